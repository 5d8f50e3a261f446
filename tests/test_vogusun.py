"""Vogusun through the framework against the plain implementation (plain_vogusun.py): configuration and names, cache groups, each
mechanism alone (the plain functions' own properties, the kernels by themselves, models of one kind of layer), and the engine's step
function under every way of cutting the work.  The ``gpu`` tests run the kernels; the others need no device."""
from __future__ import annotations

import json
import math

import numpy as np
import pytest
import torch

import plain_vogusun
import trace_tools
from kernel_steps import pieces_of, scrambled_table, step_of
from tinyllama_inference_engine_b200 import EngineConfig
from tinyllama_inference_engine_b200.cache import CacheManager
from tinyllama_inference_engine_b200.config import architecture_for, load_model_config
from tinyllama_inference_engine_b200.engine.batch import StepEntry
from tinyllama_inference_engine_b200.engine.runner import ModelRunner
from tinyllama_inference_engine_b200.errors import ConfigError
from tinyllama_inference_engine_b200.models import cache_needs, expected_tensors
from tinyllama_inference_engine_b200.models.vogusun_config import VogusunConfig
from tinyllama_inference_engine_b200.weights import SafetensorsFile, write_random_model, write_safetensors


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _rot(dims, base, scaling):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def _attention(heads, kv_heads, dim, vdim, mlp, rot=None, base=10000.0, scale=None, mix=True, scaling=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "v_mix": mix,
                                                       "scale": 2.0 * dim ** -0.5 if scale is None else scale, "rot": _rot(dim if rot is None else rot, base, scaling)}}


def _attention_2(heads, kv_heads, dim, vdim, mlp, rot=None, base=10000.0, scale=None, softcap=6.0, mix=True, scaling=(4.0, 64, 8.0, 1.0)):
    layer = _attention(heads, kv_heads, dim, vdim, mlp, rot, base, scale, mix, scaling)
    return {"type": "attention_2", "mlp": mlp, "mixer": {**layer["mixer"], "softcap": softcap}}


def _gla(heads, dim, vdim, rank, mlp, tau=4.0):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}}


def _config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Vogusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that agree nowhere: head widths that the tensor-core kernels take and that they do not, rotations of the whole vector, of a part and of
# nothing, stretched ones whose blend starts at the first pair, ends at the last or has no width, one head, heads that share key/value heads and
# that do not, key and value widths equal and not, each kind of attention as the first that mixes values, layers that do not mix among those that do,
# bounds that bite and that hardly do, decays of every rank and temper, layers with a dense feed-forward, with experts (one per token, all of
# them) and with none.
CONFIGS = {
    "all": (_config(64, 97, [_attention(4, 2, 16, 32, _dense(48), rot=8), _gla(3, 16, 32, 8, _moe(8, 3, 24), tau=16.0), _attention_2(2, 2, 48, 32, _dense(56), rot=32),
                             _attention(8, 4, 32, 16, None, base=500.0), _attention_2(3, 3, 32, 16, _moe(6, 2, 40, limit=0.4), softcap=30.0, mix=False, scaling=(2.0, 1000, 32.0, 0.5), base=200.0),
                             _gla(2, 40, 24, 20, _dense(32), tau=1.0), _attention(3, 1, 16, 64, _dense(24), mix=False)]), 3),
    "gla_first": (_config(48, 61, [_gla(1, 64, 16, 4, _moe(4, 1, 32)), _attention_2(6, 1, 32, 48, _moe(5, 5, 16, limit=3.0), scaling=(16.0, 32, 4.0, 4.0)), _gla(4, 8, 48, 1, None, tau=30.0),
                                   _attention(4, 3 + 1, 16, 12, _dense(40), rot=0)], eps=1e-3), 5),
    "attention_first": (_config(40, 53, [_attention(5, 1, 80, 16, _moe(9, 4, 8), rot=20, mix=False), _attention(2, 1, 64, 64, _dense(24), base=50.0), _attention_2(1, 1, 16, 64, None, rot=0, scaling=None, softcap=2.0),
                                         _attention(4, 4, 16, 16, _moe(12, 2, 16))], eps=1e-6), 9),
    # nothing a multiple of 8: the width, the vocabulary, the feed-forwards, the heads' widths, the ranks
    "odd": (_config(44, 37, [_attention(3, 1, 12, 10, _dense(50), rot=6), _gla(3, 10, 7, 5, _moe(6, 2, 10)), _attention_2(2, 2, 10, 5, _dense(30), scaling=(3.0, 50, 5.0, 1.0)),
                             _gla(1, 33, 20, 13, _dense(18), tau=2.5), _attention(4, 2, 6, 5, _moe(3, 1, 14), rot=2)]), 8),
}
LENGTHS = {"all": [1, 9, 70, 150, 33, 64, 17], "gla_first": [3, 40, 100, 64, 7], "attention_first": [2, 130, 65, 16, 150], "odd": [70, 3, 33, 18]}
TOLERANCE = {"float32": 3e-5, "bfloat16": 2.5e-2}     # 32-bit: of a row's largest difference; bfloat16: of its root mean square over the vocabulary
RMS = {"float32": False, "bfloat16": True}
# bfloat16 rounds what the routers read, and of some hundred tokens a few then choose another expert than the plain implementation does: such a
# row differs by many times the rounding.  32-bit rows are all held to their bound; in bfloat16 a share of the rows of a model with
# experts may lie beyond it while the median row lies within a third of it (trace_tools.run_and_compare).
LOOSE_ROWS = {"float32": 0.0, "bfloat16": 0.15}


def load_plain(folder, dtype=torch.float32):
    config = json.loads((folder / "config.json").read_text())
    file = SafetensorsFile(folder / "model.safetensors")
    tensors = {name: file.tensor(name).clone().to(dtype) for name in file.names()}
    file.close()
    return config, tensors


def _logits(config, tensors, tokens):
    return plain_vogusun.forward(config, tensors, tokens)[0]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("vogusun")
    return {key: write_random_model(base / key, config, seed) for key, (config, seed) in CONFIGS.items()}


@pytest.fixture(scope="module")
def cases(folders):
    out = {}
    for key, folder in folders.items():
        config, tensors = load_plain(folder)
        requests = trace_tools.make_requests(config["vocab"], LENGTHS[key], seed=21)
        full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
        out[key] = (folder, requests, full, max(float(v.abs().max()) for v in full.values()))
    return out


def _runner(folder, dtype, max_tokens=1024, page_size=16, requests=4):
    return ModelRunner(folder, EngineConfig(dtype=dtype, page_size=page_size, max_cache_tokens=max_tokens, max_requests=requests, max_batch_tokens=1024,
                                            device="cuda:0", poison_freed_pages=True, use_cuda_graphs=False))


def _schedules(requests, seed=3, page_size=16):
    mixed, peak = trace_tools.mixed(requests, seed=seed, page_size=page_size)
    return {"whole": (trace_tools.whole(requests), 1024), "decode": (trace_tools.tail_decode(requests), 1024), "portions": (trace_tools.portions(requests), 1024),
            "mixed": (mixed, peak)}   # a pool of exactly the peak: pages and slots are used again


# --- configuration, registry, names, cache groups -----------------------------------------------------------------------------------
def test_configuration_round_trip_registry_and_names(folders):
    architecture, config = load_model_config(folders["all"])
    assert architecture.name == "Vogusun" and isinstance(config, VogusunConfig)
    assert VogusunConfig.from_dict(config.to_dict()) == config
    assert config.layers[3]["mlp"] is None and config.layers[2]["mixer"]["rot"]["scaling"] == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    assert "scaling" not in config.layers[0]["mixer"]["rot"] and config.layers[4]["mixer"]["v_mix"] is False
    spec = architecture.build_spec(config)
    names = {t.name: tuple(t.shape) for t in expected_tensors(spec)}
    assert names["embed"] == (97, 64) and names["head"] == (97, 64) and names["final.norm"] == names["final.norm.b"] == (64,) and names["final.norm.alpha"] == ()
    assert names["l0.norm1"] == names["l0.norm1.b"] == (64,) and names["l0.norm1.alpha"] == () and "l0.norm2" not in names
    assert names["l0.mix.q"] == (64, 64) and names["l0.mix.k"] == (32, 64) and names["l0.mix.v"] == (64, 64) and names["l0.mix.g"] == (4, 64) and names["l0.mix.o"] == (64, 128)
    assert names["l0.mix.q.norm"] == names["l0.mix.k.norm"] == (16,) and names["l0.mix.vmix"] == () and "l0.mix.q.b" not in names
    assert names["l0.mlp.gate"] == names["l0.mlp.up"] == (48, 64) and names["l0.mlp.down"] == (64, 48) and "l3.mlp.gate" not in names
    assert names["l1.mix.q"] == names["l1.mix.k"] == (48, 64) and names["l1.mix.v"] == names["l1.mix.g"] == (96, 64) and names["l1.mix.norm"] == (32,)
    assert names["l1.mix.a1"] == (8, 64) and names["l1.mix.a2"] == (48, 8) and names["l1.mix.a2.b"] == (48,) and "l1.mix.vmix" not in names
    assert names["l1.mlp.e7.gate"] == (24, 64) and names["l1.mlp.e0.down"] == (64, 24) and names["l1.mlp.router"] == (8, 64) and names["l1.mlp.router.b"] == (8,)
    assert names["l2.mix.q.b"] == (96,) and names["l2.mix.v.b"] == (64,) and "l2.mix.g" not in names and "l2.mix.q.norm" not in names and "l2.mix.o.b" not in names
    assert "l4.mix.vmix" not in names
    mixes = [layer.block["mixer"].get("value_mix") for layer in spec.layers]
    assert mixes == ["first", None, "draw", "draw", None, None, None]
    assert [(e.layer, e.cache) for e in spec.order] == [(i, i) for i in range(7)]


def test_decay_rank_from_the_tensors_shape(folders, tmp_path):
    """A config.json that does not name the rank of the decays is completed from the weight file's header."""
    data = json.loads((folders["gla_first"] / "config.json").read_text())
    for layer in data["layers"]:
        layer["mixer"].pop("decay_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(data))
    (tmp_path / "model.safetensors").write_bytes((folders["gla_first"] / "model.safetensors").read_bytes())
    assert load_model_config(tmp_path)[1] == load_model_config(folders["gla_first"])[1]
    architecture = architecture_for(data)
    with pytest.raises(ConfigError, match="rank"):
        architecture.build_spec(architecture.config_class.from_dict(data))


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="lstm"), "type"),
    (lambda c: c["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "kind"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"].pop("softcap"), "softcap"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "mix values"),
    (lambda c: c["layers"][1]["mixer"].update(dim=300), "dim"),
    (lambda c: c["layers"][1]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "experts"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_refuses_what_the_design_lacks(change, message):
    data = json.loads(json.dumps(CONFIGS["all"][0]))
    change(data)
    with pytest.raises(ConfigError, match=message):
        VogusunConfig.from_dict(data)


def test_cache_groups():
    """Attention layers keep keys and values in pages, recurrent ones a state; equal needs share a group."""
    architecture = architecture_for(CONFIGS["all"][0])
    needs = cache_needs(architecture.build_spec(architecture.config_class.from_dict(CONFIGS["all"][0])))
    manager = CacheManager(needs, page_size=16, num_pages=40, max_requests=2, max_positions=4096)
    groups = sorted(g.need.page_planes() for g in manager.page_groups)
    assert groups == [((1, 16), (1, 64)), ((2, 16), (2, 32)), ((2, 48), (2, 32)), ((3, 32), (3, 16)), ((4, 32), (4, 16))]
    assert needs[1].kind == needs[5].kind == "state"


# --- the plain implementation's own mechanisms ----------------------------------------------------------------------------------------
def test_plain_curve_and_gates():
    x = torch.linspace(-40, 40, 11, dtype=torch.float64)
    y = plain_vogusun.dynamic_tanh(x, torch.full((11,), 2.0).double(), torch.full((11,), 0.5).double(), torch.tensor(0.3).double())
    assert float(y[5]) == 0.5 and float(y[-1]) == pytest.approx(2.5) and float(y[0]) == pytest.approx(-1.5)
    z = torch.randn(50, dtype=torch.float64)
    assert torch.allclose(plain_vogusun.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    one = {"m.gate": torch.eye(1), "m.up": torch.full((1, 1), -1.0), "m.down": torch.eye(1)}
    at = lambda v: float(plain_vogusun.clamped_expert(torch.tensor([[float(v)]]), one, "m", 1.5))
    assert at(9.0) == pytest.approx(1.5 / (1 + math.exp(-1.702 * 1.5)) * (-1.5 + 1.0))     # both halves at their bounds
    assert at(-9.0) == pytest.approx(-9.0 / (1 + math.exp(1.702 * 9.0)) * (1.5 + 1.0))     # the gate has no lower bound


def test_plain_one_more_in_the_denominator():
    """The weights of a row sum to less than one, by what a key of score 0 without a value would have taken."""
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(6, 2, 4, generator=g, dtype=torch.float64), torch.randn(6, 1, 4, generator=g, dtype=torch.float64)
    positions = torch.arange(6)
    ones = torch.ones(6, 1, 1, dtype=torch.float64)
    total = plain_vogusun.one_more_softmax_heads(q, k, ones, 0.5, positions)[:, :, 0]
    for i in range(6):
        score = (q[i] @ k[: i + 1, 0].T) * 0.5
        assert torch.allclose(total[i], torch.exp(score).sum(-1) / (1.0 + torch.exp(score).sum(-1)))
    assert torch.allclose(plain_vogusun.one_more_softmax_heads(q * 0, k, ones, 0.5, positions)[3, 0], torch.tensor([4.0 / 5.0]).double())
    loud = plain_vogusun.one_more_softmax_heads(q * 1e4, k * 1e2, ones, 1.0, positions)
    assert torch.isfinite(loud).all()


def test_plain_bounded_scores_and_mixed_values():
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(5, 1, d, generator=g, dtype=torch.float64) for d in (4, 4, 3))
    positions = torch.arange(5)
    loud = plain_vogusun.capped_softmax_heads(q * 1e6, k, v, 1.0, 2.0, positions)
    sign = torch.sign(q[4, 0] @ k[:, 0].T) * 2.0      # far beyond the bound only the sign is left
    assert torch.allclose(loud[4, 0], torch.softmax(sign, dim=0) @ v[:, 0])
    first = torch.randn(5, 1, 3, generator=g, dtype=torch.float64)
    assert torch.equal(plain_vogusun.mixed_values(v, None, 0.3), v) and torch.allclose(plain_vogusun.mixed_values(v, first, 0.25), 0.75 * v + 0.25 * first)


def test_plain_recurrence_is_attention_with_decayed_products():
    g = torch.Generator().manual_seed(4)
    q, k, v = (torch.randn(7, 2, d, generator=g, dtype=torch.float64) for d in (3, 3, 4))
    decay = torch.rand(7, 2, 3, generator=g, dtype=torch.float64)
    out = plain_vogusun.gated_linear_recurrence(q, k, v, decay)
    for t in (0, 3, 6):
        want = torch.zeros(2, 4, dtype=torch.float64)
        for s in range(t + 1):
            faded = decay[s + 1 : t + 1].prod(dim=0) if s < t else torch.ones(2, 3).double()     # the token's own write does not fade
            want += ((q[t] * faded * k[s]).sum(-1, keepdim=True)) * v[s]
        assert torch.allclose(out[t], want)


def test_plain_router_weighs_the_chosen_logits_alone():
    tensors = {"m.router": torch.eye(5, 8), "m.router.b": torch.tensor([0.0, 0.0, 5.0, 0.0, 0.0])}     # z = the token's first five numbers, one of them raised
    h = torch.tensor([[4.0, -9.0, -0.5, 3.8, 3.9, 3.5, 0.0, 0.0]])
    chosen, weights = plain_vogusun.route(h, tensors, "m", {"experts": 5, "top": 3})
    assert chosen == [[2, 0, 4]] and np.allclose(weights[0], torch.softmax(torch.tensor([4.5, 4.0, 3.9]), dim=0).tolist())


# --- kernels by themselves ------------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("width", [44, 45, 256, 1000])
def test_curve_and_what_joins_the_stream(dtype, atol, width):
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(width)
    stream = torch.randn(9, width, generator=g) * 3.0
    a, b = ((torch.randn(9, width, generator=g)).to(dtype) for _ in range(2))
    weight, bias = torch.randn(width, generator=g), torch.randn(width, generator=g)
    for first, second in ((a, b), (a, None), (None, None)):
        want_stream = stream.double() + sum(t.double() for t in (first, second) if t is not None)
        want = plain_vogusun.dynamic_tanh(want_stream, weight.double(), bias.double(), 0.7)
        residual, out = stream.cuda(), torch.zeros(9, width, dtype=dtype, device="cuda")
        on_device = [None if t is None else t.cuda() for t in (first, second)]
        ops.dynamic_tanh(residual, *on_device, None, weight.cuda(), bias.cuda(), 0.7, out)
        assert torch.allclose(residual.cpu().double(), want_stream, atol=2e-6)
        assert float((out.cpu().double() - want).abs().max()) <= atol * float(want.abs().max())
        only = stream.cuda()
        ops.dynamic_tanh(only, *on_device, None, weight.cuda(), bias.cuda(), 0.7, None)
        assert torch.equal(only, residual)
    rows = torch.tensor([7, 2, 2], dtype=torch.int32).cuda()
    some = torch.zeros(3, width, dtype=dtype, device="cuda")
    ops.dynamic_tanh(residual, None, None, rows, weight.cuda(), bias.cuda(), 0.7, some)
    assert torch.equal(some.cpu(), out.cpu()[[7, 2, 2]])


@pytest.mark.gpu
@pytest.mark.parametrize("rows,n,k", [(1, 72, 64), (7, 64, 520), (16, 200, 128), (3, 4096, 64)])
def test_a_completing_product_finishes_the_next_norm(rows, n, k):
    """The product adds into the stream and leaves the curve of the finished stream beside it, one kernel."""
    from types import SimpleNamespace

    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(rows)
    x, weight = torch.randn(rows, k, generator=g).bfloat16(), (torch.randn(n, k, generator=g) * k ** -0.5).bfloat16()
    stream, scale, shift = torch.randn(rows, n, generator=g) * 2.0, torch.randn(n, generator=g), torch.randn(n, generator=g)
    residual, buffer = stream.cuda(), torch.zeros(rows, n, dtype=torch.bfloat16, device="cuda")
    handle = ops.FinishedNorm(SimpleNamespace(), residual, (0.6, scale.cuda(), shift.cuda()), buffer)
    before = ops.launch_count
    ops.linear_accumulate(x.cuda(), weight.cuda(), residual, handle)
    assert ops.launch_count - before == 1 and handle.finished is buffer
    want = stream.double() + x.double() @ weight.double().T
    assert torch.allclose(residual.cpu().double(), want, atol=1e-4)
    assert torch.allclose(buffer.cpu().double(), plain_vogusun.dynamic_tanh(residual.cpu().double(), scale.double(), shift.double(), 0.6), atol=2e-2, rtol=8e-3)


def _heads_of(kind, q, k, v, sizes, positions):
    if kind == "one_more":
        return plain_vogusun.one_more_softmax_heads(q, k, v, sizes["scale"], positions)
    return plain_vogusun.capped_softmax_heads(q, k, v, sizes["scale"], sizes["softcap"], positions)


ROTARY_SHAPES = [(4, 2, 16, 32, 8, 1.0), (2, 1, 32, 16, 32, 1.2), (3, 3, 16, 16, 0, 1.0), (6, 1, 64, 64, 20, 1.0), (1, 1, 40, 24, 10, 1.3), (5, 5, 10, 6, 4, 1.0),
                 (8, 2, 128, 128, 64, 1.0), (20, 1, 16, 16, 16, 1.0), (4, 2, 80, 32, 80, 1.0), (4, 4, 64, 64, 64, 1.0)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,amplitude", ROTARY_SHAPES)
@pytest.mark.parametrize("kind,with_batch,long_tail,page_size", [("one_more", False, False, 16), ("one_more", True, False, 16), ("one_more", True, True, 64),
                                                                 ("capped", False, False, 16), ("capped", True, False, 16), ("capped", True, True, 64)])
def test_rotary_attention_kernels(dtype, atol, heads, kv, dim, vdim, rot, amplitude, kind, with_batch, long_tail, page_size):
    """Norm or biases, rotation, the values drawn towards an earlier layer's, cache write and either softmax against the plain functions: every request
    in three steps, so that the later ones read what the first cached through a scrambled block table.  With the step's context the
    kernels are chosen as the engine chooses them (tensor cores for portions, a row's keys dealt to several CTAs for steps of few
    rows); without it the general kernel runs alone.  Low scores, so that the one in the denominator weighs."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    lens, firsts = ([37, 1, 18], [30, 52, 0]) if not long_tail else ([5, 200, 9], [330, 0, 61])
    g = torch.Generator().manual_seed(heads * 100 + dim)
    table, count = scrambled_table([f + n for n, f in zip(lens, firsts)], page_size, g)
    columns = heads * dim + kv * dim + kv * vdim + heads
    columns += -columns % 8
    rows = [torch.randn(f + n, columns, generator=g).to(dtype) for n, f in zip(lens, firsts)]
    earlier = [torch.randn(f + n, kv * vdim, generator=g).to(dtype) for n, f in zip(lens, firsts)]
    planes = tuple(torch.full((count, kv, page_size, w), float("nan")).to(dtype).cuda() for w in (dim, vdim))
    cache = LayerCache(CacheNeed("pages"), True, None, table.cuda(), page_size, None, planes)
    biases = tuple(torch.randn(n, generator=g) * 0.5 for n in (heads * dim, kv * dim, kv * vdim))
    q_weight, k_weight = 1 + 0.2 * torch.randn(dim, generator=g), 1 + 0.2 * torch.randn(dim, generator=g)
    sizes, share, eps = {"scale": (2.0 if kind == "capped" else 0.7) * dim ** -0.5, "softcap": 3.0}, 0.3, 1e-5
    freq = plain_vogusun.frequencies(rot, 300.0)[0] if rot else []
    inv_freq = torch.tensor(freq, dtype=torch.float32).cuda()
    k_offset, v_offset, gate_offset = heads * dim, (heads + kv) * dim, (heads + kv) * dim + kv * vdim
    interleaved, gated = kind == "one_more", kind == "one_more"
    want = []
    for r, e in zip(rows, earlier):
        x, total = r.double(), r.shape[0]
        positions = torch.arange(total)
        q, k, v = x[:, :k_offset], x[:, k_offset:v_offset], x[:, v_offset:gate_offset]
        if kind == "capped":
            q, k, v = q + biases[0].double(), k + biases[1].double(), v + biases[2].double()
        q, k = q.view(total, heads, dim), k.view(total, kv, dim)
        if kind == "one_more":
            q, k = plain_vogusun.rms(q, eps) * q_weight.double(), plain_vogusun.rms(k, eps) * k_weight.double()
        q, k = (plain_vogusun.turn(t, positions, freq, amplitude, interleaved) for t in (q, k))
        v = plain_vogusun.mixed_values(v, e.double(), share).view(total, kv, vdim)
        o = _heads_of(kind, q, k, v, sizes, positions)
        want.append((o * torch.sigmoid(x[:, gate_offset : gate_offset + heads])[:, :, None] if gated else o).reshape(total, heads * vdim))
    got = [torch.zeros_like(w) for w in want]
    given = ([None] * 3 + [q_weight.cuda(), k_weight.cuda()]) if kind == "one_more" else ([b.cuda() for b in biases] + [None, None])
    factors, sinks = torch.full((heads,), sizes["scale"]).cuda(), torch.zeros(heads).cuda() if kind == "one_more" else None
    for pieces in pieces_of(lens, firsts):
        step_rows, positions, token_seq, sub, batch, index = step_of(rows, cache, pieces)
        first_values = torch.stack([earlier[r][p] for r, p in index]).cuda().contiguous()
        ops.norm_rotary_store(step_rows, k_offset, v_offset, given[:3], given[3], given[4], eps, factors, inv_freq, rot, interleaved, amplitude, positions, token_seq, sub,
                              heads, kv, dim, vdim, first_values=first_values, value_share=share)
        out = torch.zeros(len(index), heads * vdim, dtype=dtype, device="cuda")
        ops.mixed_heads_attention(step_rows, gate_offset if gated else -1, positions, token_seq, sub, None, None, out, heads, kv, dim, vdim, 0, 1.0,
                                  batch=batch if with_batch else None, gate_per_head=True, softcap=sizes["softcap"] if kind == "capped" else 0.0, sinks=sinks)
        for (r, p), row in zip(index, out.cpu().double()):
            got[r][p] = row
    for r in range(len(rows)):
        assert float((got[r] - want[r]).abs().max()) <= atol * max(1.0, float(want[r].abs().max())), r


@pytest.mark.gpu
def test_kept_values_are_the_layers_own():
    """The layer that keeps its values leaves them with their bias and caches the same; nothing is drawn towards anything there."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    g = torch.Generator().manual_seed(5)
    heads, kv, dim, vdim, tokens = 2, 2, 16, 24, 9
    rows = torch.randn(tokens, (heads + kv) * dim + kv * vdim, generator=g).cuda()
    planes = tuple(torch.zeros(2, kv, 16, w, device="cuda") for w in (dim, vdim))
    cache = LayerCache(CacheNeed("pages"), True, None, torch.tensor([[1]], dtype=torch.int32).cuda(), 16, None, planes)
    bias, kept = torch.randn(kv * vdim, generator=g).cuda(), torch.zeros(tokens, kv * vdim, device="cuda")
    positions, seq = torch.arange(tokens, dtype=torch.int32).cuda(), torch.zeros(tokens, dtype=torch.int32).cuda()
    ops.norm_rotary_store(rows, heads * dim, (heads + kv) * dim, (None, None, bias), None, None, 0.0, None, None, 0, True, 1.0, positions, seq, cache, heads, kv, dim, vdim,
                          first_values=kept)
    want = rows[:, (heads + kv) * dim :] + bias
    assert torch.equal(kept, want) and torch.equal(planes[1][1, :, :tokens].permute(1, 0, 2).reshape(tokens, -1), want)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["one_more", "capped", "capped_sink", "capped_loosely", "capped_high"])
@pytest.mark.parametrize("dim,vdim,heads,kv,page_size", [(64, 64, 4, 2, 64), (128, 128, 8, 2, 64), (128, 128, 3, 3, 128), (64, 64, 16, 1, 64), (192, 128, 2, 1, 64), (96, 32, 4, 2, 64), (40, 24, 3, 3, 64),
                                                         (80, 80, 4, 2, 128), (64, 128, 4, 1, 64)])
def test_rotary_attention_in_tensor_memory(dim, vdim, heads, kv, page_size, kind, monkeypatch):
    """Prompt portions run on the tcgen05 kernel (in one tensor of equal planes of 64 or 128, or in planes of any widths), decoding requests at the step's
    head on the kernel of few rows; bounds that hold scores back a lot, hardly, and so high that a maximum is taken off:
    portions from position 0 and behind cached keys, page borders, a portion of 129 rows, keys that stand out, rows all of whose scores are
    low (the one in the denominator takes most of their weight) and rows whose maximum grows from tile to tile."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.engine.batch import pack_step
    from tinyllama_inference_engine_b200.ops import fast
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    g = torch.Generator().manual_seed(dim + heads)
    lens, firsts = [1, 1, 300, 129, 200], [70, 200, 0, 130, 1]
    totals = [f + n for n, f in zip(lens, firsts)]
    table, count = scrambled_table(totals, page_size, g)
    columns = (heads + kv) * dim + kv * vdim + heads
    columns += -columns % 8
    gate_at, k_at, v_at = (heads + kv) * dim + kv * vdim, heads * dim, (heads + kv) * dim
    rows = [torch.randn(t, columns, generator=g) for t in totals]
    for r in rows:
        r[-1, :dim] = r[5, k_at : k_at + dim] * 2.0                               # a key that stands out
        r[7::9, : heads * dim] = -3.0 * torch.ones(dim).repeat(heads)             # queries against ...
        r[:, k_at:v_at] += 0.15                                                   # ... keys that lean the other way: every score of such a row is low
        r[8::9, : heads * dim] = 0.2
        r[:, k_at : k_at + dim] *= torch.linspace(0.5, 2.0, r.shape[0])[:, None]  # later keys are longer
    rows = [r.bfloat16() for r in rows]
    pages = torch.full((count, 2, kv, page_size, dim), float("nan")).bfloat16().cuda() if dim == vdim else None
    planes = () if dim == vdim else tuple(torch.full((count, kv, page_size, w), float("nan")).bfloat16().cuda() for w in (dim, vdim))
    scale, softcap = 1.5 * dim ** -0.5, {"one_more": 0.0, "capped": 4.0, "capped_sink": 4.0, "capped_loosely": 25.0, "capped_high": 90.0}[kind]
    sinks = {"one_more": torch.zeros(heads), "capped_sink": torch.linspace(-6.0, 3.0, heads)}.get(kind)
    want = []
    for r in rows:
        x, total = r.double(), r.shape[0]
        q = (x[:, :k_at].view(total, heads, dim) * scale).bfloat16().double()
        k, v = x[:, k_at:v_at].view(total, kv, dim).repeat_interleave(heads // kv, 1), x[:, v_at:gate_at].view(total, kv, vdim).repeat_interleave(heads // kv, 1)
        score = torch.einsum("ihd,jhd->hij", q, k)
        if softcap:
            score = softcap * torch.tanh(score / softcap)
        score = score.masked_fill(torch.arange(total)[:, None] < torch.arange(total)[None, :], float("-inf"))
        extra = torch.full((heads, total, 1), float("-inf"), dtype=torch.float64) if sinks is None else sinks.double()[:, None, None].expand(heads, total, 1)
        p = torch.softmax(torch.cat([score, extra], dim=-1), dim=-1)[..., :total]
        o = torch.einsum("hij,jhd->ihd", p, v)
        want.append((o * torch.sigmoid(x[:, gate_at : gate_at + heads])[:, :, None]).reshape(total, heads * vdim))
    calls = []
    name = "prefill_attention_tc" if dim == vdim and dim in (64, 128) else "prefill_attention_tc_planes"
    kernel = getattr(fast, name)
    monkeypatch.setattr(fast, name, lambda *a, **k: (calls.append(1), kernel(*a, **k)))
    factors, nothing, on_device = torch.full((heads,), scale).cuda(), torch.zeros(0, device="cuda"), None if sinks is None else sinks.cuda()
    for pieces in ([(r, 0, f) for r, f in enumerate(firsts) if f > 0], [(r, f, n) for r, (n, f) in enumerate(zip(lens, firsts))]):
        ctx = pack_step([StepEntry(r, [0] * n, []) for r, _, n in pieces], [a for _, a, _ in pieces], list(range(len(pieces))), [[table[r].tolist() for r, _, _ in pieces]],
                        torch.device("cuda:0"))
        cache = LayerCache(CacheNeed("pages"), True, pages, ctx.block_tables[0], page_size, None, planes)
        index = [(r, a + i) for r, a, n in pieces for i in range(n)]
        step_rows = torch.stack([rows[r][p] for r, p in index]).cuda().contiguous()
        ops.norm_rotary_store(step_rows, k_at, v_at, None, None, None, 1e-5, factors, nothing, 0, True, 1.0, ctx.positions, ctx.token_seq, cache, heads, kv, dim, vdim)
        out = torch.full((len(index), heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
        ops.mixed_heads_attention(step_rows, gate_at, ctx.positions, ctx.token_seq, cache, None, None, out, heads, kv, dim, vdim, 0, 1.0, batch=ctx, gate_per_head=True,
                                  softcap=softcap, sinks=on_device)
        assert int(fast.tcgen05_error_flag(out.device)) == 0, "a bounded wait inside the kernel gave up"
        for (r, p), row in zip(index, out.cpu().double()):
            rms_of = lambda v: float((v * v).mean().sqrt())
            assert rms_of(row - want[r][p]) <= 1.2e-2 * max(0.3, rms_of(want[r][p])), (r, p)
    assert len(calls) == (2 if dim % 16 == 0 else 1)     # the kernels of few rows take multiples of 16: without one the second step is the general kernel's


@pytest.mark.gpu
@pytest.mark.parametrize("capped", [False, True])
@pytest.mark.parametrize("dim,vdim,heads,kv", [(64, 64, 8, 2), (192, 128, 16, 1), (96, 48, 4, 4), (256, 16, 6, 3), (16, 128, 10, 1)])
def test_single_rows_over_parts_of_their_keys(dim, vdim, heads, kv, capped):
    """Rows of unequal requests (a first token, a page's last and the next one's first, two rows of one request, 1,500 keys cut into parts), with a gate per
    head, per element and none; the same rows alone give what they give together."""
    from tinyllama_inference_engine_b200.ops import fast

    g = torch.Generator().manual_seed(dim + vdim)
    totals, page_size = [1, 64, 65, 300, 300, 1500], 64
    of_request = [0, 1, 2, 3, 3, 4]
    positions = [0, 63, 64, 298, 299, 1499]
    table, count = scrambled_table([1, 64, 65, 300, 1500], page_size, g)
    keys, values = (torch.randn(count, kv, page_size, w, generator=g).bfloat16() for w in (dim, vdim))
    columns = heads * dim + heads * vdim
    rows = torch.randn(len(positions), columns, generator=g).bfloat16()
    sinks, scale, softcap = torch.linspace(-2.0, 3.0, heads), 1.5 * dim ** -0.5, 5.0 if capped else 0.0
    want = torch.zeros(len(positions), heads, vdim, dtype=torch.float64)
    for i, (r, p) in enumerate(zip(of_request, positions)):
        where = [(int(table[r, j // page_size]), j % page_size) for j in range(p + 1)]
        k, v = (torch.stack([t[a, :, b] for a, b in where]).double().repeat_interleave(heads // kv, 1) for t in (keys, values))
        score = torch.einsum("hd,jhd->hj", rows[i, : heads * dim].view(heads, dim).double(), k) * scale
        if capped:
            score = softcap * torch.tanh(score / softcap)
        want[i] = torch.einsum("hj,jhd->hd", torch.softmax(torch.cat([score, sinks.double()[:, None]], dim=1), dim=1)[:, : p + 1], v)
    on_device = [t.cuda() for t in (rows, torch.tensor(positions, dtype=torch.int32), torch.tensor(of_request, dtype=torch.int32), table, keys, values, sinks)]
    x, pos, seq, blocks, k, v, s = on_device
    from ctypes import c_void_p

    planes = (c_void_p(k.data_ptr()), kv * page_size * dim, c_void_p(v.data_ptr()), kv * page_size * vdim)
    for gate, per_head in ((-1, True), (heads * dim, True), (heads * dim, False)):
        z = torch.sigmoid(rows[:, heads * dim :].double())
        factor = 1.0 if gate < 0 else (z[:, :heads, None] if per_head else z.view(-1, heads, vdim))
        out = torch.full((len(positions), heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
        for _ in range(2):   # the counters of the parts are left as they were found
            fast.heads_decode(x, gate, per_head, pos, seq, blocks, planes, out, heads, kv, dim, vdim, page_size, scale, softcap, s, 1500)
            assert float((out.cpu().double().view(-1, heads, vdim) - want * factor).abs().max()) <= 2e-2 * max(1.0, float(want.abs().max()))
    one = torch.zeros(1, heads * vdim, dtype=torch.bfloat16, device="cuda")
    fast.heads_decode(x[3:4], -1, True, pos[3:4], seq[3:4], blocks, planes, one, heads, kv, dim, vdim, page_size, scale, softcap, s, 300)
    assert float((one.cpu().double().view(heads, vdim) - want[3]).abs().max()) <= 2e-2


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", [(2, 16, 32, 8, 16.0), (3, 10, 7, 5, 1.0), (1, 200, 40, 16, 4.0), (4, 64, 64, 1, 30.0), (1, 33, 130, 24, 0.5)])
def test_gated_linear_attention_kernels(dtype, atol, heads, dim, vdim, rank, tau):
    """Preparation (with the low-rank pair's second half inside, and with its product given), recurrence and the gated norm against the plain functions,
    two requests in portions whose state is carried in slots that are not the entries' own numbers."""
    from types import SimpleNamespace

    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(dim)
    lens = [61, 23]
    qk, values = heads * dim, heads * vdim
    first_at = 2 * qk + 2 * values
    rows = [torch.randn(n, first_at + rank, generator=g).to(dtype) for n in lens]
    a2, bias, weight = (torch.randn(qk, rank, generator=g) * rank ** -0.5).to(dtype), torch.randn(qk, generator=g) + 1.0, 1 + 0.2 * torch.randn(vdim, generator=g)
    want = []
    for r in rows:
        x, n = r.double(), r.shape[0]
        decay = torch.sigmoid(x[:, first_at:] @ a2.double().T + bias.double()) ** (1.0 / tau)
        o = plain_vogusun.gated_linear_recurrence(x[:, :qk].view(n, heads, dim) * dim ** -0.5, x[:, qk : 2 * qk].view(n, heads, dim), x[:, 2 * qk : 2 * qk + values].view(n, heads, vdim),
                                                  decay.view(n, heads, dim))
        gate = x[:, 2 * qk + values : first_at]
        want.append((plain_vogusun.rms(o, 1e-5) * weight.double()).reshape(n, values) * gate * torch.sigmoid(gate))
    for inside in (True, False):
        state = torch.zeros(5, ops.delta_state_words(heads, dim, vdim, 0, 1)[0], device="cuda")
        slots, got, at = [3, 1], [[], []], [0, 0]
        for counts in ((20, 2), (1, 0), (1, 1), (39, 20)):
            entries = [r for r in (0, 1) if counts[r]]
            step = torch.cat([rows[r][at[r] : at[r] + counts[r]] for r in entries]).cuda().contiguous()
            starts = torch.tensor(np.concatenate([[0], np.cumsum([counts[r] for r in entries])]), dtype=torch.int32).cuda()
            ctx = SimpleNamespace(seq_starts=starts, state_slots=torch.tensor([slots[r] for r in entries], dtype=torch.int32).cuda(), num_seqs=len(entries))
            tokens = step.shape[0]
            prep = torch.zeros(tokens, 3 * qk + values + heads, device="cuda")
            decay_in = step[:, first_at:]
            if inside:
                ops.gla_prepare(step, decay_in, a2.cuda(), bias.cuda(), tau, dim ** -0.5, prep, heads, dim, vdim)
            else:
                product = torch.zeros(tokens, qk, dtype=dtype, device="cuda")
                ops.linear(decay_in, a2.cuda(), product)
                ops.gla_prepare(step, product, None, bias.cuda(), tau, dim ** -0.5, prep, heads, dim, vdim)
            read, out = torch.zeros(tokens, values, device="cuda"), torch.zeros(tokens, values, dtype=dtype, device="cuda")
            ops.delta_rule(prep, state, ctx, read, heads, heads, dim, vdim, plain=True)
            ops.delta_gate_norm(read, step[:, 2 * qk + values : first_at], weight.cuda(), out, 1e-5, heads, vdim, gate_kind="silu")
            for index, r in enumerate(entries):
                a, b = int(starts[index]), int(starts[index + 1])
                got[r].append(out[a:b].cpu().double())
                at[r] += counts[r]
        for r in (0, 1):
            assert float((torch.cat(got[r]) - want[r]).abs().max()) <= atol * max(1.0, float(want[r].abs().max())), (inside, r)
        assert torch.equal(state[[0, 2, 4]].cpu(), torch.zeros(3, state.shape[1]))     # nobody else's slot is touched


@pytest.mark.gpu
@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 32), (1, 200, 40), (3, 33, 7), (2, 128, 64)])
@pytest.mark.parametrize("lens", [[600, 1, 128, 129, 256, 257], [30, 513], [1024]])
def test_long_entries_of_the_recurrence_in_chunks(heads, dim, vdim, lens):
    """Entries of all lengths around whole chunks beside short ones, from states that are not zero, strong and weak decays: what the chunks give is what the
    rows in order give, and so is the state they leave."""
    from types import SimpleNamespace

    from tinyllama_inference_engine_b200 import ops

    assert max(lens) >= ops.RECURRENCE_CHUNKS_MIN_ROWS
    g = torch.Generator().manual_seed(sum(lens) + dim)
    qk, values, total = heads * dim, heads * vdim, sum(lens)
    starts = np.concatenate([[0], np.cumsum(lens)])
    parts = [torch.randn(total, n, generator=g) for n in (qk, qk, values)]
    decay = torch.sigmoid(torch.randn(total, qk, generator=g) + torch.linspace(-1.0, 8.0, qk)) ** 0.25
    prep = torch.cat([*parts, torch.ones(total, heads), decay], dim=1).cuda().contiguous()
    slots = list(range(len(lens)))[::-1]
    words = ops.delta_state_words(heads, dim, vdim, 0, 1)[0]
    step = lambda a, b, order: SimpleNamespace(seq_starts=torch.tensor(np.concatenate([[0], np.cumsum([y - x for x, y in zip(a, b)])]), dtype=torch.int32).cuda(),
                                               state_slots=torch.tensor([slots[i] for i in order], dtype=torch.int32).cuda(), num_seqs=len(order), max_q_len=max(y - x for x, y in zip(a, b)))
    before, state = torch.zeros(len(lens), words, device="cuda"), None
    ops.delta_rule(prep[: len(lens)].contiguous(), before, step([0] * len(lens), [1] * len(lens), range(len(lens))), torch.zeros(len(lens), values, device="cuda"), heads, heads, dim, vdim, plain=True)
    results = {}
    for chunks in (True, False):
        kept, ops.use_recurrence_chunks = ops.use_recurrence_chunks, chunks
        try:
            state, out = before.clone(), torch.full((total, values), float("nan"), device="cuda")
            launches = ops.launch_count
            ops.delta_rule(prep, state, step(starts[:-1], starts[1:], range(len(lens))), out, heads, heads, dim, vdim, plain=True)
            assert ops.launch_count - launches == (3 if chunks else 1)
            results[chunks] = (out.cpu(), state.cpu())
        finally:
            ops.use_recurrence_chunks = kept
    for got, want in zip(*results.values()):
        assert torch.isfinite(got).all() and float((got - want).abs().max()) <= 2e-6 * float(want.abs().max())
    q, k, v, fade = (t.double() for t in (*parts, decay))
    for e, (a, b) in enumerate(zip(starts[:-1], starts[1:])):      # the row that wrote the state a request starts from comes first
        rows = [torch.cat([t[e:e + 1], t[a:b]]).view(b - a + 1, heads, -1) for t in (q, k, v, fade)]
        want = plain_vogusun.gated_linear_recurrence(*rows)[1:].reshape(b - a, values)
        assert float((results[True][0][a:b].double() - want).abs().max()) <= 2e-5 * max(1.0, float(want.abs().max())), e


@pytest.mark.gpu
@pytest.mark.parametrize("tokens", [50, 1300])    # a CTA per token; four tokens per CTA (a step of many rows), the last CTA short of rows
@pytest.mark.parametrize("experts,top,width", [(8, 3, 64), (6, 2, 44), (4, 1, 32), (64, 8, 128), (5, 5, 24), (40, 36, 48), (10, 3, 42), (7, 7, 17)])
def test_router_over_chosen_logits(tokens, experts, top, width):
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(experts * 7 + width)
    x = torch.randn(tokens, width, generator=g)
    tensors = {"m.router": torch.randn(experts, width, generator=g) * 3.0 * width ** -0.5, "m.router.b": torch.randn(experts, generator=g) * 2.0}
    chosen, weights = plain_vogusun.route(x, tensors, "m", {"experts": experts, "top": top})
    ids, got = torch.zeros(tokens, top, dtype=torch.int32, device="cuda"), torch.zeros(tokens, top, device="cuda")
    ops.moe_route(x.cuda(), tensors["m.router"].cuda(), None, ids, got, 1, 1, 1.0, scores="logits", bias=tensors["m.router.b"].cuda())
    wrong = [t for t in range(tokens) if ids[t].cpu().tolist() != chosen[t]]
    for t in wrong:      # another order of the sum may turn a choice only where two logits all but tie
        z = tensors["m.router"].double() @ x[t].double() + tensors["m.router.b"].double()
        gaps = (z[:, None] - z[None, :]).abs() + torch.eye(experts, dtype=torch.float64)
        assert float(gaps.min()) < 2e-5, t
    right = [t for t in range(tokens) if t not in wrong]
    assert len(right) >= tokens - 4
    assert torch.allclose(got.cpu()[right], torch.tensor(weights)[right], atol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("tokens,experts,top,width,ff,limit", [(5, 6, 2, 44, 10, 1.0), (16, 6, 2, 64, 100, 0.3), (70, 8, 3, 64, 24, 2.0), (300, 4, 1, 32, 16, 1.0), (130, 16, 4, 128, 48, 0.7), (1, 3, 3, 24, 8, 1.5),
                                                               (300, 4, 1, 64, 72, 1.0), (700, 6, 3, 136, 200, 0.5), (400, 3, 2, 64, 520, 1.2)])   # the last three: enough rows per expert for tcgen05
def test_clamped_expert_kernels(dtype, atol, tokens, experts, top, width, ff, limit):
    """Bounds that both halves often meet; steps of few rows read the experts' rows directly, bfloat16 prompt portions sort by expert and use the
    tensor cores.  A token's result does not depend on the step."""
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(tokens + experts)
    x = torch.randn(tokens, width, generator=g).to(dtype)
    gate, up = ((torch.randn(experts, ff, width, generator=g) * width ** -0.5).to(dtype) for _ in range(2))
    down = (torch.randn(experts, width, ff, generator=g) * ff ** -0.5).to(dtype)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32)
    ids[: tokens // 2, 0] = ids[0, 0]        # one crowded expert (a token may then name it twice; both are added)
    weights = torch.rand(tokens, top, generator=g) + 0.1
    every = torch.stack([plain_vogusun.clamped_expert(x.double(), {"m.gate": gate[e].double(), "m.up": up[e].double(), "m.down": down[e].double()}, "m", limit) for e in range(experts)], dim=1)
    want = sum(weights[:, k, None].double() * every[torch.arange(tokens), ids[:, k].long()] for k in range(top))
    stacked = torch.cat([gate, up], dim=1).contiguous().cuda()
    some = torch.arange(0, tokens, max(1, tokens // 5))
    for index in (torch.arange(tokens), some):
        got = torch.zeros(len(index), width, dtype=dtype, device="cuda")
        ops.moe_experts(x[index].cuda(), stacked, down.cuda(), ids[index].cuda(), weights[index].cuda(), None, got, "clamped_sigmoid", clamp=(limit, 1.702, 1.0))
        assert int(ops.error_flag(got.device)) == 0
        assert float((got.cpu().double() - want[index]).abs().max()) <= atol * max(1.0, float(want.abs().max()))


# --- the engine on the GPU under every way of cutting the work ---------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(CONFIGS))
def test_engine_matches_plain_under_every_schedule(cases, key, dtype):
    """Whole prompts, a tail decoded token by token, portions down to two tokens, and four live requests mixed in a pool that makes
    pages and state slots come round again (freed pages are poisoned with NaN)."""
    folder, requests, full, scale = cases[key]
    for name, (steps, pool) in _schedules(requests).items():
        runner = _runner(folder, dtype, max_tokens=pool)
        trace_tools.run_and_compare(runner, steps, full, atol=TOLERANCE[dtype] * scale, over_vocabulary=RMS[dtype], allowed_over=LOOSE_ROWS[dtype])
        runner.cache.check()
        assert not runner.cache.records, name
        if name == "mixed":
            assert all(g.pool.reuses > 0 for g in runner.cache.page_groups)


@pytest.mark.gpu
@pytest.mark.parametrize("key", ["all", "odd"])
def test_layer_outputs_match_the_plain_trace(cases, key):
    folder, requests, full, scale = cases[key]
    config, tensors = load_plain(folder)
    tokens = requests["r2"]
    want = plain_vogusun.forward(config, tensors, tokens)[1]
    trace = {}
    _runner(folder, "float32").step([StepEntry("a", tokens, [0])], trace=trace)
    assert len(trace) == len(want) == len(config["layers"])
    for index, layer in enumerate(want):
        assert float((trace[f"layer{index}.output"].cpu() - layer).abs().max()) <= 3e-5 * float(layer.abs().max()), index


# models of one kind of layer, with sizes that no other test has
ONE_KIND = {
    "attention": _config(56, 41, [_attention(6, 2, 48, 80, None, rot=24), _attention(7, 7, 16, 32, None, mix=False), _attention(5, 5, 24, 32, None)]),
    "attention_experts": _config(72, 41, [_attention(2, 2, 128, 128, _moe(16, 6, 64, limit=0.7))]),
    "attention_2": _config(56, 41, [_attention_2(5, 1, 32, 48, _dense(40), rot=12), _attention_2(4, 2, 64, 64, None, mix=False, softcap=50.0)]),
    "gla": _config(72, 41, [_gla(3, 24, 56, 12, _dense(200), tau=8.0), _gla(2, 128, 64, 32, None)]),
    "gla_experts": _config(104, 41, [_gla(5, 16, 8, 2, _moe(10, 1, 24, limit=2.0), tau=0.7)]),
}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(ONE_KIND))
def test_models_of_one_kind_of_layer(tmp_path, kind, dtype):
    folder = write_random_model(tmp_path / kind, ONE_KIND[kind], 12)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(config["vocab"], [140, 5, 66, 31], seed=8)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    for steps, pool in _schedules(requests, seed=6).values():
        trace_tools.run_and_compare(_runner(folder, dtype, max_tokens=pool), steps, full, atol=TOLERANCE[dtype] * scale, over_vocabulary=RMS[dtype], allowed_over=LOOSE_ROWS[dtype])


def _changed(folder, target, change):
    """A copy of a model folder with its tensors changed."""
    _, tensors = load_plain(folder, torch.bfloat16)
    change(tensors)
    target.mkdir()
    (target / "config.json").write_text((folder / "config.json").read_text())
    write_safetensors(target / "model.safetensors", tensors)
    return target


def _paired_tokens(tensors, heads, kv_heads, dim, fast_columns, pairs):
    """Token 100 + i becomes what token i looks for: its row is token i's with the channels in another order, and the keys' projection is the queries'
    (every head of a group has one) read through that order.  The columns that turn by a radian per token are made small."""
    g = torch.Generator().manual_seed(1)
    order = torch.randperm(tensors["embed"].shape[1], generator=g)
    tensors["embed"][100 : 100 + pairs] = tensors["embed"][:pairs][:, order]
    tensors["l0.norm1"], tensors["l0.norm1.b"] = torch.ones_like(tensors["l0.norm1"]), torch.zeros_like(tensors["l0.norm1.b"])
    tensors["l0.norm1.alpha"], tensors["final.norm.alpha"] = torch.tensor(1.0).bfloat16(), torch.tensor(0.5).bfloat16()
    queries = tensors["l0.mix.q"].view(heads, dim, -1)[:: heads // kv_heads].clone()
    queries[:, fast_columns] *= 0.2
    tensors["l0.mix.q"] = queries.repeat_interleave(heads // kv_heads, 0).reshape(heads * dim, -1)
    tensors["l0.mix.k"] = queries.reshape(kv_heads * dim, -1)[:, order].contiguous()
    for name in ("l0.mix.q.b", "l0.mix.k.b"):
        if name in tensors:
            tensors[name] = torch.zeros_like(tensors[name])


def _far_case(folder, kind):
    """A one-layer model and a request whose last tokens each look for one token hundreds of positions back."""
    make = _attention if kind == "attention" else _attention_2
    layer = make(4, 2, 32, 32, _dense(32), scale=1.0, rot=4, base=1e6, **({} if kind == "attention" else {"softcap": 40.0}))
    fast = [0, 1] if kind == "attention" else [0, 2]
    model = _changed(write_random_model(folder / "base", _config(40, 401, [layer]), 7), folder / "sharp", lambda t: _paired_tokens(t, 4, 2, 32, fast, 43))
    requests = trace_tools.make_requests(401, [400, 70, 33], seed=17)
    requests["r0"] = [t if t >= 150 else t + 150 for t in requests["r0"]]
    requests["r0"][:3] = [100, 101, 102]                # tokens of their own: the first three, and forty across page borders
    requests["r0"][10:50] = list(range(103, 143))
    requests["r0"][-43:] = [*range(3, 43), 0, 1, 2]     # what looks for them
    config, tensors = load_plain(model)
    return model, config, tensors, requests


@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_far_keys_are_what_the_last_tokens_read(tmp_path, kind):
    """What the next test relies on: changing far tokens, or the first three, moves the last rows by many times what is tolerated."""
    _, config, tensors, requests = _far_case(tmp_path, kind)
    full = _logits(config, tensors, requests["r0"])
    scale = float(full.abs().max())
    for places, last, factor in ((range(10, 50), slice(-43, -3), 2000), (range(3), slice(-3, None), 1000)):
        other = [60 + i % 7 if i in places else t for i, t in enumerate(requests["r0"])]
        assert float((_logits(config, tensors, other)[last] - full[last]).abs().max()) > factor * TOLERANCE["float32"] * scale


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_far_keys_and_first_tokens_decide(tmp_path, kind, dtype):
    """A large score scale lets single keys stand out hundreds of tokens back and across page borders: a lost key or a rotation by the wrong
    position then moves the logits far beyond the tolerance, in portions, in decoded tokens and in mixed batches."""
    folder, config, tensors, requests = _far_case(tmp_path, kind)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    for steps in (trace_tools.tail_decode(requests, tail=50), trace_tools.portions(requests), trace_tools.mixed(requests, seed=4, max_portion=90)[0]):
        trace_tools.run_and_compare(_runner(folder, dtype, max_tokens=2048), steps, full, atol=TOLERANCE[dtype] * scale * (1.0 if dtype == "float32" else 3.0), over_vocabulary=RMS[dtype])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_feel_the_one_in_the_denominator(cases, tmp_path, dtype):
    """With low scores a request's first tokens leave much of their weight to nobody: the logits without the one would differ far beyond the
    tolerance, and the engine's do not, whole and token by token from the first on."""
    folder = write_random_model(tmp_path / "low", _config(40, 53, [_attention(4, 2, 32, 32, None, scale=0.02), _attention(2, 1, 64, 64, None, scale=0.02)]), 3)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(config["vocab"], [40, 3, 1, 17], seed=3)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    kept = plain_vogusun.one_more_softmax_heads
    try:
        plain_vogusun.one_more_softmax_heads = lambda q, k, v, s, p: plain_vogusun.capped_softmax_heads(q, k, v, s, 1e9, p)
        without = _logits(config, tensors, requests["r0"])
    finally:
        plain_vogusun.one_more_softmax_heads = kept
    assert float((without - full["r0"])[:3].abs().max()) > 3 * TOLERANCE["bfloat16"] * scale
    for steps in (trace_tools.whole(requests), trace_tools.tail_decode(requests, tail=100), trace_tools.mixed(requests, seed=1)[0]):
        trace_tools.run_and_compare(_runner(folder, dtype), steps, full, atol=TOLERANCE[dtype] * scale, over_vocabulary=RMS[dtype])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_memory_of_the_recurrence(tmp_path, dtype):
    """Decays near one: what the first tokens wrote is read hundreds of tokens later, so a state lost between steps or a slot handed on dirty shows."""
    def slow(tensors):
        for name in tensors:
            if name.endswith(".a2.b"):
                tensors[name] = torch.full_like(tensors[name], 6.0)

    folder = _changed(write_random_model(tmp_path / "base", _config(40, 53, [_gla(2, 32, 24, 8, None, tau=16.0), _gla(1, 48, 16, 4, _dense(24), tau=16.0)]), 4), tmp_path / "slow", slow)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(config["vocab"], [330, 70, 33, 12, 90], seed=5)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    first = [(t + 1) % config["vocab"] if i < 3 else t for i, t in enumerate(requests["r0"])]
    assert float((_logits(config, tensors, first)[-20:] - full["r0"][-20:]).abs().max()) > 20 * TOLERANCE["float32"] * scale
    for steps in (trace_tools.tail_decode(requests, tail=40), trace_tools.portions(requests), trace_tools.mixed(requests, seed=4, max_portion=90)[0]):
        trace_tools.run_and_compare(_runner(folder, dtype, max_tokens=2048), steps, full, atol=TOLERANCE[dtype] * scale, over_vocabulary=RMS[dtype])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_other_page_sizes(cases, dtype):
    """150 tokens decoded one by one behind a prompt, with pages of 64 and of 32 tokens."""
    folder, requests, full, scale = cases["all"]
    some = {rid: requests[rid] for rid in ("r2", "r3")}
    more = dict(some, long=trace_tools.make_requests(97, [260], seed=5)["r0"])
    config, tensors = load_plain(folder)
    full = dict(full, long=_logits(config, tensors, more["long"]))
    for page_size in (64, 32):
        trace_tools.run_and_compare(_runner(folder, dtype, max_tokens=2048, page_size=page_size), trace_tools.tail_decode(more, tail=150), full,
                                    atol=TOLERANCE[dtype] * scale, over_vocabulary=RMS[dtype], allowed_over=LOOSE_ROWS[dtype])


@pytest.mark.gpu
@pytest.mark.parametrize("dim,kv", [(64, 2), (128, 1)])
def test_long_portions_beside_decoded_tokens(tmp_path, dim, kv, product_thresholds):
    """Portions of up to 200 rows beside single tokens with pages of 64: the tensor-memory kernels of both softmaxes, the kernel of few rows at the
    step's head and the ones between them, in one model; the sublayers' last products adding into the stream or not."""
    folder = write_random_model(tmp_path / "m", _config(64, 47, [_attention(4, kv, dim, dim, _dense(64)), _gla(2, 32, 32, 8, _dense(40)), _attention_2(2 * kv, kv, dim, dim, _dense(96))]), 3)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(47, [500, 230, 64, 300], seed=9)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    for steps in (trace_tools.whole(requests), trace_tools.tail_decode(requests, tail=20), trace_tools.portions(requests, sizes=(200, 65, 2, 128)),
                  trace_tools.mixed(requests, seed=2, max_portion=200)[0]):
        trace_tools.run_and_compare(_runner(folder, "bfloat16", max_tokens=2048, page_size=64), steps, full, atol=TOLERANCE["bfloat16"] * scale, over_vocabulary=True)


@pytest.mark.gpu
def test_rows_do_not_depend_on_the_batch(cases):
    """32-bit rows agree to rounding however the step is cut and whatever else is in the batch."""
    folder, requests, full, scale = cases["all"]
    alone, together = _runner(folder, "float32"), _runner(folder, "float32")
    tokens = requests["r3"]
    whole = alone.step([StepEntry("x", tokens, [len(tokens) - 1])]).cpu()
    together.step([StepEntry("y", requests["r2"][:40], []), StepEntry("x", tokens[:77], [])])
    cut = together.step([StepEntry("x", tokens[77:], [len(tokens) - 78]), StepEntry("y", requests["r2"][40:41], [0])]).cpu()
    assert float((cut[0] - whole[0]).abs().max()) <= 1e-5 * scale


# --- generation through the engine's own entry point -------------------------------------------------------------------------------------
def _plain_greedy(config, tensors, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(_logits(config, tensors, tokens)[-1].argmax()))
    return tokens[len(prompt):]


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(folders, graphs):
    """Prompts of unequal length through ``Engine.generate``: scheduler, portions under a small token budget, decode sessions (captured as
    graphs or not).  32-bit, so that the plain choice is the engine's."""
    from tinyllama_inference_engine_b200 import Engine, SamplingParams

    folder = folders["all"]
    config, tensors = load_plain(folder)
    rng = np.random.default_rng(31)
    prompts = [[int(t) for t in rng.integers(0, config["vocab"], size=n)] for n in (50, 3, 21, 34, 8)]
    engine = Engine(folder, EngineConfig(dtype="float32", page_size=16, max_cache_tokens=512, max_requests=3, max_batch_tokens=24, use_cuda_graphs=graphs))
    results = engine.generate(prompts, SamplingParams(max_tokens=16))
    for prompt, result in zip(prompts, results):
        assert result.generated_tokens == _plain_greedy(config, tensors, prompt, 16)
    again = engine.generate(prompts[:3], SamplingParams(max_tokens=16))       # pages come round again; shapes repeat, so graphs replay
    assert [r.generated_tokens for r in again] == [r.generated_tokens for r in results[:3]]
    if graphs:
        assert any(s.graph is not None for s in engine._sessions.values())
    engine.runner.cache.check()


@pytest.mark.gpu
def test_generation_in_bfloat16_and_the_command_line(folders, capsys):
    from tinyllama_inference_engine_b200 import generate
    from tinyllama_inference_engine_b200.cli import main

    rng = np.random.default_rng(2)
    prompts = [[int(t) for t in rng.integers(0, 53, size=n)] for n in (90, 12, 40)]
    first = generate(folders["attention_first"], prompts, max_tokens=24, dtype="bfloat16", page_size=16, max_cache_tokens=1024, max_requests=4, max_batch_tokens=64)
    second = generate(folders["attention_first"], prompts, max_tokens=24, dtype="bfloat16", page_size=16, max_cache_tokens=1024, max_requests=4, max_batch_tokens=64)
    assert first == second and all(len(tokens) == 24 for tokens in first)
    folder = folders["all"]
    config, tensors = load_plain(folder)
    prompt = [int(t) for t in np.random.default_rng(12).integers(0, config["vocab"], size=11)]
    text = ",".join(map(str, prompt))
    assert main(["generate", str(folder), text, "6", "--dtype", "float32", "--page-size", "16"]) == 0
    result = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert result["generated_tokens"] == _plain_greedy(config, tensors, prompt, 6) and result["prompt_tokens"] == 11
    assert main(["logits", str(folder), text, "--dtype", "float32"]) == 0
    logits = torch.tensor(json.loads(capsys.readouterr().out)["logits"])
    assert torch.allclose(logits, _logits(config, tensors, prompt)[-1], atol=3e-5 * float(logits.abs().max()))
