"""Nopuzen through the framework against the plain implementation (plain_nopuzen.py): configuration and names, cache groups, each
mechanism alone (the plain functions' own properties, the kernels by themselves, models of one kind of layer), and the engine's step
function under every way of cutting the work.  The ``gpu`` tests run the kernels; the others need no device."""
from __future__ import annotations

import json
import math

import numpy as np
import pytest
import torch

import plain_nopuzen
import trace_tools
from kernel_steps import pieces_of, scrambled_table, step_of
from tinyllama_inference_engine_b200 import EngineConfig
from tinyllama_inference_engine_b200.cache import CacheManager
from tinyllama_inference_engine_b200.config import architecture_for, load_model_config
from tinyllama_inference_engine_b200.engine.batch import StepEntry
from tinyllama_inference_engine_b200.engine.runner import ModelRunner
from tinyllama_inference_engine_b200.errors import ConfigError
from tinyllama_inference_engine_b200.models import cache_needs, expected_tensors
from tinyllama_inference_engine_b200.models.nopuzen_config import NopuzenConfig
from tinyllama_inference_engine_b200.parts.position import rotation_frequencies
from tinyllama_inference_engine_b200.weights import SafetensorsFile, write_random_model, write_safetensors


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, groups=None, shared=None, scale=1.5):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, "shared": None if shared is None else {"ff": shared}}


def _latent(heads, dim, rot, vdim, rank, q_rank, mlp, base=10000.0, scaling=None, scale=None):
    turn = {"base": base, "dims": rot}
    if scaling:
        turn["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                                                              "scale": 2.0 * (dim + rot) ** -0.5 if scale is None else scale, "rot": turn}}


def _attention(heads, kv_heads, dim, vdim, mlp, rot=None, base=10000.0, scale=None, softcap=6.0):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap,
                                                       "scale": 2.0 * dim ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": dim if rot is None else rot}}}


def _config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nopuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that agree nowhere: latent ranks that the tensor-core kernels take and that they do not, query ranks above and below the latent
# rank, rotations of the whole vector, of a part and of nothing, stretched ones whose blend starts at the first pair, ends at the last or
# has no width, one head, heads that share key/value heads and that do not, key and value widths equal and not, bounds that bite and that
# hardly do, layers with a dense feed-forward, with experts (in groups of which some are dropped, in one group, in groups of one expert, one per
# token, all of them, with and without a shared one) and with none.
CONFIGS = {
    "all": (_config(64, 97, [_latent(4, 16, 16, 32, 32, 24, _dense(48), scaling=(4.0, 64, 8.0, 1.0)), _attention(4, 2, 16, 32, _moe(8, 3, 24, groups=(4, 2), shared=40), rot=8),
                             _latent(2, 32, 8, 16, 64, 48, None), _attention(3, 3, 32, 16, _dense(56), base=500.0, softcap=30.0),
                             _latent(3, 24, 16, 8, 32, 40, _moe(6, 2, 16, shared=None), scaling=(2.0, 1000, 32.0, 0.5), base=200.0)]), 3),
    "latent_first": (_config(48, 61, [_latent(1, 16, 8, 48, 96, 16, _moe(4, 1, 32, groups=(2, 1), shared=16, scale=1.0), scaling=(16.0, 32, 4.0, 4.0)),
                                      _latent(6, 8, 32, 8, 32, 72, _dense(40))], eps=1e-6), 5),
    "attention_first": (_config(40, 53, [_attention(1, 1, 48, 32, _moe(9, 4, 8, groups=(3, 2), shared=8), rot=20), _attention(5, 1, 16, 16, None, rot=0, softcap=3.0),
                                         _attention(8, 4, 16, 64, _dense(24), base=50.0)]), 9),
    "experts": (_config(32, 50, [_attention(2, 1, 64, 64, _moe(5, 5, 16, shared=24)), _latent(2, 16, 16, 16, 32, 8, _moe(6, 2, 8, groups=(6, 3), shared=8, scale=3.0)),
                                 _attention(4, 4, 16, 16, _moe(3, 1, 40))], eps=1e-3), 4),
    # nothing a multiple of 8: the width, the vocabulary, the feed-forwards, the heads' widths, the ranks
    "odd": (_config(44, 37, [_latent(3, 10, 6, 7, 20, 13, _dense(50), scaling=(3.0, 50, 5.0, 1.0)), _attention(3, 1, 12, 10, _moe(6, 2, 10, groups=(3, 2), shared=6), rot=6),
                             _latent(2, 5, 2, 6, 9, 30, _moe(4, 2, 6, shared=10)), _attention(2, 2, 10, 7, _dense(30), rot=10)]), 8),
}
LENGTHS = {"all": [1, 9, 70, 150, 33, 64, 17], "latent_first": [3, 40, 100, 64, 7], "attention_first": [2, 130, 65, 16, 150], "experts": [90, 5, 48, 17], "odd": [70, 3, 33, 18]}
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
    return plain_nopuzen.forward(config, tensors, tokens)[0]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("nopuzen")
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
            "mixed": (mixed, peak)}   # a pool of exactly the peak: pages are used again


# --- configuration, registry, names, cache groups -----------------------------------------------------------------------------------
def test_configuration_round_trip_registry_and_names(folders):
    architecture, config = load_model_config(folders["all"])
    assert architecture.name == "Nopuzen" and isinstance(config, NopuzenConfig)
    assert NopuzenConfig.from_dict(config.to_dict()) == config
    assert config.layers[2]["mlp"] is None and config.layers[0]["mixer"]["rot"]["scaling"] == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    assert "scaling" not in config.layers[2]["mixer"]["rot"] and config.layers[4]["mlp"]["router"]["groups"] == {"count": 1, "keep": 1} and config.layers[4]["mlp"]["shared"] is None
    spec = architecture.build_spec(config)
    names = {t.name: tuple(t.shape) for t in expected_tensors(spec)}
    assert names["embed"] == (97, 64) and names["final.norm"] == (64,) and names["final.norm.b"] == (64,) and "head" not in names
    assert names["l0.norm1"] == (64,) and names["l0.norm1.b"] == (64,) and names["l0.norm2.b"] == (64,) and "l2.norm2" not in names and "l2.mlp.up" not in names
    assert names["l0.mix.dq"] == (24, 64) and names["l0.mix.dq.norm"] == (24,) and names["l0.mix.uq"] == (128, 24) and names["l0.mix.dkv"] == (48, 64)
    assert names["l0.mix.uk"] == (64, 32) and names["l0.mix.uv"] == (128, 32) and names["l0.mix.g"] == (128, 64) and names["l0.mix.o"] == (64, 128) and "l0.mix.q" not in names
    assert names["l0.mlp.up"] == (48, 64) and names["l0.mlp.down"] == (64, 48) and names["l0.mlp.act"] == (2,) and "l0.mlp.gate" not in names
    assert names["l1.mix.q"] == (64, 64) and names["l1.mix.k.b"] == (32,) and names["l1.mix.v"] == (64, 64) and names["l1.mix.o.b"] == (64,) and names["l1.mix.q.norm"] == (16,)
    assert names["l1.mix.temp"] == (4,) and names["l1.mix.pb"] == (4,) and names["l1.mix.g"] == (4, 64)
    assert names["l1.mlp.e7.up"] == (24, 64) and names["l1.mlp.e0.down"] == (64, 24) and names["l1.mlp.router"] == (8, 64) and names["l1.mlp.shared.sg"] == (1, 64)
    assert names["l1.mlp.shared.up"] == (40, 64) and "l1.mlp.e0.gate" not in names and "l1.mlp.act" not in names and "l4.mlp.shared.up" not in names and "l1.mlp.correction" not in names
    assert [(e.layer, e.cache) for e in spec.order] == [(i, i) for i in range(5)]


def test_query_rank_from_the_tensors_shape(folders, tmp_path):
    """A config.json that does not name the rank of the queries' latent is completed from the weight file's header."""
    data = json.loads((folders["latent_first"] / "config.json").read_text())
    for layer in data["layers"]:
        del layer["mixer"]["q_rank"]
    (tmp_path / "config.json").write_text(json.dumps(data))
    (tmp_path / "model.safetensors").write_bytes((folders["latent_first"] / "model.safetensors").read_bytes())
    assert load_model_config(tmp_path)[1] == load_model_config(folders["latent_first"])[1]
    architecture = architecture_for(data)
    with pytest.raises(ConfigError, match="q_rank"):
        architecture.build_spec(architecture.config_class.from_dict(data))


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="lstm"), "type"),
    (lambda c: c["layers"][0].update(mlp={"kind": "routed", "ff": 8}), "kind"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("softcap"), "softcap"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=15), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=4096), "kv_rank"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "experts"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_refuses_what_the_design_lacks(change, message):
    data = json.loads(json.dumps(CONFIGS["all"][0]))
    change(data)
    with pytest.raises(ConfigError, match=message):
        NopuzenConfig.from_dict(data)


def test_cache_groups():
    """A latent layer keeps one plane of rank + rot numbers per token, an attention layer its keys and values; equal needs share a group."""
    architecture = architecture_for(CONFIGS["all"][0])
    needs = cache_needs(architecture.build_spec(architecture.config_class.from_dict(CONFIGS["all"][0])))
    manager = CacheManager(needs, page_size=16, num_pages=40, max_requests=2, max_positions=4096)
    groups = sorted((g.need.page_planes(), len(g.streams)) for g in manager.page_groups)
    assert groups == [(((1, 48),), 2), (((1, 72),), 1), (((2, 16), (2, 32)), 1), (((3, 32), (3, 16)), 1)]


# --- the plain implementation's own mechanisms, and the host's share of the work ------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [(16, 10000.0, None), (2, 50.0, None), (48, 30000.0, (5.0, 1500, 16.0, 2.0)), (16, 10000.0, (4.0, 64, 8.0, 1.0)),
                                               (16, 200.0, (2.0, 1000, 32.0, 0.5)), (8, 10000.0, (16.0, 32, 4.0, 4.0)), (64, 1e6, (40.0, 4096, 32.0, 1.0)), (2, 3.0, (1.0, 10, 3.0, 2.0))])
def test_rotation_frequencies(dims, base, scaling):
    scaling = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    want, amplitude = plain_nopuzen.frequencies(dims, base, scaling)
    got, got_amplitude = rotation_frequencies(dims, base, scaling)
    assert got.dtype == np.float32 and np.allclose(got, want, rtol=1e-6, atol=0.0) and got_amplitude == pytest.approx(amplitude, rel=1e-12)


def test_stretched_rotation_keeps_the_fast_pairs_and_slows_the_rest():
    """Pairs that turn often over the original length keep their frequency, pairs that hardly turn are slowed by the factor, between them the
    frequency falls monotonically; the amplitude grows with the logarithm of the factor."""
    plain, one = plain_nopuzen.frequencies(64, 10000.0)
    scaled, amplitude = plain_nopuzen.frequencies(64, 10000.0, {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    turns = [4096 * f / (2 * math.pi) for f in plain]
    ratio = [s / p for s, p in zip(scaled, plain)]
    assert one == 1.0 and amplitude == pytest.approx(1.0 + 0.1 * math.log(8.0))
    assert all(r == 1.0 for r, t in zip(ratio, turns) if t > 40) and all(r == pytest.approx(1 / 8) for r, t in zip(ratio, turns) if t < 0.5)
    assert all(a >= b for a, b in zip(ratio, ratio[1:])) and any(0.2 < r < 0.9 for r in ratio)


def test_plain_rotations():
    g = torch.Generator().manual_seed(1)
    x = torch.randn(5, 3, 10, generator=g, dtype=torch.float64)
    positions = torch.arange(5)
    freq = [0.7, 0.2]
    for interleaved, partner in ((True, 1), (False, 2)):
        turned = plain_nopuzen.turn(x, positions, freq, 1.0, interleaved)
        assert torch.equal(turned[..., 4:], x[..., 4:]) and torch.equal(turned[0], x[0])
        later = plain_nopuzen.turn(x, positions + 9, freq, 1.0, interleaved)
        assert torch.allclose((turned[3, 0] * turned[1, 1]).sum(), (later[3, 0] * later[1, 1]).sum())     # a score depends on the distance only
        assert torch.allclose(turned[2, 1, 0], x[2, 1, 0] * math.cos(1.4) - x[2, 1, partner] * math.sin(1.4))
        assert torch.allclose(turned[2, 1, partner], x[2, 1, partner] * math.cos(1.4) + x[2, 1, 0] * math.sin(1.4))
        assert torch.allclose(plain_nopuzen.turn(x, positions, freq, 1.5, interleaved)[..., :4], turned[..., :4] * 1.5)


def test_plain_sigmoid_weights():
    """Weights do not depend on the other keys: a row's output is the sum of what each key alone would give; scores are bounded."""
    sizes = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "softcap": 2.0}
    g = torch.Generator().manual_seed(2)
    q, k, v = (torch.randn(6, n, d, generator=g, dtype=torch.float64) for n, d in ((2, 4), (1, 4), (1, 3)))
    temps, shifts = torch.tensor([1.0, 3.0]).double(), torch.tensor([-1.0, 0.5]).double()
    positions = torch.arange(6)
    out = plain_nopuzen.sigmoid_heads(q, k, v, temps, shifts, sizes, positions)
    total = torch.zeros_like(out[5])
    for j in range(6):
        only = v.clone()
        only[torch.arange(6) != j] = 0.0
        total += plain_nopuzen.sigmoid_heads(q, k, only, temps, shifts, sizes, positions)[5]
    assert torch.allclose(out[5], total)
    loud = plain_nopuzen.sigmoid_heads(q[:1] * 1e4, q[:1, :1] * 1e4, torch.ones(1, 1, 3).double(), temps, shifts, sizes, positions[:1])   # a score far beyond the bound
    assert torch.allclose(loud[0, 0], torch.sigmoid(torch.tensor(2.0 - 1.0)).double().expand(3))


def test_plain_router_judges_groups_by_their_best_and_keeps_the_scores():
    router = {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}}
    tensors = {"m.router": torch.eye(6, 8)}     # z = the token's first six numbers
    h = torch.tensor([[4.0, -9.0, 3.9, 3.8, 3.0, 3.5, 0.0, 0.0]])
    chosen, weights = plain_nopuzen.route(h, tensors, "m", router)
    # expert 0 is the best of all, so its group is kept although group 1's two are better together; nothing is renormalised
    s = torch.softmax(h[0, :6], dim=0)
    assert chosen == [[0, 1]] and np.allclose(weights[0], (s[:2] * 3.0).tolist())
    router["groups"] = {"count": 3, "keep": 2}
    assert plain_nopuzen.route(h, tensors, "m", router)[0] == [[0, 2]]
    router["groups"] = None
    assert plain_nopuzen.route(h, tensors, "m", dict(router, top=4))[0] == [[0, 2, 3, 5]]


def test_plain_norm_and_activation():
    x, w, b = torch.randn(3, 10, dtype=torch.float64), torch.randn(10, dtype=torch.float64), torch.randn(10, dtype=torch.float64)
    assert torch.allclose(plain_nopuzen.layer_norm(x, w, b, 1e-5), torch.nn.functional.layer_norm(x, (10,), w, b, 1e-5))
    z = torch.linspace(-6, 3, 400, dtype=torch.float64, requires_grad=True)
    y = plain_nopuzen.xielu(z, 0.3, -0.4)
    y.sum().backward()
    y = y.detach()
    assert float((y[1:] - y[:-1]).abs().max()) < 0.2 and abs(float(plain_nopuzen.xielu(torch.zeros(1).double(), 0.3, -0.4))) < 1e-12
    near = z.grad[(z.detach() > -0.05) & (z.detach() < 0.05)]
    assert float((near - 0.5).abs().max()) < 0.15                      # slope 1/2 on both sides of zero
    assert float(plain_nopuzen.xielu(torch.tensor([2.0]).double(), 0.3, -0.4)) == pytest.approx(math.log1p(math.exp(0.3)) * 4.0 + 1.0)


# --- kernels by themselves ------------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 3e-6), (torch.bfloat16, 1.2e-2)])
@pytest.mark.parametrize("width", [44, 256, 1000])
def test_norm_with_a_bias_and_the_copy_of_the_stream(dtype, atol, width):
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(width)
    stream = torch.randn(9, width, generator=g) * 3.0 + 1.0
    y = (torch.randn(9, width, generator=g) * 2.0 - 0.5).to(dtype)
    post, post_bias, following, following_bias = (torch.randn(width, generator=g) for _ in range(4))
    want_stream = stream.double() + plain_nopuzen.layer_norm(y.double(), post.double(), post_bias.double(), 1e-5)
    want_out = plain_nopuzen.layer_norm(want_stream, following.double(), following_bias.double(), 1e-5)
    device = [t.cuda() for t in (post, post_bias, following, following_bias)]
    residual, out = stream.cuda(), torch.zeros(9, width, dtype=dtype, device="cuda")
    ops.branch_norm(residual, y.cuda(), device[0], device[2], out, 1e-5, post_bias=device[1], next_bias=device[3])
    assert float((residual.cpu().double() - want_stream).abs().max()) <= 3e-6 * float(want_stream.abs().max())
    assert float((out.cpu().double() - want_out).abs().max()) <= atol * float(want_out.abs().max())
    rows = torch.tensor([7, 2, 2], dtype=torch.int32).cuda()
    some = torch.zeros(3, width, dtype=dtype, device="cuda")
    ops.branch_norm(residual, None, None, device[2], some, 1e-5, rows=rows, next_bias=device[3])
    assert torch.equal(some.cpu(), out.cpu()[[7, 2, 2]])
    again, copy = stream.cuda(), torch.zeros(9, width, dtype=dtype, device="cuda")
    ops.branch_norm(again, y.cuda(), device[0], None, copy, 1e-5, post_bias=device[1])
    assert torch.equal(again, residual) and torch.equal(copy, residual.to(dtype))


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 7, 16, 40, 300])
def test_activation_and_bias_behind_a_product(rows):
    """xIELU and the bias in the small-step product's epilogue (one kernel, up to 16 rows) and as kernels behind the product."""
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(rows)
    weight = (torch.randn(72, 64, generator=g) * 0.3).bfloat16()
    x = torch.randn(rows, 64, generator=g).bfloat16()
    product = x.double() @ weight.double().T
    p, q = 0.4, -0.7
    constants = (plain_nopuzen.softplus(p), 0.5 + plain_nopuzen.softplus(q))
    got = torch.zeros(rows, 72, dtype=torch.bfloat16, device="cuda")
    before = ops.launch_count
    ops.linear_activated(x.cuda(), weight.cuda(), got, "xielu", constants)
    assert rows > 16 or ops.launch_count - before == 1
    assert torch.allclose(got.cpu().double(), plain_nopuzen.xielu(product, p, q), atol=3e-2, rtol=3e-2)
    bias = torch.randn(72, generator=g)
    before = ops.launch_count
    ops.linear_bias(x.cuda(), weight.cuda(), bias.cuda(), got)
    assert rows > 16 or ops.launch_count - before == 1
    assert torch.allclose(got.cpu().double(), product + bias.double(), atol=3e-2, rtol=1e-2)
    x32, out = torch.cat([torch.randn(rows, 61, generator=g) * 3.0, torch.tensor([[0.0, -1e-4, -30.0]]).expand(rows, 3)], dim=1), torch.zeros(rows, 64, device="cuda")
    ops.activation("xielu", x32.cuda(), out, constants)
    assert torch.allclose(out.cpu().double(), plain_nopuzen.xielu(x32.double(), p, q), atol=1e-6, rtol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("tokens,heads,n,k", [(3, 4, 16, 32), (5, 3, 7, 20), (70, 2, 64, 96), (65, 1, 10, 9)])
def test_product_per_head_behind_a_gate(dtype, atol, tokens, heads, n, k):
    """The gate is a run of columns of wider rows; few rows have it in the product's kernel, many as a kernel behind the library's."""
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(tokens)
    x, weight = torch.randn(tokens, heads, k, generator=g).to(dtype), (torch.randn(heads, n, k, generator=g) * k ** -0.5).to(dtype)
    wide = torch.randn(tokens, heads * n + 24, generator=g).to(dtype)
    want = torch.einsum("thk,hnk->thn", x.double(), weight.double()).reshape(tokens, heads * n) * torch.sigmoid(wide[:, 16 : 16 + heads * n].double())
    out = torch.zeros(tokens, heads * n, dtype=dtype, device="cuda")
    ops.head_linear(x.cuda(), weight.cuda(), out.view(tokens, heads, n), wide.cuda()[:, 16 : 16 + heads * n])
    assert float((out.cpu().double() - want).abs().max()) <= atol * max(1.0, float(want.abs().max()))


SIGMOID_SHAPES = [(4, 2, 16, 32, 8, True, 1.0), (2, 1, 32, 16, 32, True, 1.2), (3, 3, 16, 16, 0, True, 1.0), (6, 1, 64, 64, 20, False, 1.0), (1, 1, 40, 24, 10, False, 1.3), (5, 5, 10, 6, 4, True, 1.0),
                  (8, 2, 128, 128, 64, True, 1.0), (20, 1, 16, 16, 16, True, 1.0), (4, 2, 80, 48, 80, True, 1.0), (4, 4, 64, 64, 64, True, 1.0)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 3e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,interleaved,amplitude", SIGMOID_SHAPES)
@pytest.mark.parametrize("with_batch,long_tail,page_size", [(False, False, 16), (True, False, 16), (True, True, 16), (True, True, 64)])
def test_sigmoid_attention_kernels(dtype, atol, heads, kv, dim, vdim, rot, interleaved, amplitude, with_batch, long_tail, page_size):
    """Biases, norm, rotation, temperatures, cache write and the sigmoid weights against the plain functions: every request in three steps, so
    that the later ones read what the first cached through a scrambled block table.  With the step's context the kernels are chosen as the
    engine chooses them (tensor cores for portions, a row's keys dealt to several CTAs for steps of few rows); without it the general
    kernel runs alone.  Shifts of both signs: one head weighs few keys, another nearly all."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    lens, firsts = ([37, 1, 18], [30, 52, 0]) if not long_tail else ([5, 200, 9], [330, 0, 61])
    g = torch.Generator().manual_seed(heads * 100 + dim)
    table, count = scrambled_table([f + n for n, f in zip(lens, firsts)], page_size, g)
    columns = heads * dim + kv * dim + kv * vdim + heads
    columns += -columns % 8
    rows = [torch.randn(f + n, columns, generator=g).to(dtype) for n, f in zip(lens, firsts)]
    planes = tuple(torch.full((count, kv, page_size, w), float("nan")).to(dtype).cuda() for w in (dim, vdim))
    cache = LayerCache(CacheNeed("pages"), True, None, table.cuda(), page_size, None, planes)
    biases = tuple(torch.randn(n, generator=g) * 0.5 for n in (heads * dim, kv * dim, kv * vdim))
    q_weight, k_weight = 1 + 0.2 * torch.randn(dim, generator=g), 1 + 0.2 * torch.randn(dim, generator=g)
    temps, shifts = 1 + 0.5 * torch.rand(heads, generator=g), torch.linspace(-4.0, 2.0, heads)
    sizes = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 2.5 * dim ** -0.5, "softcap": 4.0}
    eps, freq = 1e-5, plain_nopuzen.frequencies(rot, 300.0)[0] if rot else []
    inv_freq = torch.tensor(freq, dtype=torch.float32).cuda()
    k_offset, v_offset, gate_offset = heads * dim, (heads + kv) * dim, (heads + kv) * dim + kv * vdim
    want = []
    for r in rows:
        x, total = r.double(), r.shape[0]
        positions = torch.arange(total)
        q = (x[:, :k_offset] + biases[0].double()).view(total, heads, dim)
        k = (x[:, k_offset:v_offset] + biases[1].double()).view(total, kv, dim)
        v = (x[:, v_offset:gate_offset] + biases[2].double()).view(total, kv, vdim)
        q = plain_nopuzen.turn(plain_nopuzen.rms(q, eps) * q_weight.double(), positions, freq, amplitude, interleaved)
        k = plain_nopuzen.turn(plain_nopuzen.rms(k, eps) * k_weight.double(), positions, freq, amplitude, interleaved)
        o = plain_nopuzen.sigmoid_heads(q, k, v, temps.double(), shifts.double(), sizes, positions)
        want.append((o * torch.sigmoid(x[:, gate_offset : gate_offset + heads])[:, :, None]).reshape(total, heads * vdim))
    got = [torch.zeros_like(w) for w in want]
    device = [t.cuda() for t in (*biases, q_weight, k_weight, temps * sizes["scale"], shifts)]
    for pieces in pieces_of(lens, firsts):
        step_rows, positions, token_seq, sub, batch, index = step_of(rows, cache, pieces)
        ops.norm_rotary_store(step_rows, k_offset, v_offset, device[:3], device[3], device[4], eps, device[5], inv_freq, rot, interleaved, amplitude, positions, token_seq, sub,
                              heads, kv, dim, vdim)
        out = torch.zeros(len(index), heads * vdim, dtype=dtype, device="cuda")
        ops.mixed_heads_attention(step_rows, gate_offset, positions, token_seq, sub, None, None, out, heads, kv, dim, vdim, 0, 1.0, batch=batch if with_batch else None,
                                  gate_per_head=True, softcap=4.0, sigmoid=True, shifts=device[6])
        for (r, p), row in zip(index, out.cpu().double()):
            got[r][p] = row
    for r in range(len(rows)):
        size = want[r].abs().mean(dim=1, keepdim=True).clamp(min=1.0)      # sums of hundreds of unnormalised weights grow with the row's position
        assert float(((got[r] - want[r]).abs() / size).max()) <= atol * (4.0 if dtype == torch.bfloat16 else 1.0), r


@pytest.mark.gpu
@pytest.mark.parametrize("dim,heads,kv,page_size,softcap", [(64, 4, 2, 64, 4.0), (128, 8, 2, 64, 4.0), (128, 3, 3, 128, 30.0), (64, 16, 1, 64, 0.0)])
def test_sigmoid_attention_in_tensor_memory(dim, heads, kv, page_size, softcap, monkeypatch):
    """Prompt portions whose heads are 64 or 128 wide run on the tcgen05 kernel, decoding requests at the step's head on the kernel of few rows:
    portions from position 0 and behind cached keys (a request's keys in an earlier step), page borders, a portion of 129 rows, loud scores."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.engine.batch import pack_step
    from tinyllama_inference_engine_b200.ops import fast
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    g = torch.Generator().manual_seed(dim + heads)
    lens, firsts = [1, 1, 300, 129, 200], [70, 200, 0, 130, 1]
    totals = [f + n for n, f in zip(lens, firsts)]
    table, count = scrambled_table(totals, page_size, g)
    columns = (heads + 2 * kv) * dim + heads
    columns += -columns % 8
    rows = [torch.randn(t, columns, generator=g).bfloat16() for t in totals]
    for r in rows:      # some keys stand out for some queries of their head
        r[-1, :dim] = r[5, heads * dim : (heads + 1) * dim] * 2.0
    pages = torch.full((count, 2, kv, page_size, dim), float("nan")).bfloat16().cuda()
    temps, shifts = (1 + 0.5 * torch.rand(heads, generator=g)) * 2.0 * dim ** -0.5, torch.linspace(-5.0, 1.0, heads)
    gate_at, k_at, v_at = (heads + 2 * kv) * dim, heads * dim, (heads + kv) * dim
    device = [temps.cuda(), shifts.cuda(), torch.zeros(0, device="cuda")]
    want = []
    for r in rows:
        x, total = r.double(), r.shape[0]
        q = (x[:, :k_at].view(total, heads, dim) * temps.double()[:, None]).bfloat16().double()
        sizes = {"heads": heads, "kv_heads": kv, "scale": 1.0, "softcap": softcap if softcap > 0 else 1e6}
        o = plain_nopuzen.sigmoid_heads(q, x[:, k_at:v_at].view(total, kv, dim), x[:, v_at:gate_at].view(total, kv, dim), torch.ones(heads).double(), shifts.double(), sizes, torch.arange(total))
        want.append((o * torch.sigmoid(x[:, gate_at : gate_at + heads])[:, :, None]).reshape(total, heads * dim))
    calls = []
    kernel = fast.prefill_attention_tc
    monkeypatch.setattr(fast, "prefill_attention_tc", lambda *a, **k: (calls.append(1), kernel(*a, **k)))
    for pieces in ([(r, 0, f) for r, f in enumerate(firsts) if f > 0], [(r, f, n) for r, (n, f) in enumerate(zip(lens, firsts))]):
        entries = [StepEntry(r, [0] * n, []) for r, _, n in pieces]
        ctx = pack_step(entries, [a for _, a, _ in pieces], list(range(len(pieces))), [[table[r].tolist() for r, _, _ in pieces]], torch.device("cuda:0"))
        cache = LayerCache(CacheNeed("pages"), True, pages, ctx.block_tables[0], page_size)
        index = [(r, a + i) for r, a, n in pieces for i in range(n)]
        step_rows = torch.stack([rows[r][p] for r, p in index]).cuda().contiguous()
        ops.norm_rotary_store(step_rows, k_at, v_at, None, None, None, 1e-5, device[0], device[2], 0, True, 1.0, ctx.positions, ctx.token_seq, cache, heads, kv, dim, dim)
        out = torch.full((len(index), heads * dim), float("nan"), dtype=torch.bfloat16, device="cuda")
        ops.mixed_heads_attention(step_rows, gate_at, ctx.positions, ctx.token_seq, cache, None, None, out, heads, kv, dim, dim, 0, 1.0, batch=ctx, gate_per_head=True, softcap=softcap,
                                  sigmoid=True, shifts=device[1])
        assert int(fast.tcgen05_error_flag(out.device)) == 0, "a bounded wait inside the kernel gave up"
        for (r, p), row in zip(index, out.cpu().double()):
            rms_of = lambda v: float((v * v).mean().sqrt())
            assert rms_of(row - want[r][p]) <= 1e-2 * max(0.5, rms_of(want[r][p])), (r, p)
    assert len(calls) == 2


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,q_rank,interleaved", [(4, 16, 16, 32, 32, 24, False), (1, 20, 6, 10, 96, 40, False), (3, 10, 2, 7, 20, 13, True), (16, 32, 64, 32, 128, 48, False),
                                                                            (20, 16, 16, 16, 64, 32, True), (2, 64, 64, 32, 512, 40, False)])
@pytest.mark.parametrize("long_tail,singles", [(False, False), (True, False), (True, True)])
def test_latent_attention_kernels(dtype, atol, heads, dim, rot, vdim, rank, q_rank, interleaved, long_tail, singles):
    """The norms of both latents, the rotations with an amplitude, the cache write, the products moved across the attention and the gate against
    expanded keys and values, in three steps through a scrambled block table."""
    from tinyllama_inference_engine_b200 import ops
    from tinyllama_inference_engine_b200.parts.base import CacheNeed, LayerCache

    lens, firsts, page_size = ([37, 1, 18], [30, 52, 0], 16) if not long_tail else ([5, 150, 9], [330, 0, 61], 16)
    g = torch.Generator().manual_seed(rank)
    table, count = scrambled_table([f + n for n, f in zip(lens, firsts)], page_size, g)
    latent_offset, gate_offset = q_rank + (-q_rank % 8), q_rank + (-q_rank % 8) + rank + rot
    rows = [torch.randn(f + n, gate_offset + heads * vdim, generator=g).to(dtype) for n, f in zip(lens, firsts)]
    pages = torch.full((count, 1, 1, page_size, rank + rot), float("nan")).to(dtype).cuda()
    cache = LayerCache(CacheNeed("pages"), True, pages, table.cuda(), page_size)
    w_uq, w_uk, w_uv = ((torch.randn(a, b, generator=g) * b ** -0.5).to(dtype) for a, b in ((heads * (dim + rot), q_rank), (heads * dim, rank), (heads * vdim, rank)))
    q_weight, weight = 1 + 0.2 * torch.randn(q_rank, generator=g), 1 + 0.2 * torch.randn(rank, generator=g)
    eps, scale, amplitude = 1e-5, 1.5 * (dim + rot) ** -0.5, 1.2
    freq = plain_nopuzen.frequencies(rot, 300.0)[0]
    want = []
    for r in rows:
        x, total = r.double(), r.shape[0]
        positions = torch.arange(total)
        q = ((plain_nopuzen.rms(x[:, :q_rank], eps) * q_weight.double()) @ w_uq.double().T).view(total, heads, dim + rot)
        latent = plain_nopuzen.rms(x[:, latent_offset : latent_offset + rank], eps) * weight.double()
        keys, values = (latent @ w_uk.double().T).view(total, heads, dim), (latent @ w_uv.double().T).view(total, heads, vdim)
        q_rot = plain_nopuzen.turn(q[..., dim:], positions, freq, amplitude, interleaved)
        k_rot = plain_nopuzen.turn(x[:, None, latent_offset + rank : gate_offset], positions, freq, amplitude, interleaved)[:, 0]
        score = (torch.einsum("ihd,jhd->hij", q[..., :dim], keys) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * scale
        score = score.masked_fill(positions[:, None] < positions[None, :], float("-inf"))
        o = torch.einsum("hij,jhd->ihd", torch.softmax(score, dim=-1), values).reshape(total, heads * vdim)
        want.append(o * torch.sigmoid(x[:, gate_offset:]))
    got = [torch.zeros_like(w) for w in want]
    inv_freq = torch.tensor(freq, dtype=torch.float32).cuda()
    uk_t = w_uk.view(heads, dim, rank).transpose(1, 2).contiguous().cuda()
    sizes = (heads, dim, rot, rank, interleaved, amplitude)
    steps = list(pieces_of(lens, firsts))
    if singles:     # the last rows one by one: steps of single tokens, of fewer and fewer requests
        steps = steps[:2] + [[(r, a + i, 1) for r, a, n in steps[2] if i < n] for i in range(max(n for _, _, n in steps[2]))]
    for pieces in steps:
        step_rows, positions, token_seq, sub, batch, index = step_of(rows, cache, pieces)
        tokens = len(index)
        q_latent, queries = torch.zeros(tokens, q_rank, dtype=dtype, device="cuda"), torch.zeros(tokens, heads * (rank + rot), dtype=dtype, device="cuda")
        ops.latent_store(step_rows, latent_offset, weight.cuda(), eps, inv_freq, rot, positions, token_seq, sub, None, *sizes, q_latent=(0, q_weight.cuda(), q_latent))
        query_rows = torch.zeros(tokens, heads * (dim + rot), dtype=dtype, device="cuda")
        ops.linear(q_latent, w_uq.cuda(), query_rows)
        ops.latent_store(None, 0, weight.cuda(), eps, inv_freq, rot, positions, token_seq, sub, queries, *sizes, query_rows=query_rows)
        ops.head_linear(query_rows.view(tokens, heads, dim + rot)[:, :, :dim], uk_t, queries.view(tokens, heads, rank + rot)[:, :, :rank])
        summed, out = torch.zeros(tokens, heads * rank, dtype=dtype, device="cuda"), torch.zeros(tokens, heads * vdim, dtype=dtype, device="cuda")
        ops.mixed_heads_attention(queries, -1, positions, token_seq, sub, None, None, summed, heads, 1, rank + rot, rank, 0, scale, batch=batch, values_in_keys=True)
        ops.head_linear(summed.view(tokens, heads, rank), w_uv.view(heads, vdim, rank).cuda(), out.view(tokens, heads, vdim), step_rows[:, gate_offset:])
        for (r, p), row in zip(index, out.cpu().double()):
            got[r][p] = row
    for r in range(len(rows)):
        assert float((got[r] - want[r]).abs().max()) <= atol * max(1.0, float(want[r].abs().max())), r


@pytest.mark.gpu
@pytest.mark.parametrize("heads,dim,rot,vdim", [(3, 128, 64, 128), (4, 64, 64, 64), (2, 64, 128, 64), (1, 128, 64, 64), (2, 64, 64, 128)])
def test_latent_attention_over_the_steps_own_rows(heads, dim, rot, vdim):
    """A step that begins all its requests: expanded keys with a part that the heads share, through the tensor-memory kernel; row tiles that
    end inside a key tile, requests next to one another in the same matrices, a key that stands out."""
    from tinyllama_inference_engine_b200.engine.batch import pack_step
    from tinyllama_inference_engine_b200.ops import fast

    g = torch.Generator().manual_seed(dim + rot + vdim)
    lens = [300, 129, 64, 2, 200, 127]
    starts = np.concatenate([[0], np.cumsum(lens)])
    tokens = int(starts[-1])
    queries = torch.randn(tokens, heads, dim + rot, generator=g).bfloat16()
    keys, values, shared = torch.randn(tokens, heads, dim, generator=g), torch.randn(tokens, heads, vdim, generator=g), torch.randn(tokens, rot, generator=g)
    keys[3] = queries[250, :, :dim].float() * 3.0                          # far back in the first request, and late in another one
    keys[starts[4] + 150] = queries[starts[4] + 190, :, :dim].float() * 5.0
    keys, values, shared = keys.bfloat16(), values.bfloat16(), shared.bfloat16()
    scale = 1.5 * (dim + rot) ** -0.5
    want = torch.empty(tokens, heads, vdim, dtype=torch.float64)
    for a, b in zip(starts[:-1], starts[1:]):
        score = torch.einsum("ihd,jhd->hij", queries[a:b, :, :dim].double(), keys[a:b].double()) + torch.einsum("ihd,jd->hij", queries[a:b, :, dim:].double(), shared[a:b].double())
        score = (score * scale).masked_fill(torch.arange(b - a)[:, None] < torch.arange(b - a)[None, :], float("-inf"))
        want[a:b] = torch.einsum("hij,jhd->ihd", torch.softmax(score, dim=-1), values[a:b].double())
    ctx = pack_step([StepEntry(i, [0] * n, []) for i, n in enumerate(lens)], [0] * len(lens), list(range(len(lens))), [[[0]] * len(lens)], torch.device("cuda:0"))
    tiles = fast.latent_rows_tiles(ctx)
    assert tiles is not None and fast.latent_rows_fit(dim, rot, vdim, torch.bfloat16)
    later = pack_step([StepEntry(0, [0] * 300, [])], [1], [0], [[[0]]], torch.device("cuda:0"))
    assert fast.latent_rows_tiles(later) is None          # a step behind cached tokens is not for this kernel
    expanded = torch.cat([keys.reshape(tokens, -1), values.reshape(tokens, -1)], dim=1).cuda()
    out = torch.full((tokens, heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
    fast.latent_rows(queries.view(tokens, -1).cuda(), expanded, shared.cuda(), tiles, ctx, out, heads, dim, rot, vdim, scale)
    assert int(fast.tcgen05_error_flag(out.device)) == 0, "a bounded wait inside the kernel gave up"
    error = (out.cpu().double() - want.reshape(tokens, -1)).abs().max(dim=1).values
    assert float(error.max()) <= 3e-2, int(error.argmax())


@pytest.mark.gpu
@pytest.mark.parametrize("tokens", [50, 1300])    # a CTA per token; four tokens per CTA (a step of many rows), the last CTA short of rows
@pytest.mark.parametrize("experts,groups,keep,top,width", [(8, 4, 2, 3, 64), (6, 1, 1, 2, 44), (9, 3, 2, 4, 40), (4, 4, 3, 2, 32), (64, 8, 4, 8, 128), (5, 5, 1, 1, 24), (12, 2, 1, 6, 48),
                                                           (10, 5, 2, 3, 42), (7, 1, 1, 7, 17)])    # rows that are no multiple of four numbers: the general form
@pytest.mark.parametrize("gated", [True, False])
def test_softmax_router_kernel(tokens, experts, groups, keep, top, width, gated):
    """The chosen experts and their scores as they are, and the shared branch's gate from one row more, against the plain router."""
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(experts * 7 + width)
    x = torch.randn(tokens, width, generator=g)
    tensors = {"m.router": torch.randn(experts, width, generator=g) * 2.0 * width ** -0.5}
    row = torch.randn(1, width, generator=g) * width ** -0.5
    router = {"experts": experts, "top": top, "scale": 2.5, "groups": {"count": groups, "keep": keep}}
    chosen, weights = plain_nopuzen.route(x, tensors, "m", router)
    ids, got = torch.zeros(tokens, top, dtype=torch.int32, device="cuda"), torch.zeros(tokens, top, device="cuda")
    gate = torch.zeros(tokens, 1, device="cuda") if gated else None
    stacked = torch.cat([tensors["m.router"], row]) if gated else tensors["m.router"]
    ops.moe_route(x.cuda(), stacked.cuda(), None, ids, got, groups, keep, 2.5, normalize=False, scores="softmax", group_score="best", shared_gate=gate)
    wrong = [t for t in range(tokens) if ids[t].cpu().tolist() != chosen[t]]
    for t in wrong:      # another order of the sum may turn a choice only where two scores all but tie
        z = torch.softmax(tensors["m.router"].double() @ x[t].double(), dim=0)
        gaps = (z[:, None] - z[None, :]).abs() + torch.eye(experts, dtype=torch.float64)
        assert float(gaps.min()) < 1e-5, t
    right = [t for t in range(tokens) if t not in wrong]
    assert len(right) >= tokens - 2
    assert torch.allclose(got.cpu()[right], torch.tensor(weights)[right], atol=1e-5)
    if gated:
        assert torch.allclose(gate.cpu().double(), torch.sigmoid(x.double() @ row.double().T), atol=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,atol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("tokens,experts,top,width,ff,shared,gated", [(5, 6, 2, 44, 10, True, True), (16, 6, 2, 64, 100, True, False), (70, 8, 3, 64, 24, True, True), (300, 4, 1, 32, 16, False, False),
                                                                      (130, 16, 4, 128, 48, True, True), (1, 3, 3, 24, 8, False, False),
                                                                      (300, 4, 1, 64, 72, False, False), (700, 6, 3, 136, 200, True, True), (400, 3, 2, 64, 520, True, True)])   # enough rows per expert for tcgen05
def test_expert_kernels_without_a_gate(dtype, atol, tokens, experts, top, width, ff, shared, gated):
    """The chosen experts' squares of relu, weighted and summed with the shared branch times its gate: steps of few rows read the experts'
    rows directly, bfloat16 prompt portions sort by expert and use the tensor cores.  A token's result does not depend on the step."""
    from tinyllama_inference_engine_b200 import ops

    g = torch.Generator().manual_seed(tokens + experts)
    x = torch.randn(tokens, width, generator=g).to(dtype)
    up = (torch.randn(experts, ff, width, generator=g) * width ** -0.5).to(dtype)
    down = (torch.randn(experts, width, ff, generator=g) * ff ** -0.5).to(dtype)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32)
    ids[: tokens // 2, 0] = ids[0, 0]        # one crowded expert (a token may then name it twice; both are added)
    weights = torch.rand(tokens, top, generator=g) + 0.1
    branch = torch.randn(tokens, width, generator=g).to(dtype) if shared else None
    gate = torch.rand(tokens, 1, generator=g) if gated else None
    want = torch.zeros(tokens, width, dtype=torch.float64) if branch is None else branch.double() * (gate.double() if gated else 1.0)
    y = torch.einsum("ewf,tef->tew", down.double(), torch.einsum("efw,tw->tef", up.double(), x.double()).clamp(min=0.0) ** 2)
    for k in range(top):
        want = want + weights[:, k, None].double() * y[torch.arange(tokens), ids[:, k].long()]
    some = torch.arange(0, tokens, max(1, tokens // 5))
    for index in (torch.arange(tokens), some):
        got = torch.zeros(len(index), width, dtype=dtype, device="cuda")
        ops.moe_experts(x[index].cuda(), up.cuda(), down.cuda(), ids[index].cuda(), weights[index].cuda(), None if branch is None else branch[index].cuda(), got, "relu_squared",
                        shared_gate=None if gate is None else gate[index].cuda())
        assert int(ops.error_flag(got.device)) == 0
        assert float((got.cpu().double() - want[index]).abs().max()) <= atol * max(1.0, float(want.abs().max()))


# --- the engine on the GPU under every way of cutting the work ---------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(CONFIGS))
def test_engine_matches_plain_under_every_schedule(cases, key, dtype):
    """Whole prompts, a tail decoded token by token, portions down to two tokens, and four live requests mixed in a pool that makes
    pages come round again (freed pages are poisoned with NaN)."""
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
    want = plain_nopuzen.forward(config, tensors, tokens)[1]
    trace = {}
    _runner(folder, "float32").step([StepEntry("a", tokens, [0])], trace=trace)
    assert len(trace) == len(want) == len(config["layers"])
    for index, layer in enumerate(want):
        assert float((trace[f"layer{index}.output"].cpu() - layer).abs().max()) <= 3e-5 * float(layer.abs().max()), index


# models of one kind of layer, with sizes that no other test has
ONE_KIND = {
    "latent": _config(56, 41, [_latent(5, 48, 32, 40, 160, 64, None, scaling=(6.0, 40, 6.0, 0.5)), _latent(2, 16, 64, 24, 32, 32, None)]),
    "latent_dense": _config(72, 41, [_latent(2, 8, 8, 8, 64, 16, _dense(200))]),
    "attention": _config(56, 41, [_attention(6, 2, 48, 80, None, rot=24), _attention(7, 7, 16, 32, None, softcap=50.0)]),
    "attention_experts": _config(72, 41, [_attention(2, 2, 128, 128, _moe(16, 6, 64, groups=(8, 4), shared=64, scale=0.7))]),
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


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["latent_attention", "attention"])
def test_far_keys_and_first_tokens_decide(tmp_path, kind, dtype):
    """A large score scale lets single keys stand out hundreds of tokens back and across page borders (the sigmoid's shifts are so low that only
    such keys weigh anything): a lost key or a rotation by the wrong position then moves the logits far beyond the tolerance, in
    portions, in decoded tokens and in mixed batches."""
    layer = _latent(2, 32, 16, 32, 64, 40, _dense(32), scaling=(4.0, 64, 8.0, 1.0), scale=1.2) if kind == "latent_attention" else _attention(4, 2, 32, 32, _dense(32), scale=1.2, softcap=20.0)
    data = _config(40, 53, [layer])
    base = write_random_model(tmp_path / "base", data, 7)
    _, tensors = load_plain(base, torch.bfloat16)
    for name in tensors:
        if name.endswith(".pb"):
            tensors[name] = torch.full_like(tensors[name], -9.0)
    folder = tmp_path / "sharp"
    folder.mkdir()
    (folder / "config.json").write_text((base / "config.json").read_text())
    write_safetensors(folder / "model.safetensors", tensors)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(config["vocab"], [400, 70, 33], seed=17)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())

    def moved(tokens):      # the largest change of the last forty rows, hundreds of tokens behind every changed token
        return float((_logits(config, tensors, tokens)[-40:] - full["r0"][-40:]).abs().max())

    early = [(t + 1) % config["vocab"] if 10 <= i < 50 else t for i, t in enumerate(requests["r0"])]       # across page borders
    assert moved(early) > 100 * TOLERANCE["float32"] * scale
    first = [(t + 1) % config["vocab"] if i < 3 else t for i, t in enumerate(requests["r0"])]
    assert moved(first) > 20 * TOLERANCE["float32"] * scale
    for steps in (trace_tools.tail_decode(requests, tail=40), trace_tools.portions(requests), trace_tools.mixed(requests, seed=4, max_portion=90)[0]):
        trace_tools.run_and_compare(_runner(folder, dtype, max_tokens=2048), steps, full, atol=TOLERANCE[dtype] * scale * (1.0 if dtype == "float32" else 3.0), over_vocabulary=RMS[dtype])


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
def test_long_portions_beside_decoded_tokens(tmp_path, dim, kv, monkeypatch):
    """Portions of up to 200 rows beside single tokens with pages of 64: the tensor-memory kernels (steps that begin their requests attend to their
    own expanded rows in the latent layer, later portions to the cache), the kernel of few rows at the step's head and the ones between
    them, in one model."""
    from tinyllama_inference_engine_b200.ops import fast

    calls, kernel = [], fast.latent_rows
    monkeypatch.setattr(fast, "latent_rows", lambda *a: (calls.append(a[0].shape[0]), kernel(*a)))
    folder = write_random_model(tmp_path / "m", _config(64, 47, [_attention(4, kv, dim, dim, _dense(64)), _latent(4, 64, 64, 64, 64, 48, _dense(96), scaling=(4.0, 100, 8.0, 1.0))]), 3)
    config, tensors = load_plain(folder)
    requests = trace_tools.make_requests(47, [500, 230, 64, 300], seed=9)
    full = {rid: _logits(config, tensors, tokens) for rid, tokens in requests.items()}
    scale = max(float(v.abs().max()) for v in full.values())
    for steps in (trace_tools.whole(requests), trace_tools.tail_decode(requests, tail=20), trace_tools.portions(requests, sizes=(200, 65, 2, 128)),
                  trace_tools.mixed(requests, seed=2, max_portion=200)[0]):
        trace_tools.run_and_compare(_runner(folder, "bfloat16", max_tokens=2048, page_size=64), steps, full, atol=TOLERANCE["bfloat16"] * scale, over_vocabulary=True)
    assert 500 in calls and 200 in calls      # whole prompts and first portions


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
    results = engine.generate(prompts, SamplingParams(max_tokens=20))
    for prompt, result in zip(prompts, results):
        assert result.generated_tokens == _plain_greedy(config, tensors, prompt, 20)
    again = engine.generate(prompts[:3], SamplingParams(max_tokens=20))       # pages come round again; shapes repeat, so graphs replay
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
