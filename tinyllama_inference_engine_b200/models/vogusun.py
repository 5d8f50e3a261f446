"""Vogusun as data: its configuration turned into a ModelSpec.

A decoder whose layers are listed one by one.  The embedding is a table row.  A layer reads the stream once, through a curve per element (tanh) in the
place of a norm, and both of its sublayers, side by side, read that; their outputs are added to the stream together.  Three mixers: softmax
attention with normed, rotated queries and keys, one more in the denominator and an output gate per head; softmax attention with biased
projections, a rotation stretched by YaRN and bounded scores; gated linear attention with a learned decay per key channel.  The attention
layers that say so draw their values towards those of the first layer that does.  The feed-forward is a gated one with gelu, or a mixture of
experts with clamped gates under a router whose weights are a softmax over the chosen logits.  The same curve stands before an untied head.
Tensor names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1`` (norms each with ``.b`` and ``.alpha``), ``l<i>.mix.*``, ``l<i>.mlp.*``.
This file only names parts and sizes; every formula lives in the parts.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..errors import ConfigError
from ..parts.spec import LayerSpec, ModelSpec, OrderEntry, PartSpec
from .vogusun_config import VogusunConfig

MAX_POSITIONS = 1 << 17   # the design has no table of positions: this only bounds a request's block table
EXPERT_SLOPE, EXPERT_SHIFT = 1.702, 1.0   # an expert's gate is g sigmoid(1.702 g), its other half is shifted by one


def _mixer(width: int, kind: str, sizes: dict, eps: float, value_mix: str | None, where: str) -> PartSpec:
    if kind == "gla":
        if "decay_rank" not in sizes:
            raise ConfigError(f"{where}: the rank of the decays is not known (it is named by decay_rank or read from the shape of a1)")
        return PartSpec("gated_linear_attention", {"hidden_size": width, "num_heads": sizes["heads"], "key_dim": sizes["dim"], "value_dim": sizes["vdim"],
                                                   "tau": sizes["tau"], "decay_rank": sizes["decay_rank"], "eps": eps})
    rot = sizes["rot"]
    shared = {"hidden_size": width, "num_heads": sizes["heads"], "num_kv_heads": sizes["kv_heads"], "key_dim": sizes["dim"], "value_dim": sizes["vdim"],
              "scale": sizes["scale"], "rot_dims": rot["dims"], "rot_base": rot["base"], "rot_scaling": rot.get("scaling"), "value_mix": value_mix}
    if kind == "attention":
        return PartSpec("rotary_attention", {**shared, "rot_layout": "interleaved", "key_norm": True, "eps": eps, "sink": 0.0, "head_gate": True})
    return PartSpec("rotary_attention", {**shared, "rot_layout": "halves", "biases": True, "softcap": sizes["softcap"]})


def _feed_forward(width: int, mlp) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", {"hidden_size": width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh", "names": ("gate", "up", "down")})
    router = mlp["router"]
    return PartSpec("routed_experts", {
        "hidden_size": width, "experts": router["experts"], "top": router["top"], "expert_size": mlp["expert"]["ff"], "activation": "clamped_sigmoid",
        "limit": mlp["expert"]["limit"], "alpha": EXPERT_SLOPE, "shift": EXPERT_SHIFT, "scores": "logits", "router_bias": True, "correction": False,
    })


def build_vogusun_spec(config: VogusunConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    curve = {"size": width, "suffix": ""}
    layers, kept = [], False   # kept: a layer before has left its values for the layers that draw theirs towards them
    for index, layer in enumerate(config.layers):
        value_mix = None
        if layer["mixer"].get("v_mix"):
            value_mix, kept = ("draw" if kept else "first"), True
        layers.append(LayerSpec(f"l{index}", PartSpec("parallel", {
            "norm": PartSpec("dynamic_tanh", curve), "norm_name": "norm1",
            "mixer": _mixer(width, layer["type"], layer["mixer"], eps, value_mix, f"layers[{index}].mixer"), "mixer_name": "mix",
            "feed_forward": _feed_forward(width, layer["mlp"]), "feed_forward_name": "mlp",
        })))
    spec = ModelSpec(
        architecture="Vogusun", hidden_size=width, vocab_size=config.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "embed", "init_std": 1.0}),
        layers=tuple(layers), order=tuple(OrderEntry(layer=i, cache=i) for i in range(len(layers))),
        final_norm=PartSpec("dynamic_tanh", {**curve, "name": "final.norm"}),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "head", "tied_to": None}),
    )
    spec.validate()
    return spec


VOGUSUN = Architecture(name="Vogusun", config_class=VogusunConfig, build_spec=build_vogusun_spec)
register_architecture(VOGUSUN, replace=True)
