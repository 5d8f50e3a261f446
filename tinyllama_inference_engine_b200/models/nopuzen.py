"""Nopuzen as data: its configuration turned into a ModelSpec.

A decoder whose layers are listed one by one.  The embedding is a table row.  The sublayers of a layer read the stream itself; a layer
norm (weight and bias) stands on each one's output before that joins the stream.  Two mixers: latent attention whose queries pass a
latent of their own, with a rotation stretched by YaRN and an output gate per element; attention with biased projections, normed and
rotated queries and keys, a temperature per head and bounded scores that weigh every visible key by a sigmoid instead of a softmax,
with an output gate per head.  The feed-forward is two products with xIELU between them, or a mixture of experts (square of relu) chosen
by a softmax router with a limit on the groups of experts a token may use, beside a shared expert behind a gate.  The final norm, then
the embedding table as the head.
Tensor names: ``embed``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm2`` (norms each with ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``.
This file only names parts and sizes; every formula lives in the parts.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..errors import ConfigError
from ..parts.spec import LayerSpec, ModelSpec, OrderEntry, PartSpec
from .nopuzen_config import NopuzenConfig

MAX_POSITIONS = 1 << 17   # the design has no table of positions: this only bounds a request's block table


def _mixer(width: int, kind: str, sizes: dict, eps: float, where: str) -> PartSpec:
    rot = sizes["rot"]
    if kind == "attention":
        return PartSpec("sigmoid_attention", {
            "hidden_size": width, "num_heads": sizes["heads"], "num_kv_heads": sizes["kv_heads"], "key_dim": sizes["dim"], "value_dim": sizes["vdim"],
            "scale": sizes["scale"], "eps": eps, "softcap": sizes["softcap"], "rot_dims": rot["dims"], "rot_base": rot["base"], "rot_scaling": rot.get("scaling"),
            "rot_layout": "interleaved",
        })
    if "q_rank" not in sizes:
        raise ConfigError(f"{where}: the rank of the queries' latent is not known (it is named by q_rank or read from the shape of dq)")
    return PartSpec("latent_attention", {
        "hidden_size": width, "num_heads": sizes["heads"], "plain_dim": sizes["dim"], "rot_dim": sizes["rot_dim"], "value_dim": sizes["vdim"], "rank": sizes["kv_rank"],
        "query_rank": sizes["q_rank"], "scale": sizes["scale"], "eps": eps, "rot_dims": rot["dims"], "rot_base": rot["base"], "rot_scaling": rot.get("scaling"),
        "rot_layout": "halves", "sink": False, "output_gate": True,
    })


def _feed_forward(width: int, mlp) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("dense_mlp", {"hidden_size": width, "intermediate_size": mlp["ff"], "activation": "xielu"})
    router, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", {
        "hidden_size": width, "experts": router["experts"], "top": router["top"], "expert_size": mlp["expert"]["ff"], "groups": router["groups"]["count"],
        "keep_groups": router["groups"]["keep"], "route_scale": router["scale"], "activation": "relu_squared", "shared_size": shared["ff"] if shared else 0,
        "shared_gate": True, "correction": False, "normalize": False, "scores": "softmax", "group_score": "best",
    })


def build_nopuzen_spec(config: NopuzenConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    norm = PartSpec("layernorm", {"size": width, "eps": eps, "suffix": "", "bias": True})
    layers = []
    for index, layer in enumerate(config.layers):
        layers.append(LayerSpec(f"l{index}", PartSpec("output_norm", {
            "mixer": _mixer(width, layer["type"], layer["mixer"], eps, f"layers[{index}].mixer"), "mixer_name": "mix", "mixer_norm": norm, "mixer_norm_name": "norm1",
            "feed_forward": _feed_forward(width, layer["mlp"]), "feed_forward_name": "mlp", "feed_forward_norm": norm, "feed_forward_norm_name": "norm2",
        })))
    spec = ModelSpec(
        architecture="Nopuzen", hidden_size=width, vocab_size=config.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "embed"}),
        layers=tuple(layers), order=tuple(OrderEntry(layer=i, cache=i) for i in range(len(layers))),
        final_norm=PartSpec("layernorm", {"size": width, "eps": eps, "suffix": "", "bias": True, "name": "final.norm"}),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "embed", "tied_to": None}),
    )
    spec.validate()
    return spec


NOPUZEN = Architecture(name="Nopuzen", config_class=NopuzenConfig, build_spec=build_nopuzen_spec)
register_architecture(NOPUZEN, replace=True)
