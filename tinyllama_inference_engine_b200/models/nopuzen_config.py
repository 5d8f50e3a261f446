"""Typed configuration of Nopuzen, read from its own config.json keys.

``layers`` lists the layers one by one: ``{"type": "latent_attention" | "attention", "mixer": {...sizes...}, "mlp": null | {"kind": "dense", "ff": n} |
{"kind": "moe", "expert": {ff}, "router": {experts, top, scale, groups: {count, keep}}, "shared": {ff} | null}}``.  A latent mixer has heads, dim,
rot_dim, vdim, kv_rank, q_rank (read from the tensor's shape if it is not there), scale, rot = {base, dims, scaling: {factor, original, fast, slow} | absent};
an attention mixer heads, kv_heads, dim, vdim, scale, softcap, rot = {base, dims}.  Beside them: ``vocab``, ``width``, ``norm`` = {eps}.  Every size and
constant is free; what the design does not have is refused.
"""
from __future__ import annotations

from dataclasses import dataclass, replace

from ..config.model_config import as_float, as_int
from ..errors import ConfigError

MIXERS = ("latent_attention", "attention")
MLP_KINDS = ("dense", "moe")
MAX_OUTPUTS = 8192     # what a token's heads may add up to in the general attention kernel: heads * vdim, or heads * kv_rank


def _object(where: str, value) -> dict:
    if not isinstance(value, dict):
        raise ConfigError(f"{where} must be an object")
    return value


def _rotation(where: str, rot, dims: int, most: int) -> dict:
    rot = _object(where, rot)
    turned = as_int(f"{where}.dims", rot.get("dims", dims), minimum=0)
    if turned > most or turned % 2:
        raise ConfigError(f"{where}.dims ({turned}) must be even and at most {most}")
    out = {"base": as_float(f"{where}.base", rot.get("base")), "dims": turned}
    if rot.get("scaling") is not None:
        scaling = _object(f"{where}.scaling", rot["scaling"])
        out["scaling"] = {key: as_float(f"{where}.scaling.{key}", scaling.get(key)) for key in ("factor", "original", "fast", "slow")}
        if out["base"] == 1.0:
            raise ConfigError(f"{where}: frequencies that are all the same (base 1) cannot be scaled")
    return out


def _latent_sizes(where: str, mixer: dict) -> dict:
    sizes = {key: as_int(f"{where}.{key}", mixer.get(key)) for key in ("heads", "dim", "rot_dim", "kv_rank")}
    sizes["vdim"] = as_int(f"{where}.vdim", mixer.get("vdim", sizes["dim"]))
    if mixer.get("q_rank") is not None:
        sizes["q_rank"] = as_int(f"{where}.q_rank", mixer["q_rank"])
    sizes["rot"] = _rotation(f"{where}.rot", mixer.get("rot"), sizes["rot_dim"], sizes["rot_dim"])
    if sizes["rot_dim"] % 2:
        raise ConfigError(f"{where}.rot_dim ({sizes['rot_dim']}) must be even")
    if sizes["heads"] * sizes["kv_rank"] > MAX_OUTPUTS:
        raise ConfigError(f"{where}: heads * kv_rank ({sizes['heads'] * sizes['kv_rank']}) may be at most {MAX_OUTPUTS}")
    sizes["scale"] = as_float(f"{where}.scale", mixer.get("scale", (sizes["dim"] + sizes["rot_dim"]) ** -0.5))
    return sizes


def _attention_sizes(where: str, mixer: dict) -> dict:
    heads = as_int(f"{where}.heads", mixer.get("heads"))
    kv_heads = as_int(f"{where}.kv_heads", mixer.get("kv_heads", heads))
    if heads % kv_heads != 0:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    dim = as_int(f"{where}.dim", mixer.get("dim"))
    vdim = as_int(f"{where}.vdim", mixer.get("vdim", dim))
    if heads * vdim > MAX_OUTPUTS:
        raise ConfigError(f"{where}: heads * vdim ({heads * vdim}) may be at most {MAX_OUTPUTS}")
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": as_float(f"{where}.scale", mixer.get("scale", dim ** -0.5)),
            "softcap": as_float(f"{where}.softcap", mixer.get("softcap")), "rot": _rotation(f"{where}.rot", mixer.get("rot"), dim, dim)}


def _mlp_sizes(where: str, mlp):
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind", "dense") not in MLP_KINDS:
        raise ConfigError(f"{where} must be null or a feed-forward of kind {MLP_KINDS}, got {mlp!r}")
    if mlp.get("kind", "dense") == "dense":
        return {"kind": "dense", "ff": as_int(f"{where}.ff", mlp.get("ff"))}
    expert, router = _object(f"{where}.expert", mlp.get("expert")), _object(f"{where}.router", mlp.get("router"))
    experts, top = as_int(f"{where}.router.experts", router.get("experts")), as_int(f"{where}.router.top", router.get("top"))
    groups = {"count": 1, "keep": 1} if router.get("groups") is None else _object(f"{where}.router.groups", router["groups"])
    count = as_int(f"{where}.router.groups.count", groups.get("count", 1))
    keep = as_int(f"{where}.router.groups.keep", groups.get("keep", count))
    if experts % count or keep > count or top > keep * (experts // count):
        raise ConfigError(f"{where}.router: {experts} experts in {count} groups of which {keep} are kept cannot give {top} per token")
    shared = mlp.get("shared")
    if shared is not None:
        shared = {"ff": as_int(f"{where}.shared.ff", _object(f"{where}.shared", shared).get("ff"))}
    return {"kind": "moe", "expert": {"ff": as_int(f"{where}.expert.ff", expert.get("ff"))},
            "router": {"experts": experts, "top": top, "scale": as_float(f"{where}.router.scale", router.get("scale", 1.0)), "groups": {"count": count, "keep": keep}},
            "shared": shared}


@dataclass(frozen=True)
class NopuzenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                # one dictionary per layer: {"type", "mixer", "mlp"}, checked
    architecture: str = "Nopuzen"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, data: dict) -> "NopuzenConfig":
        if not isinstance(data, dict):
            raise ConfigError("config.json must hold a JSON object")
        missing = [key for key in ("vocab", "width", "norm", "layers") if key not in data]
        if missing:
            raise ConfigError("config.json lacks required keys: " + ", ".join(missing))
        if not isinstance(data["layers"], list) or not data["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers = []
        for index, layer in enumerate(data["layers"]):
            kind = _object(f"layers[{index}]", layer).get("type")
            if kind not in MIXERS:
                raise ConfigError(f"layers[{index}].type must be one of {MIXERS}, got {kind!r}")
            mixer = _object(f"layers[{index}].mixer", layer.get("mixer"))
            sizes = (_latent_sizes if kind == "latent_attention" else _attention_sizes)(f"layers[{index}].mixer", mixer)
            layers.append({"type": kind, "mixer": sizes, "mlp": _mlp_sizes(f"layers[{index}].mlp", layer.get("mlp"))})
        return cls(vocab=as_int("vocab", data["vocab"]), width=as_int("width", data["width"]), norm_eps=as_float("norm.eps", _object("norm", data["norm"]).get("eps")),
                   layers=tuple(layers), architecture=str(data.get("architecture", "Nopuzen")))

    def with_tensor_shapes(self, shapes: dict) -> "NopuzenConfig":
        """The configuration with every latent layer's query rank in place, from the tensors' shapes where the file does not name it."""
        layers = []
        for index, layer in enumerate(self.layers):
            name = f"l{index}.mix.dq"
            if layer["type"] == "latent_attention" and "q_rank" not in layer["mixer"] and name in shapes:
                layer = {**layer, "mixer": {**layer["mixer"], "q_rank": int(shapes[name][0])}}
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": [dict(layer) for layer in self.layers]}
