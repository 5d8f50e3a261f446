"""Typed configuration of Vogusun, read from its own config.json keys.

``layers`` lists the layers one by one: ``{"type": "attention" | "attention_2" | "gla", "mixer": {...sizes...}, "mlp": null | {"kind": "dense", "ff": n} |
{"kind": "moe", "expert": {ff, limit}, "router": {experts, top}}}``.  Both attention mixers have heads, kv_heads, dim, vdim, scale, v_mix, rot = {base, dims,
scaling: {factor, original, fast, slow} | absent}; the second also softcap.  A gla mixer has heads, dim, vdim, tau, decay_rank (read from the tensor's
shape if it is not there).  Beside them: ``vocab``, ``width``, ``norm`` = {eps}.  Every size and constant is free; what the design does not have is refused.
"""
from __future__ import annotations

from dataclasses import dataclass, replace

from ..config.model_config import as_float, as_int
from ..errors import ConfigError

ATTENTION_MIXERS = ("attention", "attention_2")
MIXERS = (*ATTENTION_MIXERS, "gla")
MLP_KINDS = ("dense", "moe")
MAX_OUTPUTS = 8192       # heads * vdim of the general attention kernel
MAX_KEY_CHANNELS = 256   # a recurrence's key channels per head


def _object(where: str, value) -> dict:
    if not isinstance(value, dict):
        raise ConfigError(f"{where} must be an object")
    return value


def _rotation(where: str, rot, most: int) -> dict:
    rot = _object(where, rot)
    turned = as_int(f"{where}.dims", rot.get("dims", most), minimum=0)
    if turned > most or turned % 2:
        raise ConfigError(f"{where}.dims ({turned}) must be even and at most {most}")
    out = {"base": as_float(f"{where}.base", rot.get("base")), "dims": turned}
    if rot.get("scaling") is not None:
        scaling = _object(f"{where}.scaling", rot["scaling"])
        out["scaling"] = {key: as_float(f"{where}.scaling.{key}", scaling.get(key)) for key in ("factor", "original", "fast", "slow")}
        if out["base"] == 1.0:
            raise ConfigError(f"{where}: frequencies that are all the same (base 1) cannot be scaled")
    return out


def _attention_sizes(where: str, kind: str, mixer: dict) -> dict:
    heads = as_int(f"{where}.heads", mixer.get("heads"))
    kv_heads = as_int(f"{where}.kv_heads", mixer.get("kv_heads", heads))
    if heads % kv_heads != 0:
        raise ConfigError(f"{where}: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    dim = as_int(f"{where}.dim", mixer.get("dim"))
    vdim = as_int(f"{where}.vdim", mixer.get("vdim", dim))
    if heads * vdim > MAX_OUTPUTS:
        raise ConfigError(f"{where}: heads * vdim ({heads * vdim}) may be at most {MAX_OUTPUTS}")
    sizes = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": as_float(f"{where}.scale", mixer.get("scale", dim ** -0.5)),
             "rot": _rotation(f"{where}.rot", mixer.get("rot"), dim), "v_mix": bool(mixer.get("v_mix", False))}
    if kind == "attention_2":
        sizes["softcap"] = as_float(f"{where}.softcap", mixer.get("softcap"))
        if sizes["softcap"] <= 0.0:
            raise ConfigError(f"{where}.softcap must be positive")
    return sizes


def _gla_sizes(where: str, mixer: dict) -> dict:
    sizes = {key: as_int(f"{where}.{key}", mixer.get(key)) for key in ("heads", "dim")}
    sizes["vdim"] = as_int(f"{where}.vdim", mixer.get("vdim", sizes["dim"]))
    sizes["tau"] = as_float(f"{where}.tau", mixer.get("tau"))
    if sizes["tau"] <= 0.0 or sizes["dim"] > MAX_KEY_CHANNELS:
        raise ConfigError(f"{where}: tau must be positive and dim at most {MAX_KEY_CHANNELS}")
    if mixer.get("decay_rank") is not None:
        sizes["decay_rank"] = as_int(f"{where}.decay_rank", mixer["decay_rank"])
    return sizes


def _mlp_sizes(where: str, mlp):
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind", "dense") not in MLP_KINDS:
        raise ConfigError(f"{where} must be null or a feed-forward of kind {MLP_KINDS}, got {mlp!r}")
    if mlp.get("kind", "dense") == "dense":
        return {"kind": "dense", "ff": as_int(f"{where}.ff", mlp.get("ff"))}
    expert, router = _object(f"{where}.expert", mlp.get("expert")), _object(f"{where}.router", mlp.get("router"))
    experts, top = as_int(f"{where}.router.experts", router.get("experts")), as_int(f"{where}.router.top", router.get("top"))
    if top > experts:
        raise ConfigError(f"{where}.router: {experts} experts cannot give {top} per token")
    return {"kind": "moe", "expert": {"ff": as_int(f"{where}.expert.ff", expert.get("ff")), "limit": as_float(f"{where}.expert.limit", expert.get("limit"))},
            "router": {"experts": experts, "top": top}}


@dataclass(frozen=True)
class VogusunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                # one dictionary per layer: {"type", "mixer", "mlp"}, checked
    architecture: str = "Vogusun"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, data: dict) -> "VogusunConfig":
        if not isinstance(data, dict):
            raise ConfigError("config.json must hold a JSON object")
        missing = [key for key in ("vocab", "width", "norm", "layers") if key not in data]
        if missing:
            raise ConfigError("config.json lacks required keys: " + ", ".join(missing))
        if not isinstance(data["layers"], list) or not data["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers, mixing = [], None
        for index, layer in enumerate(data["layers"]):
            kind = _object(f"layers[{index}]", layer).get("type")
            if kind not in MIXERS:
                raise ConfigError(f"layers[{index}].type must be one of {MIXERS}, got {kind!r}")
            where = f"layers[{index}].mixer"
            mixer = _object(where, layer.get("mixer"))
            sizes = _gla_sizes(where, mixer) if kind == "gla" else _attention_sizes(where, kind, mixer)
            if sizes.get("v_mix"):
                values = sizes["kv_heads"] * sizes["vdim"]
                if mixing is not None and mixing != values:
                    raise ConfigError(f"{where}: layers that mix values have one number of them per token ({mixing}), not {values}")
                mixing = values
            layers.append({"type": kind, "mixer": sizes, "mlp": _mlp_sizes(f"layers[{index}].mlp", layer.get("mlp"))})
        return cls(vocab=as_int("vocab", data["vocab"]), width=as_int("width", data["width"]), norm_eps=as_float("norm.eps", _object("norm", data["norm"]).get("eps")),
                   layers=tuple(layers), architecture=str(data.get("architecture", "Vogusun")))

    def with_tensor_shapes(self, shapes: dict) -> "VogusunConfig":
        """The configuration with every gla layer's decay rank in place, from the tensors' shapes where the file does not name it."""
        layers = []
        for index, layer in enumerate(self.layers):
            name = f"l{index}.mix.a1"
            if layer["type"] == "gla" and "decay_rank" not in layer["mixer"] and name in shapes:
                layer = {**layer, "mixer": {**layer["mixer"], "decay_rank": int(shapes[name][0])}}
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": [dict(layer) for layer in self.layers]}
