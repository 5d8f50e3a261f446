"""Attention over the paged cache with everything that may stand around a softmax over rotated keys as a parameter of its own."""
from __future__ import annotations

import torch

from .. import ops
from ..errors import ConfigError
from .base import CacheNeed, LayerCache, Mixer, register_part
from .position import rotation_frequencies
from .spec import PartSpec, TensorSpec


class RotaryAttention(Mixer):
    """Grouped heads, keys cached rotated, a causal softmax.  What may be there or not:

    ``biases``       q, k and v have one each (``<tensor>.b``), added in 32-bit.
    ``key_norm``     every q and k vector is divided by its root mean square (``eps`` inside the root) and multiplied by a weight, before it turns.
    ``rot_dims``     the first ``rot_dims`` columns of q and k turn by position * frequency: columns (2i, 2i + 1) together for ``rot_layout`` "interleaved",
                     column i with column i + rot_dims / 2 for "halves"; ``rot_base``, optional ``rot_scaling`` (``position.rotation_frequencies``).
    ``softcap``      a score is bounded, softcap * tanh(score / softcap) (0: it is not).
    ``sink``         a number s: the softmax's denominator also holds e^s (None: nothing; 0.0: one is added).
    ``head_gate``    head h's output is multiplied by sigmoid((W_g x)_h), one number per head.
    ``value_mix``    "first": the layer's values are kept for the step, for later layers; "draw": v <- (1 - l) v + l v_first with the same token's
                     values that the layer with "first" kept and l the tensor ``<prefix>.vmix``; the mixed values are what is cached and seen.

    Score of head h: (q . k) * ``scale``; ``scale`` is multiplied into the queries in 32-bit before they are rounded.
    other params: ``hidden_size``, ``num_heads``, ``num_kv_heads`` (query head h reads key/value head h // (heads / kv heads)), ``key_dim``, ``value_dim``.
    tensors: ``<prefix>.q`` [heads * key_dim, hidden], ``<prefix>.k`` [kv * key_dim, hidden], ``<prefix>.v`` [kv * value_dim, hidden], ``<prefix>.o`` [hidden,
    heads * value_dim]; ``<prefix>.{q,k,v}.b``; ``<prefix>.{q,k}.norm`` [key_dim]; ``<prefix>.g`` [heads, hidden]; ``<prefix>.vmix`` [] (with either kind of
    ``value_mix``; "first" does not use it).  q, k, v and the gate are one stacked product.  The cache holds two planes per token: keys and values.
    Norms, angles, scores, softmax, mixing and the gate are 32-bit.
    """

    capturable = True
    fuses_residual_add = True
    prepares_next_norm = True

    @classmethod
    def _sizes(cls, spec: PartSpec) -> tuple[int, int, int, int, int]:
        return int(spec["hidden_size"]), int(spec["num_heads"]), int(spec["num_kv_heads"]), int(spec["key_dim"]), int(spec["value_dim"])

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        hidden, heads, kv, dim, vdim = cls._sizes(spec)
        specs = []
        for name, rows in (("q", heads * dim), ("k", kv * dim), ("v", kv * vdim)):
            specs.append(TensorSpec(f"{prefix}.{name}", (rows, hidden), std=hidden ** -0.5))
            if spec.get("biases"):
                specs.append(TensorSpec(f"{prefix}.{name}.b", (rows,), std=0.2))
        if spec.get("key_norm"):
            specs += [TensorSpec(f"{prefix}.{name}.norm", (dim,), init="norm", std=0.1) for name in ("q", "k")]
        if spec.get("value_mix"):
            specs.append(TensorSpec(f"{prefix}.vmix", (), init="uniform", std=1.0))
        if spec.get("head_gate"):
            specs.append(TensorSpec(f"{prefix}.g", (heads, hidden), std=hidden ** -0.5))
        return specs + [TensorSpec(f"{prefix}.o", (hidden, heads * vdim), std=(heads * vdim) ** -0.5)]

    @classmethod
    def cache_need(cls, spec: PartSpec) -> CacheNeed:
        _, _, kv, dim, vdim = cls._sizes(spec)
        return CacheNeed("pages", planes=((kv, dim), (kv, vdim)))

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = self._sizes(spec)
        self.eps, self.softcap = float(spec.get("eps", 0.0) or 0.0), float(spec.get("softcap", 0.0) or 0.0)
        dtype = runtime.dtype
        names = ("q", "k", "v", "g") if spec.get("head_gate") else ("q", "k", "v")
        stacked = [weights.get(f"{prefix}.{n}", dtype) for n in names]
        self.k_offset = self.heads * self.dim
        self.v_offset = self.k_offset + self.kv_heads * self.dim
        width = self.v_offset + self.kv_heads * self.vdim
        self.gate_offset = -1
        if spec.get("head_gate"):
            self.gate_offset = width
            width += self.heads
        if width % 8:   # rows of the stacked product start on 16-byte boundaries (what the tensor-core attention kernels read them by)
            stacked.append(torch.zeros((8 - width % 8, self.hidden), dtype=dtype, device=stacked[0].device))
        self.w_in = torch.cat(stacked, dim=0).contiguous()
        self.w_o = weights.get(f"{prefix}.o", dtype).contiguous()
        vector = lambda name: weights.get(f"{prefix}.{name}", torch.float32).contiguous()
        self.biases = tuple(vector(f"{n}.b") for n in ("q", "k", "v")) if spec.get("biases") else None
        self.q_weight, self.k_weight = (vector("q.norm"), vector("k.norm")) if spec.get("key_norm") else (None, None)
        per_head = lambda value: torch.full((self.heads,), float(value), dtype=torch.float32, device=runtime.device)
        self.factors = per_head(spec["scale"])
        self.sinks = None if spec.get("sink") is None else per_head(spec["sink"])
        self.value_mix = spec.get("value_mix")
        if self.value_mix not in (None, "first", "draw"):
            raise ConfigError(f"{prefix}: values are kept (\"first\") or drawn towards kept ones (\"draw\"), not {self.value_mix!r}")
        self.value_share = float(weights.get(f"{prefix}.vmix", torch.float32)) if self.value_mix == "draw" else None
        self.rot_dims, self.interleaved = int(spec.get("rot_dims", 0) or 0), spec.get("rot_layout", "interleaved") == "interleaved"
        frequencies, self.amplitude = rotation_frequencies(self.rot_dims, spec.get("rot_base", 10000.0), spec.get("rot_scaling"))
        self.inv_freq = torch.from_numpy(frequencies).to(runtime.device)

    def adds_to_residual(self, rows: int) -> bool:
        return ops.can_accumulate(rows, self.w_o)

    def forward(self, x, ctx, cache: LayerCache, accumulate_into=None, prepare=None):
        ws, dtype, tokens = self.runtime.workspace, self.runtime.dtype, x.shape[0]
        rows = ws.get("qkv_gate", tokens, self.w_in.shape[0], dtype)
        ops.linear(x, self.w_in, rows)
        # the kept values live as long as the step: every layer that reads them runs after the one that wrote them
        kept = ws.get("first_values", tokens, self.kv_heads * self.vdim, dtype) if self.value_mix else None
        ops.norm_rotary_store(rows, self.k_offset, self.v_offset, self.biases, self.q_weight, self.k_weight, self.eps, self.factors, self.inv_freq, self.rot_dims,
                              self.interleaved, self.amplitude, ctx.positions, ctx.token_seq, cache, self.heads, self.kv_heads, self.dim, self.vdim,
                              first_values=kept, value_share=self.value_share)
        mixed = ws.get("attention", tokens, self.heads * self.vdim, dtype)
        ops.mixed_heads_attention(rows, self.gate_offset, ctx.positions, ctx.token_seq, cache, None, None, mixed, self.heads, self.kv_heads, self.dim, self.vdim, 0, 1.0,
                                  batch=ctx, gate_per_head=True, softcap=self.softcap, sinks=self.sinks)
        if accumulate_into is not None:
            ops.linear_accumulate(mixed, self.w_o, accumulate_into, prepare)
            return None
        out = ws.get("mixer_out", tokens, self.hidden, dtype)
        ops.linear(mixed, self.w_o, out)
        return out


register_part("mixer", "rotary_attention", RotaryAttention)
