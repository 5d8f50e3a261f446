"""A plain, slow implementation of Vogusun: whole sequences, no cache, scores materialised, one function per mechanism.

It shares nothing with the engine.  ``config`` is the dictionary of a config.json; ``tensors`` maps tensor names to torch tensors
(any floating dtype; everything is computed in ``dtype``, 32-bit unless said otherwise).
"""
from __future__ import annotations

import math

import torch


def dynamic_tanh(x, weight, bias, alpha):
    """What stands in the place of a norm: no statistics, a bounded curve per element."""
    return torch.tanh(alpha * x) * weight + bias


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def frequencies(dims, base, scaling=None):
    """Angle per position of every pair, and what cosines and sines are multiplied by."""
    plain = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return plain, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    turns = lambda t: dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(float(base)))   # the pair that turns t times over the original length
    lo = max(math.floor(turns(float(scaling["fast"]))), 0)
    hi = min(math.ceil(turns(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, positions, freq, amplitude, interleaved):
    """x [T, n, d]: the first 2 len(freq) columns turn by position * freq, columns (2i, 2i + 1) together if ``interleaved``, else column i
    with column i + len(freq)."""
    half = len(freq)
    angle = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=torch.float64).to(x.dtype)[None, :]
    cos, sin = (torch.cos(angle) * amplitude)[:, None, :], (torch.sin(angle) * amplitude)[:, None, :]
    out = x.clone()
    first, second = (slice(0, 2 * half, 2), slice(1, 2 * half, 2)) if interleaved else (slice(0, half), slice(half, 2 * half))
    u, v = x[..., first], x[..., second]
    out[..., first] = u * cos - v * sin
    out[..., second] = v * cos + u * sin
    return out


def rotate(x, positions, rot, interleaved):
    if not rot["dims"]:
        return x
    freq, amplitude = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    return turn(x, positions, freq, amplitude, interleaved)


def mixed_values(v, first, lam):
    """The layer's values drawn towards those of the first layer that mixes (None: this is that layer), number by number whatever the heads' widths are."""
    return v if first is None else (1.0 - lam) * v + lam * first.reshape(v.shape)


def one_more_softmax_heads(q, k, v, scale, positions):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: a softmax whose denominator is one larger than its keys' sum."""
    H, G = q.shape[1], k.shape[1]
    seen = positions[:, None] >= positions[None, :]
    out = torch.empty(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        score = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, float("-inf"))
        top = score.max(-1, keepdim=True).values.clamp(min=0.0)
        p = torch.exp(score - top)
        out[:, h] = (p / (torch.exp(-top) + p.sum(-1, keepdim=True))) @ v[:, g]
    return out


def capped_softmax_heads(q, k, v, scale, cap, positions):
    """The same shapes: bounded scores, an ordinary softmax."""
    H, G = q.shape[1], k.shape[1]
    seen = positions[:, None] >= positions[None, :]
    out = torch.empty(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        score = cap * torch.tanh((q[:, h] @ k[:, g].T) * scale / cap)
        out[:, h] = torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g]
    return out


def attention(h, tensors, prefix, sizes, eps, first=None, positions=None):
    """Returns (output, the layer's own values): normed and turned queries and keys, a softmax with one more, a gate per head."""
    T = h.shape[0]
    H, G, d, dv = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    positions = torch.arange(T) if positions is None else positions
    q = rotate(rms((h @ w("q").T).view(T, H, d), eps) * w("q.norm"), positions, sizes["rot"], interleaved=True)
    k = rotate(rms((h @ w("k").T).view(T, G, d), eps) * w("k.norm"), positions, sizes["rot"], interleaved=True)
    v = (h @ w("v").T).view(T, G, dv)
    used = mixed_values(v, first, w("vmix")) if sizes.get("v_mix") else v
    heads = one_more_softmax_heads(q, k, used, float(sizes["scale"]), positions)
    heads = heads * torch.sigmoid(h @ w("g").T)[:, :, None]
    return heads.reshape(T, H * dv) @ w("o").T, v


def attention_2(h, tensors, prefix, sizes, eps, first=None, positions=None):
    """Returns (output, the layer's own values): biased projections, a stretched rotation in halves, bounded scores."""
    T = h.shape[0]
    H, G, d, dv = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    positions = torch.arange(T) if positions is None else positions
    q = rotate((h @ w("q").T + w("q.b")).view(T, H, d), positions, sizes["rot"], interleaved=False)
    k = rotate((h @ w("k").T + w("k.b")).view(T, G, d), positions, sizes["rot"], interleaved=False)
    v = (h @ w("v").T + w("v.b")).view(T, G, dv)
    used = mixed_values(v, first, w("vmix")) if sizes.get("v_mix") else v
    heads = capped_softmax_heads(q, k, used, float(sizes["scale"]), float(sizes["softcap"]), positions)
    return heads.reshape(T, H * dv) @ w("o").T, v


def gated_linear_recurrence(q, k, v, decay):
    """q, k, decay [T, H, d], v [T, H, dv] -> [T, H, dv], token by token: the key channels' rows of a matrix fade, take the token in and
    are read."""
    T, H, d = q.shape
    state = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        state = decay[t][:, :, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (state * q[t][:, :, None]).sum(1)
    return out


def gated_linear_attention(h, tensors, prefix, sizes, eps):
    T = h.shape[0]
    H, d, dv = sizes["heads"], sizes["dim"], sizes["vdim"]
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    q = (h @ w("q").T).view(T, H, d) * d ** -0.5
    k, v = (h @ w("k").T).view(T, H, d), (h @ w("v").T).view(T, H, dv)
    z = (h @ w("a1").T) @ w("a2").T + w("a2.b")
    decay = torch.sigmoid(z) ** (1.0 / float(sizes["tau"]))
    o = rms(gated_linear_recurrence(q, k, v, decay.view(T, H, d)), eps) * w("norm")
    gate = h @ w("g").T
    return (o.reshape(T, H * dv) * (gate * torch.sigmoid(gate))) @ w("o").T


def dense_ff(h, tensors, prefix):
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    return (gelu_tanh(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def clamped_expert(h, tensors, prefix, limit):
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    g = (h @ w("gate").T).clamp(max=limit)
    u = (h @ w("up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w("down").T


def route(h, tensors, prefix, router):
    """Per token: the chosen experts (a list of indices) and their weights, a softmax over the chosen logits alone."""
    z = h.float() @ tensors[f"{prefix}.router"].float().T + tensors[f"{prefix}.router.b"].float()
    chosen, weights = [], []
    for t in range(h.shape[0]):
        picks = sorted(range(router["experts"]), key=lambda e: -float(z[t, e]))[: router["top"]]
        chosen.append(picks)
        weights.append(torch.softmax(z[t, picks], dim=-1).tolist())
    return chosen, weights


def moe_ff(h, tensors, prefix, mlp):
    chosen, weights = route(h, tensors, prefix, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t], weights[t]):
            out[t] += wt * clamped_expert(h[t:t + 1], tensors, f"{prefix}.e{e}", float(mlp["expert"]["limit"]))[0]
    return out


def feed_forward(h, tensors, prefix, mlp):
    return dense_ff(h, tensors, prefix) if mlp["kind"] == "dense" else moe_ff(h, tensors, prefix, mlp)


def forward(config, tensors, tokens, dtype=torch.float32):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps = float(config["norm"]["eps"])
    norm = lambda y, name: dynamic_tanh(y, tensors[name].to(dtype), tensors[f"{name}.b"].to(dtype), tensors[f"{name}.alpha"].to(dtype))
    x = tensors["embed"].to(dtype)[torch.as_tensor(tokens)]
    trace = []
    first = {}   # the values of the first layer that mixes
    for index, spec in enumerate(config["layers"]):
        p = f"l{index}"
        h = norm(x, f"{p}.norm1")
        if spec["type"] == "gla":
            branch = gated_linear_attention(h, tensors, f"{p}.mix", spec["mixer"], eps)
        else:
            mixer = attention if spec["type"] == "attention" else attention_2
            mixes = bool(spec["mixer"].get("v_mix"))
            branch, values = mixer(h, tensors, f"{p}.mix", spec["mixer"], eps, first.get("values") if mixes else None)
            if mixes and "values" not in first:
                first["values"] = values
        if spec.get("mlp") is not None:
            branch = branch + feed_forward(h, tensors, f"{p}.mlp", spec["mlp"])
        x = x + branch
        trace.append(x)
    logits = norm(x, "final.norm") @ tensors["head"].to(dtype).T
    return logits, torch.stack(trace)
