"""A plain, slow implementation of Nopuzen: whole sequences, no cache, scores materialised, one function per mechanism.

It shares nothing with the engine.  ``config`` is the dictionary of a config.json; ``tensors`` maps tensor names to torch tensors
(any floating dtype; everything is computed in ``dtype``, 32-bit unless said otherwise).
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, weight, bias, eps):
    """A layer norm with a weight and a bias; the variance is the mean of the squared deviations."""
    mean = x.mean(-1, keepdim=True)
    centred = x - mean
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight + bias


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def softplus(z):
    return math.log1p(math.exp(-abs(z))) + max(z, 0.0)


def xielu(z, p, q):
    """A parabola with a linear part above zero, an exponential one below; p and q are stored before their softplus."""
    above = softplus(p) * z * z + 0.5 * z
    below = (0.5 + softplus(q)) * (torch.expm1(z.clamp(max=0.0)) - z) + 0.5 * z
    return torch.where(z > 0, above, below)


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


def latent_heads(q, latent, shared_key, w_uk, w_uv, sizes, positions):
    """q [T, H, dim + rot] as projected, latent [T, rank] normed, shared_key [T, rot] as projected -> heads' outputs [T, H, vdim]: keys and
    values expanded from the latent, a rotated key part that all heads share, an ordinary causal softmax."""
    T, H, dim = q.shape[0], sizes["heads"], sizes["dim"]
    rot = sizes["rot"]
    freq, amplitude = frequencies(sizes["rot_dim"], rot["base"], rot.get("scaling"))
    q_rot = turn(q[..., dim:], positions, freq, amplitude, interleaved=False)
    k_rot = turn(shared_key[:, None, :], positions, freq, amplitude, interleaved=False)[:, 0]
    keys, values = (latent @ w_uk.T).view(T, H, dim), (latent @ w_uv.T).view(T, H, sizes["vdim"])
    seen = positions[:, None] >= positions[None, :]
    out = torch.empty(T, H, sizes["vdim"], dtype=q.dtype)
    for h in range(H):
        score = (q[:, h, :dim] @ keys[:, h].T + q_rot[:, h] @ k_rot.T) * float(sizes["scale"])
        out[:, h] = torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ values[:, h]
    return out


def latent_attention(h, tensors, prefix, sizes, eps, positions=None):
    T = h.shape[0]
    H, dim, rot, vdim, rank = (sizes[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    positions = torch.arange(T) if positions is None else positions
    q = ((rms(h @ w("dq").T, eps) * w("dq.norm")) @ w("uq").T).view(T, H, dim + rot)
    down = h @ w("dkv").T
    latent = rms(down[:, :rank], eps) * w("dkv.norm")
    heads = latent_heads(q, latent, down[:, rank:], w("uk"), w("uv"), sizes, positions).reshape(T, H * vdim)
    return (heads * torch.sigmoid(h @ w("g").T)) @ w("o").T


def sigmoid_heads(q, k, v, temps, shifts, sizes, positions):
    """q [T, H, d], k [T, G, d] normed and turned, v [T, G, dv] -> [T, H, dv]: every visible key's value times a sigmoid of its own of the
    bounded score; the weights of a row need not sum to one."""
    H, G = q.shape[1], k.shape[1]
    cap = float(sizes["softcap"])
    seen = (positions[:, None] >= positions[None, :]).to(q.dtype)
    out = torch.empty(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        score = (q[:, h] @ k[:, g].T) * float(sizes["scale"]) * temps[h]
        score = cap * torch.tanh(score / cap)
        out[:, h] = (torch.sigmoid(score + shifts[h]) * seen) @ v[:, g]
    return out


def sigmoid_attention(h, tensors, prefix, sizes, eps, positions=None):
    T = h.shape[0]
    H, G, d, dv = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
    w = lambda name: tensors[f"{prefix}.{name}"].to(h.dtype)
    positions = torch.arange(T) if positions is None else positions
    q = (h @ w("q").T + w("q.b")).view(T, H, d)
    k = (h @ w("k").T + w("k.b")).view(T, G, d)
    v = (h @ w("v").T + w("v.b")).view(T, G, dv)
    freq, amplitude = frequencies(sizes["rot"]["dims"], sizes["rot"]["base"]) if sizes["rot"]["dims"] else ([], 1.0)
    q = turn(rms(q, eps) * w("q.norm"), positions, freq, amplitude, interleaved=True)
    k = turn(rms(k, eps) * w("k.norm"), positions, freq, amplitude, interleaved=True)
    heads = sigmoid_heads(q, k, v, w("temp"), w("pb"), sizes, positions)
    heads = heads * torch.sigmoid(h @ w("g").T)[:, :, None]
    return heads.reshape(T, H * dv) @ w("o").T + w("o.b")


def relu_squared_ff(h, tensors, prefix):
    z = (h @ tensors[f"{prefix}.up"].to(h.dtype).T).clamp(min=0.0)
    return (z * z) @ tensors[f"{prefix}.down"].to(h.dtype).T


def route(h, tensors, prefix, router):
    """Per token: the chosen experts (a list of indices) and their weights: softmax scores, groups judged by their best expert, the chosen
    scores times a constant."""
    s = torch.softmax(h.float() @ tensors[f"{prefix}.router"].float().T, dim=-1)
    experts, top = router["experts"], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    per = experts // groups["count"]
    chosen, weights = [], []
    for t in range(h.shape[0]):
        best = [max(float(x) for x in s[t, g * per:(g + 1) * per]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -best[g])[: groups["keep"]]
        allowed = [e for e in range(experts) if e // per in kept]
        picks = sorted(allowed, key=lambda e: -float(s[t, e]))[:top]
        chosen.append(picks)
        weights.append([float(s[t, e]) * float(router["scale"]) for e in picks])
    return chosen, weights


def moe_ff(h, tensors, prefix, mlp):
    chosen, weights = route(h, tensors, prefix, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t], weights[t]):
            out[t] += wt * relu_squared_ff(h[t:t + 1], tensors, f"{prefix}.e{e}")[0]
    if mlp.get("shared"):
        gate = torch.sigmoid(h @ tensors[f"{prefix}.shared.sg"].to(h.dtype).T)
        out = out + gate * relu_squared_ff(h, tensors, f"{prefix}.shared")
    return out


def dense_ff(h, tensors, prefix):
    p, q = (float(v) for v in tensors[f"{prefix}.act"])
    return xielu(h @ tensors[f"{prefix}.up"].to(h.dtype).T, p, q) @ tensors[f"{prefix}.down"].to(h.dtype).T


def feed_forward(h, tensors, prefix, mlp):
    return dense_ff(h, tensors, prefix) if mlp["kind"] == "dense" else moe_ff(h, tensors, prefix, mlp)


MIXERS = {"latent_attention": latent_attention, "attention": sigmoid_attention}


def layer(x, tensors, index, spec, eps):
    """The sublayers read the stream as it is; each one's output is normed before it joins."""
    p = f"l{index}"
    norm = lambda y, name: layer_norm(y, tensors[f"{p}.{name}"].to(x.dtype), tensors[f"{p}.{name}.b"].to(x.dtype), eps)
    x = x + norm(MIXERS[spec["type"]](x, tensors, f"{p}.mix", spec["mixer"], eps), "norm1")
    if spec.get("mlp") is not None:
        x = x + norm(feed_forward(x, tensors, f"{p}.mlp", spec["mlp"]), "norm2")
    return x


def forward(config, tensors, tokens, dtype=torch.float32):
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    eps = float(config["norm"]["eps"])
    table = tensors["embed"].to(dtype)
    x = table[torch.as_tensor(tokens)]
    trace = []
    for index, spec in enumerate(config["layers"]):
        x = layer(x, tensors, index, spec, eps)
        trace.append(x)
    logits = layer_norm(x, tensors["final.norm"].to(dtype), tensors["final.norm.b"].to(dtype), eps) @ table.T
    return logits, torch.stack(trace)
