"""A plain, slow implementation of the Nurolorn design: one function per mechanism, 64-bit torch on the
CPU, whole sequences at once (the recurrence token by token).  It shares no code with the engine; the
tests compare the engine with it.

``config`` is the config.json dictionary, ``w`` maps checkpoint tensor names to tensors.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, weight, groups, eps):
    """``groups`` equal runs of neighbours, each over its own root mean square; one weight per element."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * weight


def rotate_neighbours(x, positions, dims, base):
    """x [T, H, D]: dims 2i and 2i+1 of the first ``dims`` form a pair; the rest pass."""
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def silu(z):
    return z * torch.sigmoid(z)


def causal_softmax(scores, window=None):
    """scores [H, T, T] (query, key): softmax over the keys a query sees (``window``: the last that many)."""
    T = scores.shape[-1]
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = back >= 0
    if window is not None:
        seen = seen & (back < window)
    return torch.softmax(scores.masked_fill(~seen[None], float("-inf")), -1)


def latent_attention(h, w, p, m, eps):
    """h [T, width]; tensors ``p + name``; ``m`` the mixer's configuration."""
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    q_plain, q_rot = q[..., :d], rotate_neighbours(q[..., d:], pos, m["rot"]["dims"], m["rot"]["base"])
    kv = h @ w[p + "dkv"].T
    c = unit_rms(kv[:, :rank], eps) * w[p + "dkv.norm"]
    k_rot = rotate_neighbours(kv[:, None, rank:], pos, m["rot"]["dims"], m["rot"]["base"])[:, 0]
    k_plain = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    scores = (torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", causal_softmax(scores), v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def slopes(heads):
    """The distance bias of each head per token of distance."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).view(T, H, d), eps)
    k = unit_rms((h @ w[p + "k"].T).view(T, G, d), eps).repeat_interleave(H // G, 1)
    v = (h @ w[p + "v"].T).view(T, G, dv).repeat_interleave(H // G, 1)
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(F64)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] - slopes(H)[:, None, None] * back
    o = torch.einsum("hij,jhd->ihd", causal_softmax(scores, m["mask"]["size"] if m.get("mask") else None), v)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def mingru(h, w, p, m, eps):
    z = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros(m["width"], dtype=F64)
    rows = []
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        rows.append(S)
    return (torch.stack(rows) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_ff(h, w, p):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


MIXERS = {"latent_attention": latent_attention, "mingru": mingru, "attention": attention}


def layer(x, w, i, spec, config):
    p, eps, groups, m = f"l{i}.", config["norm"]["eps"], config["norm"].get("groups", 1), config.get("residual_mult", 1.0)
    x = x + m * MIXERS[spec["type"]](grouped_norm(x, w[p + "norm1"], groups, eps), w, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        x = x + m * dense_ff(grouped_norm(x, w[p + "norm2"], groups, eps), w, p + "mlp.")
    return x


def layer_runs(config):
    """The layers in the order they run, as (layer index, the pass it starts or None)."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(config, weights, tokens, taps=None):
    """Logits [T, vocab] of one sequence (64-bit).  ``taps``: a list that receives the stream after every
    layer run."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for i, start in layer_runs(config):
        if start is not None:
            if start > 0:
                x = x + x0
            x = x + w["loop.step"][start]
        x = layer(x, w, i, config["layers"][i], config)
        if taps is not None:
            taps.append(x.clone())
    y = grouped_norm(x, w["final.norm"], config["norm"].get("groups", 1), config["norm"]["eps"])
    return (y @ w["head"].T) * config.get("logit_scale", 1.0)


def tensor_shapes(config):
    """Checkpoint tensor name -> shape, for a configuration dictionary."""
    W = config["width"]
    out = {"embed": (config["vocab"], W), "head": (config["vocab"], W), "final.norm": (W,)}
    if config.get("loop"):
        out["loop.step"] = (config["loop"]["times"], W)
    for i, spec in enumerate(config["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        out[p + "norm1"] = (W,)
        if spec["type"] == "mingru":
            n = m["width"]
            out.update({p + "mix.z": (n, W), p + "mix.z.b": (n,), p + "mix.x": (n, W), p + "mix.x.b": (n,),
                        p + "mix.g": (n, W), p + "mix.o": (W, n)})
        elif spec["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * dv, W), p + "mix.o": (W, H * dv)})
        else:
            H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({p + "mix.q": (H * (d + r), W), p + "mix.dkv": (rank + r, W), p + "mix.dkv.norm": (rank,),
                        p + "mix.uk": (H * d, rank), p + "mix.uv": (H * dv, rank), p + "mix.g": (H * dv, W),
                        p + "mix.o": (W, H * dv)})
        if spec.get("mlp") is not None:
            ff = spec["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(config, seed, gain=1.0):
    """bfloat16 tensors of a size that keeps activations of order one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        x = torch.randn(shape, generator=g)
        if name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.2 * x
        elif name.endswith("z.b"):
            t = x - 2.0                         # forget slowly: what a state has taken in stays for some tokens
        elif name.endswith("x.b"):
            t = 0.5 * x
        elif name == "loop.step":
            t = 0.5 * x
        elif name == "embed":
            t = x
        else:
            t = gain * x / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
