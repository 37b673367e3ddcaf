"""A plain, slow implementation of the Movivik design: one function per mechanism, 64-bit torch on the
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


def norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """(angle per position of each pair, factor on cos and sin)."""
    dims, base = rot["dims"], rot["base"]
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0

    def place(turns):       # the (fractional) dim that makes that many turns over the original context
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=F64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / sc["factor"] * ramp + freq * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, neighbours):
    """x [T, heads, D]: pairs (2i, 2i+1) (``neighbours``) or (i, i + dims/2) of the first ``dims`` dims."""
    dims = rot["dims"]
    freq, amp = frequencies(rot)
    ang = positions.to(F64)[:, None] * freq[None, :]
    c, s = amp * torch.cos(ang)[:, None, :], amp * torch.sin(ang)[:, None, :]
    first = slice(0, dims, 2) if neighbours else slice(0, dims // 2)
    second = slice(1, dims, 2) if neighbours else slice(dims // 2, dims)
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def visible(T, chunk=None):
    """[query, key]: keys up to the query's position, within the query's own chunk."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if chunk is not None:
        seen = seen & (i // chunk == j // chunk)
    return seen


def attend(q, k, v, scale, seen):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, 1), v.repeat_interleave(group, 1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    p = torch.softmax(scores.masked_fill(~seen[None], float("-inf")), -1)
    return torch.einsum("hij,jhd->ihd", p, v)


def head_gated(o, h, w, p):
    """Each head's output times one number, then the output projection."""
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(o.shape[0], -1) @ w[p + "o"].T


def project(h, w, p, name, heads, bias):
    y = h @ w[p + name].T
    if bias:
        y = y + w[p + name + ".b"]
    return y.view(h.shape[0], heads, -1)


def chunked_attention(h, w, p, m, eps):
    """Biases, neighbours rotated in pairs (YaRN frequencies), keys of the query's chunk only."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q = rotate(project(h, w, p, "q", H, True), pos, m["rot"], True)
    k = rotate(project(h, w, p, "k", G, True), pos, m["rot"], True)
    v = project(h, w, p, "v", G, True)
    return head_gated(attend(q, k, v, m["scale"], visible(T, m["mask"]["size"])), h, w, p)


def full_attention(h, w, p, m, eps):
    """No biases, split halves rotated, q and k over their root mean square per head after it, all earlier keys."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q = unit_rms(rotate(project(h, w, p, "q", H, False), pos, m["rot"], False), eps)
    k = unit_rms(rotate(project(h, w, p, "k", G, False), pos, m["rot"], False), eps)
    v = project(h, w, p, "v", G, False)
    return head_gated(attend(q, k, v, m["scale"], visible(T)), h, w, p)


def recurrence(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv]; returns (outputs [T, H, dv], the last state [H, d, dv])."""
    T, H, d = q.shape
    g = torch.tensor(decay, dtype=F64)[:, None, None]
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if state is None else state.clone()
    rows = []
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(rows), S


def lightning(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[p + n].T).view(T, H, -1) for n in "qkv")
    o, _ = recurrence(q, k, v, m["decay"])
    o = norm(o.reshape(T, -1), w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left = full_attention(h, w, p + "left.", m["left"], eps)
    right = lightning(h, w, p + "right.", m["right"], eps)
    return 0.5 * (norm(left, w[p + "left.out"], eps) + norm(right, w[p + "right.out"], eps))


def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"attention": chunked_attention, "parallel": parallel}


def weights_layer(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def layer(x, w, i, spec, eps):
    p = f"l{i}."
    y = MIXERS[spec["type"]](norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    x = x + norm(y, w[p + "norm1b"], eps)
    if spec.get("mlp") is not None:
        x = x + norm(dense_ff(norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
    return x


def forward(config, weights, tokens, taps=None):
    """Logits [T, vocab] of one sequence (64-bit).  ``taps``: a list that receives the stream after every
    layer."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(config["layers"]):
        x = layer(x, w, weights_layer(config, i), spec, eps)
        if taps is not None:
            taps.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T


def tensor_shapes(config):
    """Checkpoint tensor name -> shape, for a configuration dictionary."""
    W = config["width"]
    out = {"embed": (config["vocab"], W), "head": (config["vocab"], W), "final.norm": (W,)}

    def attention(p, m, bias):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
            out[p + n] = (rows, W)
            if bias:
                out[p + n + ".b"] = (rows,)
        out.update({p + "g": (H, W), p + "o": (W, H * dv)})
    for i, spec in enumerate(config["layers"]):
        if spec.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", spec["mixer"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if spec["type"] == "attention":
            attention(p + "mix.", m, True)
        else:
            attention(p + "mix.left.", m["left"], False)
            r, q = m["right"], p + "mix.right."
            qk, vv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({q + "q": (qk, W), q + "k": (qk, W), q + "v": (vv, W), q + "g": (vv, W), q + "norm": (vv,), q + "o": (W, vv),
                        p + "mix.left.out": (W,), q + "out": (W,)})
        if spec.get("mlp") is not None:
            ff = spec["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(config, seed, gain=1.0):
    """bfloat16 tensors of a size that keeps activations of order one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        x = torch.randn(shape, generator=g)
        if name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b", ".out")):
            t = 1.0 + 0.2 * x
        elif name.endswith(".b"):
            t = 0.5 * x
        elif name == "embed":
            t = x
        else:
            t = gain * x / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
