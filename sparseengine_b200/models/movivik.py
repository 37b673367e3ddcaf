"""Movivik: a decoder-only design whose ``config.json`` lists its layers one by one; a layer may use an
earlier layer's weights.

The residual stream is 32-bit, with RMS norms before and after each sublayer: ``x <- x + norm1b(mixer(norm1(x)))``
and, where the layer has a feed-forward, ``x <- x + norm2b(ff(norm2(x)))``.  A layer's mixer is one of

* ``attention``: grouped-query attention (``parts.attention``, general preparation) with biases on q, k and
  v, neighbouring dims rotated in pairs (YaRN frequencies, cos and sin times their factor), keys of the
  query's own chunk only, values of a head size of their own, and one output gate per head, ``sigmoid(W_g h)``;
* ``parallel``: two mixers on the same input (``parts.parallel``), each result normed over the width with a weight
  of its own, then half their sum.  Left: grouped-query attention over all earlier keys, split halves
  rotated, q and k over their root mean square per head after the rotation, gated per head.  Right: lightning
  attention (``parts.recurrent.RetentionMixer``): silu on q, k and v, a fixed decay per head, the
  concatenated heads normed together and multiplied by ``sigmoid(W_g h)``.

The feed-forward is dense and gated by a tanh-form gelu.  A layer that names another with ``weights_of`` runs that
layer's mixer, feed-forward and norms with a cache and state of its own.

Tensor names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.q|k|v[.b]|g|o`` or
``l<i>.mix.left.q|k|v|g|o|out`` and ``l<i>.mix.right.q|k|v|g|norm|o|out``, ``l<i>.mlp.gate|up|down``.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..config.registry import register_architecture
from ..config.specs import (AttentionSpec, DenseMLPSpec, LayerSpec, ModelSpec, ParallelMixerSpec, RetentionSpec,
                            RMSNormSpec, RotarySpec, ScheduleEntry, Source)

ARCHITECTURE = "Movivik"
MIXER_TYPES = ("attention", "parallel")
DEFAULT_MAX_POSITION = 1 << 20      # the design has no position table; the cache manager wants a bound

_ATTENTION_KEYS = ("heads", "kv_heads", "dim", "vdim")
_RIGHT_KEYS = ("heads", "dim", "vdim", "decay")
_SCALING_KEYS = ("factor", "original", "fast", "slow")


def _attention_problems(m, what) -> list:
    problems = []
    missing = [k for k in _ATTENTION_KEYS if m.get(k) is None]
    if missing:
        return [f"{what}: missing mixer keys {missing}"]
    if int(m["kv_heads"]) <= 0 or int(m["heads"]) % int(m["kv_heads"]):
        problems.append(f"{what}: 'heads' must be a multiple of 'kv_heads'")
    rot = m.get("rot")
    if rot is not None and (rot.get("dims") is None or (rot["dims"] and rot.get("base") is None)):
        problems.append(f"{what}: 'rot' needs 'dims' and 'base'")
    sc = (rot or {}).get("scaling")
    if sc is not None and any(sc.get(k) is None for k in _SCALING_KEYS):
        problems.append(f"{what}: 'rot.scaling' needs {', '.join(_SCALING_KEYS)}")
    if m.get("mask") is not None and not m["mask"].get("size"):
        problems.append(f"{what}: 'mask' needs a positive 'size'")
    return problems


@dataclass(frozen=True)
class MovivikConfig:
    vocab: int
    width: int
    layers: tuple                      # of dicts {"type", "mixer", "mlp"} as in config.json (validated)
    weights: tuple                     # per layer: the layer whose weights it uses (its own index: its own)
    norm_eps: float
    max_position: int

    @classmethod
    def from_dict(cls, raw: dict) -> "MovivikConfig":
        problems = []
        for key in ("vocab", "width", "layers"):
            if raw.get(key) is None:
                problems.append(f"missing key {key!r}")
        layers = raw.get("layers") or []
        if not isinstance(layers, list) or not layers:
            problems.append("'layers' must be a non-empty list")
            layers = []
        weights = []
        for i, layer in enumerate(layers):
            kind, m, what = layer.get("type"), layer.get("mixer") or {}, f"layer {i}"
            j = layer.get("weights_of")
            weights.append(i)
            if j is not None:
                seen = {i}
                while j is not None and 0 <= int(j) < len(layers) and int(j) not in seen:
                    seen.add(int(j))
                    weights[i], j = int(j), layers[int(j)].get("weights_of")
                if j is not None:
                    problems.append(f"{what}: 'weights_of' does not lead to a layer with weights of its own")
            if kind not in MIXER_TYPES:
                problems.append(f"{what}: unknown mixer type {kind!r} (known: {', '.join(MIXER_TYPES)})")
                continue
            if kind == "attention":
                problems += _attention_problems(m, what)
            else:
                problems += _attention_problems(m.get("left") or {}, what + " (left)")
                right = m.get("right") or {}
                missing = [k for k in _RIGHT_KEYS if right.get(k) is None]
                if missing:
                    problems.append(f"{what} (right): missing mixer keys {missing}")
                elif len(right["decay"]) != int(right["heads"]):
                    problems.append(f"{what} (right): 'decay' needs one entry per head")
            mlp = layer.get("mlp")
            if mlp is not None and (mlp.get("kind", "dense") != "dense" or mlp.get("ff") is None):
                problems.append(f"{what}: the feed-forward must be 'dense' with 'ff', or null")
        if not problems:
            for i, j in enumerate(weights):
                a, b = layers[i], layers[j]
                if any(a.get(k) != b.get(k) for k in ("type", "mixer", "mlp")):
                    problems.append(f"layer {i}: its entry differs from that of layer {j}, whose weights it uses")
        if problems:
            raise ValueError("Movivik config.json cannot be used: " + "; ".join(problems))
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), layers=tuple(layers), weights=tuple(weights),
                   norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)),
                   max_position=int(raw.get("max_position", DEFAULT_MAX_POSITION)))


def _rows(prefix, parts):
    """Sources that stack the named tensors along the first dimension."""
    out, at = [], 0
    for name, n in parts:
        out.append(Source(prefix + name, ((at, n),)))
        at += n
    return tuple(out)


def _rotary(m, pairing):
    rot = m.get("rot")
    if rot is None or int(rot["dims"]) == 0:
        return None
    sc = rot.get("scaling")
    scaling = None
    if sc is not None:
        scaling = tuple(sorted({"rope_type": "yarn", "factor": float(sc["factor"]), "beta_fast": float(sc["fast"]),
                                "beta_slow": float(sc["slow"]), "original_max_position_embeddings": float(sc["original"])}.items()))
    return RotarySpec(rotary_dim=int(rot["dims"]), theta=float(rot["base"]), pairing=pairing, frequency_scaling=scaling)


def _attention(cfg, m, p, part, left):
    """The attention of a layer of its own, or (``left``) the left branch of a parallel mixer."""
    H, G, d, dv = (int(m[k]) for k in _ATTENTION_KEYS)
    mask = m.get("mask")
    spec = AttentionSpec(hidden_size=cfg.width, num_heads=H, num_kv_heads=G, head_dim=d, v_head_dim=None if dv == d else dv,
                         scale=float(m["scale"]) if m.get("scale") is not None else d ** -0.5,
                         qk_norm="per_head_unit" if left else None, qk_norm_eps=cfg.norm_eps,
                         chunk=int(mask["size"]) if mask else None, prep="general", bias=not left, output_bias=False,
                         position=_rotary(m, "split_half" if left else "interleaved"), output_gate="head")
    parts = (("q", H * d), ("k", G * d), ("v", G * dv))
    sources = {part + "qkv": _rows(p, parts + (("g", H),)), part + "o": (Source(p + "o"),)}
    if not left:
        sources[part + "qkv_bias"] = _rows(p, tuple((n + ".b", c) for n, c in parts))
    return spec, sources


def _lightning(cfg, m, p, part):
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    spec = RetentionSpec(hidden_size=cfg.width, num_heads=H, head_dim=d, v_head_dim=dv, decays=tuple(float(g) for g in m["decay"]),
                         norm_eps=cfg.norm_eps, activation="silu", k_scale=1.0, output_norm="joint")
    return spec, {part + "in_proj": _rows(p, (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv))),
                  part + "norm_w": (Source(p + "norm"),), part + "o": (Source(p + "o"),)}


def _mixer(cfg, layer, p):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return _attention(cfg, m, p, "mixer.", left=False)
    left, sources = _attention(cfg, m["left"], p + "left.", "mixer.left_", left=True)
    right, more = _lightning(cfg, m["right"], p + "right.", "mixer.right_")
    sources.update(more)
    sources.update({"mixer.left_out_norm": (Source(p + "left.out"),), "mixer.right_out_norm": (Source(p + "right.out"),)})
    return ParallelMixerSpec(hidden_size=cfg.width, branches=(left, right), scales=(0.5, 0.5), names=("left", "right"),
                             output_norms=True, norm_eps=cfg.norm_eps), sources


def build_movivik(cfg: MovivikConfig) -> ModelSpec:
    norm = RMSNormSpec(size=cfg.width, eps=cfg.norm_eps)
    layers, place = [], {}
    for i, layer in enumerate(cfg.layers):
        if cfg.weights[i] != i:
            continue
        mixer, sources = _mixer(cfg, layer, f"l{i}.mix.")
        sources.update({"mixer_norm.weight": (Source(f"l{i}.norm1"),), "mixer_post_norm.weight": (Source(f"l{i}.norm1b"),)})
        ff, extra = None, {"mixer_post_norm": norm}
        if layer.get("mlp") is not None:
            n = int(layer["mlp"]["ff"])
            ff = DenseMLPSpec(hidden_size=cfg.width, intermediate_size=n, activation="gelu_tanh")
            extra["feed_forward_post_norm"] = norm
            sources.update({"feed_forward.w13": (Source(f"l{i}.mlp.gate", (0, (0, n))), Source(f"l{i}.mlp.up", (0, (n, n)))),
                            "feed_forward.w2": (Source(f"l{i}.mlp.down", (0,)),),
                            "feed_forward_norm.weight": (Source(f"l{i}.norm2"),),
                            "feed_forward_post_norm.weight": (Source(f"l{i}.norm2b"),)})
        place[i] = len(layers)
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, mixer_norm=norm, feed_forward_norm=norm if ff is not None else None,
                                arrangement="sandwich_norm", extra=extra, sources=sources))
    # every visit has a cache and state of its own, also one that uses another layer's weights
    order = [ScheduleEntry(layer=place[j]) for j in cfg.weights]
    return ModelSpec(architecture=ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=cfg.max_position,
                     layers=layers, order=order, final_norm=norm, final_norm_source="final.norm", embed_source="embed",
                     head_source="head", residual_stream="float32")


register_architecture(ARCHITECTURE, MovivikConfig, build_movivik)
