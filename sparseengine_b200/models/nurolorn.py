"""Nurolorn: a decoder-only design whose ``config.json`` lists its layers one by one, some of which run
several times in a row.

Every layer is pre-norm over a 32-bit stream: ``x <- x + m * mixer(norm1(x))`` and, where the layer has a
feed-forward, ``x <- x + m * ff(norm2(x))`` with ``m = residual_mult``.  The norms are RMS norms in
``norm.groups`` equal parts of the vector, each over its own root mean square.  A layer's mixer is one of

* ``latent_attention``: softmax attention over a cached latent (``parts.latent_attention``) with
  queries straight from the input, neighbouring dims rotated in pairs, all earlier keys visible, and a
  sigmoid gate on the concatenated heads;
* ``mingru``: a gated running average per channel (``parts.recurrent.MinGRUMixer``);
* ``attention``: grouped-query attention over a sliding window (``parts.attention``), q and k over
  their root mean square per head, no rotation; a distance bias: head h of H loses
  ``2 ** (-8 (h + 1) / H)`` per token between query and key.

The feed-forward is ungated with a squared relu.  ``loop``: layers ``start .. stop-1`` run ``times`` times
in a row with the same weights, each pass with a cache or state of its own; before a pass's first layer
the embedding output joins the stream (not before the first pass), then row t of ``loop.step``.  The final
norm is the layers' norm; the logits are multiplied by ``logit_scale``.

Tensor names: ``embed``, ``head``, ``final.norm``, ``loop.step``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``,
``l<i>.mlp.up|down``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from ..config.registry import register_architecture
from ..config.specs import (AttentionSpec, LatentAttentionSpec, LayerSpec, MinGRUSpec, ModelSpec, PlainMLPSpec,
                            RMSNormSpec, RotarySpec, ScheduleEntry, Source)

ARCHITECTURE = "Nurolorn"
MIXER_TYPES = ("latent_attention", "mingru", "attention")
DEFAULT_MAX_POSITION = 1 << 20      # the design has no position table; the cache manager wants a bound

_MIXER_KEYS = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank"), "mingru": ("width",),
               "attention": ("heads", "kv_heads", "dim", "vdim")}


@dataclass(frozen=True)
class NurolornConfig:
    vocab: int
    width: int
    layers: tuple                      # of dicts {"type", "mixer", "mlp"} as in config.json (validated)
    loop: Optional[tuple]              # (start, stop, times) or None
    norm_eps: float
    norm_groups: int
    residual_mult: float
    logit_scale: float
    max_position: int

    @classmethod
    def from_dict(cls, raw: dict) -> "NurolornConfig":
        problems = []
        for key in ("vocab", "width", "layers"):
            if raw.get(key) is None:
                problems.append(f"missing key {key!r}")
        layers = raw.get("layers") or []
        if not isinstance(layers, list) or not layers:
            problems.append("'layers' must be a non-empty list")
            layers = []
        for i, layer in enumerate(layers):
            kind, m = layer.get("type"), layer.get("mixer") or {}
            if kind not in MIXER_TYPES:
                problems.append(f"layer {i}: unknown mixer type {kind!r} (known: {', '.join(MIXER_TYPES)})")
                continue
            missing = [k for k in _MIXER_KEYS[kind] if m.get(k) is None]
            if missing:
                problems.append(f"layer {i} ({kind}): missing mixer keys {missing}")
            rot = m.get("rot")
            if kind == "latent_attention" and m.get("rot_dim") and (rot or {}).get("base") is None:
                problems.append(f"layer {i}: 'rot' needs 'base'")
            mask = m.get("mask")
            if mask is not None and mask.get("size") is None:
                problems.append(f"layer {i}: 'mask' needs 'size'")
            mlp = layer.get("mlp")
            if mlp is not None and (mlp.get("kind", "dense") != "dense" or mlp.get("ff") is None):
                problems.append(f"layer {i}: the feed-forward must be 'dense' with 'ff', or null")
        loop = raw.get("loop")
        if loop is not None:
            try:
                loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
                if not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
                    problems.append(f"loop {loop} does not fit {len(layers)} layers")
            except (KeyError, TypeError, ValueError):
                problems.append("'loop' needs integer 'start', 'stop' and 'times'")
        norm = raw.get("norm") or {}
        groups = int(norm.get("groups") or 1)
        if raw.get("width") is not None and (groups < 1 or int(raw["width"]) % groups):
            problems.append(f"norm.groups {groups} does not divide width {raw['width']}")
        if problems:
            raise ValueError("Nurolorn config.json cannot be used: " + "; ".join(problems))

        def number(key, default):
            return float(default if raw.get(key) is None else raw[key])
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), layers=tuple(layers), loop=loop,
                   norm_eps=float(norm.get("eps", 1e-6)), norm_groups=groups, residual_mult=number("residual_mult", 1.0),
                   logit_scale=number("logit_scale", 1.0), max_position=int(raw.get("max_position", DEFAULT_MAX_POSITION)))


def _rows(prefix, parts):
    """Sources that stack the named tensors along the first dimension."""
    out, at = [], 0
    for name, n in parts:
        out.append(Source(prefix + name, ((at, n),)))
        at += n
    return tuple(out)


def _latent_attention(cfg, m, p):
    H, d, r, dv, rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    window = (m.get("mask") or {}).get("size")
    position = None
    if r > 0:
        rot = m["rot"]
        position = RotarySpec(rotary_dim=int(rot["dims"]) if rot.get("dims") is not None else r, theta=float(rot["base"]),
                              pairing="interleaved")
    spec = LatentAttentionSpec(hidden_size=cfg.width, num_heads=H, head_dim=d, rot_dim=r, v_head_dim=dv, q_rank=0, kv_rank=rank,
                               scale=float(m.get("scale", (d + r) ** -0.5)), window=int(window) if window else None,
                               position=position, norm_eps=cfg.norm_eps, output_gate=True)
    sources = {"mixer.in_proj": _rows(p, (("q", H * (d + r)), ("dkv", rank + r), ("g", H * dv))),
               "mixer.kv_norm": (Source(p + "dkv.norm"),), "mixer.uk": (Source(p + "uk"),), "mixer.uv": (Source(p + "uv"),),
               "mixer.o": (Source(p + "o"),)}
    return spec, sources


def _mingru(cfg, m, p):
    n = int(m["width"])
    return MinGRUSpec(hidden_size=cfg.width, width=n), {
        "mixer.in_proj": _rows(p, (("z", n), ("x", n), ("g", n))), "mixer.gate_bias": _rows(p, (("z.b", n), ("x.b", n))),
        "mixer.o": (Source(p + "o"),)}


def distance_slopes(heads: int) -> tuple:
    """What each head's score loses per token of distance: a geometric row that ends at 2^-8."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _attention(cfg, m, p):
    H, G, d, dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    window = (m.get("mask") or {}).get("size")
    spec = AttentionSpec(hidden_size=cfg.width, num_heads=H, num_kv_heads=G, head_dim=d, scale=float(m.get("scale", d ** -0.5)),
                         qk_norm="per_head_unit", qk_norm_eps=cfg.norm_eps, window=int(window) if window else None,
                         prep="general", v_head_dim=None if dv == d else dv, distance_slopes=distance_slopes(H))
    return spec, {"mixer.qkv": _rows(p, (("q", H * d), ("k", G * d), ("v", G * dv))), "mixer.o": (Source(p + "o"),)}


_MIXERS = {"latent_attention": _latent_attention, "mingru": _mingru, "attention": _attention}


def layer_order(num_layers: int, loop) -> list:
    """The visits in the order they run: ``(layer, the pass it starts or None)``."""
    if loop is None:
        return [(i, None) for i in range(num_layers)]
    start, stop, times = loop
    runs = [(i, None) for i in range(start)]
    for t in range(times):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, num_layers)]


def build_nurolorn(cfg: NurolornConfig) -> ModelSpec:
    norm = RMSNormSpec(size=cfg.width, eps=cfg.norm_eps, groups=cfg.norm_groups)
    layers = []
    for i, layer in enumerate(cfg.layers):
        mixer, sources = _MIXERS[layer["type"]](cfg, layer["mixer"], f"l{i}.mix.")
        sources["mixer_norm.weight"] = (Source(f"l{i}.norm1"),)
        ff = None
        if layer.get("mlp") is not None:
            ff = PlainMLPSpec(hidden_size=cfg.width, intermediate_size=int(layer["mlp"]["ff"]), activation="relu2")
            sources.update({"feed_forward.up": (Source(f"l{i}.mlp.up"),), "feed_forward.down": (Source(f"l{i}.mlp.down"),),
                            "feed_forward_norm.weight": (Source(f"l{i}.norm2"),)})
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, mixer_norm=norm, feed_forward_norm=norm if ff is not None else None,
                                arrangement="pre_norm_stream", residual_scale=cfg.residual_mult, sources=sources))
    # every visit has a cache or state of its own, also a layer's second and third pass
    order = [ScheduleEntry(layer=i, add_embedding=t is not None and t > 0, step_vector=t)
             for i, t in layer_order(len(layers), cfg.loop)]
    return ModelSpec(architecture=ARCHITECTURE, hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=cfg.max_position,
                     layers=layers, order=order, final_norm=norm, final_norm_source="final.norm", embed_source="embed",
                     head_source="head", logit_scale=cfg.logit_scale, residual_stream="float32",
                     step_source="loop.step" if cfg.loop is not None else None,
                     step_count=cfg.loop[2] if cfg.loop is not None else 0)


register_architecture(ARCHITECTURE, NurolornConfig, build_nurolorn)
