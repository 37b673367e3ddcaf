"""The Nurolorn design without a GPU: the plain implementation's own pieces on cases worked by hand, the
premises of the GPU tests (that a window one key off, a missing or reversed distance bias, a lost state, a
forgotten pass vector and the like show in the plain logits), what the configuration reader accepts,
refuses and makes of a configuration, and the sizes the parts refuse."""
import copy

import numpy as np
import pytest
import torch

import plain_nurolorn as pn
import sparseengine_b200.models  # noqa: F401
import trace_util as tu
from sparseengine_b200.config.registry import load_model_spec
from sparseengine_b200.engine.model import Model
from test_nurolorn_gpu import CONFIGS, att, config, dense, far_key_model, gru, lat, sharp_window_model, slow_state_model

F64 = torch.float64


def moved(a, b, rows=slice(None)):
    """Root mean square of the difference of some rows, in units of the first's."""
    return float((a[rows] - b[rows]).pow(2).mean().sqrt() / a.pow(2).mean().sqrt())


def test_the_plain_mechanisms_are_what_they_claim():
    # neighbours form pairs, the rest passes
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    y = pn.rotate_neighbours(x, torch.tensor([3]), 4, 100.0)
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(y[0, 0].numpy(), [np.cos(a0) - 2 * np.sin(a0), 2 * np.cos(a0) + np.sin(a0),
                                         3 * np.cos(a1) - 4 * np.sin(a1), 4 * np.cos(a1) + 3 * np.sin(a1), 5.0])
    # two groups of two: each over its own root mean square
    n = pn.grouped_norm(torch.tensor([3.0, 4.0, 1.0, -1.0], dtype=F64), torch.tensor([1.0, 1.0, 2.0, 2.0], dtype=F64), 2, 0.0)
    assert np.allclose(n.numpy(), [3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 2.0, -2.0])
    # the row of slopes, and a head count that is no power of two
    assert pn.slopes(4).tolist() == [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8]
    assert np.allclose(pn.slopes(3).tolist(), [2 ** (-8 / 3), 2 ** (-16 / 3), 2 ** -8])
    # a window of two: the query sees itself and the key before it
    p = pn.causal_softmax(torch.zeros(1, 3, 3, dtype=F64), 2)[0]
    assert np.allclose(p.numpy(), [[1, 0, 0], [0.5, 0.5, 0], [0, 0.5, 0.5]])
    # one channel of the recurrence by hand: an open gate takes the candidate, a closed one keeps the state
    w = {"z": torch.tensor([[100.0]]), "z.b": torch.tensor([-50.0]), "x": torch.tensor([[2.0]]), "x.b": torch.tensor([0.0]),
         "g": torch.tensor([[1.0]]), "o": torch.tensor([[1.0]])}
    h = torch.tensor([[1.0], [0.0], [-1.0]], dtype=F64)
    out = pn.mingru(h, {k: v.to(F64) for k, v in w.items()}, "", {"width": 1}, 0.0)
    sig = 1 / (1 + np.exp(-1.0))
    assert np.allclose(out[:, 0].numpy(), [2.5 * sig, 0.0, -2.5 * (1 - sig)])


def test_layer_order_and_what_passes_add():
    cfg = config(8, 10, [gru(4), gru(4), gru(4)], loop=(1, 2, 3))
    assert pn.layer_runs(cfg) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]
    _, spec = load_model_spec(cfg)
    assert [(e.layer, e.add_embedding, e.step_vector) for e in spec.order] == [
        (0, False, None), (1, False, 0), (1, True, 1), (1, True, 2), (2, False, None)]
    # the first pass takes the vector alone, later ones the embedding output too
    w = pn.random_weights(cfg, 3)
    ref = pn.forward(cfg, w, [1, 2, 3])
    other = dict(w)
    other["loop.step"] = w["loop.step"].clone()
    other["loop.step"][0] += w["embed"][4]
    assert moved(ref, pn.forward(cfg, other, [1, 2, 3])) > 0.01


@pytest.mark.parametrize("dim", [16, 64, 128])
def test_the_plain_window_matters(dim):
    cfg, w = sharp_window_model(37, dim)
    toks = tu.random_prompt(80, 150, 60)
    ref = pn.forward(cfg, w, toks)
    for other in (36, 38):
        c = copy.deepcopy(cfg)
        c["layers"][0]["mixer"]["mask"]["size"] = other
        d = pn.forward(c, w, toks)
        assert float((d - ref)[:36].abs().max()) < 1e-9             # the first tokens see everything either way
        rows = (d - ref)[40:].pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
        assert float(rows.max()) > 0.35                             # beyond the widest bound of the GPU test


def test_the_plain_distance_bias_matters(monkeypatch):
    cfg = CONFIGS["wide"]
    w = pn.random_weights(cfg, 5)
    toks = tu.random_prompt(cfg["vocab"], 70, 2)
    ref = pn.forward(cfg, w, toks)
    real = pn.slopes
    for planted in (lambda n: real(n) * 0.0, lambda n: real(n).flip(0), lambda n: real(n) * 0.5):
        monkeypatch.setattr(pn, "slopes", planted)
        assert moved(ref, pn.forward(cfg, w, toks)) > 0.02
        monkeypatch.setattr(pn, "slopes", real)


def test_the_plain_far_keys_matter(monkeypatch):
    """Without the first page of 16 keys the rows near position 400 move."""
    cfg, w = far_key_model()
    toks = tu.random_prompt(80, 430, 80)
    ref = pn.forward(cfg, w, toks)
    real = pn.causal_softmax

    def blind(scores, window=None):
        scores = scores.clone()
        scores[:, 16:, :16] = float("-inf")
        return real(scores, window)
    monkeypatch.setattr(pn, "causal_softmax", blind)
    rows = (pn.forward(cfg, w, toks) - ref)[380:].pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(rows.max()) > 0.35


def test_the_plain_state_matters():
    """What a first token leaves in the state still shows a thousand tokens later, and a state that is lost at
    position 300 does so by far more than the bfloat16 bound."""
    cfg, w = slow_state_model()
    toks = tu.random_prompt(64, 1100, 70)
    ref = pn.forward(cfg, w, toks)
    changed = [(toks[0] + 1) % 64] + toks[1:]
    assert moved(ref, pn.forward(cfg, w, changed), slice(400, None)) > 1e-4
    lost = pn.forward(cfg, w, toks[300:])
    rows = (lost - ref[300:]).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(rows[:50].max()) > 0.15


def test_the_plain_constants_matter():
    """Groups, factors, eps and the pass's additions of the test models: leaving one out shows."""
    for name, change in (("hybrid", lambda c, w: c["norm"].__setitem__("groups", 1)), ("odd", lambda c, w: c["norm"].__setitem__("groups", 1)),
                         ("hybrid", lambda c, w: c.__setitem__("residual_mult", 1.0)), ("middle", lambda c, w: w["loop.step"].zero_()),
                         ("wide", lambda c, w: [w.__setitem__(k, torch.zeros_like(v)) for k, v in list(w.items()) if k.endswith("mix.g")])):
        cfg, w = copy.deepcopy(CONFIGS[name]), pn.random_weights(CONFIGS[name], 8)
        toks = tu.random_prompt(cfg["vocab"], 40, 3)
        ref = pn.forward(cfg, w, toks)
        w2 = {k: v.clone() for k, v in w.items()}
        change(cfg, w2)
        assert moved(ref, pn.forward(cfg, w2, toks)) > 0.02, name


def test_what_the_reader_makes_of_a_configuration():
    cfg = config(64, 100, [lat(4, 8, 6, 12, 20, scale=0.3, base=777.0, mlp=dense(48)), gru(40),
                           att(6, 2, 16, 10, 13, scale=0.9, mlp=dense(32))], loop=(0, 3, 2), groups=4, eps=3e-4, mult=0.4, logit_scale=2.5)
    typed, spec = load_model_spec(cfg)
    la, gr, at = (layer.mixer for layer in spec.layers)
    assert (la.num_heads, la.head_dim, la.rot_dim, la.v_head_dim, la.kv_rank, la.q_rank) == (4, 8, 6, 12, 20, 0)
    assert la.scale == 0.3 and la.window is None and not la.sink and la.output_gate and la.norm_eps == 3e-4
    assert (la.position.rotary_dim, la.position.theta, la.position.pairing) == (6, 777.0, "interleaved")
    assert gr.width == 40
    assert at.window == 13 and at.scale == 0.9 and at.qk_norm == "per_head_unit" and at.qk_norm_eps == 3e-4 and at.value_dim == 10
    assert at.position is None and list(at.distance_slopes) == pn.slopes(6).tolist()
    assert spec.logit_scale == 2.5 and spec.final_norm.groups == 4 and all(layer.residual_scale == 0.4 for layer in spec.layers)
    assert spec.layers[1].feed_forward is None and spec.layers[2].feed_forward.activation == "relu2"
    model = Model(spec, torch.bfloat16)
    names = {s.name for p in model.params() for s in p.sources}
    assert names == set(pn.tensor_shapes(cfg))
    # two passes of three layers: two latent groups of cache layers, two windows', two states
    assert [(kv.layout, n) for kv, n in model.layout.groups] == [("latent", 2), ("kv", 2)] and len(model.layout.states) == 2
    # what may be left out
    bare = {k: v for k, v in cfg.items() if k not in ("loop", "residual_mult", "logit_scale")}
    bare["norm"] = {"eps": 1e-6}
    _, spec = load_model_spec(bare)
    assert spec.step_source is None and spec.logit_scale == 1.0 and spec.final_norm.groups == 1 and spec.layers[0].residual_scale == 1.0
    bare["loop"] = None
    load_model_spec(bare)


def test_what_a_configuration_must_have():
    good = config(32, 40, [lat(2, 8, 8, 8, 8, mlp=dense(16)), gru(8), att(2, 1, 8, 8, 5)], loop=(0, 1, 2), groups=2)
    load_model_spec(good)
    for breaker, word in ((lambda c: c["layers"][0].__setitem__("type", "retention"), "unknown mixer type"),
                          (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
                          (lambda c: c["layers"][0]["mixer"].pop("rot"), "base"),
                          (lambda c: c["layers"][1]["mixer"].pop("width"), "width"),
                          (lambda c: c["layers"][2]["mixer"].__setitem__("mask", {}), "size"),
                          (lambda c: c["loop"].__setitem__("stop", 4), "does not fit"),
                          (lambda c: c["norm"].__setitem__("groups", 3), "does not divide"),
                          (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "dense"),
                          (lambda c: c.pop("vocab"), "vocab")):
        bad = copy.deepcopy(good)
        breaker(bad)
        with pytest.raises(ValueError, match=word):
            load_model_spec(bad)


def test_how_many_ctas_share_a_prompts_recurrence():
    from sparseengine_b200.csrc import ops
    plan = lambda *a: ops.min_gru_plan(*a, sms=148)
    assert [plan(1, 2048, n) for n in (1, 128, 129, 512, 513, 4096)] == [1, 1, 2, 4, 8, 8]
    assert plan(1, 4096, 2048) == 4 and plan(4, 4096, 2048) == 1 and plan(64, 64, 2048) == 4 and plan(1, 1, 10 ** 6) == 8


def test_what_the_parts_refuse():
    from sparseengine_b200.config.specs import (AttentionSpec, LatentAttentionSpec, LayerSpec, MinGRUSpec, ModelSpec, PlainMLPSpec,
                                                RMSNormSpec, RotarySpec, ScheduleEntry)
    from sparseengine_b200.csrc import ops
    from sparseengine_b200.parts.base import make_mixer, make_norm
    with pytest.raises(ValueError, match="groups"):
        make_norm(RMSNormSpec(size=64, groups=5), torch.float32)
    most = ops.LIMITS["rmsnorm_stream_max_groups"]
    make_norm(RMSNormSpec(size=2 * most, groups=most), torch.float32)
    with pytest.raises(ValueError, match=str(most)):
        make_norm(RMSNormSpec(size=4 * most, groups=2 * most), torch.float32)
    ok = dict(hidden_size=64, num_heads=4, num_kv_heads=2, head_dim=16, scale=0.25, prep="general")
    make_mixer(AttentionSpec(**ok, distance_slopes=(0.5, 0.25, 0.1, 0.0)), torch.float32)
    with pytest.raises(ValueError, match="one slope per query head"):
        make_mixer(AttentionSpec(**ok, distance_slopes=(0.5, 0.25)), torch.float32)
    with pytest.raises(ValueError, match="prep='general'"):
        make_mixer(AttentionSpec(**dict(ok, prep="rotary"), qk_norm="per_head_unit"), torch.float32)
    lat_ok = dict(hidden_size=64, num_heads=2, head_dim=16, rot_dim=16, v_head_dim=16, kv_rank=8, scale=0.1)
    make_mixer(LatentAttentionSpec(**lat_ok, q_rank=0, output_gate=True, position=RotarySpec(rotary_dim=16, pairing="interleaved")), torch.float32)
    with pytest.raises(ValueError, match="q_rank 0"):
        make_mixer(LatentAttentionSpec(**lat_ok, q_rank=8, output_gate=True), torch.float32)
    with pytest.raises(ValueError, match="pairs"):
        make_mixer(LatentAttentionSpec(**lat_ok, position=RotarySpec(rotary_dim=16, pairing="interleaved_to_split_half")), torch.float32)
    with pytest.raises(ValueError, match="positive"):
        make_mixer(MinGRUSpec(hidden_size=64, width=0), torch.float32)
    # norms in groups and what a pass adds go with the pre-norm stream only
    norm, ff, gm = RMSNormSpec(size=64, groups=2), PlainMLPSpec(hidden_size=64, intermediate_size=8), MinGRUSpec(hidden_size=64, width=8)
    sources = {"mixer.in_proj": (), "mixer.gate_bias": (), "mixer.o": (), "mixer_norm.weight": (), "feed_forward_norm.weight": (),
               "feed_forward.up": (), "feed_forward.down": ()}

    def spec(norm, arrangement, entry, **kw):
        layer = LayerSpec(mixer=gm, feed_forward=ff, mixer_norm=norm, feed_forward_norm=norm, arrangement=arrangement, sources=sources)
        return ModelSpec(architecture="t", hidden_size=64, vocab_size=8, max_position=64, layers=[layer], order=[entry], final_norm=norm, **kw)
    Model(spec(norm, "pre_norm_stream", ScheduleEntry(0, step_vector=0), residual_stream="float32", step_source="s", step_count=1), torch.float32)
    with pytest.raises(ValueError, match="norms in groups"):
        Model(spec(norm, "pre_norm", ScheduleEntry(0)), torch.float32)
    with pytest.raises(ValueError, match="add_embedding"):
        Model(spec(RMSNormSpec(size=64), "pre_norm", ScheduleEntry(0, add_embedding=True)), torch.float32)
    with pytest.raises(ValueError, match="names a row"):
        Model(spec(norm, "pre_norm_stream", ScheduleEntry(0, step_vector=1), residual_stream="float32", step_source="s", step_count=1), torch.float32)
