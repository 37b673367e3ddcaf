"""The Movivik design without a GPU: the plain implementation's own pieces on cases worked by hand, the premises of
the GPU tests (that a chunk one key off, a far key or a state that is lost, a missing gate, factor or norm show in
the plain logits), what the configuration reader accepts, refuses and makes of a configuration, what the cache
manager keeps of a chunk, and what the parts refuse."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_movivik as pm
import sparseengine_b200.models  # noqa: F401
import trace_util as tu
from sparseengine_b200.config.registry import load_model_spec
from sparseengine_b200.engine.model import Model
from test_movivik_gpu import CONFIGS, att, config, dense, far_key_model, par, sharp_chunk_model, slow_state_model

F64 = torch.float64


def moved(a, b, rows=slice(None)):
    """Root mean square of the difference of some rows, in units of the first's."""
    return float((a[rows] - b[rows]).pow(2).mean().sqrt() / a.pow(2).mean().sqrt())


def test_the_plain_mechanisms_are_what_they_claim():
    # the two pairings, a factor on cos and sin, the rest passes
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    y = pm.rotate(x, torch.tensor([3]), {"base": 100.0, "dims": 4}, True)
    assert np.allclose(y[0, 0].numpy(), [np.cos(a0) - 2 * np.sin(a0), 2 * np.cos(a0) + np.sin(a0),
                                         3 * np.cos(a1) - 4 * np.sin(a1), 4 * np.cos(a1) + 3 * np.sin(a1), 5.0])
    y = pm.rotate(x, torch.tensor([3]), {"base": 100.0, "dims": 4}, False)
    assert np.allclose(y[0, 0].numpy(), [np.cos(a0) - 3 * np.sin(a0), 2 * np.cos(a1) - 4 * np.sin(a1),
                                         3 * np.cos(a0) + np.sin(a0), 4 * np.cos(a1) + 2 * np.sin(a1), 5.0])
    # frequency scaling: pairs below the ramp keep their frequency, pairs above it are slowed, one between is blended
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 100, "fast": 6.0, "slow": 1.0}}
    place = lambda t: 8 * math.log(100 / (2 * math.pi * t)) / (2 * math.log(100.0))
    lo, hi = math.floor(place(6.0)), math.ceil(place(1.0))
    assert (lo, hi) == (0, 3)
    f, amp = pm.frequencies(rot)
    plain = [100.0 ** (-2 * i / 8) for i in range(4)]
    assert np.allclose(f.numpy(), [plain[i] * (i / 3 / 4 + 1 - i / 3) for i in range(4)]) and amp == 0.1 * math.log(4.0) + 1
    # chunks of three
    seen = pm.visible(5, 3)
    assert seen.int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [0, 0, 0, 1, 0], [0, 0, 0, 1, 1]]
    # the recurrence by hand: one head, one dim
    q, k, v = (torch.tensor(t, dtype=F64).view(3, 1, 1) for t in ([1.0, 2.0, 1.0], [1.0, 1.0, 2.0], [3.0, 1.0, -1.0]))
    o, S = pm.recurrence(q, k, v, [0.5])
    assert o.flatten().tolist() == [3.0, 5.0, -0.75] and S.item() == -0.75
    assert abs(pm.gelu_tanh(torch.tensor(1.0, dtype=F64)).item() - 0.8411919906) < 1e-9


def test_the_norm_after_a_rotation_is_that_of_the_rotated_head():
    x = torch.randn(4, 2, 12, dtype=F64, generator=torch.Generator().manual_seed(1))
    rot = {"base": 50.0, "dims": 8, "scaling": {"factor": 16.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    amp = pm.frequencies(rot)[1]
    y = pm.rotate(x, torch.arange(4), rot, False)
    counted = torch.cat([amp * x[..., :8], x[..., 8:]], -1)      # what the preparation kernel sums instead
    assert np.allclose((y * y).sum(-1).numpy(), (counted * counted).sum(-1).numpy())


def test_the_frequency_table_is_the_plain_one():
    from sparseengine_b200.parts.position import scaled_frequencies
    for dims, base, (factor, original, fast, slow) in ((16, 1e4, (4.0, 64, 32.0, 1.0)), (96, 5e5, (8.0, 4096, 32.0, 1.0)), (2, 100.0, (2.0, 50, 4.0, 1.0)),
                                                       (16, 100.0, (8.0, 512, 24.0, 0.3)), (8, 1.5, (2.0, 10 ** 6, 9.0, 8.0)), (12, 10.0, (3.0, 4, 32.0, 1.0))):
        rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
        want, amp = pm.frequencies(rot)
        got, scale = scaled_frequencies(dims, base, {"rope_type": "yarn", "factor": factor, "beta_fast": fast, "beta_slow": slow,
                                                     "original_max_position_embeddings": original})
        assert np.allclose(got.numpy(), want.numpy(), rtol=2e-6) and abs(scale - amp) < 1e-12


@pytest.mark.parametrize("dim", [16, 64, 88, 128])
def test_the_plain_chunk_matters(dim):
    cfg, w = sharp_chunk_model(37, dim)
    toks = tu.random_prompt(80, 150, 60)
    ref = pm.forward(cfg, w, toks)
    for other in (36, 38):
        c = copy.deepcopy(cfg)
        c["layers"][0]["mixer"]["mask"]["size"] = other
        d = pm.forward(c, w, toks)
        assert float((d - ref)[:36].abs().max()) < 1e-9             # the first tokens see everything either way
        rows = (d - ref)[36:].pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
        assert float(rows.max()) > 0.35                             # at least the widest bound of the GPU test


@pytest.mark.parametrize("dim", [16, 64, 96, 128])
def test_the_plain_far_keys_matter(monkeypatch, dim):
    """Without the first page of 16 keys the rows near position 400 move."""
    cfg, w = far_key_model(dim=dim)
    toks = tu.random_prompt(80, 430, 80)
    ref = pm.forward(cfg, w, toks)

    def blind(T, chunk=None):
        seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
        seen[16:, :16] = False
        return seen
    monkeypatch.setattr(pm, "visible", blind)
    rows = (pm.forward(cfg, w, toks) - ref)[300:].pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(rows.max()) > 0.45


def test_the_plain_state_matters():
    """What a first token leaves in the state still shows a thousand tokens later, and a state that is lost at
    position 300 does so by far more than the bfloat16 bound."""
    cfg, w = slow_state_model()
    toks = tu.random_prompt(64, 1100, 70)
    ref = pm.forward(cfg, w, toks)
    changed = [(toks[0] + 1) % 64] + toks[1:]
    assert moved(ref, pm.forward(cfg, w, changed), slice(400, None)) > 1e-4
    lost = pm.forward(cfg, w, toks[300:])
    rows = (lost - ref[300:]).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(rows[:50].max()) > 0.2


def test_the_plain_parts_matter(monkeypatch):
    """Gates, biases, scaling, pairings, norms and shared weights of the test models: leaving one out or swapping it
    shows."""
    def without(suffix):
        return lambda c, w: [w.__setitem__(k, torch.zeros_like(v)) for k, v in list(w.items()) if k.endswith(suffix)]

    def each(what):
        def change(c, w):
            for layer in c["layers"]:
                what(layer)
        return change
    for name, change in (("hybrid", without("mix.g")), ("hybrid", without("left.g")), ("wide", without("right.g")), ("wide", without(".b")),
                         ("hybrid", without("left.out")), ("hybrid", without("right.out")), ("odd", without("norm1b")), ("odd", without("norm2b")),
                         ("odd", lambda c, w: c["norm"].__setitem__("eps", 0.3)),
                         ("wide", each(lambda layer: (layer["mixer"].get("rot") or {}).pop("scaling", None))),
                         ("hybrid", each(lambda layer: layer["mixer"].get("right", {}).__setitem__("decay", [0.2] * layer["mixer"]["right"]["heads"])
                                         if layer["type"] == "parallel" else None)),
                         ("shared", lambda c, w: [layer.pop("weights_of", None) for layer in c["layers"]] and w.update(
                             {k: v for k, v in pm.random_weights(c, 9).items() if k not in w}))):
        cfg, w = copy.deepcopy(CONFIGS[name]), pm.random_weights(CONFIGS[name], 8)
        toks = tu.random_prompt(cfg["vocab"], 40, 3)
        ref = pm.forward(cfg, w, toks)
        w2 = {k: v.clone() for k, v in w.items()}
        change(cfg, w2)
        assert moved(ref, pm.forward(cfg, w2, toks)) > 0.02, name
    cfg, w = CONFIGS["wide"], pm.random_weights(CONFIGS["wide"], 8)
    toks = tu.random_prompt(cfg["vocab"], 40, 3)
    ref, real = pm.forward(cfg, w, toks), pm.rotate
    monkeypatch.setattr(pm, "rotate", lambda x, p, r, neighbours: real(x, p, r, not neighbours))
    assert moved(ref, pm.forward(cfg, w, toks)) > 0.02


def test_what_the_reader_makes_of_a_configuration():
    layers = [par((6, 2, 12, 20), (3, 16, 8), rot=8, base=777.0, scale=0.3, decay=[0.5, 0.9, 1.0], mlp=dense(48)),
              att(4, 1, 16, 10, 13, rot=12, base=555.0, scaling=(4.0, 64, 16.0, 2.0), scale=0.9)]
    cfg = config(64, 100, layers + [dict(copy.deepcopy(layers[0]), weights_of=0), dict(copy.deepcopy(layers[1]), weights_of=1)], eps=3e-4)
    _, spec = load_model_spec(cfg)
    assert len(spec.layers) == 2 and [e.layer for e in spec.order] == [0, 1, 0, 1] and all(e.cache is None for e in spec.order)
    both, at = (layer.mixer for layer in spec.layers)
    left, right = both.branches
    assert both.scales == (0.5, 0.5) and both.output_norms and both.norm_eps == 3e-4
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.scale) == (6, 2, 12, 20, 0.3)
    assert left.qk_norm == "per_head_unit" and left.qk_norm_eps == 3e-4 and not left.bias and left.output_gate == "head" and left.chunk is None
    assert (left.position.rotary_dim, left.position.theta, left.position.pairing, left.position.frequency_scaling) == (8, 777.0, "split_half", None)
    assert (right.num_heads, right.head_dim, right.v_head_dim, right.decays, right.k_scale) == (3, 16, 8, (0.5, 0.9, 1.0), 1.0)
    assert right.activation == "silu" and right.output_norm == "joint" and right.norm_eps == 3e-4 and right.position is None
    assert at.chunk == 13 and at.window is None and at.bias and at.output_bias is False and at.qk_norm is None and at.value_dim == 10
    assert (at.position.rotary_dim, at.position.theta, at.position.pairing) == (12, 555.0, "interleaved")
    assert dict(at.position.frequency_scaling) == {"rope_type": "yarn", "factor": 4.0, "original_max_position_embeddings": 64.0,
                                                   "beta_fast": 16.0, "beta_slow": 2.0}
    assert spec.layers[0].feed_forward.activation == "gelu_tanh" and spec.layers[1].feed_forward is None
    model = Model(spec, torch.bfloat16)
    assert {s.name for p in model.params() for s in p.sources} == set(pm.tensor_shapes(cfg))
    # a cache and a state of its own for every visit; the chunked layers' pages in a group of their own
    assert [(kv.chunk, n) for kv, n in model.layout.groups] == [(None, 2), (13, 2)] and len(model.layout.states) == 2
    assert [e.cache_layer for e in model.layout.entries] == [0, 0, 1, 1]
    # what may be left out: the rotation, the chunk, the scale
    bare = copy.deepcopy(cfg)
    bare["layers"] = [copy.deepcopy(layers[1])]
    for key in ("rot", "mask", "scale"):
        bare["layers"][0]["mixer"].pop(key)
    m = load_model_spec(bare)[1].layers[0].mixer
    assert m.position is None and m.chunk is None and m.scale == 0.25
    # a chain of shared weights
    cfg["layers"][3] = dict(copy.deepcopy(layers[0]), weights_of=2)
    assert [e.layer for e in load_model_spec(cfg)[1].order] == [0, 1, 0, 0]


def test_what_a_configuration_must_have():
    good = config(32, 40, [par((2, 1, 8, 8), (2, 8, 8), mlp=dense(16)), att(2, 1, 8, 8, 5, mlp=dense(16)),
                           dict(att(2, 1, 8, 8, 5, mlp=dense(16)), weights_of=1)])
    load_model_spec(good)
    for breaker, word in ((lambda c: c["layers"][0].__setitem__("type", "delta"), "unknown mixer type"),
                          (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), r"\(left\): missing mixer keys \['vdim'\]"),
                          (lambda c: c["layers"][0]["mixer"]["right"].pop("decay"), "decay"),
                          (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("decay", [0.5]), "one entry per head"),
                          (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 3), "multiple"),
                          (lambda c: c["layers"][1]["mixer"]["rot"].pop("base"), "base"),
                          (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
                          (lambda c: c["layers"][1]["mixer"].__setitem__("mask", {}), "size"),
                          (lambda c: c["layers"][2].__setitem__("weights_of", 3), "weights_of"),
                          (lambda c: c["layers"][2].__setitem__("weights_of", 2), "weights_of"),
                          (lambda c: c["layers"][2].__setitem__("weights_of", 0), "differs"),
                          (lambda c: c["layers"][2].__setitem__("mlp", None), "differs"),
                          (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "dense"),
                          (lambda c: c.pop("vocab"), "vocab")):
        bad = copy.deepcopy(good)
        breaker(bad)
        with pytest.raises(ValueError, match=word):
            load_model_spec(bad)


@pytest.mark.parametrize("chunk,page", [(10, 4), (4, 4), (1, 4), (37, 16), (3, 8)])
def test_the_cache_keeps_a_chunk(chunk, page):
    """Pages that hold nothing of the next query's chunk go back; what they held is not asked for again."""
    from sparseengine_b200.cache.manager import CacheManager
    from sparseengine_b200.engine.model import CacheLayout, EntryCache
    from sparseengine_b200.parts.base import KVRequest
    req = KVRequest(1, 8, chunk=chunk)
    assert [req.first_visible(p) for p in (0, chunk - 1, chunk, 2 * chunk)] == [0, 0, chunk, 2 * chunk]
    m = CacheManager(CacheLayout(((req, 1),), (), (EntryCache(0, 0, True, None),)), page_size=page, num_pages=64, max_rows=2, max_seq_len=256,
                     allocate=False)
    m.admit("a")
    n = 0
    for step in (1, 2, 5, 1, 1, 9, 3, 1, 17, 1, 1, 40, 1, 2):
        m.reserve("a", step)
        m.commit("a", step)
        n += step
        assert sorted(m._requests["a"].pages[0]) == list(range(n // chunk * chunk // page, -(-n // page))), n
        m.check()
    m.release("a")
    assert m.free_pages(0) == 64


def test_what_the_parts_refuse():
    from sparseengine_b200.config.specs import (AttentionSpec, DenseMLPSpec, LayerSpec, ModelSpec, ParallelMixerSpec, RetentionSpec,
                                                RMSNormSpec, RotarySpec, ScheduleEntry)
    from sparseengine_b200.parts.base import make_feed_forward, make_mixer
    ok = dict(hidden_size=64, num_heads=4, num_kv_heads=2, head_dim=16, scale=0.25, prep="general")
    make_mixer(AttentionSpec(**ok, chunk=5, output_gate="head", bias=True, output_bias=False,
                             position=RotarySpec(rotary_dim=8, pairing="interleaved", scaling=1.5)), torch.float32)
    for change, word in ((dict(chunk=0), "chunk"), (dict(chunk=4, window=4), "place of a window"), (dict(output_gate="row"), "output_gate"),
                         (dict(position=RotarySpec(rotary_dim=8, pairing="interleaved_to_split_half")), "neighbours")):
        with pytest.raises(ValueError, match=word):
            make_mixer(AttentionSpec(**ok, **change), torch.float32)
    with pytest.raises(ValueError, match="prep='general'"):
        make_mixer(AttentionSpec(**dict(ok, prep="rotary"), output_gate="head"), torch.float32)
    # the gate's rows follow the values'; biases cover q, k and v alone
    p = make_mixer(AttentionSpec(**ok, v_head_dim=8, output_gate="head", bias=True, output_bias=False), torch.float32).parameters()
    assert p["qkv"].shape == (64 + 32 + 16 + 4, 64) and p["qkv_bias"].shape == (112,) and "o_bias" not in p
    ret = dict(hidden_size=64, num_heads=2, head_dim=16, v_head_dim=16, decays=(0.5, 0.9))
    make_mixer(RetentionSpec(**ret, activation="silu", output_norm="joint"), torch.float32)
    with pytest.raises(ValueError, match="activation"):
        make_mixer(RetentionSpec(**ret, activation="relu"), torch.float32)
    with pytest.raises(ValueError, match="output_norm"):
        make_mixer(RetentionSpec(**ret, output_norm="row"), torch.float32)
    both = dict(hidden_size=64, scales=(0.5, 0.5), names=("left", "right"), output_norms=True)
    make_mixer(ParallelMixerSpec(**both, branches=(AttentionSpec(**ok), RetentionSpec(**ret))), torch.float32)
    with pytest.raises(ValueError, match="no bias"):
        make_mixer(ParallelMixerSpec(**both, branches=(AttentionSpec(**ok, bias=True), RetentionSpec(**ret))), torch.float32)
    make_feed_forward(DenseMLPSpec(hidden_size=8, intermediate_size=8, activation="gelu_tanh"), torch.float32)
    with pytest.raises(ValueError, match="activation"):
        make_feed_forward(DenseMLPSpec(hidden_size=8, intermediate_size=8, activation="tanh"), torch.float32)
    norm, grouped = RMSNormSpec(size=64), RMSNormSpec(size=64, groups=2)

    def spec(post, entry=ScheduleEntry(0), **kw):
        layer = LayerSpec(mixer=RetentionSpec(**ret), feed_forward=None, mixer_norm=norm, feed_forward_norm=None, arrangement="sandwich_norm",
                          extra={"mixer_post_norm": post} if post else {}, sources={})
        return ModelSpec(architecture="t", hidden_size=64, vocab_size=8, max_position=64, layers=[layer], order=[entry], final_norm=norm, **kw)
    Model(spec(norm, residual_stream="float32"), torch.float32)
    for post in (None, grouped):
        with pytest.raises(ValueError, match="mixer_post_norm"):
            Model(spec(post, residual_stream="float32"), torch.float32)
    with pytest.raises(ValueError, match="sandwich_norm blocks need"):
        Model(spec(norm), torch.float32)
    with pytest.raises(ValueError, match="add_embedding"):
        Model(spec(norm, ScheduleEntry(0, add_embedding=True), residual_stream="float32"), torch.float32)
