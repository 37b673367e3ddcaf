"""The Movivik design in the engine against the plain implementation (tests/plain_movivik.py): each mechanism
alone, whole prompts against token-by-token decoding, portions down to two tokens, mixed batches with pages
and state slots that are used again, keys far away, at both edges of every chunk and at page borders, a far
token held by the recurrence, the first tokens, long decoding, other sizes (also values equal to one another
or to 1), greedy generation through ``LLM``, and the design's kernels against one another and against the
equations written out."""
import copy
import json
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_movivik as pm
import trace_util as tu

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def dense(ff):
    return {"kind": "dense", "ff": ff}


def att(heads, kv_heads, dim, vdim, chunk, rot=None, base=10000.0, scaling=(4.0, 64, 32.0, 1.0), scale=None, mlp=None, **more):
    r = {"base": base, "dims": dim if rot is None else rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mlp": mlp, **more,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": r,
                      "scale": scale if scale is not None else 1.5 * dim ** -0.5}}


def par(left, right, rot=None, base=5000.0, scale=None, decay=None, mlp=None, **more):
    """left: (heads, kv_heads, dim, vdim), right: (heads, dim, vdim)."""
    H, G, d, dv = left
    Hr, dr, dvr = right
    if decay is None:
        decay = [1.0 - 2.0 ** (-1.0 - 6.0 * h / max(1, Hr - 1)) for h in range(Hr)]
    return {"type": "parallel", "mlp": mlp, **more,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "rot": {"base": base, "dims": d if rot is None else rot},
                               "scale": scale if scale is not None else 0.8},
                      "right": {"heads": Hr, "dim": dr, "vdim": dvr, "decay": decay}}}


def config(width, vocab, layers, eps=1e-6):
    return {"architecture": "Movivik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


def _with_again(layers, *which):
    """Insert after the listed layers a layer that uses their weights."""
    out = []
    place = {}
    for i, layer in enumerate(layers):
        place[i] = len(out)
        out.append(layer)
        if i in which:
            out.append(dict(copy.deepcopy(layer), weights_of=place[i]))
    return out


CONFIGS = {
    # both mixers, layers with and without a feed-forward, shared weights of both kinds
    "hybrid": config(96, 160, _with_again([par((6, 2, 12, 20), (3, 16, 8), rot=8, mlp=dense(128)), att(6, 3, 16, 12, 11, rot=12, mlp=dense(72)),
                                           par((2, 2, 8, 8), (2, 8, 24)), att(3, 1, 20, 16, 30, scaling=None)], 0, 1), eps=1e-5),
    # two layers, one of them shared three times, two chunk sizes (two page groups of chunks)
    "shared": config(64, 100, [att(4, 1, 8, 24, 7, mlp=dense(96)), par((4, 4, 16, 16), (4, 16, 16), mlp=dense(48)), att(2, 2, 24, 8, 20),
                               {"type": "attention", "weights_of": 0}, {"type": "parallel", "weights_of": 1}, {"type": "attention", "weights_of": 3}]),
    # sizes that bfloat16 steps give to the tensor-core kernels, exact tiles and padded ones
    "wide": config(128, 200, [par((4, 2, 64, 64), (2, 64, 64), rot=32, mlp=dense(192)), att(4, 2, 128, 128, 50, rot=64, mlp=dense(192)),
                              par((3, 1, 80, 40), (5, 40, 32), mlp=dense(160)), att(4, 1, 72, 104, 33, mlp=dense(192)),
                              att(2, 2, 112, 64, 70)], eps=1e-5),
    # sizes that are equal or 1: one head, a chunk of one key, a decay of 1, one rotated pair.  (Not values of one dim: a norm
    # over one number is its sign, which rounding decides where it is near 0.)
    "ones": config(32, 48, [att(1, 1, 32, 32, 1, mlp=dense(32)), par((1, 1, 32, 32), (1, 32, 32), decay=[1.0], mlp=dense(32)),
                            att(1, 1, 2, 6, 64, scaling=(1.0, 32, 8.0, 2.0)), par((1, 1, 2, 6), (1, 6, 6), decay=[0.5])]),
    # sizes that are multiples of nothing in particular
    "odd": config(54, 77, [par((5, 5, 6, 3), (3, 7, 5), rot=2, mlp=dense(30)), att(5, 5, 10, 3, 19, rot=6, mlp=dense(11)),
                           att(3, 1, 7, 13, 9, rot=4), par((3, 1, 13, 9), (2, 5, 11), rot=10, decay=[0.05, 0.99])], eps=1e-4),
}
for _i in (3, 4, 5):       # the rest of the entries that use another layer's weights
    _l = CONFIGS["shared"]["layers"]
    CONFIGS["shared"]["layers"][_i] = dict(copy.deepcopy(_l[{3: 0, 4: 1, 5: 0}[_i]]), weights_of=_l[_i]["weights_of"])


def write_folder(folder, cfg, seed, w=None):
    from safetensors.torch import save_file
    w = w if w is not None else pm.random_weights(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return w


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("mov_" + name))
        out[name] = (d, cfg, write_folder(d, cfg, 71 + i))
    return out


_plain_cache = {}


def plain_logits(cfg, w, seqs):
    out = {}
    for sid, toks in seqs.items():
        key = (json.dumps(cfg, sort_keys=True), float(w["embed"].float().sum()), tuple(toks))
        if key not in _plain_cache:
            _plain_cache[key] = pm.forward(cfg, w, toks).float().numpy()
        out[sid] = _plain_cache[key]
    return out


def row_errors(got, ref):
    """Difference of every logits row (mean taken off, root mean square) in units of the reference
    rows' root mean square."""
    rows = np.stack([ref[sid][p] for sid, p in got])
    rms = float(np.sqrt((rows.astype(np.float64) ** 2).mean()))
    out = {}
    for (sid, p), row in got.items():
        d = row.astype(np.float64) - ref[sid][p]
        d -= d.mean()
        e = float(np.sqrt((d * d).mean())) / rms
        out[(sid, p)] = e if e == e else float("inf")
    return out


# 32-bit: every row within 3e-5.  bfloat16: rounding alone moves the rows of these small models by one or two parts in a
# hundred, so nine rows of ten must lie within 0.06 and every row within 0.2; a fault of the cache, the state or a
# chunk moves every row behind it by its whole size.
BOUND32 = 3e-5


def assert_close(got, ref, dtype, what, bound=None):
    errs = row_errors(got, ref)
    v = np.array(list(errs.values()))
    where = max(errs, key=errs.get)
    if bound is not None or dtype == "float32":
        limit = bound or BOUND32
        assert v.max() < limit, f"{what} ({dtype}): row error {v.max():.3e} at {where}"
        return
    assert np.quantile(v, 0.9) < 0.06, f"{what} ({dtype}): nine rows of ten within {np.quantile(v, 0.9):.3e}"
    assert v.max() < 0.2, f"{what} ({dtype}): row error {v.max():.3e} at {where}"


def make_runner(folder, dtype, steps, page_size=16, rows=4, **kw):
    from sparseengine_b200.engine.factory import build_runner
    tokens = tu.max_live_tokens(steps, round_to=page_size)
    return build_runner(folder, dtype=dtype, page_size=page_size, num_pages=max(1, tokens // page_size), max_rows=rows,
                        max_seq_len=max(64, tokens), **kw)


def check_trace(folders, name, dtype, steps, seqs, what, bound=None, **kw):
    folder, cfg, w = folders[name]
    runner = make_runner(folder, dtype, steps, **kw)
    got = tu.run_trace_runner(runner, steps)
    from sparseengine_b200.csrc import ops
    ops.error_check(runner.device)
    runner.cache.check()
    assert runner.cache.free_rows == runner.cache.max_rows
    assert_close(got, plain_logits(cfg, w, seqs), dtype, f"{what}, {name}", bound)
    return runner


def prompts(cfg, lengths, seed):
    return {f"s{i}": tu.random_prompt(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


# ---- each mechanism alone ----------------------------------------------------------------------

SINGLE = {
    "chunked_attention": ([att(4, 2, 12, 20, 9)], {}),
    "chunked_attention_partly_rotated_without_scaling": ([att(4, 2, 16, 8, 15, rot=6, scaling=None)], {}),
    "frequency_scaling_where_every_pair_is_blended": ([att(2, 1, 16, 16, 40, base=100.0, scaling=(8.0, 512, 24.0, 0.3))], {}),
    "full_attention_beside_lightning": ([par((4, 2, 12, 20), (3, 8, 16), rot=6)], {}),
    "feed_forward": ([att(1, 1, 8, 8, 4, mlp=dense(80))], {}),
    "weights_of_a_layer_with_a_state": ([par((2, 1, 8, 8), (2, 8, 8), mlp=dense(24))] * 1 + [dict(par((2, 1, 8, 8), (2, 8, 8), mlp=dense(24)), weights_of=0)], {}),
    "an_eps_that_counts": ([par((2, 2, 8, 8), (2, 8, 8), mlp=dense(24)), att(2, 1, 8, 8, 6)], {"eps": 0.3}),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(SINGLE))
def test_each_mechanism_alone(tmp_path, which, dtype):
    layers, kw = SINGLE[which]
    cfg = config(40, 50, layers, **kw)
    w = write_folder(str(tmp_path), cfg, 5)
    seqs = prompts(cfg, (37, 1, 18), 3)
    for cut in (tu.trace_whole, lambda s: tu.trace_chunks(s, sizes=(2, 3, 1, 5, 2)), lambda s: tu.trace_tail_decode(s, tail=9)):
        check_trace({which: (str(tmp_path), cfg, w)}, which, dtype, cut(seqs), seqs, "alone")


# ---- ways of cutting ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_decode_chunks_mixed(folders, name, dtype):
    cfg = CONFIGS[name]
    seqs = prompts(cfg, (70, 33, 1, 18, 49, 2, 26), 20)
    check_trace(folders, name, dtype, tu.trace_whole(seqs), seqs, "whole")
    check_trace(folders, name, dtype, tu.trace_tail_decode(seqs, tail=20), seqs, "decode")
    check_trace(folders, name, dtype, tu.trace_chunks(seqs), seqs, "portions")
    check_trace(folders, name, dtype, tu.trace_chunks(seqs, sizes=(2,)), seqs, "portions of two")
    # three rows for seven requests, and a pool of the live tokens only: rows, state slots and pages are used again
    runner = check_trace(folders, name, dtype, tu.trace_mixed(seqs, live=3, chunk=6, decode_tail=5), seqs, "mixed", rows=3)
    assert all(g.pool.reused_total > 0 for g in runner.cache.groups)
    check_trace(folders, name, dtype, tu.trace_random(seqs, seed=3, live=4), seqs, "random schedule", page_size=8)


def test_a_state_slot_that_is_used_again_starts_from_zero(folders):
    """One row: every request gets the slot and the pages the one before it left; a long request
    first, so that its state is far from zero."""
    seqs = prompts(CONFIGS["shared"], (60, 5, 1, 9), 40)
    check_trace(folders, "shared", "float32", tu.trace_chunks(seqs, sizes=(7, 2)), seqs, "one slot", rows=1)


# ---- places where a fault would sit --------------------------------------------------------------

def sharp_chunk_model(chunk, dim=16, seed=9):
    """One chunked attention layer whose softmax is sharp (a large score scale), so that a query hangs on the one or
    two keys of its chunk with the highest score: a key that is lost at the chunk's start, or one that is let in from
    the chunk before, moves the row by much."""
    cfg = config(64, 80, [att(4, 2, dim, dim, chunk, scale=10.0 * dim ** -0.5, scaling=None, mlp=dense(64))])
    return cfg, pm.random_weights(cfg, seed)


@pytest.mark.parametrize("dtype,dim", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64), ("bfloat16", 88), ("bfloat16", 128)])
def test_the_chunks_two_edges_and_page_borders(tmp_path, dtype, dim):
    """Chunks of 37 over pages of 16: the first key a query sees wanders through the places of a page from chunk to
    chunk, in prompts, in portions that start and end anywhere (also at and beside a chunk's edge), and in tokens
    decoded alone over the edges; pages behind the chunk are given back and used again meanwhile.  (In bfloat16 the
    rounding of queries and keys moves such sharp weights by itself, hence the wider bound; a lost key moves the
    row by its whole size.)"""
    cfg, w = sharp_chunk_model(37, dim)
    write_folder(str(tmp_path), cfg, 0, w)
    seqs = prompts(cfg, (150, 37, 38, 36, 16, 95), 60)
    fs = {"edge": (str(tmp_path), cfg, w)}
    bound = 0.35 if dtype == "bfloat16" else 6e-5
    check_trace(fs, "edge", dtype, tu.trace_whole(seqs), seqs, "chunk, whole", bound)
    check_trace(fs, "edge", dtype, tu.trace_tail_decode(seqs, tail=80), seqs, "chunk, decoded", bound)
    check_trace(fs, "edge", dtype, tu.trace_chunks(seqs, sizes=(15, 2, 16, 33, 1, 7, 37, 38)), seqs, "chunk, portions", bound)
    check_trace(fs, "edge", dtype, tu.trace_chunks(seqs, sizes=(37,)), seqs, "chunk, a portion each", bound)
    check_trace(fs, "edge", dtype, tu.trace_chunks(seqs, sizes=(36, 2, 35)), seqs, "chunk, portions over the edge", bound)
    check_trace(fs, "edge", dtype, tu.trace_mixed(seqs, live=3, chunk=21, decode_tail=40), seqs, "chunk, mixed", bound, rows=3)


def test_pages_behind_a_chunk_are_given_back(folders):
    """After position p only the pages of p's next query's chunk are held."""
    from sparseengine_b200.engine.runner import StepEntry
    cfg, w = sharp_chunk_model(37)
    import tempfile
    with tempfile.TemporaryDirectory() as d:
        write_folder(d, cfg, 0, w)
        toks = tu.random_prompt(80, 120, 1)
        runner = make_runner(d, "float32", [{"step": 0, "entries": [{"id": "a", "tokens": toks}], "end": []}], page_size=4)
        runner.validate = True
        runner.admit("a")
        for t in range(0, 120, 3):
            runner.step([StepEntry("a", toks[t:t + 3], [2])])
            n = t + 3
            held = sorted(runner.cache._requests["a"].pages[0])
            assert held == list(range(n // 37 * 37 // 4, -(-n // 4))), n


def far_key_model(seed=13, dim=16):
    """One parallel layer whose attention has a sharp softmax over all earlier keys: queries hang on single keys
    anywhere in the sequence."""
    cfg = config(64, 80, [par((4, 2, dim, dim), (2, 8, 8), rot=dim // 2, scale=12.0, mlp=dense(64))])
    return cfg, pm.random_weights(cfg, seed)


@pytest.mark.parametrize("dtype,dim", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64), ("bfloat16", 96), ("bfloat16", 128)])
def test_far_keys_of_the_full_attention(tmp_path, dtype, dim):
    cfg, w = far_key_model(dim=dim)
    write_folder(str(tmp_path), cfg, 0, w)
    seqs = prompts(cfg, (430, 131, 64, 7), 80)
    fs = {"far": (str(tmp_path), cfg, w)}
    bound = 0.45 if dtype == "bfloat16" else 1e-4
    check_trace(fs, "far", dtype, tu.trace_whole(seqs), seqs, "far keys, whole", bound)
    check_trace(fs, "far", dtype, tu.trace_chunks(seqs, sizes=(100, 2, 33, 1, 64)), seqs, "far keys, portions", bound)
    check_trace(fs, "far", dtype, tu.trace_tail_decode(seqs, tail=40), seqs, "far keys, decoded", bound)
    check_trace(fs, "far", dtype, tu.trace_mixed(seqs, live=3, chunk=50, decode_tail=30), seqs, "far keys, mixed", bound, rows=3)


def slow_state_model(seed=12, dim=24):
    """Heads that forget slowly or not at all; the attention beside them is made blind (its values are zero), so what
    far tokens leave reaches a query through the state alone."""
    cfg = config(48, 64, [par((1, 1, 8, 8), (3, dim, 16), decay=[0.9999, 0.995, 1.0], mlp=dense(64))])
    w = pm.random_weights(cfg, seed)
    w["l0.mix.left.v"].zero_()
    return cfg, w


@pytest.mark.parametrize("dtype,dim", [("float32", 24), ("bfloat16", 24), ("bfloat16", 64)])
def test_a_far_token_held_by_the_recurrence(tmp_path, dtype, dim):
    """A state that is lost at a portion's start or copied to the wrong slot shows in every row behind it."""
    cfg, w = slow_state_model(dim=dim)
    write_folder(str(tmp_path), cfg, 0, w)
    seqs = prompts(cfg, (1100, 130, 3, 260), 70)
    fs = {"far": (str(tmp_path), cfg, w)}
    check_trace(fs, "far", dtype, tu.trace_whole(seqs), seqs, "far token, whole")
    check_trace(fs, "far", dtype, tu.trace_chunks(seqs, sizes=(300, 2, 133, 7, 1)), seqs, "far token, portions")
    check_trace(fs, "far", dtype, tu.trace_tail_decode(seqs, tail=40), seqs, "far token, decoded")
    check_trace(fs, "far", dtype, tu.trace_mixed(seqs, live=2, chunk=150, decode_tail=10), seqs, "far token, mixed", rows=2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens(folders, dtype):
    """Requests of one to four tokens, whole, in portions of one and two, and side by side."""
    seqs = prompts(CONFIGS["hybrid"], (1, 2, 3, 4, 1), 90)
    check_trace(folders, "hybrid", dtype, tu.trace_whole(seqs), seqs, "first tokens")
    check_trace(folders, "hybrid", dtype, tu.trace_chunks(seqs, sizes=(1, 2, 1)), seqs, "first tokens, portions")
    check_trace(folders, "hybrid", dtype, tu.trace_mixed(seqs, live=4, chunk=2, decode_tail=1), seqs, "first tokens, mixed")


def test_long_decoding_through_replayed_graphs(folders):
    """140 tokens decoded one by one, over several edges of every chunk, through replayed CUDA graphs."""
    for name, dtype in (("hybrid", "float32"), ("hybrid", "bfloat16"), ("wide", "bfloat16")):
        seqs = prompts(CONFIGS[name], (170, 150), 120)
        runner = check_trace(folders, name, dtype, tu.trace_tail_decode(seqs, tail=140), seqs, "long decoding")
        assert runner.graph_replays > 200


def test_a_batch_does_not_change_a_request(folders):
    """Unequal requests in one step against each alone: equal up to the order of sums in 32-bit."""
    from sparseengine_b200.engine.runner import StepEntry
    folder, cfg, w = folders["hybrid"]
    seqs = prompts(cfg, (29, 3, 11), 140)
    steps = [{"step": 0, "entries": [{"id": sid, "tokens": toks} for sid, toks in seqs.items()], "end": []}]
    runner = make_runner(folder, "float32", steps, rows=4)       # pages for all three at once
    alone = {}
    for sid, toks in seqs.items():
        runner.admit(sid)
        runner.step([StepEntry(sid, toks[:-1], [])])
        alone[sid] = runner.step([StepEntry(sid, toks[-1:], [0])]).clone()
        runner.release(sid)
    for sid in seqs:
        runner.admit(sid)
    runner.step([StepEntry(sid, toks[:-1], []) for sid, toks in seqs.items()])
    together = runner.step([StepEntry(sid, toks[-1:], [0]) for sid, toks in seqs.items()])
    for i, sid in enumerate(seqs):
        assert float((together[i] - alone[sid][0]).abs().max()) < 2e-5 * float(alone[sid][0].abs().max()), sid


def test_the_stream_after_every_layer(folders):
    """The 32-bit stream after each layer (one that uses another's weights counts too) against the plain
    implementation's."""
    from sparseengine_b200.engine.runner import StepEntry
    folder, cfg, w = folders["shared"]
    toks = tu.random_prompt(cfg["vocab"], 45, 8)
    taps = []
    pm.forward(cfg, w, toks, taps)
    runner = make_runner(folder, "float32", [{"step": 0, "entries": [{"id": "a", "tokens": toks}], "end": []}])
    runner.model.stream_taps = got = []
    runner.admit("a")
    runner.step([StepEntry("a", toks, [0])])
    assert len(got) == len(taps) == 6
    for i, (a, b) in enumerate(zip(got, taps)):
        assert float((a.cpu().double() - b).abs().max()) < 3e-5 * float(b.abs().max()), i


# ---- the entry point -----------------------------------------------------------------------------

def plain_greedy(cfg, w, prompt, steps):
    toks, out, margins = list(prompt), [], []
    for _ in range(steps):
        logits = pm.forward(cfg, w, toks)[-1]
        top = torch.topk(logits, 2).values
        margins.append(float(top[0] - top[1]))
        out.append(int(logits.argmax()))
        toks.append(out[-1])
    return out, margins


@pytest.mark.parametrize("name", ["hybrid", "odd"])
def test_greedy_generation_through_the_entry_point(folders, name):
    from sparseengine_b200 import LLM, SamplingParams
    folder, cfg, w = folders[name]
    llm = LLM(folder, dtype="float32", page_size=8, num_kvcache_slots=512, max_num_batched_tokens=16, max_model_len=128,
              max_num_seqs_in_gpu=3)
    ps = [tu.random_prompt(cfg["vocab"], n, 200 + n) for n in (5, 21, 9, 2, 14)]
    outs = llm.generate(ps, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))
    for p, o in zip(ps, outs):
        want, margins = plain_greedy(cfg, w, p, 10)
        if min(margins) > 1e-4:
            assert o["token_ids"] == want
        else:       # a near-tie: the tokens up to it
            k = next(i for i, m in enumerate(margins) if m <= 1e-4)
            assert o["token_ids"][:k] == want[:k]
    assert llm.is_finished() and llm.runner.cache.free_rows == llm.runner.cache.max_rows


def test_trace_program(folders, tmp_path):
    """bin/trace_run as a program on a folder of this design, pages and slots used again."""
    folder, cfg, w = folders["wide"]
    seqs = prompts(cfg, (40, 7, 22, 31, 3), 300)
    steps = tu.trace_mixed(seqs, live=4, chunk=9, decode_tail=4)
    for dtype in ("float32", "bfloat16"):
        out = str(tmp_path / dtype)
        got = tu.run_trace_cli(folder, dtype, steps, out, tu.max_live_tokens(steps))
        assert_close(got, plain_logits(cfg, w, seqs), dtype, "trace program")


def test_command_line(folders):
    import subprocess
    import sys
    folder, cfg, w = folders["hybrid"]
    hyper = json.dumps({"dtype": "bfloat16", "page_size": 8, "num_kvcache_slots": 1024, "max_model_len": 256})
    for extra in ([], ["--tiny_random"]):
        r = subprocess.run([sys.executable, "-m", "sparseengine_b200.cli.bench", "--model_path", folder, "--lengths", "24",
                            "--batch_sizes", "3", "--output_len", "6", "--random_prompts", "--generate", "--hyper_params", hyper,
                            *extra], cwd=tu.ROOT, capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert r.stdout.strip()


# ---- kernels against one another and against their equations ----------------------------------------

def batch(q_lens, kv_lens, dev, page, rows):
    """Positions, block table (pages in a shuffled order) and index tensors of a step's entries."""
    entries = len(q_lens)
    max_pages = -(-max(kv_lens) // page)
    perm = torch.randperm(entries * max_pages, generator=torch.Generator().manual_seed(1)).to(torch.int32)
    seq_rows = torch.tensor(rows, dtype=torch.int32, device=dev)
    table = perm.view(entries, max_pages).to(dev)[torch.argsort(seq_rows.cpu()).to(dev)].contiguous()
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    return SimpleNamespace(
        entries=entries, tokens=sum(q_lens), pages=entries * max_pages, table=table, seq_rows=seq_rows, num_seqs=entries,
        max_q_len=max(q_lens), cu=cu,
        positions=torch.cat([torch.arange(k - n, k) for n, k in zip(q_lens, kv_lens)]).to(torch.int32).to(dev),
        token_seq=torch.repeat_interleave(torch.arange(entries), torch.tensor(q_lens)).to(torch.int32).to(dev),
        cu_q=torch.tensor(cu, dtype=torch.int32, device=dev), kv_len=torch.tensor(kv_lens, dtype=torch.int32, device=dev))


def held(cache, b, e, page, kv_heads, d, dv):
    """Entry e's keys and values [positions, kv heads, size] in 64-bit from its pages."""
    c = cache.double().cpu()
    keys = c[:, :page * kv_heads * d].reshape(-1, kv_heads, page, d)
    vals = c[:, page * kv_heads * d:].reshape(-1, kv_heads, page, dv)
    pages = b.table.cpu()[b.seq_rows.cpu()[e].item()].long()
    return (keys[pages].transpose(1, 2).reshape(-1, kv_heads, d), vals[pages].transpose(1, 2).reshape(-1, kv_heads, dv))


@pytest.mark.parametrize("d,dv,heads,kv_heads,chunk,window,gated", [
    (64, 64, 4, 2, 33, None, "head"), (128, 64, 6, 1, 70, None, "head"), (104, 56, 6, 2, 50, None, "head"), (40, 24, 3, 3, 17, None, "head"),
    (128, 128, 8, 2, 100, None, "head"), (128, 128, 6, 6, 1, None, "head"), (128, 128, 4, 1, None, None, "head"), (72, 128, 20, 1, 64, None, None),
    (88, 104, 4, 2, None, 37, "element"), (120, 32, 2, 1, None, None, "element"), (128, 128, 4, 2, 64, None, "element"), (56, 40, 34, 2, 90, None, "head")])
def test_chunks_gates_and_head_sizes_in_the_attention_kernels(d, dv, heads, kv_heads, chunk, window, gated):
    """The same queries, pages and block table through the plain kernel, the split-key kernel and the prompt-portion
    kernels: keys of a query's own chunk, a gate per head or per element, head sizes between the tiles'; the plain
    kernel against the equations in 64-bit.  Some entries start, end or lie on a chunk's edge."""
    from sparseengine_b200.csrc import ops
    page = 16
    g = torch.Generator(device=DEV).manual_seed(d + heads)
    q_lens, kv_lens = [37, 1, 130, 1, 2, 1, 1, 35], [37, 64, 209, 140, 17, 3, 101, 135]
    b = batch(q_lens, kv_lens, DEV, page, [3, 0, 4, 1, 5, 2, 7, 6])
    cache = (torch.randn(b.pages, page * kv_heads * (d + dv), generator=g, device=DEV) * 0.7).to(torch.bfloat16)
    q = torch.randn(b.tokens, heads * d, generator=g, device=DEV).to(torch.bfloat16)
    cols = {"head": heads, "element": heads * dv, None: 0}[gated]
    gate_rows = torch.randn(b.tokens, cols + 11, generator=g, device=DEV).to(torch.bfloat16)
    gate = gate_rows[:, 3:3 + cols] if gated else None
    scale = d ** -0.5 * 2.0
    common = dict(num_heads=heads, num_kv_heads=kv_heads, head_dim=d, page_size=page, scale=scale, window=window, chunk=chunk,
                  v_head_dim=dv, gate=gate)
    plain = torch.full((b.tokens, heads * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    ops.paged_attention_plain(q, cache, b.table, b.seq_rows, b.token_seq, b.positions, plain, **common)
    portions, split, split_long = (torch.full_like(plain, float("nan")) for _ in range(3))
    ops.attn_prefill(q, cache, b.table, b.seq_rows, b.cu_q, b.kv_len, portions, entries=b.entries, max_q_len=b.max_q_len, **common)
    ops.attn_decode(q, cache, b.table, b.seq_rows, b.token_seq, b.positions, split, max_keys=min(max(kv_lens), chunk or window or 1 << 30), **common)
    ops.attn_decode(q[:1], cache, b.table, b.seq_rows, b.token_seq, b.positions, split_long[:1], max_keys=4096,       # several key splits
                    **dict(common, gate=gate[:1] if gated else None))
    others = [(portions, "portions"), (split, "split keys")]
    if d == dv and ops.attn_prefill_tc_supported(d, heads, kv_heads):
        tc = torch.full_like(plain, float("nan"))
        ops.attn_prefill_tc(q, cache, b.table, b.seq_rows, b.cu_q, b.kv_len, tc, entries=b.entries, max_q_len=b.max_q_len, **common)
        others.append((tc, "portions, tensor memory"))
    ops.error_check(DEV)
    want = torch.zeros(b.tokens, heads, dv, dtype=torch.float64)
    for e in range(b.entries):
        K, V = (x.repeat_interleave(heads // kv_heads, 1) for x in held(cache, b, e, page, kv_heads, d, dv))
        for t in range(b.cu[e], b.cu[e + 1]):
            p = int(b.positions[t])
            lo = p // chunk * chunk if chunk else max(0, p - window + 1) if window else 0
            s = torch.einsum("hd,jhd->hj", q[t].double().cpu().view(heads, d), K[lo:p + 1]) * scale
            want[t] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), V[lo:p + 1])
    if gated:
        want = want * torch.sigmoid(gate.double().cpu()).view(b.tokens, heads, -1)
    want = want.reshape(b.tokens, -1)
    most = float(want.abs().max())
    assert float((plain.double().cpu() - want).abs().max()) < 1.5e-2 * most
    for other, what in others:
        assert bool(torch.isfinite(other.float()).all()), what
        assert float((other.float() - plain.float()).abs().max()) < 3e-2 * most, what
    assert float((split_long[:1].float() - plain[:1].float()).abs().max()) < 3e-2 * most


@pytest.mark.parametrize("d,dv,heads,kv_heads,rot,pairing,norm,bias,scale", [
    (104, 56, 6, 2, 104, "interleaved", None, True, 1.3), (64, 64, 4, 1, 16, "split_half", "unit", False, 1.0),
    (128, 128, 8, 2, 64, "split_half", "unit", False, 1.4), (128, 40, 4, 4, 128, "interleaved", "unit", True, 0.7),
    (64, 24, 3, 1, 64, "split_half", "weights", True, 1.1), (256, 64, 4, 2, 32, "interleaved", "weights", False, 1.2),
    (16, 16, 2, 2, 16, "split_half", "unit", False, 1.5), (8, 8, 1, 1, 8, "interleaved", "unit", True, 1.5), (40, 16, 5, 1, 32, "split_half", None, True, 1.0),
    # sizes that leave the chunked kernel
    (12, 20, 4, 2, 6, "split_half", "unit", False, 1.4), (10, 3, 5, 5, 6, "interleaved", None, True, 1.2), (104, 56, 6, 2, 32, "split_half", "unit", True, 1.6),
    (104, 56, 3, 1, 24, "interleaved", "unit", False, 1.6), (13, 7, 3, 1, 4, "interleaved", "weights", True, 0.8), (24, 24, 2, 1, 0, "split_half", "unit", True, 1.0)])
def test_query_and_key_preparation(d, dv, heads, kv_heads, rot, pairing, norm, bias, scale):
    """Biases, rotations of both pairings with a factor on cos and sin, and norms per head (over the rotated head
    where they have no weights) against the equations; queries, keys and values in their places."""
    from sparseengine_b200.csrc import ops
    page, eps = 16, 1e-3
    g = torch.Generator(device=DEV).manual_seed(d + heads + rot)
    q_lens, kv_lens = [37, 1, 130, 2, 1], [37, 1, 130, 2, 1]              # whole prompts: the pages all come from this step
    b = batch(q_lens, kv_lens, DEV, page, [2, 0, 3, 1, 4])
    qn, kn, vn = heads * d, kv_heads * d, kv_heads * dv
    pitch = (qn + kn + vn + 7) // 8 * 8 + 16
    inv_freq = (300.0 ** (-torch.arange(0, max(rot, 1), 2, dtype=torch.float64) / max(rot, 1))).float().to(DEV)[:rot // 2].contiguous()
    bias_t = torch.randn(qn + kn + vn, generator=g, device=DEV) if bias else None
    for dtype, bound in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        proj = torch.randn(b.tokens, pitch, generator=g, device=DEV).to(dtype)
        w = [(1 + 0.3 * torch.randn(d, generator=g, device=DEV)).to(dtype) for _ in range(2)] if norm == "weights" else [None, None]
        cache = torch.full((b.pages, page * kv_heads * (d + dv)), float("nan"), dtype=dtype, device=DEV)
        q = torch.full((b.tokens, qn), float("nan"), dtype=dtype, device=DEV)
        ops.qk_prep_general(proj, w[0], w[1], b.positions, b.token_seq, b.seq_rows, b.table, cache, q, num_heads=heads, num_kv_heads=kv_heads,
                            head_dim=d, v_head_dim=dv, eps=eps, page_size=page, bias=bias_t, per_head=norm == "weights",
                            per_head_unit=norm == "unit", inv_freq=inv_freq if rot else None, rotary_dim=rot, pairing=pairing, rope_scale=scale)
        ops.error_check(DEV)
        P = proj.double().cpu()[:, :qn + kn + vn] + (bias_t.double().cpu() if bias else 0.0)

        def prepared(x, n, weight):
            x = x.reshape(b.tokens, n, d)
            if norm == "weights":
                x = pm.unit_rms(x, eps) * weight.double().cpu()
            if rot:
                ang = b.positions.double().cpu()[:, None] * inv_freq.double().cpu()[None, :]
                c, s = scale * torch.cos(ang)[:, None], scale * torch.sin(ang)[:, None]
                first, second = (slice(0, rot, 2), slice(1, rot, 2)) if pairing == "interleaved" else (slice(0, rot // 2), slice(rot // 2, rot))
                u, v = x[..., first].clone(), x[..., second].clone()
                x = x.clone()
                x[..., first], x[..., second] = u * c - v * s, v * c + u * s
            return pm.unit_rms(x, eps) if norm == "unit" else x
        want_q, want_k = prepared(P[:, :qn], heads, w[0]), prepared(P[:, qn:qn + kn], kv_heads, w[1])
        want_v = P[:, qn + kn:].reshape(b.tokens, kv_heads, dv)
        assert float((q.double().cpu().view(b.tokens, heads, d) - want_q).abs().max()) < bound * float(want_q.abs().max()), dtype
        for e in range(b.entries):
            K, V = held(cache, b, e, page, kv_heads, d, dv)
            lo, hi = b.cu[e], b.cu[e + 1]
            assert float((K[:hi - lo] - want_k[lo:hi]).abs().max()) < bound * float(want_k.abs().max()), dtype
            assert float((V[:hi - lo] - want_v[lo:hi]).abs().max()) < bound * float(want_v.abs().max()), dtype


@pytest.mark.parametrize("heads,d,dv", [(2, 64, 64), (3, 7, 5), (1, 1, 1), (4, 128, 32), (2, 40, 72), (1, 256, 16), (5, 16, 33)])
def test_lightning_kernels_against_the_recurrence_written_out(heads, d, dv):
    """silu on q, k and v, the walk token by token (from the projection and from prepared rows) and the chunked kernel (in
    one pass and in segments), from non-zero states, with entries of 1, 15, 64, 65 and 700 tokens in one step; outputs and
    the states they leave; the joint norm with its gate."""
    from sparseengine_b200.csrc import ops
    g = torch.Generator(device=DEV).manual_seed(heads + d)
    q_lens, rows = [15, 1, 700, 64, 65, 128], [2, 0, 4, 1, 5, 3]
    b = batch(q_lens, q_lens, DEV, 16, rows)
    n, m = heads * d, heads * dv
    decays = [1.0, 0.3, 0.999, 0.9, 0.97][:heads]
    decay = torch.tensor(decays, device=DEV)
    state0 = torch.randn(6, n * dv + 4, generator=g, device=DEV)        # rows wider than the state
    for dtype, bound in ((torch.float32, 1e-5), (torch.bfloat16, 1e-4)):
        proj = torch.randn(b.tokens, 2 * n + 2 * m + 5, generator=g, device=DEV).to(dtype)
        P = proj.double().cpu()
        q, k = (pm.silu(P[:, i * n:(i + 1) * n]).view(-1, heads, d) for i in range(2))
        v = pm.silu(P[:, 2 * n:2 * n + m]).view(-1, heads, dv)
        want, left = torch.zeros(b.tokens, heads, dv, dtype=torch.float64), state0.double().cpu().clone()
        for e in range(b.entries):
            s = slice(b.cu[e], b.cu[e + 1])
            want[s], S = pm.recurrence(q[s], k[s], v[s], decays, left[rows[e], :n * dv].view(heads, d, dv))
            left[rows[e], :n * dv] = S.reshape(-1)
        q32, k32 = (torch.full((b.tokens, n), float("nan"), device=DEV) for _ in range(2))
        ops.retention_prep(proj, 0, n, None, b.positions, q32, k32, heads=heads, head_dim=d, rotary_dim=0, k_scale=1.0, silu=True)
        assert float((q32.double().cpu() - q.reshape(-1, n)).abs().max()) < 1e-5 and float((k32.double().cpu() - k.reshape(-1, n)).abs().max()) < 1e-5
        sizes = dict(heads=heads, head_dim=d, v_head_dim=dv, silu=True)
        ways = [("direct", lambda *a: ops.retention_scan(None, None, *a, qk=(0, n, 1.0), **sizes)),
                ("prepared", lambda *a: ops.retention_scan(q32, k32, *a, **sizes)),
                ("chunks", lambda *a: ops.retention_chunk(q32, k32, *a, segments=(1, 0), **sizes)),
                ("segments", lambda *a: ops.retention_chunk(q32, k32, *a, segments=(6, 128), **sizes))]
        for name, fn in ways:
            state, o = state0.clone(), torch.full((b.tokens, m), float("nan"), device=DEV)
            fn(proj, 2 * n, decay, state, b, o)
            assert bool(torch.isfinite(o).all()), name
            assert float((o.double().cpu().view_as(want) - want).abs().max()) < bound * float(want.abs().max()), (name, dtype)
            assert float((state.double().cpu() - left).abs().max()) < bound * float(left.abs().max()), (name, dtype)
        # a factor on k and a rotation go with the activation too
        inv = torch.tensor([0.5], device=DEV)
        if d >= 2:
            ops.retention_prep(proj, 0, n, inv, b.positions, q32, k32, heads=heads, head_dim=d, rotary_dim=2, k_scale=0.25, silu=True)
            ang = b.positions.double().cpu()[:, None] * 0.5
            u, x = k[..., 0], k[..., 1]
            rot_k = torch.cat([(u * ang.cos() - x * ang.sin())[..., None], (x * ang.cos() + u * ang.sin())[..., None], k[..., 2:]], -1) * 0.25
            assert float((k32.double().cpu().view_as(k) - rot_k).abs().max()) < 2e-4
        w = (1 + 0.3 * torch.randn(m, generator=g, device=DEV)).to(dtype)
        out = torch.full((b.tokens, m), float("nan"), dtype=dtype, device=DEV)
        ops.retention_out_joint(o, proj, 2 * n + m, w, out, eps=1e-3)
        joint = pm.norm(o.double().cpu(), w.double().cpu(), 1e-3) * torch.sigmoid(P[:, 2 * n + m:2 * n + 2 * m])
        assert float((out.double().cpu() - joint).abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2) * float(joint.abs().max())
    ops.error_check(DEV)


@pytest.mark.parametrize("width", [3, 8, 40, 54, 1000, 1024, 2048, 4096, 5120, 8192, 12288, 16384, 16400, 20000])
def test_norms_around_a_sublayer(width):
    """One result, two normed results, none; with and without the norm after it, the stream, the norm before the next
    and its storing; rows picked by index: against the same in 64-bit."""
    from sparseengine_b200.csrc import ops
    g = torch.Generator(device=DEV).manual_seed(width)
    eps = (1e-3, 1e-2, 1e-4)
    for rows, dtype, bound in ((3, torch.float32, 1e-5), (3, torch.bfloat16, 8e-3), (1100, torch.bfloat16, 8e-3)):
        if rows > 3 and width > 4096:
            continue
        x0 = torch.randn(rows, width, generator=g, device=DEV) * 2
        y0, y1 = (torch.randn(rows, width, generator=g, device=DEV).to(dtype) * s for s in (1.0, 5.0))
        w0, w1, wp, wn = ((1 + 0.3 * torch.randn(width, generator=g, device=DEV)).to(dtype) for _ in range(4))
        d = [t.double() for t in (x0, y0, y1, w0, w1, wp, wn)]
        two = 0.5 * pm.norm(d[1], d[3], eps[0]) - 0.25 * pm.norm(d[2], d[4], eps[0])
        pair = ((y0, w0, 0.5), (y1, w1, -0.25), eps[0])
        idx = torch.tensor([2, 0, 2, 1], dtype=torch.int32, device=DEV)
        for y, c in ((y0, d[1]), (pair, two), (None, None)):
            for post in ((wp, eps[1]), None):
                if y is None and post is not None:
                    continue
                v = d[0] if c is None else d[0] + (pm.norm(c, d[5], eps[1]) if post else c)
                normed = pm.norm(v, d[6], eps[2])
                stream, out = x0.clone(), torch.full((rows, width), float("nan"), dtype=dtype, device=DEV)
                ops.sandwich_norm(stream, y, post=post, following=(wn, eps[2]), out=out)
                assert float((stream.double() - v).abs().max()) < 1e-5 * float(v.abs().max())
                assert float((out.double() - normed).abs().max()) < bound * float(normed.abs().max())
                stream, picked = x0.clone(), torch.full((4, width), float("nan"), dtype=dtype, device=DEV)
                ops.sandwich_norm(stream, y, post=post, following=(wn, eps[2]), out=picked, rows=idx, store=False)
                assert torch.equal(stream, x0) and torch.equal(picked, out[idx.long()])
                ops.sandwich_norm(stream, y, post=post, dtype=dtype)                     # the stream alone
                assert float((stream.double() - v).abs().max()) < 1e-5 * float(v.abs().max())
                if y is not None:                                                        # no stream: the result alone
                    ops.sandwich_norm(None, y, post=post, out=out)
                    alone = v - d[0]
                    assert float((out.double() - alone).abs().max()) < bound * float(alone.abs().max())


@pytest.mark.parametrize("kind", ["silu", "clamped_swiglu", "gelu_tanh"])
def test_gated_activations(kind):
    """The activation after a product and inside the few-row product, and the experts' kernels with the new one, against
    the equations; large arguments of both signs included."""
    from sparseengine_b200.config.specs import DenseMLPSpec, MoESpec
    from sparseengine_b200.csrc import ops
    from sparseengine_b200.parts.base import make_feed_forward
    act = (kind, 0.8, 1.702) if kind == "clamped_swiglu" else kind

    def gate(z, u):
        if kind == "silu":
            return pm.silu(z) * u
        if kind == "gelu_tanh":
            return pm.gelu_tanh(z) * u
        z = z.clamp(max=0.8)
        return z * torch.sigmoid(1.702 * z) * (u.clamp(-0.8, 0.8) + 1)
    g = torch.Generator(device=DEV).manual_seed(3)
    for rows, width in ((5, 8), (33, 1), (7, 37), (300, 256), (2, 4096)):
        for dtype, bound in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2)):
            x = (torch.randn(rows, 2 * width, generator=g, device=DEV) * 3).to(dtype)
            x[0, 0], x[1, 0] = 60.0, -60.0
            out = torch.full((rows, width), float("nan"), dtype=dtype, device=DEV)
            ops.glu(x, out, act)
            want = gate(x.double()[:, :width], x.double()[:, width:])
            assert float((out.double() - want).abs().max()) < bound * float(want.abs().max())
    for rows, n, k in ((1, 8, 32), (8, 100, 96), (5, 1, 4096), (16, 77, 4128), (9, 640, 160)):
        x, w = torch.randn(rows, k, generator=g, device=DEV).bfloat16(), (torch.randn(2 * n, k, generator=g, device=DEV) * 2 / k ** 0.5).bfloat16()
        out = torch.full((rows, n), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.gemv_glu(x, w, out, act)
        y = x.double() @ w.double().T
        want = gate(y[:, :n], y[:, n:])
        assert float((out.double() - want).abs().max()) < 2e-2 * float(want.abs().max()), (rows, n, k)
    width, ff, limit = 64, 48, dict(activation_limit=0.8) if kind == "clamped_swiglu" else {}
    w13, w2 = torch.randn(2, 2 * ff, width, generator=g, device=DEV) / 8, torch.randn(2, width, ff, generator=g, device=DEV) / 7
    for dtype, bound in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
        for rows in (3, 70, 1500):
            x = torch.randn(rows, width, generator=g, device=DEV).to(dtype)
            a, b = w13.to(dtype), w2.to(dtype)
            want = [gate(*(x.double() @ a[e].double().T).split(ff, -1)) @ b[e].double().T for e in range(2)]
            part = make_feed_forward(DenseMLPSpec(hidden_size=width, intermediate_size=ff, activation=kind, **limit), dtype)
            part.bind({"w13": a[:1].contiguous(), "w2": b[:1].contiguous()})
            assert float((part.forward(x, None).double() - want[0]).abs().max()) < bound * float(want[0].abs().max()), (dtype, rows)
            moe = make_feed_forward(MoESpec(hidden_size=width, num_experts=2, top_k=2, intermediate_size=ff, activation=kind, **limit), dtype)
            moe.bind({"w13": a, "w2": b, "gate": torch.zeros(2, width, device=DEV), "selection_bias": torch.zeros(2, device=DEV)})
            for pair in (None, 64) if dtype == torch.bfloat16 else (None,):
                moe.pair_min_rows, moe.pair_min_rows_per_expert = pair, 1
                mean = 0.5 * (want[0] + want[1])
                assert float((moe.forward(x, None).double() - mean).abs().max()) < bound * float(mean.abs().max()), (dtype, rows, pair)
    ops.error_check(DEV)


def test_the_kernels_a_step_takes(folders):
    """bfloat16 steps of the wide model run on the tensor-core attention kernels, the chunked recurrence for prompt
    portions, and the fused norms; nothing falls back to the plain attention."""
    from sparseengine_b200.csrc import ops
    from sparseengine_b200.engine.runner import StepEntry
    folder, cfg, w = folders["wide"]
    toks = tu.random_prompt(cfg["vocab"], 60, 4)
    runner = make_runner(folder, "bfloat16", [{"step": 0, "entries": [{"id": "a", "tokens": toks}], "end": []}], decode_graphs=False)
    runner.admit("a")
    before = copy.copy(ops.calls)
    runner.step([StepEntry("a", toks[:-1], [0])])
    runner.step([StepEntry("a", toks[-1:], [0])])
    ran = {k for k, v in ops.calls.items() if v > before.get(k, 0)}
    assert {"se_attn_prefill", "se_attn_prefill_tc", "se_attn_decode", "se_retention_chunk", "se_retention_scan", "se_retention_out_joint",
            "se_sandwich_norm", "se_qk_prep_general", "se_glu", "se_gemv_glu"} <= ran
    assert not {"se_paged_attention_plain", "se_add_rmsnorm_stream", "se_scaled_sum"} & ran
    assert ops.limit("sandwich_norm_max_width") == ops.LIMITS["sandwich_norm_max_width"]
