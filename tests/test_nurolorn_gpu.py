"""The Nurolorn design in the engine against the plain implementation (tests/plain_nurolorn.py): each
mechanism alone, whole prompts against token-by-token decoding, portions down to two tokens, mixed
batches with pages and state slots that are used again, keys far away, at the window's two edges and at
page borders, the distance bias, a far token held by the recurrence, the first tokens, long decoding,
other sizes (also values equal to one another or to 1), greedy generation through ``LLM``, and the
design's kernels against one another and against the equations written out."""
import copy
import json
import os
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_nurolorn as pn
import trace_util as tu

pytestmark = pytest.mark.gpu


def dense(ff):
    return {"kind": "dense", "ff": ff}


def lat(heads, dim, rot_dim, vdim, kv_rank, scale=None, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def gru(width, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def att(heads, kv_heads, dim, vdim, window, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "scale": scale if scale is not None else 2.0 * dim ** -0.5}}


def config(width, vocab, layers, loop=None, groups=1, eps=1e-6, mult=0.8, logit_scale=1.5):
    c = {"architecture": "Nurolorn", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps, "groups": groups},
         "residual_mult": mult, "logit_scale": logit_scale}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


CONFIGS = {
    # the three mixers, layers with and without feed-forward, a loop from layer 0
    "hybrid": config(96, 160, [lat(6, 16, 8, 12, 24, mlp=dense(128)), gru(40, mlp=dense(72)), att(6, 3, 16, 12, 11),
                               lat(3, 8, 16, 20, 40, base=500.0)], loop=(0, 3, 2), groups=3, eps=1e-5, mult=0.6, logit_scale=1.7),
    # a loop in the middle, run three times; two windows (two page groups)
    "middle": config(64, 100, [att(4, 1, 8, 24, 7), gru(64, mlp=dense(96)), lat(2, 16, 16, 16, 32), att(2, 2, 24, 8, 20, mlp=dense(48)),
                               gru(24)], loop=(1, 3, 3), groups=2, mult=1.3),
    # sizes that bfloat16 steps give to the tensor-core kernels (row pitches of 16 bytes)
    "wide": config(128, 200, [lat(4, 32, 32, 32, 64, mlp=dense(192)), att(4, 2, 64, 64, 33, mlp=dense(192)), gru(160, mlp=dense(192)),
                              att(2, 1, 128, 128, 50), lat(8, 16, 16, 32, 48)], loop=(1, 3, 2), groups=4, mult=0.5, logit_scale=3.0),
    # sizes that are equal or 1: one head, one group, a window of one key, a loop of one pass, factors of 1
    "ones": config(32, 48, [att(1, 1, 32, 32, 1, mlp=dense(32)), lat(1, 32, 32, 32, 32, mlp=dense(32)), gru(32, mlp=dense(32))],
                   loop=(0, 3, 1), mult=1.0, logit_scale=1.0),
    # sizes that are multiples of nothing in particular; no loop
    "odd": config(54, 77, [gru(37, mlp=dense(30)), lat(5, 6, 2, 7, 13, mlp=dense(11)), att(5, 5, 7, 3, 19), lat(3, 10, 6, 3, 5),
                           gru(1)], groups=9, eps=1e-4, mult=0.37, logit_scale=0.9),
}


def write_folder(folder, cfg, seed, w=None):
    from safetensors.torch import save_file
    w = w if w is not None else pn.random_weights(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return w


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("nur_" + name))
        out[name] = (d, cfg, write_folder(d, cfg, 61 + i))
    return out


_plain_cache = {}


def plain_logits(cfg, w, seqs):
    out = {}
    for sid, toks in seqs.items():
        key = (json.dumps(cfg, sort_keys=True), float(w["embed"].float().sum()), tuple(toks))
        if key not in _plain_cache:
            _plain_cache[key] = pn.forward(cfg, w, toks).float().numpy()
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


# 32-bit: every row within 3e-5.  bfloat16: rounding alone moves the rows of these small models by about one part in a
# hundred, so nine rows of ten must lie within 0.05 and every row within 0.15; a fault of the cache, the state or a
# window moves every row behind it by its whole size.
BOUND32 = 3e-5


def assert_close(got, ref, dtype, what, bound=None):
    errs = row_errors(got, ref)
    v = np.array(list(errs.values()))
    where = max(errs, key=errs.get)
    if bound is not None or dtype == "float32":
        limit = bound or BOUND32
        assert v.max() < limit, f"{what} ({dtype}): row error {v.max():.3e} at {where}"
        return
    assert np.quantile(v, 0.9) < 0.05, f"{what} ({dtype}): nine rows of ten within {np.quantile(v, 0.9):.3e}"
    assert v.max() < 0.15, f"{what} ({dtype}): row error {v.max():.3e} at {where}"


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
    "latent_attention": ([lat(4, 8, 6, 12, 16)], {}),
    "mingru": ([gru(52)], {}),
    "windowed_attention_with_distance_bias": ([att(4, 2, 12, 20, 9)], {}),
    "feed_forward": ([gru(8, mlp=dense(80))], {}),
    "norm_in_groups": ([gru(8, mlp=dense(16))], {"groups": 8, "eps": 0.3}),
    "residual_and_logit_factors": ([gru(24, mlp=dense(40))], {"mult": 2.5, "logit_scale": 0.3}),
    "loop": ([gru(16), att(2, 1, 8, 8, 5)], {"loop": (0, 2, 4)}),
    "loop_of_the_last_layer": ([gru(16), lat(2, 8, 4, 8, 8)], {"loop": (1, 2, 3)}),
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
    seqs = prompts(CONFIGS["middle"], (60, 5, 1, 9), 40)
    check_trace(folders, "middle", "float32", tu.trace_chunks(seqs, sizes=(7, 2)), seqs, "one slot", rows=1)


# ---- places where a fault would sit --------------------------------------------------------------

def sharp_window_model(window, dim=16, seed=9):
    """One windowed attention layer whose softmax is sharp (a large score scale), so that a query hangs
    on the one or two keys of its window with the highest score: a key that is lost at the window's far edge,
    or one that is let in from beyond it, moves the row by much."""
    cfg = config(64, 80, [att(4, 2, dim, dim, window, scale=10.0 * dim ** -0.5, mlp=dense(64))], groups=2)
    return cfg, pn.random_weights(cfg, seed)


@pytest.mark.parametrize("dtype,dim", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64), ("bfloat16", 128)])
def test_the_windows_two_edges_and_page_borders(tmp_path, dtype, dim):
    """Window 37 over pages of 16: the oldest key a query sees wanders through every place of a
    page, in prompts, in portions that start and end anywhere, and in tokens decoded alone; pages
    behind the window are given back and used again meanwhile.  (In bfloat16 the rounding of queries
    and keys moves such sharp weights by itself, hence the wider bound; a lost key moves the row by
    its whole size.)"""
    cfg, w = sharp_window_model(37, dim)
    write_folder(str(tmp_path), cfg, 0, w)
    seqs = prompts(cfg, (150, 37, 38, 36, 16, 95), 60)
    fs = {"edge": (str(tmp_path), cfg, w)}
    bound = 0.3 if dtype == "bfloat16" else None
    check_trace(fs, "edge", dtype, tu.trace_whole(seqs), seqs, "window, whole", bound)
    check_trace(fs, "edge", dtype, tu.trace_tail_decode(seqs, tail=60), seqs, "window, decoded", bound)
    check_trace(fs, "edge", dtype, tu.trace_chunks(seqs, sizes=(15, 2, 16, 33, 1, 37, 38)), seqs, "window, portions", bound)
    check_trace(fs, "edge", dtype, tu.trace_mixed(seqs, live=3, chunk=21, decode_tail=40), seqs, "window, mixed", bound, rows=3)


def far_key_model(seed=13):
    """One latent attention layer with a sharp softmax over all earlier keys: queries hang on single keys
    anywhere in the sequence."""
    cfg = config(64, 80, [lat(4, 16, 16, 16, 32, scale=1.5, mlp=dense(64))], groups=4)
    return cfg, pn.random_weights(cfg, seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_of_the_latent_attention(tmp_path, dtype):
    cfg, w = far_key_model()
    write_folder(str(tmp_path), cfg, 0, w)
    seqs = prompts(cfg, (430, 131, 64, 7), 80)
    fs = {"far": (str(tmp_path), cfg, w)}
    bound = 0.35 if dtype == "bfloat16" else 6e-5
    check_trace(fs, "far", dtype, tu.trace_whole(seqs), seqs, "far keys, whole", bound)
    check_trace(fs, "far", dtype, tu.trace_chunks(seqs, sizes=(100, 2, 33, 1, 64)), seqs, "far keys, portions", bound)
    check_trace(fs, "far", dtype, tu.trace_tail_decode(seqs, tail=40), seqs, "far keys, decoded", bound)
    check_trace(fs, "far", dtype, tu.trace_mixed(seqs, live=3, chunk=50, decode_tail=30), seqs, "far keys, mixed", bound, rows=3)


def slow_state_model(seed=12):
    cfg = config(48, 64, [gru(80, mlp=dense(64))], groups=2)
    w = pn.random_weights(cfg, seed)
    w["l0.mix.z.b"] = (w["l0.mix.z.b"].float() - 3.5).to(torch.bfloat16)         # forget slowly
    return cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_token_held_by_the_recurrence(tmp_path, dtype):
    """The model's only mixer is the recurrence and it forgets slowly: what the first tokens left reaches
    position 400 through the state alone.  A state that is lost at a portion's start or copied to the
    wrong slot shows there."""
    cfg, w = slow_state_model()
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
    """140 tokens decoded one by one, far past every window, through replayed CUDA graphs."""
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


def test_the_stream_after_every_layer_run(folders):
    """The 32-bit stream after each visit of the execution order (a looped layer counts each time)
    against the plain implementation's."""
    from sparseengine_b200.engine.runner import StepEntry
    folder, cfg, w = folders["middle"]
    toks = tu.random_prompt(cfg["vocab"], 45, 8)
    taps = []
    pn.forward(cfg, w, toks, taps)
    assert len(taps) == 1 + 3 * 2 + 2
    runner = make_runner(folder, "float32", [{"step": 0, "entries": [{"id": "a", "tokens": toks}], "end": []}])
    runner.model.stream_taps = got = []
    runner.admit("a")
    runner.step([StepEntry("a", toks, [0])])
    assert len(got) == len(taps)
    for i, (a, b) in enumerate(zip(got, taps)):
        assert float((a.cpu().double() - b).abs().max()) < 3e-5 * float(b.abs().max()), i


# ---- the entry point -----------------------------------------------------------------------------

def plain_greedy(cfg, w, prompt, steps):
    toks, out, margins = list(prompt), [], []
    for _ in range(steps):
        logits = pn.forward(cfg, w, toks)[-1]
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


@pytest.mark.parametrize("d,dv,heads,kv_heads,window,steep", [(64, 64, 4, 2, 33, 1.0), (128, 64, 6, 1, 70, 0.1), (64, 32, 2, 2, 5, 12.0),
                                                               (128, 128, 8, 2, 100, 1.0), (128, 128, 6, 6, None, 0.02), (64, 128, 3, 3, None, 1.0)])
def test_distance_bias_in_the_attention_kernels(d, dv, heads, kv_heads, window, steep):
    """The same queries, pages and block table through the plain kernel, the split-key kernel and the prompt-portion
    kernels with a bias per token of distance (steep and almost flat ones); the plain kernel against the
    equations in 64-bit; and that the bias matters."""
    from sparseengine_b200.csrc import ops
    dev, page = "cuda:0", 16
    g = torch.Generator(device=dev).manual_seed(d + heads)
    q_lens, kv_lens = [37, 1, 130, 1, 2, 1], [37, 64, 209, 140, 17, 3]
    b = batch(q_lens, kv_lens, dev, page, [3, 0, 4, 1, 5, 2])
    cache = (torch.randn(b.pages, page * kv_heads * (d + dv), generator=g, device=dev) * 0.7).to(torch.bfloat16)
    q = torch.randn(b.tokens, heads * d, generator=g, device=dev).to(torch.bfloat16)
    slopes = torch.tensor([steep * 2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float32, device=dev)
    scale = d ** -0.5 * 2.0
    common = dict(num_heads=heads, num_kv_heads=kv_heads, head_dim=d, page_size=page, scale=scale, window=window,
                  v_head_dim=dv, slopes=slopes)
    plain = torch.empty(b.tokens, heads * dv, dtype=torch.bfloat16, device=dev)
    ops.paged_attention_plain(q, cache, b.table, b.seq_rows, b.token_seq, b.positions, plain, **common)
    portions = torch.full_like(plain, float("nan"))
    ops.attn_prefill(q, cache, b.table, b.seq_rows, b.cu_q, b.kv_len, portions, entries=b.entries, max_q_len=b.max_q_len, **common)
    split = torch.full_like(plain, float("nan"))
    ops.attn_decode(q, cache, b.table, b.seq_rows, b.token_seq, b.positions, split,
                    max_keys=max(kv_lens) if window is None else min(max(kv_lens), window), **common)
    others = [(portions, "portions"), (split, "split keys")]
    if d == dv and ops.attn_prefill_tc_supported(d, heads, kv_heads):
        tc = torch.full_like(plain, float("nan"))
        ops.attn_prefill_tc(q, cache.view(-1, 2, kv_heads, page, d), b.table, b.seq_rows, b.cu_q, b.kv_len, tc, entries=b.entries,
                            max_q_len=b.max_q_len, **common)
        others.append((tc, "portions, tensor memory"))
    ops.error_check(dev)
    # the equations, with and without the bias
    want, flat = (torch.zeros(b.tokens, heads, dv, dtype=torch.float64) for _ in range(2))
    c = cache.double().cpu()
    keys = c[:, :page * kv_heads * d].reshape(-1, kv_heads, page, d)
    vals = c[:, page * kv_heads * d:].reshape(-1, kv_heads, page, dv)
    for e in range(b.entries):
        pages = b.table.cpu()[b.seq_rows.cpu()[e].item()].long()
        K = keys[pages].transpose(1, 2).reshape(-1, kv_heads, d).repeat_interleave(heads // kv_heads, 1)
        V = vals[pages].transpose(1, 2).reshape(-1, kv_heads, dv).repeat_interleave(heads // kv_heads, 1)
        for t in range(b.cu[e], b.cu[e + 1]):
            p = int(b.positions[t])
            lo = 0 if window is None else max(0, p - window + 1)
            s = torch.einsum("hd,jhd->hj", q[t].double().cpu().view(heads, d), K[lo:p + 1]) * scale
            dist = (p - torch.arange(lo, p + 1)).double()
            for out, sc in ((want, s - slopes.double().cpu()[:, None] * dist), (flat, s)):
                out[t] = torch.einsum("hj,jhd->hd", torch.softmax(sc, -1), V[lo:p + 1])
    want, flat = want.reshape(b.tokens, -1), flat.reshape(b.tokens, -1)
    most = float(want.abs().max())
    assert float((want - flat).abs().max()) > 0.1 * most
    assert float((plain.double().cpu() - want).abs().max()) < 1.5e-2 * most
    for other, what in others:
        assert bool(torch.isfinite(other.float()).all()), what
        assert float((other.float() - plain.float()).abs().max()) < 3e-2 * most, what


@pytest.mark.parametrize("rank,rot,heads,d", [(64, 32, 4, 16), (80, 48, 5, 8), (32, 16, 80, 8), (192, 64, 3, 40), (48, 2, 2, 6), (13, 6, 3, 5)])
def test_latent_attention_with_neighbouring_pairs(rank, rot, heads, d):
    """Preparation and attention with neighbours rotated in pairs, queries and latent read from the columns of one
    projection: the page rows against the equations, the kernel per token and head against the equations, and
    the tiled kernel against it where it takes the sizes."""
    from sparseengine_b200.csrc import ops
    dev, page, D, base = "cuda:0", 16, rank + rot, 300.0
    g = torch.Generator(device=dev).manual_seed(rank + heads)
    q_lens, kv_lens = [37, 1, 130, 2], [37, 1, 130, 2]              # whole prompts: the page rows all come from this step
    b = batch(q_lens, kv_lens, dev, page, [2, 0, 3, 1])
    cols, scale, eps = heads * (d + rot), 2.0 * (d + rot) ** -0.5, 1e-5
    inv_freq = (base ** (-torch.arange(0, rot, 2, dtype=torch.float64) / rot)).float().to(dev)
    kv_w = 1.0 + 0.2 * torch.randn(rank, generator=g, device=dev)
    for dtype, bound in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        proj = torch.randn(b.tokens, cols + D + 7, generator=g, device=dev).to(dtype)
        cache = torch.full((b.pages, page, D), float("nan"), dtype=dtype, device=dev)
        w = kv_w.to(dtype)
        ops.latent_prep(proj[:, cols:cols + D], None, w, inv_freq, b.positions, b.token_seq, b.seq_rows, b.table, cache, None,
                        q_rank=0, rank=rank, rot=rot, rotary_dim=rot, eps=eps, page_size=page, pairing="interleaved")
        q = proj[:, :cols]
        uk = (torch.randn(heads, d, rank, generator=g, device=dev) * d ** -0.5).to(dtype)
        q_lat = torch.einsum("thd,hdr->htr", q.float().view(b.tokens, heads, d + rot)[..., :d], uk.float()).contiguous()
        plain = torch.full((b.tokens, heads, rank), float("nan"), dtype=dtype, device=dev)
        ops.latent_attention_plain(q_lat, q, inv_freq, cache, b.table, b.seq_rows, b.token_seq, b.positions, None, plain,
                                   heads=heads, head_dim=d, rank=rank, rot=rot, rotary_dim=rot, page_size=page, scale=scale,
                                   pairing="interleaved")
        P = proj.double().cpu()
        want = torch.zeros(b.tokens, heads, rank, dtype=torch.float64)
        for e in range(b.entries):
            lo, hi = b.cu[e], b.cu[e + 1]
            pos = b.positions[lo:hi].cpu()
            lat_rows = pn.unit_rms(P[lo:hi, cols:cols + rank], eps) * w.double().cpu()
            k_rot = pn.rotate_neighbours(P[lo:hi, None, cols + rank:cols + D], pos, rot, base)[:, 0]
            pages = b.table.cpu()[b.seq_rows.cpu()[e].item()].long()
            held = cache.double().cpu()[pages].reshape(-1, D)[:hi - lo]
            assert float((held - torch.cat([lat_rows, k_rot], -1)).abs().max()) < bound * 5
            q_rot = pn.rotate_neighbours(P[lo:hi, :cols].view(-1, heads, d + rot)[..., d:], pos, rot, base)
            s = (torch.einsum("hir,jr->hij", q_lat.double().cpu()[:, lo:hi], held[:, :rank])
                 + torch.einsum("ihr,jr->hij", q_rot, held[:, rank:])) * scale
            want[lo:hi] = torch.einsum("hij,jr->ihr", pn.causal_softmax(s), held[:, :rank])
        assert float((plain.double().cpu() - want).abs().max()) < bound * float(want.abs().max()), dtype
        if dtype == torch.bfloat16 and ops.latent_attention_tiled_supported(rank, rot):
            qfull = torch.empty(b.tokens, heads, D, dtype=dtype, device=dev)
            qfull[:, :, :rank] = q_lat.transpose(0, 1)
            # the rotated parts by the kernel of their own, and by the preparation (which writes the same page rows again)
            ops.latent_q_rotate(q, inv_freq, b.positions, qfull, heads=heads, head_dim=d, rank=rank, rot=rot, rotary_dim=rot,
                                pairing="interleaved")
            again = torch.zeros_like(qfull)
            ops.latent_prep(proj[:, cols:cols + D], None, w, inv_freq, b.positions, b.token_seq, b.seq_rows, b.table, cache, None,
                            q_rank=0, rank=rank, rot=rot, rotary_dim=rot, eps=eps, page_size=page, pairing="interleaved",
                            queries=(q, heads, d, again))
            assert torch.equal(again[:, :, rank:], qfull[:, :, rank:]) and not bool(again[:, :, :rank].any())
            tiled = torch.full_like(plain, float("nan"))
            ops.latent_attention_tiled(qfull, cache, b.table, b.seq_rows, b.cu_q, b.kv_len, None, tiled, entries=b.entries,
                                       max_q_len=b.max_q_len, heads=heads, rank=rank, rot=rot, page_size=page, scale=scale)
            assert float((tiled.float() - plain.float()).abs().max()) < 3e-2 * float(want.abs().max())
    ops.error_check(dev)


@pytest.mark.parametrize("width", [1, 37, 64, 130, 512])
def test_min_gru_kernels_against_the_recurrence_written_out(width):
    """The walk token by token and the chunked kernel in clusters of one to eight CTAs, from non-zero states, with entries
    of 1, 15, 16, 17, 128, 129 and 1,100 tokens in one step; outputs and the states they leave."""
    from sparseengine_b200.csrc import ops
    dev = "cuda:0"
    g = torch.Generator(device=dev).manual_seed(width)
    q_lens = [15, 1, 1100, 16, 17, 129, 128]
    rows = [2, 0, 4, 1, 6, 5, 3]
    b = batch(q_lens, q_lens, dev, 16, rows)
    bias = torch.cat([torch.randn(width, generator=g, device=dev) - 3.0, torch.randn(width, generator=g, device=dev) * 0.5])
    state0 = torch.randn(7, width + 3, generator=g, device=dev)[:, :width + 2].contiguous()       # rows wider than the state
    for dtype, bound in ((torch.float32, 1e-5), (torch.bfloat16, 6e-3)):
        proj = torch.randn(b.tokens, 3 * width, generator=g, device=dev).to(dtype)
        P, B = proj.double().cpu(), bias.double().cpu()
        z = torch.sigmoid(P[:, :width] + B[:width])
        u = P[:, width:2 * width] + B[width:]
        cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        want, left = torch.zeros(b.tokens, width, dtype=torch.float64), state0.double().cpu().clone()
        for e in range(b.entries):
            S = left[rows[e], :width].clone()
            for t in range(b.cu[e], b.cu[e + 1]):
                S = (1 - z[t]) * S + z[t] * cand[t]
                want[t] = S
            left[rows[e], :width] = S
        want = want * pn.silu(P[:, 2 * width:])
        for fn, kw in ((ops.min_gru_scan, {}), *((ops.min_gru_chunk, {"ctas": n}) for n in (1, 2, 4, 8)), (ops.min_gru_chunk, {})):
            state = state0.clone()
            out = torch.full((b.tokens, width), float("nan"), dtype=dtype, device=dev)
            fn(proj, bias, state, b, out, **kw)
            assert bool(torch.isfinite(out.float()).all()), (fn.__name__, kw)
            assert float((out.double().cpu() - want).abs().max()) < bound * float(want.abs().max()), (fn.__name__, kw)
            assert float((state.double().cpu() - left).abs().max()) < 1e-5 * float(left.abs().max()), (fn.__name__, kw)


@pytest.mark.parametrize("width,groups", [(40, 1), (40, 5), (64, 64), (54, 9), (1024, 2), (1032, 43), (4096, 8), (8192, 4), (8192, 1024), (7, 7)])
def test_stream_norm_in_groups_with_what_a_pass_adds(width, groups):
    """x + alpha y + table[id] scale + step, and its norm in groups, against the same in 64-bit; every addend present
    and left out."""
    from sparseengine_b200.csrc import ops
    dev, rows, vocab, eps = "cuda:0", 5, 11, 1e-4
    g = torch.Generator(device=dev).manual_seed(width + groups)
    spread = torch.linspace(0.1, 5.0, width, device=dev)        # parts of very different size
    x0 = torch.randn(rows, width, generator=g, device=dev) * spread
    step = torch.randn(width, generator=g, device=dev)
    ids = torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32, device=dev)
    for dtype, bound in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        y = torch.randn(rows, width, generator=g, device=dev).to(dtype)
        w = (1.0 + 0.2 * torch.randn(width, generator=g, device=dev)).to(dtype)
        table = torch.randn(vocab, width, generator=g, device=dev).to(dtype)
        for has_y, inject in ((True, (table, ids, 0.7, step)), (True, None), (False, (None, None, 0.0, step)), (True, (table, ids, 1.0, None)),
                              (False, None)):
            v = x0.double()
            if has_y:
                v = v + 0.3 * y.double()
            if inject is not None and inject[0] is not None:
                v = v + inject[2] * table.double()[ids.long()]
            if inject is not None and inject[3] is not None:
                v = v + step.double()
            want = pn.grouped_norm(v, w.double(), groups, eps)
            x, out = x0.clone(), torch.full((rows, width), float("nan"), dtype=dtype, device=dev)
            ops.add_rmsnorm_stream(x, y if has_y else None, w, eps, out32=x, out_act=out, alpha=0.3, groups=groups, inject=inject)
            assert float((x.double() - v).abs().max()) < 1e-5 * float(v.abs().max())
            assert float((out.double() - want).abs().max()) < bound * float(want.abs().max())


@pytest.mark.parametrize("width,pitch,at", [(48, 200, 8), (48, 201, 3), (33, 77, 5), (4096, 9000, 16)])
def test_sigmoid_gate(width, pitch, at):
    from sparseengine_b200.csrc import ops
    g = torch.Generator(device="cuda:0").manual_seed(width)
    for dtype, bound in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
        x = torch.randn(9, width, generator=g, device="cuda:0").to(dtype)
        gate = (torch.randn(9, pitch, generator=g, device="cuda:0") * 4).to(dtype)[:, at:at + width]
        want = x.double() * torch.sigmoid(gate.double())
        ops.sigmoid_gate_(x, gate)
        assert float((x.double() - want).abs().max()) < bound * float(want.abs().max())


def test_the_kernels_a_step_takes(folders):
    """bfloat16 steps of the wide model run on the tensor-core attention kernels, the tiled latent attention and, for
    prompt portions, the chunked recurrence."""
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
    assert {"se_attn_prefill", "se_attn_prefill_tc", "se_attn_decode", "se_latent_attention_tiled", "se_min_gru_chunk",
            "se_min_gru_scan", "se_add_rmsnorm_stream", "se_sigmoid_gate", "se_qk_prep_general"} <= ran
    assert not {"se_paged_attention_plain", "se_latent_attention_plain"} & ran
