"""Prefill and decode throughput of the Nurolorn design (latent attention over all keys with an output gate,
minGRU, windowed attention with a distance bias, squared-relu feed-forwards between norms in groups over a
scaled 32-bit stream, a looped stack) at layer sizes that resemble a real model's, beside the engine's
closest other model (the looped design Zisevik: latent attention with a window, retention) at equal width,
feed-forward size and number of layer visits, and each of the design's own kernels alone against its
roofline, with the like kernel of the closest models beside it.

    python -m sparseengine_b200.cli.nurolorn_bench [--sizes 2048,4096] [--steps 20] [--warmup 3]

Random weights, bfloat16, one GPU, device-timed with CUDA events; inputs differ from step to step
and the weights of a step exceed the L2 cache.  ``bench.py --design nurolorn`` prints the same
record as its one JSON line.
"""
from __future__ import annotations

import argparse
import copy
import json
import sys

import torch

from .hybrid_bench import PAGE_SIZE, VOCAB, _parts, _throughput
from .kernel_bench import peaks, timed
from .zisevik_bench import zisevik_config

WINDOW = 1024


def nurolorn_config(width: int) -> dict:
    """Four layers, the two in the middle run three times (eight visits: two latent attention over all keys, three
    minGRU, three windowed attention).  Latent attention: heads of 64 + 64 (rotated) query/key dims, values of 64, a
    cached row of 192 + 64; minGRU as wide as the model; attention: head size 128, four query heads per
    key/value head, a window of 1,024; feed-forwards of 4 x width; norms in two groups."""
    heads = width // 128
    ff = {"kind": "dense", "ff": 4 * width}
    lat = {"type": "latent_attention", "mlp": ff,
           "mixer": {"heads": 2 * heads, "dim": 64, "rot_dim": 64, "vdim": 64, "kv_rank": 192, "scale": 128 ** -0.5,
                     "rot": {"base": 1e6, "dims": 64}}}
    gru = {"type": "mingru", "mlp": ff, "mixer": {"width": width}}
    att = {"type": "attention", "mlp": ff,
           "mixer": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "mask": {"size": WINDOW}}}
    return {"architecture": "Nurolorn", "vocab": VOCAB, "width": width, "layers": [lat, gru, att, copy.deepcopy(lat)],
            "loop": {"start": 1, "stop": 3, "times": 3}, "norm": {"eps": 1e-6, "groups": 2}, "residual_mult": 0.7,
            "logit_scale": 1.5, "max_position": 16384}


def closest_config(width: int) -> dict:
    """The looped design Zisevik at the same width and number of visits, every feed-forward dense and of the same size."""
    cfg = zisevik_config(width)
    for layer in cfg["layers"]:
        layer["mlp"] = {"kind": "dense", "ff": 4 * width}
    return cfg


def _kernels(width: int, cases, pk: dict) -> dict:
    """Each kernel of the design alone: microseconds, the bytes it has to move (inputs read once, outputs
    written once) or the operations it has to do, and the share of the measured copy bandwidth or bfloat16
    matrix throughput that is; ``like: ...`` are the kernels of the closest models on inputs of the same size.
    ``cases``: (tokens, requests, keys each request already holds)."""
    from types import SimpleNamespace

    from ..csrc import ops
    dev = torch.device("cuda:0")
    cfg = nurolorn_config(width)
    lat, att = cfg["layers"][0]["mixer"], cfg["layers"][2]["mixer"]
    bf = torch.bfloat16
    out = {}
    for tokens, entries, held in cases:
        per = tokens // entries
        step = SimpleNamespace(token_seq=torch.arange(tokens, device=dev, dtype=torch.int32) // per,
                               cu_q=torch.arange(entries + 1, device=dev, dtype=torch.int32) * per,
                               seq_rows=torch.arange(entries, device=dev, dtype=torch.int32), num_seqs=entries, max_q_len=per,
                               positions=(torch.arange(tokens, device=dev, dtype=torch.int32) % per) + held)
        kv_len = torch.full((entries,), held + per, device=dev, dtype=torch.int32)
        rec = {}

        def add(name, fn, nbytes=None, flops=None, iters=20):
            ms = timed(fn, iters)
            r = {"us": round(ms * 1e3, 2)}
            if nbytes is not None:
                r.update(mbytes=round(nbytes / 1e6, 2), of_hbm_measured=round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 3))
            if flops is not None:
                r.update(gflop=round(flops / 1e9, 2), of_bf16_measured=round(flops / (ms * 1e-3) / 1e12 / pk["bf16_tflops"], 3))
            rec[name] = r

        # norm over the stream: in groups, with a factor, and with what a pass adds
        x32 = torch.randn(tokens, width, device=dev)
        y = torch.randn(tokens, width, device=dev, dtype=bf)
        w = torch.ones(width, device=dev, dtype=bf)
        oa = torch.empty_like(y)
        table = torch.randn(VOCAB, width, device=dev, dtype=bf)
        ids = torch.randint(0, VOCAB, (tokens,), device=dev, dtype=torch.int32)
        vec = torch.zeros(width, device=dev)
        add("add_rmsnorm_stream (two groups, factor)", lambda: ops.add_rmsnorm_stream(x32, y, w, 1e-6, out32=x32, out_act=oa, alpha=0.1, groups=2),
            tokens * width * 12)
        add("add_rmsnorm_stream (two groups, start of a pass)", lambda: ops.add_rmsnorm_stream(
            x32, y, w, 1e-6, out32=x32, out_act=oa, alpha=0.1, groups=2, inject=(table, ids, 0.1, vec)), tokens * width * 14)
        add("like: add_rmsnorm_stream (one group)", lambda: ops.add_rmsnorm_stream(x32, y, w, 1e-6, out32=x32, out_act=oa), tokens * width * 12)
        del table
        # latent attention
        H, d, r, dv, rank = lat["heads"], lat["dim"], lat["rot_dim"], lat["vdim"], lat["kv_rank"]
        D, cols = rank + r, lat["heads"] * (lat["dim"] + lat["rot_dim"])
        pages = -(-(held + per) // PAGE_SIZE)
        btable = torch.arange(entries * pages, device=dev, dtype=torch.int32).view(entries, pages)
        cache = (torch.randn(entries * pages, PAGE_SIZE, D, device=dev) * 0.5).to(bf)
        proj = torch.randn(tokens, cols + D + H * dv, device=dev, dtype=bf)
        kw = torch.ones(rank, device=dev, dtype=bf)
        inv = (1e6 ** (-torch.arange(0, r, 2, dtype=torch.float32) / r)).to(dev)
        cq, qw = torch.empty(tokens, width // 2, device=dev, dtype=bf), torch.ones(width // 2, device=dev, dtype=bf)
        qfull = torch.zeros(tokens, H, D, device=dev, dtype=bf)
        add("latent_prep (no query latent, neighbouring pairs, queries)", lambda: ops.latent_prep(
            proj[:, cols:cols + D], None, kw, inv, step.positions, step.token_seq, step.seq_rows, btable, cache, None, q_rank=0,
            rank=rank, rot=r, rotary_dim=r, eps=1e-6, page_size=PAGE_SIZE, pairing="interleaved",
            queries=(proj[:, :cols], H, d, qfull)), tokens * (D + H * r) * 4)
        proj_q = torch.randn(tokens, width // 2 + D, device=dev, dtype=bf)
        add("like: latent_prep (query latent, split halves)", lambda: ops.latent_prep(
            proj_q, qw, kw, inv, step.positions, step.token_seq, step.seq_rows, btable, cache, cq, q_rank=width // 2, rank=rank,
            rot=r, rotary_dim=r, eps=1e-6, page_size=PAGE_SIZE), tokens * (width // 2 + D) * 4)
        q = torch.randn(tokens, cols, device=dev, dtype=bf)
        add("like: latent_q_rotate (split halves)", lambda: ops.latent_q_rotate(
            q, inv, step.positions, qfull, heads=H, head_dim=d, rank=rank, rot=r, rotary_dim=r), tokens * H * r * 4)
        qfull[:, :, :rank].normal_()
        o_lat = torch.empty(tokens, H, rank, device=dev, dtype=bf)

        def tiled(window, sink):
            most = held + per if window is None else min(held + per, window + per - 1)
            ops.latent_attention_tiled(qfull, cache, btable, step.seq_rows, step.cu_q, kv_len, sink, o_lat, entries=entries,
                                       max_q_len=per, heads=H, rank=rank, rot=r, page_size=PAGE_SIZE, scale=0.09, window=window,
                                       max_keys=most)
        for name, window, sink in (("latent_attention_tiled (all keys)", None, None),
                                   ("like: latent_attention_tiled (window, sink)", WINDOW, torch.zeros(H, device=dev))):
            seen = sum(min(window or 1 << 30, held + i + 1) for i in range(per)) * entries
            key_rows = entries * (held + per if window is None else min(held + per, window + per - 1))
            add(name, lambda: tiled(window, sink), nbytes=key_rows * D * 2 + tokens * H * (D + rank) * 2, flops=2.0 * seen * H * (D + rank))
        heads_out = torch.randn(tokens, H * dv, device=dev, dtype=bf)
        add("sigmoid_gate", lambda: ops.sigmoid_gate_(heads_out, proj[:, cols + D:]), tokens * H * dv * 6)
        # windowed attention with a distance bias
        hq, hkv = att["heads"], att["kv_heads"]
        qn, kn = hq * 128, hkv * 128
        pr = torch.randn(tokens, qn + 2 * kn, device=dev, dtype=bf)
        cache2 = (torch.randn(entries * pages, 2, hkv, PAGE_SIZE, 128, device=dev) * 0.5).to(bf)
        q2, o2 = torch.empty(tokens, qn, device=dev, dtype=bf), torch.empty(tokens, qn, device=dev, dtype=bf)
        one = torch.ones(128, device=dev, dtype=bf)

        def prep(**kw):
            ops.qk_prep_general(pr, kw.pop("q_w", None), kw.pop("k_w", None), step.positions, step.token_seq, step.seq_rows, btable, cache2,
                                q2, num_heads=hq, num_kv_heads=hkv, head_dim=128, v_head_dim=128, eps=1e-6, page_size=PAGE_SIZE, **kw)
        add("qk_prep_general (per-head norms without weights)", lambda: prep(per_head_unit=True), tokens * (qn + 2 * kn) * 4)
        add("like: qk_prep_general (per-head norms with weights)", lambda: prep(q_w=one, k_w=one, per_head=True), tokens * (qn + 2 * kn) * 4)
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / hq) for h in range(hq)], device=dev)
        seen2 = sum(min(WINDOW, held + i + 1) for i in range(per)) * entries
        for name, sl in (("(distance bias)", slopes), ("", None)):
            pre = "" if sl is not None else "like: "
            if per > 1:
                add(f"{pre}attn_prefill_tc {name}".strip(), lambda: ops.attn_prefill_tc(
                    q2, cache2, btable, step.seq_rows, step.cu_q, kv_len, o2, entries=entries, max_q_len=per, num_heads=hq,
                    num_kv_heads=hkv, head_dim=128, page_size=PAGE_SIZE, scale=0.09, window=WINDOW, slopes=sl), flops=4.0 * seen2 * hq * 128)
            else:
                add(f"{pre}attn_decode {name}".strip(), lambda: ops.attn_decode(
                    q2, cache2, btable, step.seq_rows, step.token_seq, step.positions, o2, num_heads=hq, num_kv_heads=hkv, head_dim=128,
                    page_size=PAGE_SIZE, scale=0.09, window=WINDOW, max_keys=min(held + 1, WINDOW), slopes=sl),
                    nbytes=entries * min(held + 1, WINDOW) * hkv * 128 * 4)
        # minGRU, and retention over the same number of values
        prg = torch.randn(tokens, 3 * width, device=dev, dtype=bf)
        bias, state = torch.zeros(2 * width, device=dev), torch.zeros(entries, width, device=dev)
        yg = torch.empty(tokens, width, device=dev, dtype=bf)
        gru_bytes = tokens * width * 8 + entries * width * 8
        if per > 1:
            add("min_gru_chunk", lambda: ops.min_gru_chunk(prg, bias, state, step, yg), gru_bytes)
        else:
            add("min_gru_scan", lambda: ops.min_gru_scan(prg, bias, state, step, yg), gru_bytes)
        Hr, dr = width // 128, 128
        qk = vv = Hr * dr
        q32, k32 = torch.randn(tokens, qk, device=dev), torch.randn(tokens, qk, device=dev)
        prr = torch.randn(tokens, 2 * qk + 2 * vv, device=dev, dtype=bf) * 0.3
        decay = torch.linspace(0.95, 0.9999, Hr, device=dev)
        rstate, ro = torch.zeros(entries, Hr * dr * dr, device=dev), torch.empty(tokens, vv, device=dev)
        fn = ops.retention_chunk if per > 1 else ops.retention_scan
        add("like: " + fn.__name__, lambda: fn(q32, k32, prr, 2 * qk, decay, rstate, step, ro, heads=Hr, head_dim=dr, v_head_dim=dr),
            tokens * (2 * qk * 4 + vv * 6) + entries * Hr * dr * dr * 8, iters=5)
        # the feed-forward's activation
        up = torch.randn(tokens, 4 * width, device=dev, dtype=bf)
        add("activation (squared relu)", lambda: ops.activation_(up, "relu2"), tokens * 4 * width * 4)
        up.normal_()
        add("like: activation (tanh-form gelu)", lambda: ops.activation_(up, "gelu_tanh"), tokens * 4 * width * 4)
        out[f"tokens{tokens}_requests{entries}_held{held}"] = rec
        ops.error_check(dev)
    return out


def run(sizes=(2048, 4096), steps: int = 20, warmup: int = 3, kernels: bool = True, parts: bool = True) -> dict:
    torch.cuda.set_device(0)
    pk = peaks()
    points = [("prefill", 1, 2048), ("prefill", 1, 8192), ("prefill", 4, 2048), ("decode", 8, 2048), ("decode", 64, 2048)]
    rec = {"design": "Nurolorn", "closest": "Zisevik (looped), dense feed-forwards", "dtype": "bf16", "data": "synthetic", "peaks": pk, "sizes": {}}
    for width in sizes:
        mine, other = nurolorn_config(width), closest_config(width)
        one = {"layer_visits": 8, "nurolorn": _throughput(mine, points, steps, warmup), "closest": _throughput(other, points, steps, warmup)}
        if parts:
            one["nurolorn_parts_ms"] = _parts(mine, 2048, 8)
            one["closest_parts_ms"] = _parts(other, 2048, 8)
        if kernels:
            one["kernels"] = _kernels(width, [(2048, 1, 0), (8192, 4, 0), (64, 64, 2048)], pk)
        rec["sizes"][str(width)] = one
    return rec


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-parts", action="store_true")
    a = ap.parse_args(argv)
    print(json.dumps(run(tuple(int(s) for s in a.sizes.split(",")), a.steps, max(a.warmup, 3), not a.no_kernels, not a.no_parts)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
