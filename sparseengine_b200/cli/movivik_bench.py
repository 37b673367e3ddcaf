"""Prefill and decode throughput of the Movivik design (norms before and after each sublayer over a 32-bit stream,
attention within chunks, full attention beside lightning attention, gelu-gated feed-forwards) at layer sizes that
resemble a real model's, beside the engine's closest other model (Tedisun: attention beside a matrix memory, a delta
rule) at equal width, attention and feed-forward sizes and number of layers, and each of the design's own kernels
alone against its roofline, with the like kernel of the closest models beside it.

    python -m sparseengine_b200.cli.movivik_bench [--sizes 2048,4096] [--steps 20] [--warmup 3]

Random weights, bfloat16, one GPU, device-timed with CUDA events; inputs differ from step to step
and the weights of a step exceed the L2 cache.  ``bench.py --design movivik`` prints the same
record as its one JSON line.
"""
from __future__ import annotations

import argparse
import json
import sys

import torch

from .hybrid_bench import PAGE_SIZE, VOCAB, _parts, _throughput
from .kernel_bench import peaks, timed
from .tedisun_bench import tedisun_config

CHUNK = 1024


def movivik_config(width: int) -> dict:
    """Eight layers, parallel mixer and attention in turn.  Parallel: full attention with heads of 128, four query heads
    per key/value head, half of a head rotated, beside half as many lightning heads with a 128 x 128 state; attention:
    the same heads within chunks of 1,024, rotated as a whole; feed-forwards of 4 x width."""
    heads = width // 128
    a = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    left = dict(a, rot={"base": 500000.0, "dims": 64})
    n = max(1, heads // 2)
    right = {"heads": n, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-3.0 - 7.0 * h / n) for h in range(n)]}
    local = dict(a, mask={"size": CHUNK},
                 rot={"base": 10000.0, "dims": 128, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    ff = {"kind": "dense", "ff": 4 * width}
    layers = []
    for _ in range(4):
        layers += [{"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": ff},
                   {"type": "attention", "mixer": local, "mlp": ff}]
    return {"architecture": "Movivik", "vocab": VOCAB, "width": width, "layers": layers, "norm": {"eps": 1e-6}, "max_position": 16384}


def closest_config(width: int) -> dict:
    """Tedisun at the same width and number of layers with one residual stream and one expert of the same size, which
    every token uses."""
    cfg = tedisun_config(width)
    cfg["streams"] = 1
    for layer in cfg["layers"]:
        layer["mlp"] = {"kind": "moe", "expert": {"ff": 4 * width}, "router": {"experts": 1, "identity": 0, "top": 1}}
    return cfg


def _kernels(width: int, cases, pk: dict) -> dict:
    """Each kernel of the design alone: microseconds, the bytes it has to move (inputs read once, outputs
    written once) or the operations it has to do, and the share of the measured copy bandwidth or bfloat16
    matrix throughput that is; ``like: ...`` are the kernels of the closest models on inputs of the same size.
    ``cases``: (tokens, requests, keys each request already holds)."""
    from types import SimpleNamespace

    from ..config.specs import DenseMLPSpec
    from ..csrc import ops
    from ..parts.base import make_feed_forward
    dev, bf = torch.device("cuda:0"), torch.bfloat16
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

        # norms around the sublayers
        x32 = torch.randn(tokens, width, device=dev)
        y, y2 = (torch.randn(tokens, width, device=dev, dtype=bf) for _ in range(2))
        w = torch.ones(width, device=dev, dtype=bf)
        oa = torch.empty_like(y)
        ends = dict(post=(w, 1e-6), following=(w, 1e-6), out=oa)
        add("sandwich_norm (one result)", lambda: ops.sandwich_norm(x32, y, **ends), tokens * width * 12)
        add("sandwich_norm (two normed results)", lambda: ops.sandwich_norm(x32, ((y, w, 0.5), (y2, w, 0.5), 1e-6), **ends), tokens * width * 14)
        add("like: add_rmsnorm_stream", lambda: ops.add_rmsnorm_stream(x32, y, w, 1e-6, out32=x32, out_act=oa), tokens * width * 12)
        del x32, y, y2, oa
        _attention_kernels(width, tokens, entries, held, step, kv_len, add)
        _lightning_kernels(width, tokens, entries, step, add)
        # the feed-forward: two products, the activation in the first one's epilogue
        h = torch.randn(tokens, width, device=dev, dtype=bf)
        for name, kind in (("feed-forward (tanh-form gelu)", "gelu_tanh"), ("like: feed-forward (silu)", "silu")):
            ff = make_feed_forward(DenseMLPSpec(hidden_size=width, intermediate_size=4 * width, activation=kind), bf)
            ff.bind({k: torch.randn(*p.shape, device=dev, dtype=bf) * 0.02 for k, p in ff.parameters().items()})
            add(name, lambda: ff.forward(h, None), nbytes=24 * width * width + tokens * width * 4, flops=24.0 * tokens * width * width)
            if kind == "gelu_tanh":
                w13, w2 = ff.w13[0], ff.w2[0]
                mid = torch.randn(tokens, 4 * width, device=dev, dtype=bf)
                add("like: the two products alone, cuBLAS", lambda: (torch.matmul(h, w13.t()), torch.matmul(mid, w2.t())),
                    nbytes=24 * width * width, flops=24.0 * tokens * width * width)
            del ff
        out[f"tokens{tokens}_requests{entries}_held{held}"] = rec
        ops.error_check(dev)
    return out


def _attention_kernels(width, tokens, entries, held, step, kv_len, add):
    from ..csrc import ops
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    per, hq = tokens // entries, width // 128
    hkv = max(1, hq // 4)
    pages = -(-(held + per) // PAGE_SIZE)
    table = torch.arange(entries * pages, device=dev, dtype=torch.int32).view(entries, pages)
    for d, dv in ((128, 128), (96, 64)):
        qn, kn, vn = hq * d, hkv * d, hkv * dv
        cache = (torch.randn(entries * pages, PAGE_SIZE * hkv * (d + dv), device=dev) * 0.5).to(bf)
        proj = torch.randn(tokens, qn + kn + vn + (hq + 7) // 8 * 8, device=dev, dtype=bf)
        q, o = torch.empty(tokens, qn, device=dev, dtype=bf), torch.empty(tokens, hq * dv, device=dev, dtype=bf)
        inv = (1e4 ** (-torch.arange(0, d, 2, dtype=torch.float32) / d)).to(dev)
        bias, one = torch.zeros(qn + kn + vn, device=dev), torch.ones(d, device=dev, dtype=bf)
        sizes = dict(num_heads=hq, num_kv_heads=hkv, head_dim=d, v_head_dim=dv, page_size=PAGE_SIZE)

        def prep(q_w=None, k_w=None, **kw):
            ops.qk_prep_general(proj, q_w, k_w, step.positions, step.token_seq, step.seq_rows, table, cache, q, eps=1e-6, **sizes, **kw)
        nbytes, tag = tokens * (qn + kn + vn) * 4, f"{d}/{dv}"
        add(f"qk_prep_general {tag} (biases, neighbours)", lambda: prep(bias=bias, inv_freq=inv, rotary_dim=d, pairing="interleaved", rope_scale=1.2), nbytes)
        if d == 128:
            add(f"qk_prep_general {tag} (split halves, norms without weights after)", lambda: prep(inv_freq=inv, rotary_dim=64, per_head_unit=True), nbytes)
            add(f"like: qk_prep_general {tag} (per-head norms with weights, no rotation)", lambda: prep(q_w=one, k_w=one, per_head=True), nbytes)
            add(f"like: qk_prep_general {tag} (biases, norms with weights, split halves)", lambda: prep(
                q_w=one, k_w=one, per_head=True, bias=bias, inv_freq=inv, rotary_dim=64), nbytes)
        gate = proj[:, qn + kn + vn:qn + kn + vn + hq]
        for name, kw in (("(chunk, gate per head)", dict(chunk=CHUNK, gate=gate)), ("(all keys, gate per head)", dict(gate=gate)),
                         ("like: (window)", dict(window=CHUNK)), ("like: (all keys)", {})):
            if d != 128 and name != "(chunk, gate per head)":
                continue
            chunk, window = kw.get("chunk"), kw.get("window")

            def span(p):
                return p % chunk + 1 if chunk else min(window or 1 << 30, p + 1)
            pre, name = ("like: ", name[6:]) if name.startswith("like: ") else ("", name)
            seen = sum(span(held + i) for i in range(per)) * entries
            if per > 1:
                fn = ops.attn_prefill_tc if d == 128 else ops.attn_prefill
                add(f"{pre}{fn.__name__} {tag} {name}", lambda: fn(q, cache, table, step.seq_rows, step.cu_q, kv_len, o, entries=entries,
                                                                  max_q_len=per, scale=0.09, **sizes, **kw), flops=2.0 * seen * hq * (d + dv))
            else:
                add(f"{pre}attn_decode {tag} {name}", lambda: ops.attn_decode(
                    q, cache, table, step.seq_rows, step.token_seq, step.positions, o, scale=0.09,
                    max_keys=min(held + 1, chunk or window or held + 1), **sizes, **kw), nbytes=seen * hkv * (d + dv) * 2)
        if d != 128 and per > 1:       # the same kernel at the sizes of its tiles
            cache2 = (torch.randn(entries * pages, PAGE_SIZE * hkv * 192, device=dev) * 0.5).to(bf)
            q2, o2 = torch.randn(tokens, hq * 128, device=dev, dtype=bf), torch.empty(tokens, hq * 64, device=dev, dtype=bf)
            add("like: attn_prefill 128/64 (window)", lambda: ops.attn_prefill(
                q2, cache2, table, step.seq_rows, step.cu_q, kv_len, o2, entries=entries, max_q_len=per, scale=0.09, num_heads=hq,
                num_kv_heads=hkv, head_dim=128, v_head_dim=64, page_size=PAGE_SIZE, window=CHUNK),
                flops=2.0 * sum(min(CHUNK, held + i + 1) for i in range(per)) * entries * hq * 192)


def _lightning_kernels(width, tokens, entries, step, add):
    from ..csrc import ops
    dev, bf = torch.device("cuda:0"), torch.bfloat16
    H, d = max(1, width // 256), 128
    n, per = H * d, tokens // entries
    proj = torch.randn(tokens, 4 * n, device=dev, dtype=bf) * 0.3
    q32, k32 = (torch.randn(tokens, n, device=dev) for _ in range(2))
    decay, state = torch.linspace(0.6, 0.9999, H, device=dev), torch.zeros(entries, H * d * d, device=dev)
    o, gated, w = torch.empty(tokens, n, device=dev), torch.empty(tokens, n, device=dev, dtype=bf), torch.ones(n, device=dev, dtype=bf)
    inv = (1e4 ** (-torch.arange(0, d, 2, dtype=torch.float32) / d)).to(dev)
    sizes = dict(heads=H, head_dim=d)
    nbytes = tokens * n * (4 + 8 + 2 + 4) + entries * n * d * 8
    if per > 1:
        add("retention_prep (silu)", lambda: ops.retention_prep(proj, 0, n, None, step.positions, q32, k32, rotary_dim=0, k_scale=1.0, silu=True, **sizes), tokens * n * 12)
        add("like: retention_prep (rotation)", lambda: ops.retention_prep(proj, 0, n, inv, step.positions, q32, k32, rotary_dim=d, k_scale=0.09, **sizes), tokens * n * 12)
        for name, silu in (("retention_chunk (silu)", True), ("like: retention_chunk", False)):
            add(name, lambda: ops.retention_chunk(q32, k32, proj, 2 * n, decay, state, step, o, v_head_dim=d, silu=silu, **sizes), nbytes, iters=5)
    else:
        add("retention_scan (silu, straight from the projection)", lambda: ops.retention_scan(
            None, None, proj, 2 * n, decay, state, step, o, v_head_dim=d, silu=True, qk=(0, n, 1.0), **sizes), nbytes, iters=5)
        add("like: retention_scan", lambda: ops.retention_scan(q32, k32, proj, 2 * n, decay, state, step, o, v_head_dim=d, **sizes), nbytes, iters=5)
    o.normal_()
    add("retention_out_joint", lambda: ops.retention_out_joint(o, proj, 3 * n, w, gated, eps=1e-6), tokens * n * 8)
    add("like: retention_out", lambda: ops.retention_out(o, proj, 3 * n, gated, heads=H, v_head_dim=d, eps=1e-6), tokens * n * 8)


def run(sizes=(2048, 4096), steps: int = 20, warmup: int = 3, kernels: bool = True, parts: bool = True) -> dict:
    torch.cuda.set_device(0)
    pk = peaks()
    points = [("prefill", 1, 2048), ("prefill", 1, 8192), ("prefill", 4, 2048), ("decode", 8, 2048), ("decode", 64, 2048)]
    rec = {"design": "Movivik", "closest": "Tedisun (one stream, one expert)", "dtype": "bf16", "data": "synthetic", "peaks": pk, "sizes": {}}
    for width in sizes:
        mine, other = movivik_config(width), closest_config(width)
        one = {"layers": 8, "movivik": _throughput(mine, points, steps, warmup), "closest": _throughput(other, points, steps, warmup)}
        if parts:
            one["movivik_parts_ms"] = _parts(mine, 2048, 8)
            one["closest_parts_ms"] = _parts(other, 2048, 8)
        if kernels:
            one["kernels"] = _kernels(width, [(2048, 1, 0), (8192, 4, 0), (64, 64, 3000)], pk)
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
