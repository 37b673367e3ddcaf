"""Attention over a cached latent (kernels: csrc/latent_attention.cu).

Per token the mixer projects to ``[query latent | key/value latent | shared rotated key part]`` in
one product; the preparation kernel RMS-norms the two latents (32-bit), rotates the shared key
part and writes ``[c | k_rot]`` into the token's page slot: that row is all the cache holds.
Queries ``q = W_uq c_q`` (or, without a query latent, ``q = W_q x``: the one product is then ``[queries |
key/value latent | shared rotated key part | output gate]`` and the kernels read its columns) are laid out head by head as ``[head_dim unrotated | rot_dim rotated]``.

Keys and values are never formed.  With ``k_plain = W_uk c`` and ``v = W_uv c``,

    q_plain . k_plain = (W_uk^T q_plain) . c          and        sum_j p_j v_j = W_uv (sum_j p_j c_j),

so the unrotated queries are taken into the latent's space (one batched product over the heads),
attention runs over the cached rows as if there were one key/value head of ``kv_rank + rot_dim``
dims whose first ``kv_rank`` dims are also the values, and the values' up-projection follows (one
more batched product).  Scores, weights and sums are 32-bit; the products are in the activation
type with 32-bit accumulation.
"""
from __future__ import annotations

import torch

from ..config.specs import ParamSpec
from ..csrc import ops
from .base import KVRequest, Mixer, make_position, register_mixer
from .linear import linear
from .position import RotaryArgs, as_rotary_args


class LatentAttention(Mixer):
    graph_safe = True
    max_step_entries = ops.LIMITS["grid_dim_yz"]

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        s = spec
        if min(s.hidden_size, s.num_heads, s.head_dim, s.v_head_dim, s.kv_rank) <= 0 or s.rot_dim < 0 or s.q_rank < 0:
            raise ValueError("the sizes of a latent attention must be positive (rot_dim and q_rank may be 0)")
        if s.output_gate and s.q_rank:
            raise ValueError("an output gate goes with queries straight from the input (q_rank 0)")
        if s.kv_rank + s.rot_dim > ops.LIMITS["latent_max_row"]:
            raise ValueError(f"a cached row of {s.kv_rank} + {s.rot_dim} elements is not supported (at most "
                             f"{ops.LIMITS['latent_max_row']}: a warp keeps a row in registers)")
        if s.num_heads > ops.LIMITS["grid_dim_yz"]:
            raise ValueError(f"{s.num_heads} heads are not supported (heads are a grid dimension of the kernels)")
        if s.window is not None and s.window <= 0:
            raise ValueError("window must be positive (None: all keys)")
        self.position = make_position(s.position, dtype) if s.position is not None and s.rot_dim > 0 else None
        if self.position is not None:
            if s.position.pairing not in ("split_half", "interleaved"):
                raise ValueError("the latent attention kernels rotate split halves or interleaved pairs")
            if s.position.rotary_dim > s.rot_dim:
                raise ValueError(f"the position encoding rotates {s.position.rotary_dim} dims, the rotated part has {s.rot_dim}")
        self.sink = None
        # without a query latent: the columns of the one projection
        self.q_cols = 0 if s.q_rank else s.num_heads * (s.head_dim + s.rot_dim)
        self.g_off = self.q_cols + s.kv_rank + s.rot_dim
        self.g_cols = s.num_heads * s.v_head_dim if s.output_gate else 0

    def parameters(self):
        s = self.spec
        if s.q_rank:
            out = {"down": ParamSpec((s.q_rank + s.kv_rank + s.rot_dim, s.hidden_size)),
                   "q_norm": ParamSpec((s.q_rank,), "act", "norm"),
                   "uq": ParamSpec((s.num_heads * (s.head_dim + s.rot_dim), s.q_rank))}
        else:       # queries, then what `down` holds, then the gate
            out = {"in_proj": ParamSpec((self.g_off + self.g_cols, s.hidden_size))}
        out |= {"kv_norm": ParamSpec((s.kv_rank,), "act", "norm"),
               "uk": ParamSpec((s.num_heads * s.head_dim, s.kv_rank)),
               "uv": ParamSpec((s.num_heads * s.v_head_dim, s.kv_rank)),
               "o": ParamSpec((s.hidden_size, s.num_heads * s.v_head_dim))}
        if s.sink:
            out["sink"] = ParamSpec((s.num_heads,), "float32", "bias")
        return out

    def kv_request(self):
        s = self.spec
        return KVRequest(1, s.kv_rank + s.rot_dim, s.window, None, "latent")

    def forward(self, x, step, slot):
        s = self.spec
        tokens, dev = x.shape[0], x.device
        H, d, r, rank = s.num_heads, s.head_dim, s.rot_dim, s.kv_rank
        if self.position is not None:
            rope = as_rotary_args(self.position.kernel_args(dev))
            if rope.scale != 1.0:
                raise ValueError("the latent attention kernels take no factor on cos and sin")
        else:
            rope = RotaryArgs(None, 0)
        proj = linear(x, self.down if s.q_rank else self.in_proj)
        tiled = self.takes_tiles(x.dtype)
        qfull = torch.empty(tokens, H, rank + r, dtype=x.dtype, device=dev) if tiled else None
        cq = torch.empty(tokens, s.q_rank, dtype=x.dtype, device=dev) if s.q_rank else None
        q = proj[:, :self.q_cols]                                            # [tokens, H * (d + r)]
        ops.latent_prep(proj[:, self.q_cols:self.g_off + s.q_rank], self.q_norm if s.q_rank else None, self.kv_norm,
                        rope.inv_freq, step.positions, step.token_seq, step.seq_rows, slot.table, slot.kv, cq,
                        q_rank=s.q_rank, rank=rank, rot=r, rotary_dim=rope.rotary_dim, eps=s.norm_eps,
                        page_size=slot.page_size, write_cache=slot.write_cache, pairing=rope.pairing,
                        queries=(q, H, d, qfull) if tiled and not s.q_rank else None)
        if s.q_rank:
            q = linear(cq, self.uq)
            if tiled:
                ops.latent_q_rotate(q, rope.inv_freq, step.positions, qfull, heads=H, head_dim=d, rank=rank, rot=r,
                                    rotary_dim=rope.rotary_dim, pairing=rope.pairing)
        # the unrotated queries in the latent's space: [H, tokens, d] x [H, d, rank], in the tiled kernel's query rows
        # or 32-bit
        q_plain, uk = q.unflatten(1, (H, d + r))[:, :, :d].transpose(0, 1), self.uk.view(H, d, rank)
        out_lat = torch.empty(tokens, H, rank, dtype=x.dtype, device=dev)
        if tiled:
            torch.bmm(q_plain, uk, out=qfull[:, :, :rank].transpose(0, 1))
            self.attend_tiled(qfull, out_lat, step, slot)
        else:
            q_lat = torch.bmm(q_plain, uk) if x.dtype == torch.float32 else torch.bmm(q_plain, uk, out_dtype=torch.float32)
            ops.latent_attention_plain(q_lat, q, rope.inv_freq, slot.kv, slot.table, step.seq_rows, step.token_seq,
                                       step.positions, self.sink, out_lat, heads=H, head_dim=d, rank=rank, rot=r,
                                       rotary_dim=rope.rotary_dim, page_size=slot.page_size, scale=s.scale, window=s.window,
                                       pairing=rope.pairing)
        # the values' up-projection per head, read from and written to token-major rows through strided views
        heads_out = torch.empty(tokens, H, s.v_head_dim, dtype=x.dtype, device=dev)
        torch.bmm(out_lat.transpose(0, 1), self.uv.view(H, s.v_head_dim, rank).transpose(1, 2), out=heads_out.transpose(0, 1))
        heads_out = heads_out.view(tokens, H * s.v_head_dim)
        if s.output_gate:
            ops.sigmoid_gate_(heads_out, proj[:, self.g_off:])
        return linear(heads_out, self.o)

    use_tensor_cores = None      # False: always the kernel with one block per (token, head)

    def takes_tiles(self, dtype) -> bool:
        """bfloat16 steps of sizes the tiled kernel takes (latent and rotated part in multiples of 16, a
        cached row of at most 256) run on tensor-core tiles whose rows are (token, head) pairs, prompt
        portions and single tokens alike; everything else one block per (token, head)."""
        s = self.spec
        return (self.use_tensor_cores is not False and dtype == torch.bfloat16 and s.scale > 0
                and ops.latent_attention_tiled_supported(s.kv_rank, s.rot_dim))

    def attend_tiled(self, qfull, out_lat, step, slot):
        s = self.spec
        most = step.max_kv_len if s.window is None else min(step.max_kv_len, s.window + step.max_q_len - 1)
        ops.latent_attention_tiled(qfull, slot.kv, slot.table, step.seq_rows, step.cu_q, step.kv_len, self.sink, out_lat,
                                   entries=step.num_seqs, max_q_len=step.max_q_len, heads=s.num_heads, rank=s.kv_rank,
                                   rot=s.rot_dim, page_size=slot.page_size, scale=s.scale, window=s.window, max_keys=most)


register_mixer("latent_attention", LatentAttention)
