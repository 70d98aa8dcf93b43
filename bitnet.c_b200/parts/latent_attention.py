"""Softmax attention through low-rank latents, with the latent itself as the cached key and value."""
from __future__ import annotations

from typing import Dict, Optional

import numpy as np
import torch

from ..csrc import ops
from .base import KvRequest, Mixer, ParamSpec
from .registry import build_part, register_mixer


@register_mixer("latent_attention")
class LatentAttention(Mixer):
    """c_q = norm(W_dq h), q = W_uq c_q (or, without a query latent, q = W_q h), per head [plain | rotated];
    W_dkv h = [latent | rotated key part], the
    latent normed; per head k = [W_uk c | rotated part], v = W_uv c; softmax over the window, optionally with a
    learned score per head in its denominator that has no key and no value (``sink``); the head's output
    times the logistic function of its gate (one number per head, or one per output number); output projection.

    Only the normed latent c and the rotated key part are cached, as one key row [c | k_rot] of one key/value
    head, and attention runs on those rows directly: since (W_uk c) . q = c . (W_uk^T q), every head's plain
    query part is carried into the latent space first (one small product per head), the scores are
    q' . [c | k_rot] with q' = [W_uk^T q_plain | q_rot], the weighted sum of the rows' first kv_rank numbers is
    the head's output in the latent space, and W_uv brings it back (another small product per head).  The
    values are a part of the key rows, so the cache holds no value plane.

    Runs of new tokens take the other order where the tcgen05 kernel has room for a head's keys (192 numbers) and values (128),
    or the key rows are too wide for the mma.sync one (more than 256 numbers): the rows every new token sees are read back
    from the cache, W_uk and W_uv make per-head keys [W_uk c | k_rot] and values of them (two products over all those
    rows), which go into scratch pages of the step, and the attention runs on these with the queries as projected.

    A run without a latent of its own (``own_kv`` False) reads the rows of the run its schedule entry names, with its own
    queries, W_uk and W_uv."""

    kernels = ("linear", "linear_mma", "linear_tc", "gemm_tc", "attention", "attention_prefill", "attention_prefill_tc", "rotary_pairs", "norm", "latent")
    TILED_MIN_TOKENS = 16  # runs of new tokens from this many on take the tensor-core kernel (bfloat16)
    SEEN_PER_NEW = 64  # keys and values are made per head while a step's tokens see at most so many rows each, on average
    graph_safe = True

    def __init__(self, spec, build):
        super().__init__(spec, build)
        if min(spec.n_heads, spec.head_dim, spec.rot_dim, spec.v_head_dim, spec.kv_rank) <= 0 or spec.q_rank < 0:
            raise ValueError("latent_attention: heads, head sizes and the key/value rank must be positive")
        self.element_gate = bool(getattr(spec, "element_gate", False))
        self.has_sink = bool(getattr(spec, "sink", False))
        if self.element_gate and spec.head_gate:
            raise ValueError("latent_attention: a gate per head or a gate per output number, not both")
        if spec.kv_rank + spec.rot_dim > 2048:
            raise ValueError(f"latent_attention: kv_rank + rot_dim = {spec.kv_rank + spec.rot_dim} must be at most 2048")
        s = spec
        # which forms of attention over runs of tokens its sizes allow
        self.per_head = (build.dtype == torch.bfloat16 and (s.head_dim + s.rot_dim) % 16 == 0 and s.v_head_dim % 16 == 0
                         and max(s.head_dim + s.rot_dim, s.v_head_dim) <= 256 and not (s.head_dim % 8 or s.rot_dim % 8 or s.kv_rank % 8))
        self.on_tcgen05 = self.per_head and ops.USE_TCGEN05_ATTENTION and s.head_dim + s.rot_dim <= 192 and s.v_head_dim <= 128 and s.scale > 0
        self.position = build_part("position", spec.position, build)
        self.w_dq: Optional[torch.Tensor] = None

    def children(self):
        return {"position": self.position}

    @property
    def key_row(self) -> int:
        return self.spec.kv_rank + self.spec.rot_dim

    def params(self) -> Dict[str, ParamSpec]:
        s = self.spec
        p = {"uk": ParamSpec((s.n_heads * s.head_dim, s.kv_rank)), "uv": ParamSpec((s.n_heads * s.v_head_dim, s.kv_rank)), "o": ParamSpec((s.width, s.n_heads * s.v_head_dim))}
        if s.own_kv:
            p.update({"dkv": ParamSpec((self.key_row, s.width)), "dkv.norm": ParamSpec((s.kv_rank,), init="ones")})
        if s.q_rank:
            p.update({"dq": ParamSpec((s.q_rank, s.width)), "dq.norm": ParamSpec((s.q_rank,), init="ones"),
                      "uq": ParamSpec((s.n_heads * (s.head_dim + s.rot_dim), s.q_rank))})
        else:
            p["q"] = ParamSpec((s.n_heads * (s.head_dim + s.rot_dim), s.width))
        if s.head_gate or self.element_gate:
            p["g"] = ParamSpec((self.gate_len, s.width))
        if self.has_sink:
            p["sink"] = ParamSpec((s.n_heads,))
        return p

    @property
    def gate_len(self) -> int:
        s = self.spec
        return s.n_heads * s.v_head_dim if self.element_gate else (s.n_heads if s.head_gate else 0)

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        if s.q_rank:
            self.w_dq, self.g_dq, self.w_uq = tensors["dq"], tensors["dq.norm"], tensors["uq"]
        self.g_dkv, self.w_o = tensors.get("dkv.norm"), tensors["o"]
        self.sink = tensors["sink"].float().contiguous() if self.has_sink else None
        # the latent, the rotated key part, the gates and (without a query latent) the queries are one product of
        # the mixer's input
        parts = ([tensors["dkv"]] if s.own_kv else []) + ([tensors["g"]] if self.gate_len else [])
        self.g_off = self.key_row if s.own_kv else 0
        at = self.g_off + self.gate_len
        if not s.q_rank:
            gap = -at % 8  # the queries start at a 16-byte boundary of the row
            if gap:
                parts.append(torch.zeros((gap, s.width), dtype=tensors["q"].dtype, device=tensors["q"].device))
            self.q_off = at + gap
            parts.append(tensors["q"])
            at = self.q_off + s.n_heads * (s.head_dim + s.rot_dim)
        self.w_kv, self.row = None, 0  # (nothing at all where a run has a query latent, no gates and no latent of its own)
        if parts:
            dt = parts[0].dtype if all(t.dtype == parts[0].dtype for t in parts) else torch.float32
            pad = -at % 8  # rows of the product's result stay 16-byte aligned
            if pad:
                parts.append(torch.zeros((pad, s.width), dtype=dt, device=parts[0].device))
            self.w_kv = torch.cat([t.to(dt) for t in parts], dim=0).contiguous()
            self.row = at + pad
        # per head: W_uk as [dim, kv_rank] (plain query part -> latent space), W_uv as [vdim, kv_rank]
        self.w_uk = tensors["uk"].reshape(s.n_heads, s.head_dim, s.kv_rank).contiguous()
        self.w_uv = tensors["uv"].reshape(s.n_heads, s.v_head_dim, s.kv_rank).contiguous()
        self.w_uk_flat, self.w_uv_flat = tensors["uk"], tensors["uv"]

    def cache_request(self) -> KvRequest:
        s = self.spec
        return KvRequest(n_kv_heads=1, head_dim=self.key_row, window=s.window, v_head_dim=s.kv_rank, values_in_keys=True)

    def forward(self, h, ctx, kv, state):
        s = self.spec
        n = h.shape[0]
        H, d, dr, rank, row = s.n_heads, s.head_dim, s.rot_dim, s.kv_rank, self.key_row
        dt = self.build.dtype
        if kv.owner != s.own_kv:
            raise ValueError("a latent mixer with a latent of its own owns its cache plane, one without reads another's")
        ckv = ops.linear(h, self.w_kv, out_dtype=dt) if self.w_kv is not None else None  # [n, latent | rotated key part | gates | (queries) | padding]
        if s.q_rank:
            cq = ops.linear(h, self.w_dq, out_dtype=dt)
            ops.rmsnorm_slices(cq, s.norm_eps, 0, s.q_rank, self.g_dq)
            q, q_off = ops.linear(cq, self.w_uq, out_dtype=dt), 0  # [n, H * (d + dr)]
        else:
            q, q_off = ckv, self.q_off
        # the latent normed, the heads' rotated query parts and the shared key part rotated, the key row [c | k_rot]
        # to the cache: one launch
        places = dict(q_off=q_off, n_q_heads=H, q_head_stride=d + dr, q_rot_off=d)
        if s.own_kv:
            self.position.apply(ckv, ctx, xq=q, k_off=0, n_k_heads=1, k_head_stride=row, k_rot_off=rank, k_row=row, tok_seq=ctx.tok_seq,
                                slots=ctx.slots, page_table=kv.page_table, k_cache=kv.k, norm_len=rank, norm_w=self.g_dkv,
                                norm_eps=s.norm_eps, **places)
        else:
            self.position.apply(q, ctx, **places)
        gate = ckv[:, self.g_off:] if s.head_gate else None
        egate = ckv[:, self.g_off: self.g_off + self.gate_len] if self.element_gate else None
        tiled = dt == torch.bfloat16 and not ctx.decode and ctx.tile_seq is not None and ctx.max_new >= self.TILED_MIN_TOKENS
        if q_off:
            q = q[:, q_off: q_off + H * (d + dr)]
        in_latent_space = row <= 256 and row % 16 == 0 and rank % 16 == 0  # the tensor-core kernel takes the cached rows as they are
        if (tiled and self.per_head and ctx.host_new and q.stride(0) % 8 == 0
                and (not in_latent_space or self.on_tcgen05 and sum(ctx.host_pos0) <= (self.SEEN_PER_NEW - 1) * ctx.n_tokens)):
            return self._per_head_keys(q, gate, ctx, kv, egate)
        # queries in the latent space: [W_uk^T q_plain | q_rot] per head
        q3 = q.unflatten(1, (H, d + dr))
        ql = torch.empty((n, H, row), dtype=q.dtype, device=q.device)
        torch.bmm(q3[:, :, :d].transpose(0, 1), self.w_uk.to(q.dtype), out=ql[:, :, :rank].transpose(0, 1))
        ql[:, :, rank:] = q3[:, :, d:]
        if ctx.diag is not None:
            ctx.tap("attn_q", lambda: ql.view(n, H * row))
        out = torch.empty((n, H * rank), dtype=dt, device=h.device)
        if tiled and in_latent_space:
            # runs of new tokens: 64 tokens of a sequence and a head per block on the tensor cores, the
            # softmax weights with 16 bits of mantissa
            ops.attention_prefill(ql, H * row, out, H, 1, row, s.scale, s.window, ctx.tile_seq, ctx.tile_row0, ctx.seq_start,
                                  ctx.seq_pos0, ctx.slots, kv.page_table, kv.k, None, gate=gate, gate_stride=self.row,
                                  precise=True, v_dim=rank, sink=self.sink)
        else:
            ops.attention_general(ql, H * row, out, n, H, 1, row, s.scale, s.window, ctx.tok_seq, ctx.tok_pos, ctx.slots,
                                  kv.page_table, kv.k, None, gate=gate, gate_stride=self.row, v_dim=rank,
                                  max_keys=min(ctx.max_len, s.window) if s.window > 0 else ctx.max_len, sink=self.sink)
        ctx.tap("attn_out", out)
        # back from the latent space: W_uv per head, heads side by side
        o = torch.empty((n, H, s.v_head_dim), dtype=dt, device=h.device)
        torch.bmm(out.view(n, H, rank).transpose(0, 1), self.w_uv.to(dt).transpose(1, 2), out=o.transpose(0, 1))
        o = o.view(n, H * s.v_head_dim)
        if egate is not None:
            ops.gate_rows(o, egate)
        return ops.linear(o, self.w_o, out_dtype=torch.float32)

    def _seen_rows(self, ctx, device):
        """For this step: which cached positions its new tokens see (sequence and position of each, on the device),
        and a page table of scratch pages that holds just those, by sequence of the step and page index within the
        sequence.  The same for every layer of one window, so it is made once per step."""
        key = ("latent_attention.seen", self.spec.window)
        if key not in ctx.memo:
            w = self.spec.window
            seq, pos, spans = [], [], []
            for i, (p0, n) in enumerate(zip(ctx.host_pos0, ctx.host_new)):
                lo = max(0, p0 - w + 1) if w > 0 else 0
                seq.append(np.full(p0 + n - lo, i, dtype=np.int32))
                pos.append(np.arange(lo, p0 + n, dtype=np.int32))
                spans.append((lo // ops.PAGE, (p0 + n - 1) // ops.PAGE))
            table = np.zeros((len(spans), max(b for _a, b in spans) + 1), dtype=np.int32)
            at = 0
            for i, (a, b) in enumerate(spans):
                table[i, a:b + 1] = np.arange(at, at + b - a + 1)
                at += b - a + 1
            both = torch.from_numpy(np.stack([np.concatenate(seq), np.concatenate(pos)])).pin_memory().to(device, non_blocking=True)
            ctx.memo[key] = (both[0], both[1], torch.from_numpy(table).pin_memory().to(device, non_blocking=True), at,
                             torch.arange(len(spans), dtype=torch.int32, device=device))
        return ctx.memo[key]

    def _per_head_keys(self, q, gate, ctx, kv, egate=None):
        s = self.spec
        H, d, dr, dv, rank = s.n_heads, s.head_dim, s.rot_dim, s.v_head_dim, s.kv_rank
        dt, dev = self.build.dtype, q.device
        seq, pos, table, n_pages, rows_of = self._seen_rows(ctx, dev)
        c = ops.latent_gather(kv.k, rank, seq, pos, ctx.slots, kv.page_table)
        keys, values = ops.linear(c, self.w_uk_flat, out_dtype=dt), ops.linear(c, self.w_uv_flat, out_dtype=dt)
        on_tcgen05 = self.on_tcgen05 and ctx.wide_tile_seq is not None and q.dim() == 2
        # rows of a page that no position fills are masked, but zero times what lies there must be zero: scratch pages start as
        # zeros where the kernel does not see to it (it does for what lies behind a sequence's last position on tcgen05)
        new = torch.empty if on_tcgen05 and s.window <= 0 else torch.zeros
        k_s = new((n_pages, H, ops.PAGE, d + dr), dtype=dt, device=dev)
        v_s = new((n_pages, H, ops.PAGE, dv), dtype=dt, device=dev)
        ops.latent_pages(keys, values, kv.k, rank, H, seq, pos, ctx.slots, kv.page_table, table, k_s, v_s)
        out = torch.empty((q.shape[0], H * dv), dtype=dt, device=dev)
        if on_tcgen05:
            ops.attention_prefill_tc(q, q.stride(0), out, H, H, d + dr, s.scale, s.window, ctx.wide_tile_seq, ctx.wide_tile_row0,
                                     ctx.seq_start, ctx.seq_pos0, rows_of, table, k_s, v_s, precise=True, sink=self.sink, gate=gate,
                                     gate_stride=self.row)
        else:
            ops.attention_prefill(q, q.stride(0), out, H, H, d + dr, s.scale, s.window, ctx.tile_seq, ctx.tile_row0, ctx.seq_start,
                                  ctx.seq_pos0, rows_of, table, k_s, v_s, gate=gate, gate_stride=self.row, precise=True, sink=self.sink)
        ctx.tap("attn_out", out)
        if egate is not None:
            ops.gate_rows(out, egate)
        return ops.linear(out, self.w_o, out_dtype=torch.float32)
