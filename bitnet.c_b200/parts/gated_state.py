"""Recurrent mixers with a matrix state per head under one decay per head and token: the gated delta rule with
head-wise decays, the Mamba-2 state-space layer, and linear attention under fixed decays."""
from __future__ import annotations

import math
from typing import Dict, Optional, Sequence, Tuple

import torch

from ..csrc import ops
from .base import Mixer, ParamSpec, StateRequest
from .registry import register_mixer


class GatedStateMixer(Mixer):
    """What the mixers share: one stacked product of the mixer's input whose last rows are the heads' gate
    pre-activations, the recurrence from the sequence's state (matrices, and the convolutions' last inputs, float32),
    a gated norm and the output projection.  Steps of one token per sequence take the whole product in float32 and
    the recurrence in one launch; runs of tokens in bfloat16 take the gates' rows as a float32 product of their own
    beside the others' bfloat16 rows."""

    kernels = ("linear", "linear_mma", "linear_tc", "gemm_tc", "gated_state")
    graph_safe = True
    CHUNKED_MIN_TOKENS = 16  # steps with a run of so many new tokens take the recurrence chunk by chunk
    n_heads = n_groups = dim = vdim = taps = 0  # set by the mixers
    log_decay = None  # fixed log decays per head, in place of gates

    def _check_sizes(self) -> None:
        if min(self.n_heads, self.n_groups, self.dim, self.vdim) <= 0 or self.n_heads % self.n_groups:
            raise ValueError(f"{self.spec.kind}: {self.n_heads} heads are not a multiple of {self.n_groups} groups, or a size is not positive")
        if self.dim > ops.GATED_STATE_MAX_DIM or not 1 <= self.taps <= ops.GATED_STATE_MAX_TAPS:
            raise ValueError(f"{self.spec.kind}: a state of {self.dim} rows (at most {ops.GATED_STATE_MAX_DIM}) or {self.taps} taps "
                             f"(1 to {ops.GATED_STATE_MAX_TAPS}) is not supported")

    def _stack(self, parts: Sequence[torch.Tensor], n_gates: int) -> None:
        """The input product's matrix; its last ``n_gates`` rows are the gates'."""
        dt = parts[0].dtype if all(t.dtype == parts[0].dtype for t in parts) else torch.float32
        rows = sum(t.shape[0] for t in parts)
        self.main, self.n_gates = rows - n_gates, n_gates
        pad = -rows % 8  # rows of the product's result stay 16-byte aligned
        if pad:
            parts = list(parts) + [torch.zeros((pad, parts[0].shape[1]), dtype=dt, device=parts[0].device)]
        self.w_in = torch.cat([t.to(dt) for t in parts], dim=0).contiguous()

    def state_request(self) -> StateRequest:
        return StateRequest((ops.gated_state_floats(self.n_heads, self.n_groups, self.dim, self.vdim, self.taps),), torch.float32)

    def _project(self, h, ctx) -> Tuple[torch.Tensor, torch.Tensor]:
        """(rows of the projection, the gates' float32 pre-activations)."""
        if ctx.decode or self.build.dtype == torch.float32 or self.w_in.dtype == torch.float32:
            proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
            return proj, proj[:, self.main:]
        return (ops.linear(h, self.w_in[: self.main], out_dtype=self.build.dtype),
                ops.linear(h, self.w_in[self.main:], out_dtype=torch.float32))

    def _recur(self, proj, gates, ctx, state):
        chunked = not ctx.decode and ctx.max_new >= self.CHUNKED_MIN_TOKENS and ctx.tile_seq is not None
        tiles = dict(tile_seq=ctx.tile_seq, tile_row0=ctx.tile_row0) if chunked else {}
        o = ops.gated_state(proj, self.q_off, self.k_off, self.v_off, gates, self.a_off, self.b_off, self.conv_w, self.conv_b,
                            self.dt_bias, self.a_log, self.skip, state, ctx.tok_seq, ctx.seq_start, ctx.seq_pos0, ctx.slots,
                            ctx.n_seqs, self.n_heads, self.n_groups, self.dim, self.vdim, one_token=ctx.decode,
                            log_decay=self.log_decay, **tiles)
        ctx.tap("state_raw", o)
        return o


@register_mixer("head_delta")
class HeadDelta(GatedStateMixer):
    """q, k (kv_heads x dim) and v (heads x vdim) = W h, each through a short convolution along the sequence and SiLU;
    every q and k head scaled to length one (q also by dim^-1/2).  From W_b h and W_a h every head gets a rate
    b = sigmoid(.) and a log decay l = -exp(A_log) softplus(. + dt_bias), and from the sequence's state S (zero at first)

        S' = e^l S;  u = b (v - S'^T k);  S = S' + k u^T;  o = S^T q

    Then an RMS norm per head with one gain for all heads, a gate silu(W_g h), and the output projection.  Consecutive
    heads / kv_heads heads share a q/k head."""

    def __init__(self, spec, build):
        super().__init__(spec, build)
        self.n_heads, self.n_groups, self.dim, self.vdim, self.taps = (spec.n_heads, spec.n_kv_heads, spec.head_dim,
                                                                       spec.v_head_dim, spec.conv_taps)
        self._check_sizes()
        self.w_in: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        s = self.spec
        qk, vv, H = s.n_kv_heads * s.head_dim, s.n_heads * s.v_head_dim, s.n_heads
        return {"q": ParamSpec((qk, s.width)), "q.conv": ParamSpec((qk, s.conv_taps)),
                "k": ParamSpec((qk, s.width)), "k.conv": ParamSpec((qk, s.conv_taps)),
                "v": ParamSpec((vv, s.width)), "v.conv": ParamSpec((vv, s.conv_taps)),
                "b": ParamSpec((H, s.width)), "A_log": ParamSpec((H,)), "a": ParamSpec((H, s.width)), "dt_bias": ParamSpec((H,)),
                "g": ParamSpec((vv, s.width)), "norm": ParamSpec((s.v_head_dim,), init="ones"), "o": ParamSpec((s.width, vv))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        qk, vv = s.n_kv_heads * s.head_dim, s.n_heads * s.v_head_dim
        self._stack([tensors[n] for n in ("q", "k", "v", "g", "a", "b")], 2 * s.n_heads)
        self.q_off, self.k_off, self.v_off, self.g_off = 0, qk, 2 * qk, 2 * qk + vv
        self.a_off, self.b_off = 0, s.n_heads
        self.conv_w = torch.cat([tensors[n].float() for n in ("q.conv", "k.conv", "v.conv")]).t().contiguous()
        self.conv_b = self.skip = None
        self.dt_bias, self.a_log, self.gain = (tensors[n].float().contiguous() for n in ("dt_bias", "A_log", "norm"))
        self.w_o = tensors["o"]

    def forward(self, h, ctx, kv, state):
        s = self.spec
        proj, gates = self._project(h, ctx)
        o = self._recur(proj, gates, ctx, state)
        y = ops.state_output(o, proj[:, self.g_off: self.g_off + o.shape[1]], self.gain, s.n_heads, s.norm_eps, False, self.build.dtype)
        return ops.linear(y, self.w_o, out_dtype=torch.float32)


@register_mixer("mamba2")
class Mamba2(GatedStateMixer):
    """[z | x | B | C | dt] = W_in h; x, B and C through a short convolution along the sequence (with a bias) and SiLU; the
    step size of a head d = softplus(dt + dt_bias); from the sequence's state S (zero at first)

        S = e^(-exp(A_log) d) S_before + d B x^T;  y = S^T C + D x

    with B and C shared by the heads of a group.  Then the gate, y silu(z), an RMS norm of the row cut into
    ``norm_groups`` parts, a gain, and the output projection."""

    def __init__(self, spec, build):
        super().__init__(spec, build)
        self.n_heads, self.n_groups, self.dim, self.vdim, self.taps = (spec.n_heads, spec.n_groups, spec.state, spec.v_head_dim,
                                                                       spec.conv_taps)
        self._check_sizes()
        self.inner = self.n_heads * self.vdim
        if spec.norm_groups <= 0 or self.inner % spec.norm_groups:
            raise ValueError(f"mamba2: {self.inner} numbers cannot be normed in {spec.norm_groups} equal parts")
        self.w_in: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        s = self.spec
        channels, H = self.inner + 2 * s.n_groups * s.state, s.n_heads
        return {"in": ParamSpec((self.inner + channels + H, s.width)), "conv": ParamSpec((channels, s.conv_taps)),
                "conv.b": ParamSpec((channels,)), "dt_bias": ParamSpec((H,)), "A_log": ParamSpec((H,)), "D": ParamSpec((H,)),
                "norm": ParamSpec((self.inner,), init="ones"), "o": ParamSpec((s.width, self.inner))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        bc = s.n_groups * s.state
        self._stack([tensors["in"]], s.n_heads)
        self.v_off, self.k_off, self.q_off = self.inner, 2 * self.inner, 2 * self.inner + bc  # x, B, C
        self.a_off, self.b_off = 0, -1
        # the file's channels are [x | B | C]; the recurrence's are [C | B | x]
        order = lambda t: torch.cat([t[self.inner + bc:], t[self.inner: self.inner + bc], t[: self.inner]]).float()
        self.conv_w = order(tensors["conv"]).t().contiguous()
        self.conv_b = order(tensors["conv.b"]).contiguous()
        self.dt_bias, self.a_log, self.skip, self.gain = (tensors[n].float().contiguous() for n in ("dt_bias", "A_log", "D", "norm"))
        self.w_o = tensors["o"]

    def forward(self, h, ctx, kv, state):
        s = self.spec
        proj, gates = self._project(h, ctx)
        o = self._recur(proj, gates, ctx, state)
        y = ops.state_output(o, proj[:, : self.inner], self.gain, s.norm_groups, s.norm_eps, True, self.build.dtype)
        return ops.linear(y, self.w_o, out_dtype=torch.float32)


@register_mixer("lightning")
class Lightning(GatedStateMixer):
    """q, k (heads x dim) and v (heads x vdim) = SiLU(W h); per head, from the sequence's state S (zero at first), under one
    fixed decay per head

        S = decay S_before + k v^T;  o = S^T q

    Then one RMS norm over all heads with a gain, the logistic function of W_g h, and the output projection."""

    NO_DECAY_LEFT = -100.0  # log decay of a head that forgets everything: e^-100 is zero in single precision

    def __init__(self, spec, build):
        super().__init__(spec, build)
        self.n_heads = self.n_groups = spec.n_heads
        self.dim, self.vdim, self.taps = spec.head_dim, spec.v_head_dim, 1
        self._check_sizes()
        if len(spec.decay) != spec.n_heads or not all(0.0 <= d <= 1.0 for d in spec.decay):
            raise ValueError(f"lightning: one decay from 0 to 1 for each of {spec.n_heads} heads, not {spec.decay!r}")
        self.w_in: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        s = self.spec
        qk, vv = s.n_heads * s.head_dim, s.n_heads * s.v_head_dim
        return {"q": ParamSpec((qk, s.width)), "k": ParamSpec((qk, s.width)), "v": ParamSpec((vv, s.width)),
                "g": ParamSpec((vv, s.width)), "o": ParamSpec((s.width, vv)), "norm": ParamSpec((vv,), init="ones")}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        qk, vv = s.n_heads * s.head_dim, s.n_heads * s.v_head_dim
        self._stack([tensors[n] for n in ("q", "k", "v", "g")], 0)
        self.q_off, self.k_off, self.v_off, self.g_off = 0, qk, 2 * qk, 2 * qk + vv
        self.a_off, self.b_off = 0, -1
        self.conv_w = self.conv_b = self.dt_bias = self.a_log = self.skip = None
        self.log_decay = torch.tensor([max(math.log(d), self.NO_DECAY_LEFT) if d > 0 else self.NO_DECAY_LEFT for d in s.decay],
                                      dtype=torch.float32, device=self.w_in.device)
        self.gain, self.w_o = tensors["norm"].float().contiguous(), tensors["o"]

    def forward(self, h, ctx, kv, state):
        s = self.spec
        proj = ops.linear(h, self.w_in, out_dtype=self.build.dtype)
        o = self._recur(proj, None, ctx, state)
        y = ops.state_output(o, proj[:, self.g_off: self.g_off + o.shape[1]], self.gain, 1, s.norm_eps, False, self.build.dtype, logistic=True)
        return ops.linear(y, self.w_o, out_dtype=torch.float32)
