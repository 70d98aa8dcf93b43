"""A real-gated linear recurrence per channel behind a short convolution, beside a GELU branch."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..csrc import ops
from .base import Mixer, ParamSpec, StateRequest
from .registry import register_mixer


@register_mixer("gated_linear")
class GatedLinear(Mixer):
    """y = gelu_tanh(W_y h + b) and u = conv(W_x h + b), a causal convolution per channel; r and i = the logistic function of
    block-diagonal matrices times u; per channel, from the sequence's state S (zero at first)

        l = -8 r softplus(lam);  S = e^l S_before + sqrt(1 - e^(2 l)) i u

    and W_o (S y).  The projections are one product [y | x]; its result and u are in the compute type, all behind it is
    float32.  The state and the convolution's last inputs are kept per sequence, float32."""

    kernels = ("linear", "linear_mma", "linear_tc", "gemm_tc", "gated_linear")
    graph_safe = True
    shares_products = True
    leaves_tail = True

    def __init__(self, spec, build):
        super().__init__(spec, build)
        s = spec
        if min(s.inner, s.parts) <= 0 or s.inner % s.parts:
            raise ValueError(f"gated_linear: {s.inner} channels do not form {s.parts} equal parts")
        if s.inner // s.parts > ops.GATED_LINEAR_MAX_PART or not 1 <= s.conv_taps <= ops.GATED_LINEAR_MAX_TAPS:
            raise ValueError(f"gated_linear: parts of {s.inner // s.parts} channels (at most {ops.GATED_LINEAR_MAX_PART}) or {s.conv_taps} taps "
                             f"(1 to {ops.GATED_LINEAR_MAX_TAPS}) are not supported")
        self.inner_dim = s.inner
        self.w_in: Optional[torch.Tensor] = None

    def params(self) -> Dict[str, ParamSpec]:
        s = self.spec
        n, b, p = s.inner, s.parts, s.inner // s.parts
        return {"y": ParamSpec((n, s.width)), "y.b": ParamSpec((n,)), "x": ParamSpec((n, s.width)), "x.b": ParamSpec((n,)),
                "conv": ParamSpec((n, s.conv_taps)), "conv.b": ParamSpec((n,)), "ra": ParamSpec((b, p, p)), "ra.b": ParamSpec((b, p)),
                "ri": ParamSpec((b, p, p)), "ri.b": ParamSpec((b, p)), "lam": ParamSpec((n,)), "o": ParamSpec((s.width, n))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n, dt = self.spec.inner, self.build.dtype
        f32 = lambda t: t.float().contiguous()
        y, x = tensors["y"], tensors["x"]
        wd = y.dtype if y.dtype == x.dtype else torch.float32
        self.x_off = n + -n % 8  # both branches start at a 16-byte boundary of the row
        self.w_in = torch.zeros((2 * self.x_off, y.shape[1]), dtype=wd, device=y.device)
        self.b_in = torch.zeros(2 * self.x_off, dtype=torch.float32, device=y.device)
        for at, w, b in ((0, y, "y.b"), (self.x_off, x, "x.b")):
            self.w_in[at: at + n], self.b_in[at: at + n] = w, tensors[b]
        self.conv_w, self.conv_b, self.lam = f32(tensors["conv"].t()), f32(tensors["conv.b"]), f32(tensors["lam"])
        # part by part: the rows of r, then of i
        self.w_gates = torch.cat([tensors["ra"], tensors["ri"]], dim=1).to(dt).contiguous()
        self.gate_b = f32(torch.cat([tensors["ra.b"], tensors["ri.b"]], dim=1))
        self.w_o, self.b_o = tensors["o"], None

    def state_request(self) -> StateRequest:
        return StateRequest((ops.gated_linear_floats(self.spec.inner, self.spec.conv_taps),), torch.float32)

    def forward(self, h, ctx, kv, state):
        proj = ops.linear(h, self.w_in, out_dtype=self.build.dtype, bias=self.b_in)
        out = torch.empty((h.shape[0], self.inner_dim), dtype=self.build.dtype, device=h.device)
        self.inner(proj, 0, out, 0, 1.0, ctx, kv, state)
        return ops.linear(out, self.w_o, out_dtype=torch.float32)

    def inner(self, proj, at, out, out_at, factor, ctx, kv, state, tail=0):
        n = self.spec.inner
        ops.gated_linear(proj[:, at + self.x_off: at + self.x_off + n], proj[:, at: at + n], self.conv_w, self.conv_b, self.w_gates,
                         self.gate_b, self.lam, state, ctx.tok_seq, ctx.seq_start, ctx.seq_pos0, ctx.slots, ctx.n_seqs,
                         out[:, out_at: out_at + n + tail], scale=factor, tail=tail, one_token=ctx.decode, tile_seq=ctx.tile_seq,
                         tile_row0=ctx.tile_row0)
        ctx.tap("state_out", out[:, out_at: out_at + n])
