"""Two mixers side by side on the same input."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..csrc import ops
from .base import KvRequest, Mixer, StateRequest
from .registry import build_part, register_mixer


@register_mixer("pair")
class Pair(Mixer):
    """left_scale left(h) + right_scale right(h).  Mixers that share their products (``Mixer.shares_products``) run between two
    common ones: [left's rows | right's rows] times h with their biases, and one product over [left's inner result times its
    factor | right's | tail] whose matrix lies side by side alike; the factors act on the inner results before they are
    rounded.  The output biases, times their factors, are two columns of that matrix (the bias rounded to the weights' type
    and what the rounding left), which the ones in the tail pick.  Other mixers run one after the other."""

    kernels = ("linear", "linear_mma", "linear_tc", "gemm_tc")
    graph_safe = True

    def __init__(self, spec, build):
        super().__init__(spec, build)
        self.left = build_part("mixer", spec.left, build)
        self.right = build_part("mixer", spec.right, build)
        if self.left.cache_request() is not None and self.right.cache_request() is not None:
            raise ValueError("a pair of mixers that both cache keys and values is not built")
        self.together = self.left.shares_products and self.right.shares_products and self.right.leaves_tail
        self.w_in: Optional[torch.Tensor] = None

    def children(self):
        return {"left": self.left, "right": self.right}

    def bound(self) -> None:
        if not self.together:
            return
        a, b = self.left, self.right
        dt = a.w_in.dtype if a.w_in.dtype == b.w_in.dtype else torch.float32
        dev = a.w_in.device
        self.at = a.w_in.shape[0]
        self.w_in = torch.cat([a.w_in.to(dt), b.w_in.to(dt)])
        self.b_in = None
        if a.b_in is not None or b.b_in is not None:
            self.b_in = torch.zeros(self.w_in.shape[0], dtype=torch.float32, device=dev)
            for at, m in ((0, a), (self.at, b)):
                if m.b_in is not None:
                    self.b_in[at: at + m.w_in.shape[0]] = m.b_in
        n = a.inner_dim + b.inner_dim
        bias = None
        for f, m in ((self.spec.left_scale, a), (self.spec.right_scale, b)):
            if m.b_o is not None:
                bias = f * m.b_o if bias is None else bias + f * m.b_o
        # the tail fills the rows up to whole 16-byte pieces; with a bias it is at least its two columns
        self.tail = -n % 8
        if bias is not None and self.tail < 2:
            self.tail += 8
        od = a.w_o.dtype if a.w_o.dtype == b.w_o.dtype else torch.float32
        self.w_o = torch.zeros((a.w_o.shape[0], n + self.tail), dtype=od, device=dev)
        self.w_o[:, : a.inner_dim], self.w_o[:, a.inner_dim: n] = a.w_o, b.w_o
        if bias is not None:
            self.w_o[:, n] = bias
            self.w_o[:, n + 1] = bias - self.w_o[:, n].float()
        for m in (a, b):  # their own copies are not needed any more
            m.w_in = m.w_o = m.b_in = None

    def cache_request(self) -> Optional[KvRequest]:
        return self.left.cache_request() or self.right.cache_request()

    def state_request(self) -> Optional[Dict[str, StateRequest]]:
        own = {name: m.state_request() for name, m in self.children().items()}
        return {name: r for name, r in own.items() if r is not None} or None

    def forward(self, h, ctx, kv, state):
        s = self.spec
        of = lambda name: state.get(name) if state else None
        if not self.together:
            d = self.left.forward(h, ctx, kv, of("left")) * s.left_scale
            return d.add_(self.right.forward(h, ctx, kv, of("right")), alpha=s.right_scale)
        dt = self.build.dtype
        proj = ops.linear(h, self.w_in, out_dtype=dt, bias=self.b_in)
        out = torch.empty((h.shape[0], self.w_o.shape[1]), dtype=dt, device=h.device)
        self.left.inner(proj, 0, out, 0, s.left_scale, ctx, kv, of("left"))
        self.right.inner(proj, self.at, out, self.left.inner_dim, s.right_scale, ctx, kv, of("right"), tail=self.tail)
        return ops.linear(out, self.w_o, out_dtype=torch.float32)
