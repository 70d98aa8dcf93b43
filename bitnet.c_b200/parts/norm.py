"""Norms with the residual add fused in front of them."""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import Norm, ParamSpec, StreamDelta
from .registry import register_norm


@register_norm("rmsnorm")
class RmsNorm(Norm):
    """out = v / sqrt(mean(v^2) + eps) * weight with v = x + delta, statistics in float32
    (src/transformer/rmsnorm_scalar.c:4-13; fused with the residual as src/gpu_cuda.cu:5077)."""

    kernels = ("norm",)
    graph_safe = True

    def params(self) -> Dict[str, ParamSpec]:
        one_plus = bool(getattr(self.spec, "one_plus", False))
        return {"weight": ParamSpec((self.spec.width,), init="around_zero" if one_plus else "ones",
                                    optional=bool(getattr(self.spec, "optional", False)))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"]
        if self.weight is not None and getattr(self.spec, "one_plus", False):
            # a gain kept as its offset from one: the factor 1 + w, made once in float32 (in bfloat16 the sum would lose the
            # stored gain's low bits); the kernels read gains of either type
            self.weight = (1.0 + self.weight.float()).contiguous()

    def sink(self, x, ctx):
        # a product in bfloat16 of few rows, or of many, can add to the residual and prepare this norm's output
        if self.build.dtype != torch.bfloat16 or not ops.USE_FUSED_NORM or x.dtype != torch.float32:
            return None
        if (x.shape[0] <= ops.MMA_MAX_ROWS and ops.USE_TCGEN05) or ops.own_gemm_sink_rows(x.shape[0]):
            return ops.NormSink(x, self.weight, self.spec.eps)
        return None

    def add_norm(self, x, delta, ctx, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.spec.width), dtype=self.build.dtype, device=x.device)
        return ops.add_rmsnorm(x, delta, self.weight, self.spec.eps, out, rows=rows)

    def scaled_add_norm(self, x, alpha, delta):
        """The norm after the sum: x = norm(alpha * x + delta) in place on the float32 residual; returns
        the same rows in the compute type (x itself when that is float32)."""
        if self.build.dtype == torch.float32:
            ops.scaled_add_rmsnorm(x, alpha, delta, self.weight, self.spec.eps)
            return x
        out = torch.empty(x.shape, dtype=self.build.dtype, device=x.device)
        return ops.scaled_add_rmsnorm(x, alpha, delta, self.weight, self.spec.eps, out)


@register_norm("layernorm")
class LayerNorm(Norm):
    """out = (v - mean) / sqrt(mean((v - mean)^2) + eps) * weight + bias with v = x + delta, statistics in float32.  The
    residual may hold several streams side by side: v is then what ``streams_norm`` is told to read of them (by default
    their sum), and a delta comes as ``StreamDelta``."""

    kernels = ("streams",)
    graph_safe = True

    def __init__(self, spec, build):
        super().__init__(spec, build)
        if spec.width > ops.STREAMS_MAX_WIDTH:
            raise ValueError(f"layernorm: width={spec.width} must be at most {ops.STREAMS_MAX_WIDTH}")

    def params(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.spec.width,), init="ones"), "bias": ParamSpec((self.spec.width,), init="around_zero")}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight, self.bias = tensors["weight"], tensors["bias"]

    def streams_norm(self, x, pending, read=None, rows=None, **convolution):
        """Bring ``pending`` (None or a ``StreamDelta``) into the streams of x and norm sum_s read[s] x_s; the rest as
        for ``ops.streams_norm``."""
        update = dict(delta=pending.delta, mix=pending.mix, scale=pending.scale, mult=pending.mult) if pending is not None else {}
        return ops.streams_norm(x, x.shape[1] // self.spec.width, self.weight, self.bias, self.spec.eps, self.build.dtype,
                                read=read, rows=rows, **update, **convolution)

    def add_norm(self, x, delta, ctx, rows=None):
        if delta is not None and not isinstance(delta, StreamDelta):
            delta = StreamDelta(delta.sum(0) if delta.dim() == 3 else delta, 1, None, None, 1.0)
        return self.streams_norm(x, delta, rows=rows)
