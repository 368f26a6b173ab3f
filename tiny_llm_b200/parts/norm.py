"""Norms.  RMSNorm: y_j = (w_j x_j) / sqrt(mean_j(x_j^2) + eps), statistics in 32-bit
(tiny_llm/ops/cuda/norm.cu:16-49).  Any width; the reference stops at 2048.  With `one_plus` the stored weight lies
around zero and the norm multiplies by 1 + w_j.  LayerNorm: y_j = (x_j - mean) / sqrt(var + eps) w_j (+ b_j)."""
from __future__ import annotations

from .. import ops
from ..weights import FLOAT32, WeightSpec
from .registry import register_part


class RMSNorm:
    graph_safe = True   # launches kernels only: a step through this part can be captured in a CUDA graph

    def __init__(self, size: int, eps: float, weight_suffix: str = ".weight", one_plus: bool = False,
                 scalar: bool = False):
        """`weight_suffix`: what the weight is called behind the part's name ("" when the name is the tensor's).
        `one_plus`: the norm multiplies by 1 + the stored weight (added once, in 32-bit, when the weight is loaded).
        `scalar`: the stored weight is ONE number for all coordinates (a tensor without dimensions); it is spread over
        the row when it is loaded."""
        self.size = size
        self.scalar = scalar
        self.eps = float(eps)
        self.weight_suffix = weight_suffix
        self.one_plus = one_plus
        self.weight = None

    def weight_specs(self, prefix: str):
        init = {"init": ("normal", 0.1)} if self.one_plus else ({"init": ("uniform", 0.5, 1.5)} if self.scalar else {})
        return [WeightSpec(prefix + self.weight_suffix, () if self.scalar else (self.size,), FLOAT32, **init)]

    def load(self, prefix: str, weights) -> None:
        w = weights[prefix + self.weight_suffix]
        if self.scalar:
            w = w.reshape(1).expand(self.size).contiguous()
        self.weight = (w + 1.0).contiguous() if self.one_plus else w

    def add_into(self, ctx, branch, resid, copy=None, then=None):
        """resid += norm(branch): for a block that norms a branch's output before it joins the stream.  `branch` is a
        zeroed float32 buffer that products added into; it is handed back zeroed.  `copy` (bfloat16) also receives the
        new stream, rounded.  `then`: the norm that reads the new stream next; a norm that can take it along returns what
        `then.forward(ctx, resid)` would (this one returns None)."""
        ops.rms_norm_add(branch, self.weight, self.eps, 1.0, resid, copy=copy)

    def forward(self, ctx, x, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        out = ctx.workspace.get("norm_out", (n, self.size), ctx.dtype)
        ops.rms_norm(x, self.weight, self.eps, out, rows)
        return out


class DynamicTanh:
    """Dynamic Tanh: y_j = tanh(alpha x_j) w_j + b_j with one learned number alpha.  It takes the place of a norm and
    computes no mean or variance, so a row's output does not depend on the row's other values.  The weight is
    stored under the part's own name, the bias and alpha beside it as `<name>.b` and `<name>.alpha`."""
    graph_safe = True

    def __init__(self, size: int):
        self.size = size
        self.weight = self.bias = self.alpha = None

    def weight_specs(self, prefix: str):
        return [WeightSpec(prefix, (self.size,), FLOAT32),
                WeightSpec(prefix + ".b", (self.size,), FLOAT32, init=("normal", 0.05)),
                WeightSpec(prefix + ".alpha", (), FLOAT32, init=("const", 0.75))]

    def load(self, prefix: str, weights) -> None:
        self.weight = weights[prefix]
        self.bias = weights[prefix + ".b"]
        self.alpha = weights[prefix + ".alpha"].reshape(1).contiguous()

    def forward(self, ctx, x, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        out = ctx.workspace.get("norm_out", (n, self.size), ctx.dtype)
        ops.dyt_norm(x, self.weight, self.bias, self.alpha, out, rows)
        return out


class LayerNorm:
    """y_j = (x_j - mean) / sqrt(mean((x - mean)^2) + eps) * w_j + b_j, all in 32-bit.  The weight is stored under the
    part's own name, the bias beside it as `<name>.b` (`has_bias=False`: there is none)."""
    graph_safe = True

    def __init__(self, size: int, eps: float, has_bias: bool = True):
        self.size, self.eps, self.has_bias = size, float(eps), has_bias
        self.weight = self.bias = None

    def weight_specs(self, prefix: str):
        specs = [WeightSpec(prefix, (self.size,), FLOAT32, init=("uniform", 0.5, 1.5))]
        if self.has_bias:
            specs.append(WeightSpec(prefix + ".b", (self.size,), FLOAT32, init=("normal", 0.2)))
        return specs

    def load(self, prefix: str, weights) -> None:
        self.weight, self.bias = weights[prefix], weights[prefix + ".b"] if self.has_bias else None

    def add_into(self, ctx, branch, resid, copy=None, then=None):
        """resid += norm(branch), as RMSNorm.add_into; a following layer norm `then` of the new stream is taken in the same
        kernel and its output returned."""
        if not isinstance(then, LayerNorm) or then.size != self.size:
            ops.layer_norm_add(branch, resid, self.weight, self.bias, self.eps, copy=copy)
            return None
        out = ctx.workspace.get("norm_out", (resid.shape[0], self.size), ctx.dtype)
        ops.layer_norm_add(branch, resid, self.weight, self.bias, self.eps, copy=copy,
                           then=(then.weight, then.bias, then.eps), out=out)
        return out

    def join(self, ctx, branch, resid, stream_scale, out_bias=None, copy=None, depth=None) -> None:
        """resid <- norm(stream_scale * resid + branch + out_bias): for a block that norms the sum.  `branch` is a zeroed
        float32 buffer that products added into; it is handed back zeroed.  `copy` (bfloat16) also receives the new
        stream, rounded.  `depth` (stages, how many hold results, weights, whether to keep this one): the result is
        averaged with the earlier ones on its way into the stream."""
        stages, done, mix, keep = depth if depth is not None else (None, 0, None, False)
        ops.post_norm_join(branch, resid, self.weight, self.bias, self.eps, stream_scale, out_bias=out_bias, copy=copy,
                           stages=stages, done=done, mix=mix, keep=keep)

    def forward(self, ctx, x, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        out = ctx.workspace.get("norm_out", (n, self.size), ctx.dtype)
        ops.layer_norm(x, self.weight, self.bias, self.eps, out, rows)
        return out


register_part("norm", "rms_norm", RMSNorm)
register_part("norm", "layer_norm", LayerNorm)
register_part("norm", "dynamic_tanh", DynamicTanh)
