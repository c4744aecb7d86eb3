"""An element-wise squashing in a norm's place, and a learned scale of what a sublayer adds to the stream.

``TanhNorm``: y = tanh(alpha x) * w + b with a learned number alpha and learned vectors w and b; no mean and no
variance enter. The stream x, the sum into it and the arithmetic are float32 on every path; y is rounded once to the
path's dtype. With ``branch_scale`` the norm also owns the learned vector by which the sublayer behind it is multiplied,
element by element, when its output comes back: it leaves that vector on the stream (``Stream.fold``) and the next norm
computes x + scale * output in float32, as it folds any pending output.
"""

from __future__ import annotations

import torch

from .base import Norm, Stream, TensorSpec, register_norm
from .norm import Normed


class TanhNorm(Norm):
    """params: size, branch_scale (bool, default False)."""

    def __init__(self, params):
        super().__init__(params)
        self.size = int(params["size"])
        self.branch_scale = bool(params.get("branch_scale", False))
        self.gain = self.shift = self.scale = None
        self.alpha = 1.0
        self.dtype = None

    def tensor_specs(self):
        specs = {"weight": TensorSpec((self.size,), "gain"), "alpha": TensorSpec((), "gain"),
                 "b": TensorSpec((self.size,), "vector")}
        if self.branch_scale:
            specs["scale"] = TensorSpec((self.size,), "gain")
        return specs

    def bind(self, tensors, runtime):
        f = lambda key: tensors[key].float().contiguous()
        self.gain, self.shift = f("weight"), f("b")
        self.alpha = float(tensors["alpha"].float().item())
        self.scale = f("scale") if self.branch_scale else None
        self.dtype = runtime.dtype

    def forward(self, ctx, stream: Stream) -> Normed:
        x, branch = stream.x, stream.branch
        if x.dtype != torch.float32:
            raise TypeError("this norm follows a float32 residual stream")
        if stream.branch2 is not None or stream.scale != 1.0:
            raise TypeError("this norm folds one pending output at a time")
        x_new = ctx.ops.empty_like(x) if branch is not None else x
        rows = ctx.ops.tanh_norm(x, branch, stream.fold if branch is not None else None, self.alpha, self.gain, self.shift,
                                 x_new, self.dtype)
        normed = Normed(ctx.ops, x, branch, self.gain, 0.0, x_new)
        normed.mark_fused(rows)
        stream.x = x_new
        stream.branch = None
        stream.fold = self.scale  # the sublayer behind this norm comes back multiplied by it
        return normed


register_norm("tanh_norm", TanhNorm)
