"""Norm parts: LayerNorm (with or without bias) and RMSNorm.

LayerNorm: y = (x - mean) * rsqrt(var + eps) * gamma + beta with var = mean((x-mean)^2);
RMSNorm: y = x * rsqrt(mean(x^2) + eps) * gamma; with ``weight_offset`` c the stored scale w is an offset,
gamma = c + w (formed once, in float32, when the tensors are loaded).  Statistics are float32.  With
``branch_scale`` the norm also stores a scale s per channel for what a block adds before it, and ``post`` runs the
norm after the sum: x <- norm(a x + s * branch) with a = ``residual_scale``, in place.  ``output_scale`` c multiplies the
result (folded into gamma and beta when they are loaded).  ``one_number``: the stored scale is a single number for all
coordinates.  The
reference's norm shader has both as modes (crates/thuban_kernel/wgsl/norm.wgsl:66-83,
112-121) and picks by config key (crates/thuban_architectures/src/phi.rs:55-63).
"""
from __future__ import annotations

import torch

from ..registry import NORMS
from ..weights.sources import WeightSpec
from .base import Norm, vec


class _RowNorm(Norm):
    mode = "layer"
    graph_safe = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.width = int(params["width"])
        self.eps = float(params["eps"])
        self.has_bias = bool(params.get("bias", False))
        # a scale stored as an offset: the row is multiplied by weight_offset + w (0: by w itself)
        self.weight_offset = float(params.get("weight_offset", 0.0))
        # for a block that norms after the sum: the residual's weight, and whether a scale of the branch is stored
        self.residual_scale = float(params.get("residual_scale", 1.0))
        self.has_branch_scale = bool(params.get("branch_scale", False))
        self.output_scale = float(params.get("output_scale", 1.0))
        self.one_number = bool(params.get("one_number", False))
        self.gamma = self.beta = self.branch_scale = None

    def weights(self):
        init = "normal" if self.weight_offset else "gamma"
        w = {"weight": WeightSpec((), role="vector", init=init) if self.one_number else vec(self.width, init=init)}
        if self.has_bias:
            w["bias"] = vec(self.width)
        if self.has_branch_scale:
            w["branch_scale"] = vec(self.width, init="gamma")
        return w

    def load(self, tensors):
        self.gamma = tensors["weight"]
        if self.one_number:
            self.gamma = self.gamma.to(torch.float32).expand(self.width).contiguous()
        if self.weight_offset:
            self.gamma = (self.gamma.to(torch.float32) + self.weight_offset).contiguous()
        self.beta = tensors.get("bias")
        if self.output_scale != 1.0:
            self.gamma = (self.gamma.to(torch.float32) * self.output_scale).contiguous()
            self.beta = (self.beta.to(torch.float32) * self.output_scale).contiguous() if self.beta is not None else None
        self.branch_scale = tensors.get("branch_scale")

    supports_pending = True
    supports_router = True

    def post(self, x, branch, copy=None):
        """x <- norm(residual_scale x + branch_scale * branch) in place; ``branch``: a ``Pending`` of partial sums
        (and a bias).  ``copy``: a tensor of another element type that receives the result too."""
        self.ops.post_norm(x, branch.partials, branch.bias, self.branch_scale, self.residual_scale, self.gamma, self.beta,
                           self.eps, self.mode, out_copy=copy)

    def forward(self, x, want, row_index=None, pending=None, router=None, out=None, gather=None):
        """``out``: {element type: tensor} to write into instead of new tensors (then ``want`` is ignored).  ``gather``
        [S]: x is [T, S, width] and its weighted sum over the streams is normed."""
        rows = row_index.numel() if row_index is not None else x.shape[0]
        if out is None:
            out = {}
            for dt in set(want):
                out[dt] = torch.empty((rows, self.width), dtype=dt, device=x.device)
        kw = {} if gather is None else {"gather": gather}
        self.ops.row_norm(x, self.gamma, self.beta, self.eps, self.mode, out_f32=out.get(torch.float32),
                          out_bf16=out.get(torch.bfloat16), row_index=row_index, pending=pending, router=router, **kw)
        return out


@NORMS.register("layernorm")
class LayerNorm(_RowNorm):
    mode = "layer"


@NORMS.register("rmsnorm")
class RMSNorm(_RowNorm):
    mode = "rms"

    def __init__(self, params, ctx):
        super().__init__({**params, "bias": False}, ctx)
