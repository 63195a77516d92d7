"""A mixer that reads its rows through a causal convolution over time: h <- x + conv(x) per channel,

    conv(x)_t = sum_j w[:, j] x_(t - taps + 1 + j),   zeros before the sequence,

then any registered mixer on h.  The rows are read as they are kept (float32); their last taps - 1 are fixed-size state of
the request and lie before the inner mixer's state in one row of the cache manager's slab.  The reference has no such
convolution; its hybrid family convolves behind the projections, inside the mixer
(crates/thuban_architectures/src/qwen35/state.rs:5-55).
"""
from __future__ import annotations

import torch

from ..cache.manager import StateSpec
from ..errors import ConfigError, ModelError
from ..registry import MIXERS
from .base import Mixer
from .block import branch_of, settle
from .recurrent import conv_weight


@MIXERS.register("input_conv")
class InputConv(Mixer):
    """params: hidden_size, taps (1 to 64), mixer (PartSpec).  tensors: ``input_conv.weight`` [hidden, taps] and the inner
    mixer's own."""

    returns_pending = True
    CONV = "input_conv.weight"

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.taps = int(params["hidden_size"]), int(params["taps"])
        if not 1 <= self.taps <= 64:
            raise ConfigError(f"input_conv: {self.taps} taps are not supported (1 to 64)")
        inner = params["mixer"]
        self.inner = MIXERS.get(inner.kind)(inner.params, ctx)
        spec = self.inner.state_spec()
        if spec is not None and (len(spec.shape) != 1 or spec.dtype != torch.float32):
            raise ConfigError("input_conv: the inner mixer's state must be one float32 row")
        self.n_conv, self.n_inner = (self.taps - 1) * self.hidden, spec.shape[0] if spec is not None else 0
        self.graph_safe = self.inner.graph_safe

    def weights(self):
        return {self.CONV: conv_weight(self.hidden, self.taps), **self.inner.weights()}

    def subparts(self):
        return [self.inner]

    def fused(self):
        return self.inner.fused()

    def load(self, t):
        self.w_conv = t[self.CONV]
        self.inner.load({k: v for k, v in t.items() if k != self.CONV})

    def input_dtypes(self):
        return (torch.float32,)

    def cache_spec(self):
        return self.inner.cache_spec()

    def state_spec(self):
        n = self.n_conv + self.n_inner
        return StateSpec((n,), torch.float32) if n else None

    def step_needs(self):
        return self.inner.step_needs()

    def plan_key(self):
        return (type(self), self.inner.plan_key())

    def plan_step(self, step, captured):
        return self.inner.plan_step(step, captured)

    def _run(self, rows, carry, step, cache, state, writes_cache):
        if state is None and self.n_conv + self.n_inner:
            raise ModelError("input_conv needs a state slab")
        ring = state[:, :self.n_conv] if self.n_conv else None
        inner_state = state[:, self.n_conv:] if self.n_inner else None
        want = list(dict.fromkeys(self.inner.input_dtypes()))
        h = torch.empty(rows.shape, dtype=want[0] if len(want) == 1 else torch.float32, device=rows.device)
        if rows.shape[0] == len(step.entries):         # single tokens: what is pending and the convolution in one launch
            self.ops.row_post(rows, carry, out=h, conv=(self.w_conv, ring, step.pos, step.slot))
        else:
            settle(self, rows, carry)
            self.ops.short_conv(rows, 0, self.w_conv, None, "plus_input", step.pos, step.slot, ring, h)
        x = {h.dtype: h}
        for dt in want:
            if dt not in x:
                x[dt] = torch.empty(rows.shape, dtype=dt, device=rows.device)
                self.ops.cast_rows(h, x[dt])
        return branch_of(self.inner, rows, lambda r: self.inner.forward(x, r, step, cache, inner_state, writes_cache))

    def from_rows(self, residual, carry, step, cache, state, writes_cache=True):
        return self._run(residual, carry, step, cache, state, writes_cache)

    def forward(self, x, residual, step, cache, state, writes_cache=True):
        return self._run(x[torch.float32], None, step, cache, state, writes_cache)
