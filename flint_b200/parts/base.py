"""What every part of a layer looks like to the model that holds it.

A part gets its sizes and constants as parameters, names the tensors it expects under
its own prefix, receives them once, and then runs on whatever rows a step brings.
No part knows which architecture it is in; the reference's ops take spec structs in
the same spirit (``NormSpec``, ``AttnSpec``, ``RopeArgs``, ``MlpSpec``:
crates/thuban_model/src/ops/*.rs).

Interfaces
----------
Norm          ``forward(x, want, row_index=None, pending=None, router=None) -> {dtype: tensor}``
              x is the float32 residual stream [T, H] (or, with ``gather``, several streams [T, S, H] whose weighted
              sum is normed); ``want`` is the set of element
              types the next part asked for.  A norm with ``supports_pending`` applies a
              ``Pending`` addition to x first; one with ``supports_router`` can fill a
              ``RouterRequest``.  Both are optional abilities; the block works without them.
Mixer         ``input_dtypes()``, ``cache_spec()``, ``state_spec()``, optionally ``step_needs()`` (rows cut into
              tiles), ``plan_step(step, captured)`` (how this step's work is cut) and ``plan_key()`` (which mixers plan alike),
              ``forward(x, residual, step, cache, state, writes_cache=True)``:
              adds its output into ``residual`` (float32 [T, H]) in place and returns None,
              or returns a ``Pending`` that the block hands to the next norm.  One with
              ``from_rows(residual, carry, step, cache, state, writes_cache)`` forms its input from the rows
              themselves, with the addition ``carry`` (or None) applied to them on the way, and returns a ``Pending``.
FeedForward   ``input_dtypes()``, ``forward(x, residual, step)``: adds into ``residual`` or
              returns a ``Pending``.  A feed-forward with ``router_request(n_rows)`` gets the
              filled request back as ``forward(..., routed=request)``.
PositionEncoding  ``rotary_dim``, ``style`` ("half": dims i and i + rotary_dim/2 rotate together, "interleaved":
              dims 2i and 2i + 1), ``tables() -> (cos, sin)`` float32 [positions, rotary_dim/2]; one named by
              ``ModelSpec.embed_position`` instead has ``after_embedding(h, step)`` and adds to the embedded rows.
Block         ``forward(residual, step, cache, state, writes_cache)``: the arrangement of
              the parts of one layer.
StreamMix     ``weights()``, ``gather`` [S], ``mix`` [S, S] and ``spread`` [S] float32: how a part of a layer with several
              residual streams reads them and how what it adds goes into them.
EmbedAddition ``weights()``, ``state_spec()`` (per-request state, or None), ``forward(h, step, state)``: adds to the
              embedded rows h [T, H] in place (a table row chosen by the token and its predecessor, and the like).
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..weights.sources import WeightSpec


@dataclass
class Pending:
    """An addition to the residual stream that its producer has not applied: the next norm's
    kernel applies it while it reads the row anyway (or ``ops.apply_pending`` does, for a norm
    that cannot).  Either partial sums of a product whose K range was split
    (``partials`` [S, T, H] float32, plus an optional ``bias`` [H]), or the selected experts'
    outputs (``y`` [kT, H] with ``row_of`` [T, k] and ``gates`` [T, k], k choices a token), or both.  For a residual of
    several streams ``mix`` [S, S] ([from, to]) and ``spread`` [S] say how it goes into them: with r the addition,
    x_t <- sum_s mix[s, t] x_s + spread[t] r for all t at once.  ``branches``: several products' partial sums, each with a
    bias (or None) and a constant weight.  With ``gamma`` [H] the sum of all of it is divided by its root mean square (``eps``
    inside the root) and scaled before it is added."""
    partials: torch.Tensor | None = None
    bias: torch.Tensor | None = None
    y: torch.Tensor | None = None
    row_of: torch.Tensor | None = None
    gates: torch.Tensor | None = None
    mix: torch.Tensor | None = None
    spread: torch.Tensor | None = None
    branches: tuple = ()
    gamma: torch.Tensor | None = None
    eps: float = 0.0

    @property
    def alone(self) -> bool:
        """Whether it is added by a kernel of its own (a norm's kernel cannot apply it on the way)."""
        return self.gamma is not None or bool(self.branches)


@dataclass
class RouterRequest:
    """What a feed-forward asks a norm to compute while the normalised row is at hand: router logits over
    ``weight`` [E, H] and the choice of experts, into ``expert_ids`` and ``gates`` ([T, k] each).  The rule is
    sparsemixer top-2 with ``jitter_eps`` (``top`` 0), or, with ``top`` > 0, a softmax whose choice is limited to
    the ``keep`` best of ``groups`` equal groups of neighbouring experts, ``top`` experts a token, gates times
    ``scale``.  With ``rule`` "sigmoid": scores sigmoid(logit) over the first rows of ``weight``, the ``top`` largest
    chosen, ``gates`` their scores as they are; the last ``extra`` rows of ``weight`` are gates of always-on parts,
    and ``weights`` [T, top + extra] gets 1 for every chosen expert and those rows' sigmoids.  With ``rule``
    "sigmoid_grouped": choice scores sigmoid(logit) + ``correction`` [E] (or None), a group of neighbouring experts scores
    as the sum of its two largest choice scores, ``top`` experts of the ``keep`` best of ``groups`` groups are chosen,
    ``gates`` their sigmoids, over their sum if ``normalize``, times ``scale``.  ``rule`` "softmax_corrected": the same with
    the softmax of all logits as scores.  ``logits`` ([T, E]
    float32, optional): the logits the choice was made from are written there too (tests compare them).  ``rows``
    (optional, [*, H] float32): the float32 normalised rows are wanted as its last T rows."""
    weight: torch.Tensor
    jitter_eps: float
    expert_ids: torch.Tensor
    gates: torch.Tensor
    logits: torch.Tensor | None = None
    top: int = 0
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    rule: str = ""
    extra: int = 0
    weights: torch.Tensor | None = None
    correction: torch.Tensor | None = None
    normalize: bool = True
    rows: torch.Tensor | None = None


@dataclass
class BuildContext:
    """What parts need to know about where they run."""
    ops: object                    # the kernel set
    device: torch.device
    compute: str                   # "bfloat16" or "float32"
    shared: dict = field(default_factory=dict)   # things built once per model (position tables)
    max_context: int | None = None               # positions the model is built to serve (None: the architecture's limit)

    @property
    def act_dtype(self):
        return torch.bfloat16 if self.compute == "bfloat16" else torch.float32


class Part:
    """Base of all parts: parameters in, tensor specs out, tensors in."""

    # True if ``forward`` only launches work that reads the step's metadata from device memory
    # (so a decode step can be captured once as a CUDA graph and replayed).  A part that looks at
    # the host-side entries of the step must leave this False; the model then runs it eagerly.
    graph_safe = False

    def __init__(self, params: dict, ctx: BuildContext):
        self.params = dict(params)
        self.ctx = ctx
        self.ops = ctx.ops

    def weights(self) -> dict:
        """name (under this part's prefix) -> WeightSpec"""
        return {}

    def fused(self) -> dict:
        """Fused tensors a checkpoint may store instead of some of ``weights()``: fused name -> the names it
        stands for, stacked by rows in that order (all under this part's prefix)."""
        return {}

    def subparts(self) -> list:
        """The parts this one is made of (their tensors are its own)."""
        return []

    def load(self, tensors: dict):
        """Receives the tensors named by ``weights()`` (already on the device and typed
        by the loader's policy)."""

    def input_dtypes(self):
        return (self.ctx.act_dtype,)


class Mixer(Part):
    def cache_spec(self):
        return None

    def state_spec(self):
        return None

    def step_needs(self):
        """A ``StepNeeds`` if the mixer wants the step's rows cut into tiles (see ``engine/step.py``), else None."""
        return None

    def plan_key(self):
        """Mixers with the same key plan a step alike: one of them is asked."""
        return type(self)

    def plan_step(self, step, captured: bool):
        """Called once per step (on one mixer of each kind) before the layers run, with the host-side view of
        the batch: the mixer may work out how it will cut its work (into ``step.plans[kind]`` or the fields it
        reads later) and returns a hashable value naming everything about the plan that shapes its launches,
        or None.  A decode step that is captured as a CUDA graph (``captured``) is keyed by these values, so a
        graph is only replayed on steps that would launch the same work."""
        return None

    def forward(self, x, residual, step, cache, state, writes_cache=True):
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x, residual, step):
        raise NotImplementedError


class Norm(Part):
    supports_pending = False
    supports_router = False

    def forward(self, x, want, row_index=None, pending=None, router=None):
        raise NotImplementedError


class StreamMix(Part):
    """How one part of a layer reads and feeds the residual streams."""
    gather = mix = spread = None


class EmbedAddition(Part):
    """Something added to the embedded rows before the first layer; it may keep fixed-size state per request."""

    def state_spec(self):
        return None

    def forward(self, h, step, state):
        raise NotImplementedError


class PositionEncoding(Part):
    rotary_dim = 0
    style = "half"          # which dims of a head rotate together: "half" (i, i + rotary_dim/2) or "interleaved" (2i, 2i + 1)

    def tables(self):
        raise NotImplementedError


def matmul_dtype(*ws):
    """The element type a product over these stored matrices runs in: bfloat16 only if
    all of them are bfloat16, else float32."""
    return torch.bfloat16 if all(w.dtype == torch.bfloat16 for w in ws) else torch.float32


def vec(n, init="normal", optional=False):
    return WeightSpec((n,), role="vector", init=init, optional=optional)


def mat(*shape):
    return WeightSpec(tuple(shape), role="matrix")
