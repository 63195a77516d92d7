"""Sokipel as a ``ModelSpec``.

Every layer is an ``outnorm`` block: x <- x + m n1(mixer(x + conv(x))); x <- x + m n2(experts(x)) (RMS norms whose scale is one
number for all coordinates, applied to what a part adds; m rides on that scale; the second half is absent in a layer without
a feed-forward).  Every mixer reads its rows through a short convolution over time (``input_conv``).  The mixer is grouped-query
attention with q and k normed over the whole projection, an interleaved rotation with banded frequencies, a sink per head and a
mask that cuts the sequence into chunks (``attention`` with these options); a gated delta rule with one decay a head and a SiLU
gate (``gated_delta``); or the weighted sum of both kinds side by side (``branches``), the attention then with biases, norms per
head, a half-layout rotation with divided frequencies, no chunks and a gate per head.  The feed-forward is a mixture of clamped
gated experts with a sigmoid router whose scores multiply what the experts read (``sigmoid_topk_moe`` with ``gated``).  The
embedded rows are scaled and the logits capped by a tanh.  Checkpoints name tensors ``embed``, ``l<i>.canon1``, ``l<i>.norm1``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm`` and ``head``.  The reference registers its families in one table keyed by the
checkpoint's architecture string (crates/thuban_architectures/src/loader.rs:39-60).
"""
from __future__ import annotations

from ..config.sokipel import DEFAULT_MAX_POSITIONS, Attention, DeltaRule, SokipelConfig
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..registry import ARCHITECTURES

UNIT_NORM_EPS = 1e-6      # the design fixes the constant under the root of the delta rule's unit norms
SWISH_SLOPE = 1.702       # of the experts' clamped activation
ATTENTION_NAMES = (("q_proj.weight", "q"), ("k_proj.weight", "k"), ("v_proj.weight", "v"), ("o_proj.weight", "o"),
                   ("q_proj.bias", "q.b"), ("k_proj.bias", "k.b"), ("v_proj.bias", "v.b"), ("q_norm.weight", "q.norm"),
                   ("k_norm.weight", "k.norm"), ("gate_proj.weight", "g"), ("sinks", "sink"))


def _position(rot, style):
    if rot is None:
        return None
    params = {"rotary_dim": rot.dims, "theta": rot.base, "style": style, "max_positions": DEFAULT_MAX_POSITIONS}
    if rot.banded is not None:
        params["banded"] = dict(zip(("factor", "low", "high", "original"), rot.banded))
    if rot.linear is not None:
        params["linear"] = rot.linear
    return PartSpec("rope", params)


def _attention(cfg, a, style, more):
    return PartSpec("attention", {
        "hidden_size": cfg.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.vdim,
        "scale": a.scale, "position": _position(a.rot, style), "chunk": a.chunk, "sinks": True, "qk_norm_eps": cfg.eps, **more})


def _delta(cfg, d):
    return PartSpec("gated_delta", {
        "hidden_size": cfg.width, "num_heads": d.heads, "num_kv_heads": d.kv_heads, "dim": d.dim, "value_dim": d.vdim,
        "conv_taps": d.taps, "unit_eps": UNIT_NORM_EPS, "norm_eps": cfg.eps, "head_decay": True, "full_gate": True,
        "gate_act": "silu"})


@ARCHITECTURES.register("Sokipel")
class SokipelArchitecture:
    config_class = SokipelConfig

    @staticmethod
    def parse_config(d: dict) -> SokipelConfig:
        return SokipelConfig.from_dict(d)

    @staticmethod
    def model_spec(cfg: SokipelConfig) -> ModelSpec:
        norm = {"width": cfg.width, "eps": cfg.eps, "one_number": True}
        out_norm = PartSpec("rmsnorm", {**norm, "output_scale": cfg.residual_mult})
        layers, stored = [], {}
        for i, layer in enumerate(cfg.layers):
            m, pre = layer.mixer, f"l{i}."
            if isinstance(m, Attention):
                mixer, sub = _attention(cfg, m, "interleaved", {"qk_norm": "whole"}), "mix."
            elif isinstance(m, DeltaRule):
                mixer, sub = _delta(cfg, m), None
            else:
                left = _attention(cfg, m.left, "half", {"qkv_bias": True, "qk_norm": "head", "head_gate": True})
                mixer, sub = PartSpec("branches", {
                    "hidden_size": cfg.width, "combine": "weighted", "scales": (m.left_scale, m.right_scale), "leave_branches": True,
                    "branches": (("left", left), ("right", _delta(cfg, m.right)))}), "mix.left."
            if sub is not None:
                for ours, theirs in ATTENTION_NAMES:
                    stored[f"{pre}{sub}{ours}"] = f"{pre}{sub}{theirs}"
            parts = {"norm1": out_norm,
                     "mixer": PartSpec("input_conv", {"hidden_size": cfg.width, "taps": cfg.canon_taps, "mixer": mixer})}
            stored[f"{pre}mix.input_conv.weight"] = f"{pre}canon1"
            stored[f"{pre}norm1.weight"] = f"{pre}norm1"
            f = layer.mlp
            if f is not None:
                parts["norm2"] = out_norm
                stored[f"{pre}norm2.weight"] = f"{pre}norm2"
                parts["ffn"] = PartSpec("sigmoid_topk_moe", {
                    "hidden_size": cfg.width, "intermediate_size": f.ff, "num_experts": f.experts, "top": f.top, "gated": True,
                    "act": "swish_clamped", "act_slope": SWISH_SLOPE, "act_limit": f.limit})
            layers.append(LayerSpec("outnorm", parts, pre, {"norm1": "norm1.", "mixer": "mix.", "norm2": "norm2.", "ffn": "mlp."}))
        stored.update({"embed.weight": "embed", "final.norm.weight": "final.norm", "head.weight": "head"})
        return ModelSpec(
            architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=DEFAULT_MAX_POSITIONS,
            layers=tuple(layers), order=tuple(LayerCall(i) for i in range(len(layers))), final_norm=PartSpec("rmsnorm", norm),
            embed_name="embed.", final_norm_name="final.norm.", head_name="head.", embed_scale=cfg.embed_scale,
            logit_softcap=cfg.softcap, stored_names=stored)
