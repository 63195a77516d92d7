"""Sinilorn as a ``ModelSpec``.

The rows travel as ``streams`` copies (block ``streams``): a part reads norm(sum_s in[s] x_s), a LayerNorm with a scale and
no bias, and what it adds goes into every stream, x_t <- sum_s mix[s, t] x_s + out[t] y (``hyper_connection``); the
final norm reads the streams' sum.  The mixer is latent attention with queries through a latent of their own, a sliding
window, a sink per head, an output gate and a rotated part in the half layout with YaRN frequencies
(``latent_attention``; a layer with ``kv_from`` reads the latent rows another layer cached, which then stay reachable for
the longest window among their readers), or Griffin's recurrent block (``rglru``).  The feed-forward is a SiLU-gated unit
with biases (``gated_mlp``), a mixture of clamped gated experts with a softmax router that has a correction for the
choice and identity experts (``grouped_topk_moe``), or absent.  The logits are scaled by a constant, which rides on the
final norm's scale.  Checkpoints name tensors ``embed``, ``l<i>.norm1``, ``l<i>.hc1.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm`` and ``head``.  The reference registers its families in one table keyed by the checkpoint's architecture
string (crates/thuban_architectures/src/loader.rs:39-60).
"""
from __future__ import annotations

from ..config.sinilorn import DEFAULT_MAX_POSITIONS, DenseMlp, LatentAttention, SinilornConfig
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..registry import ARCHITECTURES

DECAY_SCALE = 8.0         # log a = -8 r softplus(lam)
SWISH_SLOPE = 1.702       # of the experts' clamped activation
DENSE_NAMES = (("gate_proj.weight", "gate"), ("up_proj.weight", "up"), ("down_proj.weight", "down"),
               ("gate_proj.bias", "gate.b"), ("up_proj.bias", "up.b"), ("down_proj.bias", "down.b"))


def _latent(cfg, m, cache_window):
    position = None
    if m.rot is not None:
        params = {"rotary_dim": m.rot_dim, "theta": m.rot.base, "style": "half", "max_positions": DEFAULT_MAX_POSITIONS}
        if m.rot.yarn is not None:
            params["yarn"] = dict(zip(("factor", "original", "fast", "slow"), m.rot.yarn))
        position = PartSpec("rope", params)
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
        "kv_rank": m.kv_rank, "scale": m.scale, "norm_eps": cfg.eps, "window": m.window, "own_cache": m.kv_from is None,
        "cache_window": cache_window, "position": position, "q_rank": m.q_rank, "sinks": True, "out_gate": True})


@ARCHITECTURES.register("Sinilorn")
class SinilornArchitecture:
    config_class = SinilornConfig

    @staticmethod
    def parse_config(d: dict) -> SinilornConfig:
        return SinilornConfig.from_dict(d)

    @staticmethod
    def model_spec(cfg: SinilornConfig) -> ModelSpec:
        norm = PartSpec("layernorm", {"width": cfg.width, "eps": cfg.eps})
        hc = PartSpec("hyper_connection", {"streams": cfg.streams})
        # latent rows stay in the cache for the longest window of the layers that read them (0: for good)
        reach = {}
        for i, layer in enumerate(cfg.layers):
            if isinstance(layer.mixer, LatentAttention):
                owner = i if layer.mixer.kv_from is None else layer.mixer.kv_from
                reach.setdefault(owner, []).append(layer.mixer.window)
        layers, order, stored = [], [], {}
        for i, layer in enumerate(cfg.layers):
            m, pre = layer.mixer, f"l{i}."
            kv_from = None
            if isinstance(m, LatentAttention):
                kv_from = m.kv_from
                windows = reach[i] if kv_from is None else [m.window]
                mixer = _latent(cfg, m, max(windows) if min(windows) else 0)
            else:
                mixer = PartSpec("rglru", {"hidden_size": cfg.width, "width": m.width, "blocks": m.blocks, "conv_taps": m.taps,
                                           "decay_scale": DECAY_SCALE})
            parts = {"hc1": hc, "norm1": norm, "mixer": mixer}
            stored[f"{pre}norm1.weight"] = f"{pre}norm1"
            f = layer.mlp
            if f is not None:
                parts.update({"hc2": hc, "norm2": norm})
                stored[f"{pre}norm2.weight"] = f"{pre}norm2"
                if isinstance(f, DenseMlp):
                    parts["ffn"] = PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": f.ff, "act": "silu",
                                                          "bias": True, "pending": True})
                    for ours, theirs in DENSE_NAMES:
                        stored[f"{pre}mlp.{ours}"] = f"{pre}mlp.{theirs}"
                else:
                    parts["ffn"] = PartSpec("grouped_topk_moe", {
                        "hidden_size": cfg.width, "intermediate_size": f.ff, "num_experts": f.experts, "identity": f.identity,
                        "top": f.top, "correction": True, "act": "swish_clamped", "act_slope": SWISH_SLOPE,
                        "act_limit": f.limit})
            layers.append(LayerSpec("streams", parts, pre, {"hc1": "hc1.", "norm1": "norm1.", "mixer": "mix.", "hc2": "hc2.",
                                                            "norm2": "norm2.", "ffn": "mlp."}))
            order.append(LayerCall(i, cache_of=kv_from))
        stored.update({"embed.weight": "embed", "final.norm.weight": "final.norm", "head.weight": "head"})
        final = PartSpec("layernorm", {"width": cfg.width, "eps": cfg.eps, "output_scale": cfg.logit_scale})
        return ModelSpec(
            architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width,
            max_positions=DEFAULT_MAX_POSITIONS, layers=tuple(layers), order=tuple(order), final_norm=final,
            embed_name="embed.", final_norm_name="final.norm.", head_name="head.", stored_names=stored, streams=cfg.streams)
