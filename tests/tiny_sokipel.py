"""Tiny Sokipel configurations that differ in every size, constant and in the order of layers, and a writer of model folders
whose random weights are large enough that every mechanism shows in the logits (attention is peaked, sinks take a real share,
the delta rule remembers over a few tokens up to hundreds, the convolutions reach back, the experts' clamps bite, scores are
spread so that their use on the input and not on the output shows)."""
from __future__ import annotations

import math
import random

import torch

from tiny_puledra import write_model as _write_folder

BANDED = ("factor", "low", "high", "original")


def _rot(dims, base, banded=None, linear=None):
    r = {"dims": dims, "base": base}
    if banded:
        r["scaling"] = dict(zip(BANDED, banded))
    if linear:
        r["scaling"] = {"factor": linear}
    return r


def _heads(heads, kv_heads, dim, vdim):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim}


def _attention(heads, kv_heads, dim, vdim, chunk, rot, scale=None):
    return {**_heads(heads, kv_heads, dim, vdim), "mask": {"size": chunk}, "rot": rot, "scale": scale or dim ** -0.5}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {**_heads(heads, kv_heads, dim, vdim), "conv": conv}


def _parallel(left, rot, right, scales, scale=None):
    return {"left": {**_heads(*left), "rot": rot, "scale": scale or left[2] ** -0.5}, "right": _delta(*right),
            "left_scale": scales[0], "right_scale": scales[1]}


def _moe(ff, limit, experts, top):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _model(vocab, width, eps, scale, mult, taps, cap, layers):
    return {"architecture": "Sokipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "canon": {"taps": taps}, "logit_softcap": cap, "layers": layers}


# K1: a width that is no multiple of 4 (rows on the separate kernels, products on the float32 pipes), values of an odd size
# under the gate, three query heads a key head, a chunk shorter than a page and one across page borders, heads rotated partly,
# fully and hardly, keys of the delta rule over more than one lane a column (40) and two value heads a key head, one
# expert a token and several, a layer without a feed-forward
K1 = _model(71, 30, 1e-5, 3.0, 0.7, 4, 9.0, [
    _layer("parallel", _parallel((3, 1, 10, 7), _rot(6, 300.0, linear=3.0), (2, 2, 12, 5, 3), (0.8, 1.3)), _moe(10, 0.8, 5, 2)),
    _layer("attention", _attention(6, 2, 6, 9, 11, _rot(6, 200.0, (4.0, 1.0, 4.0, 60))), None),
    _layer("delta", _delta(4, 2, 40, 6, 2), _moe(7, 1.5, 3, 1)),
    _layer("attention", _attention(2, 1, 14, 4, 37, _rot(2, 500.0, (2.0, 0.5, 8.0, 300)), scale=0.4), _moe(9, 1.0, 4, 4)),
])

# K2: sizes in multiples of 16 (every product on the tensor cores in bfloat16, attention in tiles), two taps, a chunk of a
# page, heads of 16 to 64, one delta rule with as many key as value heads and one with four value heads a key head
K2 = _model(160, 64, 1e-6, 4.0, 0.4, 2, 20.0, [
    _layer("delta", _delta(4, 1, 32, 32, 4), _moe(32, 1.5, 8, 3)),
    _layer("attention", _attention(4, 2, 32, 48, 64, _rot(16, 10000.0, (8.0, 1.0, 4.0, 64))), _moe(16, 2.0, 6, 1)),
    _layer("parallel", _parallel((8, 2, 64, 32), _rot(64, 10000.0, linear=2.0), (2, 2, 64, 16, 4), (1.1, 0.6)), _moe(32, 1.0, 4, 2)),
    _layer("delta", _delta(2, 2, 16, 80, 5), None),
])

# K3: one tap in front of the mixers (no state of it), a convolution of one tap inside, one head, chunks of 1 and of 3, no
# frequency scaling
K3 = _model(64, 48, 1e-6, 1.0, 1.0, 1, 30.0, [
    _layer("attention", _attention(1, 1, 16, 16, 3, _rot(8, 100.0)), _moe(24, 1.2, 2, 2)),
    _layer("parallel", _parallel((2, 2, 8, 8), _rot(4, 50.0), (3, 1, 8, 12, 1), (1.0, 1.0)), None),
    _layer("attention", _attention(4, 4, 8, 12, 1, _rot(8, 100.0, (2.0, 1.0, 1.0, 30))), _moe(8, 3.0, 7, 5)),
])

# K4: the widest keys (four and eight lanes a column of the state), five taps in front, more experts than a warp has lanes
K4 = _model(90, 72, 1e-5, 2.0, 0.3, 5, 12.0, [
    _layer("delta", _delta(2, 1, 144, 24, 3), _moe(16, 1.0, 37, 4)),
    _layer("parallel", _parallel((4, 1, 24, 40), _rot(12, 1000.0, linear=4.0), (4, 2, 100, 8, 6), (0.5, 1.5)), _moe(40, 0.6, 3, 1)),
])

CONFIGS = {"K1": K1, "K2": K2, "K3": K3, "K4": K4}


def _delta_shapes(m, W, p):
    H, G, D, V, t = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
    return {p + "q": (G * D, W), p + "q.conv": (G * D, t), p + "k": (G * D, W), p + "k.conv": (G * D, t), p + "v": (H * V, W),
            p + "v.conv": (H * V, t), p + "b": (H, W), p + "a": (H, W), p + "dt_bias": (H,), p + "A_log": (H,), p + "g": (H * V, W),
            p + "norm": (V,), p + "o": (W, H * V)}


def _attention_shapes(m, W, p, left):
    H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    out = {p + "q": (H * D, W), p + "k": (G * D, W), p + "v": (G * V, W), p + "sink": (H,), p + "o": (W, H * V)}
    if left:
        out.update({p + "q.b": (H * D,), p + "k.b": (G * D,), p + "v.b": (G * V,), p + "q.norm": (D,), p + "k.norm": (D,), p + "g": (H, W)})
    else:
        out.update({p + "q.norm": (H * D,), p + "k.norm": (G * D,)})
    return out


def tensor_shapes(cfg):
    """Every tensor of a checkpoint by name, written down here independently of the package."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out.update({p + "norm1": (), p + "canon1": (W, cfg["canon"]["taps"])})
        if layer["type"] == "delta":
            out.update(_delta_shapes(m, W, p + "mix."))
        elif layer["type"] == "attention":
            out.update(_attention_shapes(m, W, p + "mix.", False))
        else:
            out.update(_attention_shapes(m["left"], W, p + "mix.left.", True))
            out.update(_delta_shapes(m["right"], W, p + "mix.right."))
        f = layer.get("mlp")
        if f:
            out.update({p + "norm2": (), p + "mlp.router": (f["router"]["experts"], W)})
            for e in range(f["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (f["expert"]["ff"], W), f"{p}mlp.e{e}.up": (f["expert"]["ff"], W),
                            f"{p}mlp.e{e}.down": (W, f["expert"]["ff"])})
    out.update({"final.norm": (), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0):
    """bfloat16 tensors.  Rows of the embedding are scaled so that the residual's entries are near one; matrices N(0, g^2 /
    fan_in) with larger g for routers and gates; scales of norms 1 + N(0, 0.1) (of q and k around 2, so that attention
    is peaked); sinks N(1, 1); convolutions N(0, 0.5); A_log and dt_bias so that decays lie between nearly one and a few
    hundredths; other vectors N(0, 0.5)."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda shape: torch.randn(shape, generator=g)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith((".q.norm", ".k.norm")):
            t = 1.6 + 0.3 * rn(shape)
        elif name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t = 1.0 + 0.1 * rn(shape)
        elif name.endswith(".sink"):
            t = 1.0 + rn(shape)
        elif name.endswith((".conv", ".canon1")):
            t = 0.5 * rn(shape)
        elif name.endswith(".A_log"):
            t = 0.5 * rn(shape)
        elif name.endswith(".dt_bias"):
            t = -3.0 + 1.5 * rn(shape)
        elif len(shape) == 1:
            t = 0.5 * rn(shape)
        elif name == "embed":
            t = rn(shape) / cfg["embedding"]["scale"]
        else:
            gain = 2.5 if name.endswith((".router", ".left.g", ".b")) else 1.3
            t = rn(shape) * gain / math.sqrt(shape[-1])
        w[name] = t.to(torch.bfloat16)
    return w


def write_model(folder, cfg, seed=0, weights=None):
    return _write_folder(folder, cfg, seed, weights if weights is not None else random_weights(cfg, seed))


def random_config(seed):
    """A configuration drawn at random: one to six layers in any order, odd sizes, chunks of 1 to 100 positions, one to six taps,
    feed-forwards present or not."""
    r = random.Random(seed)

    def heads(dims, vdims):
        kv = r.choice([1, 2, 3])
        return kv * r.choice([1, 2, 3]), kv, r.choice(dims), r.choice(vdims)

    def rot(dim):
        return 2 * r.randint(1, dim // 2), r.choice([50.0, 10000.0])

    layers = []
    for _ in range(r.randint(1, 6)):
        kind = r.choice(["attention", "delta", "parallel"])
        delta = (*heads([4, 9, 16, 33, 48, 70], [3, 8, 16, 20]), r.choice([1, 2, 3, 4, 6]))
        att = heads([4, 6, 8, 16, 24], [3, 8, 16])
        dims, base = rot(att[2])
        if kind == "delta":
            m = _delta(*delta)
        elif kind == "attention":
            m = _attention(*att, r.choice([1, 2, 5, 16, 17, 40, 100]), _rot(dims, base, r.choice([None, (4.0, 1.0, 4.0, 40), (2.0, 0.5, 2.0, 9)])))
        else:
            m = _parallel(att, _rot(dims, base, linear=r.choice([None, 2.0, 8.0])), delta, (r.choice([1.0, 0.5]), r.choice([1.0, 1.4])))
        experts = r.choice([1, 2, 5, 8])
        f = r.choice([None, _moe(r.choice([5, 8, 16]), r.choice([0.5, 2.0]), experts, r.randint(1, min(experts, 4)))])
        layers.append(_layer(kind, m, f))
    return _model(r.choice([50, 97]), r.choice([24, 30, 32, 40]), r.choice([1e-5, 1e-6]), r.choice([1.0, 5.0]), r.choice([0.3, 1.0]),
                  r.choice([1, 2, 3, 4, 6]), r.choice([8.0, 30.0]), layers)
