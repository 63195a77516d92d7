"""Tiny Sinilorn configurations that differ in every size, constant and in the order of layers, and a writer of model
folders whose random weights are large enough that every mechanism shows in the logits (attention is peaked, sinks take
a real share, the recurrent unit remembers over a few tokens up to hundreds, streams differ from one another, the
experts' clamps bite, router scores and corrections are spread so that identity experts are chosen and the choice
differs from the scores' own order)."""
from __future__ import annotations

import math
import random

import torch

from tiny_puledra import write_model as _write_folder


def _rot(dims, base=10000.0, yarn=None):
    r = {"dims": dims, "base": base}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return r


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, size=None, base=10000.0, yarn=None, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": _rot(rot_dim, base, yarn), "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _unit(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, limit, experts, identity, top):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# S1: sizes that are no multiples of 8 (products on the float32 pipes, latent rows padded, values of an odd size), two
# streams, recurrent blocks of 5 channels with 3 taps and one block of all channels with 1 tap, windows shorter than a
# page, a reader with a longer window than the layer whose rows it reads and one that sees everything, a layer without a
# feed-forward, one expert a token, more identity experts than experts, YaRN on one layer and its reader.
S1 = {
    "architecture": "Sinilorn", "vocab": 83, "width": 36, "streams": 2, "norm": {"eps": 1e-5}, "logit_scale": 0.7,
    "layers": [
        _layer("rglru", _unit(20, 4, 3), _moe(12, 0.8, 2, 5, 3)),
        _layer("latent_attention", _latent(3, 10, 6, 7, 14, 20, size=7, base=300.0, yarn=(3.0, 24, 8.0, 1.0)), _dense(22)),
        _layer("latent_attention", _latent(2, 6, 6, 9, 10, 20, size=21, base=300.0, yarn=(3.0, 24, 8.0, 1.0), kv_from=1), None),
        _layer("latent_attention", _latent(5, 4, 2, 6, 18, 11, size=1), _moe(8, 2.0, 5, 0, 1)),
        _layer("rglru", _unit(14, 1, 1), _dense(9)),
        _layer("latent_attention", _latent(1, 8, 2, 5, 6, 11, kv_from=3), _moe(8, 1.2, 3, 1, 4)),
    ],
}

# S2: sizes in multiples of 16 (every product on the tensor cores in bfloat16), three streams, recurrent blocks of 32 and
# of 8 channels with 4 and 5 taps, a window of a page and one of more than a page, a layer and a reader of equal cache
# needs in one page group, experts with one identity expert.
S2 = {
    "architecture": "Sinilorn", "vocab": 160, "width": 64, "streams": 3, "norm": {"eps": 1e-6}, "logit_scale": 3.0,
    "layers": [
        _layer("latent_attention", _latent(4, 32, 16, 32, 48, 48, size=16, base=500000.0), _dense(96)),
        _layer("latent_attention", _latent(8, 16, 16, 16, 32, 48, size=40, base=500000.0, kv_from=0), _moe(32, 1.5, 8, 1, 3)),
        _layer("rglru", _unit(96, 3, 4), _moe(16, 1.0, 4, 4, 2)),
        _layer("latent_attention", _latent(4, 32, 16, 32, 48, 48, size=40, base=500000.0), _dense(64)),
        _layer("rglru", _unit(64, 8, 5), None),
    ],
}

# S3: five streams (more than the row kernel holds), no window at all, one layer of each kind, two taps
S3 = {
    "architecture": "Sinilorn", "vocab": 64, "width": 32, "streams": 5, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
    "layers": [
        _layer("rglru", _unit(48, 2, 2), _dense(40)),
        _layer("latent_attention", _latent(2, 16, 8, 16, 24, 24), _moe(16, 3.0, 4, 2, 2)),
    ],
}

# S4: one stream, whose mixing still is not a plain residual sum; the recurrent unit last
S4 = {
    "architecture": "Sinilorn", "vocab": 72, "width": 40, "streams": 1, "norm": {"eps": 1e-5}, "logit_scale": 1.5,
    "layers": [
        _layer("latent_attention", _latent(6, 8, 8, 24, 16, 32, size=12, yarn=(4.0, 16, 4.0, 1.0)), _moe(24, 1.0, 6, 3, 4)),
        _layer("rglru", _unit(40, 5, 4), _dense(48)),
    ],
}

CONFIGS = {"S1": S1, "S2": S2, "S3": S3, "S4": S4}


def tensor_shapes(cfg):
    """Every tensor of a checkpoint by name, written down here independently of the package."""
    W, S = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out.update({p + "norm1": (W,), p + "hc1.in": (S,), p + "hc1.out": (S,), p + "hc1.mix": (S, S)})
        if layer["type"] == "rglru":
            n, B = m["width"], m["blocks"]
            out.update({p + "mix.y": (n, W), p + "mix.y.b": (n,), p + "mix.x": (n, W), p + "mix.x.b": (n,),
                        p + "mix.conv": (n, m["conv"]), p + "mix.conv.b": (n,), p + "mix.ra": (B, n // B, n // B),
                        p + "mix.ra.b": (B, n // B), p + "mix.ri": (B, n // B, n // B), p + "mix.ri.b": (B, n // B),
                        p + "mix.lam": (n,), p + "mix.o": (W, n)})
        else:
            H, D, R, V, Q, C = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            out.update({p + "mix.dq": (Q, W), p + "mix.dq.norm": (Q,), p + "mix.uq": (H * (D + R), Q), p + "mix.uk": (H * D, C),
                        p + "mix.uv": (H * V, C), p + "mix.sink": (H,), p + "mix.g": (H * V, W), p + "mix.o": (W, H * V)})
            if m.get("kv_from") is None:
                out.update({p + "mix.dkv": (C + R, W), p + "mix.dkv.norm": (C,)})
        f = layer.get("mlp")
        if not f:
            continue
        out.update({p + "norm2": (W,), p + "hc2.in": (S,), p + "hc2.out": (S,), p + "hc2.mix": (S, S)})
        if f["kind"] == "dense":
            out.update({p + "mlp.gate": (f["ff"], W), p + "mlp.gate.b": (f["ff"],), p + "mlp.up": (f["ff"], W),
                        p + "mlp.up.b": (f["ff"],), p + "mlp.down": (W, f["ff"]), p + "mlp.down.b": (W,)})
        else:
            n = f["router"]["experts"] + f["router"].get("identity", 0)
            out.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            for e in range(f["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (f["expert"]["ff"], W), f"{p}mlp.e{e}.up": (f["expert"]["ff"], W),
                            f"{p}mlp.e{e}.down": (W, f["expert"]["ff"])})
    out.update({"final.norm": (W,), "head": (cfg["vocab"], W)})
    return out


def random_weights(cfg, seed=0):
    """bfloat16 tensors: matrices N(0, g^2 / fan_in) with g = 2.5 for queries, keys, routers and gates; norm scales
    1 + N(0, 0.1); the streams' reading weights 1 / S + N(0, 0.4), their mixing near the identity plus N(0, 0.2), what a
    part adds N(1, 0.5); sinks N(1, 1); corrections N(0, 0.15); lam uniform in (-7, 0.5) (decays from near one to almost
    none); other vectors N(0, 0.5)."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda shape: torch.randn(shape, generator=g)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith((".norm1", ".norm2", "final.norm", ".dq.norm", ".dkv.norm")):
            t = 1.0 + 0.1 * rn(shape)
        elif name.endswith((".hc1.in", ".hc2.in")):
            t = 1.0 / shape[0] + 0.4 * rn(shape)
        elif name.endswith((".hc1.out", ".hc2.out")):
            t = 1.0 + 0.5 * rn(shape)
        elif name.endswith((".hc1.mix", ".hc2.mix")):
            t = 0.8 * torch.eye(shape[0]) + 0.2 * rn(shape)
        elif name.endswith(".sink"):
            t = 1.0 + rn(shape)
        elif name.endswith(".correction"):
            t = 0.15 * rn(shape)
        elif name.endswith(".lam"):
            t = -7.0 + 7.5 * torch.rand(shape, generator=g)
        elif name.endswith(".conv"):
            t = 0.6 * rn(shape)
        elif len(shape) == 1 or name.endswith((".ra.b", ".ri.b")):
            t = 0.5 * rn(shape)
        elif name == "embed":
            t = rn(shape)
        else:
            gain = 2.5 if name.endswith((".uq", ".uk", ".router", ".mix.g", ".ra", ".ri")) else 1.3
            t = rn(shape) * gain / math.sqrt(shape[-1])
        w[name] = t.to(torch.bfloat16)
    return w


def write_model(folder, cfg, seed=0, weights=None):
    return _write_folder(folder, cfg, seed, weights if weights is not None else random_weights(cfg, seed))


def random_config(seed):
    """A configuration drawn at random: one to six layers in any order, odd sizes, windows of 1 to 40 positions or none,
    one to six streams, layers that read an earlier layer's latent rows with a window of their own."""
    r = random.Random(seed)
    layers = []
    for i in range(r.randint(1, 6)):
        if r.random() < 0.4:
            blocks = r.choice([1, 2, 3, 4])
            kind, m = "rglru", _unit(blocks * r.choice([1, 3, 8, 16]), blocks, r.choice([1, 2, 3, 4, 6]))
        else:
            kind = "latent_attention"
            owners = [j for j, l in enumerate(layers) if l["type"] == kind and "kv_from" not in l["mixer"]]
            size = r.choice([None, 1, 2, 5, 16, 17, 40])
            heads, dim, vdim, q_rank = r.choice([1, 2, 3, 5]), r.choice([4, 7, 8, 16]), r.choice([3, 8, 16]), r.choice([5, 8, 24])
            if owners and r.random() < 0.5:
                j = r.choice(owners)
                o = layers[j]["mixer"]
                m = _latent(heads, dim, o["rot_dim"], vdim, q_rank, o["kv_rank"], size=size, kv_from=j)
                m["rot"] = dict(o["rot"])
            else:
                m = _latent(heads, dim, r.choice([2, 4, 8]), vdim, q_rank, r.choice([6, 8, 24]), size=size, base=r.choice([50.0, 10000.0]),
                            yarn=r.choice([None, (2.0, 16, 8.0, 1.0)]))
        experts, identity = r.choice([1, 2, 5, 8]), r.choice([0, 1, 4])
        f = r.choice([None, _dense(r.choice([5, 16, 24])), _moe(r.choice([5, 8, 16]), r.choice([0.5, 2.0]), experts, identity,
                                                              r.randint(1, min(experts + identity, 6)))])
        layers.append(_layer(kind, m, f))
    return {"architecture": "Sinilorn", "vocab": r.choice([50, 97]), "width": r.choice([24, 30, 32, 40]), "streams": r.choice([1, 2, 3, 4, 6]),
            "norm": {"eps": r.choice([1e-5, 1e-6])}, "logit_scale": r.choice([1.0, 0.5, 2.5]), "layers": layers}
