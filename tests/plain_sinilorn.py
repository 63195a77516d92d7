"""Sinilorn, plainly: one function per mechanism, whole sequences from position 0, float64, slow.

Nothing here is shared with the package: the tests compare the engine against these functions.  ``cfg`` is the
parsed config.json (a dict), ``w`` maps tensor names to float64 tensors.

The rows travel as ``streams`` copies.  For every part (mixer, then feed-forward) of every layer:
u = sum_s in[s] x_s;  y = part(norm(u));  x_t <- sum_s mix[s, t] x_s + out[t] y for all t at once; after the last layer
the copies are added up.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as nnf

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norms and activations
def rms_norm(x, g, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * g


def layer_norm(x, g, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * g


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------ streams
def gather_streams(x, hc_in):
    """x [s, T, W] -> [T, W]"""
    return torch.einsum("s,stw->tw", hc_in, x)


def spread_streams(x, y, hc_mix, hc_out):
    """every stream from the old ones (mix indexed [from, to]) and what the part adds"""
    return torch.einsum("st,snw->tnw", hc_mix, x) + hc_out[:, None, None] * y[None]


# ------------------------------------------------------------------------------------------------ rotation
def rotary_frequencies(rot):
    """(frequencies [dims/2], factor on cos and sin)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def dim_of(t):
        return dims * math.log(original / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1


def rotate(x, pos, rot):
    """x [T, heads, dim]: dim i turns with dim i + dims/2 by the row's position."""
    dims = int(rot["dims"])
    f, mag = rotary_frequencies(rot)
    ang = pos.to(F64)[:, None] * f[None, :]
    c, s = (torch.cos(ang) * mag)[:, None, :], (torch.sin(ang) * mag)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ------------------------------------------------------------------------------------------------ latent attention
def latent_rows(h, w, pre, m, eps):
    """(c [T, kv_rank], rotated shared key part [T, rot_dim]) of every token: what a cache holds."""
    C, R = int(m["kv_rank"]), int(m["rot_dim"])
    d = h @ w[pre + "dkv"].T
    c = rms_norm(d[:, :C], w[pre + "dkv.norm"], eps)
    return c, rotate(d[:, None, C:C + R], torch.arange(h.shape[0]), m["rot"])[:, 0]


def latent_queries(h, w, pre, m, eps):
    """(plain part [T, H, dim], rotated part [T, H, rot_dim])"""
    H, D, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"])
    q = (rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).view(h.shape[0], H, D + R)
    return q[..., :D], rotate(q[..., D:], torch.arange(h.shape[0]), m["rot"])


def sink_softmax(s, sink):
    """s [H, T, J] with -inf where nothing is seen; one more term exp(sink_h) in every denominator."""
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def window_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i >= j) & ((i - j < size) if size else torch.ones((), dtype=torch.bool))


def latent_attention(h, w, pre, m, eps, held=None):
    """``held``: the latent rows of the layer this one reads, or None if it makes its own.  Returns (output, rows)."""
    T = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    c, r = held if held is not None else latent_rows(h, w, pre, m, eps)
    qp, qr = latent_queries(h, w, pre, m, eps)
    k = (c @ w[pre + "uk"].T).view(T, H, D)
    v = (c @ w[pre + "uv"].T).view(T, H, V)
    s = (torch.einsum("thd,jhd->htj", qp, k) + torch.einsum("thr,jr->htj", qr, r)) * float(m["scale"])
    mask = m.get("mask")
    s = s.masked_fill(~window_mask(T, int(mask["size"]) if mask else 0)[None], -math.inf)
    o = torch.einsum("htj,jhd->thd", sink_softmax(s, w[pre + "sink"]), v).reshape(T, H * V)
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, (c, r)


# ------------------------------------------------------------------------------------------------ the linear recurrent unit
def causal_conv(u, taps, bias):
    """u [T, C], taps [C, n], the last column belongs to the row's own input; zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([u.new_zeros(n - 1, u.shape[1]), u], 0)
    return sum(padded[k:k + u.shape[0]] * taps[:, k] for k in range(n)) + bias


def block_gate(u, mats, bias):
    """sigmoid of a block-diagonal product: u [T, C], mats [B, C/B, C/B] (out, in), bias [B, C/B]"""
    B, n, _ = mats.shape
    return torch.sigmoid(torch.einsum("bij,tbj->tbi", mats, u.view(-1, B, n)) + bias).reshape(u.shape)


def rglru(h, w, pre, m):
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    r, i = block_gate(u, w[pre + "ra"], w[pre + "ra.b"]), block_gate(u, w[pre + "ri"], w[pre + "ri.b"])
    log_a = -8.0 * r * nnf.softplus(w[pre + "lam"])
    a = torch.exp(log_a)
    b = torch.sqrt(1 - a * a) * i * u
    S = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return (out * y) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def dense(h, w, pre):
    g = h @ w[pre + "gate"].T + w[pre + "gate.b"]
    u = h @ w[pre + "up"].T + w[pre + "up.b"]
    return (g * torch.sigmoid(g) * u) @ w[pre + "down"].T + w[pre + "down.b"]


def expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, w, pre, f, forced=None):
    """(chosen [T, top], weights [T, top]): numbers from ``experts`` on are identity experts.  ``forced``: choices to
    use instead of the rule's own (their weights still follow the scores)."""
    s = torch.softmax(h @ w[pre + "router"].T, -1)
    if forced is None:
        ids = torch.sort(s + w[pre + "correction"], dim=-1, descending=True, stable=True).indices[:, :int(f["router"]["top"])]
    else:
        ids = forced.to(torch.long)
    chosen = s.gather(1, ids)
    return ids, chosen / (chosen.sum(-1, keepdim=True) + 1e-20)


def moe(h, w, pre, f, forced=None):
    E, limit = int(f["router"]["experts"]), float(f["expert"]["limit"])
    ids, weights = route(h, w, pre, f, forced)
    out = torch.zeros_like(h)
    for e in range(E):
        t, c = (ids == e).nonzero(as_tuple=True)
        if len(t):
            out.index_add_(0, t, weights[t, c][:, None] * expert(h[t], w[f"{pre}e{e}.gate"], w[f"{pre}e{e}.up"],
                                                                 w[f"{pre}e{e}.down"], limit))
    return out + (weights * (ids >= E)).sum(-1, keepdim=True) * h, ids


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, w, tokens, forced=None):
    """logits [T, vocab], the summed streams after every layer [layers, T, width], the choices of every layer (or None)."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].expand(int(cfg["streams"]), -1, -1).clone()
    held, after, chosen = {}, [], []
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = layer_norm(gather_streams(x, w[pre + "hc1.in"]), w[pre + "norm1"], eps)
        if layer["type"] == "rglru":
            y = rglru(h, w, pre + "mix.", m)
        else:
            y, held[i] = latent_attention(h, w, pre + "mix.", m, eps, held[m["kv_from"]] if m.get("kv_from") is not None else None)
        x = spread_streams(x, y, w[pre + "hc1.mix"], w[pre + "hc1.out"])
        f, ids = layer.get("mlp"), None
        if f:
            h = layer_norm(gather_streams(x, w[pre + "hc2.in"]), w[pre + "norm2"], eps)
            if f["kind"] == "dense":
                y = dense(h, w, pre + "mlp.")
            else:
                y, ids = moe(h, w, pre + "mlp.", f, forced[i] if forced is not None else None)
            x = spread_streams(x, y, w[pre + "hc2.mix"], w[pre + "hc2.out"])
        chosen.append(ids)
        after.append(x.sum(0))
    logits = layer_norm(x.sum(0), w["final.norm"], eps) @ w["head"].T * float(cfg.get("logit_scale", 1.0))
    return logits, torch.stack(after), chosen
