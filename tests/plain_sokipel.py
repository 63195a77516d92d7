"""Sokipel, plainly: one function per mechanism, whole sequences from position 0, float64, slow.

Nothing here is shared with the package: the tests compare the engine against these functions.  ``cfg`` is the parsed
config.json (a dict), ``w`` maps tensor names to float64 tensors; h [T, W] are the rows a part reads, rows 0 .. T - 1 are the
positions of one sequence.

A layer, with m = residual_mult:  x <- x + m * n1(mixer(x + conv(x)));  x <- x + m * n2(experts(x)).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norms, convolutions
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_number_norm(x, g, eps):
    """an RMS norm whose weight is a single number"""
    return unit_rms(x, eps) * g


def unit_length(x, eps):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: row t gets sum_j taps[:, j] u[t - n + 1 + j], nothing before the start"""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u], 0)
    return sum(taps[:, j] * padded[j:j + u.shape[0]] for j in range(n))


def input_conv(x, taps):
    """what a mixer reads: the row and the convolution of the rows up to it"""
    return x + causal_conv(x, taps)


# ------------------------------------------------------------------------------------------------ rotation
def base_frequencies(rot):
    i = torch.arange(int(rot["dims"]) // 2, dtype=F64)
    return float(rot["base"]) ** (-2.0 * i / int(rot["dims"]))


def banded_frequencies(rot):
    """Short wavelengths stay, long ones are stretched by the factor, in between by a share of both."""
    f = base_frequencies(rot)
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for x in f.tolist():
        length = 2 * math.pi / x
        if length < s["original"] / s["high"]:
            out.append(x)
        elif length > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
            out.append((1 - share) * x / s["factor"] + share * x)
    return torch.tensor(out, dtype=F64)


def linear_frequencies(rot):
    f = base_frequencies(rot)
    return f / float(rot["scaling"]["factor"]) if rot.get("scaling") else f


def turn(x, freq, interleaved):
    """x [T, heads, d]: the leading 2 * len(freq) dims turn by position * freq, in pairs (2i, 2i + 1) or (i, i + half)"""
    n = freq.numel()
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    a, b = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    out[..., a] = x[..., a] * c - x[..., b] * s
    out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def visible(T, chunk):
    """[T, T] bool: row i sees row j <= i, with a chunk length only of its own chunk (counted from position 0)"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i // chunk == j // chunk) if chunk else ok


def sink_softmax(score, sink):
    """score [H, T, T]; sink [H] joins every row's denominator once"""
    s = torch.cat([score, sink[:, None, None].expand(-1, score.shape[1], 1)], -1)
    return torch.softmax(s, -1)[..., :-1]


def attend(q, k, v, scale, seen, sink):
    H, G = q.shape[1], k.shape[1]
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    score = torch.einsum("ihd,jhd->hij", q, kk) * scale
    p = sink_softmax(score.masked_fill(~seen, -math.inf), sink)
    return torch.einsum("hij,jhv->ihv", p, vv)


def chunked_attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    # one root mean square over all heads of q, and one over all of k
    q = (unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    f = banded_frequencies(m["rot"])
    q, k = turn(q, f, True), turn(k, f, True)
    o = attend(q, k, v, m["scale"], visible(T, m["mask"]["size"]), w[p + "sink"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


def gated_attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = lambda n: h @ w[p + n].T + w[p + n + ".b"]
    q = unit_rms(proj("q").view(T, H, d), eps) * w[p + "q.norm"]
    k = unit_rms(proj("k").view(T, G, d), eps) * w[p + "k.norm"]
    f = linear_frequencies(m["rot"])
    q, k = turn(q, f, False), turn(k, f, False)
    o = attend(q, k, proj("v").view(T, G, dv), m["scale"], visible(T, 0), w[p + "sink"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ the delta rule
def delta_step(S, q, k, v, g, beta):
    """One token of all heads: S [H, d, dv], q, k [H, d], v [H, dv], g, beta [H].  The read-out sees the write."""
    S = g[:, None, None] * S
    u = beta[:, None] * (v - torch.einsum("hdv,hd->hv", S, k))
    S = S + k[:, :, None] * u[:, None, :]
    return S, torch.einsum("hdv,hd->hv", S, q)


def gated_delta(h, w, p, m, eps, unit_eps=1e-6):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mixed = lambda n: silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    q = (unit_length(mixed("q").view(T, G, d), unit_eps) * d ** -0.5).repeat_interleave(H // G, 1)
    k = unit_length(mixed("k").view(T, G, d), unit_eps).repeat_interleave(H // G, 1)
    v = mixed("v").view(T, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    S, o = torch.zeros(H, d, dv, dtype=F64), torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        S, o[t] = delta_step(S, q[t], k[t], v[t], g[t], beta[t])
    o = unit_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def two_mixers(h, w, p, m, eps):
    return m["left_scale"] * gated_attention(h, w, p + "left.", m["left"], eps) \
        + m["right_scale"] * gated_delta(h, w, p + "right.", m["right"], eps)


# ------------------------------------------------------------------------------------------------ experts
def expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, w, p, f, forced=None):
    """(chosen experts [T, top], their scores): sigmoids as they are"""
    s = torch.sigmoid(h @ w[p + "router"].T)
    ids = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :f["router"]["top"]] if forced is None else forced.long()
    return ids, s.gather(1, ids)


def experts(h, w, p, f, forced=None):
    """The score multiplies what the expert reads.  Returns (rows, the router's own or the forced choice)."""
    ids, s = route(h, w, p, f, forced)
    out = torch.zeros_like(h)
    for e in ids.unique().tolist():
        rows, c = (ids == e).nonzero(as_tuple=True)
        out.index_add_(0, rows, expert(s[rows, c][:, None] * h[rows], *(w[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")), f["expert"]["limit"]))
    return out, ids


# ------------------------------------------------------------------------------------------------ the model
MIXERS = {"attention": chunked_attention, "delta": gated_delta, "parallel": two_mixers}


def forward(cfg, w, tokens, forced=None):
    """(logits [T, vocab], the rows behind every layer, the experts chosen by every layer or None) of one sequence.
    ``forced``: a list with the experts to use per layer ([T, top], or None for the router's own)."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    after, chosen = [], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](input_conv(x, w[p + "canon1"]), w, p + "mix.", layer["mixer"], eps)
        x = x + mult * one_number_norm(y, w[p + "norm1"], eps)
        ids = None
        if layer.get("mlp") is not None:
            y, ids = experts(x, w, p + "mlp.", layer["mlp"], forced[i] if forced is not None else None)
            x = x + mult * one_number_norm(y, w[p + "norm2"], eps)
        after.append(x)
        chosen.append(ids)
    logits = one_number_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(logits / cap), after, chosen
