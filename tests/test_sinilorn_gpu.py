"""Sinilorn on the GPU: each new kernel beside its plain reference or the plain function of its mechanism (sinks, keys
planted at window edges, page borders and far back, in prompts and in decoding, with forced splits; the recurrent unit
under every cut; residual streams; identity experts; biased and clamped gated products), and the whole model under every
cut, in long decoding and in generation, beside the plain implementation."""
import json
import math
import os
import random
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_sinilorn as P
import tiny_sinilorn as tiny
import traces
from flint_b200.cache.manager import CacheView, KVSpec
from flint_b200.engine.engine import Engine
from flint_b200.engine.model import load_model
from flint_b200.engine.replay import Replayer
from flint_b200.parts.base import Pending, RouterRequest
from flint_b200.sampling.params import SamplingParams
from kernel_refs import RefOps

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LENGTHS = (1, 2, 9, 37, 70, 130)


@pytest.fixture(scope="module")
def ops():
    from flint_b200.csrc.ops import get_ops
    return get_ops(DEV)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


# ------------------------------------------------------------------------------------------------ latent attention
def latent_cache(lengths, C, R, P_, dtype, seed=0):
    """Random latent rows of several requests in pages that lie in a shuffled order: (view on the device, rows per
    request as float64)."""
    rn, rnd = gen(seed), random.Random(seed)
    row_w = -(-(C + R) // 8) * 8
    n_pages = sum(-(-n // P_) for n in lengths) + 3
    order = list(range(n_pages))
    rnd.shuffle(order)
    k = torch.zeros(n_pages, 1, P_, row_w, dtype=dtype)
    bt = torch.full((len(lengths), max(-(-n // P_) for n in lengths) + 1), -1, dtype=torch.int32)
    dense = []
    for s, n in enumerate(lengths):
        rows = rn(n, C + R).to(dtype)
        for lp in range(-(-n // P_)):
            bt[s, lp] = order.pop()
            m = min(P_, n - lp * P_)
            k[bt[s, lp], 0, :m, :C + R] = rows[lp * P_:lp * P_ + m]
        dense.append(rows.double())
    view = CacheView(k.to(DEV), torch.zeros(n_pages, 1, P_, 0, dtype=dtype, device=DEV), bt.to(DEV), P_, KVSpec(1, row_w, 0, 0))
    return view, dense


def dense_attention(qa, dense, pos, slot, C, scale, window, sinks):
    out = torch.zeros(qa.shape[0], qa.shape[1], C, dtype=F64)
    for t in range(qa.shape[0]):
        lo = max(0, int(pos[t]) + 1 - window) if window else 0
        k = dense[int(slot[t])][lo:int(pos[t]) + 1]
        s = torch.cat([(qa[t].double() @ k.T) * scale, sinks.double()[:, None]], 1)
        out[t] = torch.softmax(s, -1)[:, :-1] @ k[:, :C]
    return out


def step_of(pos, slot, n_entries):
    pos = torch.as_tensor(pos, dtype=torch.int32, device=DEV)
    return SimpleNamespace(pos=pos, slot=torch.as_tensor(slot, dtype=torch.int32, device=DEV), max_kv_len=int(pos.max()) + 1,
                           entries=[None] * n_entries, n_tokens=pos.numel(), status=torch.zeros(1, dtype=torch.int32, device=DEV))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,R,H", [(40, 8, 5), (20, 6, 1), (104, 24, 7), (256, 64, 33)])
@pytest.mark.parametrize("window", [0, 1, 7, 64, 77, 200])
def test_latent_attention_with_sinks_finds_planted_keys(ops, dtype, C, R, H, window):
    """Single rows whose query points at one key (the row's own, the window's first, the one that has just left it, page
    borders, the first token), with sinks from negligible to dominant: a key too many or too few, or a sink that is
    scaled, left out or counted once per split, shows at once."""
    P_, lengths = 16, [333, 150]
    view, dense = latent_cache(lengths, C, R, P_, dtype, seed=C + window)
    rows = []
    for s, n in enumerate(lengths):
        for p in sorted({n - 1, n // 2, 2 * P_, 2 * P_ - 1, max(window - 1, 0), window, window + 1, 1, 0}):
            if p < n:
                for j in sorted({p, p - 1, p - window + 1, p - window, (p // P_) * P_, (p // P_) * P_ - 1, 0, 1, p // 3}):
                    if 0 <= j <= p:
                        rows.append((s, p, j))
    rn = gen(H + window)
    qa = 0.3 * rn(len(rows), H, C + R).double()
    for t, (s, p, j) in enumerate(rows):
        aim = dense[s][j]
        qa[t, t % H] += 14.0 * aim / aim.norm() ** 2 / 0.5
    qa = qa.to(dtype)
    sinks = torch.linspace(-30.0, 12.0, H) if H > 1 else torch.tensor([3.0])
    pos, slot = [p for _, p, _ in rows], [s for s, _, _ in rows]
    want = dense_attention(qa, dense, pos, slot, C, 0.5, window, sinks)
    span = min(max(pos) + 1, window) if window else max(pos) + 1
    for kernel in ("simt",) if dtype == torch.float32 else ("simt", "mma"):
        for splits in (None, (64, -(-span // 64)), (32, -(-span // 32))):
            out = torch.zeros(len(rows), H, C, dtype=dtype, device=DEV)
            ops.latent_attention(qa.to(DEV), view, step_of(pos, slot, len(rows)), out, H, C, window, 0.5, splits=splits, kernel=kernel,
                                 sinks=sinks.to(DEV))
            err = (out.cpu().double() - want).abs().amax((1, 2))
            assert err.max().item() < (3e-5 if dtype == torch.float32 else 4e-2), (kernel, splits, rows[int(err.argmax())], err.max().item())


@pytest.mark.parametrize("C,R,H", [(104, 24, 7), (48, 16, 1), (24, 8, 3), (512, 64, 16), (128, 32, 32)])
@pytest.mark.parametrize("window", [0, 5, 64, 77, 128, 130])
def test_latent_attention_windows_over_tiles_of_tokens(ops, C, R, H, window):
    """Portions of prompts on the tensor cores: a block's tokens see a window each, so between them more keys than one
    window (a window of exactly a key tile, one more, one less than a multiple)."""
    P_, lengths = 16, [333, 150]
    view, dense = latent_cache(lengths, C, R, P_, torch.bfloat16, seed=C + window + 1)
    portions = [(0, 0, 150), (1, 0, 64), (0, 150, 17), (1, 64, 2), (0, 167, 166), (1, 66, 84)]
    pos = [p0 + i for _, p0, c in portions for i in range(c)]
    slot = [s for s, _, c in portions for _ in range(c)]
    rn = gen(H)
    qa = (rn(len(pos), H, C + R) * (2.0 / math.sqrt(C + R))).double()
    for t in range(len(pos)):            # the key at the window's far edge, and the one just outside, stand out in turn
        j = pos[t] - window + (1 if t % 2 else 0) if window else pos[t] // 5
        if 0 <= j <= pos[t]:
            aim = dense[slot[t]][j]
            qa[t, t % H] += 9.0 * aim / aim.norm() ** 2
    qa = qa.to(torch.bfloat16)
    sinks = 2.0 * gen(3)(H)
    want = dense_attention(qa, dense, pos, slot, C, 1.0, window, sinks)
    for kernel in ("mma", "simt"):
        out = torch.zeros(len(pos), H, C, dtype=torch.bfloat16, device=DEV)
        ops.latent_attention(qa.to(DEV), view, step_of(pos, slot, len(portions)), out, H, C, window, 1.0, kernel=kernel, sinks=sinks.to(DEV))
        err = (out.cpu().double() - want).abs().amax((1, 2))
        assert err.max().item() < 4e-2, (kernel, int(err.argmax()), pos[int(err.argmax())], err.max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [3, 200])
@pytest.mark.parametrize("Q,C,R,rot,H,D,S", [(24, 16, 8, 8, 3, 8, 3), (37, 11, 6, 4, 2, 5, 1), (1536, 512, 64, 64, 4, 128, 9), (5, 20, 2, 2, 1, 0, 2)])
def test_the_latents_on_their_way_in(ops, dtype, T, Q, C, R, rot, H, D, S):
    """The query latent's norm, the cached row, and the queries' rotation, from partial sums, for few rows (several
    blocks a row) and many, with rows of whole 16-byte units and not."""
    rn, P_ = gen(Q + T), 16
    W = Q + C + R + 13
    proj, q_proj = rn(S, T, W), rn(S, T, H * (D + R))
    qw, kw = 1 + 0.1 * rn(Q), 1 + 0.1 * rn(C)
    ang = torch.arange(260, dtype=F64)[:, None] * 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)[None, :]
    cos, sin = (1.1 * torch.cos(ang)).float(), (1.1 * torch.sin(ang)).float()
    pos = torch.tensor([(7 * t) % 16 + 16 * (t // 16) for t in range(T)], dtype=torch.int32)
    slot = torch.zeros(T, dtype=torch.int32)
    row_w = -(-(C + R) // 8) * 8
    res = []
    for device, o, dt in (("cpu", RefOps(F64), F64), (DEV, ops, dtype)):
        mv = lambda t: t.to(device)
        n = -(-260 // P_)
        view = CacheView(torch.full((n, 1, P_, row_w), 3.0, dtype=dt, device=device), None, torch.arange(n, dtype=torch.int32, device=device)[None],
                         P_, KVSpec(1, row_w, 0, 0))
        st = torch.zeros(1, dtype=torch.int32, device=device)
        c_q, c_q2 = torch.zeros(T, Q, dtype=dt, device=device), torch.zeros(T, Q, dtype=dt, device=device)
        args = (mv(pos), mv(slot), mv(cos), mv(sin), rot, "half", mv(kw), 1e-5)
        o.latent_down(mv(proj), Q, mv(qw), *args, c_q, view, R, C, True, st)
        o.latent_down(mv(proj), Q, mv(qw), *args[:6], None, 1e-5, c_q2, view, R, C, False, st)
        qp, qa = torch.zeros(T, H, D, dtype=dt, device=device), torch.zeros(T, H, C + R, dtype=dt, device=device)
        o.latent_prepare(mv(q_proj), *args[:6], None, 1e-5, qp, qa, view, H, D, R, C, False, st)
        res.append([t.cpu().double() for t in (c_q, c_q2, view.k, qp, qa)])
        assert int(st) == 0
    tol = 3e-5 if dtype == torch.float32 else 5e-2
    for a, b in zip(*res):
        assert a.numel() == 0 or (a - b).abs().max() < tol * max(1.0, float(a.abs().max()) / 4), (a - b).abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 8, 16, 17, 150])
@pytest.mark.parametrize("H,N,K,S", [(3, 24, 40, 1), (7, 72, 104, 4), (2, 7, 13, 3), (5, 33, 16, 2)])
def test_products_per_head_with_a_gate(ops, dtype, T, H, N, K, S):
    rn = gen(T + N)
    x, w, proj = rn(T, H, K).to(dtype), (rn(H, N, K) / math.sqrt(K)).to(dtype), rn(S, T, 5 + H * N)
    want, out = torch.zeros(T, H, N, dtype=F64), torch.zeros(T, H, N, dtype=dtype, device=DEV)
    RefOps(F64).head_products(x, w, want, gate=proj[:, :, 5:])
    ops.head_products(x.to(DEV), w.to(DEV), out, gate=proj.to(DEV)[:, :, 5:])
    assert (out.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 3e-2)


# ------------------------------------------------------------------------------------------------ the linear recurrent unit
def unit_weights(W, B, taps, dtype, seed):
    rn = gen(seed)
    n = W // B
    lam = -7.0 + 7.5 * torch.rand(W, generator=torch.Generator().manual_seed(seed + 1))
    return dict(w_r=(2.0 * rn(B, n, n) / math.sqrt(n)).to(dtype), b_r=0.5 * rn(W), w_i=(2.0 * rn(B, n, n) / math.sqrt(n)).to(dtype),
                b_i=0.5 * rn(W), rate=-8.0 * torch.nn.functional.softplus(lam), conv_w=0.6 * rn(W, taps), conv_b=0.3 * rn(W), b_in=0.3 * rn(2 * W))


@pytest.mark.parametrize("kernel,dtype", [("simt", torch.float32), ("simt", torch.bfloat16), ("mma", torch.bfloat16)])
@pytest.mark.parametrize("W,B,T", [(64, 4, 70), (96, 3, 64), (40, 5, 1), (512, 2, 131), (36, 1, 65), (35, 5, 10)])
def test_the_block_diagonal_gates(ops, kernel, dtype, W, B, T):
    """Both kernels keep float32 accuracy: on the tensor cores u enters as three bfloat16 parts."""
    n = W // B
    if kernel == "mma" and n % 8:
        pytest.skip("blocks of a multiple of 8 channels only")
    w = unit_weights(W, B, 1, dtype, W + T)
    u = 3.0 * gen(T)(T, W)
    wa, wb = torch.zeros(T, W, dtype=F64), torch.zeros(T, W, dtype=F64)
    RefOps(F64).rglru_gates(u, w["w_r"], w["b_r"], w["w_i"], w["b_i"], w["rate"], wa, wb)
    a, b = torch.zeros(T, W, device=DEV), torch.zeros(T, W, device=DEV)
    d = {k: v.to(DEV) for k, v in w.items()}
    ops.rglru_gates(u.to(DEV), d["w_r"], d["b_r"], d["w_i"], d["b_i"], d["rate"], a, b, kernel=kernel)
    assert (a.cpu().double() - wa).abs().max() < 1e-5
    assert ((b.cpu().double() - wb).abs() / (1e-3 + wb.abs())).max() < 2e-3 and (b.cpu().double() - wb).abs().max() < 2e-5


@pytest.mark.parametrize("W", [40, 129, 512])
def test_the_scan_over_chunks(ops, W):
    """Requests of unequal length side by side (single rows, whole chunks, one row more and less), from carried state, in
    any order of slots; a slot nobody names stays as it was."""
    lengths = [1, 64, 65, 2, 200, 63, 128, 129, 7]
    rn = gen(W)
    T, n = sum(lengths), len(lengths)
    a = torch.exp(-torch.rand(T, W, generator=torch.Generator().manual_seed(W)) * torch.logspace(-3, 1, W))
    b, proj, state = rn(T, W), rn(T, 2 * W + 3), rn(n + 2, 3 * W)
    slots = [4, 0, 7, 9, 2, 5, 1, 10, 3]
    slot = torch.tensor([s for s, c in zip(slots, lengths) for _ in range(c)], dtype=torch.int32)
    starts = torch.tensor([sum(lengths[:i]) for i in range(n + 1)], dtype=torch.int32)
    st_ref, want = state.double(), torch.zeros(T, W, dtype=F64)
    RefOps(F64).rglru_scan(a, b, proj[:, :W], slot, starts, n, max(lengths), st_ref, want)
    for dt in (torch.float32, torch.bfloat16):
        st, out = state.to(DEV), torch.zeros(T, W, dtype=dt, device=DEV)
        ops.rglru_scan(a.to(DEV), b.to(DEV), proj.to(DEV)[:, :W], slot.to(DEV), starts.to(DEV), n, max(lengths), st, out)
        scale = float(want.abs().max())
        assert (out.cpu().double() - want).abs().max() < (2e-6 if dt == torch.float32 else 1e-2) * scale
        assert (st.cpu().double() - st_ref).abs().max() < 2e-6 * scale
        assert torch.equal(st.cpu()[[6, 8]], state[[6, 8]]) and torch.equal(st.cpu()[:, W:], state[:, W:])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,B,taps", [(64, 4, 4), (40, 5, 3), (36, 1, 1), (35, 5, 2), (320, 1, 6), (512, 2, 4)])
def test_the_recurrent_unit_under_every_cut(ops, dtype, W, B, taps):
    """Convolution, gates and recurrence over whole prompts, portions and single tokens (one launch), in slots that an
    earlier request left, beside the plain functions over the whole sequence: every cut gives the same numbers."""
    w = unit_weights(W, B, taps, dtype, W + taps)
    d = {k: v.to(DEV) for k, v in w.items()}
    lens = {0: 150, 1: 37}
    rn = gen(W)
    x = {s: rn(n, 2 * W) for s, n in lens.items()}              # what the projection leaves, without its biases
    want = {}
    for s, n in lens.items():
        z = (x[s] + w["b_in"]).double()
        u = P.causal_conv(z[:, W:], w["conv_w"].double(), w["conv_b"].double())
        r, i = (P.block_gate(u, w[k].double(), w[c].double().view(B, -1)) for k, c in (("w_r", "b_r"), ("w_i", "b_i")))
        a = torch.exp(w["rate"].double() * r)
        S, out = torch.zeros(W, dtype=F64), torch.zeros(n, W, dtype=F64)
        for t in range(n):
            S = a[t] * S + torch.sqrt(1 - a[t] * a[t]) * i[t] * u[t]
            out[t] = S
        want[s] = out * P.gelu_tanh(z[:, :W])
    for cut in ((150,), (3, 2, 1, 1, 64, 5, 2, 200), (1,), (2,), (130, 1, 1, 2, 1)):
        state = 5.0 * gen(9)(3, W * (1 + taps)).to(DEV)             # what an earlier request left
        state[:2] = 0                                              # admission zeroes a slot
        idle = state[2].clone()
        done, got, k = {0: 0, 1: 0}, {0: [], 1: []}, 0
        while any(done[s] < lens[s] for s in lens):
            portions = []
            for s in lens:
                c = min(cut[k % len(cut)], lens[s] - done[s])
                if c > 0:
                    portions.append((s, done[s], c))
            k += 1
            pos = torch.tensor([p + i for _, p, c in portions for i in range(c)], dtype=torch.int32, device=DEV)
            slot = torch.tensor([s for s, _, c in portions for _ in range(c)], dtype=torch.int32, device=DEV)
            rows = torch.cat([x[s][p:p + c] for s, p, c in portions]).to(DEV)
            T, n = pos.numel(), len(portions)
            out = torch.zeros(T, W, device=DEV)
            if T == n:
                parts = torch.stack([0.25 * rows, 0.5 * rows, 0.25 * rows])
                ops.rglru_step(parts, d["b_in"], d["conv_w"], d["conv_b"], d["w_r"], d["b_r"], d["w_i"], d["b_i"], d["rate"], pos, slot,
                               state, out)
            else:
                proj, u, a, b = rows + d["b_in"], *(torch.zeros(T, W, device=DEV) for _ in range(3))
                starts = torch.tensor([sum(c for _, _, c in portions[:i]) for i in range(n + 1)], dtype=torch.int32, device=DEV)
                ops.short_conv(proj, W, d["conv_w"], d["conv_b"], "none", pos, slot, state[:, W:], u, ring_rows=taps)
                ops.rglru_gates(u, d["w_r"], d["b_r"], d["w_i"], d["b_i"], d["rate"], a, b)
                ops.rglru_scan(a, b, proj[:, :W], slot, starts, n, max(c for _, _, c in portions), state[:, :W], out)
            o = 0
            for s, p, c in portions:
                got[s].append(out[o:o + c].cpu())
                done[s] += c
                o += c
        for s in lens:
            err = (torch.cat(got[s]).double() - want[s]).abs().max().item()
            assert err < 2e-5 * max(1.0, float(want[s].abs().max())), (cut, s, err)
        assert torch.equal(state[2], idle)


@pytest.mark.parametrize("T", [1, 7, 9])
def test_single_tokens_of_many_requests(ops, T):
    """More tokens than a block of the single-token kernel takes, positions before and after the convolution is filled."""
    W, B, taps = 96, 3, 4
    w = unit_weights(W, B, taps, torch.bfloat16, T)
    proj, state = gen(T)(2, T, 2 * W), gen(T + 1)(T + 3, W * (1 + taps))
    pos = torch.tensor([(0, 1, 2, 3, 4, 100, 5, 7, 1023)[t] for t in range(T)], dtype=torch.int32)
    slot = torch.tensor([T + 1 - t for t in range(T)], dtype=torch.int32)
    st_ref, want = state.double(), torch.zeros(T, W, dtype=F64)
    names = ("b_in", "conv_w", "conv_b", "w_r", "b_r", "w_i", "b_i", "rate")
    RefOps(F64).rglru_step(proj, *(w[k] for k in names), pos, slot, st_ref, want)
    st, out = state.to(DEV), torch.zeros(T, W, device=DEV)
    ops.rglru_step(proj.to(DEV), *(w[k].to(DEV) for k in names), pos.to(DEV), slot.to(DEV), st, out)
    assert (out.cpu().double() - want).abs().max() < 2e-5 and (st.cpu().double() - st_ref).abs().max() < 2e-5


# ------------------------------------------------------------------------------------------------ residual streams
def pending_case(rn, T, W, S, which):
    p = Pending(mix=0.5 * rn(S, S), spread=rn(S))
    if "partials" in which:
        p.partials = rn(3, T, W)
    if "bias" in which:
        p.bias = rn(W)
    if "rows" in which:
        k = 3
        p.y, p.gates = rn((k + 1) * T, W), torch.rand(T, k, generator=torch.Generator().manual_seed(T))
        p.row_of = torch.randint(0, (k + 1) * T, (T, k), generator=torch.Generator().manual_seed(W)).to(torch.int32)
    return p


def pend_on(p, device):
    return Pending(**{k: (v.to(device) if isinstance(v, torch.Tensor) else v) for k, v in vars(p).items()})


@pytest.mark.parametrize("S", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("T,W", [(1, 208), (8, 2048), (16, 1024), (300, 200), (2048, 512), (5, 8192), (40, 37)])
def test_streams_are_mixed_and_normed(ops, S, T, W):
    """One kernel for the mixing of what is pending and the norm of the streams' weighted sum: a block a row, a cluster a
    row, many rows, widths and numbers of streams that go to the separate kernels; the additions alone; the final
    norm's row list, which leaves the streams in memory as they are."""
    rn = gen(S * T + W)
    x, gamma, gather = rn(T, S, W), 1 + 0.1 * rn(W), rn(S)
    ref = RefOps(F64)
    index = torch.tensor(sorted({0, T // 2, T - 1}), dtype=torch.int32)
    for which in ("", "partials", "partials bias", "rows", "partials bias rows"):
        pend = pending_case(rn, T, W, S, which) if which else None
        for mode, rows in (("layer", None), ("rms", None), ("layer", index), ("none", None)):
            if mode == "none" and pend is None:
                continue
            a, b = x.double(), x.to(DEV)
            n = rows.numel() if rows is not None else T
            wf, of, ob = torch.zeros(n, W), torch.zeros(n, W, device=DEV), torch.zeros(n, W, dtype=torch.bfloat16, device=DEV)
            kw = dict(out_f32=wf, row_index=rows) if mode != "none" else {}
            kd = dict(out_f32=of, out_bf16=ob, row_index=rows.to(DEV) if rows is not None else None) if mode != "none" else {}
            gm = gamma if mode != "none" else None
            m = mode if mode != "none" else "layer"
            ref.row_norm(a, gm, None, 1e-5, m, pending=pend, gather=gather, **kw)
            ops.row_norm(b, gm.to(DEV) if gm is not None else None, None, 1e-5, m, pending=pend_on(pend, DEV) if pend is not None else None,
                         gather=gather.to(DEV), **kd)
            assert (b.cpu().double() - a).abs().max() < 3e-5, (which, mode)
            if mode != "none":
                assert (of.cpu() - wf).abs().max() < 1e-4 and (ob.float().cpu() - wf).abs().max() < 4e-2, (which, mode)
            if rows is not None:
                assert torch.equal(b.cpu(), x)


@pytest.mark.parametrize("S,T,W", [(2, 1, 208), (4, 8, 2048), (3, 300, 200), (6, 40, 72), (4, 2048, 256), (2, 9, 38)])
@pytest.mark.parametrize("E,top", [(13, 3), (80, 6), (5, 1)])
def test_the_corrected_softmax_router_rides_on_the_streams_norm(ops, S, T, W, E, top):
    """The choice is exactly the rule applied to the logits the kernel reports, and those agree with the plain product;
    the weights are the scores without the correction."""
    rn = gen(S + T + E)
    x, gamma, gather, pend = rn(T, S, W), 1 + 0.1 * rn(W), rn(S), pending_case(rn, T, W, S, "partials")
    wr, corr = (2.5 * rn(E, W) / math.sqrt(W)).to(torch.bfloat16), 0.15 * rn(E)
    y = torch.zeros(3 * T, W, device=DEV)
    req = RouterRequest(wr.to(DEV), 0.0, torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV),
                        logits=torch.zeros(T, E, device=DEV), top=top, rule="softmax_corrected", correction=corr.to(DEV), rows=y)
    ops.row_norm(x.to(DEV), gamma.to(DEV), None, 1e-5, "layer", out_f32=y[2 * T:], pending=pend_on(pend, DEV), gather=gather.to(DEV), router=req)
    a, normed = x.double(), torch.zeros(T, W, dtype=torch.float32)
    RefOps(F64).row_norm(a, gamma, None, 1e-5, "layer", out_f32=normed, pending=pend, gather=gather)
    assert (y[2 * T:].cpu() - normed).abs().max() < 1e-4
    assert (req.logits.cpu().double() - normed.double() @ wr.double().T).abs().max() < 5e-4
    s = torch.softmax(req.logits.cpu().double(), -1)
    ids = torch.sort(s + corr.double(), dim=-1, descending=True, stable=True).indices[:, :top]
    same = (ids == req.expert_ids.cpu().long()).all(-1)
    assert int((~same).sum()) <= max(1, T // 200)               # float32 scores against float64 ones: a tie at most
    g = s.gather(1, ids)
    assert (req.gates.cpu().double() - g / g.sum(-1, keepdim=True))[same].abs().max() < 1e-5


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,E,identity,top", [(1, 2, 2, 3), (8, 10, 3, 4), (60, 3, 5, 4), (64, 4, 4, 4), (65, 4, 4, 4), (500, 16, 4, 2), (40, 1, 6, 2)])
@pytest.mark.parametrize("kind", ["drawn", "all identity", "no identity"])
def test_identity_experts_take_no_rows_of_the_plan(ops, T, E, identity, top, kind):
    if (kind == "all identity" and identity < top) or (kind == "no identity" and E < top):
        pytest.skip("too few of a kind")
    g = torch.Generator().manual_seed(T + E)
    lo, hi = (E, E + identity) if kind == "all identity" else (0, E) if kind == "no identity" else (0, E + identity)
    ids = torch.stack([lo + torch.randperm(hi - lo, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    x = torch.randn(T, 24, generator=g)
    plan, xs = ops.moe_dispatch(ids.to(DEV), E, 16, x.to(DEV))
    off, row_of, token_of = plan.offsets.cpu(), plan.row_of.cpu().long(), plan.token_of.cpu().long()
    live = int((ids < E).sum())
    assert int(off[E]) == live and torch.equal(plan.counts.cpu().long(), torch.bincount(ids[ids < E].long(), minlength=E)[:E])
    assert int(plan.n_tiles) == int(sum(-(-int(c) // 16) for c in plan.counts.cpu()))
    assert bool((token_of[live:] == -1).all())
    seen = set()
    for t in range(T):
        for c in range(top):
            e, r = int(ids[t, c]), int(row_of[t, c])
            if e >= E:
                assert r == top * T + t
            else:
                assert off[e] <= r < off[e + 1] and int(token_of[r]) == t and torch.equal(xs[r].cpu(), x[t])
                seen.add(r)
    assert len(seen) == live


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M", [1, 8, 100, 130, 300])
@pytest.mark.parametrize("N,K", [(40, 64), (112, 208), (23, 40), (17, 21)])
def test_gated_products_with_biases_and_clamps(ops, dtype, M, N, K):
    """Dense: biases of gate and up before the activation, plain and clamped; few rows (partial sums and an activation
    kernel) and many (the tile's epilogue)."""
    rn = gen(M + N)
    x, wg, wu = rn(M, K).to(dtype), (2 * rn(N, K) / math.sqrt(K)).to(dtype), (2 * rn(N, K) / math.sqrt(K)).to(dtype)
    bg, bu = rn(N), rn(N)
    w, b = ops.pair_gate_up(wg.to(DEV), wu.to(DEV)).contiguous(), ops.pair_gate_up(bg[:, None].to(DEV), bu[:, None].to(DEV)).reshape(-1).contiguous()
    ref = RefOps(F64)
    wr, br = ref.pair_gate_up(wg, wu), torch.cat([bg, bu])
    for act, params in (("silu", None), ("swish_clamped", (1.702, 1.5)), ("gelu_pytorch_tanh", None)):
        for bias in (False, True):
            want, out = torch.zeros(M, N, dtype=F64), torch.zeros(M, N, dtype=dtype, device=DEV)
            ref.gated_gemm(x, wr, want, act, act_params=params, bias=br if bias else None)
            ops.gated_gemm(x.to(DEV), w, out, act, act_params=params, bias=b if bias else None)
            assert (out.cpu().double() - want).abs().max() < (3e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want.abs().max())), (act, bias)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,identity,top,N,K", [(1, 4, 4, 2, 32, 64), (1, 2, 6, 4, 16, 64), (7, 10, 3, 4, 112, 208), (200, 10, 3, 4, 112, 208), (90, 3, 2, 3, 13, 40),
                                                   (300, 2, 1, 2, 20, 36), (300, 2, 1, 2, 20, 40)])
def test_a_mixture_with_identity_experts_beside_the_plain_one(ops, dtype, T, E, identity, top, N, K):
    """The whole part, from the normalised rows to the pending rows, beside the plain mixture following its choices; also
    when no expert with weights is chosen at all."""
    from flint_b200.parts.base import BuildContext
    from flint_b200.parts.ffn import GroupedTopKMoE
    rn = gen(T + E)
    for push in (0.0, 50.0):                                # 50: only identity experts are chosen
        part = GroupedTopKMoE({"hidden_size": K, "intermediate_size": N, "num_experts": E, "identity": identity, "top": min(top, identity) if push else top,
                               "correction": True, "act": "swish_clamped", "act_slope": 1.702, "act_limit": 1.2},
                              BuildContext(ops, torch.device(DEV), "bfloat16" if dtype == torch.bfloat16 else "float32"))
        w = {n: (rn(*s.shape) * (2.0 / math.sqrt(s.shape[-1]) if len(s.shape) > 1 else 0.1)).to(dtype if len(s.shape) > 1 else torch.float32)
             for n, s in part.weights().items()}
        w["correction"][E:] += push
        part.load({n: t.to(DEV) for n, t in w.items()})
        h = rn(T, K).to(dtype)
        step = SimpleNamespace(record={})
        x = {dtype: h.to(DEV), torch.float32: h.float().to(DEV)}
        pend = part.forward(x, None, step)
        out = torch.zeros(T, K, device=DEV)
        ops.moe_combine(out, pend.y, pend.row_of, pend.gates)
        ids = step.record["experts"][0].cpu()
        if push:
            assert bool((ids >= E).all())
        f = {"router": {"experts": E, "identity": identity, "top": part.top}, "expert": {"ff": N, "limit": 1.2}}
        want, own = P.moe(h.double(), {"m." + n: t.double() for n, t in w.items()}, "m.", f, forced=ids)
        assert (out.cpu().double() - want).abs().max() < (5e-5 if dtype == torch.float32 else 3e-2) * max(1.0, float(want.abs().max()))
        _, own = P.moe(h.double(), {"m." + n: t.double() for n, t in w.items()}, "m.", f)
        assert int((own.sort(-1).values != ids.long().sort(-1).values).any(-1).sum()) <= 1


def test_the_small_changes_to_shared_kernels(ops):
    rn = gen(4)
    # embedded rows written once per stream
    table, ids = rn(11, 20).to(torch.bfloat16), torch.tensor([3, 0, 10], dtype=torch.int32)
    out = torch.zeros(3, 4, 20, device=DEV)
    ops.embed(ids.to(DEV), table.to(DEV), out, copies=4)
    assert torch.equal(out.cpu(), table[ids.long()].float()[:, None].expand(-1, 4, -1))
    # the convolution over many rows in 16-byte units gives the bits of the row-by-row kernel
    for C, taps in ((64, 4), (512, 2), (516, 8), (64, 1)):
        T = 200
        u, w, b = rn(T, C + 8).to(DEV), rn(C, taps).to(DEV), rn(C).to(DEV)
        pos = torch.tensor(list(range(3, 133)) + list(range(70)), dtype=torch.int32, device=DEV)
        slot = torch.tensor([1] * 130 + [0] * 70, dtype=torch.int32, device=DEV)
        state = rn(2, taps * C).to(DEV)
        y = torch.zeros(T, C, device=DEV)
        s1 = state.clone()
        ops.short_conv(u, 4, w, b, "silu", pos, slot, s1, y, ring_rows=taps)
        one, s2 = torch.zeros(T, C, device=DEV), state.clone()
        for lo, hi in ((0, 100), (100, 130), (130, 200)):
            ops.short_conv(u[lo:hi], 4, w, b, "silu", pos[lo:hi].contiguous(), slot[lo:hi].contiguous(), s2, (o := torch.zeros(hi - lo, C, device=DEV)), ring_rows=taps)
            one[lo:hi] = o
        assert torch.equal(y, one)
        for sl, end in ((1, 133), (0, 70)):                   # the inputs that the next token's convolution reads
            for p in range(end - taps + 1, end):
                r = p % taps
                assert torch.equal(s1[sl, r * C:(r + 1) * C], s2[sl, r * C:(r + 1) * C])


# ------------------------------------------------------------------------------------------------ the whole model
@pytest.fixture(scope="module", params=["S1", "S2", "S3", "S4"])
def setup(request, tmp_path_factory):
    which = request.param
    cfg = tiny.CONFIGS[which]
    folder, w = tiny.write_model(tmp_path_factory.mktemp("sinilorn") / which, cfg, seed=3)
    reqs = traces.make_requests(cfg["vocab"], LENGTHS, seed=7)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    return which, cfg, folder, w, reqs, plain


def replay(folder, steps, dtype, page_size=64, record=None):
    rp = Replayer(folder, dtype=dtype, max_tokens=traces.max_tokens_needed(steps), page_size=page_size, max_requests=4, device=DEV)
    out, recs = {}, {}
    for s in steps:
        rec = dict(record, **({"rows_after": []} if "rows_after" in record else {})) if record is not None else None
        lg = rp.run_step(s["entries"], s["end"], record=rec)
        if lg is not None:
            out[s["step"]] = lg
        recs[s["step"]] = rec
        rp.model.cache.check()
    assert all(g.pages.pool.used_pages == 0 for g in rp.model.cache.groups)
    return out, recs, rp


def followed(cfg, w, reqs, folder, dtype):
    """The plain implementation run with the experts the engine chose for the whole prompts (in bfloat16 a near-tie of
    two choice scores may fall the other way), and how many (row, layer) choices differ from the plain router's own."""
    steps = traces.whole(reqs)
    _, recs, _ = replay(folder, steps, dtype, record={})
    routed = [i for i, l in enumerate(cfg["layers"]) if l["mlp"] and l["mlp"]["kind"] == "moe"]
    out, flips = {}, 0
    for s in steps:
        rid = s["entries"][0]["id"]
        forced = [None] * len(cfg["layers"])
        for k, i in enumerate(routed):
            forced[i] = recs[s["step"]]["experts"][k].cpu()
        own = P.forward(cfg, w, reqs[rid])[2]
        out[rid] = P.forward(cfg, w, reqs[rid], forced=forced)[0]
        flips += sum(int((own[i].sort(-1).values != forced[i].long().sort(-1).values).any(-1).sum()) for i in routed)
    return out, flips


def rel_err(got, want):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    c = want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / c.pow(2).mean(-1).sqrt().clamp(min=1e-6))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_matches_plain_under_every_cut(setup, dtype):
    which, cfg, folder, w, reqs, plain = setup
    if dtype == "bfloat16":
        base, flips = followed(cfg, w, reqs, folder, dtype)
        assert flips <= 0.1 * sum(LENGTHS) * len(cfg["layers"])
    else:
        base = plain
    limit = 1e-4 if dtype == "float32" else 8e-2
    cuts = {"whole": traces.whole, "tail": lambda r: traces.tail_decoded(r, tail=40), "portions": traces.portions,
            "twos": lambda r: traces.portions(r, sizes=(2, 2, 1, 2, 3, 128)), "mixed": lambda r: traces.mixed(r, seed=3)}
    for name, cut in cuts.items():
        steps = cut(reqs)
        out, _, rp = replay(folder, steps, dtype, page_size=16 if name == "mixed" else 64)
        exp = traces.expected_rows(steps, base)
        assert set(out) == set(exp)
        errs = torch.cat([rel_err(out[k], torch.stack(rows)) for k, rows in exp.items()])
        bad = int((errs > limit).sum())
        assert bad <= (0 if dtype == "float32" else 0.1 * len(errs)), f"{name}: {bad} of {len(errs)} rows, worst {float(errs.max()):.3g}"
        if name == "mixed":
            assert max(max(g.pages.pool.served) for g in rp.model.cache.groups) >= 2


def test_every_layer_leaves_what_the_plain_model_does(setup):
    which, cfg, folder, w, reqs, plain = setup
    _, recs, _ = replay(folder, traces.whole({"r4": reqs["r4"]}), "float32", record={"rows_after": []})
    after = P.forward(cfg, w, reqs["r4"])[1]
    for i, r in enumerate(recs[0]["rows_after"]):
        assert (r.cpu().double() - after[i]).abs().max() < 1e-4 * max(1.0, float(after[i].abs().max())), f"layer {i}"


def test_a_cut_changes_float32_logits_by_rounding_only(setup):
    which, cfg, folder, w, reqs, plain = setup
    one = {"r5": reqs["r5"]}
    a, _, _ = replay(folder, traces.whole(one), "float32")
    steps = traces.portions(one, sizes=(3, 2, 17, 64, 2, 1, 5))
    b, _, _ = replay(folder, steps, "float32", page_size=16)
    got = torch.cat([b[s["step"]] for s in steps if s["step"] in b])
    assert float(rel_err(got, a[0].double()).max()) < 3e-5


@pytest.mark.parametrize("seed", [11, 12, 13, 14, 15, 16, 17, 18, 19, 20])
def test_configurations_drawn_at_random(seed, tmp_path):
    cfg = tiny.random_config(seed)
    folder, w = tiny.write_model(tmp_path / "m", cfg, seed=seed)
    reqs = traces.make_requests(cfg["vocab"], (1, 2, 23, 50, 85, 170), seed=seed)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    for cut in (traces.whole, lambda r: traces.tail_decoded(r, tail=45), lambda r: traces.portions(r, sizes=(2, 3, 16, 1, 2, 64)),
                lambda r: traces.mixed(r, seed=seed)):
        steps = cut(reqs)
        out, _, _ = replay(folder, steps, "float32", page_size=16)
        exp = traces.expected_rows(steps, plain)
        errs = torch.cat([rel_err(out[k], torch.stack(rows)) for k, rows in exp.items()])
        assert float(errs.max()) < 1e-4, (cfg, float(errs.max()))


def test_long_decoding_token_by_token(setup):
    """Two requests decoded side by side, one token a step each, over several pages and past every window, after
    prompts of unequal length: the captured decode step is replayed many times, and the recurrent state and the
    convolution's inputs are carried through all of them."""
    which, cfg, folder, w, reqs, plain = setup
    a, b = reqs["r5"], reqs["r4"]
    rp = Replayer(folder, dtype="float32", max_tokens=512, page_size=16, max_requests=2, device=DEV)
    rp.run_step([{"id": "a", "tokens": a[:40], "want": []}, {"id": "b", "tokens": b[:3], "want": []}])
    worst = 0.0
    for i in range(66):
        out = rp.run_step([{"id": "a", "tokens": [a[40 + i]], "want": [0]}, {"id": "b", "tokens": [b[3 + i]], "want": [0]}])
        worst = max(worst, float(rel_err(out, torch.stack([plain["r5"][40 + i], plain["r4"][3 + i]])).max()))
    assert worst < 1e-4
    assert len(rp.model._graphs) >= 1


def test_greedy_generation_through_the_entry_point(setup):
    which, cfg, folder, w, reqs, plain = setup
    prompts = [reqs["r2"], reqs["r3"][:14], reqs["r0"]]
    expected = []
    for p in prompts:
        toks, out = list(p), []
        for _ in range(12):
            t = int(torch.argmax(P.forward(cfg, w, toks)[0][-1]))
            out.append(t)
            toks.append(t)
        expected.append(out)
    for n_pages in (16, 3):
        m = load_model(folder, dtype="float32", device=DEV, page_size=16, n_pages=n_pages, max_slots=4, max_step_tokens=24,
                       max_context=256)
        eng = Engine(m, SamplingParams.greedy(), prefill_chunk=16)
        assert eng.generate(prompts, 12) == expected
        assert all(g.pages.pool.used_pages == 0 for g in m.cache.groups) and m.cache.free_slots == 4
    assert eng.scheduler.preemptions > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_as_a_program(setup, tmp_path, dtype):
    """bin/trace_run in a process of its own, fed a mixed trace over standard input."""
    which, cfg, folder, w, reqs, plain = setup
    if which not in ("S1", "S2"):
        pytest.skip("two configurations are enough")
    steps = traces.mixed(reqs, seed=5)
    out_dir = tmp_path / "out"
    proc = subprocess.run([sys.executable, f"{REPO}/bin/trace_run", "--model", str(folder), "--dtype", dtype, "--out", str(out_dir),
                           "--max-tokens", str(traces.max_tokens_needed(steps))],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.split("\n") if l] == [f"done {s['step']}" for s in steps]
    exp = traces.expected_rows(steps, plain)
    errs = []
    for s in steps:
        f = out_dir / f"{s['step']}.f32"
        n = sum(len(e["want"]) for e in s["entries"])
        assert f.exists() == (n > 0)
        if n:
            got = torch.from_numpy(np.fromfile(f, dtype="<f4").reshape(n, cfg["vocab"]))
            errs.append(rel_err(got, torch.stack(exp[s["step"]])))
    errs = torch.cat(errs)
    if dtype == "float32":
        assert float(errs.max()) < 1e-4
    else:       # a near-tie of two choice scores may fall the other way at some rows
        assert float(errs.median()) < 5e-2


def test_chat_program_with_random_weights(tmp_path):
    """bin/flint_chat with ``--random-config FILE --seed N``, token ids in and out, greedy: the tokens of the folder
    that the random-weights mode writes for that configuration and seed, under the plain implementation."""
    from flint_b200.engine.loading import write_random_model
    from flint_b200.weights.safetensors_io import SafetensorsFile
    seed, cfg = 4, tiny.S4
    folder = write_random_model(tmp_path / "model", cfg, seed=seed)
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.read(n).double() for n in f.names()}
    prompt = [3, 50, 50, 7, 70, 0, 12, 13, 14, 15, 16]
    cfg_file = tmp_path / "only_config.json"
    cfg_file.write_text(json.dumps(cfg))
    proc = subprocess.run([sys.executable, f"{REPO}/bin/flint_chat", "--random-config", str(cfg_file), "--prompt", " ".join(map(str, prompt)),
                           "--max-tokens", "8", "--temperature", "0", "--seed", str(seed), "--dtype", "float32", "--ctx-size", "128"],
                          capture_output=True, text=True, timeout=600, env={**os.environ, "VERIFY_IDS": "1"})
    assert proc.returncode == 0, proc.stderr[-2000:]
    got = [int(x) for x in proc.stdout.split()]
    toks, want = list(prompt), []
    for _ in range(8):
        t = int(torch.argmax(P.forward(cfg, w, toks)[0][-1]))
        want.append(t)
        toks.append(t)
    assert got == want
