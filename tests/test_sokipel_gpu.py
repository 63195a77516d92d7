"""Sokipel on the GPU: each new kernel beside its plain reference or the plain function of its mechanism (the row kernel that
norms, adds, convolves and routes; single rows of attention on the tensor cores with keys planted at the edges of chunks and
windows, page borders and far back; the delta rule with a decay a head under every cut, single tokens in one launch; experts that
read rows times their scores), and the whole model under every cut, in long decoding and in generation, beside the plain
implementation."""
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

import plain_sokipel as P
import tiny_sokipel as tiny
import traces
from flint_b200.cache.manager import CacheView, KVSpec
from flint_b200.engine.engine import Engine
from flint_b200.engine.model import load_model
from flint_b200.engine.replay import Replayer
from flint_b200.parts.base import BuildContext, Pending, RouterRequest
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


def ints(x):
    return torch.as_tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------------ attention of single rows
def paged_keys(lengths, nkv, hd, vd, P_, dtype, seed):
    """Random keys and values of several requests in pages that lie in a shuffled order: (view on the device, keys and values
    per request as float64)."""
    rn, rnd = gen(seed), random.Random(seed)
    n_pages = sum(-(-n // P_) for n in lengths) + 3
    order = list(range(n_pages))
    rnd.shuffle(order)
    k, v = torch.zeros(n_pages, nkv, P_, hd, dtype=dtype), torch.zeros(n_pages, nkv, P_, vd, dtype=dtype)
    bt = torch.full((len(lengths), max(-(-n // P_) for n in lengths) + 1), -1, dtype=torch.int32)
    dense = []
    for s, n in enumerate(lengths):
        kk, vv = rn(n, nkv, hd).to(dtype), rn(n, nkv, vd).to(dtype)
        for lp in range(-(-n // P_)):
            bt[s, lp] = order.pop()
            m = min(P_, n - lp * P_)
            k[bt[s, lp], :, :m] = kk[lp * P_:lp * P_ + m].transpose(0, 1)
            v[bt[s, lp], :, :m] = vv[lp * P_:lp * P_ + m].transpose(0, 1)
        dense.append((kk.double(), vv.double()))
    return CacheView(k.to(DEV), v.to(DEV), bt.to(DEV), P_, KVSpec(nkv, hd, 0, vd)), dense


def dense_row(q, k, v, seen, sinks, scale):
    G = q.shape[0] // k.shape[1]
    out = torch.zeros(q.shape[0], v.shape[2], dtype=F64)
    for h in range(q.shape[0]):
        s = torch.cat([k[seen, h // G] @ q[h] * scale, sinks[h:h + 1]])
        out[h] = torch.softmax(s, 0)[:-1] @ v[seen, h // G]
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,hd,vd", [(4, 2, 32, 48), (6, 1, 48, 48), (20, 1, 64, 16), (8, 8, 128, 128), (6, 2, 20, 7), (33, 1, 16, 80)])
@pytest.mark.parametrize("mask", [{}, {"chunk": 1}, {"chunk": 17}, {"chunk": 64}, {"chunk": 100}, {"window": 37}, {"window": 70, "keep_first": 5}])
def test_single_rows_find_planted_keys(ops, dtype, nq, nkv, hd, vd, mask):
    """Rows whose query points at one key (the row's own, the chunk's or window's first, the one just outside, page borders, the
    first tokens, far back), with sinks from negligible to dominant; both kernels, any splits: a key too many or too few, or a
    sink that is scaled, left out or counted once per split, shows at once."""
    P_, lengths = 16, [333, 150]
    view, dense = paged_keys(lengths, nkv, hd, vd, P_, dtype, hd + vd)
    chunk, window, keep = mask.get("chunk", 0), mask.get("window", 0), mask.get("keep_first", 0)
    rows = []
    for s, n in enumerate(lengths):
        for p in sorted({n - 1, 2 * P_, 2 * P_ - 1, chunk, chunk - 1, 2 * chunk, window, window + keep, 1, 0}):
            if 0 <= p < n:
                lo = p // chunk * chunk if chunk else p + 1 - window if window else 0
                for j in sorted({p, p - 1, lo, lo - 1, (p // P_) * P_, (p // P_) * P_ - 1, 0, keep - 1, keep, p // 3}):
                    if 0 <= j <= p:
                        rows.append((s, p, j))
    if len(rows) > 60:
        rows = random.Random(1).sample(rows, 60)
    q = 0.3 * gen(nq)(len(rows), nq, hd).double()
    for t, (s, p, j) in enumerate(rows):
        for h in range(t % 3, nq, 3):
            aim = dense[s][0][j, h // (nq // nkv)]
            q[t, h] += 14.0 * aim / aim.norm() ** 2 / 0.5
    q = q.to(dtype)
    sinks = torch.linspace(-30.0, 12.0, nq) if nq > 1 else torch.tensor([3.0])
    want, spans = [], []
    for t, (s, p, j) in enumerate(rows):
        i = torch.arange(p + 1)
        seen = i[(i // chunk == p // chunk) if chunk else (((p - i) < window) | (i < keep)) if window else i >= 0]
        spans.append(len(seen))
        want.append(dense_row(q[t].double(), *dense[s], seen, sinks.double(), 0.5))
    want = torch.stack(want)
    step = SimpleNamespace(pos=ints([p for _, p, _ in rows]), slot=ints([s for s, _, _ in rows]), max_kv_len=max(p for _, p, _ in rows) + 1)
    mma_ok = ops.sink_attention_tiles_ok(dtype, dtype, hd, vd)
    span = min(step.max_kv_len, window + keep) if window else min(step.max_kv_len, chunk) if chunk else step.max_kv_len
    for kernel in ("simt", "mma") if mma_ok else ("simt",):
        for splits in (None, (64, -(-span // 64)), (span, 1), (24, -(-span // 24))):
            out = torch.zeros(len(rows), nq * vd, dtype=dtype, device=DEV)
            ops.sink_attention(q.reshape(len(rows), nq * hd).to(DEV), view, step, out, nq, nkv, hd, vd, window, keep, sinks.to(DEV), 0.5,
                               splits=splits, chunk=chunk, kernel=kernel)
            err = (out.cpu().double().view(len(rows), nq, vd) - want).abs().amax((1, 2))
            assert err.max().item() < (5e-5 if dtype == torch.float32 else 5e-2), (kernel, splits, rows[int(err.argmax())], err.max().item())


def test_rows_of_a_list_beside_tiles(ops):
    """Rows that lie in no tile are computed in their places, the others left alone; without sinks too."""
    nq, nkv, hd, vd = 4, 2, 32, 32
    view, dense = paged_keys([90, 40], nkv, hd, vd, 16, torch.bfloat16, 5)
    pos, slot = [89, 3, 39, 64], [0, 0, 1, 0]
    q = gen(2)(4, nq, hd).to(torch.bfloat16)
    step = SimpleNamespace(pos=ints(pos), slot=ints(slot), max_kv_len=90)
    for sinks in (None, torch.zeros(nq)):
        out = torch.full((4, nq * vd), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.sink_attention(q.reshape(4, -1).to(DEV), view, step, out, nq, nkv, hd, vd, 0, 0, sinks.to(DEV) if sinks is not None else None, 0.3,
                           rows=ints([3, 0]), chunk=50)
        assert bool((out[1:3] == 7.0).all())
        for t in (0, 3):
            lo = pos[t] // 50 * 50
            s = sinks.double() if sinks is not None else torch.full((nq,), -1e30, dtype=F64)
            want = dense_row(q[t].double(), *dense[slot[t]], torch.arange(lo, pos[t] + 1), s, 0.3)
            assert (out[t].cpu().double().view(nq, vd) - want).abs().max() < 2e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [3, 100])
@pytest.mark.parametrize("nq,nkv,hd,vd,rot,style,S", [(6, 2, 12, 7, 12, "interleaved", 3), (8, 2, 64, 32, 32, "half", 6), (16, 4, 128, 128, 128, "interleaved", 9)])
def test_projections_normed_and_rotated_from_partial_sums(ops, dtype, T, nq, nkv, hd, vd, rot, style, S):
    """q, k and v from partial sums and a bias, with norms per head and over the whole projection, beside the float64
    reference; few rows (several blocks a row) and many; then the gates, from partial sums too, on heads of any size."""
    rn, W = gen(T + hd), (nq + nkv) * hd + nkv * vd
    y, bias = rn(S, T, W + nq), rn(W)
    ang = torch.arange(120, dtype=F64)[:, None] * 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)[None, :]
    cos, sin = torch.cos(ang).float(), torch.sin(ang).float()
    pos, slot = torch.tensor([(7 * t) % 120 for t in range(T)], dtype=torch.int32), torch.zeros(T, dtype=torch.int32)
    if T > 50:
        pos = torch.arange(T, dtype=torch.int32)
    for whole in (False, True):
        qw, kw = (1 + 0.2 * rn(nq * hd), 1 + 0.2 * rn(nkv * hd)) if whole else (1 + 0.2 * rn(hd), 1 + 0.2 * rn(hd))
        res = []
        for device, o, dt in (("cpu", RefOps(F64), F64), (DEV, ops, dtype)):
            mv = lambda t: t.to(device)
            view = CacheView(torch.zeros(8, nkv, 16, hd, dtype=dt, device=device), torch.zeros(8, nkv, 16, vd, dtype=dt, device=device),
                             torch.arange(8, dtype=torch.int32, device=device)[None], 16, KVSpec(nkv, hd, 0, vd))
            q = torch.zeros(T, nq * hd, dtype=dt, device=device)
            st = torch.zeros(1, dtype=torch.int32, device=device)
            o.qk_norm_write(mv(y)[:, :, :W], mv(qw), mv(kw), 1e-5, mv(pos), mv(slot), mv(cos), mv(sin), rot, style, None, None, "half", q, view,
                            nq, nkv, hd, vd, st, whole=whole, bias=mv(bias))
            attn, out = mv(gen(3)(T, nq * vd)).to(dt), torch.zeros(T, nq * vd, dtype=dt, device=device)
            o.head_finish(attn, mv(pos), None, None, "half", mv(y)[:, :, W:], out, nq, vd)
            res.append([x.cpu().double() for x in (q, view.k, view.v, out)])
        for a, b in zip(*res):
            assert (a - b).abs().max() < (3e-5 if dtype == torch.float32 else 5e-2) * max(1.0, float(a.abs().max()) / 4)


# ------------------------------------------------------------------------------------------------ rows: norm, sum, convolution, router
def pending_case(rn, T, W, which):
    p = Pending()
    if "partials" in which:
        p.partials, p.bias = rn(3, T, W), rn(W) if "bias" in which else None
    if "branches" in which:
        p.branches = ((rn(5, T, W), rn(W), 0.7), (rn(1, T, W), None, -1.3))
    if "rows" in which:
        p.y, p.gates = rn(3 * T, W), torch.rand(T, 3, generator=torch.Generator().manual_seed(T))
        p.row_of = torch.randint(0, 3 * T, (T, 3), generator=torch.Generator().manual_seed(W)).to(torch.int32)
    if "norm" in which:
        p.gamma, p.eps = 1 + 0.1 * rn(W), 1e-2
    return p


def on(v, device):
    if isinstance(v, torch.Tensor):
        return v.to(device)
    return tuple(on(x, device) for x in v) if isinstance(v, tuple) else v


def pend_on(p, device):
    return Pending(**{k: on(v, device) for k, v in vars(p).items()})


@pytest.mark.parametrize("T,W", [(1, 208), (8, 2048), (16, 1024), (300, 200), (2048, 512), (5, 8192), (40, 37), (3, 16388)])
def test_rows_get_what_is_added_normed(ops, T, W):
    """A block a row, a cluster a row, many rows, widths that go to the separate kernels; products with scales, expert rows,
    with and without the norm; the copy in another type."""
    rn = gen(T + W)
    x = rn(T, W)
    for which in ("partials", "partials bias norm", "branches norm", "rows norm", "partials bias branches rows norm", "branches"):
        p = pending_case(rn, T, W, which)
        a, b = x.double(), x.to(DEV)
        RefOps(F64).row_post(a, p)
        for dt in (torch.bfloat16, torch.float32, None):
            b.copy_(x)
            out = torch.zeros(T, W, dtype=dt, device=DEV) if dt is not None else None
            ops.row_post(b, pend_on(p, DEV), out=out)
            scale = float(a.abs().max())
            assert (b.cpu().double() - a).abs().max() < 3e-6 * max(scale, 3.0), which
            if dt is not None:
                assert (out.cpu().double() - a).abs().max() < (3e-6 if dt == torch.float32 else 8e-3) * max(scale, 3.0), which
        c = x.to(DEV)                    # what a norm that cannot take it along does
        ops.apply_pending(c, pend_on(p, DEV))
        assert torch.equal(c, b) if p.alone else (c - b).abs().max() < 1e-5 * max(scale, 3.0)


@pytest.mark.parametrize("T,W", [(1, 208), (8, 2048), (300, 200), (2048, 256), (9, 38), (16, 1028)])
@pytest.mark.parametrize("E,top,gain", [(13, 3, 2.5), (70, 6, 2.5), (5, 1, 2.5), (40, 2, 12.0)])
def test_the_sigmoid_router_rides_on_the_sum(ops, T, W, E, top, gain):
    """The choice is exactly the rule applied to the logits the kernel reports, also where many scores round to 1 in float32,
    and those agree with the plain product."""
    rn = gen(T + E)
    x, p, wr = rn(T, W), pending_case(rn, T, W, "partials norm"), (gain * rn(E, W) / math.sqrt(W)).to(torch.bfloat16)
    req = RouterRequest(wr.to(DEV), 0.0, torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV),
                        logits=torch.zeros(T, E, device=DEV), top=top, rule="sigmoid", weights=torch.zeros(T, top, device=DEV))
    a, b = x.double(), x.to(DEV)
    RefOps(F64).row_post(a, p)
    ops.row_post(b, pend_on(p, DEV), router=req)
    assert (b.cpu().double() - a).abs().max() < 1e-4
    assert (req.logits.cpu().double() - a @ wr.double().T).abs().max() < 2e-4 * gain
    s = torch.sigmoid(req.logits.cpu().double())
    ids = torch.sort(req.logits.cpu(), dim=-1, descending=True, stable=True).indices[:, :top]
    same = (ids == req.expert_ids.cpu().long()).all(-1)
    assert bool(same.all())
    assert (req.gates.cpu().double() - s.gather(1, ids)).abs().max() < 1e-5 and bool((req.weights == 1).all())


@pytest.mark.parametrize("W,taps", [(64, 3), (37, 4), (1024, 2), (2048, 5), (40, 1), (72, 6)])
def test_the_input_convolution_under_every_cut(ops, W, taps):
    """Whole prompts, portions (few rows and many) and single tokens (together with the sum before them) over the same rows, in
    slots that an earlier request left: every cut gives the same numbers, and a slot nobody names stays as it was."""
    lens = {0: 150, 1: 37}
    rn, w = gen(W), 0.5 * gen(taps)(W, taps)
    x = {s: rn(n, W) for s, n in lens.items()}
    want = {s: P.input_conv(x[s].double(), w.double()) for s in lens}
    wd = w.to(DEV)
    for cut in ((150,), (3, 2, 1, 1, 64, 5, 2, 200), (1,), (2,), (130, 1, 1, 2, 1)):
        for dt in (torch.float32, torch.bfloat16):
            state = 5.0 * gen(9)(3, 4 + (taps - 1) * W + 8).to(DEV)
            state[:2] = 0
            idle = state[2].clone()
            ring = state[:, 4:]
            done, got, k = {0: 0, 1: 0}, {0: [], 1: []}, 0
            while any(done[s] < lens[s] for s in lens):
                portions = [(s, done[s], min(cut[k % len(cut)], lens[s] - done[s])) for s in lens if done[s] < lens[s]]
                k += 1
                pos, slot = ints([p + i for _, p, c in portions for i in range(c)]), ints([s for s, _, c in portions for _ in range(c)])
                rows = torch.cat([x[s][p:p + c] for s, p, c in portions]).to(DEV)
                out = torch.zeros(rows.shape, dtype=dt, device=DEV)
                if len(portions) == pos.numel():
                    half = (0.25 * rows).unsqueeze(0).expand(2, -1, -1).contiguous()
                    base = 0.5 * rows
                    ops.row_post(base, Pending(partials=half), out=out, conv=(wd, ring if taps > 1 else None, pos, slot))
                    assert (base - rows).abs().max() < 1e-6
                else:
                    ops.short_conv(rows, 0, wd, None, "plus_input", pos, slot, ring if taps > 1 else None, out)
                o = 0
                for s, p, c in portions:
                    got[s].append(out[o:o + c].cpu())
                    done[s] += c
                    o += c
            for s in lens:
                err = (torch.cat(got[s]).double() - want[s]).abs().max().item()
                assert err < (3e-6 if dt == torch.float32 else 1e-2) * float(want[s].abs().max()), (cut, s, err)
            assert torch.equal(state[2], idle)


# ------------------------------------------------------------------------------------------------ the delta rule with a decay a head
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,V,taps", [(2, 2, 12, 5, 3), (4, 2, 40, 6, 2), (4, 1, 32, 32, 4), (2, 1, 144, 24, 1), (16, 8, 128, 128, 4), (3, 3, 64, 68, 6),
                                          (2, 1, 256, 130, 2), (3, 1, 20, 260, 5)])
def test_the_delta_rule_under_every_cut(ops, dtype, H, G, D, V, taps):
    """From the projected columns to the gated heads over whole prompts, portions and single tokens (one launch), in slots
    that an earlier request left, beside the plain recurrence over the whole sequence."""
    rn = gen(D + V)
    C, N = 2 * G * D + H * V, 2 * G * D + 2 * H * V + 2 * H
    lens = {0: 70, 1: 23}
    proj = {s: rn(n, N) for s, n in lens.items()}
    conv_w, dt_bias, a_log, norm_w = 0.5 * rn(C, taps), -2.0 + rn(H), 0.5 * rn(H), 1 + 0.1 * rn(V)
    want = {}
    for s, n in lens.items():
        z = proj[s].double()
        y = P.silu(P.causal_conv(z[:, :C], conv_w.double()))
        q = (P.unit_length(y[:, :G * D].view(n, G, D), 1e-6) * D ** -0.5).repeat_interleave(H // G, 1)
        k = P.unit_length(y[:, G * D:2 * G * D].view(n, G, D), 1e-6).repeat_interleave(H // G, 1)
        v, beta = y[:, 2 * G * D:].view(n, H, V), torch.sigmoid(z[:, C:C + H])
        g = torch.exp(-torch.exp(a_log.double()) * P.softplus(z[:, C + H:C + 2 * H] + dt_bias.double()))
        S, o = torch.zeros(H, D, V, dtype=F64), torch.zeros(n, H, V, dtype=F64)
        for t in range(n):
            S, o[t] = P.delta_step(S, q[t], k[t], v[t], g[t], beta[t])
        want[s] = (P.unit_rms(o, 1e-5) * norm_w.double() * P.silu(z[:, C + 2 * H:]).view(n, H, V)).view(n, H * V)
    d = {n: t.to(DEV) for n, t in dict(conv_w=conv_w, dt_bias=dt_bias, a_log=a_log, norm_w=norm_w).items()}
    ring = taps if taps > 1 else 0
    for cut in ((70,), (3, 2, 1, 1, 33, 5, 2, 200), (1,), (40, 1, 1, 2, 1)):
        state = 5.0 * gen(9)(3, 3 + H * D * V + ring * C).to(DEV)[:, (0 if D % 4 == 0 and V % 4 == 0 else 3):]
        state[:2] = 0
        idle = state[2].clone()
        done, got, k = {0: 0, 1: 0}, {0: [], 1: []}, 0
        while any(done[s] < lens[s] for s in lens):
            portions = [(s, done[s], min(cut[k % len(cut)], lens[s] - done[s])) for s in lens if done[s] < lens[s]]
            k += 1
            pos, slot = ints([p + i for _, p, c in portions for i in range(c)]), ints([s for s, _, c in portions for _ in range(c)])
            rows = torch.cat([proj[s][p:p + c] for s, p, c in portions]).to(DEV)
            T, n = pos.numel(), len(portions)
            out = torch.zeros(T, H * V, dtype=dtype, device=DEV)
            if T == n:
                parts = torch.stack([0.25 * rows, 0.5 * rows, 0.25 * rows])
                ops.delta_token(parts, d["conv_w"], d["dt_bias"], d["a_log"], d["norm_w"], "silu", pos, slot, state, 1e-6, 1e-5, out, H, G, D, V)
            else:
                f = lambda *s: torch.zeros(*s, device=DEV)
                y, qk, decay, beta, o = f(T, C), f(T, 2 * G * D), f(T, H), f(T, H), f(T, H * V)
                starts = ints([sum(c for _, _, c in portions[:i]) for i in range(n + 1)])
                ops.short_conv(rows, 0, d["conv_w"], None, "silu", pos, slot, state[:, H * D * V:] if ring else None, y, ring_rows=ring or None)
                ops.delta_prepare(y, rows[:, C:C + H], rows[:, C + H:C + 2 * H], d["dt_bias"], d["a_log"], qk, decay, beta, H, G, D, 1e-6)
                ops.recurrence_scan(qk[:, :G * D], qk[:, G * D:], y[:, 2 * G * D:], decay, True, beta, None, None, slot, starts, n, state, o, H, G, D, V)
                ops.gated_norm(o, rows[:, C + 2 * H:], "silu", False, d["norm_w"], 1e-5, H, out)
            at = 0
            for s, p, c in portions:
                got[s].append(out[at:at + c].cpu())
                done[s] += c
                at += c
        for s in lens:
            err = (torch.cat(got[s]).double() - want[s]).abs().max().item()
            assert err < (3e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(want[s].abs().max())), (cut, s, err)
        assert torch.equal(state[2], idle)


def test_single_tokens_of_many_requests(ops):
    """More requests than multiprocessors have room for at once, positions before and after the convolution is filled, a sigmoid
    gate, slots in any order."""
    H, G, D, V, taps, n = 6, 3, 16, 48, 4, 40
    C, N = 2 * G * D + H * V, 2 * G * D + 2 * H * V + 2 * H
    rn = gen(1)
    proj, state = rn(2, n, N), rn(n + 3, H * D * V + taps * C)
    w = [0.5 * rn(C, taps), rn(H), rn(H), 1 + 0.1 * rn(V)]
    pos = torch.tensor([(0, 1, 2, 3, 4, 100, 5, 7, 1023)[t % 9] for t in range(n)], dtype=torch.int32)
    slot = torch.tensor([n + 1 - t for t in range(n)], dtype=torch.int32)
    st_ref, want = state.double(), torch.zeros(n, H * V, dtype=F64)
    RefOps(F64).delta_token(proj, *w, "sigmoid", pos, slot, st_ref, 1e-6, 1e-5, want, H, G, D, V)
    st, out = state.to(DEV), torch.zeros(n, H * V, device=DEV)
    ops.delta_token(proj.to(DEV), *(t.to(DEV) for t in w), "sigmoid", pos.to(DEV), slot.to(DEV), st, 1e-6, 1e-5, out, H, G, D, V)
    assert (out.cpu().double() - want).abs().max() < 3e-5 and (st.cpu().double() - st_ref).abs().max() < 3e-5


# ------------------------------------------------------------------------------------------------ experts that read scaled rows
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,top,N,K", [(1, 4, 2, 32, 64), (7, 10, 3, 112, 208), (200, 10, 3, 112, 208), (90, 3, 3, 13, 40), (300, 2, 1, 20, 36), (300, 5, 4, 24, 38),
                                         (1, 1, 1, 16, 30)])
def test_a_mixture_whose_scores_multiply_the_input(ops, dtype, T, E, top, N, K):
    """The whole part, from the float32 rows to the pending rows, beside the plain mixture following its choices (few choices:
    plan and rows in one launch; many; rows of no whole 16-byte units)."""
    from flint_b200.parts.ffn import SigmoidTopKMoE
    rn = gen(T + E)
    part = SigmoidTopKMoE({"hidden_size": K, "intermediate_size": N, "num_experts": E, "top": top, "gated": True, "act": "swish_clamped",
                           "act_slope": 1.702, "act_limit": 1.2}, BuildContext(ops, torch.device(DEV), "bfloat16" if dtype == torch.bfloat16 else "float32"))
    w = {n: (rn(*s.shape) * (2.0 / math.sqrt(s.shape[-1]))).to(dtype) for n, s in part.weights().items()}
    part.load({n: t.to(DEV) for n, t in w.items()})
    h = rn(T, K)
    step = SimpleNamespace(record={})
    pend = part.forward({torch.float32: h.to(DEV)}, None, step)
    out = torch.zeros(T, K, device=DEV)
    ops.moe_combine(out, pend.y, pend.row_of, pend.gates)
    ids = step.record["experts"][0].cpu()
    f = {"router": {"experts": E, "top": top}, "expert": {"ff": N, "limit": 1.2}}
    wd = {"m." + n: t.double() for n, t in w.items()}
    want, _ = P.experts(h.double(), wd, "m.", f, forced=ids)
    assert (out.cpu().double() - want).abs().max() < (5e-5 if dtype == torch.float32 else 3e-2) * max(1.0, float(want.abs().max()))
    own, _ = P.route(h.double(), wd, "m.", f)
    assert int((own.sort(-1).values != ids.long().sort(-1).values).any(-1).sum()) <= 1


# ------------------------------------------------------------------------------------------------ the whole model
@pytest.fixture(scope="module", params=list(tiny.CONFIGS))
def setup(request, tmp_path_factory):
    which = request.param
    cfg = tiny.CONFIGS[which]
    folder, w = tiny.write_model(tmp_path_factory.mktemp("sokipel") / which, cfg, seed=3)
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
    """The plain implementation run with the experts the engine chose for the whole prompts (in bfloat16 a near-tie of two
    scores may fall the other way), and how many (row, layer) choices differ from the plain router's own."""
    steps = traces.whole(reqs)
    _, recs, _ = replay(folder, steps, dtype, record={})
    routed = [i for i, l in enumerate(cfg["layers"]) if l["mlp"]]
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
    base = plain
    if dtype == "bfloat16":
        base, flips = followed(cfg, w, reqs, folder, dtype)
        assert flips <= 0.1 * sum(LENGTHS) * len(cfg["layers"])
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
            assert all(max(g.pages.pool.served) >= 2 for g in rp.model.cache.groups)


def test_every_layer_leaves_what_the_plain_model_does(setup):
    which, cfg, folder, w, reqs, plain = setup
    _, recs, _ = replay(folder, traces.whole({"r4": reqs["r4"]}), "float32", record={"rows_after": []})
    after = P.forward(cfg, w, reqs["r4"])[1]
    assert len(recs[0]["rows_after"]) == len(after)
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


@pytest.mark.parametrize("seed", [11, 12, 13, 14, 15, 16, 17, 18])
def test_configurations_drawn_at_random(seed, tmp_path):
    cfg = tiny.random_config(seed)
    folder, w = tiny.write_model(tmp_path / "m", cfg, seed=seed)
    reqs = traces.make_requests(cfg["vocab"], (1, 2, 23, 50, 85, 140), seed=seed)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    for cut in (traces.whole, lambda r: traces.tail_decoded(r, tail=45), lambda r: traces.portions(r, sizes=(2, 3, 16, 1, 2, 64)),
                lambda r: traces.mixed(r, seed=seed)):
        steps = cut(reqs)
        out, _, _ = replay(folder, steps, "float32", page_size=16)
        exp = traces.expected_rows(steps, plain)
        errs = torch.cat([rel_err(out[k], torch.stack(rows)) for k, rows in exp.items()])
        assert float(errs.max()) < 1e-4, (cfg, float(errs.max()))


def test_long_decoding_token_by_token(setup):
    """Two requests decoded side by side, one token a step each, over several pages and past every chunk's edge, after prompts
    of unequal length: the captured decode step is replayed many times, and the states are carried through all of them."""
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
    if which not in ("K1", "K2"):
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
            errs.append(rel_err(torch.from_numpy(np.fromfile(f, dtype="<f4").reshape(n, cfg["vocab"])), torch.stack(exp[s["step"]])))
    errs = torch.cat(errs)
    if dtype == "float32":
        assert float(errs.max()) < 1e-4
    else:       # a near-tie of two scores may fall the other way at some rows
        assert float(errs.median()) < 5e-2


def test_chat_program_with_random_weights(tmp_path):
    """bin/flint_chat with ``--random-config FILE --seed N``, token ids in and out, greedy: the tokens of the folder that the
    random-weights mode writes for that configuration and seed, under the plain implementation."""
    from flint_b200.engine.loading import write_random_model
    from flint_b200.weights.safetensors_io import SafetensorsFile
    seed, cfg = 4, tiny.K3
    folder = write_random_model(tmp_path / "model", cfg, seed=seed)
    f = SafetensorsFile(folder / "model.safetensors")
    w = {n: f.read(n).double() for n in f.names()}
    prompt = [3, 50, 50, 7, 60, 0, 12, 13, 14, 15, 16]
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
