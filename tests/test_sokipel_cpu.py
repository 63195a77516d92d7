"""Sokipel through the engine's plumbing on the CPU (the kernels replaced by their plain references): hand-computed cases of the
plain mechanisms, the configuration reader, tensor names, rotation tables, what every layer leaves, state across steps and slots,
and replay under every cut against the plain implementation."""
import copy
import math

import pytest
import torch

import plain_sokipel as P
import tiny_sokipel as tiny
import traces
from flint_b200.engine.engine import Engine
from flint_b200.engine.loading import expected_from_config, write_random_model
from flint_b200.engine.model import load_model
from flint_b200.engine.replay import Replayer
from flint_b200.errors import ConfigError, WeightError
from flint_b200.parts.base import BuildContext
from flint_b200.parts.rope import RotaryEncoding
from flint_b200.sampling.params import SamplingParams
from kernel_refs import RefOps

LENGTHS = (1, 2, 9, 37, 70, 130)
F64 = torch.float64


@pytest.fixture(scope="module", params=list(tiny.CONFIGS))
def setup(request, tmp_path_factory):
    which = request.param
    cfg = tiny.CONFIGS[which]
    folder, w = tiny.write_model(tmp_path_factory.mktemp("sokipel") / which, cfg, seed=3)
    reqs = traces.make_requests(cfg["vocab"], LENGTHS, seed=7)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    return which, cfg, folder, w, reqs, plain


def replay(folder, steps, page_size=16, record=False):
    rp = Replayer(folder, dtype="float32", max_tokens=traces.max_tokens_needed(steps), page_size=page_size, max_requests=4,
                  device="cpu", ops=RefOps())
    out, recs = {}, {}
    for s in steps:
        rec = {"rows_after": []} if record else None
        lg = rp.run_step(s["entries"], s["end"], record=rec)
        if lg is not None:
            out[s["step"]] = lg
        recs[s["step"]] = rec
        rp.model.cache.check()
    assert all(g.pages.pool.used_pages == 0 for g in rp.model.cache.groups)
    return out, recs, rp


def compare(out, steps, plain, tol=3e-4):
    exp = traces.expected_rows(steps, plain)
    assert set(out) == set(exp)
    for k, rows in exp.items():
        want = torch.stack(rows)
        err = (out[k].double() - want).abs().max().item()
        assert err < tol * max(1.0, float(want.abs().max())), f"step {k}: max error {err:.2e}"


# ------------------------------------------------------------------------------------------------ the plain mechanisms
def test_the_plain_norms_and_convolutions():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    # one number for all coordinates, eps inside the root
    assert torch.allclose(P.one_number_norm(x, torch.tensor(2.0, dtype=F64), 12.5), 2 * x / 5)
    assert torch.allclose(P.unit_length(x, 0.0), x / 5)
    # the last tap is the row's own, nothing before the start; a mixer reads the row plus the convolution
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    w = torch.tensor([[2.0, 3.0, 5.0]], dtype=F64)
    assert P.causal_conv(u, w)[:, 0].tolist() == [5.0, 53.0, 532.0]
    assert P.input_conv(u, w)[:, 0].tolist() == [6.0, 63.0, 632.0]


def test_the_plain_rotations():
    rot = {"dims": 4, "base": 100.0}
    f = P.base_frequencies(rot)
    assert torch.allclose(f, torch.tensor([1.0, 0.1], dtype=F64))
    assert torch.allclose(P.linear_frequencies({**rot, "scaling": {"factor": 4.0}}), f / 4)
    # wavelengths 6.28 and 62.8: below original / high kept, above original / low divided, between a share of both
    sc = lambda original: {**rot, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": original}}
    assert torch.allclose(P.banded_frequencies(sc(1000)), f)
    assert torch.allclose(P.banded_frequencies(sc(5)), f / 8)
    assert torch.allclose(P.banded_frequencies(sc(40)), torch.tensor([1.0, 0.1 / 8], dtype=F64))
    share = (20 / (2 * math.pi) - 1) / 3
    assert torch.allclose(P.banded_frequencies(sc(20))[0], torch.tensor((1 - share) / 8 + share, dtype=F64))
    # the pairs: (0, 1), (2, 3) or (0, 2), (1, 3); dims beyond the rotating ones stay
    x = torch.zeros(2, 1, 5, dtype=F64)
    x[1, 0] = torch.tensor([1.0, 0.0, 0.0, 0.0, 7.0], dtype=F64)
    c, s = math.cos(1.0), math.sin(1.0)
    assert torch.allclose(P.turn(x, f, True)[1, 0], torch.tensor([c, s, 0, 0, 7.0], dtype=F64))
    assert torch.allclose(P.turn(x, f, False)[1, 0], torch.tensor([c, 0, s, 0, 7.0], dtype=F64))


def test_the_plain_attention_mask_and_sink():
    m = P.visible(7, 3)                    # chunks 0 1 2 | 3 4 5 | 6
    assert m[2].tolist() == [True] * 3 + [False] * 4 and m[4].tolist() == [False] * 3 + [True] * 2 + [False] * 2
    assert m[6].tolist() == [False] * 6 + [True] and torch.equal(P.visible(4, 0), torch.ones(4, 4, dtype=torch.bool).tril())
    # equal scores of 0 and a sink of 0: n keys share n / (n + 1); the sink is not scaled and counts once
    p = P.sink_softmax(torch.zeros(3, 1, 4, dtype=F64), torch.tensor([0.0, 30.0, -30.0], dtype=F64))
    assert torch.allclose(p[0], torch.full((1, 4), 0.2, dtype=F64)) and float(p[1].sum()) < 1e-9 and abs(float(p[2].sum()) - 1) < 1e-9
    # query head h reads key head floor(h / (H / G)), and the scores are scaled
    q, k, v = torch.ones(1, 4, 1, dtype=F64), torch.tensor([[[0.0], [2.0]]], dtype=F64), torch.tensor([[[1.0], [10.0]]], dtype=F64)
    o = P.attend(q, k, v, 0.5, P.visible(1, 0), torch.zeros(4, dtype=F64))[0, :, 0]
    e = math.e / (math.e + 1)
    assert torch.allclose(o, torch.tensor([0.5, 0.5, 10 * e, 10 * e], dtype=F64))


def test_the_plain_delta_rule():
    # one head, one key dim, one value dim: S decays, then moves towards v for the key, and the read-out sees the write
    one = lambda x: torch.tensor([[x]], dtype=F64)
    S = torch.tensor([[[2.0]]], dtype=F64)
    S, o = P.delta_step(S, one(3.0), one(1.0), one(5.0), torch.tensor([0.5], dtype=F64), torch.tensor([0.25], dtype=F64))
    assert float(S[0, 0, 0]) == 1.0 + 0.25 * (5.0 - 1.0) and float(o[0, 0]) == 6.0
    # a unit key written with strength one is read back whole, whatever was there
    S, o = P.delta_step(torch.randn(1, 3, 2, dtype=F64), torch.eye(3, dtype=F64)[:1], torch.eye(3, dtype=F64)[:1],
                        torch.tensor([[4.0, -1.0]], dtype=F64), torch.tensor([0.3], dtype=F64), torch.ones(1, dtype=F64))
    assert torch.allclose(o[0], torch.tensor([4.0, -1.0], dtype=F64))


def test_the_plain_router_and_experts():
    f = {"router": {"experts": 3, "top": 2}, "expert": {"ff": 1, "limit": 1.5}}
    w = {"m.router": torch.tensor([[1.0], [-1.0], [2.0]], dtype=F64)}
    h = torch.ones(1, 1, dtype=F64)
    ids, s = P.route(h, w, "m.", f)
    assert ids[0].tolist() == [2, 0] and torch.allclose(s[0], torch.sigmoid(torch.tensor([2.0, 1.0], dtype=F64)))   # not renormalised
    # the clamp: the gate from above only, the other factor on both sides
    one = lambda x: torch.tensor([[x]], dtype=F64)
    assert abs(float(P.expert(one(1.0), one(9.0), one(-9.0), one(1.0), 1.5)) - 1.5 / (1 + math.exp(-1.702 * 1.5)) * (1 - 1.5)) < 1e-12
    assert abs(float(P.expert(one(1.0), one(-9.0), one(0.0), one(1.0), 1.5)) - (-9.0 / (1 + math.exp(1.702 * 9)))) < 1e-12
    # the score multiplies the input: expert(s h), not s expert(h)
    for e in range(3):
        w.update({f"m.e{e}.gate": one(1.0), f"m.e{e}.up": one(0.0), f"m.e{e}.down": one(float(e + 1))})
    y, _ = P.experts(h, w, "m.", f)
    unit = lambda z: z / (1 + math.exp(-1.702 * z))
    assert abs(float(y) - (3 * unit(float(s[0, 0])) + 1 * unit(float(s[0, 1])))) < 1e-12


# ------------------------------------------------------------------------------------------------ configuration and tensors
def test_rotation_tables_follow_the_plain_frequencies():
    ctx = BuildContext(ops=None, device=torch.device("cpu"), compute="float32", max_context=300)
    for params, freq in (({"linear": 3.0}, P.linear_frequencies({"dims": 12, "base": 77.0, "scaling": {"factor": 3.0}})),
                         *(({"banded": dict(zip(tiny.BANDED, b))},
                            P.banded_frequencies({"dims": 12, "base": 77.0, "scaling": dict(zip(tiny.BANDED, b))}))
                           for b in ((4.0, 1.0, 4.0, 60), (8.0, 0.5, 8.0, 200), (2.0, 1.0, 1.0, 30), (2.0, 1.0, 2.0, 1)))):
        cos, sin = RotaryEncoding({"rotary_dim": 12, "theta": 77.0, "max_positions": 1000, **params}, ctx).tables()
        ang = torch.arange(300, dtype=F64)[:, None] * freq
        assert (cos.double() - torch.cos(ang)).abs().max() < 1e-7 and (sin.double() - torch.sin(ang)).abs().max() < 1e-7


def test_config_names_every_size_and_refuses_what_it_cannot_read():
    for which, cfg in tiny.CONFIGS.items():
        spec, expected = expected_from_config(cfg)
        assert {spec.stored_names.get(n, n): tuple(ws.shape) for n, ws in expected.items()} == tiny.tensor_shapes(cfg)
        assert all(l.block == "outnorm" for l in spec.layers)
    spec, _ = expected_from_config(tiny.K1)
    assert "ffn" not in spec.layers[1].parts and "norm2" not in spec.layers[1].parts
    for key, value, message in ((("layers", 0, "type"), "conv", "unknown layer type"),
                                (("layers", 1, "mixer", "heads"), 5, "multiple of kv_heads"),
                                (("layers", 2, "mixer", "kv_heads"), 3, "multiple of kv_heads"),
                                (("layers", 1, "mixer", "rot", "dims"), 8, "at most dim"),
                                (("layers", 1, "mixer", "rot", "dims"), 3, "must be even"),
                                (("layers", 1, "mixer", "rot", "scaling", "factor"), -1.0, "must be positive"),
                                (("layers", 1, "mixer", "rot", "scaling", "high"), 0.5, "at least low"),
                                (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0.0, "must be positive"),
                                (("layers", 1, "mixer", "mask", "size"), 0, "size"),
                                (("layers", 0, "mlp", "router", "top"), 6, "exceeds"),
                                (("layers", 0, "mlp", "kind"), "dense", "unknown kind"),
                                (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
                                (("canon", "taps"), 0, "taps"), (("logit_softcap",), 0.0, "logit_softcap"),
                                (("layers", 2, "mixer", "dim"), 300, "not supported"), (("canon", "taps"), 65, "not supported")):
        bad = copy.deepcopy(tiny.K1)
        d = bad
        for k in key[:-1]:
            d = d[k]
        d[key[-1]] = value
        with pytest.raises(ConfigError, match=message):
            expected_from_config(bad)
    for path in (("layers", 1, "mixer", "scale"), ("layers", 0, "mixer", "left_scale"), ("layers", 0, "mixer", "right", "conv"),
                 ("layers", 1, "mixer", "rot", "scaling", "original"), ("residual_mult",), ("embedding", "scale"), ("canon",)):
        bad = copy.deepcopy(tiny.K1)
        d = bad
        for k in path[:-1]:
            d = d[k]
        del d[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            expected_from_config(bad)


def test_a_missing_or_misshaped_tensor_is_named(tmp_path):
    w = tiny.random_weights(tiny.K1, 1)
    del w["l1.mix.sink"], w["l0.canon1"]
    w["l2.mix.dt_bias"] = w["l2.mix.dt_bias"][:2]
    w["l0.norm2"] = torch.ones(30, dtype=torch.bfloat16)              # a norm's scale is one number
    w["l1.mix.g"] = torch.ones(6, 30, dtype=torch.bfloat16)           # attention in chunks has no gate
    folder, _ = tiny.write_model(tmp_path / "m", tiny.K1, weights=w)
    with pytest.raises(WeightError) as e:
        load_model(folder, dtype="float32", device="cpu", ops=RefOps(), page_size=16, n_pages=4, max_slots=2, max_context=64)
    assert all(n in str(e.value) for n in ("l1.mix.sink", "l0.mix.input_conv", "l2.mix.dt_bias", "l0.norm2", "l1.mix.gate_proj"))


def test_random_weights_mode_writes_the_design_s_own_names(tmp_path):
    folder = write_random_model(tmp_path / "m", tiny.K2, seed=5)
    from flint_b200.weights.safetensors_io import SafetensorsFile
    assert set(SafetensorsFile(folder / "model.safetensors").names()) == set(tiny.tensor_shapes(tiny.K2))
    m = load_model(folder, dtype="float32", device="cpu", ops=RefOps(), page_size=16, n_pages=8, max_slots=2, max_context=128)
    # every layer keeps its rows' last inputs; two layers own keys and values, of different sizes
    assert sorted(m.cache.state) == [0, 1, 2, 3] and sorted(c for g in m.cache.groups for c in g.calls) == [1, 2]
    assert m.cache.state[1].shape[1] == (tiny.K2["canon"]["taps"] - 1) * tiny.K2["width"]
    inner = m.layers[0].parts["mixer"].inner
    assert m.cache.state[0].shape[1] == (tiny.K2["canon"]["taps"] - 1) * tiny.K2["width"] + inner.state_spec().shape[0]
    # the bytes of inner parts count
    assert m.weight_bytes() >= 4 * sum(math.prod(s) for n, s in tiny.tensor_shapes(tiny.K2).items() if n.endswith((".q", ".o", ".gate", ".up", ".down")))


# ------------------------------------------------------------------------------------------------ the engine against the plain model
def test_every_layer_leaves_what_the_plain_model_does(setup):
    which, cfg, folder, w, reqs, plain = setup
    _, after, _ = P.forward(cfg, w, reqs["r3"])
    _, recs, _ = replay(folder, traces.whole({"r3": reqs["r3"]}), record=True)
    rows = recs[0]["rows_after"]
    assert len(rows) == len(cfg["layers"])
    for i, r in enumerate(rows):
        assert (r.double() - after[i]).abs().max() < 3e-4 * max(1.0, float(after[i].abs().max())), f"layer {i}"


def test_replay_matches_plain_whole_and_cut(setup):
    which, cfg, folder, w, reqs, plain = setup
    for cut in (traces.whole, lambda r: traces.tail_decoded(r, tail=40), traces.portions,
                lambda r: traces.portions(r, sizes=(2, 2, 1, 2, 3, 128))):
        steps = cut(reqs)
        out, _, _ = replay(folder, steps)
        compare(out, steps, plain)


def test_replay_matches_plain_in_mixed_batches_with_slots_and_pages_used_again(setup):
    which, cfg, folder, w, reqs, plain = setup
    more = dict(reqs)
    more.update({f"x{k}": v for k, v in traces.make_requests(cfg["vocab"], (33, 5, 64, 17), seed=11).items()})
    full = dict(plain)
    full.update({rid: P.forward(cfg, w, t)[0] for rid, t in more.items() if rid not in full})
    for seed in (3, 4):
        steps = traces.mixed(more, seed=seed)
        out, _, rp = replay(folder, steps)
        compare(out, steps, full)
        assert all(max(g.pages.pool.served) >= 2 for g in rp.model.cache.groups)      # pages were used again


def test_state_starts_anew_in_a_slot_that_was_used(setup):
    """One slot, three requests one after the other: each must see the state and the convolutions' inputs of a new sequence,
    decoded from its first token on."""
    which, cfg, folder, w, reqs, plain = setup
    rp = Replayer(folder, dtype="float32", max_tokens=192, page_size=16, max_requests=1, device="cpu", ops=RefOps())
    for rid, head in (("r4", 5), ("r3", 1), ("r4", 2)):
        t = reqs[rid]
        a = rp.run_step([{"id": rid, "tokens": t[:head], "want": [head - 1]}])
        b = rp.run_step([{"id": rid, "tokens": t[head:head + 1], "want": [0]}])
        c = rp.run_step([{"id": rid, "tokens": t[head + 1:], "want": [len(t) - head - 2]}], end=[rid])
        got = torch.cat([a, b, c]).double()
        want = torch.stack([plain[rid][head - 1], plain[rid][head], plain[rid][-1]])
        assert (got - want).abs().max() < 3e-4 * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_configurations_drawn_at_random(seed, tmp_path):
    cfg = tiny.random_config(seed)
    folder, w = tiny.write_model(tmp_path / "m", cfg, seed=seed)
    reqs = traces.make_requests(cfg["vocab"], (1, 2, 23, 50, 85), seed=seed)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    for cut in (traces.whole, lambda r: traces.tail_decoded(r, tail=45), lambda r: traces.portions(r, sizes=(2, 3, 16, 1, 2, 64)),
                lambda r: traces.mixed(r, seed=seed)):
        steps = cut(reqs)
        out, _, _ = replay(folder, steps)
        compare(out, steps, plain)


def test_greedy_generation_through_the_engine_with_preemption(setup):
    which, cfg, folder, w, reqs, plain = setup
    prompts = [reqs["r2"], reqs["r3"][:14], reqs["r0"]]
    expected = []
    for p in prompts:
        toks, out = list(p), []
        for _ in range(10):
            t = int(torch.argmax(P.forward(cfg, w, toks)[0][-1]))
            out.append(t)
            toks.append(t)
        expected.append(out)
    for n_pages in (16, 3):
        m = load_model(folder, dtype="float32", device="cpu", ops=RefOps(), page_size=16, n_pages=n_pages, max_slots=4,
                       max_step_tokens=24, max_context=256, use_graphs=False)
        eng = Engine(m, SamplingParams.greedy(), prefill_chunk=16)
        assert eng.generate(prompts, 10) == expected
        assert all(g.pages.pool.used_pages == 0 for g in m.cache.groups) and m.cache.free_slots == 4
    assert eng.scheduler.preemptions > 0


def test_every_mechanism_shows_in_the_logits(setup, monkeypatch):
    """A plain implementation with one mechanism left out or one off gives other logits, far beyond the tolerance of the
    comparisons above: the tests' weights hide none of them."""
    which, cfg, folder, w, reqs, plain = setup
    t, base = reqs["r5"], plain["r5"]
    layers = cfg["layers"]
    has = {k: any(l["type"] == k for l in layers) for k in ("attention", "delta", "parallel")}
    deltas = [l["mixer"] if l["type"] == "delta" else l["mixer"]["right"] for l in layers if l["type"] != "attention"]
    o = {n: getattr(P, n) for n in ("visible", "sink_softmax", "turn", "causal_conv", "input_conv", "delta_step", "expert", "experts",
                                    "route", "silu", "banded_frequencies", "linear_frequencies", "unit_length", "one_number_norm")}
    older = lambda taps: torch.cat([0 * taps[:, :1], taps[:, 1:]], 1)
    late = lambda S, q, k, v, g, b: (o["delta_step"](S, q, k, v, g, b)[0], torch.einsum("hdv,hd->hv", g[:, None, None] * S, q))
    cases = {
        "a sink left out": {"sink_softmax": lambda s, sink: torch.softmax(s, -1)},
        "no rotation": {"turn": lambda x, f, il: x},
        "the other pairs rotate": {"turn": lambda x, f, il: o["turn"](x, f, not il)},
        "no convolution in front of the mixers": {"input_conv": lambda x, taps: x},
        "only the convolution in front": {"input_conv": o["causal_conv"]},
        "norms left out": {"one_number_norm": lambda x, g, eps: x * g},
        "an expert without its clamp": {"expert": lambda h, g, u, d, lim: o["expert"](h, g, u, d, 1e9)},
        "scores normalised": {"route": lambda *a, **k: (lambda i, s: (i, s / s.sum(-1, keepdim=True)))(*o["route"](*a, **k))},
    }
    if has["attention"]:
        cases["a chunk one longer"] = {"visible": lambda T, c: o["visible"](T, c + 1 if c else 0)}
        if any(l["type"] == "attention" and l["mixer"]["mask"]["size"] > 1 for l in layers):
            cases["chunks counted from elsewhere"] = {"visible": lambda T, c: o["visible"](T + 1, c)[1:, 1:] if c else o["visible"](T, 0)}
        if any(l["type"] == "attention" and l["mixer"]["rot"].get("scaling") for l in layers) and which != "K3":
            cases["frequencies as they are"] = {"banded_frequencies": P.base_frequencies}
    if has["parallel"] and any(l["type"] == "parallel" and l["mixer"]["left"]["rot"].get("scaling") for l in layers):
        cases["undivided frequencies"] = {"linear_frequencies": P.base_frequencies}
    if deltas:
        cases.update({"the read-out before the write": {"delta_step": late},
                      "no decay": {"delta_step": lambda S, q, k, v, g, b: o["delta_step"](S, q, k, v, torch.ones_like(g), b)},
                      "a plain write": {"delta_step": lambda S, q, k, v, g, b: (lambda N: (N, torch.einsum("hdv,hd->hv", N, q)))(
                          g[:, None, None] * S + b[:, None, None] * k[:, :, None] * v[:, None, :])},
                      "keys of any length": {"unit_length": lambda x, eps: x}})
    if any(d["conv"] > 1 for d in deltas) or cfg["canon"]["taps"] > 1:
        cases["convolutions without their oldest input"] = {"causal_conv": lambda u, taps: o["causal_conv"](u, older(taps) if taps.shape[1] > 1 else taps)}
    if not any(l["mlp"] for l in layers):
        del cases["an expert without its clamp"]
    for name, patch in cases.items():
        with monkeypatch.context() as m:
            for k, v in patch.items():
                m.setattr(P, k, v)
            other = P.forward(cfg, w, t)[0]
        d = (other - base).abs().max(-1).values / base.abs().max()
        assert float(d.max()) > 1e-2, name
        assert int((d > 3e-3).sum()) >= 10, name
