"""Sinilorn through the engine's plumbing on the CPU (the kernels replaced by their plain references): hand-computed cases
of the plain mechanisms, the configuration reader, tensor names, the reach of cached latent rows, what every layer leaves
in the streams, state across steps and slots, and replay under every cut against the plain implementation."""
import copy
import math

import pytest
import torch

import plain_sinilorn as P
import tiny_sinilorn as tiny
import traces
from flint_b200.engine.engine import Engine
from flint_b200.engine.loading import expected_from_config, write_random_model
from flint_b200.engine.model import load_model
from flint_b200.engine.replay import Replayer
from flint_b200.errors import ConfigError, WeightError
from flint_b200.sampling.params import SamplingParams
from kernel_refs import RefOps

LENGTHS = (1, 2, 9, 37, 70, 130)
F64 = torch.float64


@pytest.fixture(scope="module", params=["S1", "S2", "S3", "S4"])
def setup(request, tmp_path_factory):
    which = request.param
    cfg = tiny.CONFIGS[which]
    folder, w = tiny.write_model(tmp_path_factory.mktemp("sinilorn") / which, cfg, seed=3)
    reqs = traces.make_requests(cfg["vocab"], LENGTHS, seed=7)
    plain = {rid: P.forward(cfg, w, t)[0] for rid, t in reqs.items()}
    return which, cfg, folder, w, reqs, plain


def replay(folder, steps, page_size=16, record=False):
    n = traces.max_tokens_needed(steps)
    rp = Replayer(folder, dtype="float32", max_tokens=n, page_size=page_size, max_requests=4, device="cpu", ops=RefOps())
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
def test_the_plain_streams_norm_and_rotation():
    g = torch.Generator().manual_seed(1)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    # streams: mix is indexed [from, to], every new stream is made from the old ones
    x, y = rn(2, 3, 4), rn(3, 4)
    mix, out = torch.tensor([[0.0, 1.0], [2.0, 0.0]], dtype=F64), torch.tensor([3.0, -1.0], dtype=F64)
    new = P.spread_streams(x, y, mix, out)
    assert torch.allclose(new[0], 2 * x[1] + 3 * y) and torch.allclose(new[1], x[0] - y)
    assert torch.allclose(P.gather_streams(x, torch.tensor([2.0, -1.0], dtype=F64)), 2 * x[0] - x[1])
    # layer norm: the mean of the squared deviations, eps inside the root
    v = torch.tensor([[1.0, 3.0]], dtype=F64)
    assert torch.allclose(P.layer_norm(v, torch.ones(2, dtype=F64), 3.0), torch.tensor([[-0.5, 0.5]], dtype=F64))
    # YaRN: frequencies below the ramp stay, those above it are divided by the factor
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 4.0, "original": 32, "fast": 16.0, "slow": 1.0}}
    f, mag = P.rotary_frequencies(rot)
    plain_f, one = P.rotary_frequencies({"dims": 8, "base": 100.0})
    assert one == 1.0 and abs(mag - (0.1 * math.log(4.0) + 1)) < 1e-12
    assert torch.all(f <= plain_f + 1e-15) and torch.all(f >= plain_f / 4 - 1e-15) and f[0] == plain_f[0]
    r = rn(5, 3, 8)
    z = P.rotate(r, torch.arange(5), {"dims": 8, "base": 100.0})
    assert torch.allclose(z[0], r[0])
    assert torch.allclose(z[2, 1, 0] ** 2 + z[2, 1, 4] ** 2, r[2, 1, 0] ** 2 + r[2, 1, 4] ** 2)      # dim i turns with i + dims/2


def test_the_plain_attention_mask_and_sink():
    # a window of 3: position 4 sees 2, 3, 4
    m = P.window_mask(6, 3)
    assert m[4].tolist() == [False, False, True, True, True, False] and m[1].tolist() == [True, True] + [False] * 4
    assert torch.equal(P.window_mask(5, 0), torch.ones(5, 5, dtype=torch.bool).tril())
    # equal scores of 0 and a sink of 0: n keys share n / (n + 1); a large sink takes almost everything, a small one nothing
    s = torch.zeros(3, 1, 4, dtype=F64)
    p = P.sink_softmax(s, torch.tensor([0.0, 30.0, -30.0], dtype=F64))
    assert torch.allclose(p[0], torch.full((1, 4), 0.2, dtype=F64)) and float(p[1].sum()) < 1e-9 and abs(float(p[2].sum()) - 1) < 1e-9
    # the sink is not scaled and counts once, whatever the scores
    s = torch.tensor([[[2.0, -math.inf]]], dtype=F64)
    assert torch.allclose(P.sink_softmax(s, torch.tensor([1.0], dtype=F64))[0, 0, 0], torch.sigmoid(torch.tensor(1.0, dtype=F64)))


def test_the_plain_recurrent_unit():
    g = torch.Generator().manual_seed(2)
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    # the convolution: the last tap is the row's own input, zeros before the start
    u, taps = rn(4, 2), rn(2, 3)
    c = P.causal_conv(u, taps, torch.tensor([0.5, -1.0], dtype=F64))
    assert torch.allclose(c[0], taps[:, 2] * u[0] + torch.tensor([0.5, -1.0], dtype=F64))
    assert torch.allclose(c[3], taps[:, 0] * u[1] + taps[:, 1] * u[2] + taps[:, 2] * u[3] + torch.tensor([0.5, -1.0], dtype=F64))
    # block-diagonal gates [out, in]: a channel reads its own block only
    mats = torch.zeros(2, 2, 2, dtype=F64)
    mats[1, 0, 1] = 1.0                                     # channel 2 reads channel 3
    z = P.block_gate(rn(1, 4), mats, torch.zeros(2, 2, dtype=F64))
    assert torch.allclose(z[0, [0, 1, 3]], torch.full((3,), 0.5, dtype=F64)) and abs(float(z[0, 2]) - 0.5) > 1e-3
    # one channel with gates of 1/2 and lam = 0: a = exp(-4 ln 2) = 1/16; S_1 = a S_0 + sqrt(1 - a^2) u_1 / 2, and the first
    # token has no special case
    m = {"width": 1, "blocks": 1, "conv": 1}
    h = rn(3, 1)
    w = {"p.y": torch.zeros(1, 1, dtype=F64), "p.y.b": torch.full((1,), 2.0, dtype=F64), "p.x": torch.ones(1, 1, dtype=F64),
         "p.x.b": torch.zeros(1, dtype=F64), "p.conv": torch.ones(1, 1, dtype=F64), "p.conv.b": torch.zeros(1, dtype=F64),
         "p.ra": torch.zeros(1, 1, 1, dtype=F64), "p.ra.b": torch.zeros(1, 1, dtype=F64), "p.ri": torch.zeros(1, 1, 1, dtype=F64),
         "p.ri.b": torch.zeros(1, 1, dtype=F64), "p.lam": torch.zeros(1, dtype=F64), "p.o": torch.ones(1, 1, dtype=F64)}
    o = P.rglru(h, w, "p.", m)
    y, a = P.gelu_tanh(torch.tensor(2.0, dtype=F64)), 1 / 16
    k = math.sqrt(1 - a * a) / 2
    assert torch.allclose(o[0], k * h[0] * y) and torch.allclose(o[1], (a * k * h[0] + k * h[1]) * y)


def test_the_plain_router_and_experts():
    f = {"router": {"experts": 2, "identity": 2, "top": 2}, "expert": {"ff": 1, "limit": 1.5}}
    z = torch.tensor([[1.0], [0.0], [2.0], [-1.0]], dtype=F64)
    w = {"m.router": z, "m.correction": torch.zeros(4, dtype=F64)}
    h = torch.ones(1, 1, dtype=F64)
    s = torch.softmax(z[:, 0], 0)
    ids, weights = P.route(h, w, "m.", f)
    assert ids[0].tolist() == [2, 0] and torch.allclose(weights[0], s[[2, 0]] / s[[2, 0]].sum())
    # a correction changes the choice, not the weights
    w["m.correction"] = torch.tensor([0.0, 0.0, -1.0, 5.0], dtype=F64)
    ids, weights = P.route(h, w, "m.", f)
    assert ids[0].tolist() == [3, 0] and torch.allclose(weights[0], s[[3, 0]] / s[[3, 0]].sum())
    # an identity expert hands the input on; the clamp: gate from above only, up on both sides
    w.update({"m.e0.gate": torch.tensor([[9.0]], dtype=F64), "m.e0.up": torch.tensor([[-9.0]], dtype=F64), "m.e0.down": torch.tensor([[1.0]], dtype=F64),
              "m.e1.gate": torch.zeros(1, 1, dtype=F64), "m.e1.up": torch.zeros(1, 1, dtype=F64), "m.e1.down": torch.zeros(1, 1, dtype=F64)})
    y, _ = P.moe(h, w, "m.", f)
    e0 = 1.5 / (1 + math.exp(-1.702 * 1.5)) * (-1.5 + 1)
    assert torch.allclose(y[0, 0], weights[0, 0] * 1.0 + weights[0, 1] * e0)
    low = P.expert(torch.tensor([[1.0]], dtype=F64), torch.tensor([[-9.0]], dtype=F64), torch.tensor([[0.0]], dtype=F64), torch.ones(1, 1, dtype=F64), 1.5)
    assert abs(float(low) - (-9.0 / (1 + math.exp(1.702 * 9)))) < 1e-12


# ------------------------------------------------------------------------------------------------ configuration and tensors
def test_config_names_every_size_and_refuses_what_it_cannot_read():
    for which, cfg in tiny.CONFIGS.items():
        spec, expected = expected_from_config(cfg)
        stored = {spec.stored_names.get(n, n): tuple(ws.shape) for n, ws in expected.items()}
        assert stored == tiny.tensor_shapes(cfg)
        assert spec.streams == cfg["streams"] and all(l.block == "streams" for l in spec.layers)
    spec, _ = expected_from_config(tiny.S1)
    assert "ffn" not in spec.layers[2].parts and "norm2" not in spec.layers[2].parts and "hc2" not in spec.layers[2].parts
    assert [c.cache_of for c in spec.order] == [None, None, 1, None, None, 3]
    for key, value, message in ((("layers", 0, "type"), "conv", "unknown layer type"),
                                (("layers", 0, "mixer", "blocks"), 3, "multiple of blocks"),
                                (("layers", 1, "mixer", "rot", "dims"), 4, "must equal rot_dim"),
                                (("layers", 1, "mixer", "rot", "scaling", "factor"), -1.0, "must be positive"),
                                (("layers", 2, "mixer", "kv_from"), 0, "latent rows of its own"),
                                (("layers", 2, "mixer", "kv_from"), 5, "latent rows of its own"),
                                (("layers", 5, "mixer", "kv_from"), 2, "latent rows of its own"),
                                (("layers", 2, "mixer", "kv_from"), 3, "earlier latent_attention"),
                                (("layers", 2, "mixer", "kv_rank"), 19, "must be equal"),
                                (("layers", 2, "mixer", "rot", "base"), 301.0, "must be equal"),
                                (("layers", 0, "mlp", "router", "top"), 8, "exceeds"),
                                (("layers", 0, "mlp", "kind"), "mlp", "unknown kind"),
                                (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
                                (("layers", 1, "mixer", "mask", "size"), 0, "size"),
                                (("streams",), 0, "streams"), (("streams",), 40, "streams")):
        bad = copy.deepcopy(tiny.S1)
        d = bad
        for k in key[:-1]:
            d = d[k]
        d[key[-1]] = value
        with pytest.raises(ConfigError, match=message):
            expected_from_config(bad)
    for path in (("layers", 1, "mixer", "q_rank"), ("layers", 1, "mixer", "scale"), ("layers", 0, "mixer", "conv"), ("streams",)):
        bad = copy.deepcopy(tiny.S1)
        d = bad
        for k in path[:-1]:
            d = d[k]
        del d[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            expected_from_config(bad)


def test_cached_rows_reach_as_far_as_their_longest_reader_sees():
    spec, _ = expected_from_config(tiny.S1)
    reach = lambda i: (spec.layers[i].parts["mixer"].params["window"], spec.layers[i].parts["mixer"].params["cache_window"])
    assert reach(1) == (7, 21) and reach(2) == (21, 21)          # layer 2 reads layer 1's rows behind layer 1's own window
    assert reach(3) == (1, 0)                                    # layer 5 sees everything of layer 3's rows
    spec, _ = expected_from_config(tiny.S2)
    assert spec.layers[0].parts["mixer"].params["cache_window"] == 40 == spec.layers[3].parts["mixer"].params["cache_window"]


def test_a_missing_or_misshaped_tensor_is_named(tmp_path):
    w = tiny.random_weights(tiny.S1, 1)
    del w["l1.mix.sink"]
    w["l0.mix.lam"] = w["l0.mix.lam"][:2]
    w["l4.hc2.mix"] = w["l4.hc2.mix"][:1]
    w["l2.mix.dkv"] = w["l1.mix.dkv"]                       # a layer that reads another's rows has none of its own
    folder, _ = tiny.write_model(tmp_path / "m", tiny.S1, weights=w)
    with pytest.raises(WeightError) as e:
        load_model(folder, dtype="float32", device="cpu", ops=RefOps(), page_size=16, n_pages=4, max_slots=2, max_context=64)
    assert all(n in str(e.value) for n in ("l1.mix.sink", "l0.mix.lam", "l4.hc2.mix", "l2.mix.dkv"))


def test_random_weights_mode_writes_the_design_s_own_names(tmp_path):
    folder = write_random_model(tmp_path / "m", tiny.S2, seed=5)
    from flint_b200.weights.safetensors_io import SafetensorsFile
    names = set(SafetensorsFile(folder / "model.safetensors").names())
    assert names == set(tiny.tensor_shapes(tiny.S2))
    m = load_model(folder, dtype="float32", device="cpu", ops=RefOps(), page_size=16, n_pages=8, max_slots=2, max_context=128)
    # two layers own latent rows, in one page group (equal sizes, equal reach); two recurrent units own state
    assert len(m.cache.groups) == 1 and m.cache.groups[0].calls == [0, 3] and sorted(m.cache.state) == [2, 4]


# ------------------------------------------------------------------------------------------------ the engine against the plain model
def test_every_layer_leaves_what_the_plain_model_does(setup):
    which, cfg, folder, w, reqs, plain = setup
    t = reqs["r3"]
    _, after, _ = P.forward(cfg, w, t)
    _, recs, _ = replay(folder, traces.whole({"r3": t}), record=True)
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
        assert max(max(g.pages.pool.served) for g in rp.model.cache.groups) >= 2      # pages were used again


def test_state_starts_anew_in_a_slot_that_was_used(setup):
    """One slot, three requests one after the other: each must see the state and the convolution's inputs of a new
    sequence, decoded from its first token on."""
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


def test_pages_behind_every_reader_s_window_go_back(tmp_path):
    """The rows of a layer whose reader sees further back stay until the reader has passed them, and no longer."""
    cfg = copy.deepcopy(tiny.S1)
    cfg["layers"] = cfg["layers"][:3]
    folder, w = tiny.write_model(tmp_path / "m", cfg, seed=3)
    toks = traces.make_requests(cfg["vocab"], (200,), seed=5)["r0"]
    plain = P.forward(cfg, w, toks)[0]
    rp = Replayer(folder, dtype="float32", max_tokens=256, page_size=16, max_requests=1, device="cpu", ops=RefOps())
    rp.run_step([{"id": "a", "tokens": toks[:100], "want": []}])
    pool = rp.model.cache.groups[0].pages.pool
    assert rp.model.cache.groups[0].spec.window == 21
    for i in range(100, 200):
        out = rp.run_step([{"id": "a", "tokens": [toks[i]], "want": [0]}])
        assert pool.used_pages <= 3                        # 21 positions touch at most three pages of 16
        assert (out[0].double() - plain[i]).abs().max() < 3e-4 * max(1.0, float(plain[i].abs().max())), i


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
    windows = [l for l in cfg["layers"] if l["type"] == "latent_attention" and "mask" in l["mixer"]]
    moes = [i for i, l in enumerate(cfg["layers"]) if l["mlp"] and l["mlp"]["kind"] == "moe"]
    orig = {n: getattr(P, n) for n in ("window_mask", "sink_softmax", "rotate", "causal_conv", "gelu_tanh", "spread_streams", "expert", "route")}
    cases = {
        "a sink left out": {"sink_softmax": lambda s, sink: torch.softmax(s, -1)},
        "no rotation": {"rotate": lambda x, pos, rot: x},
        "the convolution without its oldest input": {"causal_conv": lambda u, taps, b: orig["causal_conv"](u, torch.cat([0 * taps[:, :1], taps[:, 1:]], 1), b)},
        "the gate branch without its activation": {"gelu_tanh": lambda z: z},
        "mix indexed the other way": {"spread_streams": lambda x, y, mix, out: orig["spread_streams"](x, y, mix.T, out)},
        "an expert without its clamp": {"expert": lambda h, g, u, d, limit: orig["expert"](h, g, u, d, 1e9)},
        "a choice without the correction": {"route": lambda h, w_, pre, f, forced=None: orig["route"](h, {**w_, pre + "correction": 0 * w_[pre + "correction"]}, pre, f, forced)},
    }
    if windows:
        cases["a window one longer"] = {"window_mask": lambda T, n: orig["window_mask"](T, n + 1 if n else 0)}
        cases["a window one shorter"] = {"window_mask": lambda T, n: orig["window_mask"](T, max(n - 1, 1) if n else 0)}
    if not moes:
        del cases["an expert without its clamp"], cases["a choice without the correction"]
    if all(l["mixer"]["conv"] == 1 for l in cfg["layers"] if l["type"] == "rglru"):
        del cases["the convolution without its oldest input"]
    if cfg["streams"] == 1:
        del cases["mix indexed the other way"]
    for name, patch in cases.items():
        with monkeypatch.context() as m:
            for k, v in patch.items():
                m.setattr(P, k, v)
            other = P.forward(cfg, w, t)[0]
        d = (other - base).abs().max(-1).values / base.abs().max()
        assert float(d.max()) > 1e-2, name
        assert int((d > 3e-3).sum()) >= 10, name
