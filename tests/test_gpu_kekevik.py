"""Kekevik decoders on the GPU against the plain implementation in ``layered_oracle`` (float64 on the CPU)."""
import io
import json

import layered_gpu as H
import layered_models as M
import layered_oracle as O
import numpy as np
import pytest
import torch
from layered_gpu import engine, feed, poison

pytestmark = pytest.mark.gpu

# median and worst row; H.TOL where a norm of something near zero amplifies rounding (a head of few values, an empty state)
TOL = {"f32": (2e-6, 5e-5), "bf16": (0.008, 0.03)}


def check(got, want, kv, what="", tol=TOL):
    H.check(got, want, kv, what, tol)


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    return M.Model(tmp_path_factory.mktemp("kekevik") / "mixed", M.kekevik_mixed(), seed=5)


@pytest.fixture(scope="module", params=["f32", "bf16"])
def mixed_engine(request, mixed):
    return request.param, engine(mixed, request.param)


# ---- row-wise steps ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("act", ["sigmoid", "silu"])
@pytest.mark.parametrize("first", [False, True])
@pytest.mark.parametrize("parts,width", [(3, 40), (1, 77), (4, 512), (1, 2080), (2, 5000)])
def test_gated_norm(parts, width, first, act):
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(width)
    n, T, eps = parts * width, 7, 1e-3
    o, gate, w = torch.randn(T, n, generator=g), torch.randn(T, n + 8, generator=g) * 2, torch.randn(n, generator=g)
    a = {"sigmoid": torch.sigmoid, "silu": O.silu}[act](gate[:, 4:4 + n].double())
    v = o.double() * a if first else o.double()
    for weight in (w, None):
        want = O.grouped_rms(v, parts, eps) * 1.7 * (1.0 if first else a) * (1.0 if weight is None else w.double())
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 0.02)):
            out = torch.zeros(T, n, dtype=dtype, device="cuda")
            L.gated_norm(o.cuda(), 2, gate.cuda(), 4, None if weight is None else w.cuda(), eps, T - 2, parts, width, out, act, first, 1.7)
            assert float(((out.cpu().double() - want)[2:] / (want.abs()[2:] + 1)).abs().max()) < tol and float(out[:2].abs().max()) == 0


@pytest.mark.parametrize("width", [40, 77, 1024, 5002])
def test_norms_around_a_sublayer(width):
    """x += norm(y) w, and the next input: x itself or its norm; likewise behind the embedding."""
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(width)
    T, eps, ld = 5, 1e-4, L.round_up(width, 128)
    x0, y, w, w2 = (torch.randn(*s, generator=g) for s in ((T, width), (T, L.round_up(width, 4)), (width,), (width,)))
    table = torch.randn(9, width, generator=g).bfloat16()
    tokens = torch.tensor([3, 0, 8, 3, 1], dtype=torch.int32)
    want = x0.double() + O.rms_norm(y[:, :width].double(), w.double(), eps)
    emb = table[tokens.long()].double() * 2.5
    for nxt in (None, w2):
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 0.02)):
            for src, target in (("add", want), ("embed", emb)):
                x, h = x0.cuda(), torch.zeros(T, ld, dtype=dtype, device="cuda")
                n = None if nxt is None else nxt.cuda()
                if src == "add":
                    L.norm_add(x, y.cuda(), w.cuda(), eps, T, h, n)
                else:
                    L.embed(table.cuda(), tokens.cuda(), 2.5, T, width, x, h, n, eps)
                assert float((x.cpu().double() - target).abs().max()) < 1e-5
                wh = target if nxt is None else O.rms_norm(target, w2.double(), eps)
                assert float(((h.cpu().double()[:, :width] - wh) / (wh.abs() + 1)).abs().max()) < tol and float(h[:, width:].abs().sum()) == 0


# ---- each mechanism alone -----------------------------------------------------------------------------------------------------------
ALONE = {
    "retention": lambda: [M.retention()],
    "retention, part of the head rotated": lambda: [M.retention(2, 36, 70, 50.0, 10)],
    "retention, nothing rotated": lambda: [M.retention(2, 16, 130, dims=0)],
    "lightning": lambda: [M.lightning()],
    "attention": lambda: [M.parallel(scales=(1.1, 0.0))],
    "attention, values wider than keys": lambda: [M.parallel(M.capped(8, 1, 20, 100, 0.4, 2.0, 2.0, 1), scales=(0.4, 0.0))],
    "state space": lambda: [M.parallel(scales=(0.0, 0.9))],
    "state space, one tap": lambda: [M.parallel(right=M.ssd(4, 40, 64, 4, 1, 1), scales=(0.0, 2.0))],
    "state space, seven taps": lambda: [M.parallel(right=M.ssd(3, 7, 13, 3, 7, 7), scales=(0.0, 1.0))],
    "feed-forward": lambda: [M.retention(ff=333)],
}
CUTS = {"whole": [], "twos": [2] * 20 + [3] * 5, "ones": [1] * 40, "mixture": [5, 1, 1, 64, 1, 63, 2, 65, 1], "decode": [100] + [1] * 100}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", ALONE)
def test_alone(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.kekevik(ALONE[name](), width=88, vocab=120), seed=len(name))
    eng = engine(m, kv, max_batch=2)
    tokens = m.tokens(205)
    want = m.logits(tokens)
    for n, cuts in CUTS.items():
        poison(eng)
        check(feed(eng, tokens, cuts, slot=1), want, kv, what=f"{name}, {n}")


# ---- the whole design: portions, batches, generation ---------------------------------------------------------------------------------
@pytest.mark.parametrize("cuts", CUTS)
def test_portions(mixed, mixed_engine, cuts):
    kv, eng = mixed_engine
    tokens = mixed.tokens(260, seed=len(cuts))
    poison(eng)
    check(feed(eng, tokens, CUTS[cuts]), mixed.logits(tokens), kv, what=cuts)


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5])
def test_first_tokens(mixed, mixed_engine, n):
    kv, eng = mixed_engine
    tokens = mixed.tokens(n, seed=n)
    for cuts in ([], [1] * n, [2]):
        poison(eng)
        check(feed(eng, tokens, cuts, slot=2), mixed.logits(tokens), kv, what=f"{n} tokens, {cuts}")


def test_batches_match_single_requests(mixed, mixed_engine):
    kv, eng = mixed_engine
    H.run_unequal_requests(mixed, eng, kv, TOL)


def test_the_cut_and_the_company_only_round(mixed, mixed_engine):
    """One position computed in several ways: as part of a prompt, decoded alone, decoded beside others."""
    kv, eng = mixed_engine
    a, b, c = mixed.tokens(150, 1), mixed.tokens(97, 2), mixed.tokens(40, 3)
    alone = feed(eng, a, [149])[149]
    for slot, toks in ((0, b[:96]), (2, a[:149]), (3, c[:10])):
        eng.reserve(slot, len(toks) + 31)
        eng.feed([(slot, toks, 0)], [[]])
    out = eng.feed([(3, c[10:40], 10), (0, b[96:], 96), (2, a[149:], 149)], [[29], [0], [0]])
    for s in (0, 2, 3):
        eng.close_sequence(s)
    want = [mixed.logits(c)[39], mixed.logits(b)[96], mixed.logits(a)[149]]
    check(out, torch.stack(want), kv)
    check(out[2:], alone.cpu()[None], kv)
    check(feed(eng, a, [])[149:], alone.cpu()[None], kv)


# ---- things that random weights would hide ---------------------------------------------------------------------------------------------
MARK, ASK = 7, 11


def plain_tokens(m, n, seed=1):
    return [t if t not in (MARK, ASK) else 1 for t in m.tokens(n, seed)]


def standout(w):
    """Token ASK's queries match token MARK's keys: whether a MARK is seen shows."""
    k = w["l0.mix.left.k"]
    H, G, d = w["l0.mix.left.q"].shape[0], k.shape[0], w["l0.mix.left.q"].shape[1]
    dim = 36
    w["l0.mix.left.q"] = -k.view(G // dim, 1, dim, d).expand(-1, H // G, -1, -1).reshape(H, d).clone()
    w["embed"][MARK] = -w["embed"][ASK]


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("group", [1, 4])
def test_far_keys(tmp_path, kv, group):
    """One key that stands out, hundreds of tokens back and at page borders, asked for in a prompt and in decoding."""
    cfg = M.kekevik([M.parallel(M.capped(2 * group, 2, 36, 36, 0.6, 40.0, 0.1, 50), scales=(1.0, 0.1))], vocab=60, width=64)
    m = M.Model(tmp_path / "m", cfg, seed=9, tweak=standout)
    eng = engine(m, kv, max_batch=1)
    for ask, marks in ((330, (0, 1, 63, 64, 65, 127, 128, 255, 256, 319, 320, 329)), (128, (0, 64, 127)), (64, (0, 63)), (2, (0, 1))):
        base = plain_tokens(m, ask + 3)
        base[ask] = ASK
        nothing = m.logits(base)[ask]
        for mark in marks:
            tokens = list(base)
            tokens[mark] = MARK
            want = m.logits(tokens)
            assert float((want[ask] - nothing).abs().max()) > 0.5
            poison(eng)
            for cuts in ([], [ask] + [1] * 3, [mark + 1, 2]):
                check(feed(eng, tokens, cuts), want, kv, what=f"mark {mark}, ask {ask}, cuts {cuts}")


def rows_are_close(a, b, tol):
    d = a - b
    d = d - d.mean()
    return float(d.pow(2).mean().sqrt() / (b - b.mean()).pow(2).mean().sqrt()) < tol


def test_query_temperature_and_cap_show(tmp_path):
    """The step of the temperature at a multiple of ``every`` and the cap are visible in the reference, so the comparison sees them."""
    left = M.capped(2, 1, 36, 36, 0.5, 3.0, 9.0, 50)
    m = M.Model(tmp_path / "m", M.kekevik([M.parallel(left, scales=(1.0, 0.0))], vocab=60, width=64, scale=1.0), seed=3)
    tokens = m.tokens(120)
    want = m.logits(tokens)
    for key, value in (("softcap", 1e3), ("q_temp", {"coef": 9.0, "every": 51})):
        other = M.kekevik([M.parallel({**left, key: value}, scales=(1.0, 0.0))], vocab=60, width=64, scale=1.0)
        moved = O.forward(other, m.w, tokens)
        assert not rows_are_close(moved[49], want[49], 0.1)
        if key == "q_temp":
            assert rows_are_close(moved[48], want[48], 1e-6) and rows_are_close(moved[50], want[50], 1e-6)
    for kv in ("f32", "bf16"):
        eng = engine(m, kv, max_batch=1)
        for cuts in ([], [48] + [1] * 4, [49, 2], [98, 1, 1, 1]):
            check(feed(eng, tokens, cuts), want, kv, what=str(cuts))


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("kind", ["retention", "lightning", "ssd"])
def test_state_carries_far(tmp_path, kind, kv):
    """Heads that hardly forget and keys that one token alone makes large: a MARK near the start decides the output hundreds of
    tokens on, across chunks, portions and decoding."""
    layer = {"retention": M.retention(2, 30, 20, 1e4, 4, [0.9999, 1.0]), "lightning": M.lightning(2, 30, 20, [1.0, 0.9995]),
             "ssd": M.parallel(right=M.ssd(2, 20, 30, 1, 1, 4), scales=(0.0, 1.0))}[kind]

    def tweak(w):
        w["embed"] *= 0.1                                            # what the layer adds stays visible in the sum
        p = "l0.mix.right." if kind == "ssd" else "l0.mix."
        g = torch.Generator().manual_seed(1)
        rows = torch.randn(30 if kind == "ssd" else 60, 1, generator=g)
        e = w["embed"][MARK] / w["embed"][MARK].norm()
        others = torch.arange(70) != MARK
        w["embed"][others] -= 0.8 * (w["embed"][others] @ e)[:, None] * e[None, :]
        key = rows * (2.0 * e / w["l0.norm1"])[None, :]              # (the input's part along MARK) times a random key
        if kind == "ssd":
            w[p + "in"][80:110] = key
            w[p + "A_log"] = torch.tensor([-9.0, -7.0])
            w[p + "D"] *= 0.1
        else:
            w[p + "k"] = key
    m = M.Model(tmp_path / "m", M.kekevik([layer], vocab=70, width=256, scale=1.0), seed=2, tweak=tweak)
    tokens = plain_tokens(m, 330)
    plain = m.logits(tokens)
    tokens[3] = MARK
    want = m.logits(tokens)
    assert not rows_are_close(want[320], plain[320], 0.15) and not rows_are_close(want[64], plain[64], 0.15)
    eng = engine(m, kv, max_batch=1)
    for cuts in ([], [1] * 20 + [64, 1, 63], [300] + [1] * 30, [2] * 5 + [3] * 30):
        check(feed(eng, tokens, cuts), want, kv, str(cuts[:3]), H.TOL)


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_convolution_window(tmp_path, kv):
    """A channel input that stands out reaches exactly the next taps - 1 tokens, whichever way the portions are cut."""
    taps = 5

    def tweak(w):
        p = "l0.mix.right."
        w[p + "A_log"] = torch.full((2,), 5.0)                       # the state forgets at once: only the convolution reaches back
        w[p + "dt_bias"] = torch.full((2,), 3.0)
        w["embed"][MARK] *= 3.0
    m = M.Model(tmp_path / "m", M.kekevik([M.parallel(right=M.ssd(2, 20, 30, 1, 1, taps), scales=(0.0, 1.0))], vocab=70, width=64, scale=1.0), seed=6, tweak=tweak)
    eng = engine(m, kv, max_batch=1)
    for mark in (0, 62, 66):
        tokens = plain_tokens(m, 90)
        base = m.logits(tokens)
        tokens[mark] = MARK
        want = m.logits(tokens)
        for back in range(1, taps + 2):
            assert rows_are_close(want[mark + back], base[mark + back], 0.1) == (back >= taps)
        for cuts in ([], [mark + 1] + [1] * 8, [mark + 1, 2, 2, 2, 2], [mark + 2, 3], [mark + 4, 1, 1, 2]):
            poison(eng)
            check(feed(eng, tokens, cuts), want, kv, f"mark {mark}, cuts {cuts}", H.TOL)


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_fast_decays(tmp_path, kv):
    """Decays down to nothing, and steps so long that a token wipes the state, beside ones that keep it.  A head that forgets at once
    gives (q . k) v, whose norm keeps little but a sign; the wide eps takes that edge off."""
    layers = [M.retention(3, 20, 30, decay=[0.0, 1e-30, 0.3]), M.lightning(2, 20, 30, decay=[0.0, 1e-4]), M.parallel(right=M.ssd(3, 20, 24, 1, 1, 2))]

    def tweak(w):
        w["l2.mix.right.A_log"] = torch.tensor([4.0, 1.0, -3.0])
        w["l2.mix.right.dt_bias"] = torch.tensor([5.0, -8.0, 6.0])
    m = M.Model(tmp_path / "m", M.kekevik(layers, vocab=70, width=64, eps=0.03), seed=12, tweak=tweak)
    eng = engine(m, kv, max_batch=1)
    tokens = m.tokens(200)
    want = m.logits(tokens)
    for cuts in ([], [70, 2, 1, 1, 60], [1] * 30):
        check(feed(eng, tokens, cuts), want, kv, what=str(cuts[:3]))


@pytest.mark.parametrize("d,e", [(20, 70), (100, 40), (200, 66)])
def test_long_prompts_in_segments(tmp_path, d, e):
    """Prompts long enough for the recurrences to be cut into segments, from position 0 and from a state, alone and together."""
    from oxibonsai_b200.models.layered import plan_segments
    layers = [M.retention(2, d, e, decay=[0.998, 0.9]), M.parallel(M.capped(2, 1, 16, 16), M.ssd(2, e, d, 1, 1, 4))]
    m = M.Model(tmp_path / "m", M.kekevik(layers, vocab=70, width=64), seed=d, tweak=lambda w: w["l1.mix.right.A_log"].copy_(torch.tensor([-5.0, -2.0])))
    eng = engine(m, "bf16", max_batch=3, max_seq=1024, chunk=2048)
    poison(eng)
    tokens = m.tokens(900)
    want = m.logits(tokens)
    assert eng.runner.segment_plans and all(plan_segments(n, p, 148) for p in eng.runner.segment_plans for n in ([900], [600, 700]))
    check(feed(eng, tokens, []), want, "bf16", "whole")
    check(feed(eng, tokens, [77, 700, 2]), want, "bf16", "resumed")
    for s, n in ((0, 601), (1, 1), (2, 901)):
        eng.reserve(s, n)
    eng.feed([(2, tokens[:200], 0)], [[]])
    out = eng.feed([(0, tokens[:600], 0), (1, tokens[:1], 0), (2, tokens[200:], 200)], [list(range(600)), [0], list(range(700))])
    check(out, torch.cat([want[:600], want[:1], want[200:]]), "bf16", "together")
    check(eng.feed([(0, tokens[600:601], 600), (2, [5], 900)], [[0], []]), want[600:601], "bf16", "decode after")


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_long_decoding(tmp_path, kv):
    m = M.Model(tmp_path / "m", M.kekevik([M.parallel(M.capped(2, 1, 24, 24), M.ssd(2, 16, 16, 1, 1, 4), ff=64), M.retention(2, 16, 24)], vocab=70, width=64), seed=8)
    eng = engine(m, kv, max_batch=1, max_seq=640)
    poison(eng)
    tokens = m.tokens(600)
    check(feed(eng, tokens, [3] + [1] * 597), m.logits(tokens), kv)


# ---- other sizes --------------------------------------------------------------------------------------------------------------------------
SIZES = {
    "one head each": [M.retention(1, 16, 16, ff=33), M.lightning(1, 8, 8), M.parallel(M.capped(1, 1, 8, 8), M.ssd(1, 8, 8, 1, 1, 2), ff=5)],
    "many query heads": [M.parallel(M.capped(40, 2, 8, 16), M.ssd(12, 8, 16, 4, 6, 4))],
    "wide heads": [M.parallel(M.capped(2, 1, 256, 200, 0.05), M.ssd(2, 128, 256, 2, 4, 4)), M.retention(2, 256, 256, 1e6)],
    "three quarters": [M.parallel(M.capped(3, 3, 96, 64, 0.1), M.ssd(2, 96, 72, 1, 1, 3)), M.parallel(M.capped(4, 2, 130, 192, 0.07), M.ssd(2, 66, 128, 2, 2, 4), ff=31)],
    "long keys, many values": [M.retention(1, 300, 600, dims=300), M.lightning(2, 400, 520), M.parallel(M.capped(2, 2, 17, 33), M.ssd(1, 530, 270, 1, 5, 2))],
    "nothing even": [M.retention(3, 13, 7, dims=6, ff=21), M.lightning(7, 11, 5), M.parallel(M.capped(9, 3, 11, 9), M.ssd(3, 5, 11, 3, 5, 3), ff=5)],
    "parts across heads": [M.parallel(M.capped(2, 1, 16, 16), M.ssd(3, 20, 16, 1, 2, 4)), M.lightning(4, 64, 64), M.retention(4, 128, 64, ff=64)],
}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", SIZES)
def test_sizes(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.kekevik(SIZES[name], width={"wide heads": 264, "nothing even": 75}.get(name, 72), vocab=97, eps=1e-6, scale=1.5), seed=len(name))
    eng = engine(m, kv, max_batch=2)
    poison(eng)
    tokens = m.tokens(140)
    want = m.logits(tokens)
    for cuts in ([], [66, 1, 2, 1], [1] * 5 + [80] + [1] * 60):
        check(feed(eng, tokens, cuts, slot=1), want, kv, f"{name} {cuts[:4]}", H.TOL if name in ("one head each", "nothing even") else TOL)


# ---- generation through the framework's entry points -----------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def sharp(tmp_path_factory):
    """A model whose logits are far enough apart for greedy generation to be the same in both modes."""
    return M.Model(tmp_path_factory.mktemp("kekevik") / "sharp", M.kekevik_mixed(), seed=31, tweak=lambda w: w["final.norm"].mul_(3.0))


def test_greedy_generation_matches_oracle(sharp):
    eng = engine(sharp, "f32")
    prompts = [sharp.tokens(n, seed=n) for n in (1, 5, 70)]
    want = [sharp.greedy(p, 8)[0] for p in prompts]
    assert [eng.generate(p, 8) for p in prompts] == want
    assert eng.generate_batch(prompts, 8) == want
    info = eng.model_info()
    assert info["arch"] == "Kekevik" and info["recurrent_layers"] == 6 and info["attention_layers"] == 2
    eng.runner.check_status()


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_scheduler_generation(sharp, kv):
    """Continuous batching with prompts that ride in decode steps: every request as if it were alone."""
    from oxibonsai_b200.runtime.presets import SamplingPreset
    from oxibonsai_b200.runtime.scheduler import BatchScheduler
    eng = engine(sharp, kv, max_batch=3, pages=12)
    poison(eng)
    prompts = [sharp.tokens(n, seed=n) for n in (6, 90, 33, 1, 150, 64, 2)]
    counts = [20, 8, 15, 25, 3, 9, 12]
    alone = engine(sharp, kv, max_batch=1)
    want = [alone.generate(p, k) for p, k in zip(prompts, counts)]
    sched = BatchScheduler(eng, prefill_chunk_tokens=32)
    reqs = [sched.submit(p, SamplingPreset.GREEDY.params(), k) for p, k in zip(prompts, counts)]
    sched.start()
    got = [r.wait(timeout=120) for r in reqs]
    sched.stop()
    assert sched.mixed_steps > 0 and len(eng.kv.free_pages) == 12 and len(eng.runner.states.free_rows) == 3
    if kv == "f32":
        assert got == want
    for p, g in zip(prompts, got):           # in 16 bits a near tie may fall the other way: the chosen logits are near the best ones
        lg = sharp.logits(p + g)[len(p) - 1:-1]
        chosen = lg[torch.arange(len(g)), torch.tensor(g)]
        assert float((lg.max(-1).values - chosen).max()) < 0.1 * float(lg.std())


def test_unsupported_features_are_refused(sharp):
    eng = engine(sharp, "bf16")
    assert not eng.supports_prefix_cache
    with pytest.raises(ValueError):
        eng.enable_prefix_cache()
    with pytest.raises(NotImplementedError):
        eng.verify_greedy([1, 2], 0)


def test_trace_replay(mixed, mixed_engine, tmp_path):
    from oxibonsai_b200.runtime.trace import replay
    kv, eng = mixed_engine
    a, b = mixed.tokens(80, 3), mixed.tokens(30, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:29], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:52], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[29:], "want": [0]}, {"id": "a", "tokens": a[52:], "want": [27]}], "end": ["a", "b"]}]
    assert replay(eng, [json.dumps(s) for s in steps], str(tmp_path), io.StringIO()) == 3
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).view(-1, mixed.cfg["vocab"])
    la, lb = mixed.logits(a), mixed.logits(b)
    check(read(0), la[[0, 49]], kv)
    check(read(1), la[[51]], kv)
    check(read(2), torch.stack([lb[29], la[79]]), kv)
    assert len(eng.kv.free_pages) == eng.kv.num_pages and len(eng.runner.states.free_rows) == 4
