"""Kutepel decoders on the GPU against the plain implementation in ``layered_oracle`` (float64 on the CPU)."""
import io
import json

import layered_gpu as H
import layered_models as M
import layered_oracle as O
import numpy as np
import pytest
import torch
from layered_gpu import engine, feed

pytestmark = pytest.mark.gpu

TOL = {"f32": (2e-6, 5e-5), "bf16": (0.008, 0.03)}      # median and worst row
NAN = float("nan")


def check(got, want, kv, what="", tol=TOL):
    H.check(got, want, kv, what, tol)


def poison(eng):
    """Cache and scratch that a step must write before it reads them."""
    H.poison(eng)
    r = eng.runner
    r.expanded.fill_(NAN)
    for q, part, ml in r._absorbed.values():
        for t in (q, part, ml):
            t.fill_(NAN)
    for e in r.experts.values():
        e.s.out.fill_(NAN)


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    return M.Model(tmp_path_factory.mktemp("kutepel") / "mixed", M.kutepel_mixed(), seed=5)


@pytest.fixture(scope="module", params=["f32", "bf16"])
def mixed_engine(request, mixed):
    return request.param, engine(mixed, request.param)


# ---- row-wise steps ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [40, 77, 1024, 5002])
def test_sublayers_side_by_side(width):
    """x += mult * (y + the token's expert rows) and the next input; likewise behind the embedding and for selected rows."""
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(width)
    T, top, eps, ld = 6, 3, 1e-4, L.round_up(width, 128)
    x0, y, w = torch.randn(T, width, generator=g) + 0.7, torch.randn(T, L.round_up(width, 4), generator=g), torch.randn(width, generator=g)
    rows = torch.randn(T * top, L.round_up(width, 8), generator=g).bfloat16()
    at = torch.randperm(T * top, generator=g).int()
    table, tokens = (torch.randn(9, width, generator=g) + 0.5).bfloat16(), torch.tensor([3, 0, 8, 3, 1, 2], dtype=torch.int32)

    class Rows:
        def __init__(self, e):
            self.e, self.at, self.counts = e.cuda(), at.cuda(), torch.ones(70, dtype=torch.int32, device="cuda")
            self.outputs = (self.e.data_ptr(), self.e.stride(0), int(e.dtype == torch.float32), self.at.data_ptr(), top, self.counts.data_ptr(), 70)
    plain = x0.double() + 0.3 * y[:, :width].double()
    with_rows = plain + 0.3 * rows[at.long()].view(T, top, -1)[..., :width].double().sum(1)
    norm = {True: O.layer_norm, False: O.rms_norm}
    for center in (True, False):
        for nxt in (None, w):
            for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 0.02)):
                for e, want in ((None, plain), (rows, with_rows), (rows.float(), with_rows), ("embed", table[tokens.long()].double() * 2.5)):
                    x, h, n = x0.cuda(), torch.zeros(T, ld, dtype=dtype, device="cuda"), None if nxt is None else nxt.cuda()
                    if isinstance(e, str):
                        L.embed(table.cuda(), tokens.cuda(), 2.5, T, width, x, h, n, eps, center)
                    else:
                        r = None if e is None else Rows(e)
                        L.side_by_side(x, y.cuda(), r, 0.3, T, h, n, eps, center)
                        assert r is None or int(r.counts.abs().sum()) == 0
                    assert float((x.cpu().double() - want).abs().max()) < 1e-5
                    wh = want if nxt is None else norm[center](want, w.double(), eps)
                    assert float(((h.cpu().double()[:, :width] - wh) / (wh.abs() + 1)).abs().max()) < tol and float(h[:, width:].abs().sum()) == 0
        out, pick = torch.zeros(2, ld, device="cuda"), torch.tensor([4, 1], dtype=torch.int32, device="cuda")
        L.norm_rows(x0.cuda(), pick.data_ptr(), 2, w.cuda(), eps, out, center)
        assert float((out.cpu().double()[:, :width] - norm[center](x0.double(), w.double(), eps)[[4, 1]]).abs().max()) < 2e-5


# ---- the router and the experts ------------------------------------------------------------------------------------------------------
def routing(E, top, groups, keep, ff, width, rows, exact, seed=0, scale=1.3, correction=None):
    """One expert layer on its own: (call, logits buffer, weights in float64)."""
    from oxibonsai_b200.models.layered_config import ExpertsSpec, RouterSpec
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(seed)
    dev = torch.device("cuda")
    w = {f"e{e}.{n}": (torch.randn(s, generator=g) * s[1] ** -0.5).bfloat16() for e in range(E) for n, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    spec = ExpertsSpec(RouterSpec(E, top, groups, keep, scale), ff)
    up = L.DenseWeight([torch.cat([w[f"e{e}.{c}"] for e in range(E)]) for c in ("gate", "up")], dev, interleave=True)
    down = L.DenseWeight([torch.cat([w[f"e{e}.down"] for e in range(E)])], dev)
    c = 0.4 * torch.randn(E, generator=g) - 0.4 if correction is None else correction
    logits = torch.zeros(rows, L.round_up(E, 4) + 8, device=dev)
    r = L.Routing(spec, up, down, c.cuda(), logits, 4, L.ExpertScratch(rows, width, [spec], exact, dev))
    return r, logits, {**{k: v.double() for k, v in w.items()}, "correction": c.double()}


ROUTERS = [(5, 2, 1, 1), (16, 2, 4, 3), (33, 5, 11, 4), (64, 8, 8, 4), (130, 6, 13, 2), (260, 32, 4, 1), (512, 8, 16, 5), (12, 4, 12, 7), (6, 6, 1, 1), (1, 1, 1, 1), (8, 4, 2, 1)]


@pytest.mark.parametrize("E,top,groups,keep", ROUTERS)
def test_router_chooses_and_sorts(E, top, groups, keep):
    r, logits, w = routing(E, top, groups, keep, 8, 16, 300, False)
    from oxibonsai_b200.ops import layered_ops as L
    scratch = L.GemmScratch(torch.device("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    h = torch.randn(300, 128, device="cuda").bfloat16()
    for T in (1, 2, 31, 64, 65, 300):
        z = 2.0 * torch.randn(T, E, generator=torch.Generator().manual_seed(T))
        logits.fill_(NAN)
        logits[:T, 4:4 + E] = z.cuda()
        r(h, T, scratch)
        r.s.counts.zero_()
        at, token, weight = (t[: T * top].cpu() for t in (r.s.at, r.s.token, r.s.weight))
        offsets, chosen = r.s.lists[: E + 1].cpu().tolist(), int(r.s.lists[E + 1])
        active = r.s.lists[E + 2:E + 2 + chosen].cpu().tolist()
        assert sorted(at.tolist()) == list(range(T * top)) and offsets[0] == 0 and offsets[-1] == T * top
        owner = torch.bucketize(torch.arange(T * top), torch.tensor(offsets[1:]), right=True)
        assert active == sorted(set(owner.tolist()))
        for t in range(T):
            pairs = at[t * top:(t + 1) * top].long()
            want, ww = O.route(z[t].double(), w["correction"], top, groups, keep, 1.3)
            assert owner[pairs].tolist() == want and torch.equal(token[pairs], torch.full((top,), t, dtype=torch.int32))
            assert torch.allclose(weight[pairs].double(), ww, rtol=2e-5)


@pytest.mark.parametrize("exact", [True, False])
@pytest.mark.parametrize("E,top,ff,width", [(6, 2, 40, 72), (9, 3, 130, 264), (40, 4, 64, 128), (3, 2, 200, 600)])
def test_experts(E, top, ff, width, exact):
    """Few and many rows per expert, even and uneven shares (one expert with all tokens, others with none)."""
    from oxibonsai_b200.ops import layered_ops as L
    scratch = L.GemmScratch(torch.device("cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"))
    ways = set()
    for case in ("even", "uneven"):
        c = torch.zeros(E) if case == "even" else torch.cat([torch.full((top - 1,), 9.0), torch.full((1,), 5.0), torch.full((E - top,), 0.0)])
        c[-1] = -9.0
        r, logits, w = routing(E, top, 1, 1, ff, width, 900, exact, seed=E, correction=c)
        for T in (1, 5, 32, 33, 260, 900):
            g = torch.Generator().manual_seed(T)
            z = torch.randn(T, E, generator=g)
            logits.fill_(NAN)
            logits[:T, 4:4 + E] = z.cuda()
            act = torch.randn(T, width, generator=g).bfloat16()
            h = torch.zeros(900, L.round_up(width, 128), device="cuda", dtype=torch.float32 if exact else torch.bfloat16)
            h[:T, :width] = act.cuda().to(h.dtype)
            r.s.out.fill_(NAN)
            r(h, T, scratch)
            x = torch.zeros(T, width, device="cuda")
            L.side_by_side(x, torch.zeros(T, L.round_up(width, 4), device="cuda"), r, 1.0, T, None, None, 1e-5, True)
            want, a = torch.zeros(T, width, dtype=torch.float64), act.double()
            choice = [O.route(z[t].double(), w["correction"], top, 1, 1, 1.3) for t in range(T)]
            for e in range(E):
                mine = [(t, wt[ids.index(e)]) for t, (ids, wt) in enumerate(choice) if e in ids]
                if mine:
                    rows = torch.tensor([t for t, _ in mine])
                    want[rows] += O.expert(a[rows], w, f"e{e}.") * torch.stack([f for _, f in mine])[:, None]
            err = (x.cpu().double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
            assert float(err.max()) < (2e-6 if exact else 0.012), (case, T, float(err.max()))
            ways.add("f32" if exact else ("few" if r.few(T) else ("wide" if T * top > 96 * E else "narrow")))
    assert int(scratch.status) == 0
    assert ways == ({"f32"} if exact else {"few", "wide", "narrow"} if E < 40 else {"few", "narrow"})


# ---- each mechanism alone -----------------------------------------------------------------------------------------------------------
ALONE = {
    "latent": lambda: [M.latent()],
    "latent, stretched": lambda: [M.latent(2, 8, 40, 33, 20, 0.4, 300.0, M.STRETCH)],
    "latent, seventeen heads": lambda: [M.latent(17, 12, 4, 9, 40)],
    "latent, forty heads": lambda: [M.latent(40, 4, 2, 6, 200, 0.5)],
    "attention": lambda: [M.rotary()],
    "attention, part of the head rotated": lambda: [M.rotary(8, 1, 20, 100, 0.4, 6, 30.0, M.STRETCH)],
    "attention, nothing rotated": lambda: [M.rotary(3, 3, 16, 16, 0.3, 0)],
    "shared keys": lambda: [M.rotary(4, 2), M.rotary(8, 2, kv_from=0, dims=12), M.rotary(2, 2, 16, 72), M.rotary(2, 2, kv_from=0, scaling=M.STRETCH)],
    "experts": lambda: [M.rotary(2, 1, 16, 16, mlp=M.experts(50, 9, 2, 3, 1, 1.5))],
    "experts, all of them": lambda: [M.rotary(2, 1, 16, 16, mlp=M.experts(20, 4, 4, 2, 2, 0.5))],
    "one expert": lambda: [M.latent(2, 16, 8, 16, 24, mlp=M.experts(70, 1, 1, 1, 1, 2.0))],
}
CUTS = {"whole": [], "twos": [2] * 20 + [3] * 5, "ones": [1] * 40, "mixture": [5, 1, 1, 64, 1, 63, 2, 65, 1], "decode": [100] + [1] * 100,
        "around the short limit": [31, 32, 33, 34, 2, 33]}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", ALONE)
def test_alone(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.kutepel(ALONE[name](), width=88, vocab=120), seed=len(name))
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


def test_layers_leave_the_stream_of_the_oracle(mixed, tmp_path):
    """Models of the first layers only: the residual stream itself, through an identity in place of the head."""
    for n in (1, 2, 4):
        cfg = {**M.kutepel_mixed(), "layers": mixed.cfg["layers"][:n]}
        m = M.Model(tmp_path / str(n), cfg, seed=n)
        eng = engine(m, "f32", max_batch=1)
        tokens = m.tokens(70)
        _, kept = O.forward(m.cfg, m.w, tokens, True)
        feed(eng, tokens, [])
        got = eng.runner.x[:70].cpu().double()
        assert float((got - kept[-1]).abs().max()) < 2e-5 * float(kept[-1].abs().max())


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


def test_contexts_in_several_groups(mixed):
    """Long portions whose cached tokens exceed the expansion scratch together, short ones beyond its rows, and decoded tokens."""
    eng = engine(mixed, "bf16", max_batch=14, pages=90)
    poison(eng)
    r = eng.runner
    toks = {s: mixed.tokens(360, seed=s) for s in range(14)}
    want = {s: mixed.logits(toks[s]) for s in (0, 1, 2)}
    for s in range(14):
        eng.reserve(s, 360 if s < 3 else 90)
    for s in (0, 1, 2):
        eng.feed([(s, toks[s][:300], 0)], [[]])
    eng.feed([(3, toks[3][:50], 0)], [[]])
    entries = [(s, toks[s][300:340], 300) for s in (2, 0, 1)] + [(3, toks[3][50:51], 50)] + [(s, toks[s][:30], 0) for s in range(4, 14)]
    assert 3 * 340 > r.context_rows and 1 + 10 * 30 > r.short_rows
    out = eng.feed(entries, [list(range(len(t))) for _, t, _ in entries]).split([len(t) for _, t, _ in entries])
    for (s, t, pos0), got in zip(entries, out):
        ref = want[s] if s in want else mixed.logits(toks[s][:pos0 + len(t)])
        check(got, ref[pos0:pos0 + len(t)], "bf16", f"slot {s}")
    out = eng.feed([(s, toks[s][340:341], 340) for s in (0, 1, 2)], [[0]] * 3)
    check(out, torch.stack([want[s][340] for s in (0, 1, 2)]), "bf16", "decoded after")


# ---- things that random weights would hide ---------------------------------------------------------------------------------------------
MARK, ASK = 7, 11


def plain_tokens(m, n, seed=1):
    return [t if t not in (MARK, ASK) else 1 for t in m.tokens(n, seed)]


def pointer(w, p, token):
    """Rows that read a token's embedding out of the layer's input, where it has length sqrt(width)."""
    e = w["embed"][token] - w["embed"][token].mean()
    return e / e.norm() / w[p + "norm1"]


def point_latent(w, l, dim, rot_dim, gain=1.2):
    """Token ASK's queries match the unrotated keys that token MARK's latent expands to."""
    p, H = f"l{l}.mix.", w[f"l{l}.mix.sink"].shape[0] if f"l{l}.mix.sink" in w else w[f"l{l}.mix.uk"].shape[0] // dim
    R = w[p + "uk"].shape[1]
    v = torch.randn(R, generator=torch.Generator().manual_seed(4))
    w[p + "dkv"][:R] += 0.3 * v[:, None] * pointer(w, f"l{l}.", MARK)[None, :]
    key = (w[p + "uk"] @ (v * w[p + "dkv.norm"])).view(H, dim)
    q = w[p + "q"].view(H, dim + rot_dim, -1)
    q[:, :dim] += gain * (key / key.norm(dim=1, keepdim=True))[:, :, None] * pointer(w, f"l{l}.", ASK)[None, None, :]


def point_heads(w, l, source, heads, kv_heads, dim, turned, gain=1.0):
    """The same with keys of their own (of layer ``source``), in the dimensions that are not rotated."""
    g = torch.Generator().manual_seed(5)
    dirs = torch.randn(kv_heads, dim, generator=g)
    dirs[:, :turned] = 0.0
    dirs /= dirs.norm(dim=1, keepdim=True)
    w[f"l{source}.mix.k"].view(kv_heads, dim, -1).add_(gain * dirs[:, :, None] * pointer(w, f"l{source}.", MARK)[None, None, :])
    q = w[f"l{l}.mix.q"].view(kv_heads, heads // kv_heads, dim, -1)
    q.add_(gain * dirs[:, None, :, None] * pointer(w, f"l{l}.", ASK)[None, None, None, :])


FAR = {
    "latent": (lambda: [M.latent(4, 24, 4, 30, 40, 0.5, 50.0)], lambda w: point_latent(w, 0, 24, 4)),
    "latent, twenty heads": (lambda: [M.latent(20, 24, 4, 10, 140, 0.5, 50.0)], lambda w: point_latent(w, 0, 24, 4)),
    "attention": (lambda: [M.rotary(2, 2, 36, 20, 0.3, 6, 50.0)], lambda w: point_heads(w, 0, 0, 2, 2, 36, 6)),
    "attention, groups of four": (lambda: [M.rotary(8, 2, 36, 20, 0.3, 6, 50.0, M.STRETCH)], lambda w: point_heads(w, 0, 0, 8, 2, 36, 6)),
    "shared keys": (lambda: [M.rotary(4, 2, 36, 20, 0.3, 6, 50.0), M.rotary(8, 2, 36, 20, 0.3, 6, 50.0, kv_from=0)],
                    lambda w: (w["l0.mix.o"].zero_(), w["l0.mix.q"].zero_(), point_heads(w, 1, 0, 8, 2, 36, 6))),
}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("kind", FAR)
def test_far_keys(tmp_path, kind, kv):
    """One key that stands out, hundreds of tokens back and at page borders, asked for in a prompt and in decoding."""
    layers, tweak = FAR[kind]
    m = M.Model(tmp_path / "m", M.kutepel(layers(), vocab=60, width=96, mult=1.0), seed=9, tweak=tweak)
    eng = engine(m, kv, max_batch=1)
    for ask, marks in ((330, (0, 1, 63, 64, 65, 127, 128, 255, 256, 319, 320, 329)), (128, (0, 64, 127)), (64, (0, 63)), (2, (0, 1))):
        base = plain_tokens(m, ask + 3)
        base[ask] = ASK
        nothing = m.logits(base)[ask]
        for mark in marks:
            tokens = list(base)
            tokens[mark] = MARK
            want = m.logits(tokens)
            assert float((want[ask] - nothing).abs().max()) > 0.4
            poison(eng)
            for cuts in ([], [ask] + [1] * 3, [mark + 1, 2], [max(1, ask - 20)]):
                check(feed(eng, tokens, cuts), want, kv, what=f"mark {mark}, ask {ask}, cuts {cuts}")


def apart(a, b):
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / (b - b.mean(-1, keepdim=True)).pow(2).mean().sqrt()).max())


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_sinks_show(tmp_path, kv):
    """Sinks from none to nearly everything, counted once however the keys are split; the reference without them is another model."""
    values = torch.tensor([-30.0, 0.0, 3.0, 6.0, 9.0, 30.0])
    m = M.Model(tmp_path / "m", M.kutepel([M.rotary(6, 2, 32, 40, 0.25)], vocab=90, width=96, mult=1.0), seed=3, tweak=lambda w: w["l0.mix.sink"].copy_(values))
    tokens = m.tokens(330)
    want = m.logits(tokens)
    for change, least in ((-1e9, 0.1), (1.0, 0.02)):
        w = dict(m.w)
        w["l0.mix.sink"] = w["l0.mix.sink"] + change
        assert apart(O.forward(m.cfg, w, tokens)[100:], want[100:]) > least
    eng = engine(m, kv, max_batch=1)
    for cuts in ([], [1] * 70 + [200], [270] + [1] * 60):
        poison(eng)
        check(feed(eng, tokens, cuts), want, kv, what=str(cuts[-2:]))


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_rotations_show(tmp_path, kv):
    """Pairing, base, stretch and the ramp matter to the reference at late positions, so the comparison sees them."""
    layers = [M.latent(3, 4, 24, 30, 40, 0.8, 400.0, M.STRETCH), M.rotary(4, 2, 24, 20, 0.8, 24, 400.0, M.STRETCH)]
    cfg = M.kutepel(layers, vocab=90, width=96, mult=1.0)
    m = M.Model(tmp_path / "m", cfg, seed=13)
    tokens = m.tokens(300)
    want = m.logits(tokens)
    for key, value in (("factor", 7.0), ("low", 2.5), ("high", 3.0), ("original", 60)):
        for l in (0, 1):
            other = json.loads(json.dumps(cfg))
            other["layers"][l]["mixer"]["rot"]["scaling"][key] = value
            assert apart(O.forward(other, m.w, tokens)[200:], want[200:]) > 0.05, (key, l)
    eng = engine(m, kv, max_batch=1)
    for cuts in ([], [250] + [1] * 50, [40] * 7):
        check(feed(eng, tokens, cuts), want, kv, what=str(cuts[:2]))


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_long_context(tmp_path, kv):
    """Decoding over several splits, prompts of many tiles, from position 0 and behind cached tokens."""
    m = M.Model(tmp_path / "m", M.kutepel([M.latent(4, 24, 8, 30, 40, 0.6, mlp=M.experts(16, 6, 2, 3, 2)), M.rotary(4, 2, 36, 20, 0.4), M.rotary(2, 2, 36, 20, 0.4, kv_from=1)],
                                          vocab=70, width=64), seed=8)
    eng = engine(m, kv, max_batch=3, max_seq=1024, chunk=1024)
    tokens = m.tokens(900)
    want = m.logits(tokens)
    assert kv == "f32" or eng.runner.mixers[0][0].splits(1) == (16, 8)
    for cuts in ([], [77, 700, 2], [860] + [1] * 40, [500, 33, 32, 1, 200]):
        poison(eng)
        check(feed(eng, tokens, cuts), want, kv, str(cuts[:3]))


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_long_decoding(tmp_path, kv):
    m = M.Model(tmp_path / "m", M.kutepel([M.latent(2, 16, 8, 16, 24, mlp=M.experts(32, 6, 2, 2, 1)), M.rotary(2, 1, 24, 24)], vocab=70, width=64), seed=8)
    eng = engine(m, kv, max_batch=1, max_seq=640)
    poison(eng)
    tokens = m.tokens(600)
    check(feed(eng, tokens, [3] + [1] * 597), m.logits(tokens), kv)


# ---- other sizes --------------------------------------------------------------------------------------------------------------------------
SIZES = {
    "as small as possible": [M.latent(1, 1, 2, 1, 1, 1.0, mlp=M.experts(1, 1, 1, 1, 1, 1.0)), M.rotary(1, 1, 2, 1, 1.0, mlp=M.experts(2, 2, 1, 2, 1))],
    "real heads": [M.latent(20, 128, 64, 128, 512, 0.07, 1e4, M.STRETCH), M.rotary(8, 2, 128, 128, 0.09, 128, 5e5, M.STRETCH)],
    "wide heads": [M.latent(16, 190, 64, 256, 300, 0.06), M.rotary(2, 1, 256, 200, 0.06), M.latent(2, 64, 62, 130, 400, 0.1), M.latent(2, 8, 128, 20, 512, 0.1)],
    "many heads": [M.latent(70, 8, 4, 5, 33), M.rotary(64, 1, 8, 16, mlp=M.experts(17, 70, 9, 10, 4))],
    "nothing even": [M.latent(3, 13, 6, 7, 11, mlp=M.experts(21, 9, 5, 3, 3)), M.rotary(9, 3, 11, 9, 0.3, 6, mlp=M.experts(5, 15, 2, 5, 2)), M.rotary(21, 3, 11, 9, 0.3, 4, kv_from=1)],
    "keys wider than values": [M.latent(4, 64, 32, 16, 64, 0.1), M.rotary(4, 2, 96, 16, 0.1)],
    "values wider than keys": [M.latent(4, 8, 8, 120, 96, 0.3), M.rotary(4, 2, 16, 120, 0.3)],
}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", SIZES)
def test_sizes(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.kutepel(SIZES[name], width={"wide heads": 264, "nothing even": 75}.get(name, 72), vocab=97, eps=1e-6, mult=0.7), seed=len(name))
    eng = engine(m, kv, max_batch=2)
    poison(eng)
    tokens = m.tokens(140)
    want = m.logits(tokens)
    for cuts in ([], [66, 1, 2, 1], [1] * 5 + [80] + [1] * 60):
        check(feed(eng, tokens, cuts, slot=1), want, kv, f"{name} {cuts[:4]}")


# ---- generation through the framework's entry points -----------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def sharp(tmp_path_factory):
    """A model whose logits are far enough apart for greedy generation to be the same in both modes."""
    return M.Model(tmp_path_factory.mktemp("kutepel") / "sharp", M.kutepel_mixed(), seed=31, tweak=lambda w: w["final.norm"].mul_(3.0))


def test_greedy_generation_matches_oracle(sharp):
    eng = engine(sharp, "f32")
    prompts = [sharp.tokens(n, seed=n) for n in (1, 5, 70)]
    want = [sharp.greedy(p, 8)[0] for p in prompts]
    assert [eng.generate(p, 8) for p in prompts] == want
    assert eng.generate_batch(prompts, 8) == want
    info = eng.model_info()
    assert info["arch"] == "Kutepel" and info["recurrent_layers"] == 0 and info["attention_layers"] == 7 and info["state_bytes"] == 0
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
    sched = BatchScheduler(eng, prefill_chunk_tokens=48)
    reqs = [sched.submit(p, SamplingPreset.GREEDY.params(), k) for p, k in zip(prompts, counts)]
    sched.start()
    got = [r.wait(timeout=120) for r in reqs]
    sched.stop()
    assert sched.mixed_steps > 0 and len(eng.kv.free_pages) == 12
    if kv == "f32":
        assert got == want
    for p, g in zip(prompts, got):           # in 16 bits a near tie may fall the other way: the chosen logits are near the best ones
        lg = sharp.logits(p + g)[len(p) - 1:-1]
        chosen = lg[torch.arange(len(g)), torch.tensor(g)]
        assert float((lg.max(-1).values - chosen).max()) < 0.1 * float(lg.std())


def test_prefix_cache(sharp):
    """A prompt whose first pages are cached continues from them, latents and shared keys included."""
    eng = engine(sharp, "f32", max_batch=1)
    cache = eng.enable_prefix_cache(4)
    prompt = sharp.tokens(150)
    want = sharp.greedy(prompt, 5)[0]
    assert eng.generate(prompt, 5) == want and eng.generate(prompt, 5) == want
    assert len(cache.lookup(prompt, max_tokens=149)) == 2


def test_step_counts_its_launches(mixed, monkeypatch):
    """A decode step of two sequences makes as many launches as it claims (each of its calls is one)."""
    from oxibonsai_b200.ops import cuda_ops as K
    eng = engine(mixed, "bf16", max_batch=2)
    r = eng.runner
    for s in (0, 1):
        eng.reserve(s, 80)
        eng.feed([(s, mixed.tokens(70, s), 0)], [[]])
    r.positions[:2].fill_(70)
    calls, check_call = [], K.check
    monkeypatch.setattr(K, "check", lambda rc, what: (calls.append(what), check_call(rc, what))[1])
    r.step_eager(2)
    torch.cuda.synchronize()
    assert len(calls) == r.kernel_launches(2) and calls.count("latent_decode") == 3 and calls.count("route") == 5


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
    assert len(eng.kv.free_pages) == eng.kv.num_pages
