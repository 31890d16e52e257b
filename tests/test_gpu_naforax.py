"""Naforax decoders on the GPU against the plain implementation in ``layered_oracle`` (float64 on the CPU)."""
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

TOL = {"f32": (3e-6, 6e-5), "bf16": (0.012, 0.05)}      # median and worst row
NAN = float("nan")


def check(got, want, kv, what="", tol=TOL):
    H.check(got, want, kv, what, tol)


def poison(eng):
    """Cache, state and scratch that a step must write before it reads them."""
    H.poison(eng)
    r = eng.runner
    for t in (*r.scan_scratch, r.n32, r.y, r.router_out):
        t.fill_(NAN)
    for x, bc, dt, low in r._scan_buffers.values():
        dt.fill_(NAN)
    for e in r.experts.values():
        e.s.out.fill_(NAN)


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    return M.Model(tmp_path_factory.mktemp("naforax") / "mixed", M.naforax_mixed(), seed=5)


@pytest.fixture(scope="module", params=["f32", "bf16"])
def mixed_engine(request, mixed):
    return request.param, engine(mixed, request.param)


class FakeRows:
    """Rows of a batch: (slot, first position, tokens) of each entry, single tokens first; every slot has the state row ``slot`` + 1."""

    def __init__(self, entries, vocab=9):
        from oxibonsai_b200.models.layered import StepShape
        from oxibonsai_b200.ops import layered_ops as L
        i32 = dict(dtype=torch.int32, device="cuda")
        n = sum(e[2] for e in entries)
        self.tokens = torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(n)).int().cuda()
        self.positions = torch.tensor([p + i for _, p, k in entries for i in range(k)], **i32)
        self.slots = torch.tensor([s for s, _, k in entries for _ in range(k)], **i32)
        singles = sum(e[2] == 1 for e in entries)
        lists, tiles, row = [], [], singles
        for s, p, k in entries[singles:]:
            tiles += [(len(lists), t) for t in range(0, k, L.lib().bonsai_lay_conv_rows())]
            lists.append((row, k, s, p))
            row += k
        self.lists, self.tiles = torch.tensor(lists + [(0, 0, 0, 0)], **i32), torch.tensor(tiles + [(0, 0)], **i32)
        self.shape = StepShape(n, singles, singles, len(lists), self.lists.data_ptr(), {L.lib().bonsai_lay_conv_rows(): (self.tiles.data_ptr(), len(tiles))})
        self.rows = n


STATE_ROWS = 6


def state_table():
    return torch.arange(1, STATE_ROWS, dtype=torch.int32, device="cuda")


# ---- row steps and convolutions --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,groups", [(40, 1), (77, 7), (96, 8), (1024, 1), (1024, 4), (1536, 3), (2304, 9), (4100, 2), (4096, 1), (6002, 2), (16384, 16), (9216, 1)])
def test_row_step(width, groups):
    """Every part on its own and all together, against float64."""
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(width)
    T, top, eps, up = 5, 3, 1e-3, L.round_up(width, 128)
    rand = lambda *s: torch.randn(*s, generator=g)
    pad = lambda t, m: torch.nn.functional.pad(t, (0, L.round_up(t.shape[1], m) - t.shape[1])).cuda()
    x0, y, bias, w, nxt, step = rand(T, width), rand(T, width), rand(width), rand(width), rand(width), rand(width)
    gate, table, rows, at = rand(T, 3), rand(9, width).bfloat16(), rand(T * top, width), torch.randperm(T * top, generator=g).int()
    fake = FakeRows([(s, 0, 1) for s in range(T)])
    tokens = fake.tokens.cpu().long()

    class Rows:
        def __init__(self, dtype):
            self.e, self.at, self.counts = pad(rows, 8).to(dtype), at.cuda(), torch.ones(70, dtype=torch.int32, device="cuda")
            self.outputs = (self.e.data_ptr(), self.e.stride(0), int(dtype == torch.float32), self.at.data_ptr(), top, self.counts.data_ptr(), 70)
            self.sum = self.e.cpu().double()[at.long()].view(T, top, -1)[..., :width].sum(1)
    d = lambda t: t.double()
    norm = lambda v, f: O.grouped_norm(v, d(f), groups, eps)
    for case in ("all", "all, 32-bit rows", "plain", "normed", "embedding", "only experts"):
        f32 = "32" in case
        experts = Rows(torch.float32 if f32 else torch.bfloat16) if "all" in case or "only" in case else None
        a, want = {}, d(x0)
        u = torch.zeros(T, width, dtype=torch.float64)
        if "only" not in case and case != "embedding":
            a["y"], u = pad(y, 4), d(y)
        if "all" in case:
            gates = gate.cuda()
            a.update(bias=bias.cuda(), gate=gates[:, 1:])
            u = (u + d(bias)) * torch.sigmoid(d(gate))[:, 1:2]
        if experts is not None:
            u = u + experts.sum
        if case in ("all", "all, 32-bit rows", "normed"):
            a["w"] = w.cuda()
            u = norm(u, w)
        want = want + 0.7 * u
        if case == "embedding":
            a.update(fresh=True, table=pad(table.float(), 128).bfloat16(), scale=1.5, step=step.cuda())
            want = 1.5 * d(table)[tokens] + d(step)
        elif "all" in case:
            a.update(table=pad(table.float(), 128).bfloat16(), scale=0.5, step=step.cuda())
            want = want + 0.5 * d(table)[tokens] + d(step)
        after = norm(want, nxt)
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 0.02)):
            x, h = x0.cuda(), torch.zeros(T, up, dtype=dtype, device="cuda")
            if a.get("fresh"):
                x.fill_(NAN)
            L.RowStep(x, h, fake, state_table(), eps=eps, groups=groups, mult=0.7, next_norm=nxt.cuda(), **a)(T, fake.shape, experts)
            assert experts is None or int(experts.counts.abs().sum()) == 0
            assert float(((x.cpu().double() - want) / (want.abs() + 1)).abs().max()) < 2e-5, case
            assert float(((h.cpu().double()[:, :width] - after) / (after.abs() + 1)).abs().max()) < tol and float(h[:, width:].abs().sum()) == 0, case
    out, pick = torch.zeros(2, up, device="cuda"), torch.tensor([4, 1], dtype=torch.int32, device="cuda")
    x = x0.cuda()
    L.RowStep(x, out, fake, state_table(), eps=eps, groups=groups, next_norm=nxt.cuda())(2, None, norm_of=pick.data_ptr())
    assert float((out.cpu().double()[:, :width] - norm(d(x0), nxt)[[4, 1]]).abs().max()) < 5e-5 and torch.equal(x.cpu(), x0)


@pytest.mark.parametrize("width", [36, 130, 1028])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 16])
def test_input_convolution(width, taps):
    """Single tokens, short and long portions in turn: the next input is n + conv(n), from the ring whatever the cut."""
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(width + taps)
    n = 90
    x, w, nxt = torch.randn(2, n, width, generator=g), torch.randn(width, taps, generator=g), torch.randn(width, generator=g)
    want = torch.stack([O.plus_conv(O.grouped_norm(x[s].double(), nxt.double(), 2, 1e-5), w.double()) for s in range(2)])
    ring = torch.full((STATE_ROWS, taps, width), NAN, device="cuda")
    weight = L.conv_weight(w.cuda())
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 0.02)):
        ring.fill_(NAN)
        at, got = [0, 0], [[], []]
        for a, b in [(1, 1), (1, 2), (3, 1), (1, 1), (1, 17), (2, 33), (16, 1), (15, 1), (1, 1), (40, 30)]:
            parts = sorted([(0, a), (1, b)], key=lambda p: p[1] != 1)
            fake = FakeRows([(s + 1, at[s], k) for s, k in parts])
            stream = torch.cat([x[s, at[s]:at[s] + k] for s, k in parts]).cuda()
            h, n32 = torch.zeros(fake.rows, L.round_up(width, 128), dtype=dtype, device="cuda"), torch.full((fake.rows, L.round_up(width, 4)), NAN, device="cuda")
            L.RowStep(stream, h, fake, state_table(), eps=1e-5, groups=2, next_norm=nxt.cuda(), conv=(weight, ring), n32=n32)(fake.rows, fake.shape)
            for (s, k), part in zip(parts, h[:, :width].cpu().double().split([k for _, k in parts])):
                got[s].append(part)
                at[s] += k
        for s in range(2):
            o = torch.cat(got[s])
            assert float(((o - want[s, :len(o)]) / (want[s, :len(o)].abs() + 1)).abs().max()) < tol and len(o) > 70


# ---- recurrences ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("exact", [True, False])
@pytest.mark.parametrize("width", [20, 33, 100, 256])
def test_mingru(width, exact):
    """Prompts over clusters of every size and decoded tokens, each continuing from the one before."""
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    g, n = torch.Generator().manual_seed(width), 1500
    up = L.round_up(width, 4)
    proj = torch.full((n, 3 * up + 8), NAN)
    cols = (4, 4 + up, 4 + 2 * up)
    z, u, gate = (torch.randn(n, width, generator=g) for _ in range(3))
    z = 2.0 * z - 1.5
    for c, t in zip(cols, (z, u, gate)):
        proj[:, c:c + width] = t
    zb, ub = torch.randn(width, generator=g), torch.randn(width, generator=g)
    d = lambda t: t.double()
    want = O.mingru_scan(torch.sigmoid(d(z) + d(zb)), O.mingru_candidate(d(u) + d(ub))) * O.silu(d(gate))
    S = torch.full((STATE_ROWS, width), NAN, device="cuda")
    proj, zb, ub = proj.cuda(), zb.cuda(), ub.cuda()
    lib, dtype, tol = L.lib(), torch.float32 if exact else torch.bfloat16, 3e-6 if exact else 5e-3
    for cluster in (1, 2, 4, 8):
        S.fill_(NAN)
        at = 0
        for k in (5, 1, 1, 127, 130, 1, 2, 600, 1, 632):
            fake = FakeRows([(2, at, k)])
            out = torch.zeros(k, L.round_up(width, 128), dtype=dtype, device="cuda")
            part = proj[at:at + k]
            call = L.MixerCall([part, zb, ub, S, fake.positions, fake.slots, state_table(), out], [part.stride(0), *cols, out.stride(0), width], [])
            if k == 1:
                K.check(lib.bonsai_lay_gru_step(*call.args, 1, int(exact), K.stream()), "gru_step")
            else:
                K.check(lib.bonsai_lay_gru_scan(*call.args, fake.lists.data_ptr(), 1, cluster, int(exact), K.stream()), "gru_scan")
            got, ref = out[:, :width].cpu().double(), want[at:at + k]
            assert float(((got - ref) / (ref.abs() + 0.3)).abs().max()) < tol, (cluster, at, k)
            assert float(out[:, width:].abs().sum()) == 0
            at += k
        assert at == n


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("state", [1, 3, 16, 17, 32, 50, 64, 100, 128, 129, 256])
def test_selective_scan_states(tmp_path, monkeypatch, state, kv):
    """Every split of the states over lanes; prompts whole and in segments, decoding, and back to prompts."""
    from oxibonsai_b200.models import layered
    m = M.Model(tmp_path / "m", M.naforax([M.mamba1({256: 130, 3: 41}.get(state, 62), state, 5, 3)], width=64, vocab=60), seed=state)
    tokens = m.tokens(230)
    want = m.logits(tokens)
    eng = engine(m, kv, max_batch=2)
    for size in (0, 1, 2):
        monkeypatch.setattr(layered, "plan_segments", lambda lengths, plan, sms: size)
        poison(eng)
        check(feed(eng, tokens, [150, 1, 1, 2, 1], slot=1), want, kv, f"{state} states, segments of {size} chunks")


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_strong_and_weak_decays(tmp_path, kv):
    """Decays from next to none to all at once, step sizes from tiny to large: no overflow, and old inputs count where they should."""
    def tweak(w):
        w["l0.mix.A_log"].copy_(torch.linspace(-9.0, 5.0, w["l0.mix.A_log"].numel()).view(w["l0.mix.A_log"].shape))
        w["l0.mix.dt.b"].copy_(torch.linspace(-6.0, 6.0, w["l0.mix.dt.b"].numel()))
        w["l1.mix.z.b"].copy_(torch.linspace(-9.0, 9.0, w["l1.mix.z.b"].numel()))
    m = M.Model(tmp_path / "m", M.naforax([M.mamba1(64, 16, 4, 4), M.mingru(96)], (0, 2, 2), width=64, vocab=60), seed=3, tweak=tweak)
    tokens = m.tokens(350)
    want = m.logits(tokens)
    eng = engine(m, kv, max_batch=1)
    for cuts in ([], [300] + [1] * 50, [2] * 100):
        poison(eng)
        check(feed(eng, tokens, cuts), want, kv, str(cuts[:2]))


# ---- routing and epilogues ------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(5, 2), (33, 5), (64, 64 // 2), (130, 6), (512, 8), (6, 6), (1, 1)])
def test_softmax_router(E, top):
    from oxibonsai_b200.models.layered_config import ExpertsSpec, RouterSpec
    from oxibonsai_b200.ops import layered_ops as L
    g, dev = torch.Generator().manual_seed(E), torch.device("cuda")
    spec = ExpertsSpec(RouterSpec(E, top, softmax=True, normalized=False, corrected=False), 8)
    up = L.DenseWeight([torch.zeros(8 * E, 16).bfloat16()] * 2, dev, interleave=True)
    logits = torch.full((300, L.round_up(E, 4) + 8), NAN, device=dev)
    r = L.Routing(spec, up, L.DenseWeight([torch.zeros(16 * E, 8).bfloat16()], dev), None, logits, 4, L.ExpertScratch(300, 16, [spec], False, dev))
    scratch, h = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev)), torch.zeros(300, 128, device=dev).bfloat16()
    for T, spread in ((1, 2.0), (31, 2.0), (65, 60.0), (300, 2.0)):       # a wide spread underflows the scores of the last choices
        z = spread * torch.randn(T, E, generator=g)
        logits[:T, 4:4 + E] = z.cuda()
        r(h, T, scratch)
        r.s.counts.zero_()
        at, weight = r.s.at[: T * top].cpu().long().view(T, top), r.s.weight[: T * top].cpu().double()
        owner = torch.bucketize(torch.arange(T * top), r.s.lists[1: E + 1].cpu(), right=True)
        for t in range(T):
            want, ww = O.softmax_route(z[t].double(), top)
            assert owner[at[t]].tolist() == want and torch.allclose(weight[at[t]], ww, rtol=2e-5, atol=1e-37)


@pytest.mark.parametrize("T", [3, 20, 32, 40, 65, 300])
@pytest.mark.parametrize("n,k", [(70, 60), (333, 200), (130, 4096)])
def test_epilogues(n, k, T):
    """The gelu gate and the capped head in all three projection kernels."""
    from oxibonsai_b200.models.layered_config import gelu_mlp
    from oxibonsai_b200.ops import layered_ops as L
    g, dev, spec = torch.Generator().manual_seed(n + T), torch.device("cuda"), gelu_mlp(n)
    scratch = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
    a, b, x = (torch.randn(s, generator=g) * s[1] ** -0.5 * 3 for s in ((n, k), (n, k), (T, k)))
    a, b, x = a.bfloat16(), b.bfloat16(), (x * k ** 0.5 / 3).bfloat16()
    p, q = (O.linear(x.double(), w.double()) for w in (a, b))
    both, one = L.DenseWeight([a, b], dev, interleave=True), L.DenseWeight([a], dev)
    for exact in (True, False):
        act = torch.float32 if exact else torch.bfloat16
        h = torch.zeros(T, one.kp, dtype=act, device=dev)
        h[:, :k] = x.to(dev, act)
        out, raw = torch.zeros(T, L.round_up(n, 128), dtype=act, device=dev), torch.zeros(T, L.round_up(n, 4), device=dev)
        L.linear(both, h, T, out, scratch, L.Glu(spec.limit, spec.alpha, spec.offset, spec.cubic))
        L.linear(one, h, T, raw, scratch, L.SoftCap(2.5))
        want = O.gelu_tanh(p) * q
        assert float(((out[:, :n].cpu().double() - want) / (want.abs() + 1)).abs().max()) < (2e-5 if exact else 0.01)
        want = 2.5 * torch.tanh(p / 2.5)
        assert float((raw[:, :n].cpu().double() - want).abs().max()) < 6e-5 and float(p.abs().max()) > 4.0
    assert int(scratch.status) == 0


# ---- each mechanism alone -----------------------------------------------------------------------------------------------------------
ALONE = {
    "attention": lambda: [M.differential()],
    "attention, one key head": lambda: [M.differential(8, 1, 16, 40, 0.4, 33, 16, 30.0, 0.0)],
    "attention, twenty heads a group": lambda: [M.differential(20, 1, 12, 24, 0.4, 50, 2, 30.0, 0.9)],
    "attention, nothing rotated": lambda: [M.differential(3, 3, 16, 16, 0.3, 64, 0, 1.0, 0.25)],
    "attention, chunks of one": lambda: [M.differential(4, 2, 16, 16, 0.3, 1, 4)],
    "minGRU": lambda: [M.mingru()],
    "Mamba": lambda: [M.mamba1()],
    "Mamba, one tap": lambda: [M.mamba1(40, 5, 1, 1)],
    "dense": lambda: [M.mingru(24, mlp=M.gelu())],
    "experts": lambda: [M.mingru(24, mlp=M.moe())],
    "experts, none shared": lambda: [M.mingru(24, mlp=M.moe(50, 9, 2, 1.4, None))],
    "experts, all of them": lambda: [M.mingru(24, mlp=M.moe(20, 4, 4, 0.5, (8, 0.6)))],
    "one expert": lambda: [M.mingru(24, mlp=M.moe(70, 1, 1, 3.0))],
}
CUTS = {"whole": [], "twos": [2] * 20 + [3] * 5, "ones": [1] * 40, "mixture": [5, 1, 1, 64, 1, 63, 2, 65, 1], "decode": [100] + [1] * 100}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", ALONE)
def test_alone(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.naforax(ALONE[name](), width=88, vocab=120), seed=len(name))
    eng = engine(m, kv, max_batch=2)
    tokens = m.tokens(205)
    want = m.logits(tokens)
    for n, cuts in CUTS.items():
        poison(eng)
        check(feed(eng, tokens, cuts, slot=1), want, kv, what=f"{name}, {n}")


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("loop", [(0, 3, 2), (1, 2, 4), (2, 3, 3), (1, 3, 1), (0, 1, 1)])
def test_loops(tmp_path, loop, kv):
    """Loops at the start, the end and in between; every pass has its own keys and state."""
    m = M.Model(tmp_path / "m", M.naforax([M.mingru(40), M.differential(4, 2, 16, 16, size=45), M.mamba1(48, 6, 3, 3)], loop, width=72, vocab=80), seed=sum(loop))
    eng = engine(m, kv, max_batch=1)
    tokens = m.tokens(150)
    want = m.logits(tokens)
    for cuts in ([], [100] + [1] * 50, [3, 2, 60]):
        poison(eng)
        check(feed(eng, tokens, cuts), want, kv, what=f"{loop} {cuts[:2]}")


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
    """The residual stream behind the first layer runs, of models cut off there."""
    layers = mixed.cfg["layers"]
    for n, loop in ((1, (0, 1, 1)), (2, (1, 2, 1)), (2, (0, 2, 3)), (4, (1, 4, 2))):
        m = M.Model(tmp_path / f"{n}{loop}", {**M.naforax_mixed(), "layers": layers[:n], "loop": dict(zip(("start", "stop", "times"), loop))}, seed=n)
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


# ---- things that random weights would hide ---------------------------------------------------------------------------------------------
MARK, ASK = 7, 11


def plain_tokens(m, n, seed=1):
    return [t if t not in (MARK, ASK) else 1 for t in m.tokens(n, seed)]


def point_maps(w, m, gain=4.0, which=(0,)):
    """Token ASK's queries match token MARK's keys in the given maps, in the dimensions that are not rotated; no convolution blurs it, and
    both maps count (lambda is 0.39 above ``diff``)."""
    H, G, d, turned = m["heads"], m["kv_heads"], m["dim"], m["rot"]["dims"]
    w["l0.canon1"].zero_()
    read = lambda t: w["embed"][t] / w["embed"][t].norm() / w["l0.norm1"]
    dirs = torch.randn(G, d, generator=torch.Generator().manual_seed(5))
    dirs[:, :turned] = 0.0
    dirs /= dirs.norm(dim=1, keepdim=True)
    k, q = w["l0.mix.k"].view(G, 2, d, -1), w["l0.mix.q"].view(G, H // G, 2, d, -1)
    for n, value in (("lq1", 0.0), ("lk1", 0.0), ("lq2", 1.0), ("lk2", -0.5 / d)):
        w["l0.mix." + n].fill_(value)
    for i in which:
        k[:, i] += gain * dirs[:, :, None] * read(MARK)[None, None, :]
        q[:, :, i] += gain * dirs[:, None, :, None] * read(ASK)[None, None, None, :]


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("which", [(0,), (1,)])
@pytest.mark.parametrize("heads,size", [((2, 2, 30, 20), 64), ((8, 2, 30, 44), 37), ((4, 1, 36, 70), 200), ((3, 3, 24, 24), 1000)])
def test_far_keys_and_chunk_edges(tmp_path, heads, size, which, kv):
    """One key that stands out in one of the maps, just inside and just outside the chunk, at page borders and far away, asked for in a
    prompt and in decoding.  Outside, the answer is that of a prompt without it."""
    layer = M.differential(*heads, scale=0.5, size=size, dims=6, base=50.0, diff=0.5)
    m = M.Model(tmp_path / "m", M.naforax([layer], vocab=60, width=96, mult=1.0, cap=30.0), seed=9, tweak=lambda w: point_maps(w, layer["mixer"], which=which))
    eng = engine(m, kv, max_batch=1)
    for ask in (330, 2 * size, 2 * size - 1, 128, 64):
        ask = min(ask, 350)
        start = ask - ask % size
        inside = {p for p in (start, start + 1, ask - 1, ask - 2, 63, 64, 128, 256, 319, 320) if start <= p < ask}
        outside = {p for p in (start - 1, start - 2, 0, 63) if 0 <= p < start}
        base = plain_tokens(m, ask + 3)
        base[ask] = ASK
        nothing = m.logits(base)[ask]
        for mark in sorted(inside) + sorted(outside):
            tokens = list(base)
            tokens[mark] = MARK
            want = m.logits(tokens)
            moved = float((want[ask] - nothing).abs().max())
            assert moved > 0.12 if mark in inside else moved < 1e-9
            poison(eng)
            for cuts in ([], [ask] + [1] * 3, [mark + 1, 2], [max(1, ask - 20)]):
                check(feed(eng, tokens, cuts), want, kv, what=f"mark {mark}, ask {ask}, cuts {cuts}")


def apart(a, b):
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / (b - b.mean(-1, keepdim=True)).pow(2).mean().sqrt()).max())


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_constants_show(tmp_path, kv):
    """What the configuration's numbers do is larger than the tolerance, so the comparison sees each of them."""
    cfg = M.naforax([M.differential(4, 2, 24, 20, 0.6, 90, 20, 400.0, 0.35, mlp=M.moe(30, 5, 2, 0.4, (24, 0.5))), M.mingru(48), M.mamba1(48, 6, 3, 3)], (0, 2, 2),
                    vocab=90, width=96, mult=0.8, cap=4.0, groups=3)
    m = M.Model(tmp_path / "m", cfg, seed=13, scale=2.0, tweak=lambda w: w["l2.mix.D"].mul_(6.0))
    tokens = m.tokens(200)
    want = m.logits(tokens)
    changes = {"scale": lambda c: c["layers"][0]["mixer"].update(scale=0.8), "chunk": lambda c: c["layers"][0]["mixer"]["mask"].update(size=91),
               "diff": lambda c: c["layers"][0]["mixer"].update(diff=0.5), "base": lambda c: c["layers"][0]["mixer"]["rot"].update(base=700.0),
               "rotated": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "limit": lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.6),
               "shared limit": lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.8), "top": lambda c: c["layers"][0]["mlp"]["router"].update(top=1),
               "mult": lambda c: c.update(residual_mult=0.6), "cap": lambda c: c.update(logit_softcap=5.0), "groups": lambda c: c["norm"].update(groups=1),
               "stop": lambda c: c["loop"].update(stop=1), "start": lambda c: c["loop"].update(start=1)}
    for name, change in changes.items():
        other = json.loads(json.dumps(cfg))
        change(other)
        assert apart(O.forward(other, m.w, tokens), want) > 0.05, name
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.mix.o.b", "l0.mix.lq1", "l1.mix.z.b", "l1.mix.x.b", "l2.mix.conv.b", "l2.mix.D", "l2.mix.dt.b", "loop.step", "l1.canon1", "l0.canon2"):
        assert apart(O.forward(cfg, {**m.w, name: torch.zeros_like(m.w[name])}, tokens), want) > 0.05, name
    eng = engine(m, kv, max_batch=1)
    for cuts in ([], [150] + [1] * 50, [40] * 5):
        check(feed(eng, tokens, cuts), want, kv, what=str(cuts[:2]), tol={"f32": TOL["f32"], "bf16": (0.02, 0.06)})


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_long_context(tmp_path, kv):
    """Decoding over several splits, prompts of many tiles and several rounds of the scans, from position 0 and behind earlier tokens."""
    m = M.Model(tmp_path / "m", M.naforax([M.differential(4, 2, 36, 20, 0.4, 700, 20), M.mingru(40), M.mamba1(40, 20, 4, 4)], (1, 2, 2), vocab=70, width=64), seed=8)
    eng = engine(m, kv, max_batch=2, max_seq=1408, chunk=1408)
    tokens = m.tokens(1300)
    want = m.logits(tokens)
    assert eng.runner.mixers[0][0].splits(1) >= 4 and eng.runner.mixers[1][0].cluster(1, 1300) == 8
    for cuts in ([], [77, 1100, 2], [1260] + [1] * 40, [699, 2, 33, 1, 1, 200]):
        poison(eng)
        check(feed(eng, tokens, cuts), want, kv, str(cuts[:3]))


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_long_decoding(tmp_path, kv):
    m = M.Model(tmp_path / "m", M.naforax([M.mamba1(32, 8, 3, 4, mlp=M.moe(16, 4, 2)), M.differential(2, 1, 12, 24, size=130, dims=8), M.mingru(32)], (0, 2, 2), vocab=70, width=64), seed=8)
    eng = engine(m, kv, max_batch=1, max_seq=640)
    poison(eng)
    tokens = m.tokens(600)
    check(feed(eng, tokens, [3] + [1] * 597), m.logits(tokens), kv)


# ---- other sizes --------------------------------------------------------------------------------------------------------------------------
TINY = [M.differential(1, 1, 1, 1, 1.0, 1, 0, mlp=M.moe(1, 1, 1, 1.0, (1, 1.0))), M.mingru(1, mlp=M.gelu(1)), M.mamba1(1, 1, 1, 1)]
SIZES = {          # layers, width, groups, taps
    "as small as possible": (TINY, 20, 1, 1),
    "one column a group": (TINY, 18, 18, 2),
    "real heads": ([M.differential(8, 4, 64, 128, 0.12, 100, 64, 5e5), M.mamba1(288, 16, 40, 4), M.mingru(520)], 256, 2, 4),
    "wide heads": ([M.differential(2, 1, 128, 256, 0.09, 90, 128), M.differential(2, 2, 90, 130, 0.09, 90, 50), M.differential(2, 2, 48, 192, 0.09, 90, 48)], 264, 4, 3),
    "many heads": ([M.differential(64, 1, 8, 16, 0.4, 60, 4, mlp=M.moe(17, 70, 9, 1.0)), M.differential(36, 12, 8, 30, 0.4, 60, 4)], 72, 4, 5),
    "nothing even": ([M.differential(9, 3, 11, 9, 0.3, 47, 6, mlp=M.moe(21, 9, 5, 0.8, (13, 1.7))), M.mamba1(37, 7, 5, 3, mlp=M.gelu(31)), M.mingru(45, mlp=M.moe(5, 15, 2))], 75, 5, 7),
    "keys wider than values": ([M.differential(4, 2, 96, 16, 0.1, 70, 30)], 72, 2, 2),
    "values wider than keys": ([M.differential(4, 2, 10, 120, 0.3, 70, 10)], 72, 8, 16),
    "many states": ([M.mamba1(30, 200, 60, 8), M.mamba1(200, 33, 130, 2)], 72, 3, 3),
}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", SIZES)
def test_sizes(tmp_path, name, kv):
    layers, width, groups, taps = SIZES[name]
    m = M.Model(tmp_path / "m", M.naforax(layers, (len(layers) - 1, len(layers), 2), width, 97, 1e-6, groups, taps, 0.7, 20.0), seed=len(name))
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
    return M.Model(tmp_path_factory.mktemp("naforax") / "sharp", {**M.naforax_mixed(), "logit_softcap": 30.0}, seed=31, tweak=lambda w: w["final.norm"].mul_(3.0))


def test_greedy_generation_matches_oracle(sharp):
    eng = engine(sharp, "f32")
    prompts = [sharp.tokens(n, seed=n) for n in (1, 5, 70)]
    want = [sharp.greedy(p, 8)[0] for p in prompts]
    assert [eng.generate(p, 8) for p in prompts] == want
    assert eng.generate_batch(prompts, 8) == want
    info = eng.model_info()
    assert info["arch"] == "Naforax" and info["recurrent_layers"] == 4 and info["attention_layers"] == 3 and info["state_bytes"] > 0
    assert not eng.supports_prefix_cache
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
    assert sched.mixed_steps > 0 and len(eng.kv.free_pages) == 12 and len(eng.runner.states.free_rows) == 3
    if kv == "f32":
        assert got == want
    for p, g in zip(prompts, got):           # in 16 bits a near tie may fall the other way: the chosen logits are near the best ones
        lg = sharp.logits(p + g)[len(p) - 1:-1]
        chosen = lg[torch.arange(len(g)), torch.tensor(g)]
        assert float((lg.max(-1).values - chosen).max()) < 0.1 * float(lg.std())


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
    assert len(calls) == r.kernel_launches(2) and calls.count("scan_step") == 4 and calls.count("route") == 7 and calls.count("attn_decode") == 7


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
