"""Layer-list decoders on the GPU against the plain implementation in ``layered_oracle`` (float64 on the CPU)."""
import io
import json
import os
import subprocess
import sys

import layered_models as M
import layered_oracle as O
import numpy as np
import pytest
import torch
from layered_gpu import check, engine, feed, poison, run_unequal_requests

pytestmark = pytest.mark.gpu

@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    return M.Model(tmp_path_factory.mktemp("layered") / "mixed", M.mixed_config(), seed=5)


@pytest.fixture(scope="module", params=["f32", "bf16"])
def mixed_engine(request, mixed):
    return request.param, engine(mixed, request.param)


# ---- projections -------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 2, 8, 9, 16, 17, 32, 33, 64, 65, 300])
@pytest.mark.parametrize("n,k", [(5, 40), (77, 152), (331, 384), (130, 1000), (301, 8200)])      # the last one is split along K between CTAs
def test_linear(T, n, k):
    from oxibonsai_b200.ops import layered_ops as L
    g = torch.Generator().manual_seed(T * 1000 + n)
    a, b = (torch.randn(n, k, generator=g).bfloat16() for _ in range(2))
    x = torch.randn(T, k, generator=g) * k ** -0.5
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    scratch = L.GemmScratch(torch.device("cuda"), status)
    single, pair = L.DenseWeight([a], "cuda"), L.DenseWeight([a, b], "cuda", interleave=True)
    x16 = torch.zeros(T, single.kp, dtype=torch.bfloat16, device="cuda")
    x16[:, :k] = x.bfloat16().cuda()
    limit, alpha, offset = 0.9, 1.3, 0.7
    for act in (x16, x.cuda()):
        exact = act.dtype == torch.float32
        xd = (x if exact else x.bfloat16()).double()
        out = torch.full((T, n + 3), 7.0, device="cuda")[:, :n]
        L.linear(single, act, T, out, scratch)
        want = xd @ a.double().T
        assert float((out.cpu().double() - want).abs().max()) < 2e-5 * max(1.0, k / 1000)      # f32 sums of k terms
        gl = torch.zeros(T, n, dtype=act.dtype, device="cuda")
        L.linear(pair, act, T, gl, scratch, L.Glu(limit, alpha, offset))
        gg, uu = torch.clamp(want, max=limit), torch.clamp(xd @ b.double().T, -limit, limit)
        want = gg * torch.sigmoid(alpha * gg) * (uu + offset)
        assert float((gl.cpu().double() - want).abs().max()) < (2e-5 * max(1.0, k / 1000) if exact else 0.02)
        L.linear(single, act, T, gl, scratch, L.SQUARED_RELU)
        want = torch.relu(xd @ a.double().T) ** 2
        assert float((gl.cpu().double() - want).abs().max()) < (6e-5 * max(1.0, k / 1000) if exact else 0.1)
    assert int(status.item()) == 0


# ---- whole sequences, portions, decoding ---------------------------------------------------------------------------------------------
CUTS = {"whole": [], "twos": [2] * 40 + [3] * 5, "ones": [1] * 90, "mixture": [5, 1, 1, 64, 1, 63, 2, 65, 1], "edges": [37, 2, 61, 2, 1, 90],
        "decode": [150] + [1] * 200}


@pytest.mark.parametrize("cuts", CUTS)
def test_portions(mixed, mixed_engine, cuts):
    kv, eng = mixed_engine
    n = 90 if cuts == "ones" else (260 if cuts == "decode" else 215)
    tokens = mixed.tokens(n, seed=len(cuts))
    poison(eng)
    check(feed(eng, tokens, CUTS[cuts]), mixed.logits(tokens), kv, what=cuts)


def test_batches_match_single_requests(mixed, mixed_engine):
    """Unequal requests share steps: portions beside decoded tokens, left out now and then, ending at different times; their
    pages and slots go to new requests, over a pool that starts full of NaN."""
    kv, eng = mixed_engine
    run_unequal_requests(mixed, eng, kv)


def test_wanted_places(mixed, mixed_engine):
    kv, eng = mixed_engine
    a, b = mixed.tokens(50, 1), mixed.tokens(9, 2)
    for s, t in ((0, a), (3, b)):
        eng.reserve(s, len(t))
    out = eng.feed([(0, a, 0), (3, b, 0)], [[49, 0, 7], []])
    check(out, mixed.logits(a)[[49, 0, 7]], kv)
    assert eng.feed([(0, [1], 50), (3, [2], 9)], [[], []]).shape == (0, mixed.cfg["vocab"])
    eng.close_sequence(0), eng.close_sequence(3)


def test_bad_entries(mixed, mixed_engine):
    _, eng = mixed_engine
    for entries in ([(0, [mixed.cfg["vocab"]], 0)], [(0, [-1, 2], 0)], [(9, [1, 2], 0)], [(0, [1, 2], 383)], [(0, [1, 2], 0), (0, [3, 4], 2)], []):
        with pytest.raises(ValueError):
            eng.feed(entries, [[] for _ in entries])
    with pytest.raises(MemoryError):
        eng.reserve(0, 384), eng.reserve(1, 384), eng.reserve(2, 384), eng.reserve(3, 384), eng.kv.alloc(1)
    for s in range(4):
        eng.close_sequence(s)


# ---- windows, kept tokens, far keys: one key that stands out -------------------------------------------------------------------------
MARK, ASK = 7, 11


def standout(w):
    """Token ASK's queries match token MARK's keys, whose values are three times as long: whether a MARK is seen shows."""
    for p in [k[:-1] for k in w if k.endswith("mix.q") and k + ".norm" in w]:
        d = w[p + "q.norm"].shape[0]
        k = w[p + "k"]
        group = w[p + "q"].shape[0] // k.shape[0]
        w[p + "q"] = k.view(-1, 1, d, k.shape[1]).expand(-1, group, -1, -1).reshape(-1, k.shape[1]).clone()
    w["embed"][MARK] = -3.0 * w["embed"][ASK]


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("size,keep,group", [(70, 4, 3), (64, 0, 1), (1, 1, 2), (33, 70, 4), (5, 1, 8)])
def test_window_edges(tmp_path, kv, size, keep, group):
    """A marked key just inside and just outside the window and the kept tokens, at page borders, for prompts and decoding."""
    def tweak(w):
        standout(w)
        w["l0.mix.k.norm"] = -w["l0.mix.k.norm"].abs()          # MARK's key is ASK's reversed; the negative norm weight turns it back
        w["l0.mix.q.norm"] = w["l0.mix.q.norm"].abs()
    m = M.Model(tmp_path / "m", M.config([M.attention(heads=group * 2, kv_heads=2, dim=36, scale=0.6, size=size, keep=keep)], vocab=60), seed=9, tweak=tweak)
    eng = engine(m, kv, max_batch=1)
    n = 200
    shown = 0
    for ask in (127, 128, 129, 191):
        for mark in sorted({ask - size - 1, ask - size, ask - size + 1, ask - 1, keep - 1, keep, 0, 63, 64, 65, 127} & set(range(ask))):
            tokens = [t if t not in (MARK, ASK) else 1 for t in m.tokens(n, seed=mark)]
            plain = list(tokens)
            plain[ask] = ASK
            tokens[ask], tokens[mark] = ASK, MARK
            want = m.logits(tokens)
            if ask == 127 or mark % 2:
                shown += float((want[ask] - m.logits(plain)[ask]).abs().max()) > 0.05
            poison(eng)
            for cuts in ([], [ask] + [1] * 3, [mark, 2, 1, ask - mark - 3, 2] if ask - mark > 3 else [mark, 1, 1]):
                got = feed(eng, tokens[: ask + 2], cuts)
                check(got, want[: ask + 2], kv, what=f"mark {mark}, ask {ask}, cuts {cuts}")
    assert shown >= 1


@pytest.mark.parametrize("kv", ["f32", "bf16"])
def test_state_carries_far(tmp_path, kv):
    """A forget gate that is almost open and one strong input gate: the first tokens' values reach hundreds of tokens on."""
    def tweak(w):
        w["l0.mix.f.b"] = torch.tensor([9.0, 2.0])
        w["l0.mix.i.b"] = torch.tensor([-6.0, 0.0])
        w["l0.mix.f"] *= 0.1
        w["l0.mix.i"][0] = 0.2 * w["embed"][MARK]
    m = M.Model(tmp_path / "m", M.config([M.mlstm(heads=2, dim=30, vdim=20, cap=12.0)], vocab=70), seed=2, tweak=tweak)
    eng = engine(m, kv, max_batch=1)
    tokens = [t if t != MARK else 1 for t in m.tokens(330)]
    plain = m.logits(tokens)
    tokens[3] = MARK
    want = m.logits(tokens)
    assert float((want[320] - plain[320]).abs().max()) > 0.05
    for cuts in ([], [1] * 20 + [64, 1, 63], [300] + [1] * 30, [2] * 5 + [3] * 30):
        check(feed(eng, tokens, cuts), want, kv, what=str(cuts[:3]))


@pytest.mark.parametrize("d,e", [(20, 70), (100, 40), (200, 66)])
def test_long_prompts_in_segments(tmp_path, d, e):
    """Prompts long enough for the recurrence to be cut into segments, from position 0 and from a state, alone and together."""
    from oxibonsai_b200.models.layered import plan_segments
    m = M.Model(tmp_path / "m", M.config([M.mlstm(heads=2, dim=d, vdim=e)], vocab=70, width=64), seed=d,
                tweak=lambda w: w["l0.mix.f.b"].copy_(torch.tensor([6.0, 1.0])))
    eng = engine(m, "bf16", max_batch=3, max_seq=1024, chunk=2048)
    poison(eng)
    tokens = m.tokens(900)
    want = m.logits(tokens)
    (plan,) = eng.runner.segment_plans
    assert plan_segments([900], plan, 148) and plan_segments([600, 700], plan, 148)
    check(feed(eng, tokens, []), want, "bf16", "whole")
    check(feed(eng, tokens, [77, 700, 2]), want, "bf16", "resumed")
    for s, n in ((0, 600), (1, 1), (2, 900)):
        eng.reserve(s, n)
    eng.feed([(2, tokens[:200], 0)], [[]])
    out = eng.feed([(0, tokens[:600], 0), (1, tokens[:1], 0), (2, tokens[200:], 200)], [list(range(600)), [0], list(range(700))])
    check(out, torch.cat([want[:600], want[:1], want[200:]]), "bf16", "together")
    check(eng.feed([(0, tokens[600:601], 600), (2, [5], 900)], [[0], []]), want[600:601], "bf16", "decode after")


# ---- other sizes --------------------------------------------------------------------------------------------------------------------------
SIZES = {
    "one head each": [M.attention(heads=1, kv_heads=1, dim=32, size=9, keep=1, ff=64), M.mlstm(heads=1, dim=16, vdim=16, cap=1.0, ff=33)],
    "many query heads": [M.attention(heads=40, kv_heads=2, dim=8, size=80, keep=2), M.mlstm(heads=5, dim=64, vdim=64)],
    "wide heads": [M.attention(heads=2, kv_heads=1, dim=256, scale=0.05, size=50, keep=5), M.mlstm(heads=2, dim=256, vdim=200)],
    "three quarters": [M.attention(heads=3, kv_heads=3, dim=96, scale=0.1), M.attention(heads=4, kv_heads=2, dim=192, scale=0.07, ff=31), M.mlstm(dim=128, vdim=64)],
    "long keys, many values": [M.mlstm(heads=1, dim=300, vdim=600), M.attention(heads=2, kv_heads=2, dim=17, size=300, keep=0)],
    "nothing even": [M.mlstm(heads=3, dim=13, vdim=7, ff=21), M.attention(heads=9, kv_heads=3, dim=11, size=23, keep=2, ff=5)],
    "only recurrent": [M.mlstm(heads=2, dim=65, vdim=129, cap=30.0, ff=100)],
}


@pytest.mark.parametrize("kv", ["f32", "bf16"])
@pytest.mark.parametrize("name", SIZES)
def test_sizes(tmp_path, name, kv):
    m = M.Model(tmp_path / "m", M.config(SIZES[name], width={"wide heads": 264, "nothing even": 75}.get(name, 72), vocab=97, eps=1e-6), seed=len(name))
    eng = engine(m, kv, max_batch=2)
    poison(eng)
    tokens = m.tokens(140)
    want = m.logits(tokens)
    for cuts in ([], [66, 1, 2, 1], [1] * 5 + [80] + [1] * 60):
        check(feed(eng, tokens, cuts, slot=1), want, kv, what=f"{name} {cuts[:4]}")


# ---- generation through the framework's entry points -----------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def sharp(tmp_path_factory):
    """A model whose logits are far enough apart for greedy generation to be the same in both modes."""
    def tweak(w):
        w["final.norm"] *= 3.0
    return M.Model(tmp_path_factory.mktemp("layered") / "sharp", M.mixed_config(), seed=31, tweak=tweak)


def test_greedy_generation_matches_oracle(sharp):
    eng = engine(sharp, "f32")
    prompts = [sharp.tokens(n, seed=n) for n in (1, 5, 70)]
    want = [sharp.greedy(p, 12)[0] for p in prompts]
    assert [eng.generate(p, 12) for p in prompts] == want
    assert eng.generate_batch(prompts, 12) == want
    assert eng.last_stats.generated_tokens == 12 and eng.model_info()["recurrent_layers"] == 2
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
    want = [sharp.greedy(p, k)[0] if kv == "f32" and len(p) < 70 else alone.generate(p, k) for p, k in zip(prompts, counts)]
    sched = BatchScheduler(eng, prefill_chunk_tokens=32)
    reqs = [sched.submit(p, SamplingPreset.GREEDY.params(), k) for p, k in zip(prompts, counts)]
    sched.start()
    got = [r.wait(timeout=120) for r in reqs]
    sched.stop()
    assert sched.mixed_steps > 0 and len(eng.kv.free_pages) == 12 and len(eng.runner.states.free_rows) == 3
    if kv == "f32":
        assert got == want
    else:                    # a near tie may fall the other way in 16 bits: compare the logits along the generated text instead
        for p, g in zip(prompts, got):
            lg = sharp.logits(p + g)[len(p) - 1:-1]
            chosen = lg[torch.arange(len(g)), torch.tensor(g)]
            assert float((lg.max(-1).values - chosen).max()) < 0.1 * float(lg.std())
    bad = BatchScheduler(eng)
    r = bad.submit([0, sharp.cfg["vocab"]], SamplingPreset.GREEDY.params(), 3)
    bad.start()
    with pytest.raises(ValueError):
        r.wait(timeout=60)
    bad.stop()


def test_constrained_and_sampled_generation(sharp):
    from oxibonsai_b200.runtime.presets import SamplingParams
    eng = engine(sharp, "bf16")

    class Evens:
        def reset(self): pass
        def advance(self, t): pass
        def finished(self): return False
        def allowed_mask(self): return np.full((sharp.cfg["vocab"] + 31) // 32, 0x55555555, dtype=np.uint32)
    out = eng.generate(sharp.tokens(20), 10, constraint=Evens())
    assert len(out) == 10 and all(t % 2 == 0 for t in out)
    p = SamplingParams(temperature=1.0, top_k=0, top_p=1.0, seed=3)
    a, b = eng.generate(sharp.tokens(20), 10, p), eng.generate(sharp.tokens(20), 10, p)
    assert a == b and all(0 <= t < sharp.cfg["vocab"] for t in a)


def test_unsupported_features_are_refused(sharp):
    eng = engine(sharp, "bf16")
    assert not eng.supports_prefix_cache and eng.enable_kv_formats() == ["bf16"]
    with pytest.raises(ValueError):
        eng.enable_prefix_cache()
    with pytest.raises(NotImplementedError):
        eng.verify_greedy([1, 2], 0)
    with pytest.raises(ValueError):
        engine(sharp, "q8")


def test_prefix_cache_without_recurrence(tmp_path):
    """An attention-only model resumes from cached prompt pages."""
    m = M.Model(tmp_path / "m", M.config([M.attention(size=90, ff=64), M.attention(heads=2, kv_heads=1, size=200, keep=1)]), seed=4,
                tweak=lambda w: w["final.norm"].mul_(3.0))
    eng = engine(m, "f32", max_batch=1)
    cache = eng.enable_prefix_cache(4)
    prompt = m.tokens(150)
    want = m.greedy(prompt, 5)[0]
    assert eng.generate(prompt, 5) == want and eng.generate(prompt, 5) == want
    assert len(cache.lookup(prompt, max_tokens=149)) == 2


# ---- trace replay -------------------------------------------------------------------------------------------------------------------------------
def test_trace_replay(mixed, mixed_engine, tmp_path):
    from oxibonsai_b200.runtime.trace import replay
    kv, eng = mixed_engine
    a, b = mixed.tokens(80, 3), mixed.tokens(30, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:29], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:51], "want": []}], "end": []},
             {"step": 5, "entries": [{"id": "b", "tokens": b[29:], "want": [0]}, {"id": "a", "tokens": a[51:], "want": [28]}], "end": ["a", "b"]}]
    answer = io.StringIO()
    assert replay(eng, [json.dumps(s) for s in steps] + ["\n"], str(tmp_path), answer) == 3
    assert answer.getvalue().split("\n") == ["done 0", "done 1", "done 5", ""] and sorted(os.listdir(tmp_path)) == ["0.f32", "5.f32"]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).view(-1, mixed.cfg["vocab"])
    la, lb = mixed.logits(a), mixed.logits(b)
    check(read(0), la[[0, 49]], kv)
    check(read(5), torch.stack([lb[29], la[79]]), kv)
    assert len(eng.kv.free_pages) == eng.kv.num_pages


def test_trace_run_program(mixed, tmp_path):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = mixed.tokens(70, 6)
    lines = [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": toks[:69], "want": [68]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "x", "tokens": toks[69:], "want": [0]}], "end": ["x"]})]
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", mixed.path, "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "128"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    got = torch.cat([torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4")).view(1, -1) for s in (0, 1)])
    check(got, mixed.logits(toks)[68:70], "f32")
