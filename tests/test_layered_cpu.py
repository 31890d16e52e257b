"""Layer-list decoders without a GPU: configuration, registry, pools, scheduler batches, and the oracle against itself."""
import json

import layered_models as M
import layered_oracle as O
import pytest
import torch

from oxibonsai_b200.models import registry as R
from oxibonsai_b200.models.layered_config import LayeredConfigError, keripel_config
from oxibonsai_b200.models.paged import PagePool, StatePool
from oxibonsai_b200.models.rope_scaling import alibi_slopes, geometric_slopes


def test_config_reads_every_layer():
    raw = M.mixed_config()
    c = keripel_config(raw, "tiny")
    assert (c.width, c.vocab, c.eps, c.layers, c.name) == (152, 331, 1e-5, 4, "tiny")
    assert c.attention_layers == [0, 2] and c.recurrent_layers == [1, 3]
    a, b = c.layer_specs[0].mixer, c.layer_specs[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.scale, a.window, a.keep_first, a.group) == (6, 2, 40, 0.2, 37, 3, 3)
    assert (b.window, b.keep_first, b.group) == (100, 0, 1) and c.max_visible == 100
    assert c.layer_specs[1].mlp is None and c.layer_specs[3].mlp.ff == 90 and c.layer_specs[3].mixer.gate_cap == 4.0
    assert c.tensor_shapes() == {k: tuple(v) for k, v in O.tensor_shapes(raw).items()}


@pytest.mark.parametrize("change", [
    lambda r: r.pop("width"), lambda r: r.pop("norm"), lambda r: r["layers"].clear(), lambda r: r["layers"][0].pop("mlp"),
    lambda r: r["layers"][0].update(type="conv"), lambda r: r["layers"][0]["mixer"].update(vdim=48), lambda r: r["layers"][0]["mixer"].update(heads=5),
    lambda r: r["layers"][0]["mixer"].update(dim=300, vdim=300), lambda r: r["layers"][0]["mixer"]["mask"].pop("keep_first"),
    lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), lambda r: r["layers"][1]["mixer"].update(dim=513), lambda r: r["layers"][1]["mixer"].pop("gate_cap"),
    lambda r: r["layers"][0]["mlp"].update(kind="moe"), lambda r: r["layers"][0]["mlp"].update(limit="x"), lambda r: r.update(vocab=1.5)])
def test_config_errors(change):
    raw = json.loads(json.dumps(M.mixed_config()))
    change(raw)
    with pytest.raises(LayeredConfigError):
        keripel_config(raw)


def test_registry_and_validation(tmp_path):
    m = M.Model(tmp_path / "tiny", M.mixed_config())
    assert R.is_model_dir(m.path) and not R.is_model_dir(tmp_path)
    assert R.load_model_dir_config(m.path).arch == "Keripel"
    assert R.validate_model_dir(m.path).ok
    w = {k: v.float() for k, v in m.w.items() if k != "l1.mix.f.b"}
    w["l0.mix.o"] = w["l0.mix.o"][:, :-1]
    w["spare"] = torch.zeros(3)
    M.write(m.path, m.cfg, w)
    v = R.validate_model_dir(m.path)
    assert not v.ok and any("l1.mix.f.b" in e for e in v.errors) and any("l0.mix.o" in e for e in v.errors) and v.warnings == ["unused tensor spare"]
    (tmp_path / "other").mkdir()
    (tmp_path / "other" / "config.json").write_text('{"architecture": "Unknown"}')
    assert not R.is_model_dir(tmp_path / "other")
    with pytest.raises(LayeredConfigError):
        R.load_model_dir_config(tmp_path / "other")


def test_cli_info_and_validate(tmp_path, capsys):
    from oxibonsai_b200 import cli
    m = M.Model(tmp_path / "tiny", M.mixed_config())
    assert cli.main(["info", "-m", m.path, "--json"]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Keripel" and info["config"]["recurrent_layers"] == [1, 3] and info["valid"]
    assert cli.main(["info", "-m", m.path]) == 0 and "layer 3: mixer mlstm" in capsys.readouterr().out
    assert cli.main(["validate", "-m", m.path]) == 0


def test_slopes():
    for h in (1, 2, 3, 6, 8, 12):
        s = geometric_slopes(h)
        assert torch.allclose(s, torch.tensor([O.alibi_slope(i, h) for i in range(h)]))
    assert torch.allclose(geometric_slopes(8), alibi_slopes(8)) and not torch.allclose(geometric_slopes(6), alibi_slopes(6))


def test_pools():
    p = PagePool(4, 64)
    a = p.alloc(3)
    assert sorted(a) == [0, 1, 2] and p.utilization == 0.75
    p.retain(a[:1])
    p.release(a)
    assert a[0] not in p.alloc(3)                 # still held by the second owner
    p.release(a[:1])
    assert p.alloc(1) == a[:1]
    with pytest.raises(MemoryError):
        PagePool(1, 64).alloc(2)
    s = StatePool({1: {"S": (2, 4, 4), "m": (2,)}}, 2, "cpu")
    r0, r1 = s.alloc(), s.alloc()
    assert {r0, r1} == {0, 1} and s.nbytes == 2 * (32 + 2) * 4
    with pytest.raises(MemoryError):
        s.alloc()
    s.release(r0)
    assert s.alloc() == r0



# ---- the oracle ------------------------------------------------------------------------------------------------------------------
def test_oracle_window_and_kept_tokens():
    m = O.window_mask(12, 4, 2)
    for i in range(12):
        assert [j for j in range(12) if m[i, j]] == [j for j in range(i + 1) if i - j < 4 or j < 2]
        assert all(bool(m[i, j]) == O.visible(i, j, 4, 2) for j in range(12))


def test_oracle_recurrence_is_the_weighted_sum():
    """The token-by-token recurrence equals its closed form: weights e^(F_t - F_s + i_s - m_t)."""
    g = torch.Generator().manual_seed(3)
    n, d, e = 23, 5, 7
    q, k, v = (torch.randn(n, c, generator=g, dtype=torch.float64) for c in (d, d, e))
    i = 3 * torch.randn(n, generator=g, dtype=torch.float64)
    f = torch.nn.functional.logsigmoid(3 * torch.randn(n, generator=g, dtype=torch.float64))
    o, (S, nrm, m) = O.matrix_memory(q, k, v, i, f)
    F = f.cumsum(0)
    for t in range(n):
        a = F[t] - F[: t + 1] + i[: t + 1]
        mt = torch.maximum(a.max(), F[t])
        w = torch.exp(a - mt) * (k[: t + 1] @ q[t])
        want = (w[:, None] * v[: t + 1]).sum(0) / (torch.maximum(w.sum().abs(), torch.exp(-mt)) + 1e-6)
        assert torch.allclose(o[t], want, rtol=1e-9, atol=1e-12)
    # resuming from the state is the same sequence
    o1, st = O.matrix_memory(q[:9], k[:9], v[:9], i[:9], f[:9])
    o2, _ = O.matrix_memory(q[9:], k[9:], v[9:], i[9:], f[9:], st)
    assert torch.allclose(torch.cat([o1, o2]), o)


def test_oracle_clamped_glu():
    g, u = torch.tensor([-3.0, 0.5, 9.0]), torch.tensor([-9.0, 0.2, 9.0])
    gc, uc = torch.tensor([-3.0, 0.5, 2.0]), torch.tensor([-2.0, 0.2, 2.0])
    assert torch.allclose(O.clamped_glu(g, u, 2.0), gc * torch.sigmoid(1.702 * gc) * (uc + 1))


# ---- scheduler: prompt chunks that ride in decode steps -----------------------------------------------------------------------------
class FakeMixedEngine:
    """Slot interface whose next token is a function of the sequence's length; records what a step held."""
    supports_mixed_steps, prefill_min_tokens, max_seq_len, max_batch, step_token_limit, eos_token = True, 16, 4096, 4, 64, -1

    def __init__(self):
        self.cached, self.log, self.closed = {}, [], []

    def bind_thread(self): pass

    def begin_sequence(self, prompt, total, slot, params, kv_format=None):
        assert slot not in self.cached
        if 999 in prompt:
            raise ValueError("bad token")
        self.cached[slot] = 0
        return 0

    def prefill(self, prompt, slot, pos0):
        assert self.cached[slot] == pos0
        self.cached[slot] += len(prompt)
        self.log.append(("prefill", len(prompt)))

    def finish_sequence(self, prompt, slot, mask=None):
        assert self.cached[slot] == len(prompt)
        return 10 + len(prompt)

    def _decode(self, positions):
        for s, p in enumerate(positions):
            assert self.cached[s] == p, (s, p, self.cached)
            self.cached[s] += 1
        return [10 + p + 1 for p in positions]

    def step_batch(self, positions, masks=None):
        self.log.append(("step", len(positions)))
        return self._decode(positions)

    def step_mixed(self, positions, chunk, slot, pos0, last, masks=None):
        assert slot >= len(positions) and self.cached[slot] == pos0 and len(chunk) + len(positions) <= self.step_token_limit
        self.cached[slot] += len(chunk)
        self.log.append(("mixed", len(positions), len(chunk)))
        return self._decode(positions)

    def move_slot(self, src, dst):
        self.cached[dst] = self.cached.pop(src)

    def close_sequence(self, slot):
        self.closed.append(slot)
        self.cached.pop(slot, None)


def test_scheduler_mixed_steps():
    from oxibonsai_b200.runtime.presets import SamplingPreset
    from oxibonsai_b200.runtime.scheduler import BatchScheduler
    eng = FakeMixedEngine()
    sched = BatchScheduler(eng, prefill_chunk_tokens=32)
    p = SamplingPreset.GREEDY.params()
    reqs = [sched.submit([1] * n, p, k) for n, k in ((20, 30), (150, 9), (1, 25), (70, 4), (33, 12), (90, 1))]
    bad = sched.submit([1, 999], p, 5)
    sched.start()
    outs = [r.wait(timeout=30) for r in reqs]
    with pytest.raises(ValueError):
        bad.wait(timeout=30)
    sched.stop()
    for r, out in zip(reqs, outs):
        assert out == [10 + len(r.prompt) + j for j in range(r.max_tokens)]
    mixed = [x for x in eng.log if x[0] == "mixed"]
    assert len(mixed) == sched.mixed_steps >= 5 and not eng.cached
    # prompts only run on their own while nothing is live
    assert eng.log[0][0] == "prefill" and sum(x[0] == "prefill" for x in eng.log) <= 2


def test_scheduler_cancel_pending_mixed():
    from oxibonsai_b200.runtime.presets import SamplingPreset
    from oxibonsai_b200.runtime.scheduler import BatchScheduler
    eng = FakeMixedEngine()
    sched = BatchScheduler(eng, prefill_chunk_tokens=16)
    p = SamplingPreset.GREEDY.params()
    second = None
    first = sched.submit([1] * 5, p, 40, on_token=lambda t: second.cancel() if len(first.tokens) == 5 else None)
    second = sched.submit([1] * 3000, p, 5)
    sched.start()
    assert len(first.wait(timeout=30)) == 40
    second.wait(timeout=30)
    sched.stop()
    assert second.finish_reason == "cancelled" and not second.tokens


def test_segment_plan():
    from oxibonsai_b200.models.layered import CHUNK, MAX_SEGMENTS, MLSTM_COST, RECURRENCE_COST, WIDE_RECURRENCE_COST, SegmentPlan, plan_segments
    for cost in (MLSTM_COST, RECURRENCE_COST, WIDE_RECURRENCE_COST):
        plan = lambda ctas: SegmentPlan(ctas, cost)
        assert plan_segments([100], plan(64), 148) == 0 and plan_segments([512] * 8, plan(64), 148) == 0 and plan_segments([2], plan(1), 148) == 0
        for lengths, ctas in (([4096], 64), ([4096], 2), ([100_000], 1), ([900, 2, 700], 4), ([64 * 9 + 1], 3), ([2000] * 30, 1)):
            size = plan_segments(lengths, plan(ctas), 148)
            segs = sum(-(-n // (size * CHUNK)) for n in lengths) if size else 0
            assert segs <= MAX_SEGMENTS and (size == 0 or size >= cost.shortest)
            assert size > 0 or len(lengths) > MAX_SEGMENTS
