"""Naforax decoders without a GPU: configuration, registry, command line, state and weights, and the oracle's mechanisms against other forms."""
import json
import math

import layered_models as M
import layered_oracle as O
import pytest
import torch

from oxibonsai_b200.models import registry as R
from oxibonsai_b200.models.layered_config import LayeredConfigError, Run, naforax_config


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ---- configuration ------------------------------------------------------------------------------------------------------------------
def test_config_reads_every_layer():
    raw = M.naforax_mixed()
    c = naforax_config(raw, "tiny")
    assert (c.width, c.vocab, c.eps, c.layers, c.residual_mult, c.norm_groups, c.input_taps, c.logit_cap, c.own_head) == (152, 331, 1e-5, 7, 0.6, 4, 3, 9.0, True)
    assert (c.pre_norm, c.side_by_side, c.layer_norm, c.embed_scale, c.row_steps, c.has_state) == (True, False, False, 1.0, True, True)
    assert c.attention_layers == [1, 3, 6] and c.recurrent_layers == [0, 2, 4, 5] and c.expert_layers == [0, 2, 3] and c.max_visible == 100
    g, a, s = (c.layer_specs[i].mixer for i in (0, 1, 2))
    assert g.width == 100 and (s.channels, s.states, s.rank, s.conv) == (90, 12, 9, 4)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.window, a.difference, a.maps, a.row_dim, a.visible) == (6, 2, 20, 28, 0.3, 70, 0, 0.4, 2, 40, 70)
    assert (a.rotary.base, a.rotary.dims, a.rotary.interleaved, a.biases, a.element_gate, a.norm_weights, a.sink) == (900.0, 12, True, True, True, True, False)
    e = c.experts(0)
    assert (e.ff, e.limit, e.alpha, e.offset, e.router.experts, e.router.top, e.router.softmax, e.router.normalized, e.router.corrected) == (40, 0.9, 1.702, 1.0, 11, 3, True, False, False)
    assert (e.shared.ff, e.shared.limit, e.shared.alpha) == (56, 1.3, 1.702) and c.experts(2).shared is None and c.layer_specs[4].mlp is None
    assert c.norm_names(4) == [("l4.norm1", "l4.norm1b")] and len(c.norm_names(0)) == 2
    assert c.tensor_shapes() == {k: tuple(v) for k, v in O.tensor_shapes(raw).items()}
    assert c.param_count() == sum(math.prod(s) for s in O.tensor_shapes(raw).values())


@pytest.mark.parametrize("loop", [(0, 1, 1), (0, 7, 2), (1, 4, 3), (6, 7, 5), (2, 3, 1)])
def test_runs(loop):
    c = naforax_config({**M.naforax_mixed(), "loop": dict(zip(("start", "stop", "times"), loop))})
    assert [(r.layer, r.begins) for r in c.runs] == [(i, t if i == loop[0] else None) for i, t in O.loop_runs(7, dict(zip(("start", "stop", "times"), loop)))]
    assert sum(r.begins is not None for r in c.runs) == loop[2] and c.tensor_shapes()["loop.step"] == (loop[2], 152)


def test_without_a_loop():
    raw = M.naforax_mixed()
    del raw["loop"]
    c = naforax_config(raw)
    assert c.runs == tuple(Run(i) for i in range(7)) and "loop.step" not in c.tensor_shapes()


L = lambda i: lambda r: r["layers"][i]["mixer"]
MLP = lambda i: lambda r: r["layers"][i]["mlp"]


@pytest.mark.parametrize("change", [
    lambda r: r.pop("residual_mult"), lambda r: r.pop("logit_softcap"), lambda r: r.update(logit_softcap=0), lambda r: r.pop("canon"), lambda r: r["canon"].update(taps=0),
    lambda r: r["canon"].update(taps=17), lambda r: r["norm"].pop("groups"), lambda r: r["norm"].update(groups=5), lambda r: r.update(width=1 << 16),
    lambda r: r["loop"].update(start=4), lambda r: r["loop"].update(stop=8), lambda r: r["loop"].update(times=0), lambda r: r["loop"].pop("times"),
    lambda r: L(0)(r).pop("width"), lambda r: L(2)(r).update(state=257), lambda r: L(2)(r).update(state=0), lambda r: L(2)(r).pop("dt_rank"), lambda r: L(2)(r).update(conv=17),
    lambda r: L(1)(r).pop("mask"), lambda r: L(1)(r)["mask"].update(size=0), lambda r: L(1)(r).pop("diff"), lambda r: L(1)(r).update(kv_heads=4), lambda r: L(1)(r).update(dim=129),
    lambda r: L(1)(r).update(vdim=300), lambda r: L(1)(r)["rot"].update(dims=21), lambda r: L(1)(r)["rot"].update(dims=22), lambda r: L(1)(r).pop("rot"),
    lambda r: MLP(0)(r)["router"].update(top=12), lambda r: MLP(0)(r)["router"].update(experts=513), lambda r: MLP(0)(r)["expert"].pop("limit"),
    lambda r: MLP(0)(r)["shared"].pop("limit"), lambda r: MLP(0)(r).update(kind="mixture"), lambda r: MLP(1)(r).pop("ff"), lambda r: r["layers"][0].update(type="gru"),
    lambda r: r["layers"][0].pop("mlp")])
def test_config_errors(change):
    raw = json.loads(json.dumps(M.naforax_mixed()))
    change(raw)
    with pytest.raises(LayeredConfigError):
        naforax_config(raw)


def test_registry_validation_and_command_line(tmp_path, capsys):
    from oxibonsai_b200 import cli
    m = M.Model(tmp_path / "tiny", M.naforax_mixed())
    assert R.is_model_dir(m.path) and R.load_model_dir_config(m.path).arch == "Naforax" and R.validate_model_dir(m.path).ok
    assert cli.main(["info", "-m", m.path, "--json"]) == 0
    info = json.loads(capsys.readouterr().out)
    layers = info["config"]["layer_list"]
    assert info["architecture"] == "Naforax" and info["valid"] and [l["mixer"] for l in layers[:3]] == ["mingru", "attention", "selective"]
    assert info["config"]["loop"] == {"start": 1, "stop": 4, "times": 3} and layers[1]["chunk"] == 70 and layers[0]["mlp"]["shared"]["ff"] == 56
    assert cli.main(["info", "-m", m.path]) == 0
    out = capsys.readouterr().out
    assert "layer 3: mixer attention" in out and "feed-forward 40 x 3 of 11" in out and "layers 1-3 run 3 times" in out
    assert cli.main(["validate", "-m", m.path]) == 0
    w = {k: v.float() for k, v in m.w.items() if k != "l0.mlp.shared.sg"}
    w["l0.mlp.correction"] = torch.zeros(11)
    M.write(m.path, m.cfg, w)
    v = R.validate_model_dir(m.path)
    assert any("l0.mlp.shared.sg" in e for e in v.errors) and v.warnings == ["unused tensor l0.mlp.correction"]


def test_scan_weights():
    """The projections a selective scan reads start at multiples of four columns."""
    from oxibonsai_b200.models.layered import ScanWeights
    spec = naforax_config(M.naforax([M.mamba1(50, 7, 5, 3)])).layer_specs[0].mixer
    x, dt = rand(19, 50).bfloat16(), rand(50, 5, seed=1).bfloat16()
    w = ScanWeights.load(spec, x, dt, "cpu")
    assert w.read.columns == [0, 8, 16] and (w.read.n, w.read.kp, w.step.n, w.step.kp) == (24, 128, 50, 128)
    assert torch.equal(w.read.data[:5, :50], x[:5]) and torch.equal(w.read.data[8:15, :50], x[5:12]) and torch.equal(w.read.data[16:23, :50], x[12:])
    assert not w.read.data[5:8].any() and not w.read.data[:, 50:].any() and not w.step.data[:, 5:].any()


def test_conv_weight_order():
    from oxibonsai_b200.ops.layered_ops import conv_weight
    w, x = rand(6, 3), rand(9, 6, seed=1)
    t = conv_weight(w)
    want = O.causal_conv(x, w, torch.zeros(6, dtype=torch.float64))
    assert torch.allclose(want[5], x[5] * t[0] + x[4] * t[1] + x[3] * t[2]) and torch.allclose(want[0], x[0] * t[0])


def test_scans_are_cut_by_a_plan():
    from oxibonsai_b200.models.layered import SCAN_COST, SegmentPlan, plan_segments
    few, many = SegmentPlan(16, SCAN_COST), SegmentPlan(1200, SCAN_COST)
    assert plan_segments([4096], few, 148) > 0 and plan_segments([4096], many, 148) == 0 and plan_segments([64], few, 148) == 0


# ---- the oracle -----------------------------------------------------------------------------------------------------------------------
def test_chunks():
    m = O.chunk_mask(9, 4)
    assert [int(r.sum()) for r in m] == [1, 2, 3, 4, 1, 2, 3, 4, 1] and m[7, 4] and not m[7, 3] and not m[4, 3] and not m[4, 5]


def test_differential_attention_of_equal_maps():
    """With both maps alike the difference is a multiple of one attention, which the norm takes out."""
    raw = M.differential(2, 1, 6, 5, 0.3, 40, 4)["mixer"]
    w = {k: rand(*s, seed=i) for i, (k, s) in enumerate((("q", (24, 8)), ("k", (12, 8)), ("v", (5, 8)), ("g", (10, 8)), ("o", (8, 10)), ("q.b", (24,)), ("k.b", (12,)),
                                                           ("v.b", (5,)), ("o.b", (8,)), ("q.norm", (6,)), ("k.norm", (6,))))}
    w.update({n: 0.2 * rand(6, seed=40 + i) for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))})
    lam = O.difference_factor(w, "", raw["diff"])
    assert abs(float(lam) - (math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.4)) < 1e-12
    for n, heads in (("q", 2), ("k", 1)):
        for t in (w[n], w[n + ".b"]):
            v = t.view(heads, 2, 6, -1)
            v[:, 1] = v[:, 0]
    h = rand(7, 8, seed=90)
    got = O.differential_mixer(h, w, "", raw, 1e-12)
    q = O.rotate_pairs(O.rms_norm((O.linear(h, w["q"]) + w["q.b"]).view(7, 4, 6), w["q.norm"], 1e-12), 0, raw["rot"])
    k = O.rotate_pairs(O.rms_norm((O.linear(h, w["k"]) + w["k.b"]).view(7, 2, 6), w["k.norm"], 1e-12), 0, raw["rot"])
    v = O.linear(h, w["v"]) + w["v.b"]
    out = [0.6 * O.rms(torch.sign(1 - lam) * O.masked_attention(q[:, 2 * a], k[:, 0], v, 0.3, O.chunk_mask(7, 40)), 1e-12) for a in range(2)]
    want = O.linear(torch.cat(out, dim=1) * torch.sigmoid(O.linear(h, w["g"])), w["o"]) + w["o.b"]
    assert torch.allclose(got, want, atol=1e-8)


def test_mingru_state():
    z, c = torch.sigmoid(rand(12, 5)), rand(12, 5, seed=1)
    whole = O.mingru_scan(z, c)
    assert torch.allclose(whole[7:], O.mingru_scan(z[7:], c[7:], whole[6]))
    a = 1.0 - z                                        # closed form
    assert torch.allclose(whole[3], z[3] * c[3] + a[3] * (z[2] * c[2] + a[2] * (z[1] * c[1] + a[1] * z[0] * c[0])))
    u = torch.tensor([-2.0, 0.0, 3.0], dtype=torch.float64)
    assert torch.allclose(O.mingru_candidate(u), torch.tensor([torch.sigmoid(u[0]), 0.5, 3.5], dtype=torch.float64))


def test_selective_scan_state():
    x, dt, A, B, C, D = rand(9, 4), rand(9, 4, seed=1).exp(), -rand(4, 3, seed=2).exp(), rand(9, 3, seed=3), rand(9, 3, seed=4), rand(4, seed=5)
    whole, last = O.selective_scan(x, dt, A, B, C, D)
    first, mid = O.selective_scan(x[:5], dt[:5], A, B[:5], C[:5], D)
    rest, end = O.selective_scan(x[5:], dt[5:], A, B[5:], C[5:], D, mid)
    assert torch.allclose(whole, torch.cat([first, rest])) and torch.allclose(last, end)
    want = sum((C[2] * B[s] * torch.exp(A * dt[s + 1:3].sum(0)[:, None])).sum(-1) * dt[s] * x[s] for s in range(3)) + D * x[2]
    assert torch.allclose(whole[2], want)
    # a segment's state carries over as the start of the next one
    _, local = O.selective_scan(x[5:], dt[5:], A, B[5:], C[5:], D)
    assert torch.allclose(last, torch.exp(A * dt[5:].sum(0)[:, None]) * mid + local)


def test_gelu_through_a_sigmoid():
    """The gate of the kernels: alpha = 2 sqrt(2 / pi), a cubic term inside the sigmoid."""
    from oxibonsai_b200.models.layered_config import gelu_mlp
    z, m = torch.linspace(-8, 8, 400, dtype=torch.float64), gelu_mlp(8)
    assert torch.allclose(O.gelu_tanh(z), z * torch.sigmoid(m.alpha * (z + m.cubic * z ** 3)), atol=1e-12) and m.limit == math.inf and m.offset == 0.0
    assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


def test_softmax_routing():
    z = torch.tensor([2.0, -1.0, 0.5, 3.0], dtype=torch.float64)
    chosen, weights = O.softmax_route(z, 2)
    s = torch.softmax(z, 0)
    assert chosen == [3, 0] and torch.allclose(weights, s[[3, 0]]) and float(weights.sum()) < 1.0


def test_grouped_norm():
    x, w = rand(3, 12), rand(12, seed=1)
    assert torch.allclose(O.grouped_norm(x, w, 1, 1e-3), O.rms_norm(x, w, 1e-3))
    assert torch.allclose(O.grouped_norm(x, w, 3, 1e-3)[:, 4:8], O.rms_norm(x[:, 4:8], w[4:8], 1e-3))


def oracle_model(seed, cfg=None):
    m = M.Model.__new__(M.Model)
    m.cfg = cfg or M.naforax_mixed()
    m.w = {k: v.double() for k, v in O.random_weights(m.cfg, seed).items()}
    return m


def test_loop_is_its_layers_written_out():
    """Two passes are the layers in a row, with the embedding and the steps added between."""
    m = oracle_model(1, M.naforax([M.mingru(20), M.differential(2, 2, 8, 8, dims=4, mlp=M.gelu(16))], (0, 2, 2), width=64, vocab=40))
    tokens = m.tokens(9)
    x = first = m.w["embed"][torch.tensor(tokens)]
    for t in range(2):
        x = x + m.w["loop.step"][t] + (first if t else 0.0)
        for i in range(2):
            x = O.naforax_layer(x, m.w, f"l{i}.", m.cfg["layers"][i], m.cfg["norm"], m.cfg["residual_mult"])
    logits, kept = O.forward(m.cfg, m.w, tokens, True)
    assert torch.allclose(kept[-1], x) and kept.shape[0] == 4
    raw = O.linear(O.grouped_norm(x, m.w["final.norm"], 4, 1e-5), m.w["head"])
    assert torch.allclose(logits, 9.0 * torch.tanh(raw / 9.0)) and float(raw.abs().max()) > 2.0


def test_model_is_causal():
    m = oracle_model(3)
    a = m.tokens(30)
    assert torch.allclose(m.logits(a)[:20], m.logits(a[:20]), atol=1e-9)


def test_seeded_routers_leave_no_close_call():
    """The tests' models choose experts far from any other choice, and use them all."""
    m = oracle_model(4)
    tokens = m.tokens(120)
    runs = O.loop_runs(7, m.cfg["loop"])
    _, kept = O.forward(m.cfg, m.w, tokens, True)
    for n, (l, _) in enumerate(runs):
        mlp = m.cfg["layers"][l]["mlp"]
        if mlp is None or mlp["kind"] != "moe":
            continue
        z = O.linear(O.grouped_norm(kept[n], m.w[f"l{l}.norm2"], 4, 1e-5), m.w[f"l{l}.mlp.router"])       # the code's dimensions of every layer are the same
        top = mlp["router"]["top"]
        order = torch.sort(z, dim=-1, descending=True).values
        if top < mlp["router"]["experts"]:
            assert float((order[:, top - 1] - order[:, top]).min()) > 0.15
        assert len({e for row in z for e in O.softmax_route(row, top)[0]}) == mlp["router"]["experts"]
