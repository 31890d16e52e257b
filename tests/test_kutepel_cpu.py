"""Kutepel decoders without a GPU: configuration, registry, command line, batches of portions, and the oracle's mechanisms against other forms."""
import json
import math

import layered_models as M
import layered_oracle as O
import pytest
import torch

from oxibonsai_b200.models import registry as R
from oxibonsai_b200.models.layered_config import LayeredConfigError, kutepel_config


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ---- configuration ------------------------------------------------------------------------------------------------------------------
def test_config_reads_every_layer():
    raw = M.kutepel_mixed()
    c = kutepel_config(raw, "tiny")
    assert (c.width, c.vocab, c.eps, c.layers, c.residual_mult, c.side_by_side, c.layer_norm, c.embed_scale) == (152, 331, 1e-5, 7, 0.4, True, True, 1.0)
    assert c.attention_layers == list(range(7)) and c.recurrent_layers == [] and c.max_visible is None and c.expert_layers == [0, 1, 3, 5, 6]
    a, b, s = (c.layer_specs[i].mixer for i in (0, 1, 3))
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.rank, a.scale, a.rotary.base, a.rotary.interleaved, a.rotary.scaling) == (3, 20, 12, 28, 72, 0.3, 700.0, True, None)
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.sink, b.normed, b.kv_from, b.rotary.dims) == (6, 2, 40, 24, True, False, None, 40)
    assert s.kv_from == 1 and [n for n, _ in s.sections] == ["q"] and [n for n, _ in b.sections] == ["q", "k", "v"]
    e = c.experts(6)
    assert (e.ff, e.router.experts, e.router.top, e.router.groups, e.router.keep, e.router.scale) == (64, 20, 4, 10, 2, 2.0)
    assert c.norm_names(0) == [("l0.norm1", None)] and c.layer_specs[2].mlp is None
    assert c.tensor_shapes() == {k: tuple(v) for k, v in O.tensor_shapes(raw).items()}
    assert c.param_count() == sum(math.prod(s) for s in O.tensor_shapes(raw).values())
    for i in (0, 1, 2, 5):
        got, want = c.layer_specs[i].mixer.rotary.frequencies, O.frequencies(raw["layers"][i]["mixer"]["rot"])
        assert len(got) == len(want) and all(abs(x - y) < 1e-15 for x, y in zip(got, want))


def test_optional_parts():
    raw = M.kutepel([M.latent(mlp=M.experts(8, 4, 2, 1, 1)), M.rotary(dims=0)])
    del raw["layers"][0]["mlp"]["router"]["groups"]
    raw["layers"][1]["mixer"]["kv_from"] = None
    c = kutepel_config(raw)
    assert (c.experts(0).router.groups, c.experts(0).router.keep) == (1, 1) and c.layer_specs[1].mixer.rotary is None and c.layer_specs[1].mixer.kv_from is None


L = lambda i: lambda r: r["layers"][i]["mixer"]
ROUTER = lambda r: r["layers"][0]["mlp"]["router"]


@pytest.mark.parametrize("change", [
    lambda r: r.pop("residual_mult"), lambda r: r["layers"][0].pop("mlp"), lambda r: r["layers"][0].update(type="latent"), lambda r: r["layers"][0]["mlp"].update(kind="dense"),
    lambda r: L(0)(r).pop("kv_rank"), lambda r: L(0)(r).update(kv_rank=513), lambda r: L(0)(r).update(rot_dim=10), lambda r: L(0)(r)["rot"].update(dims=6),
    lambda r: L(0)(r).update(dim=250), lambda r: L(0)(r).update(vdim=300), lambda r: L(2)(r).update(kv_rank=512, rot_dim=160, rot={"base": 10.0, "dims": 160}),
    lambda r: L(1)(r)["rot"]["scaling"].pop("original"), lambda r: L(1)(r)["rot"]["scaling"].update(low=6.0), lambda r: L(1)(r)["rot"].update(base=-1),
    lambda r: L(1)(r).update(kv_heads=4), lambda r: L(1)(r).pop("rot"), lambda r: L(3)(r).update(kv_from=0), lambda r: L(3)(r).update(kv_from=3),
    lambda r: L(3)(r).update(kv_from=5), lambda r: L(5)(r).update(kv_from=3), lambda r: L(3)(r).update(kv_from=4), lambda r: L(3)(r).update(kv_from=-1),
    lambda r: ROUTER(r).update(top=9), lambda r: ROUTER(r).update(experts=13), lambda r: ROUTER(r)["groups"].update(keep=4), lambda r: ROUTER(r)["groups"].pop("count"),
    lambda r: ROUTER(r).pop("scale"), lambda r: ROUTER(r).update(experts=600), lambda r: r["layers"][0]["mlp"].pop("expert")])
def test_config_errors(change):
    raw = json.loads(json.dumps(M.kutepel_mixed()))
    change(raw)
    with pytest.raises(LayeredConfigError):
        kutepel_config(raw)


def test_registry_validation_and_command_line(tmp_path, capsys):
    from oxibonsai_b200 import cli
    m = M.Model(tmp_path / "tiny", M.kutepel_mixed())
    assert R.is_model_dir(m.path) and R.load_model_dir_config(m.path).arch == "Kutepel" and R.validate_model_dir(m.path).ok
    assert cli.main(["info", "-m", m.path, "--json"]) == 0
    info = json.loads(capsys.readouterr().out)
    layers = info["config"]["layer_list"]
    assert info["architecture"] == "Kutepel" and info["valid"] and [l["mixer"] for l in layers[:2]] == ["latent", "attention"]
    assert layers[1]["rotary"]["scaling"]["factor"] == 5.0 and layers[0]["mlp"]["router"]["top"] == 3 and layers[0]["mlp"]["limit"] is None
    assert cli.main(["info", "-m", m.path]) == 0
    out = capsys.readouterr().out
    assert "layer 3: mixer attention" in out and "feed-forward 64 x 4 of 20" in out
    assert cli.main(["validate", "-m", m.path]) == 0
    w = {k: v.float() for k, v in m.w.items() if k != "l0.mlp.e3.up"}
    w["l3.mix.k"] = torch.zeros(80, 152)
    M.write(m.path, m.cfg, w)
    v = R.validate_model_dir(m.path)
    assert any("l0.mlp.e3.up" in e for e in v.errors) and v.warnings == ["unused tensor l3.mix.k"]


def test_contexts_are_grouped():
    from oxibonsai_b200.models.layered import group_contexts
    lists = [(0, 40, 0, 0), (40, 50, 1, 100), (90, 33, 2, 400), (123, 60, 3, 0)]
    assert group_contexts(lists, 1000) == [lists] and group_contexts([], 10) == []
    assert group_contexts(lists, 433) == [lists[:2], [lists[2]], [lists[3]]]
    assert group_contexts(lists, 193) == [lists[:2], [lists[2]], [lists[3]]]        # one that does not fit stands alone
    assert group_contexts(lists, 189) == [[e] for e in lists]


def test_latent_weights():
    """The padded forms hold the same matrices."""
    from oxibonsai_b200.models.layered import LatentWeights
    raw = M.kutepel([M.latent(3, 13, 6, 21, 50)])
    spec = kutepel_config(raw).layer_specs[0].mixer
    uk, uv = rand(39, 50).bfloat16(), rand(63, 50, seed=1).bfloat16()
    w = LatentWeights.load(spec, uk, uv, "cpu")
    assert w.keys.shape == (3, 64, 32) and w.values.shape == (3, 21, 64) and (w.expand.n, w.expand.kp) == (3 * 40, 128)
    assert torch.equal(w.keys[:, :50, :13], uk.view(3, 13, 50).transpose(1, 2)) and torch.equal(w.values[:, :, :50], uv.view(3, 21, 50))
    e = w.expand.data.view(3, 40, 128)
    assert torch.equal(e[:, :13, :50], uk.view(3, 13, 50)) and torch.equal(e[:, 16:37, :50], uv.view(3, 21, 50))
    for t, used in ((w.keys, 39 * 50), (w.values, 63 * 50), (w.expand.data, 102 * 50)):
        assert int((t != 0).sum()) <= used


# ---- the oracle -----------------------------------------------------------------------------------------------------------------------
def test_rotation_is_relative():
    x, y, rot = rand(1, 2, 10), rand(1, 2, 10, seed=1), M.rotation(6, 100.0, {"factor": 3.0, "low": 1.0, "high": 2.0, "original": 30})
    dot = lambda p, r: (O.rotate_pairs(x, p, rot) * O.rotate_pairs(y, r, rot)).sum(-1)
    assert torch.allclose(dot(9, 4), dot(25, 20)) and not torch.allclose(dot(9, 4), dot(9, 5))
    r = O.rotate_pairs(x, 3, rot)
    a = 3 * O.frequencies(rot)[1]
    assert torch.equal(r[..., 6:], x[..., 6:])
    assert torch.allclose(r[0, 0, 2], x[0, 0, 2] * math.cos(a) - x[0, 0, 3] * math.sin(a)) and torch.allclose(r[0, 0, 3], x[0, 0, 3] * math.cos(a) + x[0, 0, 2] * math.sin(a))


def test_stretched_frequencies():
    f = [1000.0 ** (-2 * i / 16) for i in range(8)]
    got = O.frequencies(M.rotation(16, 1000.0, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}))
    kinds = set()
    for a, b in zip(f, got):
        length = 2 * math.pi / a
        if length < 25:
            assert b == a
            kinds.add("kept")
        elif length > 100:
            assert b == a / 4
            kinds.add("stretched")
        else:
            assert a / 4 < b < a
            kinds.add("between")
    assert kinds == {"kept", "stretched", "between"}


def test_sink_takes_weight():
    q, k, v = rand(5, 4), rand(5, 4, seed=1), rand(5, 3, seed=2)
    plain = O.sink_attention(q, k, v, 0.5)
    assert torch.allclose(plain, torch.nn.functional.scaled_dot_product_attention(q[None], k[None], v[None], is_causal=True, scale=0.5)[0])
    s = torch.tensor(0.7, dtype=torch.float64)
    z = torch.stack([torch.exp((q[t] @ k[: t + 1].T) * 0.5).sum() for t in range(5)])
    assert torch.allclose(O.sink_attention(q, k, v, 0.5, s), plain * (z / (z + math.exp(0.7)))[:, None])


def test_latent_is_attention_over_latents():
    """Expanding the keys and values, and attending to the latents themselves, are the same."""
    m = M.latent(2, 6, 4, 5, 9, 0.4)["mixer"]
    w = {k: rand(*s, seed=i) for i, (k, s) in enumerate((("q", (20, 8)), ("dkv", (13, 8)), ("dkv.norm", (9,)), ("uk", (12, 9)), ("uv", (10, 9)), ("g", (10, 8)), ("o", (8, 10))))}
    h = rand(7, 8, seed=9)
    q = O.linear(h, w["q"]).view(7, 2, 10)
    c = O.rms_norm(O.linear(h, w["dkv"])[:, :9], w["dkv.norm"], 1e-5)
    row = torch.cat([c, O.rotate_pairs(O.linear(h, w["dkv"])[:, None, 9:], 0, m["rot"])[:, 0]], dim=1)
    out = []
    for a in range(2):
        qa = torch.cat([q[:, a, :6] @ w["uk"][6 * a:6 * a + 6], O.rotate_pairs(q[:, a:a + 1, 6:], 0, m["rot"])[:, 0]], dim=1)
        out.append(O.sink_attention(qa, row, c, 0.4) @ w["uv"][5 * a:5 * a + 5].T)
    want = O.linear(torch.cat(out, dim=1) * torch.sigmoid(O.linear(h, w["g"])), w["o"])
    assert torch.allclose(O.latent_attention_mixer(h, w, "", m, 1e-5), want)


def test_routing():
    z = torch.tensor([2.0, -1.0, 0.5, 0.4, -3.0, 3.0], dtype=torch.float64)
    s, none = torch.sigmoid(z), torch.zeros(6, dtype=torch.float64)
    chosen, weights = O.route(z, none, 2, 1, 1, 1.0)
    assert chosen == [5, 0] and torch.allclose(weights, s[[5, 0]] / (s[5] + s[0]))
    # groups (0, 1), (2, 3), (4, 5): sums 1.15, 1.22, 1.0; the best two leave out expert 5, the best single one
    assert O.route(z, none, 2, 3, 2, 1.0)[0] == [0, 2]
    # the correction moves the choice, not the weights, and may make every choice negative
    chosen, weights = O.route(z, torch.tensor([-3.0, -3.0, -2.0, -2.0, -1.5, -1.5], dtype=torch.float64), 2, 3, 1, 0.5)
    assert chosen == [5, 4] and torch.allclose(weights, 0.5 * s[[5, 4]] / (s[5] + s[4]))
    assert abs(O.route_margin(z, none, 2, 3, 2) - min(float(s[0] + s[1] - s[4] - s[5]), float(s[2] - s[3]))) < 1e-12
    assert O.route_margin(z, none, 6, 1, 1) == math.inf


def test_layer_norm():
    x, w = rand(3, 12), rand(12, seed=1)
    assert torch.allclose(O.layer_norm(x, w, 1e-3), torch.nn.functional.layer_norm(x, (12,), w, None, 1e-3))


def oracle_model(seed):
    m = M.Model.__new__(M.Model)
    m.cfg = M.kutepel_mixed()
    m.w = {k: v.double() for k, v in O.random_weights(m.cfg, seed).items()}
    return m


def test_model_is_causal():
    m = oracle_model(3)
    a = m.tokens(30)
    assert torch.allclose(m.logits(a)[:20], m.logits(a[:20]), atol=1e-9)


def test_seeded_routers_leave_no_close_call():
    """The tests' models choose experts by the token alone, far from any other choice, and use them all."""
    m = oracle_model(4)
    tokens = m.tokens(120)
    _, kept = O.forward(m.cfg, m.w, tokens, True)
    x = m.w["embed"][torch.tensor(tokens)]
    for l, layer in enumerate(m.cfg["layers"]):
        if layer["mlp"] is not None:
            p, r = f"l{l}.mlp.", layer["mlp"]["router"]
            z = O.linear(O.layer_norm(x, m.w[f"l{l}.norm1"], 1e-5), m.w[p + "router"])
            a = (m.w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"])
            assert min(O.route_margin(row, *a) for row in z) > 0.008
            assert len({e for row in z for e in O.route(row, *a, 1.0)[0]}) >= r["experts"] // 2
        x = kept[l]
