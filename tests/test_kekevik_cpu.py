"""Kekevik decoders without a GPU: configuration, registry, command line, and the oracle's mechanisms against other forms."""
import json
import math

import layered_models as M
import layered_oracle as O
import pytest
import torch

from oxibonsai_b200.models import registry as R
from oxibonsai_b200.models.layered_config import LayeredConfigError, kekevik_config


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ---- configuration ------------------------------------------------------------------------------------------------------------------
def test_config_reads_every_layer():
    raw = M.kekevik_mixed()
    c = kekevik_config(raw, "tiny")
    assert (c.width, c.vocab, c.eps, c.layers, c.embed_scale, c.pre_norm) == (152, 331, 1e-5, 6, 3.5, True)
    assert c.attention_layers == [0, 3] and c.recurrent_layers == [0, 1, 2, 3, 4, 5] and c.max_visible is None
    left, right = (b.spec for b in c.layer_specs[0].mixer.branches)
    assert [b.scale for b in c.layer_specs[0].mixer.branches] == [0.7, 1.3]
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.softcap, left.temp_coef, left.temp_every) == (6, 2, 40, 24, 0.3, 6.0, 0.7, 19.0)
    assert (left.window, left.slope_exponent, left.norm_weights, left.gated, left.group) == (0, None, False, False, 3)
    assert (right.heads, right.dim, right.vdim, right.groups, right.norm_parts, right.conv) == (6, 28, 20, 2, 3, 4)
    assert right.decay is None and right.gate_first and right.conv_channels == 120 + 2 * 2 * 28
    ret, light = c.layer_specs[1].mixer, c.layer_specs[2].mixer
    assert ret.rotary.dims == 24 and ret.rotary.base == 5000.0 and ret.key_scale == 24 ** -0.5 and ret.norm_parts == 3 and not ret.norm_weight and ret.gate == "silu"
    assert light.activation and light.norm_parts == 1 and light.norm_weight and light.rotary is None and light.key_scale == 1.0 and light.gate == "sigmoid"
    assert c.layer_specs[1].mlp is None and c.layer_specs[2].mlp.ff == 90
    assert c.tensor_shapes() == {k: tuple(v) for k, v in O.tensor_shapes(raw).items()}
    assert c.param_count() == sum(math.prod(s) for s in O.tensor_shapes(raw).values())


L = lambda i: lambda r: r["layers"][i]["mixer"]


@pytest.mark.parametrize("change", [
    lambda r: r.pop("embedding"), lambda r: r["embedding"].pop("scale"), lambda r: r["layers"][1].update(type="mlstm"), lambda r: r["layers"][0].pop("mlp"),
    lambda r: L(1)(r)["decay"].pop(), lambda r: L(1)(r).pop("decay"), lambda r: L(2)(r)["decay"].__setitem__(0, 1.5), lambda r: L(2)(r)["decay"].__setitem__(0, "a"),
    lambda r: L(1)(r)["rot"].update(dims=7), lambda r: L(1)(r)["rot"].update(dims=26), lambda r: L(1)(r)["rot"].update(base=0), lambda r: L(1)(r).update(dim=513),
    lambda r: L(0)(r)["left"].update(kv_heads=4), lambda r: L(0)(r)["left"].update(softcap=0), lambda r: L(0)(r)["left"]["q_temp"].update(every=0),
    lambda r: L(0)(r)["left"].update(vdim=300), lambda r: L(0)(r)["right"].update(groups=4), lambda r: L(0)(r)["right"].update(norm_groups=7),
    lambda r: L(0)(r)["right"].update(conv=0), lambda r: L(0)(r).pop("left_scale"), lambda r: L(0)(r).pop("right"), lambda r: r["layers"][0]["mlp"].update(kind="moe")])
def test_config_errors(change):
    raw = json.loads(json.dumps(M.kekevik_mixed()))
    change(raw)
    with pytest.raises(LayeredConfigError):
        kekevik_config(raw)


def test_registry_validation_and_command_line(tmp_path, capsys):
    from oxibonsai_b200 import cli
    m = M.Model(tmp_path / "tiny", M.kekevik_mixed())
    assert R.is_model_dir(m.path) and R.load_model_dir_config(m.path).arch == "Kekevik" and R.validate_model_dir(m.path).ok
    assert cli.main(["info", "-m", m.path, "--json"]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Kekevik" and info["valid"] and info["config"]["attention_layers"] == [0, 3]
    parts = info["config"]["layer_list"][0]["parts"]
    assert [(p["prefix"], p["output_scale"], p["mixer"]) for p in parts] == [("left.", 0.7, "attention"), ("right.", 1.3, "recurrence")] and parts[0]["scale"] == 0.3
    assert cli.main(["info", "-m", m.path]) == 0 and "layer 3: mixer parallel" in capsys.readouterr().out
    assert cli.main(["validate", "-m", m.path]) == 0
    w = {k: v.float() for k, v in m.w.items() if k != "l0.norm1b"}
    M.write(m.path, m.cfg, w)
    assert any("l0.norm1b" in e for e in R.validate_model_dir(m.path).errors)


def test_branches_share_a_buffer():
    from oxibonsai_b200.models.layered import branch_offsets
    assert branch_offsets([7]) == ([0], 7) and branch_offsets([7, 16, 3]) == ([0, 8, 24], 27) and branch_offsets([32, 5]) == ([0, 32], 37)


# ---- the oracle -----------------------------------------------------------------------------------------------------------------------
def test_recurrence_is_the_weighted_sum():
    """Token by token equals the closed form with weights b_s a_(s+1) .. a_t, and resuming from the state the same sequence."""
    n, d, e = 19, 5, 4
    q, k, v, a, b = rand(n, d), rand(n, d, seed=1), rand(n, e, seed=2), torch.rand(n, dtype=torch.float64), torch.rand(n, dtype=torch.float64)
    o, S = O.decayed_memory(q, k, v, a, b)
    for t in range(n):
        w = torch.stack([b[s] * a[s + 1:t + 1].prod() * (k[s] @ q[t]) for s in range(t + 1)])
        assert torch.allclose(o[t], w @ v[: t + 1])
    o1, S1 = O.decayed_memory(q[:8], k[:8], v[:8], a[:8], b[:8])
    o2, S2 = O.decayed_memory(q[8:], k[8:], v[8:], a[8:], b[8:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)


def test_rotation_is_relative():
    x, y = rand(1, 2, 10), rand(1, 2, 10, seed=1)
    dot = lambda p, r: (O.rotate_half(x, p, 100.0, 6) * O.rotate_half(y, r, 100.0, 6)).sum(-1)
    assert torch.allclose(dot(9, 4), dot(25, 20)) and not torch.allclose(dot(9, 4), dot(9, 5))
    r = O.rotate_half(x, 3, 100.0, 6)
    assert torch.equal(r[..., 6:], x[..., 6:])
    a = 3 * 100.0 ** (-2 / 6)
    assert torch.allclose(r[0, 0, 1], x[0, 0, 1] * math.cos(a) - x[0, 0, 4] * math.sin(a)) and torch.allclose(r[0, 0, 4], x[0, 0, 4] * math.cos(a) + x[0, 0, 1] * math.sin(a))


def test_convolution_is_causal():
    x, w, b = rand(6, 3), rand(3, 4, seed=1), rand(3, seed=2)
    y = O.causal_conv(x, w, b)
    for t in range(6):
        assert torch.allclose(y[t], b + sum(w[:, 3 - j] * x[t - j] for j in range(4) if t >= j))
    assert torch.allclose(O.causal_conv(x[:2], w, b), y[:2])


def test_temperature_and_cap():
    t = O.query_temperature(9, 0.5, 3)
    assert torch.allclose(t, torch.tensor([1.0 + 0.5 * math.log(f) for f in (1, 1, 2, 2, 2, 3, 3, 3, 4)], dtype=torch.float64))
    s = torch.tensor([-100.0, 0.01, 100.0])
    assert torch.allclose(O.soft_cap(s, 5.0), torch.tensor([-5.0, 0.01, 5.0]), atol=1e-4)
    q, k, v = rand(5, 4), rand(5, 4, seed=1), rand(5, 3, seed=2)
    assert torch.allclose(O.capped_attention(q, k, v, 0.5, 2.0)[0], v[0])
    assert torch.allclose(O.capped_attention(q, k, v, 0.5, 1e9), torch.nn.functional.scaled_dot_product_attention(q[None], k[None], v[None], is_causal=True, scale=0.5)[0])


def test_grouped_norm():
    x = rand(3, 12)
    y = O.grouped_rms(x, 4, 0.0)
    assert torch.allclose(y.view(3, 4, 3).pow(2).mean(-1), torch.ones(3, 4, dtype=torch.float64)) and torch.allclose(O.grouped_rms(x, 1, 1e-3), O.rms(x, 1e-3))


def test_model_is_causal():
    m = M.Model.__new__(M.Model)
    m.cfg = M.kekevik_mixed()
    m.w = {k: v.double() for k, v in O.random_weights(m.cfg, 3).items()}
    a = m.tokens(30)
    assert torch.allclose(m.logits(a)[:20], m.logits(a[:20]), atol=1e-9)
