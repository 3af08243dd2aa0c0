"""CPU side of the Bivizen integration: configuration, registry, cache geometry, weight checks, and sanity of the
float64 oracle itself (causality, value mixing, the cap, the convolution's reach, the recurrences against closed forms)."""
import json

import pytest
import torch

from oracle import bivizen_oracle as O
from tests.test_bivizen_gpu import CONFIGS
from vila_b200.model.bivizen import BivizenConfig, BivizenForCausalLM
from vila_b200.model.moronex import stack_rows
from vila_b200.model.registry import LANGUAGE_MODELS, language_model_architecture

F64 = torch.float64


def random_weights(cfg_dict, rank, seed=0):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in BivizenConfig.from_dict(cfg_dict).tensor_shapes().items():
        s = tuple(rank if k < 0 else k for k in s)
        out[n] = (torch.randn(s, generator=g) * (0.3 if len(s) < 2 else 1.5 / s[-1] ** 0.5)).to(torch.bfloat16)
    return out


@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_shapes_and_cache_geometry(name):
    d, rank = CONFIGS[name]
    cfg = BivizenConfig.from_dict(d)
    assert cfg.to_dict() == json.loads(json.dumps(d))
    shapes = cfg.tensor_shapes()
    model = BivizenForCausalLM(cfg, "cpu")
    pools, states = model.latent_widths(), model.state_shapes()
    for i, spec in enumerate(d["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        assert ((p + "ls2") in shapes) == (spec["mlp"] is not None) == ((p + "mlp.down") in shapes)
        assert shapes[p + "mix.o"] == (d["width"], m["heads"] * m["vdim"])
        if spec["type"] == "attention":
            assert pools[i] == m["kv_heads"] * (m["dim"] + m["vdim"]) and (i, "scan") not in states
            assert ((p + "mix.vmix") in shapes) == m["v_mix"] and shapes[p + "mix.v.b"] == (m["kv_heads"] * m["vdim"],)
        else:
            assert i not in pools and states[(i, "scan")] == (m["heads"], m["vdim"], m["dim"])
        if spec["type"] == "delta":
            chans = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
            assert states.get((i, "conv")) == ((m["conv"] - 1, chans) if m["conv"] > 1 else None)
            assert shapes[p + "mix.k.conv"] == (m["kv_heads"] * m["dim"], m["conv"])
        if spec["type"] == "gla":
            assert shapes[p + "mix.a1"] == (-1, d["width"]) and shapes[p + "mix.a2"] == (m["heads"] * m["dim"], -1)


def test_bad_configs_are_refused():
    for change in (lambda d: d["layers"][0].update(type="something_else"),
                   lambda d: d["layers"][0]["mixer"].update(kv_heads=4),        # 6 heads over 4 query / key heads
                   lambda d: d["layers"][0]["mixer"].update(conv=0),
                   lambda d: d["layers"][0]["mixer"].update(dim=1000),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=14),    # more columns than the head has
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=5),
                   lambda d: d["layers"][1]["mixer"].update(softcap=-1.0),
                   lambda d: d["layers"][2]["mixer"].update(tau=0.0),
                   lambda d: d["layers"][4]["mixer"].update(vdim=24),           # cannot be mixed with the first mixing layer's values
                   lambda d: d["layers"][0]["mlp"].update(kind="moe")):
        d = json.loads(json.dumps(CONFIGS["odd"][0]))
        change(d)
        with pytest.raises(ValueError):
            BivizenConfig.from_dict(d)


def test_registry_names_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["ones"][0]))
    assert language_model_architecture(tmp_path) == "Bivizen" and LANGUAGE_MODELS["Bivizen"] is BivizenForCausalLM


def test_weights_are_checked_against_the_config():
    d, rank = CONFIGS["odd"]
    w = random_weights(d, rank)
    make = lambda: BivizenForCausalLM(BivizenConfig.from_dict(d), "cpu", torch.float32)
    model = make().load_weights(w)
    L = model.layers[2]
    assert L.in_off["a1"][1] == rank and L.a2.shape == (24, rank)         # 21 key channels, rows padded to a multiple of 8
    assert model.layers[4].v_mix == pytest.approx(float(w["l4.mix.vmix"]))
    assert model.layers[0].conv.shape == (2 * 3 * 10 + 6 * 14, 3)
    assert torch.equal(model.layers[1].in_b[:48], w["l1.mix.q.b"].float()) and float(model.layers[1].in_b[-4:].abs().max()) == 0.0
    bad = dict(w)
    bad["l0.mlp.down"] = bad["l0.mlp.down"][:-1]
    with pytest.raises(ValueError):
        make().load_weights(bad)
    bad = dict(w)
    bad["l2.mix.a2"] = torch.zeros(21, rank + 1)                          # another rank than a1
    with pytest.raises(ValueError):
        make().load_weights(bad)
    del bad["l3.mix.g"]
    with pytest.raises(KeyError):
        make().load_weights(bad)


def test_stacked_projections_start_at_multiples_of_eight_rows():
    a, b = torch.arange(6.0).view(3, 2), torch.ones(9, 2)
    w, off = stack_rows([("a", a), ("b", b)])
    assert w.shape == (24, 2) and off == {"a": (0, 3), "b": (8, 9)}
    assert torch.equal(w[:3], a) and torch.equal(w[8:17], b) and float(w[3:8].abs().max()) == 0.0


@pytest.mark.parametrize("name", list(CONFIGS))
def test_oracle_is_causal(name):
    d, rank = CONFIGS[name]
    w = random_weights(d, rank, seed=1)
    toks = torch.randint(0, d["vocab"], (40,), generator=torch.Generator().manual_seed(2)).tolist()
    a = O.forward(d, w, toks)
    other = list(toks)
    other[25] = (other[25] + 1) % d["vocab"]
    b = O.forward(d, w, other)
    assert torch.allclose(a[:25], b[:25], rtol=0, atol=1e-12) and not torch.allclose(a[25:], b[25:])


def test_oracle_value_mixing_and_the_unused_first_number():
    d, rank = CONFIGS["odd"]
    w = random_weights(d, rank, seed=3)
    toks = list(range(20))
    base = O.forward(d, w, toks)
    for name, changes in (("l1.mix.vmix", False), ("l4.mix.vmix", True)):   # the first mixing layer has nothing to mix in
        w2 = dict(w)
        w2[name] = torch.tensor(0.9, dtype=torch.bfloat16)
        assert torch.equal(O.forward(d, w2, toks), base) != changes
    # with a mixing number of one, the later layer's own values do not matter
    w2 = dict(w)
    w2["l4.mix.vmix"] = torch.tensor(1.0)
    w3 = dict(w2)
    w3["l4.mix.v"] = w2["l4.mix.v"] * 3
    assert torch.allclose(O.forward(d, w2, toks), O.forward(d, w3, toks))


def test_oracle_cap_and_rotation():
    s = torch.tensor([-1e6, -1.0, 0.0, 0.01, 1e6], dtype=F64)
    c = O.softcap(s, 20.0)
    assert c[0] == -20 and c[-1] == 20 and c[2] == 0 and abs(float(c[3]) - 0.01) < 1e-8
    assert torch.equal(O.softcap(s, 0.0), s)
    u = torch.randn(9, 1, 8, dtype=F64, generator=torch.Generator().manual_seed(1))
    r = O.rotate_halves(u, 6, 100.0)
    assert torch.equal(r[..., 6:], u[..., 6:]) and torch.allclose(r.norm(dim=-1), u.norm(dim=-1)) and torch.equal(r[0], u[0])
    # column 0 turns with column 3 by one radian per position
    one = torch.zeros(2, 1, 8, dtype=F64)
    one[:, 0, 0] = 1.0
    assert torch.allclose(O.rotate_halves(one, 6, 100.0)[1, 0, [0, 3]], torch.tensor([0.5403023058681398, 0.8414709848078965], dtype=F64))


def test_oracle_recurrences_against_closed_forms():
    out = O.causal_conv(torch.eye(6, dtype=F64)[:, 3:4].expand(-1, 2), torch.tensor([[1.0, 2.0, 3.0], [4.0, 5.0, 6.0]], dtype=F64))
    assert out[3].tolist() == [3.0, 6.0] and out[5].tolist() == [1.0, 4.0] and float(out[:3].abs().max()) == 0.0
    v = torch.randn(5, 2, dtype=F64, generator=torch.Generator().manual_seed(1))
    k = torch.eye(3, dtype=F64)[[0, 1, 0, 2, 0]]
    one = torch.ones(5, dtype=F64)
    o, S = O.delta_rule(k, k, v, one, one)                # a full write under a unit key is read back, and replaces
    assert torch.allclose(o, v) and torch.allclose(S, torch.stack([v[4], v[1], v[3]]))
    o, S = O.delta_rule(k, k, v, one * 0.0, one)
    assert float(o.abs().max()) == 0.0                    # a step size of zero writes nothing
    q = torch.ones(4, 2, dtype=F64)
    kk = torch.tensor([[1.0, 1.0]] + [[0.0, 0.0]] * 3, dtype=F64)
    al = torch.tensor([[0.5, 0.25]] * 4, dtype=F64)
    o, _ = O.gated_linear_rule(q, kk, torch.ones(4, 1, dtype=F64), al)
    assert torch.allclose(o[:, 0], torch.tensor([2.0, 0.75, 0.3125, 0.140625], dtype=F64))
    z = torch.tensor([-50.0, 0.0, 50.0], dtype=F64)
    assert torch.allclose(O.softplus(z), torch.nn.functional.softplus(z))
