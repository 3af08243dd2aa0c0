"""CPU side of the Nibelix integration: configuration, registry, cache geometry, weight checks, and sanity of the
float64 oracle itself (causality, the window, the router's rules, the recurrence and the maps against closed forms)."""
import json
import math

import pytest
import torch

from oracle import nibelix_oracle as O
from tests.test_nibelix_gpu import CONFIGS
from vila_b200.model.nibelix import NibelixConfig, NibelixForCausalLM
from vila_b200.model.registry import LANGUAGE_MODELS, language_model_architecture

F64 = torch.float64


def random_weights(cfg_dict, seed=0):
    g = torch.Generator().manual_seed(seed)
    return {n: (torch.randn(s, generator=g) * (0.3 if len(s) < 2 else 1.5 / s[-1] ** 0.5)).to(torch.bfloat16)
            for n, s in NibelixConfig.from_dict(cfg_dict).tensor_shapes().items()}


@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_shapes_and_cache_geometry(name):
    d = CONFIGS[name]
    cfg = NibelixConfig.from_dict(d)
    assert cfg.to_dict() == json.loads(json.dumps(d))
    shapes = cfg.tensor_shapes()
    model = NibelixForCausalLM(cfg, "cpu")
    pools, states = model.latent_widths(), model.state_shapes()
    for i, spec in enumerate(d["layers"]):
        p, m, f = f"l{i}.", spec["mixer"], spec["mlp"]
        assert ((p + "ls2") in shapes) == ((p + "norm2.alpha") in shapes) == (f is not None)
        assert shapes[p + "norm1.alpha"] == () and shapes[p + "norm1.b"] == (d["width"],)
        assert shapes[p + "mix.o"] == (d["width"], m["heads"] * m["vdim"])
        if spec["type"] == "attention":
            assert pools[i] == m["kv_heads"] * (2 * m["dim"] + m["vdim"]) and (i, "scan") not in states
            assert shapes[p + "mix.k"] == (2 * m["kv_heads"] * m["dim"], d["width"]) and shapes[p + "mix.lq1"] == (m["dim"],)
        else:
            assert i not in pools and states[(i, "scan")] == (m["heads"], m["vdim"], m["dim"])
            assert shapes[p + "mix.norm"] == (m["heads"] * m["vdim"],)
        if f is not None and f["kind"] == "moe":
            r = f["router"]
            assert shapes[p + "mlp.router"] == (r["experts"] + r["identity"], d["width"])
            assert (p + f"mlp.e{r['experts'] - 1}.up") in shapes and (p + f"mlp.e{r['experts']}.up") not in shapes
            assert ((p + "mlp.shared.sg") in shapes) == ("shared" in f)


def test_parts_that_may_be_missing_from_a_configuration():
    d = json.loads(json.dumps(CONFIGS["odd"]))
    for k in ("logit_softcap", "residual_mult"):
        del d[k]
    r = d["layers"][4]["mlp"]["router"]
    for k in ("groups", "identity", "scale"):
        del r[k]
    d["layers"][2]["mixer"]["mask"] = None
    cfg = NibelixConfig.from_dict(d)
    assert (cfg.logit_softcap, cfg.residual_mult, cfg.layers[2].window) == (0.0, 1.0, 0)
    lc = cfg.layers[4]
    assert (lc.groups, lc.keep, lc.identity, lc.router_scale) == (1, 1, 0, 1.0)


def test_bad_configs_are_refused():
    for change in (lambda d: d["layers"][0].update(type="something_else"),
                   lambda d: d["layers"][0]["mixer"].update(kv_heads=4),                 # 6 heads over 4
                   lambda d: d["layers"][0]["mixer"]["rot"].update(dims=12),             # more columns than a map has
                   lambda d: d["layers"][0]["mixer"]["rot"].update(dims=5),
                   lambda d: d["layers"][1]["mixer"].update(decay=[0.5, 0.5]),           # 3 heads
                   lambda d: d["layers"][1]["mixer"].update(dim=1000),
                   lambda d: d["layers"][0]["mlp"]["router"].update(identity=2),         # 11 outputs in 4 groups
                   lambda d: d["layers"][0]["mlp"]["router"].update(top=7),              # 2 groups of 3 are kept
                   lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=5),
                   lambda d: d["layers"][1]["mlp"].update(kind="gated"),
                   lambda d: d.update(logit_softcap=-1.0)):
        d = json.loads(json.dumps(CONFIGS["odd"]))
        change(d)
        with pytest.raises(ValueError):
            NibelixConfig.from_dict(d)


def test_registry_names_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["ones"]))
    assert language_model_architecture(tmp_path) == "Nibelix" and LANGUAGE_MODELS["Nibelix"] is NibelixForCausalLM


def test_weights_are_checked_against_the_config():
    d = CONFIGS["odd"]
    w = random_weights(d)
    make = lambda: NibelixForCausalLM(NibelixConfig.from_dict(d), "cpu", torch.float32)
    model = make().load_weights(w)
    W = {k: v.double() for k, v in w.items()}
    lam, scale, eps = model.layers[0].diff
    assert lam == pytest.approx(float(O.diff_lambda(W, "l0.mix.", 0.7))) and scale == pytest.approx(0.3) and eps == 1e-5
    assert len(model.layers[0].norms) == 2 and len(model.layers[2].norms) == 1      # no feed-forward, no second norm
    assert model.layers[0].norms[1].alpha == float(w["l0.norm2.alpha"])
    assert model.layers[1].in_off["k"] == (24, 21) and model.layers[0].up.shape == (9, 20, 92)
    extra = dict(w, unused=torch.zeros(3))
    make().load_weights(extra)
    bad = dict(w)
    bad["l0.mlp.e3.down"] = bad["l0.mlp.e3.down"][:-1]
    with pytest.raises(ValueError):
        make().load_weights(bad)
    bad = dict(w)
    del bad["l4.mlp.shared.sg"]
    with pytest.raises(KeyError):
        make().load_weights(bad)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_oracle_is_causal(name):
    d = CONFIGS[name]
    w = random_weights(d, seed=1)
    toks = torch.randint(0, d["vocab"], (40,), generator=torch.Generator().manual_seed(2)).tolist()
    a = O.forward(d, w, toks)
    other = list(toks)
    other[25] = (other[25] + 1) % d["vocab"]
    b = O.forward(d, w, other)
    assert torch.allclose(a[:25], b[:25], rtol=0, atol=1e-12) and not torch.allclose(a[25:], b[25:])


def test_oracle_window_reaches_as_far_as_it_says():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(20, n, dtype=F64, generator=g) for n in (4, 4, 3))
    base = O.windowed_map(q, k, v, 0.5, 6)
    for j in range(20):
        v2 = v.clone()
        v2[j] += 1.0
        moved = (O.windowed_map(q, k, v2, 0.5, 6) != base).any(-1)
        assert moved.tolist() == [0 <= i - j < 6 for i in range(20)]
    assert torch.allclose(O.windowed_map(q, k, v, 0.5, 1), v)                      # a token that sees itself only
    assert torch.allclose(O.windowed_map(q, k, v, 0.5, 20), O.windowed_map(q, k, v, 0.5, 0))


def test_oracle_combination_of_maps():
    a = torch.tensor([[3.0, -4.0]], dtype=F64)
    r = O.combine_maps(a, torch.zeros(1, 2, dtype=F64), 5.0, 0.2, 0.0)
    assert torch.allclose(r, 0.8 * a / math.sqrt(12.5))
    assert torch.allclose(O.combine_maps(0 * a, a, 2.0, 0.2, 0.0), -r)               # the second map counts with minus its factor
    assert float(O.combine_maps(a, a, 1.0, 0.2, 1e-5).abs().max()) == 0.0
    z = torch.zeros(3, dtype=F64)
    W = {"lq1": z + 0.5, "lk1": z + 2.0, "lq2": z, "lk2": z}
    assert float(O.diff_lambda(W, "", 0.25)) == pytest.approx(math.exp(3.0) - 1.0 + 0.25)


def test_oracle_recurrence_against_closed_forms():
    k = torch.tensor([[1.0, 1.0]] + [[0.0, 0.0]] * 3, dtype=F64)
    o, S = O.lightning_rule(torch.ones(4, 2, dtype=F64), k, torch.ones(4, 1, dtype=F64), 0.5)
    assert torch.allclose(o[:, 0], torch.tensor([2.0, 1.0, 0.5, 0.25], dtype=F64)) and torch.allclose(S, torch.full((2, 1), 0.125, dtype=F64))
    v = torch.randn(5, 2, dtype=F64, generator=torch.Generator().manual_seed(1))
    o, _ = O.lightning_rule(torch.ones(5, 1, dtype=F64), torch.ones(5, 1, dtype=F64), v, 1.0)
    assert torch.allclose(o, v.cumsum(0))
    z = torch.linspace(-4, 4, 9, dtype=F64)
    assert torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert torch.allclose(O.gelu_erf(z), torch.nn.functional.gelu(z)) and torch.allclose(O.silu(z), torch.nn.functional.silu(z))


def test_oracle_router_rules():
    h, w = torch.ones(1, 1, dtype=F64), torch.log(torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=F64))
    zero = torch.zeros(4, dtype=F64)
    idx, wt = O.route(h, w, zero, {"top": 2, "scale": 2.0})
    assert idx[0].tolist() == [3, 2] and torch.allclose(wt[0], torch.tensor([0.8, 0.6], dtype=F64))   # not renormalised
    corr = torch.tensor([0.5, 0.0, 0.0, 0.0], dtype=F64) - 3.0
    r = {"top": 2, "scale": 1.0, "groups": {"count": 2, "keep": 1}}
    idx, wt = O.route(h, w, corr, r)                 # the corrected group wins; barred outputs do not win with zero
    assert idx[0].tolist() == [0, 1] and torch.allclose(wt[0], torch.tensor([0.1, 0.2], dtype=F64))


def test_oracle_identity_experts_and_the_shared_gate():
    d = {"kind": "moe", "expert": {"ff": 4}, "shared": {"ff": 3}, "router": {"experts": 2, "identity": 2, "top": 1, "scale": 3.0}}
    g = torch.Generator().manual_seed(1)
    W = {n: torch.randn(s, dtype=F64, generator=g) for n, s in (("e0.up", (4, 5)), ("e0.down", (5, 4)), ("e1.up", (4, 5)), ("e1.down", (5, 4)),
                                                               ("router", (4, 5)), ("shared.up", (3, 5)), ("shared.down", (5, 3)), ("shared.sg", (1, 5)))}
    W["correction"] = torch.tensor([0.0, 0.0, 5.0, 0.0], dtype=F64)      # always the first identity expert
    h = torch.randn(6, 5, dtype=F64, generator=g)
    s = torch.softmax(h @ W["router"].T, -1)[:, 2:3]
    want = 3.0 * s * h + torch.sigmoid(h @ W["shared.sg"].T) * O.expert_ff(h, W, "shared.")
    assert torch.allclose(O.moe_ff(h, W, "", d), want)
