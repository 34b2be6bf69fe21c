"""Tutizen models without a GPU: the configuration reader, the tensor list, the plain statement of the mathematics against
closed forms."""
import copy

import numpy as np
import pytest

import nfai_b200
from nfai_b200 import NfaiError, registry

from . import plain_tutizen as P
from . import tutizen_util as U


def test_tensor_list_follows_the_configuration():
    t = nfai_b200.config_tensors(U.CONFIGS["even"])
    assert t["embed"] == t["head"] == (200, 112) and t["final.norm"] == () and t["l0.norm1"] == t["l0.norm2"] == ()
    assert t["l0.mix.q"] == (192, 112) and t["l0.mix.q.b"] == (192,) and t["l0.mix.k"] == (64, 112) and t["l0.mix.v.b"] == (96,)
    assert t["l0.mix.g"] == (6, 112) and "l0.mix.g.b" not in t and t["l0.mix.o"] == (112, 288) and t["l0.mix.o.b"] == (112,)
    assert "l1.mix.k" not in t and "l1.mix.v" not in t and "l1.mix.k.b" not in t and t["l1.mix.q"] == (192, 112)
    assert t["l0.mlp.gate"] == (136, 112) and "l0.mlp.gate.b" not in t and t["l0.mlp.down"] == (112, 136)
    assert t["l1.mlp.e11.up"] == (40, 112) and "l1.mlp.e12.up" not in t and t["l1.mlp.router"] == (12, 112)
    assert t["l1.mlp.correction"] == (12,) and t["l1.mlp.shared.down"] == (112, 56) and t["l1.mlp.shared.sg"] == (1, 112)
    assert "l2.norm2" not in t and "l2.mlp.gate" not in t


@pytest.mark.parametrize("change", [
    lambda c: c.pop("residual_mult"),
    lambda c: c.update(norm={}),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="mamba2"),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"].update(kv_from=0),
    lambda c: c["layers"][1]["mixer"].update(kv_from=1),
    lambda c: c["layers"][1]["mixer"].update(kv_from=3),
    lambda c: c["layers"][1]["mixer"].update(kv_from=-1),
    lambda c: c["layers"][1]["mixer"].update(kv_from=0.5),
    lambda c: c["layers"][3]["mixer"].update(kv_from=1),  # borrows itself
    lambda c: c["layers"][3]["mixer"].update(kv_from=2),  # other head sizes
    lambda c: c["layers"][1]["mixer"].update(dim=40),
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mlp"].pop("limit"),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=9),  # the kept groups hold eight
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4),
    lambda c: c["layers"][1]["mlp"]["router"].update(experts=100000),
    lambda c: c["layers"][1]["mlp"]["router"].pop("scale"),
    lambda c: c["layers"][1]["mlp"].pop("expert"),
    lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"),
    lambda c: c["layers"][1]["mlp"]["expert"].update(ff=0),
])
def test_bad_configurations_are_refused(change):
    cfg = copy.deepcopy(U.CONFIGS["even"])
    change(cfg)
    with pytest.raises(NfaiError) as e:
        nfai_b200.config_tensors(cfg)
    assert e.value.code == nfai_b200._lib.ERR_ARG


def test_registry_names_the_architecture():
    assert "Tutizen" in registry.CONFIG_ARCHITECTURES


# ---- the plain statement against closed forms ------------------------------------------------------------------------
def test_plain_positions():
    v = P.position_vector(3, 6)
    assert np.allclose(v, [np.sin(3), np.cos(3), np.sin(3 / 10000 ** (1 / 3)), np.cos(3 / 10000 ** (1 / 3)),
                           np.sin(3 / 10000 ** (2 / 3)), np.cos(3 / 10000 ** (2 / 3))])
    assert np.allclose(P.position_vector(0, 5), [0, 1, 0, 1, 0]) and len(P.position_vector(9, 5)) == 5


def test_plain_bias_and_softmax():
    assert np.allclose(P.slopes(8), [0.5 ** (h + 1) for h in range(8)]) and np.allclose(P.slopes(3)[2], 2.0 ** -8)
    K, V = np.zeros((4, 2)), np.eye(4)
    w = P.attend(np.ones(2), K, V, 1.0, np.log(2.0), 3)  # equal scores: every step back halves the weight
    assert np.allclose(w, np.array([1, 2, 4, 8]) / 15)
    assert np.allclose(P.unit_rms(np.array([3.0, 4.0]), 0.0), np.array([3.0, 4.0]) / np.sqrt(12.5))


def test_plain_clamp():
    f = P.clamped_glu
    assert np.isclose(f(9.0, 0.3, 2.0), 2.0 / (1 + np.exp(-3.404)) * 1.3)   # the gate is held from above ...
    assert np.isclose(f(-9.0, 0.3, 2.0), -9.0 / (1 + np.exp(15.318)) * 1.3)  # ... only
    assert np.isclose(f(1.0, 5.0, 2.0), 3.0 * P.sigmoid(1.702)) and np.isclose(f(1.0, -5.0, 2.0), -P.sigmoid(1.702))


def test_plain_routing():
    r = {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 2}}
    logit = lambda s: np.log(np.array(s) / (1 - np.array(s)))  # noqa: E731
    s = [0.9, 0.1, 0.6, 0.5, 0.55, 0.5]
    chosen, w = P.route(logit(s), np.zeros(6), r)  # groups score 1.0, 1.1, 1.05: the first, with the best expert, is out
    assert chosen == [2, 4] and np.allclose(w, np.array([0.6, 0.55]) / 1.15 * 3)
    chosen, w = P.route(logit(s), np.array([0, 0, 0, 0, 0, 0.2]), r)  # a correction moves the choice, not the weight
    assert chosen == [5, 2] and np.allclose(w, np.array([0.5, 0.6]) / 1.1 * 3)
    one = dict(r, groups={"count": 3, "keep": 1}, top=2)
    chosen, _ = P.route(logit(s), np.array([-3.0, -3, -2, -2.5, -3, -3]), one)  # negative scores still beat what is left out
    assert chosen == [2, 3]


def test_clear_choices_survive_rounding():
    for name in ("even", "odd", "wide"):
        cfg = U.CONFIGS[name]
        W = U.weights(cfg)
        toks = U.tokens(cfg, W, 12)
        W64 = {k: v.astype(np.float64) for k, v in W.items()}
        r = lambda v: U.bf16_round(np.asarray(v, np.float32)).astype(np.float64)  # noqa: E731
        a, b = P.forward(cfg, W64, toks), P.forward(cfg, W64, toks, act=r, cache=r)
        assert U.error(b, a) < 3e-2
