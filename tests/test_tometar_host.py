"""Tometar models without a GPU: the configuration reader, the tensor list, the plain statement of the mathematics against
closed forms, and the trace replay's handling of several sequences."""
import copy
import json

import numpy as np
import pytest

import nfai_b200
from nfai_b200 import NfaiError, registry, trace

from . import plain_tometar as P
from . import tometar_util as U


def test_tensor_list_follows_the_configuration():
    cfg = U.CONFIGS["even"]
    t = nfai_b200.config_tensors(cfg)
    assert t["embed"] == t["head"] == (200, 112) and t["final.norm"] == (112,)
    assert t["l0.mix.q"] == (4 * 48, 112) and t["l0.mix.dkv"] == (64 + 16, 112) and t["l0.mix.uk"] == (128, 64)
    assert t["l0.mix.uv"] == (192, 64) and t["l0.mix.g"] == (192, 112) and t["l0.mix.o"] == (112, 192)
    assert t["l1.mix.in"] == (2 * 96 + 2 * 2 * 32 + 6, 112) and t["l1.mix.conv"] == (96 + 128, 4) and t["l1.mix.norm"] == (96,)
    assert "l1.norm2" not in t and "l1.hc2.in" not in t and "l1.mlp.gate" not in t
    assert t["l2.mlp.gate.b"] == (96,) and t["l2.mlp.down"] == (112, 96) and t["l2.hc2.mix"] == (3, 3)


@pytest.mark.parametrize("change", [
    lambda c: c.pop("architecture"),
    lambda c: c.update(architecture="Nameless"),
    lambda c: c.pop("streams"),
    lambda c: c.update(streams=0),
    lambda c: c.update(width=12.5),
    lambda c: c.update(width=-4),
    lambda c: c.update(width=1e30),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="convolution"),
    lambda c: c["layers"][0].pop("mixer"),
    lambda c: c["layers"][0]["mixer"].pop("kv_rank"),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"),
    lambda c: c["layers"][1]["mixer"].update(groups=4),
    lambda c: c["layers"][1]["mixer"].update(norm_groups=5),
    lambda c: c["layers"][1]["mixer"].update(heads=16000000),
])
def test_bad_configurations_are_refused(change):
    cfg = copy.deepcopy(U.CONFIGS["even"])
    change(cfg)
    with pytest.raises(NfaiError) as e:
        nfai_b200.config_tensors(cfg)
    assert e.value.code == nfai_b200._lib.ERR_ARG


@pytest.mark.parametrize("text", [b"", b"{", b'{"a": 1,}', b'{"a": tru}', b"[1, 2", b'"\\u12"', b'{"architecture": "Tometar"} x', b"1e999",
                                  b"[" * 10000])
def test_malformed_json_is_an_error(text):
    lib = nfai_b200._lib.load()
    assert lib.nfai_config_probe(text, len(text), None, None, 0, None, None, 0) == nfai_b200._lib.ERR_ARG


def test_json_strings_and_nesting():
    cfg = dict(U.CONFIGS["ones"], note="é\U0001f600\\\"/\n", extra=[[], {}, [1, -2.5e-3, None, True, False]])
    assert nfai_b200.config_tensors(cfg) == nfai_b200.config_tensors(U.CONFIGS["ones"])


def test_registry_names_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(U.CONFIGS["ones"]))
    assert registry.architecture_of(str(tmp_path)) in registry.CONFIG_ARCHITECTURES
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Other"}))
    assert registry.try_create(None, nfai_b200.ModelOptions(ModelPath=str(tmp_path))) is None


# ---- the plain statement against closed forms ------------------------------------------------------------------------
def test_plain_rotation_is_relative():
    rng = np.random.default_rng(0)
    a, b = rng.standard_normal(10), rng.standard_normal(10)
    f = lambda v, p: P.rotate_half(v, p, 100.0, 8)  # noqa: E731
    assert np.allclose(f(a, 7) @ f(b, 3), f(a, 14) @ f(b, 10))
    assert np.allclose(f(a, 0), a) and np.allclose(f(a, 5)[8:], a[8:])
    one = f(np.eye(10)[1], 2)  # entry 1 turns into entries 1 and 5 by 2 * 100^(-2/8)
    ang = 2 * 100.0 ** -0.25
    assert np.allclose([one[1], one[5]], [np.cos(ang), np.sin(ang)]) and np.isclose(np.linalg.norm(one), 1)


def test_plain_recurrence_equals_its_sum():
    rng = np.random.default_rng(1)
    T, H, N, V, G = 9, 4, 3, 5, 2
    x, B, C = rng.standard_normal((T, H, V)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A_log, D = rng.uniform(0.1, 1, (T, H)), rng.standard_normal(H), rng.standard_normal(H)
    S = np.zeros((H, N, V))
    for t in range(T):
        S, y = P.ssm_step(S, x[t], B[t], C[t], dt[t], A_log, D, G)
        for h in range(H):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                want = want + (C[t, h // 2] @ B[j, h // 2]) * np.exp(-np.exp(A_log[h]) * dt[j + 1:t + 1, h].sum()) * dt[j, h] * x[j, h]
            assert np.allclose(y[h], want)


def test_plain_window_and_streams():
    cfg = U.config([U.layer(U.latent(2, 6, 4, 5, 7, 3))], 8, 20, 2)
    W = {n: a.astype(np.float64) for n, a in U.weights(cfg, 3).items()}
    a, b = [1, 2, 3, 4, 5], [9, 8, 3, 4, 5]
    assert np.allclose(P.forward(cfg, W, a)[-1], P.forward(cfg, W, b)[-1])      # tokens behind the window do not matter
    assert not np.allclose(P.forward(cfg, W, a)[-2], P.forward(cfg, W, b)[-2])  # the one just inside does
    X = np.array([[1.0, 2.0], [3.0, 5.0]])
    assert np.allclose(P.hyper_write(X, np.array([1.0, 1.0]), np.array([[0.0, 1.0], [0.0, 0.0]]), np.array([0.0, 2.0])),
                       [[0, 0], [3, 4]])  # stream 0 goes to stream 1
    assert np.allclose(P.hyper_read(X, np.array([2.0, -1.0])), [-1, -1])


# ---- several sequences on one model ------------------------------------------------------------------------------------
class FakeModel:
    """Logits say what was fed since the last reset."""

    def __init__(self):
        self.fed, self.snaps = [], 0

    def reset(self):
        self.fed = []

    def snapshot(self):
        kept, me = list(self.fed), self
        me.snaps += 1

        class Snap:
            def restore(self):
                me.fed = list(kept)

            def close(self):
                me.snaps -= 1
        return Snap()

    def forward(self, tokens, want):
        out = []
        for i, t in enumerate(tokens):
            self.fed.append(t)
            if i in want:
                out.append([sum(self.fed), len(self.fed)])
        return np.array(out, np.float32).reshape(len(out), 2)


def test_replay_interleaves_sequences(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [3], "want": [0]}, {"id": "b", "tokens": [20, 30], "want": [1, 0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [7], "want": [0]}], "end": ["a", "b"]}]
    m, said = FakeModel(), []
    trace.replay(m, [json.dumps(s) + "\n" for s in steps], str(tmp_path), said.append)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 2).tolist()  # noqa: E731
    assert said == ["done 0", "done 1", "done 2", "done 3"]
    assert read(0) == [[3, 2]] and not (tmp_path / "1.f32").exists()
    assert read(2) == [[6, 3], [60, 3], [30, 2]]
    assert read(3) == [[7, 1]]  # "a" ended and starts anew
    assert m.snaps == 0
