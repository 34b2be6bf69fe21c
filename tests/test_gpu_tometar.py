"""Tometar models on a GPU against the plain float64 statement (tests/plain_tometar.py): every mechanism, prompts, portions,
decoding, reuse, window edges, generation. float32 models are held to float32 accuracy, bfloat16 models to what rounding
activations to bfloat16 costs."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nfai_b200 import ModelOptions, NfaiError, PlannedModel, _lib, trace, try_create

from . import plain_tometar as P
from . import tometar_util as U
from .gpu_util import call, dev, host, ptr

pytestmark = pytest.mark.gpu
torch = pytest.importorskip("torch")

TOL = {"f32": 2e-5, "bf16": 4e-2}
CTX = 320
_cache = {}


def plain(name, n=300, seed=0):
    """(config, weights, tokens, logits [n][V], layer outputs [n][L][H]) of a named configuration, computed once."""
    key = (name, n, seed)
    if key not in _cache:
        cfg = U.CONFIGS[name]
        W = U.weights(cfg, seed)
        toks = np.random.default_rng(seed + 100).integers(0, cfg["vocab"], n).tolist()
        taps = []
        logits = P.forward(cfg, {k: v.astype(np.float64) for k, v in W.items()}, toks, taps=taps)
        _cache[key] = (cfg, W, toks, logits, np.array(taps))
    return _cache[key]


def build(ctx, cfg, W, dtype, size=CTX):
    return PlannedModel.from_tensors(ctx, cfg, U.tensors(W), size, dtype)


@pytest.fixture(params=[(n, d) for n in U.CONFIGS for d in ("f32", "bf16")], ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, cuda_ctx):
    name, dtype = request.param
    m = build(cuda_ctx, U.CONFIGS[name], plain(name)[1], dtype)
    yield (m, dtype) + plain(name)
    m.Dispose()


def test_whole_prompt(case):
    m, dtype, cfg, W, toks, want, taps = case
    places = list(range(0, len(toks), 3)) + [len(toks) - 1]
    assert U.error(m.forward(toks, sorted(set(places))), want[sorted(set(places))]) < TOL[dtype]
    for l in range(m.L):
        assert U.error(m.read_hidden(l), taps[-1, l]) < TOL[dtype]
    assert m.position == len(toks)


def test_token_by_token(case):
    m, dtype, cfg, W, toks, want, taps = case
    n = 110
    got = [m.decode(t)[0] for t in toks[:n]]
    assert U.error(got, want[:n]) < TOL[dtype]
    for l in range(m.L):
        assert U.error(m.read_hidden(l), taps[n - 1, l]) < TOL[dtype]


def test_portions(case):
    """Cut anywhere: portions below the batched path's minimum, around the kernels' tiles, and single tokens in between."""
    m, dtype, cfg, W, toks, want, _ = case
    for sizes in ([2, 3, 1, 8, 9, 7, 16, 31, 1, 33, 2, 64, 15], [129, 2, 130, 1], [37, 37, 2, 5], [2]):
        m.reset()
        got, at, i = [], 0, 0
        end = 60 if sizes == [2] else len(toks)
        while at < end:
            n = min(sizes[i % len(sizes)], end - at)
            got += list(m.forward(toks[at:at + n], range(n)))
            at, i = at + n, i + 1
        assert U.error(got, want[:end]) < TOL[dtype], sizes


def test_prompt_then_decoding(case):
    m, dtype, cfg, W, toks, want, _ = case
    for cut in (1, 2, 33, 200):
        m.reset()
        logits, am = m.prefill(toks[:cut])
        assert U.error(logits, want[cut - 1]) < TOL[dtype] and am == int(np.argmax(logits))
        got = [m.decode(t)[0] for t in toks[cut:cut + 45]]
        assert U.error(got, want[cut:cut + 45]) < TOL[dtype]


def test_reuse_leaves_no_trace(case):
    """A sequence gives the same bits whatever ran before it, from a reset and from a snapshot."""
    m, dtype, cfg, W, toks, want, _ = case
    run = lambda: np.vstack([m.forward(toks[:50], range(0, 50, 7)), [m.decode(t)[0] for t in toks[50:60]]])  # noqa: E731
    first = run()
    other = [(t * 7 + 3) % cfg["vocab"] for t in toks]
    m.reset()
    m.forward(other[:170])
    m.reset()
    assert np.array_equal(run(), first)
    with_snap = m.snapshot()
    a = np.array([m.decode(t)[0] for t in toks[60:70]])
    m.reset()
    m.forward(other[:90])
    with_snap.restore()
    assert m.position == 60
    assert np.array_equal(np.array([m.decode(t)[0] for t in toks[60:70]]), a)
    with_snap.close()


def test_several_passes(cuda_ctx, monkeypatch):
    """A prompt longer than one pass of the batched path."""
    monkeypatch.setenv("NFAI_PREFILL_CHUNK", "48")
    for name in ("even", "odd"):
        cfg, W, toks, want, taps = plain(name)
        for dtype in ("f32", "bf16"):
            m = build(cuda_ctx, cfg, W, dtype)
            assert U.error(m.forward(toks, range(len(toks))), want) < TOL[dtype]
            assert U.error(m.read_hidden(m.L - 1), taps[-1, -1]) < TOL[dtype]
            m.Dispose()


def test_any_size_kernels_of_the_prompt_path(tmp_path):
    """The token-by-token scan and the any-size attention on bfloat16 models (switches are read once per process)."""
    cfg, W, toks, want, _ = plain("wide")
    U.write_folder(tmp_path / "m", cfg, W)
    code = ("import sys, numpy as np; sys.path.insert(0, sys.argv[1]); from nfai_b200 import *; "
            "m = try_create(CudaContext(0), ModelOptions(ModelPath=sys.argv[2], KVCacheSize=320)); "
            "np.save(sys.argv[3], m.forward(eval(sys.argv[4]), range(0, 300, 5)))")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = str(tmp_path / "o.npy")
    subprocess.run([sys.executable, "-c", code, root, str(tmp_path / "m"), out, str(toks)], check=True, timeout=120,
                   env=dict(os.environ, NFAI_SSM_CHUNK="0", NFAI_PREFILL_ATTN="0"))
    assert U.error(np.load(out), want[::5]) < TOL["bf16"]


# ---- mechanisms alone -----------------------------------------------------------------------------------------------------
def bf16(v):
    return U.bf16_round(np.asarray(v, np.float32)).astype(np.float64)


def alone(cuda_ctx, cfg, W, toks, dtype):
    """A prompt and token-by-token decoding. bfloat16 models are compared with the plain statement rounded where they round
    (prompts: operands and cache rows; decoding: cache rows only), so that the bounds stay close: what is left are
    values that fall on the other side of a rounding boundary."""
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    m = build(cuda_ctx, cfg, W, dtype, len(toks))
    ref = P.forward(cfg, W64, toks, **(dict(act=bf16, cache=bf16) if dtype == "bf16" else {}))
    assert U.error(m.forward(toks, range(len(toks))), ref) < {"f32": 3e-5, "bf16": 2e-2}[dtype]
    m.reset()
    ref = P.forward(cfg, W64, toks, **(dict(cache=bf16) if dtype == "bf16" else {}))
    assert U.error([m.decode(t)[0] for t in toks], ref) < {"f32": 3e-5, "bf16": 1e-3}[dtype]
    m.Dispose()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("mixer,ff", [
    (U.latent(5, 40, 24, 56, 88, 33), None), (U.latent(2, 128, 64, 128, 256, 64), None), (U.latent(9, 8, 4, 130, 20, 500), None),
    (U.ssm(3, 64, 128, 3, 4, 1), None), (U.ssm(8, 32, 16, 4, 3, 8), None), (U.ssm(2, 130, 24, 1, 6, 2), None), (U.ssm(2, 8, 300, 2, 2, 1), None),
], ids=str)
def test_one_mixer(cuda_ctx, mixer, ff, dtype):
    cfg = U.config([U.layer(mixer, ff)], 64, 96, 2)
    toks = np.random.default_rng(5).integers(0, 96, 150).tolist()
    alone(cuda_ctx, cfg, U.weights(cfg, 11), toks, dtype)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_feed_forward_alone(cuda_ctx, dtype):
    """The mixer's output matrix is zero: what is left is the biased relu-gated feed-forward and the streams."""
    cfg = U.config([U.layer(U.latent(1, 4, 2, 8, 8, 4), 200), U.layer(U.ssm(1, 8, 4, 1, 2, 1), 24)], 72, 50, 4)
    W = U.weights(cfg, 2)
    for i in (0, 1):
        W[f"l{i}.mix.o"][:] = 0
        W[f"l{i}.mlp.gate.b"] = U.bf16_round(W[f"l{i}.mlp.gate.b"] * 4)
    alone(cuda_ctx, cfg, W, list(range(50)), dtype)


@pytest.mark.parametrize("streams", [1, 2, 5, 8, 9, 16])
def test_stream_counts(cuda_ctx, streams):
    cfg = U.config([U.layer(U.latent(2, 16, 8, 16, 24, 9), 40), U.layer(U.ssm(2, 16, 8, 1, 3, 2))], 48, 40, streams)
    W = U.weights(cfg, streams)
    for k in W:
        if k.endswith(".mix") and ".hc" in k:  # far from symmetric: from and to must not be mixed up
            W[k] = U.bf16_round(W[k] + np.triu(np.ones_like(W[k]), 1) * 0.3 / streams)
    alone(cuda_ctx, cfg, W, [int(t) for t in np.random.default_rng(0).integers(0, 40, 40)], "f32")


def test_the_state_carries_far(cuda_ctx):
    """Decays near one: a token hundreds of positions back still shows, in prompts, across portions and in decoding."""
    cfg = U.config([U.layer(U.ssm(4, 16, 24, 2, 3, 2))], 48, 60, 2)
    W = U.weights(cfg, 4)
    W["l0.mix.A_log"][:] = U.bf16_round(np.full(4, -7.0, np.float32))
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    base = np.random.default_rng(1).integers(0, 60, 400).tolist()
    changed = [(base[0] + 1) % 60] + base[1:]
    a, b = P.forward(cfg, W64, base), P.forward(cfg, W64, changed)
    effect = U.error(a[-1], b[-1])
    assert effect > 1e-3  # well above what float32 loses: a lost or stale state would show
    m = build(cuda_ctx, cfg, W, "f32", 400)
    for toks, ref in ((base, a), (changed, b)):
        for sizes in ([400], [130, 100, 2, 168], [260] + [1] * 140):
            m.reset()
            at = 0
            for n in sizes:
                got = m.forward(toks[at:at + n], [n - 1])
                at += n
            assert U.error(got, ref[-1]) < effect / 20
    m.Dispose()
    for dtype in ("f32", "bf16"):
        alone(cuda_ctx, cfg, W, base, dtype)


# ---- window edges -----------------------------------------------------------------------------------------------------------
def needle_model(window, seed=0):
    """One latent layer whose scores are sharp, and tokens (query, needle, fillers): a query that sees the needle puts nearly
    all its weight on it, wherever it lies; fillers score low."""
    cfg = U.config([U.layer(U.latent(2, 32, 8, 24, 48, window, scale=1.0, base=1e6))], 56, 128, 2)
    W = U.weights(cfg, seed)
    for part in ("q", "dkv"):  # position matters little: the needle's score must survive any distance
        a = W[f"l0.mix.{part}"]
        rows = np.r_[32:40, 72:80] if part == "q" else np.r_[48:56]
        a[rows] = U.bf16_round(a[rows] * 0.05)
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    E = W64["embed"]
    h = np.array([P.rms_norm(e * W64["l0.hc1.in"].sum(), W64["l0.norm1"], 1e-5) for e in E])
    q = (h @ W64["l0.mix.q"].T).reshape(128, 2, 40)[:, :, :32]
    c = np.array([P.rms_norm(v, W64["l0.mix.dkv.norm"], 1e-5) for v in h @ W64["l0.mix.dkv"][:48].T])
    k = (c @ W64["l0.mix.uk"].T).reshape(128, 2, 32)
    s = np.einsum("qhd,khd->qkh", q, k).min(axis=2)  # both heads must agree
    query, needle = np.unravel_index(np.argmax(s - np.diag(s)[:, None]), s.shape)
    both = np.einsum("hd,khd->kh", q[query], k).max(axis=1)
    fillers = [int(t) for t in np.argsort(both) if t not in (query, needle)][:30]
    return cfg, W, W64, int(query), int(needle), fillers


@pytest.mark.parametrize("window", [3, 17, 64, 65, 150])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_window_edges(cuda_ctx, window, dtype):
    cfg, W, W64, query, needle, fillers = needle_model(window)
    m = build(cuda_ctx, cfg, W, dtype, 512)
    rng = np.random.default_rng(window)
    for pos in (window, window + 1, window + 40, 2 * window + 63):
        toks = [fillers[i] for i in rng.integers(0, len(fillers), pos + 1)]
        toks[pos] = query
        ref_none = P.forward(cfg, W64, toks)[-1]
        for back in (1, window - 1, window):
            t = list(toks)
            t[pos - back] = needle
            ref = P.forward(cfg, W64, t)[-1]
            seen = U.error(ref, ref_none)
            assert seen > 0.3 if back < window else seen < 1e-12  # the test sees what it is about
            m.reset()
            assert U.error(m.forward(t, [pos]), ref) < TOL[dtype], (pos, back, "prompt")
            for cut in (pos, max(1, pos - 1), max(1, pos - back), max(1, pos - back + 1), max(1, pos - 9)):
                m.reset()
                m.forward(t[:cut])
                assert U.error(m.forward(t[cut:], [pos - cut]), ref) < TOL[dtype], (pos, back, cut)
            m.reset()
            m.forward(t[:max(1, pos - 20)])
            for x in t[max(1, pos - 20):]:
                got, _ = m.decode(x)
            assert U.error(got, ref) < TOL[dtype], (pos, back, "decoded")
    m.Dispose()


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [(20, 16, 16, 24, 64, 50), (17, 8, 32, 8, 48, 300), (33, 8, 16, 16, 32, 7)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_many_heads(cuda_ctx, heads, dim, rot, vdim, rank, window, dtype):
    """More heads than one operand tile of the decode kernels holds."""
    cfg = U.config([U.layer(U.latent(heads, dim, rot, vdim, rank, window))], 40, 64, 2)
    alone(cuda_ctx, cfg, U.weights(cfg, heads), np.random.default_rng(1).integers(0, 64, 110).tolist(), dtype)


def test_runs_of_several_stages(cuda_ctx):
    """A window so long, for so many heads, that a CTA of the decode kernel walks its share of the cache in several stages."""
    cfg = U.config([U.layer(U.latent(100, 4, 16, 4, 272, 760))], 40, 64, 2)
    W = U.weights(cfg, 9)
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    toks = np.random.default_rng(2).integers(0, 64, 790).tolist()
    narrow = json.loads(json.dumps(cfg))
    narrow["layers"][0]["mixer"]["mask"]["size"] = 1  # what one layer leaves in the cache does not depend on its window
    st = P.State(narrow)
    P.forward(narrow, W64, toks[:740], st, cache=bf16)
    ref = P.forward(cfg, W64, toks[740:], st, cache=bf16)
    m = build(cuda_ctx, cfg, W, "bf16", 800)
    m.forward(toks[:740])
    assert U.error([m.decode(t)[0] for t in toks[740:]], ref) < 1e-3
    m.Dispose()


def test_cached_rows(cuda_ctx):
    """The cache holds the normed latent and the rotated key part, whichever path wrote it."""
    cfg, W, toks, _, _ = plain("even")
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    st = P.State(cfg)
    P.forward(cfg, W64, toks[:40], st)
    m = build(cuda_ctx, cfg, W, "f32")
    m.forward(toks[:30])
    for t in toks[30:40]:
        m.decode(t)
    for i in (0, 3):
        for pos in (0, 1, 29, 30, 39):
            c, kr = m.read_latent(i, pos)
            assert np.abs(c - st.layers[i][pos][0]).max() < 1e-4 and np.abs(kr - st.layers[i][pos][1]).max() < 1e-4
    m.Dispose()


# ---- generation ----------------------------------------------------------------------------------------------------------------
def test_greedy_generation(cuda_ctx):
    cfg, W, toks, _, _ = plain("even")
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    m = build(cuda_ctx, cfg, W, "f32", 300)
    st = P.State(cfg)
    lg = P.forward(cfg, W64, toks[:20], st)[-1]
    want = [int(np.argmax(lg))]
    while len(want) < 200:
        want.append(int(np.argmax(P.step(cfg, W64, st, want[-1]))))
    assert m.run_tokens(toks[:20], 60) == want[:60]
    m.reset()
    _, tk = m.prefill(toks[:20])
    got, ms = m.decode_greedy(tk, 199)  # long decoding, fed back on the device
    assert [tk] + got.tolist() == want and ms > 0
    m.Dispose()


def test_sampled_generation(cuda_ctx):
    cfg, W, toks, _, _ = plain("even")
    m = build(cuda_ctx, cfg, W, "bf16", 300)
    us = np.random.default_rng(3).random(12, dtype=np.float32)
    _, tk = m.prefill(toks[:20])
    got, _ = m.decode_sampled(tk, us, temperature=1.3)
    m.reset()
    m.prefill(toks[:20])
    x, stepped = tk, []
    for u in us:
        m.decode(x)
        x = m.sample_top_p(temperature=1.3, u=float(u))
        stepped.append(x)
    assert got.tolist() == stepped and len(set(stepped)) > 1
    m.Dispose()


# ---- files, replay, errors -------------------------------------------------------------------------------------------------------
def test_folder_and_replay(cuda_ctx, tmp_path):
    """A model folder through the registry, and two interleaved sequences replayed against each alone."""
    cfg, W, toks, want, _ = plain("odd")
    path = U.write_folder(tmp_path / "model", cfg, W)
    m = try_create(cuda_ctx, ModelOptions(ModelPath=path, KVCacheSize=CTX, WeightDType="f32"))
    other = [(t + 5) % cfg["vocab"] for t in toks[:70]]
    ref_other = P.forward(cfg, {k: v.astype(np.float64) for k, v in W.items()}, other)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": other[:9], "want": [8]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[33:35], "want": [0, 1]}, {"id": "y", "tokens": other[9:70], "want": [60]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": toks[35:200], "want": [164]}], "end": ["x"]}]
    trace.replay(m, [json.dumps(s) for s in steps], str(tmp_path), lambda s: None)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])  # noqa: E731
    assert U.error(read(0), want[[0, 32]]) < TOL["f32"] and U.error(read(1), ref_other[8]) < TOL["f32"]
    assert U.error(read(2), np.vstack([want[[33, 34]], ref_other[[69]]])) < TOL["f32"]
    assert U.error(read(3), want[199]) < TOL["f32"]
    m.Dispose()


def test_trace_program(tmp_path):
    cfg, W, toks, want, _ = plain("ones")
    U.write_folder(tmp_path / "model", cfg, W)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [39]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[40:41], "want": [0]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "41"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert r.stdout.splitlines()[-2:] == ["done 0", "done 1"]
    got = np.vstack([np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(1, -1) for n in (0, 1)])
    assert U.error(got, want[39:41]) < TOL["f32"]


def test_misuse_is_an_error(cuda_ctx, tmp_path):
    cfg, W, toks, _, _ = plain("ones")
    t = U.tensors(W)
    with pytest.raises(NfaiError) as e:
        PlannedModel.from_tensors(cuda_ctx, cfg, t[:-1], 32, "bf16")
    assert e.value.code == _lib.ERR_STATE and t[-1][0] in str(e.value)
    with pytest.raises(NfaiError) as e:
        PlannedModel.from_tensors(cuda_ctx, cfg, [(t[0][0], t[0][1].T, t[0][2])], 32, "bf16")
    assert e.value.code == _lib.ERR_ARG
    with pytest.raises(NfaiError) as e:
        PlannedModel.from_tensors(cuda_ctx, cfg, [("l9.mix.q", t[0][1], t[0][2])], 32, "bf16")
    assert e.value.code == _lib.ERR_ARG
    m = build(cuda_ctx, cfg, W, "bf16", 32)
    m.forward(toks[:20])
    with pytest.raises(NfaiError) as e:
        m.set_position(10)
    assert e.value.code == _lib.ERR_STATE and "snapshot" in str(e.value)
    for n in (13, 5):
        with pytest.raises(NfaiError) as e:
            m.forward(toks[:13], [0, 12])
        assert e.value.code == _lib.ERR_CONTEXT_FULL or e.value.code == _lib.ERR_ARG
    with pytest.raises(NfaiError):
        m.forward([cfg["vocab"]] * 9, [0])
    for bad in ([1, 0], [0, 0], [5]):
        with pytest.raises(NfaiError) as e:
            m.forward(toks[:5], bad)
        assert e.value.code == _lib.ERR_ARG
    m.Dispose()
    # damaged weight files
    path = U.write_folder(tmp_path / "m", cfg, W)
    raw = open(os.path.join(path, "model.safetensors"), "rb").read()
    for damaged in (b"", raw[:5], raw[:200], raw[:-2], b"\xff" * 8 + raw[8:], raw.replace(b'"BF16"', b'"I128"', 1),
                    raw.replace(b'"data_offsets": [0', b'"data_offsets": [1', 1)):
        with open(os.path.join(path, "model.safetensors"), "wb") as f:
            f.write(damaged)
        with pytest.raises(NfaiError) as e:
            try_create(cuda_ctx, ModelOptions(ModelPath=path, KVCacheSize=32))
        assert e.value.code == _lib.ERR_ARG


# ---- the shared products in bfloat16 and float32 ------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 40, 24), (130, 300, 136), (300, 512, 1024), (77, 35, 51), (2048, 3072, 256)])
@pytest.mark.parametrize("dtype", [_lib.F32, _lib.BF16])
def test_gemm(cuda_ctx, M, N, K, dtype):
    g = torch.Generator().manual_seed(M + N + K)
    td = torch.float32 if dtype == _lib.F32 else torch.bfloat16
    A, W = torch.randn(M, K, generator=g).to(td), torch.randn(N, K, generator=g).to(td)
    C = torch.full((M, N), float("nan"), device="cuda")
    dA, dW = A.cuda(), W.cuda()
    call(cuda_ctx, "nfai_op_gemm", ptr(dA), ptr(dW), dtype, M, N, K, ptr(C))
    ref = A.double() @ W.double().T
    assert (C.cpu().double() - ref).abs().max() < 1e-5 * K ** 0.5 * 4


@pytest.mark.parametrize("N,K", [(7, 8), (513, 1000), (64, 51), (2048, 2048)])
def test_bfloat16_gemv(cuda_ctx, N, K):
    rng = np.random.default_rng(N)
    W = U.bf16_round(rng.standard_normal((N, K)).astype(np.float32))
    x, gain, res = (rng.standard_normal(n).astype(np.float32) for n in (K, K, N))
    y = torch.full((N,), float("nan"), device="cuda")
    dW = torch.from_numpy(U.bf16_bits(W).view(np.int16)).cuda()
    dx, dg, dr = dev(x), dev(gain), dev(res)
    call(cuda_ctx, "nfai_op_gemv", ptr(dW), _lib.BF16, N, K, ptr(dx), ptr(dg), 1e-5, ptr(dr), ptr(y))
    x64 = x.astype(np.float64)
    ref = W.astype(np.float64) @ (x64 / np.sqrt((x64 * x64).mean() + 1e-5) * gain) + res
    assert np.abs(host(y) - ref).max() < 2e-4
