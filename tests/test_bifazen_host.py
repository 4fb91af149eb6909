"""Bifazen without a GPU: the float64 restatement's own pieces against closed forms, the model-folder checks of the loader."""
import math
import subprocess

import numpy as np
import pytest

import bifazen_oracle as bo


@pytest.fixture(scope="module")
def tools():
    from kuiperllama_b200 import build
    return build.build_seq_tools()


def small():
    cfg = bo.make_config(layers=[(bo.latent_mixer(), 20), (bo.plain_mixer(), None), (bo.plain_mixer(), 12)])
    return cfg, bo.make_weights(cfg)


def trace_cmd(tools, d, out):
    return [str(tools / "kuiper_trace"), "--model", str(d), "--out", str(out), "--dtype", "float32"]


def test_missing_tensors_and_unknown_kinds_are_reported(tools, tmp_path):
    cfg, w = small()
    for missing in ("l0.mix.dkv.norm", "l0.mix.uk", "l0.hc1.mix", "l0.hc2.out", "l0.norm2", "l0.mlp.gate", "l1.mix.q.b",
                    "l1.mix.k.norm", "l1.mix.o.b", "l1.hc1.in", "l2.mix.vmix", "l2.mix.g", "final.norm", "embed"):
        d = bo.write_model(tmp_path / missing, cfg, {k: v for k, v in w.items() if k != missing})
        r = subprocess.run(trace_cmd(tools, d, tmp_path), capture_output=True, text=True)
        assert r.returncode == 2 and missing in r.stderr, (missing, r.stderr)
    bad = dict(cfg, layers=[dict(cfg["layers"][0], type="convolution")])
    r = subprocess.run(trace_cmd(tools, bo.write_model(tmp_path / "bad", bad, w), tmp_path), capture_output=True, text=True)
    assert r.returncode == 2 and "convolution" in r.stderr
    bad = dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "routed", "ff": 20})])
    r = subprocess.run(trace_cmd(tools, bo.write_model(tmp_path / "bad2", bad, w), tmp_path), capture_output=True, text=True)
    assert r.returncode == 2 and "routed" in r.stderr


def test_rotation_pairs_neighbours():
    v = (np.arange(6, dtype=np.float64) + 1).reshape(1, 1, 6).repeat(4, axis=0)
    r = bo.rotate_pairs(v, 4, 100.0)[3, 0]
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(r[:4], [1 * math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + 1 * math.sin(a0),
                               3 * math.cos(a1) - 4 * math.sin(a1), 4 * math.cos(a1) + 3 * math.sin(a1)])
    assert np.allclose(r[4:], [5.0, 6.0])
    assert np.allclose(bo.rotate_pairs(v, 4, 100.0)[0], v[0]) and np.allclose(bo.rotate_pairs(v, 0, 9.0), v)


def test_window():
    want = np.array([[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]], dtype=bool)
    assert (bo.window_mask(4, 2) == want).all()
    assert (bo.window_mask(4, 1) == np.eye(4, dtype=bool)).all()
    assert (bo.window_mask(4, 0) == np.tril(np.ones((4, 4), dtype=bool))).all()


def test_gelu_and_norms():
    assert bo.gelu_tanh(np.array(0.0)) == 0.0
    assert math.isclose(bo.gelu_tanh(np.array(1.0)), 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715)))
    assert np.allclose(bo.gelu_tanh(np.array([9.0, -9.0])), [9.0, 0.0])
    x = np.array([[3.0, 4.0]])
    assert np.allclose(bo.centred_norm(x, np.zeros(2), 0.0), x / math.sqrt(12.5))
    assert np.allclose(bo.centred_norm(x, np.array([1.0, -1.0]), 3.5), [[3.0 / 4.0 * 2.0, 0.0]])  # eps inside the root


def test_streams():
    x = np.array([[[1.0, 2.0]], [[10.0, 20.0]]])   # two streams, one token
    y = np.array([[100.0, 200.0]])
    w = {"p.in": np.array([2.0, 0.5]), "p.out": np.array([1.0, 3.0]), "p.mix": np.array([[0.0, 1.0], [0.5, 0.0]])}
    assert np.allclose(bo.read_streams(x, w, "p."), [[7.0, 14.0]])
    # stream 0 is made of half of stream 1, stream 1 of stream 0 as it was
    assert np.allclose(bo.write_streams(x, y, w, "p."), [[[105.0, 210.0]], [[301.0, 602.0]]])


def test_values_are_blended_with_the_first_blending_layer():
    """The second blending layer with lambda 1 and uniform attention returns the running mean of the FIRST layer's values."""
    m = bo.plain_mixer(heads=1, kv_heads=1, dim=4, vdim=3, window=0)
    cfg = bo.make_config(width=6, layers=[(m, None)])
    w = bo.make_weights(cfg, seed=4)
    p = "l0.mix."
    w[p + "q"][:], w[p + "q.b"][:] = 0.0, 0.0
    w[p + "g"][:] = 0.0                      # gate 1/2
    w[p + "o"], w[p + "o.b"] = np.eye(6)[:, :3], np.zeros(6)
    w[p + "vmix"] = np.float64(1.0)
    h = np.random.default_rng(0).standard_normal((5, 6))
    out, raw = bo.plain_attention(h, w, p, m, 1e-6, None)
    own = h @ w[p + "v"].T + w[p + "v.b"]
    assert np.allclose(raw, own)
    means = np.cumsum(own, axis=0) / np.arange(1, 6)[:, None]
    assert np.allclose(out[:, :3], 0.5 * means)
    first = np.random.default_rng(1).standard_normal((5, 3))
    out, raw = bo.plain_attention(h, w, p, m, 1e-6, first)
    assert raw is None and np.allclose(out[:, :3], 0.5 * np.cumsum(first, axis=0) / np.arange(1, 6)[:, None])
