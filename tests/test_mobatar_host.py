"""Mobatar without a GPU: the float64 restatement's own pieces against closed forms, the model-folder checks of the loader."""
import math
import subprocess

import numpy as np
import pytest

import mobatar_oracle as mo
from seq_util import write_model


@pytest.fixture(scope="module")
def tools():
    from kuiperllama_b200 import build
    return build.build_seq_tools()


def small():
    cfg = mo.make_config(layers=[(mo.sink_mixer(), (20, 2.0)), (mo.parallel_mixer(), None), (mo.latent_mixer(), (12, 1.0)), 0, 1])
    return cfg, mo.make_weights(cfg)


def trace_cmd(tools, d, out):
    return [str(tools / "kuiper_trace"), "--model", str(d), "--out", str(out), "--dtype", "float32"]


def test_missing_tensors_and_unknown_kinds_are_reported(tools, tmp_path):
    cfg, w = small()
    for missing in ("embed", "bigram", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mlp.gate.b", "l0.mlp.down.b",
                    "l1.mix.left.q.norm", "l1.mix.left.g", "l1.mix.right.g", "l1.mix.right.o", "l2.mix.dkv.norm", "l2.mix.uv"):
        d = write_model(tmp_path / missing, cfg, {k: v for k, v in w.items() if k != missing})
        r = subprocess.run(trace_cmd(tools, d, tmp_path), capture_output=True, text=True)
        assert r.returncode == 2 and missing in r.stderr, (missing, r.stderr)
    layers = cfg["layers"]
    for i, (entry, word) in enumerate(((dict(layers[0], type="convolution"), "convolution"),
                                       (dict(layers[0], mlp={"kind": "routed", "ff": 20}), "routed"),
                                       (dict(layers[0], weights_of=9), "weights_of"), (dict(layers[0], weights_of=0), "weights_of"))):
        d = write_model(tmp_path / f"bad{i}", dict(cfg, layers=[entry]), w)
        r = subprocess.run(trace_cmd(tools, d, tmp_path), capture_output=True, text=True)
        assert r.returncode == 2 and word in r.stderr, (word, r.stderr)


def test_rotation_pairs():
    v = (np.arange(6, dtype=np.float64) + 1).reshape(1, 1, 6).repeat(4, axis=0)
    rot = mo.rotation(4, 100.0)
    a0, a1 = 3.0, 3.0 * 100.0 ** -0.5
    r = mo.rotate(v, rot, neighbours=True)[3, 0]
    assert np.allclose(r, [1 * math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + 1 * math.sin(a0),
                           3 * math.cos(a1) - 4 * math.sin(a1), 4 * math.cos(a1) + 3 * math.sin(a1), 5.0, 6.0])
    r = mo.rotate(v, rot)[3, 0]
    assert np.allclose(r, [1 * math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1),
                           3 * math.cos(a0) + 1 * math.sin(a0), 4 * math.cos(a1) + 2 * math.sin(a1), 5.0, 6.0])
    assert np.allclose(mo.rotate(v, rot)[0], v[0])


def test_frequency_bands():
    """Wavelengths below original / high keep their frequency, above original / low it is divided, in between blended."""
    plain = mo.frequencies(mo.rotation(16, 1000.0))
    assert np.allclose(mo.frequencies(mo.rotation(16, 1000.0, {"factor": 4.0})), plain / 4.0)
    f = mo.frequencies(mo.rotation(16, 1000.0, mo.BANDS))
    length = 2 * math.pi / plain
    short, long = length < 20.0, length > 60.0
    assert short.any() and long.any() and (~short & ~long).any()
    assert np.allclose(f[short], plain[short]) and np.allclose(f[long], plain[long] / 5.0)
    for k in np.where(~short & ~long)[0]:
        s = (60.0 / length[k] - 1.0) / 2.0
        assert 0.0 < s < 1.0 and math.isclose(f[k], plain[k] * (s + (1.0 - s) / 5.0))


def test_masks():
    assert (mo.window_mask(4, 2) == np.array([[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]], dtype=bool)).all()
    assert (mo.chunk_mask(5, 2) == np.array([[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0],
                                             [0, 0, 0, 0, 1]], dtype=bool)).all()
    assert (mo.chunk_mask(4, 1) == np.eye(4, dtype=bool)).all() and (mo.chunk_mask(4, 9) == mo.causal_mask(4)).all()


def test_the_denominator_gains_one():
    s = np.array([[0.0, math.log(3.0)], [500.0, 500.0]])
    p = mo.softmax_rows(s, np.ones((2, 2), dtype=bool), extra=1.0)
    assert np.allclose(p, [[1.0 / 5.0, 3.0 / 5.0], [0.5, 0.5]])
    p = mo.softmax_rows(np.array([[-2.0, 9.0]]), np.array([[True, False]]), extra=1.0)
    assert np.allclose(p, [[math.exp(-2.0) / (1.0 + math.exp(-2.0)), 0.0]])


def test_bigram_rows():
    b = {"buckets": 10, "mul_prev": 7, "mul_cur": 3}
    assert mo.bigram_rows([4, 4, 9], b) == [10, (28 + 12) % 10, (28 + 27) % 10]
    assert mo.bigram_rows([2 ** 31 - 1] * 2, dict(b, mul_prev=2 ** 30)) == [10, ((2 ** 31 - 1) * (2 ** 30 + 3)) % 10]


def test_retention_is_a_decayed_sum():
    """Token by token, against o_t = sum_j decay^(t - j) (q_t . k_j) v_j written out."""
    m = mo.retention_mixer(heads=2, dim=4, vdim=3, rot_dims=4, decay=[0.5, 0.9])
    rng = np.random.default_rng(0)
    w = {"p." + n: rng.standard_normal((rows, 6)) for n, rows in (("q", 8), ("k", 8), ("v", 6), ("g", 6))}
    w["p.o"] = np.eye(6)
    h, eps = rng.standard_normal((7, 6)), 1e-5
    q = mo.rotate((h @ w["p.q"].T).reshape(7, 2, 4), m["rot"])
    k = mo.rotate((h @ w["p.k"].T).reshape(7, 2, 4), m["rot"]) / 2.0
    v = (h @ w["p.v"].T).reshape(7, 2, 3)
    o = np.zeros((7, 2, 3))
    for t in range(7):
        for head, l in enumerate((0.5, 0.9)):
            o[t, head] = sum(l ** (t - j) * (q[t, head] @ k[j, head]) * v[j, head] for j in range(t + 1))
    z = h @ w["p.g"].T
    want = (o / np.sqrt((o ** 2).mean(-1, keepdims=True) + eps)).reshape(7, 6) * z / (1.0 + np.exp(-z))
    assert np.allclose(mo.retention(h, w, "p.", m, eps), want)


def test_clamped_feed_forward():
    w = {"p.gate": np.array([[1.0], [1.0]]), "p.gate.b": np.array([0.0, 5.0]), "p.up": np.array([[1.0], [-9.0]]),
         "p.up.b": np.array([0.25, 0.0]), "p.down": np.eye(2), "p.down.b": np.array([10.0, 20.0])}
    got = mo.clamped_ff(np.array([[1.0]]), w, "p.", 2.0)[0]
    assert np.allclose(got, [10.0 + 1.0 / (1.0 + math.exp(-1.702)) * 2.25, 20.0 + 2.0 / (1.0 + math.exp(-3.404)) * (1.0 - 2.0)])
    got = mo.clamped_ff(np.array([[-8.0]]), w, "p.", 2.0)[0]   # the gate has no lower clamp
    assert np.allclose(got[0], 10.0 - 8.0 / (1.0 + math.exp(8.0 * 1.702)) * (1.0 - 2.0))


def test_shared_weights_resolve_to_their_owner():
    cfg, w = small()
    assert [mo.owner(cfg, i) for i in range(5)] == [0, 1, 2, 0, 1]
    cfg["layers"].append(dict(cfg["layers"][3], weights_of=3))
    assert mo.owner(cfg, 5) == 0
    assert not any(k.startswith(("l3.", "l4.")) for k in w)
