"""Mobatar through the product path (bin/trace_run -> registry -> BatchScheduler -> sequence-batch engine and its
kernels) against the plain float64 restatement in tests/mobatar_oracle.py.  Small random models with bf16-representable
weights; --dtype float32 is compared tightly, bfloat16 loosely."""
import subprocess

import numpy as np
import pytest

import mobatar_oracle as mo
import seq_util
from seq_util import bf16_round, random_tokens as toks, rel_err, row_errors, run_trace, single, whole, write_model

pytestmark = pytest.mark.gpu
TOL32 = 1e-4   # fp32 kernels against float64: rounding only (a lost key or state costs > 1e-2)
TOL16 = 4e-2   # bf16 products
SINK, CHUNK, RET, PAR, LAT = mo.sink_mixer, mo.chunk_mixer, mo.retention_mixer, mo.parallel_mixer, mo.latent_mixer


def ref_logits(cfg, w, tokens):
    return mo.forward(cfg, w, tokens)[0]


def assert_rows(got, ref, tol=TOL32):
    seq_util.assert_rows(got, ref, tol)


def assert_loosely(got, ref):
    """bf16 rows of models without a smooth spread: most rows well inside the tolerance, none far outside."""
    err = row_errors(got, ref)
    assert np.median(err) < TOL16 / 2 and (err > 2 * TOL16).mean() <= 0.02, np.sort(err)[-5:]


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    """All three kinds of layer, with sizes that differ wherever they can: heads, key and value sizes, latent ranks, windows
    and chunks that are no multiple of a key tile or a page, with and without a feed-forward; three layers run again, one of
    them by way of another entry that does."""
    layers = [(SINK(heads=4, kv_heads=2, dim=12, vdim=10), (40, 1.5)),
              (PAR(CHUNK(heads=6, kv_heads=3, chunk=21), RET(heads=5, dim=10, vdim=12)), (56, 0.7)),
              (LAT(heads=2, dim=8, rot_dim=8, vdim=12, kv_rank=36, window=33, base=50.0), None),
              (PAR(CHUNK(heads=2, kv_heads=2, dim=6, vdim=9, chunk=70), RET(heads=2, dim=14, vdim=6), 1.25, 0.5), None),
              1, 2, 0, 4]
    cfg = mo.make_config(width=48, vocab=61, layers=layers)
    w = mo.make_weights(cfg, seed=1, sharp=2.0)
    return cfg, w, write_model(tmp_path_factory.mktemp("moba_base"), cfg, w)


# ---- every mechanism on its own -------------------------------------------------------------------------------------
def only(side, **kw):
    """A pair of mixers one of which has no weight in the sum."""
    return PAR(CHUNK(**kw), RET(), 1.0, 0.0) if side == "left" else PAR(CHUNK(), RET(**kw), 0.0, 1.0)


CASES = {
    "sink": [(SINK(), None)],
    "sink_one_key_head": [(SINK(heads=4, kv_heads=1, dim=16, vdim=6), None)],
    "sink_every_head_its_keys": [(SINK(heads=3, kv_heads=3), None)],
    "sink_divided_frequencies": [(SINK(scaling={"factor": 6.0}), None)],
    "sink_plain_frequencies": [(SINK(scaling=None), None)],
    "sink_other_bands": [(SINK(dim=20, rot_dims=20, scaling={"factor": 2.0, "low": 0.5, "high": 8.0, "original": 200}), None)],
    "sink_two_rotated": [(SINK(rot_dims=2), None)],
    "sink_scaled": [(SINK(scale=1.7), None)],
    "sink_wide": [(SINK(heads=2, kv_heads=1, dim=136, vdim=72, rot_dims=96, scale=0.03), None)],
    "sink_values_beyond_the_tiles": [(SINK(heads=2, kv_heads=1, dim=8, vdim=260), None)],
    "sink_keys_beyond_the_tiles": [(SINK(heads=4, kv_heads=2, dim=520, vdim=6, rot_dims=32, scale=0.01), None)],
    "chunk": [(only("left"), None)],
    "chunk_of_one": [(only("left", chunk=1), None)],
    "chunk_of_two": [(only("left", chunk=2), None)],
    "chunk_of_a_key_tile": [(only("left", chunk=64), None)],
    "chunk_of_half_a_key_tile": [(only("left", chunk=32), None)],
    "chunk_past_the_prompt": [(only("left", chunk=500), None)],
    "chunk_one_key_head": [(only("left", heads=4, kv_heads=1, dim=16, vdim=20), None)],
    "chunk_one_head": [(only("left", heads=1, kv_heads=1), None)],
    "chunk_all_rotated": [(only("left", dim=12, rot_dims=12, factor=1.0), None)],
    "chunk_wide": [(only("left", heads=2, kv_heads=1, dim=136, vdim=72, rot_dims=64, chunk=40), None)],
    "chunk_values_beyond_the_tiles": [(only("left", heads=2, kv_heads=1, dim=8, vdim=260, chunk=40), None)],
    "retention": [(only("right"), None)],
    "retention_one_head": [(only("right", heads=1), None)],
    "retention_all_rotated": [(only("right", dim=12, rot_dims=12), None)],
    "retention_two_rotated": [(only("right", rot_dims=2), None)],
    "retention_one_decay": [(only("right", heads=4, decay=[0.96] * 4), None)],
    "retention_no_decay": [(only("right", heads=2, decay=[1.0, 1.0]), None)],
    "retention_forgets_at_once": [(only("right", heads=2, decay=[0.0, 2.0 ** -12]), None)],
    "retention_wide": [(only("right", heads=2, dim=72, vdim=100, rot_dims=40), None)],
    "retention_flat": [(only("right", heads=3, dim=2, vdim=40, rot_dims=2), None)],
    "parallel": [(PAR(), None)],
    "parallel_other_scales": [(PAR(left_scale=-2.0, right_scale=0.125), None)],
    "latent": [(LAT(), None)],
    "latent_one_head": [(LAT(heads=1), None)],
    "latent_window_one": [(LAT(window=1), None)],
    "latent_window_past_the_prompt": [(LAT(window=500), None)],
    "latent_two_rotated": [(LAT(rot_dim=2, base=7.0), None)],
    "latent_rank_past_a_key_tile": [(LAT(heads=2, kv_rank=136, dim=24, rot_dim=16, vdim=72), None)],
    "latent_rank_smaller_than_a_head": [(LAT(kv_rank=3, dim=12), None)],
    "ff": [(SINK(), (30, 1.0))],
    "ff_tight_clamp": [(SINK(), (30, 0.25))],
    "ff_wide_clamp": [(SINK(), (30, 50.0))],
    "ff_past_a_block": [(LAT(), (136, 1.0))],
    "weights_again": [(PAR(), (20, 1.0)), 0, (LAT(), None), 2, 0],
    "weights_again_by_way_of_another": [(SINK(), (20, 1.0)), 0, 1, 2],
}


@pytest.mark.parametrize("case", sorted(CASES))
def test_mechanism_alone(tmp_path, case):
    # a large eps in some cases: it must reach every norm (outputs, whole projections, unit norms, latents, heads)
    big_eps = case in ("sink", "chunk", "retention", "latent", "parallel", "ff", "chunk_one_head")
    cfg = mo.make_config(width=40, vocab=50, layers=CASES[case], eps=0.05 if big_eps else 3e-6)
    w = mo.make_weights(cfg, seed=3, sharp=2.0)
    if case.startswith("ff"):  # the mixer's output projection is zero: what is left of the layer is the feed-forward
        w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    d = write_model(tmp_path, cfg, w)
    t = toks(85, cfg["vocab"], 5)
    ref, trace = mo.forward(cfg, w, t)
    logits, resid = run_trace(d, [whole("a", t)], residual=True)
    got = resid[0].reshape(trace.shape)
    assert np.abs(got - trace).max() < 1e-4 * max(1.0, np.abs(trace).max())
    assert_rows(logits[0], ref)
    # without the residual trace, and decoded
    logits, _ = run_trace(d, [whole("b", t[:80], want=[0, 3, 64, 79], end=False)] + single("b", t[80:]))
    assert_rows(np.concatenate(logits), ref[[0, 3, 64, 79, 80, 81, 82, 83, 84]])


def test_residual_after_every_layer_run(base):
    cfg, w, d = base
    t = toks(33, cfg["vocab"], 7)
    _, trace = mo.forward(cfg, w, t)
    assert trace.shape[0] == 8
    _, resid = run_trace(d, [whole("a", t)], residual=True)
    got = resid[0].reshape(trace.shape)
    for r in range(trace.shape[0]):
        assert np.abs(got[r] - trace[r]).max() < 1e-4 * max(1.0, np.abs(trace[r]).max()), f"layer run {r}"


@pytest.mark.parametrize("order", ["PL", "LSS", "SPLPS"])
def test_layer_orders(tmp_path, order):
    kinds = {"P": PAR(CHUNK(chunk=9)), "L": LAT(window=7), "S": SINK()}
    cfg = mo.make_config(width=40, vocab=60, layers=[(kinds[c], (24, 1.0) if i % 2 else None) for i, c in enumerate(order)])
    w = mo.make_weights(cfg, seed=101, sharp=2.0)
    d = write_model(tmp_path, cfg, w)
    t = toks(45, cfg["vocab"], 102)
    logits, _ = run_trace(d, [whole("a", t[:30], end=False)] + single("a", t[30:]))
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


def test_a_layer_that_runs_again_has_a_cache_of_its_own(tmp_path):
    """The same weights three times in a row: with one cache (or one state) for the three runs, the later runs would find
    the first one's keys."""
    for mixer in (SINK(), PAR(), LAT()):
        cfg = mo.make_config(width=32, vocab=40, layers=[(mixer, None), 0, 0])
        w = mo.make_weights(cfg, seed=12, sharp=2.0)
        t = toks(40, cfg["vocab"], 13)
        d = write_model(tmp_path, cfg, w)
        logits, _ = run_trace(d, [whole("a", t[:20], end=False)] + single("a", t[20:]), page=8)
        assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


# ---- the bigram embedding -------------------------------------------------------------------------------------------
def bigram_model(**kw):
    cfg = mo.make_config(width=24, vocab=30, layers=[(SINK(), None)], **kw)
    w = mo.make_weights(cfg, seed=21)
    w["embed"] = bf16_round(w["embed"] * 0.125)  # the bigram's row is most of a token's embedding
    return cfg, w


@pytest.mark.parametrize("kw", [{}, {"buckets": 1}, {"buckets": 1021, "mul_prev": 2000003, "mul_cur": 1}, {"mul_prev": 0},
                                {"mul_cur": 0}, {"buckets": 999, "mul_prev": 2147483647, "mul_cur": 2147480003}])
def test_bigram_rows(tmp_path, kw):
    """The previous token is state: across a prompt, across portions, in single-token steps and in a batch."""
    cfg, w = bigram_model(**kw)
    d = write_model(tmp_path, cfg, w)
    t, u = toks(30, cfg["vocab"], 22), toks(12, cfg["vocab"], 23)
    steps = [{"entries": [{"id": "t", "tokens": t[:11], "want": list(range(11))}, {"id": "u", "tokens": u[:1], "want": [0]}]},
             {"entries": [{"id": "u", "tokens": u[1:3], "want": [0, 1]}, {"id": "t", "tokens": t[11:20], "want": list(range(9))}]}]
    for j in range(9):
        steps.append({"entries": [{"id": "t", "tokens": [t[20 + j]], "want": [0]}, {"id": "u", "tokens": [u[3 + j]], "want": [0]}]})
    logits, _ = run_trace(d, steps)
    got_t = np.concatenate([logits[0][:11], logits[1][2:]] + [lg[:1] for lg in logits[2:]])
    got_u = np.concatenate([logits[0][11:], logits[1][:2]] + [lg[1:] for lg in logits[2:]])
    assert_rows(got_t, ref_logits(cfg, w, t)[:29])
    assert_rows(got_u, ref_logits(cfg, w, u))


def test_the_first_token_takes_the_row_behind_the_buckets(tmp_path):
    """Also when its slot was another sequence's before."""
    cfg, w = bigram_model()
    w["bigram"][-1] *= 8.0
    t, u = toks(9, cfg["vocab"], 24), toks(5, cfg["vocab"], 25)
    ref = ref_logits(cfg, w, u)
    w2 = dict(w, bigram=np.concatenate([w["bigram"][:-1], w["bigram"][:1]]))
    assert rel_err(ref_logits(cfg, w2, u)[:1], ref[:1]) > 0.1
    d = write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("t", t)] + single("u", u, end=True) + [whole("v", u)], extra=["--max-seqs", "1"])
    assert_rows(np.concatenate(logits[1:6]), ref)
    assert_rows(logits[6], ref)


# ---- keys at the edges of windows and chunks, far keys --------------------------------------------------------------
def edge_model(kind, reach, special, vocab=30, width=24, seed=9):
    """One layer, made so that ONE token's key outweighs all others while it is seen.  Input coordinate 1 is the same for
    every token and feeds the last (unrotated) coordinate of every query head; input coordinate 0 is zero except for the
    special token and feeds the same coordinate of the keys (a latent attention: by way of latent coordinate 0), and nothing
    else does."""
    if kind == "latent":
        m, p, per = LAT(heads=2, dim=8, rot_dim=4, vdim=6, kv_rank=10, window=reach, scale=3.0), "l0.mix.", 12
    elif kind == "sink":
        m, p, per = SINK(heads=2, kv_heads=1, dim=8, vdim=6, rot_dims=6, scale=3.0), "l0.mix.", 8
    elif kind == "chunk":
        m, p, per = PAR(CHUNK(heads=2, kv_heads=1, dim=8, vdim=6, rot_dims=6, chunk=reach, scale=3.0), RET(), 1.0, 0.0), "l0.mix.left.", 8
    else:
        m, p, per = PAR(CHUNK(), RET(heads=2, dim=8, vdim=6, rot_dims=6, decay=[reach, reach]), 0.0, 1.0), "l0.mix.right.", 8
    # the bigram's row depends on the token alone: a special token leaves no trace but its key and value
    cfg = mo.make_config(width=width, vocab=vocab, layers=[(m, None)], mul_prev=0)
    w = mo.make_weights(cfg, seed=seed)
    w["embed"][:, 0] = 0.0
    w["embed"][special, 0] = 8.0
    w["embed"][:, 1] = 2.0
    w["bigram"][:, :2] = 0.0
    w["bigram"] = bf16_round(w["bigram"] * 0.25)
    w[p + "q"] = bf16_round(w[p + "q"] * 0.05)
    for head in range(2):
        w[p + "q"][head * per + 7] = 0.0
        w[p + "q"][head * per + 7, 1] = 4.0
    if kind == "latent":
        w[p + "dkv"][:, :2] = 0.0
        w[p + "dkv"][0] = 0.0
        w[p + "dkv"][0, 0] = 4.0
        w[p + "uk"][:, 0] = 0.0
        for head in range(2):
            w[p + "uk"][head * 8 + 7] = 0.0
            w[p + "uk"][head * 8 + 7, 0] = 2.0
    else:
        if kind == "chunk":
            w[p + "q.norm"][:] = 1.0
            w[p + "k.norm"][:] = 1.0
        w[p + "k"][:, :2] = 0.0
        for head in range(len(w[p + "k"]) // 8):
            w[p + "k"][head * 8 + 7] = 0.0
            w[p + "k"][head * 8 + 7, 0] = 32.0 if kind == "retention" else 2.0
    return cfg, w


def plain_tokens(n, cfg, special, seed, places=()):
    t = [x if x != special else special + 1 for x in toks(n, cfg["vocab"], seed)]
    for p in places:
        t[p] = special
    return t


def without(t, place, special):
    """The special token's place taken by another."""
    return t[:place] + [special + 1] + t[place + 1:]


@pytest.mark.parametrize("window", [2, 17, 64, 65, 100])
def test_the_key_at_the_window_edge_carries_the_output(tmp_path, window):
    """One special key leaves the window inside the prompt, another while tokens are decoded one by one (across key tiles and
    pages).  The last position that still sees it depends on it heavily, the next one not at all."""
    special, n_prompt = 7, 150
    cfg, w = edge_model("latent", window, special)
    places = (20, n_prompt - 5)
    t = plain_tokens(n_prompt + window + 20, cfg, special, 13, places)
    ref = ref_logits(cfg, w, t)
    for p in places:  # the construction works
        other = ref_logits(cfg, w, without(t, p, special))
        assert rel_err(other[p + window - 1:p + window], ref[p + window - 1:p + window]) > 0.1
        assert rel_err(other[p + window:p + window + 1], ref[p + window:p + window + 1]) < 1e-9
    d = write_model(tmp_path, cfg, w)
    steps = [whole("a", t[:n_prompt], end=False)] + single("a", t[n_prompt:])
    for dtype, tol in (("float32", TOL32), ("bfloat16", TOL16)):
        logits, _ = run_trace(d, steps, page=16, dtype=dtype)
        assert rel_err(np.concatenate(logits), ref) < tol


@pytest.mark.parametrize("chunk", [2, 17, 64, 65, 100])
def test_keys_at_the_edges_of_a_chunk(tmp_path, chunk):
    """Special keys on the first and on the last place of a chunk, in the prompt and where the chunk's end is decoded: the
    first carries the output up to the chunk's end and not a position further, the last only its own."""
    special = 7
    cfg, w = edge_model("chunk", chunk, special)
    c0 = 2 * chunk                       # a chunk inside the prompt
    n_prompt = 4 * chunk + (chunk + 1) // 2
    c1 = 4 * chunk                       # a chunk that starts in the prompt and ends in decoding
    n_all = 6 * chunk + 3
    places = (c0, c0 + 2 * chunk - 1, c1, n_all - 4)  # n_all - 4: the last place of a decoded chunk
    t = plain_tokens(n_all, cfg, special, 14, places)
    ref = ref_logits(cfg, w, t)

    def differs(place, at):
        return rel_err(ref_logits(cfg, w, without(t, place, special))[at:at + 1], ref[at:at + 1])
    for first in (c0, c1):
        assert differs(first, first + chunk - 1) > 0.1 and differs(first, first + chunk) < 1e-9
    last = c0 + 2 * chunk - 1
    assert differs(last, last) > 0.1 and differs(last, last + 1) < 1e-9
    d = write_model(tmp_path, cfg, w)
    steps = [whole("a", t[:n_prompt], end=False)] + single("a", t[n_prompt:])
    for dtype, tol in (("float32", TOL32), ("bfloat16", TOL16)):
        logits, _ = run_trace(d, steps, page=16, dtype=dtype)
        assert rel_err(np.concatenate(logits), ref) < tol


def test_chunks_count_from_the_start_of_the_sequence(tmp_path):
    """Portions that end inside, at and just past a chunk's edge."""
    special, chunk = 7, 16
    cfg, w = edge_model("chunk", chunk, special)
    t = plain_tokens(100, cfg, special, 15, (0, 15, 31, 32, 50, 79))
    ref = ref_logits(cfg, w, t)
    d = write_model(tmp_path, cfg, w)
    for sizes in ((16, 16, 68), (15, 2, 31, 52), (17, 30, 1, 52), (7, 7, 7, 7, 7, 65), (2,) * 50):
        steps, at = [], 0
        for n in sizes:
            steps.append(whole("p", t[at:at + n], end=False))
            at += n
        logits, _ = run_trace(d, steps, page=8)
        assert_rows(np.concatenate(logits), ref)


@pytest.mark.parametrize("kind", ["sink", "retention"])
def test_a_far_key(tmp_path, kind):
    """One key among hundreds, far back, carries the output at the end of the prompt and while decoding."""
    special = 7
    cfg, w = edge_model(kind, 0.9999, special)
    t = plain_tokens(420, cfg, special, 16, (3,))
    ref = ref_logits(cfg, w, t)
    assert rel_err(ref_logits(cfg, w, without(t, 3, special))[-1:], ref[-1:]) > 0.1
    d = write_model(tmp_path, cfg, w)
    for dtype, tol in (("float32", TOL32), ("bfloat16", TOL16)):
        logits, _ = run_trace(d, [whole("a", t[:400], end=False)] + single("a", t[400:]), dtype=dtype)
        assert rel_err(np.concatenate(logits), ref) < tol


def test_retention_decays_with_each_token(tmp_path):
    """The far token again under a decay that has faded it by a known amount: twice the distance, the square of it."""
    special = 7
    cfg, w = edge_model("retention", 0.98, special)
    t = plain_tokens(330, cfg, special, 17, (2,))
    ref = ref_logits(cfg, w, t)
    slow = ref_logits(dict(cfg, layers=[dict(cfg["layers"][0], mixer=PAR(CHUNK(), dict(cfg["layers"][0]["mixer"]["right"], decay=[0.985, 0.98]), 0.0, 1.0))]), w, t)
    assert rel_err(slow[250:], ref[250:]) > 0.02
    d = write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("a", t[:300], end=False)] + single("a", t[300:]))
    assert_rows(np.concatenate(logits), ref)


def test_the_one_in_the_denominator(tmp_path):
    """Two heads whose scores differ: the added one takes more of the head that scores low, so it shows through the norm of
    the output -- most at the first tokens, where few keys share the sum."""
    m = SINK(heads=2, kv_heads=2, dim=8, vdim=6, scale=0.4)
    cfg = mo.make_config(width=24, vocab=30, layers=[(m, None)])
    w = mo.make_weights(cfg, seed=31)
    w["l0.mix.k"] = w["l0.mix.q"].copy()
    w["l0.mix.k"][8:] *= -1.0            # head 0 scores its own position high, head 1 low
    t = toks(40, cfg["vocab"], 32)
    ref = ref_logits(cfg, w, t)
    saved, mo.MIXERS["attention"] = mo.MIXERS["attention"], lambda h, w_, p, m_, eps: no_sink(h, w_, p, m_, eps)

    def no_sink(h, w_, p, m_, eps):
        T, H, G, dim, vd = h.shape[0], m_["heads"], m_["kv_heads"], m_["dim"], m_["vdim"]
        q, k = (mo.rms_unit(mo.rotate((h @ w_[p + n].T).reshape(T, x, dim), m_["rot"]), eps) for n, x in (("q", H), ("k", G)))
        v = (h @ w_[p + "v"].T).reshape(T, G, vd)
        return mo.grouped_softmax(q, k, v, mo.causal_mask(T), m_["scale"]).reshape(T, H * vd) @ w_[p + "o"].T
    try:
        assert rel_err(ref_logits(cfg, w, t)[:2], ref[:2]) > 0.05
    finally:
        mo.MIXERS["attention"] = saved
    d = write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("a", t), whole("b", t[:1], end=False)] + single("b", t[1:]))
    assert_rows(logits[0], ref)
    assert_rows(np.concatenate(logits[1:]), ref)


@pytest.mark.parametrize("kind", ["sink", "retention", "latent"])
def test_the_rotation_is_seen_at_far_positions(tmp_path, kind):
    """Scores from rotated coordinates alone at positions in the hundreds: a wrong pairing, base, scaling or position changes
    which keys win."""
    m = {"sink": SINK(heads=2, kv_heads=1, dim=16, rot_dims=16, scale=1.5),
         "retention": PAR(CHUNK(), RET(heads=2, dim=16, vdim=8, rot_dims=16, decay=[0.999, 0.9995]), 0.0, 1.0),
         "latent": LAT(heads=2, dim=4, rot_dim=16, kv_rank=12, window=90, base=5e5)}[kind]
    cfg = mo.make_config(width=32, vocab=40, layers=[(m, None)])
    w = mo.make_weights(cfg, seed=18)
    if kind == "latent":
        for head in range(2):
            w["l0.mix.q"][head * 20:head * 20 + 4] = 0.0
            w["l0.mix.q"][head * 20 + 4:head * 20 + 20] *= 4.0
    t = toks(330, cfg["vocab"], 19)
    d = write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("a", t[:300], end=False)] + single("a", t[300:]))
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


# ---- prompt against token-by-token decoding, long prompts, long decoding, portions -----------------------------------
@pytest.mark.parametrize("page", [4, 16, 64])
def test_long_prompt_every_position(base, page):
    cfg, w, d = base
    t = toks(203, cfg["vocab"], 11)  # past three key tiles of 64, no multiple of a page
    logits, _ = run_trace(d, [whole("a", t)], page=page)
    assert_rows(logits[0], ref_logits(cfg, w, t))


def test_prefill_equals_stepwise_decoding(base):
    cfg, w, d = base
    t = toks(90, cfg["vocab"], 17)
    ref = ref_logits(cfg, w, t)
    split = [whole("p", t[:2], end=False)] + single("p", t[2:])
    logits, _ = run_trace(d, single("s", t) + split, page=8)   # "s": from the very first token
    a, b = np.concatenate(logits[:len(t)]), np.concatenate(logits[len(t):])
    assert_rows(a, ref)
    assert_rows(b, ref)


def test_long_decoding(base):
    """Decoding far past every window, chunk, key tile and page."""
    cfg, w, d = base
    t = toks(40 + 260, cfg["vocab"], 19)
    logits, _ = run_trace(d, [whole("a", t[:40], end=False)] + single("a", t[40:]), page=16)
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 2, 2, 2), (5, 64, 3, 17), (33, 2, 70), (1, 99, 2), (1, 1, 2, 1, 40, 1, 2), (65, 66, 67)])
def test_prompt_in_portions(base, tmp_path, sizes, dtype):
    """A prompt fed in several steps: every portion starts from the cache and the state that the portions before it left.  A
    second request of another length rides along."""
    cfg, w, d = base
    if dtype == "bfloat16":  # softmaxes that are not sharpened: a peaky one amplifies the rounding of its scores
        w = mo.make_weights(cfg, seed=1)
        d = write_model(tmp_path, cfg, w)
    t = toks(sum(sizes), cfg["vocab"], 81)
    other = toks(2 * len(sizes) + 1, cfg["vocab"], 82)
    steps, at = [], 0
    for i, n in enumerate(sizes):
        o = other[2 * i:2 * i + 2] if i + 1 < len(sizes) else other[2 * i:]
        steps.append({"entries": [{"id": "o", "tokens": o, "want": list(range(len(o)))},
                                  {"id": "p", "tokens": t[at:at + n], "want": list(range(n))}]})
        at += n
    logits, _ = run_trace(d, steps, page=8, max_tokens=512, dtype=dtype)
    got_o = np.concatenate([lg[:len(st["entries"][0]["tokens"])] for lg, st in zip(logits, steps)])
    got_p = np.concatenate([lg[len(st["entries"][0]["tokens"]):] for lg, st in zip(logits, steps)])
    for got, seq in ((got_p, t), (got_o, other)):
        if dtype == "float32":
            assert_rows(got, ref_logits(cfg, w, seq))
        else:
            assert np.median(row_errors(got, ref_logits(cfg, w, seq))) < TOL16


# ---- batches ----------------------------------------------------------------------------------------------------------
def test_unequal_batch_equals_each_alone(base):
    cfg, w, d = base
    prompts = {"x": toks(1, cfg["vocab"], 21), "y": toks(67, cfg["vocab"], 22), "z": toks(130, cfg["vocab"], 23)}
    tails = {k: toks(n, cfg["vocab"], 30 + i) for i, (k, n) in enumerate({"x": 3, "y": 30, "z": 7}.items())}
    steps = [{"entries": [{"id": k, "tokens": p, "want": list(range(len(p)))} for k, p in prompts.items()]}]
    for j in range(30):
        live = [k for k in prompts if j < len(tails[k])]
        steps.append({"entries": [{"id": k, "tokens": [tails[k][j]], "want": [0]} for k in live],
                      "end": [k for k in live if j == len(tails[k]) - 1]})
    logits, _ = run_trace(d, steps, page=8, max_tokens=320)
    for k in prompts:
        rows, at = [], 0
        for kk, p in prompts.items():
            if kk == k:
                rows.append(logits[0][at:at + len(p)])
            at += len(p)
        for j in range(len(tails[k])):
            live = [kk for kk in prompts if j < len(tails[kk])]
            rows.append(logits[1 + j][live.index(k)][None])
        assert_rows(np.concatenate(rows), ref_logits(cfg, w, prompts[k] + tails[k]))


def test_prompts_beside_decoding_requests(base):
    """A step that brings a new prompt, a portion and single tokens at once."""
    cfg, w, d = base
    a, b, c = toks(60, cfg["vocab"], 24), toks(50, cfg["vocab"], 25), toks(20, cfg["vocab"], 26)
    steps = [{"entries": [{"id": "a", "tokens": a[:57], "want": [56]}, {"id": "b", "tokens": b[:20], "want": [19]}]},
             {"entries": [{"id": "a", "tokens": a[57:58], "want": [0]}, {"id": "b", "tokens": b[20:49], "want": list(range(29))},
                          {"id": "c", "tokens": c[:18], "want": list(range(18))}]},
             {"entries": [{"id": "c", "tokens": c[18:20], "want": [0, 1]}, {"id": "a", "tokens": a[58:59], "want": [0]},
                          {"id": "b", "tokens": b[49:50], "want": [0]}]}]
    logits, _ = run_trace(d, steps, page=8, max_tokens=256)
    ra, rb, rc = (ref_logits(cfg, w, x) for x in (a, b, c))
    assert_rows(np.concatenate([logits[0][0:1], logits[1][0:1], logits[2][2:3]]), ra[56:59])
    assert_rows(np.concatenate([logits[0][1:2], logits[1][1:30], logits[2][3:4]]), rb[19:50])
    assert_rows(np.concatenate([logits[1][30:], logits[2][0:2]]), rc)


def test_pages_and_slots_are_reused(base):
    """The pool holds one request at a time: each runs in the pages and the slot that the one before it gave back, and
    must see nothing of it."""
    cfg, w, d = base
    reqs = [toks(n, cfg["vocab"], 40 + i) for i, n in enumerate([50, 33, 64, 7, 50])]
    steps = []
    for i, t in enumerate(reqs):
        steps.append(whole(f"r{i}", t[:-3], end=False))
        steps += single(f"r{i}", t[-3:], end=True)
    logits, _ = run_trace(d, steps, page=4, max_tokens=64, extra=["--max-seqs", "1"])
    for i, t in enumerate(reqs):
        assert_rows(np.concatenate(logits[4 * i:4 * i + 4]), ref_logits(cfg, w, t))


def test_a_freed_slot_starts_afresh(base):
    """Two slots; requests come and go in an order that hands a slot with a long history to a request that starts by
    decoding from its first token."""
    cfg, w, d = base
    a, b, c = toks(80, cfg["vocab"], 61), toks(12, cfg["vocab"], 62), toks(9, cfg["vocab"], 63)
    steps = [{"entries": [{"id": "a", "tokens": a, "want": [79]}, {"id": "b", "tokens": b[:6], "want": [5]}], "end": ["a"]}]
    for j in range(6):  # c takes a's slot and decodes from its first token beside b
        steps.append({"entries": [{"id": "b", "tokens": [b[6 + j]], "want": [0]}, {"id": "c", "tokens": [c[j]], "want": [0]}]})
    logits, _ = run_trace(d, steps, max_tokens=128, extra=["--max-seqs", "2"])
    assert_rows(np.concatenate([logits[0][1:2]] + [lg[0:1] for lg in logits[1:]]), ref_logits(cfg, w, b)[5:])
    assert_rows(np.concatenate([lg[1:2] for lg in logits[1:]]), ref_logits(cfg, w, c)[:6])
    assert_rows(logits[0][0:1], ref_logits(cfg, w, a)[79:])


def test_first_tokens_and_single_token_requests(base):
    cfg, w, d = base
    ts = [toks(n, cfg["vocab"], 50 + n) for n in (1, 2, 3, 4)]
    logits, _ = run_trace(d, [whole(f"q{i}", t) for i, t in enumerate(ts)])
    for t, lg in zip(ts, logits):
        assert_rows(lg, ref_logits(cfg, w, t))


def test_steps_without_wanted_rows(base):
    cfg, w, d = base
    t = toks(30, cfg["vocab"], 55)
    steps = [whole("a", t[:20], want=[], end=False), whole("a", t[20:21], want=[], end=False), whole("a", t[21:], end=True)]
    logits, _ = run_trace(d, steps)
    assert logits[0] is None and logits[1] is None
    assert_rows(logits[2], ref_logits(cfg, w, t)[21:])


def test_many_requests_in_one_batch(base):
    """80 prompts of 1..5 tokens in one step, then decoded together."""
    cfg, w, d = base
    reqs = [toks(1 + i % 5, cfg["vocab"], 200 + i) + toks(2, cfg["vocab"], 400 + i) for i in range(80)]
    steps = [{"entries": [{"id": f"r{i}", "tokens": r[:-2], "want": [len(r) - 3]} for i, r in enumerate(reqs)]}]
    for j in (2, 1):
        steps.append({"entries": [{"id": f"r{i}", "tokens": [r[-j]], "want": [0]} for i, r in enumerate(reqs)]})
    logits, _ = run_trace(d, steps, max_tokens=1024)
    for i, r in enumerate(reqs):
        assert_rows(np.stack([logits[0][i], logits[1][i], logits[2][i]]), ref_logits(cfg, w, r)[-3:])


# ---- bf16, other sizes, generation ------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind,dim,vdim,reach", [("latent", 24, 40, 17), ("latent", 96, 64, 150), ("latent", 20, 24, 30),
                                                 ("sink", 24, 24, 0), ("sink", 64, 128, 0), ("sink", 128, 64, 0),
                                                 ("chunk", 24, 24, 17), ("chunk", 64, 32, 64), ("chunk", 128, 64, 150),
                                                 ("chunk", 40, 200, 40), ("chunk", 16, 120, 63)])
def test_bfloat16_prompts_on_the_tensor_cores(tmp_path, kind, dim, vdim, reach):
    """bf16 prompt steps with head sizes that are multiples of 8 take the tensor-core attention: against the float64
    restatement, and against single-token steps of the same run.  A latent head of 20 and values of 200 fall back to the
    split-key kernel."""
    mixer = {"latent": lambda: LAT(heads=4, dim=dim, rot_dim=16, vdim=vdim, kv_rank=56, window=reach),
             "sink": lambda: SINK(heads=6, kv_heads=2, dim=dim, vdim=vdim, rot_dims=16, scale=dim ** -0.5),
             "chunk": lambda: PAR(CHUNK(heads=6, kv_heads=2, dim=dim, vdim=vdim, rot_dims=8, chunk=reach),
                                  RET(heads=4, dim=24, vdim=40, rot_dims=16))}[kind]()
    cfg = mo.make_config(width=64, vocab=80, layers=[(mixer, (136, 1.5)), 0])
    w = mo.make_weights(cfg, seed=41, sharp=1.25)
    d = write_model(tmp_path, cfg, w)
    t = toks(260, cfg["vocab"], 42)
    ref = ref_logits(cfg, w, t)
    steps = [whole("a", t, end=True), whole("b", t[:200], end=False)] + single("b", t[200:])
    logits, _ = run_trace(d, steps, dtype="bfloat16")
    assert_loosely(logits[0], ref)
    assert_loosely(np.concatenate(logits[1:]), ref)
    assert_loosely(np.concatenate(logits[2:]), logits[0][200:])


@pytest.mark.parametrize("dim,vdim,rot_dims", [(16, 16, 16), (48, 96, 24), (64, 112, 36), (80, 32, 6), (128, 128, 128)])
def test_retention_of_long_entries_on_the_tensor_cores(tmp_path, monkeypatch, dim, vdim, rot_dims):
    """bf16 steps with long entries: entries around multiples of the chunk beside short ones, a second portion that starts from
    the first one's state, decays from nothing to none -- against the float64 restatement, and closely against the same run on
    the fp32 kernels (both round the same projections)."""
    right = RET(heads=5, dim=dim, vdim=vdim, rot_dims=rot_dims, base=2000.0, decay=[0.0, 0.6, 0.97, 0.9995, 1.0])
    cfg = mo.make_config(width=64, vocab=80, layers=[(PAR(CHUNK(), right, 0.0, 1.0), None)])
    w = mo.make_weights(cfg, seed=61)
    d = write_model(tmp_path, cfg, w)
    sizes = {"a": (63, 70), "b": (64, 65), "c": (129, 2), "d": (5, 192), "e": (200, 1)}
    reqs = {k: toks(sum(n), cfg["vocab"], 62 + i) for i, (k, n) in enumerate(sizes.items())}
    steps, at = [], {k: 0 for k in sizes}
    for part in range(2):
        steps.append({"entries": [{"id": k, "tokens": reqs[k][at[k]:at[k] + n[part]], "want": list(range(n[part]))}
                                  for k, n in sizes.items()]})
        at = {k: n[0] for k, n in sizes.items()}
    steps.append({"entries": [{"id": k, "tokens": [7], "want": [0]} for k in sizes]})
    logits, _ = run_trace(d, steps, dtype="bfloat16")
    monkeypatch.setenv("KLLM_SEQ_LINEAR_MMA", "0")
    plain, _ = run_trace(d, steps, dtype="bfloat16")
    for got, want in zip(logits, plain):
        assert row_errors(got, want).max() < 1e-2
    for k, n in sizes.items():
        ref = ref_logits(cfg, w, reqs[k] + [7])
        rows, i = [], list(sizes).index(k)
        for part in range(2):
            b = sum(sizes[x][part] for x in list(sizes)[:i])
            rows.append(logits[part][b:b + n[part]])
        assert_loosely(np.concatenate(rows + [logits[2][i:i + 1]]), ref)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_fit_no_vector(tmp_path, dtype):
    """Odd sizes everywhere: no 16-byte vector load, no tensor-core tile and no warp-sized loop fits."""
    layers = [(LAT(heads=3, dim=5, rot_dim=2, vdim=3, kv_rank=11, window=7), (11, 1.0)),
              (PAR(CHUNK(heads=3, kv_heads=1, dim=7, vdim=5, chunk=13, rot_dims=2), RET(heads=3, dim=5, vdim=3, rot_dims=2)), (9, 0.5)),
              (SINK(heads=5, kv_heads=5, dim=3, vdim=1, rot_dims=2), None), 1]
    cfg = mo.make_config(width=21, vocab=23, layers=layers, buckets=19)
    w = mo.make_weights(cfg, seed=51)
    d = write_model(tmp_path, cfg, w)
    t = toks(97, cfg["vocab"], 52)
    logits, _ = run_trace(d, [whole("a", t[:90], end=False)] + single("a", t[90:]), dtype=dtype)
    got, ref = np.concatenate(logits), ref_logits(cfg, w, t)
    if dtype == "float32":
        assert_rows(got, ref)
    else:
        assert np.median(row_errors(got, ref)) < TOL16


def random_design(seed):
    rng = np.random.default_rng(seed)

    def pick(*xs):
        return xs[int(rng.integers(len(xs)))]

    def mixer():
        kind, g = pick("latent", "sink", "parallel", "parallel"), pick(1, 2, 3)
        if kind == "latent":
            return LAT(heads=pick(1, 2, 5), dim=pick(3, 8, 16), rot_dim=pick(2, 8), vdim=pick(3, 8, 16), kv_rank=pick(4, 16, 70),
                       window=pick(1, 5, 30, 66), base=pick(100.0, 10000.0, 5e5))
        if kind == "sink":
            return SINK(heads=g * pick(1, 2, 4), kv_heads=g, dim=pick(4, 8, 12), vdim=pick(3, 8, 16), rot_dims=pick(2, 4),
                        scaling=pick(None, {"factor": 2.0}, mo.BANDS), scale=pick(0.2, 0.5))
        left = CHUNK(heads=g * pick(1, 2, 4), kv_heads=g, dim=pick(4, 8, 12), vdim=pick(3, 8, 16), chunk=pick(1, 5, 30, 66),
                     rot_dims=pick(2, 4), factor=pick(1.0, 8.0))
        dim = pick(2, 8, 12)
        right = RET(heads=pick(1, 2, 5), dim=dim, vdim=pick(4, 16, 33), rot_dims=pick(2, dim))
        return PAR(left, right, pick(0.5, 1.0, 1.5), pick(0.5, 1.0))

    layers = []
    for i in range(int(rng.integers(2, 8))):
        layers.append(pick(*range(i)) if i and pick(0, 0, 1) else (mixer(), pick(None, (8, 1.0), (30, 2.5))))
    return mo.make_config(width=pick(16, 24, 40), vocab=pick(17, 50), layers=layers, eps=pick(1e-6, 1e-3), buckets=pick(5, 64),
                          mul_prev=pick(3, 1000), mul_cur=pick(1, 77))


@pytest.mark.parametrize("seed", range(1, 11))
def test_random_designs(tmp_path, seed):
    """Layer order, sizes, shared weights and constants drawn at random; a ragged batch that is prefilled together and decoded
    together, in float32 (tight) and bfloat16 (loose)."""
    cfg = random_design(seed)
    w = mo.make_weights(cfg, seed=100 + seed, sharp=1.25)
    d = write_model(tmp_path, cfg, w)
    reqs = {"a": toks(90, cfg["vocab"], 300 + seed), "b": toks(23, cfg["vocab"], 400 + seed), "c": toks(6, cfg["vocab"], 500 + seed)}
    ragged_batch(cfg, w, d, reqs, 5, 256)


def ragged_batch(cfg, w, d, reqs, n_dec, max_tokens):
    steps = [{"entries": [{"id": k, "tokens": r[:-n_dec], "want": list(range(len(r) - n_dec))} for k, r in reqs.items()]}]
    for j in range(n_dec):
        steps.append({"entries": [{"id": k, "tokens": [r[len(r) - n_dec + j]], "want": [0]} for k, r in reqs.items()]})
    refs = {k: ref_logits(cfg, w, r) for k, r in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        logits, _ = run_trace(d, steps, dtype=dtype, page=8, max_tokens=max_tokens)
        at, loose = 0, []
        for i, (k, r) in enumerate(reqs.items()):
            n = len(r) - n_dec
            got = np.concatenate([logits[0][at:at + n]] + [logits[1 + j][i:i + 1] for j in range(n_dec)])
            at += n
            if dtype == "float32":
                assert_rows(got, refs[k])
            else:
                loose.append(row_errors(got, refs[k]))
        if loose:
            err = np.concatenate(loose)
            assert np.median(err) < TOL16 and (err > 4 * TOL16).mean() <= 0.03, np.sort(err)[-5:]


def test_a_mid_sized_model(tmp_path):
    """Sizes between the toy models above and a real one: every product past one tile, heads on the tensor-core sizes, a
    ragged batch decoded together."""
    layers = [(SINK(heads=8, kv_heads=4, dim=48, vdim=40, rot_dims=32, scale=0.14), (520, 1.5)),
              (PAR(CHUNK(heads=8, kv_heads=2, dim=40, vdim=56, chunk=100, rot_dims=24), RET(heads=4, dim=72, vdim=96, rot_dims=48)), (392, 1.0)),
              (LAT(heads=5, dim=48, rot_dim=16, vdim=32, kv_rank=104, window=100, base=1e5), None), 1,
              (PAR(CHUNK(heads=4, kv_heads=1, dim=64, vdim=112, chunk=250), RET(heads=6, dim=32, vdim=64)), (520, 1.0)), 0]
    cfg = mo.make_config(width=384, vocab=500, layers=layers, eps=2e-5, buckets=777)
    w = mo.make_weights(cfg, seed=123)
    d = write_model(tmp_path, cfg, w)
    reqs = {"a": toks(330, cfg["vocab"], 124), "b": toks(70, cfg["vocab"], 125), "c": toks(9, cfg["vocab"], 126)}
    ragged_batch(cfg, w, d, reqs, 6, 1024)


def test_greedy_generation_through_the_scheduler(base):
    from kuiperllama_b200 import build
    cfg, w, d = base
    tools = build.build_seq_tools()
    prompts = [toks(9, cfg["vocab"], 71), toks(30, cfg["vocab"], 72), toks(2, cfg["vocab"], 73)]
    cmd = [str(tools / "kuiper_generate"), "--model", str(d), "--dtype", "float32", "--new", "12", "--page", "8"]
    for p in prompts:
        cmd += ["--prompt", " ".join(map(str, p))]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [[int(x) for x in ln.split()] for ln in r.stdout.strip().splitlines()]
    for p, g in zip(prompts, got):
        assert g == mo.greedy(cfg, w, p, 12)


def test_tensors_of_the_wrong_shape_are_reported(base, tmp_path):
    from kuiperllama_b200 import build
    cfg, w, _ = base
    for name in ("l0.mix.q", "l1.mix.left.g", "l1.mix.right.v", "l1.mix.left.k.norm", "l2.mix.dkv", "l0.mlp.up.b", "bigram"):
        w2 = dict(w)
        w2[name] = w[name][:-1]
        d = write_model(tmp_path / name, cfg, w2)
        r = subprocess.run([str(build.build_seq_tools() / "kuiper_trace"), "--model", str(d), "--out", str(tmp_path), "--dtype",
                            "float32"], capture_output=True, text=True)
        assert r.returncode == 2 and name.split(".")[0] in r.stderr, (name, r.stderr)


def test_many_heads_in_single_token_steps(tmp_path):
    """More heads than a CTA has warps for: the kernels of single-token steps walk them in turns."""
    layers = [(PAR(CHUNK(heads=40, kv_heads=5, dim=8, vdim=6, chunk=12), RET(heads=37, dim=4, vdim=5, rot_dims=4)), None),
              (SINK(heads=36, kv_heads=6, dim=4, vdim=3, rot_dims=4), None)]
    cfg = mo.make_config(width=32, vocab=40, layers=layers)
    w = mo.make_weights(cfg, seed=77, sharp=2.0)
    d = write_model(tmp_path, cfg, w)
    t = toks(30, cfg["vocab"], 78)
    logits, _ = run_trace(d, [whole("a", t[:10], end=False)] + single("a", t[10:]))
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))
