"""Bifazen through the product path (bin/trace_run -> registry -> BatchScheduler -> sequence-batch engine and its
kernels) against the plain float64 restatement in tests/bifazen_oracle.py.  Small random models with bf16-representable
weights; --dtype float32 is compared tightly, bfloat16 loosely."""
import subprocess

import numpy as np
import pytest

import bifazen_oracle as bo
from seq_util import rel_err, run_trace, whole

pytestmark = pytest.mark.gpu
TOL32 = 1e-4   # fp32 kernels against float64: rounding only (a lost key, stream or blend costs > 1e-2)
TOL16 = 4e-2   # bf16 products


def toks(n, vocab, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def ref_logits(cfg, w, tokens):
    return bo.forward(cfg, w, tokens)[0]


def single(rid, tokens, end=False):
    """One step per token."""
    steps = [{"entries": [{"id": rid, "tokens": [x], "want": [0]}]} for x in tokens]
    if end and steps:
        steps[-1]["end"] = [rid]
    return steps


def row_errors(got, ref):
    return np.array([rel_err(got[i:i + 1], ref[i:i + 1]) for i in range(len(ref))])


def assert_rows(got, ref, tol=TOL32):
    err = row_errors(got, ref)
    assert err.max() < tol, f"first bad position {int(np.argmax(err >= tol))} of {len(ref)}, worst {err.max():.3g}"


@pytest.fixture(scope="module")
def base(tmp_path_factory):
    """Both kinds of layer, with sizes that differ wherever they can: query and key/value heads, key and value sizes,
    latent ranks, windows that are no multiple of a key tile or a page, with and without a feed-forward; three layers
    that blend their values (not next to one another) and one attention that does not."""
    layers = [(bo.latent_mixer(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, window=21), 40),
              (bo.plain_mixer(heads=4, kv_heads=2, dim=12, vdim=10, window=19), 56),
              (bo.latent_mixer(heads=2, dim=8, rot_dim=8, vdim=12, kv_rank=36, window=33, base=50.0), None),
              (bo.plain_mixer(heads=6, kv_heads=2, dim=6, vdim=10, window=9), None),
              (bo.plain_mixer(heads=3, kv_heads=3, dim=8, vdim=5, window=13, v_mix=False), 24),
              (bo.plain_mixer(heads=4, kv_heads=4, dim=5, vdim=5, window=27), 24)]
    cfg = bo.make_config(width=48, vocab=61, layers=layers, streams=3)
    w = bo.make_weights(cfg, seed=1, sharp=3.0)
    return cfg, w, bo.write_model(tmp_path_factory.mktemp("bifa_base"), cfg, w)


# ---- every mechanism on its own -------------------------------------------------------------------------------------
LAT, ATT = bo.latent_mixer, bo.plain_mixer
CASES = {  # layers, streams
    "latent": ([(LAT(), None)], 2),
    "latent_one_head": ([(LAT(heads=1), None)], 2),
    "latent_window_one": ([(LAT(window=1), None)], 2),
    "latent_window_past_the_prompt": ([(LAT(window=500), None)], 2),
    "latent_no_window": ([(LAT(window=0), None)], 2),
    "latent_partly_rotated": ([(LAT(rot_dim=8, rot_dims=4), None)], 2),
    "latent_slow_rotation": ([(LAT(rot_dim=8, base=5e5), None)], 2),
    "latent_two_rotated": ([(LAT(rot_dim=2, base=7.0), None)], 2),
    "latent_rank_past_a_key_tile": ([(LAT(heads=2, kv_rank=136, dim=24, rot_dim=16, vdim=72), None)], 2),
    "latent_rank_beyond_the_tiles": ([(LAT(heads=2, kv_rank=300, dim=12, rot_dim=4, vdim=9, window=40), None)], 2),
    "latent_rank_smaller_than_a_head": ([(LAT(kv_rank=3, dim=12), None)], 2),
    "latent_scaled": ([(LAT(scale=0.9), None)], 2),
    "attention": ([(ATT(v_mix=False), None)], 2),
    "attention_one_key_head": ([(ATT(heads=4, kv_heads=1, dim=16, vdim=6), None)], 2),
    "attention_every_head_its_keys": ([(ATT(heads=3, kv_heads=3), None)], 2),
    "attention_one_head": ([(ATT(heads=1, kv_heads=1), None)], 2),
    "attention_window_one": ([(ATT(window=1), None)], 2),
    "attention_no_window": ([(ATT(window=0), None)], 2),
    "attention_wide": ([(ATT(heads=2, kv_heads=1, dim=136, vdim=72, window=40), None)], 2),
    "attention_values_beyond_the_tiles": ([(ATT(heads=2, kv_heads=1, dim=8, vdim=260, window=40), None)], 2),
    "attention_keys_beyond_the_tiles": ([(ATT(heads=4, kv_heads=2, dim=520, vdim=6, window=40), None)], 2),
    "blend": ([(ATT(), None), (ATT(heads=2, kv_heads=1, vdim=20), None), (ATT(heads=4, kv_heads=4, vdim=5), None)], 2),
    "blend_over_a_gap": ([(LAT(), None), (ATT(), 20), (ATT(v_mix=False, vdim=7), None), (LAT(), None), (ATT(), None)], 2),
    "one_stream": ([(LAT(), 20), (ATT(), 20)], 1),
    "four_streams": ([(LAT(), 20), (ATT(), None)], 4),
    "five_streams": ([(ATT(), None), (LAT(), 20)], 5),
    "eight_streams": ([(LAT(), 20), (ATT(), 20)], 8),
    "eleven_streams": ([(ATT(), 20), (LAT(), None)], 11),
    "ff_only": ([(LAT(), 30)], 2),
    "ff_past_a_block": ([(ATT(), 136)], 2),
}


@pytest.mark.parametrize("case", sorted(CASES))
def test_mechanism_alone(tmp_path, case):
    layers, streams = CASES[case]
    # a large eps in some cases: it must reach every norm (the layers', the latent's, the whole projections')
    big_eps = case in ("latent", "attention", "ff_only", "four_streams")
    cfg = bo.make_config(width=40, vocab=50, layers=layers, eps=0.05 if big_eps else 3e-6, streams=streams)
    w = bo.make_weights(cfg, seed=3, sharp=3.0)
    if case == "ff_only":  # the mixer's output projection is zero: what is left of the layer is the feed-forward
        w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    if case == "blend":  # nothing of a layer's own values, and more than all of the first layer's
        w["l1.mix.vmix"], w["l2.mix.vmix"] = np.float64(1.0), np.float64(1.5)
        w["l0.mix.vmix"] = np.float64(77.0)   # the first blending layer does not read its own
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(75, cfg["vocab"], 5)
    ref, trace = bo.forward(cfg, w, t)
    logits, resid = run_trace(d, [whole("a", t)], residual=True)
    got = resid[0].reshape(trace.shape)
    assert np.abs(got - trace).max() < 1e-4 * max(1.0, np.abs(trace).max())
    assert_rows(logits[0], ref)
    # without the residual trace (the last boundary then runs on the wanted rows only), and decoded
    logits, _ = run_trace(d, [whole("b", t[:70], want=[0, 3, 64, 69], end=False)] + single("b", t[70:]))
    assert_rows(np.concatenate(logits), ref[[0, 3, 64, 69, 70, 71, 72, 73, 74]])


def test_residual_after_every_layer(base):
    cfg, w, d = base
    t = toks(33, cfg["vocab"], 7)
    _, trace = bo.forward(cfg, w, t)
    assert trace.shape[0] == 6
    _, resid = run_trace(d, [whole("a", t)], residual=True)
    got = resid[0].reshape(trace.shape)
    for r in range(trace.shape[0]):
        assert np.abs(got[r] - trace[r]).max() < 1e-4 * max(1.0, np.abs(trace[r]).max()), f"layer {r}"


def test_streams_are_mixed_from_rows_to_columns(tmp_path):
    """A mix matrix that moves stream 0 into stream 2 and forgets the rest, and a next sublayer that reads stream 2 only:
    the transposed matrix, or streams updated one after the other, would read something else entirely."""
    cfg = bo.make_config(width=24, vocab=30, layers=[(LAT(), None), (ATT(), None)], streams=3)
    w = bo.make_weights(cfg, seed=8)
    w["l0.hc1.in"] = np.array([0.25, 0.5, -0.5])
    w["l0.hc1.mix"] = np.array([[0.0, 0.0, 2.0], [1.0, 0.0, 0.0], [0.0, 1.0, 0.0]])
    w["l0.hc1.out"] = np.array([0.0, 4.0, 0.5])
    w["l1.hc1.in"] = np.array([0.0, 0.0, 1.0])
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(20, cfg["vocab"], 9)
    ref = ref_logits(cfg, w, t)
    w2 = dict(w)
    w2["l0.hc1.mix"] = w["l0.hc1.mix"].T.copy()
    assert rel_err(ref_logits(cfg, w2, t), ref) > 0.1  # the construction works
    logits, _ = run_trace(d, [whole("a", t[:15], end=False)] + single("a", t[15:]))
    assert_rows(np.concatenate(logits), ref)


@pytest.mark.parametrize("order", ["AL", "LLA", "ALAAL"])
def test_layer_orders(tmp_path, order):
    """Any order of the two kinds of layer; every layer has a cache of its own."""
    layers = [((ATT(window=9) if c == "A" else LAT(window=7)), 24 if i % 2 else None) for i, c in enumerate(order)]
    cfg = bo.make_config(width=40, vocab=60, layers=layers)
    w = bo.make_weights(cfg, seed=101, sharp=2.0)
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(45, cfg["vocab"], 102)
    logits, _ = run_trace(d, [whole("a", t[:30], end=False)] + single("a", t[30:]))
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


def test_a_plain_residual_when_there_are_no_streams(tmp_path):
    """Without "streams" the model has one plain residual: the same layers through the engine's other norm kernel."""
    cfg = bo.make_config(width=40, vocab=60, layers=[(LAT(), 24), (ATT(), None)], streams=1)
    w = bo.make_weights(cfg, seed=103)
    for k in list(w):
        if ".hc" in k:
            w[k] = np.ones_like(w[k])   # one stream, all coefficients one: x + sublayer(x)
    t = toks(40, cfg["vocab"], 104)
    ref = ref_logits(cfg, w, t)
    plain = {k: v for k, v in cfg.items() if k != "streams"}
    d = bo.write_model(tmp_path, plain, {k: v for k, v in w.items() if ".hc" not in k})
    logits, _ = run_trace(d, [whole("a", t[:30], end=False)] + single("a", t[30:]))
    assert_rows(np.concatenate(logits), ref)


@pytest.mark.parametrize("page", [4, 16, 64])
def test_long_prompt_every_position(base, page):
    cfg, w, d = base
    t = toks(203, cfg["vocab"], 11)  # past three key tiles of 64, no multiple of a page
    logits, _ = run_trace(d, [whole("a", t)], page=page)
    assert_rows(logits[0], ref_logits(cfg, w, t))


# ---- keys at the edge of the window ---------------------------------------------------------------------------------
def edge_model(kind, window, special, vocab=30, width=24, seed=9):
    """One attention layer, made so that ONE token's key wins every softmax it takes part in.  Input coordinate 1 is the
    same for every token and feeds the last unrotated coordinate of every query head; input coordinate 0 is zero except
    for the special token and feeds the same coordinate of the keys (by way of latent coordinate 0), and nothing else
    does.  While the special key is seen, a head's output is (almost) that token's value."""
    if kind == "latent":
        m = bo.latent_mixer(heads=2, dim=8, rot_dim=4, vdim=6, kv_rank=10, window=window, scale=3.0)
    else:
        m = bo.plain_mixer(heads=2, kv_heads=1, dim=8, vdim=6, window=window, scale=3.0)
    cfg = bo.make_config(width=width, vocab=vocab, layers=[(m, None)], streams=2)
    w = bo.make_weights(cfg, seed=seed)
    p = "l0.mix."
    w["l0.norm1"][:] = 0.0
    w["l0.hc1.in"] = np.array([0.75, 0.5])
    w["embed"][:, 0] = 0.0
    w["embed"][special, 0] = 8.0
    w["embed"][:, 1] = 2.0
    per = 12 if kind == "latent" else 8   # query rows of a head
    w[p + "q"] = bo.bf16_round(w[p + "q"] * 0.05)
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
        for n in ("q.b", "k.b"):
            w[p + n][:] = 0.0
        w[p + "q.norm"][:] = 1.0
        w[p + "k.norm"][:] = 1.0
        w[p + "k"][:, :2] = 0.0
        w[p + "k"][7] = 0.0
        w[p + "k"][7, 0] = 2.0
    return cfg, w


@pytest.mark.parametrize("kind", ["latent", "plain"])
@pytest.mark.parametrize("window", [2, 17, 64, 65, 100])
def test_the_key_at_the_window_edge_carries_the_output(tmp_path, kind, window):
    """The special key is placed so that it leaves the window inside the prompt, and a second one so that it leaves
    while tokens are decoded one by one (across key tiles and pages).  The last position that still sees it depends on
    it heavily; the next one does not depend on it at all."""
    special = 7
    cfg, w = edge_model(kind, window, special)
    n_prompt, n_all = 150, 150 + window + 20
    t = [x if x != special else special + 1 for x in toks(n_all, cfg["vocab"], 13)]
    places = (20, n_prompt - 5)  # leaves the window inside the prompt / during decoding
    for p in places:
        t[p] = special
    ref = ref_logits(cfg, w, t)
    for p in places:  # the construction works
        t2 = list(t)
        t2[p] = special + 1
        other = ref_logits(cfg, w, t2)
        assert rel_err(other[p + window - 1:p + window], ref[p + window - 1:p + window]) > 0.1
        assert rel_err(other[p + window:p + window + 1], ref[p + window:p + window + 1]) < 1e-9
    d = bo.write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("a", t[:n_prompt], end=False)] + single("a", t[n_prompt:]), page=16)
    assert_rows(np.concatenate(logits), ref)
    lb, _ = run_trace(d, [whole("a", t[:n_prompt], end=False)] + single("a", t[n_prompt:]), page=16, dtype="bfloat16")
    assert rel_err(np.concatenate(lb), ref) < TOL16


@pytest.mark.parametrize("kind", ["latent", "plain"])
def test_the_first_token_leaves_with_the_window(tmp_path, kind):
    """Nothing keeps the first tokens: position 0 is gone once the window has passed."""
    special, window = 7, 12
    cfg, w = edge_model(kind, window, special)
    t = [x if x != special else special + 1 for x in toks(40, cfg["vocab"], 14)]
    t[0] = special
    ref = ref_logits(cfg, w, t)
    t2 = [special + 1] + t[1:]
    other = ref_logits(cfg, w, t2)
    assert rel_err(other[window - 1:window], ref[window - 1:window]) > 0.1 and rel_err(other[window:], ref[window:]) < 1e-9
    d = bo.write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, single("a", t) + [whole("b", t)], page=8)
    assert_rows(np.concatenate(logits[:40]), ref)
    assert_rows(logits[40], ref)


@pytest.mark.parametrize("kind", ["latent", "plain"])
def test_a_far_key_without_a_window(tmp_path, kind):
    """One key among hundreds, far back, carries the output at the end of the prompt and while decoding."""
    special = 7
    cfg, w = edge_model(kind, 0, special)
    t = [x if x != special else special + 1 for x in toks(420, cfg["vocab"], 16)]
    t[3] = special
    ref = ref_logits(cfg, w, t)
    t2 = list(t)
    t2[3] = special + 1
    assert rel_err(ref_logits(cfg, w, t2)[-1:], ref[-1:]) > 0.1
    d = bo.write_model(tmp_path, cfg, w)
    for dtype, tol in (("float32", TOL32), ("bfloat16", TOL16)):
        logits, _ = run_trace(d, [whole("a", t[:400], end=False)] + single("a", t[400:]), dtype=dtype)
        assert rel_err(np.concatenate(logits), ref) < tol


def test_the_rotation_is_seen_at_far_positions(tmp_path):
    """Scores from the rotated part alone, sharpened, at positions in the hundreds: a wrong pairing, base or position
    changes which keys win."""
    cfg = bo.make_config(width=32, vocab=40, layers=[(LAT(heads=2, dim=4, rot_dim=16, kv_rank=12, window=90, base=5e5), None)])
    w = bo.make_weights(cfg, seed=18)
    for head in range(2):
        w["l0.mix.q"][head * 20:head * 20 + 4] = 0.0
        w["l0.mix.q"][head * 20 + 4:head * 20 + 20] *= 4.0
    t = toks(330, cfg["vocab"], 19)
    ref = ref_logits(cfg, w, t)
    d = bo.write_model(tmp_path, cfg, w)
    logits, _ = run_trace(d, [whole("a", t[:300], end=False)] + single("a", t[300:]))
    assert_rows(np.concatenate(logits), ref)


# ---- prompt against token-by-token decoding, long decoding ----------------------------------------------------------
def test_prefill_equals_stepwise_decoding(base):
    cfg, w, d = base
    t = toks(90, cfg["vocab"], 17)
    ref = ref_logits(cfg, w, t)
    split = [whole("p", t[:2], end=False)] + single("p", t[2:])
    logits, _ = run_trace(d, single("s", t) + split, page=8)   # "s": from the very first token
    a, b = np.concatenate(logits[:len(t)]), np.concatenate(logits[len(t):])
    assert_rows(a, ref)
    assert_rows(b, ref)
    assert_rows(a, b)


def test_long_decoding(base):
    """Decoding far past every window, key tile and page."""
    cfg, w, d = base
    t = toks(40 + 260, cfg["vocab"], 19)
    logits, _ = run_trace(d, [whole("a", t[:40], end=False)] + single("a", t[40:]), page=16)
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))


@pytest.mark.parametrize("dtype,tol", [("float32", TOL32), ("bfloat16", TOL16)])
@pytest.mark.parametrize("sizes", [(2, 2, 2, 2), (5, 64, 3, 17), (33, 2, 70), (1, 99, 2), (1, 1, 2, 1, 40, 1, 2)])
def test_prompt_in_portions(base, tmp_path, sizes, dtype, tol):
    """A prompt fed in several steps: every portion starts from the cache that the portions before it left.  A second
    request of another length rides along."""
    cfg, w, d = base
    if dtype == "bfloat16":  # softmaxes that are not sharpened: a peaky one amplifies the rounding of its scores
        w = bo.make_weights(cfg, seed=1)
        d = bo.write_model(tmp_path, cfg, w)
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
    assert_rows(got_p, ref_logits(cfg, w, t), tol)
    assert_rows(got_o, ref_logits(cfg, w, other), tol)


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
    at = 0
    for t in reqs:
        assert_rows(np.concatenate(logits[at:at + 4]), ref_logits(cfg, w, t))
        at += 4


def test_a_freed_slot_starts_afresh(base):
    """Two slots; requests come and go in an order that hands a slot with a long history to a request that starts by
    decoding from its first token."""
    cfg, w, d = base
    a, b, c = toks(80, cfg["vocab"], 61), toks(12, cfg["vocab"], 62), toks(9, cfg["vocab"], 63)
    steps = [{"entries": [{"id": "a", "tokens": a, "want": [79]}, {"id": "b", "tokens": b[:6], "want": [5]}], "end": ["a"]}]
    for j in range(6):  # c takes a's slot and decodes from its first token beside b
        steps.append({"entries": [{"id": "b", "tokens": [b[6 + j]], "want": [0]}, {"id": "c", "tokens": [c[j]], "want": [0]}]})
    logits, _ = run_trace(d, steps, max_tokens=128, extra=["--max-seqs", "2"])
    got_b = np.concatenate([logits[0][1:2]] + [lg[0:1] for lg in logits[1:]])
    got_c = np.concatenate([lg[1:2] for lg in logits[1:]])
    assert_rows(got_b, ref_logits(cfg, w, b)[5:])
    assert_rows(got_c, ref_logits(cfg, w, c)[:6])
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
        got = np.stack([logits[0][i], logits[1][i], logits[2][i]])
        assert_rows(got, ref_logits(cfg, w, r)[-3:])


# ---- bf16, other sizes, generation ------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind,dim,vdim,window", [("latent", 24, 40, 17), ("latent", 48, 128, 64), ("latent", 96, 64, 150),
                                                  ("latent", 200, 72, 0), ("latent", 20, 24, 30), ("plain", 24, 24, 17),
                                                  ("plain", 64, 128, 64), ("plain", 128, 64, 150), ("plain", 40, 200, 40)])
def test_bfloat16_prompts_on_the_tensor_cores(tmp_path, kind, dim, vdim, window):
    """bf16 prompt steps with head sizes that are multiples of 8 take the tensor-core attention (latents expanded into
    per-head keys and values in one product): against the float64 restatement, and against single-token steps of the same
    run.  A latent head of 20 and values of 200 fall back to the split-key kernel."""
    if kind == "latent":
        layers = [(LAT(heads=4, dim=dim, rot_dim=16, vdim=vdim, kv_rank=56, window=window), 136)]
    else:
        layers = [(ATT(heads=6, kv_heads=2, dim=dim, vdim=vdim, window=window), 136), (ATT(heads=4, kv_heads=2, dim=dim, vdim=vdim, window=window), None)]
    cfg = bo.make_config(width=64, vocab=80, layers=layers, streams=4)
    w = bo.make_weights(cfg, seed=41, sharp=1.5)
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(260, cfg["vocab"], 42)
    ref = ref_logits(cfg, w, t)
    steps = [whole("a", t, end=True), whole("b", t[:200], end=False)] + single("b", t[200:])
    logits, _ = run_trace(d, steps, dtype="bfloat16")
    assert rel_err(logits[0], ref) < TOL16
    assert rel_err(np.concatenate(logits[1:]), ref) < TOL16
    assert rel_err(np.concatenate(logits[2:]), logits[0][200:]) < TOL16


@pytest.mark.parametrize("dtype,tol", [("float32", TOL32), ("bfloat16", TOL16)])
def test_sizes_that_fit_no_vector(tmp_path, dtype, tol):
    """Odd sizes everywhere: no 16-byte vector load, no tensor-core tile and no warp-sized loop fits."""
    layers = [(LAT(heads=3, dim=5, rot_dim=2, vdim=3, kv_rank=11, window=7), 11),
              (ATT(heads=3, kv_heads=1, dim=7, vdim=5, window=13), 9),
              (LAT(heads=1, dim=1, rot_dim=6, vdim=13, kv_rank=5, window=3), None),
              (ATT(heads=5, kv_heads=5, dim=3, vdim=1, window=4), 7)]
    cfg = bo.make_config(width=22, vocab=23, layers=layers[:2] + [layers[2]], streams=3)
    w = bo.make_weights(cfg, seed=51)
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(77, cfg["vocab"], 52)
    logits, _ = run_trace(d, [whole("a", t[:70], end=False)] + single("a", t[70:]), dtype=dtype)
    err = row_errors(np.concatenate(logits), ref_logits(cfg, w, t))
    assert err.max() < tol if dtype == "float32" else (np.median(err) < tol / 2 and (err > tol).mean() <= 0.05), np.sort(err)[-5:]
    cfg = bo.make_config(width=21, vocab=23, layers=[layers[0], layers[3]], streams=7)  # a width of no even divisor
    w = bo.make_weights(cfg, seed=53)
    d = bo.write_model(tmp_path / "b", cfg, w)
    logits, _ = run_trace(d, [whole("a", t[:70], end=False)] + single("a", t[70:]), dtype=dtype)
    err = row_errors(np.concatenate(logits), ref_logits(cfg, w, t))
    assert err.max() < tol if dtype == "float32" else (np.median(err) < tol / 2 and (err > tol).mean() <= 0.05), np.sort(err)[-5:]


def random_design(seed):
    rng = np.random.default_rng(seed)

    def pick(*xs):
        return xs[int(rng.integers(len(xs)))]

    values = pick(6, 12)   # kv_heads * vdim of the layers that blend

    def mixer():
        if pick("latent", "plain") == "latent":
            return LAT(heads=pick(1, 2, 5), dim=pick(3, 8, 16), rot_dim=pick(2, 8), vdim=pick(3, 8, 16), kv_rank=pick(4, 16, 70),
                       window=pick(1, 5, 30, 66), base=pick(100.0, 10000.0, 5e5))
        g = pick(1, 2, 3)
        mix = pick(True, True, False)
        return ATT(heads=g * pick(1, 2, 4), kv_heads=g, dim=pick(4, 8, 12), vdim=values // g if mix else pick(3, 8, 16),
                   window=pick(1, 5, 30, 66), v_mix=mix)

    layers = [(mixer(), pick(None, 8, 30)) for _ in range(int(rng.integers(2, 7)))]
    return bo.make_config(width=pick(16, 24, 40), vocab=pick(17, 50), layers=layers, eps=pick(1e-6, 1e-3), streams=pick(1, 2, 3, 4, 6))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_random_designs(tmp_path, seed):
    """Layer order, sizes and constants drawn at random; a ragged batch that is prefilled together and decoded together,
    in float32 (tight) and bfloat16 (loose)."""
    cfg = random_design(seed)
    w = bo.make_weights(cfg, seed=100 + seed, sharp=1.5)
    d = bo.write_model(tmp_path, cfg, w)
    reqs = {"a": toks(90, cfg["vocab"], 300 + seed), "b": toks(23, cfg["vocab"], 400 + seed), "c": toks(6, cfg["vocab"], 500 + seed)}
    n_dec = 5
    steps = [{"entries": [{"id": k, "tokens": r[:-n_dec], "want": list(range(len(r) - n_dec))} for k, r in reqs.items()]}]
    for j in range(n_dec):
        steps.append({"entries": [{"id": k, "tokens": [r[len(r) - n_dec + j]], "want": [0]} for k, r in reqs.items()]})
    refs = {k: ref_logits(cfg, w, r) for k, r in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        logits, _ = run_trace(d, steps, dtype=dtype, page=8, max_tokens=256)
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
            assert np.median(err) < TOL16 / 2 and (err > 2 * TOL16).mean() <= 0.02, np.sort(err)[-5:]


def test_a_mid_sized_model(tmp_path):
    """Sizes between the toy models above and a real one: every product past one tile, heads on the tensor-core sizes, a
    ragged batch decoded together -- float32 tight, bfloat16 loose."""
    layers = [(LAT(heads=5, dim=48, rot_dim=16, vdim=32, kv_rank=96, window=100, base=1e5), 520),
              (ATT(heads=8, kv_heads=2, dim=40, vdim=56, window=60), 392),
              (LAT(heads=4, dim=32, rot_dim=32, vdim=64, kv_rank=160, window=250), None),
              (ATT(heads=4, kv_heads=1, dim=64, vdim=112, window=200), 520)]
    cfg = bo.make_config(width=384, vocab=500, layers=layers, eps=2e-5, streams=4)
    w = bo.make_weights(cfg, seed=123)
    d = bo.write_model(tmp_path, cfg, w)
    reqs = {"a": toks(330, cfg["vocab"], 124), "b": toks(70, cfg["vocab"], 125), "c": toks(9, cfg["vocab"], 126)}
    n_dec = 6
    steps = [{"entries": [{"id": k, "tokens": r[:-n_dec], "want": list(range(len(r) - n_dec))} for k, r in reqs.items()]}]
    for j in range(n_dec):
        steps.append({"entries": [{"id": k, "tokens": [r[len(r) - n_dec + j]], "want": [0]} for k, r in reqs.items()]})
    refs = {k: ref_logits(cfg, w, r) for k, r in reqs.items()}
    for dtype, tol in (("float32", TOL32), ("bfloat16", TOL16)):
        logits, _ = run_trace(d, steps, dtype=dtype, max_tokens=1024)
        at = 0
        for i, (k, r) in enumerate(reqs.items()):
            n = len(r) - n_dec
            got = np.concatenate([logits[0][at:at + n]] + [logits[1 + j][i:i + 1] for j in range(n_dec)])
            at += n
            assert rel_err(got, refs[k]) < tol, k


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
        assert g == bo.greedy(cfg, w, p, 12)


def test_tensors_of_the_wrong_shape_are_reported(base, tmp_path):
    from kuiperllama_b200 import build
    cfg, w, _ = base
    for name in ("l1.mix.q", "l0.mix.dkv", "l3.mix.v.b", "l0.hc2.in", "l1.mix.q.norm", "l0.mlp.gate"):
        w2 = dict(w)
        w2[name] = w[name][:-1]
        d = bo.write_model(tmp_path / name, cfg, w2)
        r = subprocess.run([str(build.build_seq_tools() / "kuiper_trace"), "--model", str(d), "--out", str(tmp_path), "--dtype",
                            "float32"], capture_output=True, text=True)
        assert r.returncode == 2 and name.split(".")[0] + "." in r.stderr, (name, r.stderr)


def test_many_heads_in_single_token_steps(tmp_path):
    """More query and key heads than a CTA has warps for: the preparation of single-token steps walks them in turns."""
    layers = [(ATT(heads=40, kv_heads=5, dim=8, vdim=6, window=12), None), (LAT(heads=36, dim=4, rot_dim=2, vdim=4, kv_rank=16), None)]
    cfg = bo.make_config(width=32, vocab=40, layers=layers)
    w = bo.make_weights(cfg, seed=77, sharp=2.0)
    d = bo.write_model(tmp_path, cfg, w)
    t = toks(30, cfg["vocab"], 78)
    logits, _ = run_trace(d, [whole("a", t[:10], end=False)] + single("a", t[10:]))
    assert_rows(np.concatenate(logits), ref_logits(cfg, w, t))
