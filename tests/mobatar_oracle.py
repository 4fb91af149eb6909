"""A slow float64 restatement of the Mobatar family, one function per mechanism.

It shares no code with the product path: numpy only, whole sequences, no cache and no state (every function sees the
complete sequence).  `weights` maps tensor names to float64 arrays; `config` is the parsed config.json.

    tokens --embed + bigram rows--> x --> layers --> centred RMS norm --> head

    layer:     x += N1(mixer(x)), then x += N2(ff(x)); the sublayers read x itself
    mixers:    'attention'         (rotation with frequencies divided band by band, unit norms after it, one more term in
                                    the softmax denominator)
               'latent_attention'  (keys and values through a low-rank latent, one rotated key part for all heads, a window)
               'parallel'          (a chunked attention and a retention on the same rows, summed with a weight each)
    ff:        down(act(gate x, up x)), a clamped gate, a bias in every product
"""
from __future__ import annotations

import math

import numpy as np


# ---- small pieces ------------------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def bigram_rows(tokens, b):
    """The bigram table's row of every token; the row behind the hashed ones for the first."""
    return [b["buckets"] if t == 0 else (int(tokens[t - 1]) * b["mul_prev"] + int(tokens[t]) * b["mul_cur"]) % b["buckets"]
            for t in range(len(tokens))]


def frequencies(rot):
    """Angle per position of every rotated pair."""
    f = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    sc = rot.get("scaling")
    if not sc:
        return np.array(f)
    if "original" not in sc:
        return np.array(f) / sc["factor"]
    out = []
    for v in f:
        wavelength = 2.0 * math.pi / v
        if wavelength < sc["original"] / sc["high"]:
            out.append(v)
        elif wavelength > sc["original"] / sc["low"]:
            out.append(v / sc["factor"])
        else:
            s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * v / sc["factor"] + s * v)
    return np.array(out)


def rotate(v, rot, neighbours=False):
    """v [T, ..., n]: the first rot.dims coordinates turn in pairs, (i, i + dims/2) or (2i, 2i + 1)."""
    T, n = v.shape[0], rot["dims"] // 2
    out = v.copy()
    for i, f in enumerate(frequencies(rot)):
        a = (np.arange(T) * f).reshape((T,) + (1,) * (v.ndim - 2))
        one, two = (2 * i, 2 * i + 1) if neighbours else (i, i + n)
        x, y = v[..., one], v[..., two]
        out[..., one] = x * np.cos(a) - y * np.sin(a)
        out[..., two] = y * np.cos(a) + x * np.sin(a)
    return out


def causal_mask(T):
    return np.tril(np.ones((T, T), dtype=bool))


def window_mask(T, window):
    """mask[i, j]: does position i see position j?"""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < window)


def chunk_mask(T, size):
    c = np.arange(T) // size
    return causal_mask(T) & (c[:, None] == c[None, :])


def softmax_rows(s, mask, extra=0.0):
    """Weights over the visible keys; `extra` = 1 adds a term exp(0) without a value to the denominator."""
    s = np.where(mask, s, -np.inf)
    top = np.maximum(s.max(-1, keepdims=True), 0.0) if extra else s.max(-1, keepdims=True)
    p = np.exp(s - top)
    return p / (p.sum(-1, keepdims=True) + extra * np.exp(-top))


# ---- mixers ------------------------------------------------------------------------------------------------------------
def grouped_softmax(q, k, v, mask, scale, extra=0.0):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_rows(q[:, h] @ k[:, g].T * scale, mask, extra) @ v[:, g]
    return out


def sink_attention(h, w, p, m, eps):
    T, H, G, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(rotate((h @ w[p + "q"].T).reshape(T, H, dim), m["rot"]), eps)
    k = rms_unit(rotate((h @ w[p + "k"].T).reshape(T, G, dim), m["rot"]), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, vd)
    return grouped_softmax(q, k, v, causal_mask(T), m["scale"], extra=1.0).reshape(T, H * vd) @ w[p + "o"].T


def chunk_attention(h, w, p, m, eps):
    T, H, G, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms_unit(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).reshape(T, H, dim)
    k = (rms_unit(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).reshape(T, G, dim)
    v = (h @ w[p + "v"].T).reshape(T, G, vd)
    o = grouped_softmax(rotate(q, m["rot"]), rotate(k, m["rot"]), v, chunk_mask(T, m["mask"]["size"]), m["scale"])
    return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * vd) @ w[p + "o"].T


def retention(h, w, p, m, eps):
    """The recurrence token by token, from a zero state."""
    T, H, dim, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + "q"].T).reshape(T, H, dim), m["rot"])
    k = rotate((h @ w[p + "k"].T).reshape(T, H, dim), m["rot"]) * dim ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, vd)
    decay = np.asarray(m["decay"], dtype=np.float64)
    S, o = np.zeros((H, dim, vd)), np.zeros((T, H, vd))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return (rms_unit(o, eps).reshape(T, H * vd) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return m["left_scale"] * chunk_attention(h, w, p + "left.", m["left"], eps) \
        + m["right_scale"] * retention(h, w, p + "right.", m["right"], eps)


def latent_attention(h, w, p, m, eps):
    T, H, dim, rd, vd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim + rd)
    down = h @ w[p + "dkv"].T
    c = rms_unit(down[:, :rank], eps) * w[p + "dkv.norm"]
    k_rot = rotate(down[:, rank:], m["rot"], neighbours=True)
    q_rot = rotate(q[:, :, dim:], m["rot"], neighbours=True)
    k = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    mask = window_mask(T, m["mask"]["size"])
    out = np.zeros((T, H, vd))
    for i in range(H):
        s = (q[:, i, :dim] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = softmax_rows(s, mask) @ v[:, i]
    return out.reshape(T, H * vd) @ w[p + "o"].T


MIXERS = {"attention": sink_attention, "parallel": side_by_side, "latent_attention": latent_attention}


def clamped_ff(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T + w[p + "gate.b"], limit)
    u = np.clip(h @ w[p + "up"].T + w[p + "up.b"], -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T + w[p + "down.b"]


# ---- the model ---------------------------------------------------------------------------------------------------------
def owner(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config, w, tokens):
    """(logits [T, vocab], residual after every layer [layers, T, width])."""
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] + w["bigram"][bigram_rows(tokens, config["embedding"]["bigram"])]
    trace = []
    for i, L in enumerate(config["layers"]):
        p = f"l{owner(config, i)}."
        x = x + centred_norm(MIXERS[L["type"]](x, w, p + "mix.", L["mixer"], eps), w[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + centred_norm(clamped_ff(x, w, p + "mlp.", L["mlp"]["limit"]), w[p + "norm2"], eps)
        trace.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T, np.stack(trace)


def greedy(config, weights, prompt, n_new):
    """n_new greedy tokens after `prompt` (lowest index on ties), recomputing the whole sequence every time."""
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(np.argmax(forward(config, weights, seq)[0][-1])))
    return seq[len(prompt):]


# ---- small configurations and random weights for the tests ---------------------------------------------------------------
def rotation(dims, base=1000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(scaling)
    return r


BANDS = {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 60}


def sink_mixer(heads=4, kv_heads=2, dim=12, vdim=10, rot_dims=8, base=1000.0, scaling=BANDS, scale=0.35):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
            "rot": rotation(rot_dims, base, scaling)}


def chunk_mixer(heads=4, kv_heads=2, dim=10, vdim=6, chunk=13, rot_dims=6, base=300.0, factor=3.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
            "scale": dim ** -0.5 if scale is None else scale, "rot": rotation(rot_dims, base, {"factor": factor})}


def retention_mixer(heads=3, dim=8, vdim=7, rot_dims=6, base=500.0, decay=None):
    if decay is None:
        decay = [(0.9, 0.99, 0.75, 0.998, 1.0)[i % 5] for i in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": rotation(rot_dims, base)}


def parallel_mixer(left=None, right=None, left_scale=0.75, right_scale=1.5):
    return {"left": left or chunk_mixer(), "right": right or retention_mixer(), "left_scale": left_scale,
            "right_scale": right_scale}


def latent_mixer(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, window=14, base=1000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
            "rot": rotation(rot_dim, base), "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}


def make_config(width=48, vocab=61, layers=(), eps=3e-6, buckets=37, mul_prev=11, mul_cur=5):
    """layers: (mixer, (ff size, limit) or None), the mixer's kind read off its keys; or the number of an earlier layer whose
    weights run again."""
    out = []
    for spec in layers:
        if isinstance(spec, int):
            out.append(dict(out[spec], weights_of=spec))
            continue
        mixer, ff = spec
        kind = "latent_attention" if "kv_rank" in mixer else "parallel" if "left" in mixer else "attention"
        out.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff[0], "limit": ff[1]} if ff else None})
    return {"architecture": "Mobatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random bf16-representable weights.  `sharp` multiplies the query weights of the softmax attentions that do not
    unit-norm their queries (the norm weights of those that norm them): > 1 makes the softmax peaky, so that single keys
    (those at an edge too) carry the output."""
    from seq_util import bf16_round
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, std=1.0, mean=0.0):
        return bf16_round(mean + std * rng.standard_normal(shape))

    def fan(rows, cols, gain=1.0):
        return rnd(rows, cols, std=gain * cols ** -0.5)

    w = {"embed": rnd(V, W, std=0.7), "bigram": rnd(cfg["embedding"]["bigram"]["buckets"] + 1, W, std=0.7),
         "final.norm": rnd(W, std=0.2), "head": fan(V, W)}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        w[p + "norm1"] = rnd(W, std=0.2)
        if L["type"] == "latent_attention":
            H = m["heads"]
            w[q + "q"] = fan(H * (m["dim"] + m["rot_dim"]), W, sharp)
            w[q + "dkv"] = fan(m["kv_rank"] + m["rot_dim"], W, 1.5)
            w[q + "dkv.norm"] = rnd(m["kv_rank"], mean=1.0, std=0.2)
            w[q + "uk"] = fan(H * m["dim"], m["kv_rank"], 1.5)
            w[q + "uv"] = fan(H * m["vdim"], m["kv_rank"])
            w[q + "o"] = fan(W, H * m["vdim"])
        else:
            a, r = (m["left"], m["right"]) if L["type"] == "parallel" else (m, None)
            lp = q + "left." if r else q
            H, G = a["heads"], a["kv_heads"]
            w[lp + "q"], w[lp + "k"] = fan(H * a["dim"], W), fan(G * a["dim"], W)
            w[lp + "v"], w[lp + "o"] = fan(G * a["vdim"], W), fan(W, H * a["vdim"])
            if r:
                w[lp + "q.norm"] = rnd(H * a["dim"], mean=sharp, std=0.2 * sharp)
                w[lp + "k.norm"] = rnd(G * a["dim"], mean=1.5, std=0.3)
                w[lp + "g"] = fan(H, W, 2.0)
                rp, R = q + "right.", r["heads"]
                w[rp + "q"], w[rp + "k"] = fan(R * r["dim"], W), fan(R * r["dim"], W)
                w[rp + "v"], w[rp + "g"] = fan(R * r["vdim"], W), fan(R * r["vdim"], W)
                w[rp + "o"] = fan(W, R * r["vdim"])
        if L.get("mlp"):
            ff = L["mlp"]["ff"]
            w[p + "norm2"] = rnd(W, std=0.2)
            for n, rows, cols in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                w[p + "mlp." + n] = fan(rows, cols)
                w[p + "mlp." + n + ".b"] = rnd(rows, std=0.3)
    return w
