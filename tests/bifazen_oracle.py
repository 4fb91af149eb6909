"""A slow float64 restatement of the Bifazen family, one function per mechanism.

It shares no code with the product path: numpy only, whole sequences, no cache and no state (every function sees the
complete sequence).  `weights` maps tensor names to float64 arrays; `config` is the parsed config.json.

    tokens --embed--> S equal streams --> layers --> sum of the streams --> centred RMS norm --> embed^T

    layer:     two sublayers (mixer, feed-forward).  A sublayer reads a weighted sum of the streams, u = sum_s in_s x_s,
               and its output y joins every stream: x_t <- sum_s mix_st x_s + out_t y
    mixers:    'latent_attention' (keys and values through a low-rank latent, one rotated key part for all heads, a window)
               'attention'        (biases, one norm over all query rows and one over all key rows, no positions, a window,
                                   values blended with those of the first blending layer, a gate per head)
    ff:        down(gelu(gate h) * up h)
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(v, dims, base):
    """v [T, ..., n]: coordinates (2i, 2i + 1) of the first `dims` turn by position * base^(-2i / dims)."""
    T = v.shape[0]
    out = v.copy()
    for i in range(dims // 2):
        a = (np.arange(T) * base ** (-2.0 * i / dims)).reshape((T,) + (1,) * (v.ndim - 2))
        x, y = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = x * np.cos(a) - y * np.sin(a)
        out[..., 2 * i + 1] = y * np.cos(a) + x * np.sin(a)
    return out


def window_mask(T, window):
    """mask[i, j]: does position i see position j?"""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < window) if window else True)


def softmax_rows(s, mask):
    s = np.where(mask, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


# ---- mixers ------------------------------------------------------------------------------------------------------------
def latent_attention(h, w, p, m, eps):
    T, H, dim, rd, vd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim + rd)
    down = h @ w[p + "dkv"].T
    c = rms_unit(down[:, :rank], eps) * w[p + "dkv.norm"]
    rot = m.get("rot")
    turn = (lambda x: rotate_pairs(x, rot["dims"], rot["base"])) if rot else (lambda x: x)
    k_rot = turn(down[:, rank:])
    k = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    q_rot = turn(q[:, :, dim:])
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else 0)
    out = np.zeros((T, H, vd))
    for i in range(H):
        s = (q[:, i, :dim] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = softmax_rows(s, mask) @ v[:, i]
    return out.reshape(T, H * vd) @ w[p + "o"].T


def blended_values(v, first, lam):
    """(1 - lam) v + lam first; the first blending layer has nothing to blend with."""
    return v if first is None else (1.0 - lam) * v + lam * first


def plain_attention(h, w, p, m, eps, first_values):
    """Returns (output, the values before blending when this layer is the first to blend, else None)."""
    T, H, G, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    q = (rms_unit(q, eps) * w[p + "q.norm"]).reshape(T, H, dim)
    k = (rms_unit(k, eps) * w[p + "k.norm"]).reshape(T, G, dim)
    raw = None
    if m.get("v_mix"):
        if first_values is None:
            raw = v
        else:
            v = blended_values(v, first_values, float(w[p + "vmix"]))
    v = v.reshape(T, G, vd)
    gate = sigmoid(h @ w[p + "g"].T)
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else 0)
    out = np.zeros((T, H, vd))
    for i in range(H):
        g = i // (H // G)
        out[:, i] = softmax_rows(q[:, i] @ k[:, g].T * m["scale"], mask) @ v[:, g] * gate[:, i:i + 1]
    return out.reshape(T, H * vd) @ w[p + "o"].T + w[p + "o.b"], raw


def gated_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- streams -----------------------------------------------------------------------------------------------------------
def read_streams(x, w, p):
    """x [S, T, width] -> what the sublayer reads."""
    return np.tensordot(w[p + "in"], x, axes=(0, 0))


def write_streams(x, y, w, p):
    """mix is indexed [from, to]."""
    S = x.shape[0]
    mix, out = w[p + "mix"], w[p + "out"]
    return np.stack([sum(mix[s, t] * x[s] for s in range(S)) + out[t] * y for t in range(S)])


# ---- the model ---------------------------------------------------------------------------------------------------------
def forward(config, w, tokens):
    """(logits [T, vocab], sum of the streams after every layer [layers, T, width])."""
    eps = config["norm"]["eps"]
    x = np.repeat(w["embed"][np.asarray(tokens)][None], config["streams"], axis=0)
    first_values, trace = None, []
    for i, L in enumerate(config["layers"]):
        p = f"l{i}."
        h = centred_norm(read_streams(x, w, p + "hc1."), w[p + "norm1"], eps)
        if L["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", L["mixer"], eps)
        else:
            y, raw = plain_attention(h, w, p + "mix.", L["mixer"], eps, first_values)
            first_values = raw if raw is not None else first_values
        x = write_streams(x, y, w, p + "hc1.")
        if L.get("mlp"):
            h = centred_norm(read_streams(x, w, p + "hc2."), w[p + "norm2"], eps)
            x = write_streams(x, gated_ff(h, w, p + "mlp."), w, p + "hc2.")
        trace.append(x.sum(0))
    return centred_norm(x.sum(0), w["final.norm"], eps) @ w["embed"].T, np.stack(trace)


def greedy(config, weights, prompt, n_new):
    """n_new greedy tokens after `prompt` (lowest index on ties), recomputing the whole sequence every time."""
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(np.argmax(forward(config, weights, seq)[0][-1])))
    return seq[len(prompt):]


# ---- small configurations and random weights for the tests ---------------------------------------------------------------
def latent_mixer(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, window=14, base=1000.0, scale=None, rot_dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "rot": {"dims": rot_dim if rot_dims is None else rot_dims, "base": base},
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if window:
        m["mask"] = {"size": window}
    return m


def plain_mixer(heads=4, kv_heads=2, dim=12, vdim=10, window=11, scale=None, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window}
    return m


def make_config(width=48, vocab=61, layers=(), eps=3e-6, streams=3):
    """layers: (mixer, ff size or None); the mixer's kind is read off its keys."""
    out = []
    for mixer, ff in layers:
        out.append({"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer,
                    "mlp": {"kind": "dense", "ff": ff} if ff else None})
    return {"architecture": "Bifazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "layers": out}


def bf16_round(a):
    """Round float64 values to the nearest bfloat16 (ties to even); the result is exactly representable."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7fff + ((u >> 16) & 1)) & 0xffff0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def make_weights(cfg, seed=0, sharp=1.0):
    """Random bf16-representable weights.  `sharp` multiplies the attentions' query weights (the norm weights of those
    that norm their queries): > 1 makes the softmax peaky, so that single keys (those at a window's edge too) carry the
    output."""
    rng = np.random.default_rng(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def rnd(*shape, std=1.0, mean=0.0):
        return bf16_round(mean + std * rng.standard_normal(shape))

    def fan(rows, cols, gain=1.0):
        return rnd(rows, cols, std=gain * cols ** -0.5)

    w = {"embed": rnd(V, W, std=0.5), "final.norm": rnd(W, std=0.2)}
    for i, L in enumerate(cfg["layers"]):
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
            H, G = m["heads"], m["kv_heads"]
            for n, rows in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"])):
                w[q + n] = fan(rows, W)
                w[q + n + ".b"] = rnd(rows, std=0.4)
            w[q + "q.norm"] = rnd(H * m["dim"], mean=sharp, std=0.2 * sharp)
            w[q + "k.norm"] = rnd(G * m["dim"], mean=1.5, std=0.3)
            if m.get("v_mix"):
                w[q + "vmix"] = rnd(mean=0.4, std=0.2)
            w[q + "g"] = fan(H, W, 2.0)
            w[q + "o"] = fan(W, H * m["vdim"])
            w[q + "o.b"] = rnd(W, std=0.2)
        for n in (1, 2) if L.get("mlp") else (1,):
            w[p + f"hc{n}.in"] = rnd(S, mean=1.0 / S, std=0.5 / S)
            w[p + f"hc{n}.out"] = rnd(S, mean=0.7, std=0.4)
            w[p + f"hc{n}.mix"] = bf16_round(0.8 * np.eye(S) + 0.2 / S + 0.1 * rng.standard_normal((S, S)))
        if L.get("mlp"):
            ff = L["mlp"]["ff"]
            w[p + "norm2"] = rnd(W, std=0.2)
            w[p + "mlp.gate"] = fan(ff, W, 1.5)
            w[p + "mlp.up"] = fan(ff, W)
            w[p + "mlp.down"] = fan(W, ff)
    return w


def write_model(folder, cfg, weights):
    """config.json and model.safetensors (bfloat16) in `folder`."""
    import json
    import struct
    from pathlib import Path
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for name, a in weights.items():
        u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
        assert not (u & 0xffff).any(), f"{name} is not bf16-representable"
        raw = (u >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder
