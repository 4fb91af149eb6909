"""Drive bin/trace_run (the product's own entry: registry -> scheduler -> sequence-batch engine) from the tests: model
folders, traces of steps, comparisons of rows of logits."""
from __future__ import annotations

import json
import struct
import subprocess
import tempfile
from pathlib import Path

import numpy as np

ROOT = Path(__file__).resolve().parent.parent
TRACE_RUN = ROOT / "bin" / "trace_run"


def run_trace(model_dir, steps, dtype="float32", max_tokens=2048, page=None, residual=False, vocab=None, extra=()):
    """steps: [{"entries": [{"id", "tokens", "want"}], "end": [...]}].  Returns (logits per step, residual per step):
    logits[i] is [wanted rows, vocab] (None when nothing was wanted)."""
    out = tempfile.mkdtemp(prefix="kllm_trace_")
    cmd = [str(TRACE_RUN), "--model", str(model_dir), "--dtype", dtype, "--out", out, "--max-tokens", str(max_tokens)]
    if page:
        cmd += ["--page", str(page)]
    if residual:
        cmd += ["--residual"]
    cmd += list(extra)
    text = "".join(json.dumps({"step": i, "entries": s["entries"], "end": s.get("end", [])}) + "\n"
                   for i, s in enumerate(steps))
    r = subprocess.run(cmd, input=text, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, f"trace_run exit {r.returncode}\n{r.stderr[-3000:]}"
    done = [ln for ln in r.stdout.splitlines() if ln.startswith("done ")]
    assert done == [f"done {i}" for i in range(len(steps))], r.stdout[-2000:]
    if vocab is None:
        vocab = json.loads((Path(model_dir) / "config.json").read_text())["vocab"]
    logits, resid = [], []
    for i, s in enumerate(steps):
        n = sum(len(e.get("want", [])) for e in s["entries"])
        f = Path(out) / f"{i}.f32"
        logits.append(np.fromfile(f, dtype="<f4").reshape(n, vocab) if n else None)
        assert n or not f.exists()
        rf = Path(out) / f"{i}.residual.f32"
        resid.append(np.fromfile(rf, dtype="<f4") if residual else None)
    return logits, resid


def whole(rid, tokens, want=None, end=True):
    return {"entries": [{"id": rid, "tokens": list(tokens), "want": list(range(len(tokens))) if want is None else want}],
            "end": [rid] if end else []}


def rel_err(got, ref):
    """Root-mean-square difference of the rows (mean over the vocabulary taken off), relative to the reference's own
    spread: the largest over the rows."""
    got = np.asarray(got, dtype=np.float64)
    ref = np.asarray(ref, dtype=np.float64)
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    spread = (ref - ref.mean(-1, keepdims=True)).std()
    return float(np.sqrt((d ** 2).mean(-1)).max() / spread)


def row_errors(got, ref):
    """rel_err of every row on its own."""
    return np.array([rel_err(got[i:i + 1], ref[i:i + 1]) for i in range(len(ref))])


def assert_rows(got, ref, tol):
    assert len(got) == len(ref)
    err = row_errors(got, ref)
    assert err.max() < tol, f"first bad position {int(np.argmax(err >= tol))} of {len(ref)}, worst {err.max():.3g}"


def single(rid, tokens, end=False):
    """One step per token."""
    steps = [{"entries": [{"id": rid, "tokens": [x], "want": [0]}]} for x in tokens]
    if end and steps:
        steps[-1]["end"] = [rid]
    return steps


def random_tokens(n, vocab, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def bf16_round(a):
    """Round float64 values to the nearest bfloat16 (ties to even); the result is exactly representable."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7fff + ((u >> 16) & 1)) & 0xffff0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


def write_model(folder, cfg, weights):
    """config.json and model.safetensors (bfloat16) in `folder`."""
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
