"""What the tests of the layer-stack models share: folders in the published format, portions through a session, comparison."""
import json
import struct

import numpy as np

LIMIT32 = 3e-5  # of the logits' root mean square
COMPUTE = ["float32", "bfloat16"]


def bf16_round(a):
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).reshape(np.shape(a))


def bf16(x):
    return bf16_round(x).astype(np.float64)


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def write_folder(path, cfg, w):
    """config.json and model.safetensors (bf16) in folder `path`."""
    with open(path / "config.json", "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, a in w.items():
        b = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = dict(dtype="BF16", shape=list(np.shape(a)), data_offsets=[at, at + len(b)])
        blobs.append(b)
        at += len(b)
    h = json.dumps(head).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def err(got, want):
    """Per position: rms over the vocabulary of the difference (mean taken off), relative to the rms of the expected logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean())


def check(got, want, compute, rows=slice(None)):
    """want: (exact logits, error of every position when operands are rounded to bf16).  32-bit: within LIMIT32, and where the model
    itself magnifies rounding (which the second shows) as much more.  16-bit: no more than a few times what rounding the operands alone
    costs, in the median, the 95th percentile and at the worst position."""
    want, rounding = want
    e = err(got, want[rows])
    assert np.isfinite(e).all()
    worst = (compute, int(e.argmax()), float(e.max()), float(np.median(e)), None if rounding is None else (float(rounding.max()), float(np.median(rounding))))
    if compute == "float32":
        more = 1.0 if rounding is None else np.maximum(1.0, rounding[rows] / (3 * np.median(rounding)))
        assert (e <= LIMIT32 * more).all(), worst
    else:
        assert e.max() <= 3 * rounding.max(), worst
        if e.size > 20:
            assert np.median(e) <= 2 * np.median(rounding), worst
        if e.size > 100:
            assert np.quantile(e, 0.95) <= 2.5 * np.quantile(rounding, 0.95), worst


def build(pkg, cfg, w, seq_len, compute):
    return pkg.LanguageModel(pkg.StackConfig(cfg, seq_len, compute), None, pkg.StackWeights(w))


def feed(pkg, state, toks, sizes):
    """The tokens in portions of the given sizes (the last one repeated); logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(pkg.extend(state, toks[at:at + n], at, range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)
