"""Plain restatement of the Perezen design for the tests: numpy, float64, one function per mechanism, no cache (every call sees whole
sequences; the recurrence goes token by token).  It shares no code with the library; weights are a dict name -> float array, the
configuration is the parsed config.json.

`operand` is applied to what enters a matrix product or the cache.  The identity gives the exact result; rounding to bf16 gives what
a 16-bit computation of the same design may lose."""
import numpy as np


def exact(x):
    return x


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def rotate_half(v, positions, base, dims):
    """v [..., tokens, n]: dimensions i and i + dims/2, i < dims/2, turned by position * base^(-2i/dims); the rest unchanged."""
    half = dims // 2
    a = positions[:, None] * (base ** (-2.0 * np.arange(half) / dims))[None, :]
    u, w = v[..., :half], v[..., half:dims]
    out = v.copy()
    out[..., :half] = u * np.cos(a) - w * np.sin(a)
    out[..., half:dims] = w * np.cos(a) + u * np.sin(a)
    return out


def visible(T, size):
    """[queries, keys]: what is not later and lies in the same chunk of `size` positions (0: no chunks)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def softmax(s):
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def differential_weight(w, diff):
    return np.exp((w["lq1"] * w["lk1"]).sum()) - np.exp((w["lq2"] * w["lk2"]).sum()) + diff


def attention_keys_values(h, w, m, eps, operand=exact):
    """Keys [kv heads, maps, tokens, dim] (normed, rotated) and values [kv heads, tokens, vdim] as the cache holds them."""
    T, G, d = h.shape[0], m["kv_heads"], m["dim"]
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, 2, d).transpose(1, 2, 0, 3)
    k = rotate_half(rms_norm(k, w["k.norm"], eps), np.arange(T, dtype=np.float64), m["rot"]["base"], m["rot"]["dims"])
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, m["vdim"]).transpose(1, 0, 2)
    return operand(k), operand(v)


def differential_attention(h, w, m, eps, keys_values, operand=exact):
    """h [tokens, width]; w: this mixer's tensors by their short names; m: the mixer's sizes; keys_values: from this layer or another."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    k, v = keys_values
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, 2, d).transpose(1, 2, 0, 3)
    q = operand(rotate_half(rms_norm(q, w["q.norm"], eps), np.arange(T, dtype=np.float64), m["rot"]["base"], m["rot"]["dims"]))
    seen = visible(T, m["mask"]["size"] if m.get("mask") else 0)
    lam = differential_weight(w, m["diff"])
    heads = []
    for i in range(H):
        g = i // (H // G)
        a = [operand(softmax(np.where(seen, (q[i, c] @ k[g, c].T) * m["scale"], -np.inf))) @ v[g] for c in range(2)]
        heads.append(unit_rms(a[0] - lam * a[1], eps) * (1.0 - m["diff"]))
    return operand(np.concatenate(heads, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def mlstm_denominator(nq, m):
    return max(abs(nq), np.exp(-m)) + 1e-6


def mlstm_recurrence(q, k, v, log_i, log_f):
    """One head, token by token: q, k [tokens, dim], v [tokens, vdim], log gates [tokens] -> [tokens, vdim]."""
    S, n, m = np.zeros((k.shape[1], v.shape[1])), np.zeros(k.shape[1]), 0.0
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        top = max(log_f[t] + m, log_i[t])
        keep, add = np.exp(log_f[t] + m - top), np.exp(log_i[t] - top)
        S, n, m = keep * S + add * np.outer(k[t], v[t]), keep * n + add * k[t], top
        out[t] = (S.T @ q[t]) / mlstm_denominator(n @ q[t], m)
    return out


def mlstm(h, w, m, eps, operand=exact):
    T, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = operand(h @ w["q"].T).reshape(T, H, d) * d ** -0.5
    k = operand(h @ w["k"].T).reshape(T, H, d)
    v = operand(h @ w["v"].T).reshape(T, H, dv)
    log_i = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    log_f = log_sigmoid(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o = np.stack([unit_rms(mlstm_recurrence(q[:, i], k[:, i], v[:, i], log_i[:, i], log_f[:, i]), eps) for i in range(H)], 1).reshape(T, H * dv)
    return operand(o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def gated_mlp(h, gate, up, down, operand=exact):
    return operand(silu(h @ gate.T) * (h @ up.T)) @ down.T


def embedding(W, tokens):
    return W["embed"][tokens] + W["pos"][:len(tokens)]


def forward(cfg, weights, tokens, residuals=None, operand=exact):
    """Logits [tokens, vocab]; residuals (a list, optional) receives the residual stream after every layer."""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]
    x = embedding(W, tokens)
    kv = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mix = {k[len(p) + 4:]: v for k, v in W.items() if k.startswith(p + "mix.")}
        h = operand(rms_norm(x, W[p + "norm1"], eps))
        if layer["type"] == "mlstm":
            y = mlstm(h, mix, m, eps, operand)
        else:
            j = m.get("kv_from")
            kv[i] = attention_keys_values(h, mix, m, eps, operand) if j is None else kv[j]
            y = differential_attention(h, mix, m, eps, kv[i], operand)
        x = x + rms_norm(y, W[p + "norm1b"], eps)
        if layer.get("mlp"):
            h = operand(rms_norm(x, W[p + "norm2"], eps))
            x = x + rms_norm(gated_mlp(h, W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"], operand), W[p + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x)
    return operand(rms_norm(x, W["final.norm"], eps)) @ W["head"].T * cfg["logit_scale"]
