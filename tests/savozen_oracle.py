"""Plain restatement of the Savozen design for the tests: numpy, float64, one function per mechanism, no cache (every call
sees whole sequences).  It shares no code with the library; weights are a dict name -> float array, the configuration is the
parsed config.json.

`operand` is applied to what enters a matrix product or the cache.  The identity gives the exact result; rounding to bf16 gives
what a 16-bit computation of the same design may lose."""
import math

import numpy as np


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def dynamic_tanh(x, alpha, weight, bias):
    return np.tanh(alpha * x) * weight + bias


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_interleaved(v, positions, base, dims):
    """v [..., tokens, n]: dimensions (2i, 2i+1), i < dims/2, turned by position * base^(-2i/dims); the rest unchanged."""
    out = v.copy()
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    a = positions[:, None] * f[None, :]
    u, w = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - w * np.sin(a)
    out[..., 1:dims:2] = w * np.cos(a) + u * np.sin(a)
    return out


def sink_softmax(scores, sink):
    """scores [heads, queries, keys] (-inf where masked); the denominator also holds exp(sink_h)."""
    m = np.maximum(scores.max(-1, keepdims=True), sink[:, None, None])
    e = np.exp(scores - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def exact(x):
    return x


def latent_attention(h, w, m, eps, positions=None, operand=exact):
    """h [tokens, width]; w: this mixer's tensors by their short names; m: the mixer's sizes."""
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T, dtype=np.float64) if positions is None else positions
    q = (h @ w["q"].T).reshape(T, H, d + r).transpose(1, 0, 2)
    q_plain = operand(q[..., :d])
    q_rot = operand(rotate_interleaved(q[..., d:], pos, m["rot"]["base"], m["rot"]["dims"]))
    down = h @ w["dkv"].T
    c = operand(rms_norm(down[:, :R], w["dkv.norm"], eps))
    k_rot = operand(rotate_interleaved(down[:, R:], pos, m["rot"]["base"], m["rot"]["dims"]))
    k = operand(c @ w["uk"].T).reshape(T, H, d).transpose(1, 0, 2)
    v = operand(c @ w["uv"].T).reshape(T, H, dv).transpose(1, 0, 2)
    s = (q_plain @ k.transpose(0, 2, 1) + q_rot @ k_rot.T[None]) * m["scale"]
    s = np.where(np.tril(np.ones((T, T), bool))[None], s, -np.inf)
    o = (operand(sink_softmax(s, w["sink"])) @ v).transpose(1, 0, 2).reshape(T, H * dv)
    return operand(o * sigmoid(h @ w["g"].T)) @ w["o"].T


def gated_mlp(h, gate, up, down, operand=exact):
    return operand(gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def token_side(x, e, gate, proj, norm, eps, operand=exact):
    y = operand(gelu_tanh(operand(x) @ gate.T) * e) @ proj.T
    return x + rms_norm(y, norm, eps)


def layer_runs(cfg):
    """(layer index, pass number if this run begins a pass of the loop else None) in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, weights, tokens, residuals=None, operand=exact):
    """Logits [tokens, vocab]; residuals (a list, optional) receives the residual stream after every layer run."""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]

    def norm(name, x):
        return operand(dynamic_tanh(x, W[name + ".alpha"], W[name], W[name + ".b"]))
    x = W["embed"][tokens] * cfg["embedding"]["scale"]
    side = cfg.get("token_side")
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + W["loop.step"][t]
        p = f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in W.items() if k.startswith(p + "mix.")}
        x = x + latent_attention(norm(p + "norm1", x), mix, cfg["layers"][i]["mixer"], eps, operand=operand)
        if cfg["layers"][i].get("mlp"):
            x = x + gated_mlp(norm(p + "norm2", x), W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"], operand)
        if side:
            e = W["side.embed"][tokens][:, i * side["dim"]:(i + 1) * side["dim"]]
            x = token_side(x, e, W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"], eps, operand)
        if residuals is not None:
            residuals.append(x)
    return norm("final.norm", x) @ W["head"].T
