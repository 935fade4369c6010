"""Seeded synthetic weights, prompts and configurations of the benchmark shapes.  All bytes come from the
counter-based generators of the test-support library (libl2b_synth.so, include/l2b_synth.h), so every machine builds the same model from a seed."""
import numpy as np

from . import _lib as L
from .model import ModelConfig, QuantMatrix, StackWeights, TransformerLayerWeights, TransformerWeights

Q4, Q5, Q6, F32 = L.TYPE_Q4_K, L.TYPE_Q5_K, L.TYPE_Q6_K, L.TYPE_F32


def normal_f32(n, seed, std):
    a = np.empty(int(n), dtype=np.float32)
    L.synth_check(L.synth_lib().l2b_synth_f32(L.ptr(a), a.size, int(seed), float(std), 0))
    return a


def kquant_bytes(ggml_type, n_blocks, seed):
    a = np.empty(int(n_blocks) * L.BLOCK_BYTES[ggml_type], dtype=np.uint8)
    L.synth_check(L.synth_lib().l2b_synth_kquant(ggml_type, L.ptr(a), int(n_blocks), int(seed)))
    return a


def tokens(n, seed, lo, hi):
    a = np.empty(int(n), dtype=np.int32)
    L.synth_check(L.synth_lib().l2b_synth_tokens(L.ptr(a), a.size, int(seed), int(lo), int(hi)))
    return a


def matrix(ggml_type, in_dim, out_dim, seed, std=0.02):
    """(in, out) weight matrix of the given storage type."""
    if ggml_type == F32:
        return normal_f32(in_dim * out_dim, seed, std).reshape(out_dim, in_dim)
    return QuantMatrix(ggml_type, kquant_bytes(ggml_type, (in_dim // 256) * out_dim, seed), in_dim, out_dim)


def _seed(base, layer, role):
    return (base * 1000003 + layer * 101 + role) & 0xFFFFFFFFFFFF


def model_weights(c: ModelConfig, types: dict, seed: int, tied_output=False, distinct_layers: int = 0) -> TransformerWeights:
    """types maps 'wq','wk','wv','wo','w1','w2','w3','token_embd','output' to a ggml type.  Norm gains are 1.
    distinct_layers = k > 0: only the first k layers are generated and layer l reuses the host arrays of layer l % k
    (every layer still gets its own device copy), for shapes whose full host copy would not fit in memory."""
    hs = c.dim // c.n_heads
    kv = hs * c.n_kv_heads
    ones = np.ones(c.dim, dtype=np.float32)
    layers = []
    for l in range(c.n_layers):
        if distinct_layers and l >= distinct_layers:
            layers.append(layers[l % distinct_layers])
            continue
        layers.append(TransformerLayerWeights(
            ones, ones,
            matrix(types["wq"], c.dim, c.dim, _seed(seed, l, 1)), matrix(types["wk"], c.dim, kv, _seed(seed, l, 2)),
            matrix(types["wv"], c.dim, kv, _seed(seed, l, 3)), matrix(types["wo"], c.dim, c.dim, _seed(seed, l, 4)),
            matrix(types["w1"], c.dim, c.hidden_dim, _seed(seed, l, 5)), matrix(types["w2"], c.hidden_dim, c.dim, _seed(seed, l, 6)),
            matrix(types["w3"], c.dim, c.hidden_dim, _seed(seed, l, 7))))
    emb = matrix(types["token_embd"], c.dim, c.vocab_size, _seed(seed, 999, 8))
    out = emb if tied_output else matrix(types["output"], c.dim, c.vocab_size, _seed(seed, 999, 9))
    return TransformerWeights(emb, layers, ones, out)


ALL = lambda t: {k: t for k in ("wq", "wk", "wv", "wo", "w1", "w2", "w3", "token_embd", "output")}

# the configurations the benchmark specification names
TINY_F32 = dict(config=ModelConfig(288, 768, 6, 6, 6, 32000, 256, 10000.0, False), types=ALL(F32), tied=True,
                n_prompt=16, n_decode=240)
LLAMA3_8B_Q4_K_S = dict(config=ModelConfig(4096, 14336, 32, 32, 8, 128256, 512, 500000.0, False),
                        types=dict(wq=Q4, wk=Q4, wv=Q5, wo=Q4, w1=Q4, w2=Q5, w3=Q4, token_embd=Q4, output=Q6), tied=False,
                        n_prompt=128, n_decode=256)
PHI3_MINI_Q5_K_M = dict(config=ModelConfig(3072, 8192, 32, 32, 32, 32064, 4096, 10000.0, True),
                        types=dict(ALL(Q5), output=Q6), tied=False, n_prompt=2048, n_decode=512)
LLAMA2_70B_Q4_K = dict(config=ModelConfig(8192, 28672, 80, 64, 8, 32000, 4096, 10000.0, False),
                       types=dict(ALL(Q4), output=Q6), tied=False, n_prompt=512, n_decode=256)


def scaled(spec, n_layers=None, vocab_size=None, seq_len=None):
    """The same shape with fewer layers / a smaller vocabulary / a shorter context (for parity runs the
    CPU oracle finishes in seconds)."""
    c = spec["config"]
    c2 = ModelConfig(c.dim, c.hidden_dim, n_layers or c.n_layers, c.n_heads, c.n_kv_heads, vocab_size or c.vocab_size,
                     seq_len or c.seq_len, c.rope_freq_base, c.rope_is_neox)
    return dict(spec, config=c2)


def prompt_tokens(spec, seed):
    c = spec["config"]
    return tokens(spec["n_prompt"], seed ^ 0xABCDEF, 3, c.vocab_size)


# ---- layer-stack models ------------------------------------------------------------------------------------
def _savozen(width, ff, heads, dim, rot, vdim, rank, side, layers, vocab):
    mix = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=(dim + rot) ** -0.5, rot=dict(base=500000.0, dims=rot))
    return dict(architecture="Savozen", embedding=dict(scale=1.0), norm=dict(eps=1e-5), vocab=vocab, width=width, token_side=dict(dim=side),
                layers=[dict(type="latent_attention", mixer=mix, mlp=dict(kind="dense", ff=ff)) for _ in range(layers)])


# Layers of the size of a real model's, and the llama shape of equal width, feed-forward and head count that they are measured beside.
SAVOZEN_SIZES = {
    "2k": dict(raw=_savozen(2048, 8192, 16, 128, 64, 128, 512, 128, 8, 32768), llama=ModelConfig(2048, 8192, 8, 16, 16, 32768, 2048, 500000.0, False)),
    "4k": dict(raw=_savozen(4096, 14336, 32, 128, 64, 128, 512, 256, 8, 32768), llama=ModelConfig(4096, 14336, 8, 32, 8, 32768, 2048, 500000.0, False)),
}


def bf16_matrix(out_dim, in_dim, seed):
    """Random bf16 bit patterns with magnitudes around 1/64 (two octaves, both signs)."""
    bits = np.random.default_rng(seed).integers(0, 65536, size=(out_dim, in_dim), dtype=np.uint16)
    return (bits & np.uint16(0x80FF)) | np.uint16(0x3C00)


def savozen_weights(raw, seed):
    """Weights of a Savozen configuration by tensor name; layers of one size share their host arrays (every layer has its own device
    copy)."""
    D, V, shared = raw["width"], raw["vocab"], {}

    def mat(key, out, inn):
        if (key, out, inn) not in shared:
            shared[(key, out, inn)] = bf16_matrix(out, inn, seed + len(shared))
        return shared[(key, out, inn)]
    w = StackWeights(embed=mat("embed", V, D), head=mat("head", V, D))

    def norm(name):
        w[name] = np.ones(D, np.float32)
        w[name + ".b"] = np.zeros(D, np.float32)
        w[name + ".alpha"] = np.float32(0.5)
    norm("final.norm")
    if raw.get("loop"):
        w["loop.step"] = normal_f32(raw["loop"]["times"] * D, seed, 0.1).reshape(-1, D)
    side = raw["token_side"]["dim"] if raw.get("token_side") else 0
    if side:
        w["side.embed"] = mat("side.embed", V, side * len(raw["layers"]))
    for i, l in enumerate(raw["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        norm(p + "norm1")
        for name, out, inn in (("q", H * (d + r), D), ("dkv", R + r, D), ("uk", H * d, R), ("uv", H * dv, R), ("g", H * dv, D), ("o", D, H * dv)):
            w[p + "mix." + name] = mat(name, out, inn)
        w[p + "mix.dkv.norm"] = np.ones(R, np.float32)
        w[p + "mix.sink"] = np.zeros(H, np.float32)
        if l["mlp"]:
            norm(p + "norm2")
            ff = l["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat("gate", ff, D), mat("up", ff, D), mat("down", D, ff)
        if side:
            w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = mat("sgate", side, D), mat("sproj", D, side), np.full(D, 0.5, np.float32)
    return w


def savozen_flops_per_token(raw, npos):
    """Multiply-adds x 2 of one prompt token's matrix products, and of its attention over npos positions (expanded form)."""
    D, side = raw["width"], raw["token_side"]["dim"] if raw.get("token_side") else 0
    dense = att = 0
    for l in raw["layers"]:
        m = l["mixer"]
        H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        dense += D * (H * (d + r) + R + r + H * dv) + H * (d + dv) * R + H * dv * D + 3 * D * (l["mlp"]["ff"] if l["mlp"] else 0) + 2 * D * side
        att += H * npos * (d + r + dv)
    return 2 * dense, 2 * att


def _perezen(width, ff, heads, kv_heads, dim, vdim, mheads, mdim, mvdim, layers, vocab, chunk=8192):
    """Layers in threes: attention, mLSTM (no feed-forward), attention on the keys and values of the first."""
    att = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5, diff=0.4, rot=dict(base=500000.0, dims=dim), mask=dict(size=chunk))
    rec = dict(heads=mheads, dim=mdim, vdim=mvdim, gate_cap=15.0)
    mlp = dict(kind="dense", ff=ff)
    return dict(architecture="Perezen", norm=dict(eps=1e-5), vocab=vocab, width=width, max_positions=2048, logit_scale=1.0,
                layers=[dict(type="mlstm", mixer=rec, mlp=None) if i % 3 == 1 else dict(type="attention", mixer=dict(att, kv_from=i - 2) if i % 3 == 2 else att, mlp=mlp)
                        for i in range(layers)])


# Layers of the size of a real model's; each is measured beside the Savozen layers of the same name (equal width, feed-forward and heads).
PEREZEN_SIZES = {
    "2k": _perezen(2048, 8192, 16, 4, 64, 128, 4, 256, 512, 8, 32768),
    "4k": _perezen(4096, 14336, 32, 8, 64, 128, 8, 256, 512, 8, 32768),
}


def perezen_weights(raw, seed):
    """Weights of a Perezen configuration by tensor name; layers of one size share their host arrays."""
    D, V, shared = raw["width"], raw["vocab"], {}

    def mat(out, inn):
        if (out, inn) not in shared:
            shared[(out, inn)] = bf16_matrix(out, inn, seed + len(shared))
        return shared[(out, inn)]
    w = StackWeights({"embed": mat(V, D), "head": mat(V, D), "pos": mat(raw["max_positions"], D), "final.norm": np.ones(D, np.float32)})
    for i, l in enumerate(raw["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = np.ones(D, np.float32), np.full(D, 0.5, np.float32)
        w[p + "mix.g"], w[p + "mix.o"] = mat(H * dv, D), mat(D, H * dv)
        if l["type"] == "mlstm":
            w[p + "mix.q"], w[p + "mix.k"], w[p + "mix.v"], w[p + "mix.norm"] = mat(H * d, D), mat(H * d, D), mat(H * dv, D), np.ones(H * dv, np.float32)
            w[p + "mix.i"], w[p + "mix.f"] = mat(H, D), mat(H, D)
            w[p + "mix.i.b"], w[p + "mix.f.b"] = np.zeros(H, np.float32), np.linspace(2.0, 8.0, H, dtype=np.float32)
        else:
            G = m["kv_heads"]
            parts = [("q", H * 2 * d)] + ([("k", G * 2 * d), ("v", G * dv)] if m.get("kv_from") is None else [])
            for n, rows in parts:
                w[p + "mix." + n], w[p + "mix." + n + ".b"] = mat(rows, D), np.zeros(rows, np.float32)
                if n != "v":
                    w[p + "mix." + n + ".norm"] = np.ones(d, np.float32)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + "mix." + n] = normal_f32(d, seed, 0.1)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            w[p + "norm2"], w[p + "norm2b"] = np.ones(D, np.float32), np.full(D, 0.5, np.float32)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, D), mat(ff, D), mat(D, ff)
    return w


def perezen_flops_per_token(raw, npos):
    """Multiply-adds x 2 of one prompt token's matrix products, and of its mixers: attention over npos positions (within the chunk), the
    recurrence's update and read of the state."""
    D = raw["width"]
    dense = mix = 0
    for l in raw["layers"]:
        m = l["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "mlstm":
            dense += D * (H * (2 * d + 2 * dv + 2) + H * dv)
            mix += 2 * H * d * dv
        else:
            G = m["kv_heads"] if m.get("kv_from") is None else 0
            dense += D * (2 * H * d + G * (2 * d + dv) + 2 * H * dv)
            mix += 2 * H * min(npos, m["mask"]["size"]) * (d + dv)
        dense += 3 * D * (l["mlp"]["ff"] if l["mlp"] else 0)
    return 2 * dense, 2 * mix


def perezen_cache_bytes(raw, npos):
    """Bytes of cache and state a decode step at position npos reads and writes (bf16 rows; f32 states)."""
    b = 0
    for l in raw["layers"]:
        m = l["mixer"]
        b += 8 * m["heads"] * m["dim"] * m["vdim"] if l["type"] == "mlstm" else 2 * m["kv_heads"] * (2 * m["dim"] + m["vdim"]) * min(npos, m["mask"]["size"])
    return b


def savozen_cache_bytes(raw, npos):
    return sum(2 * (l["mixer"]["kv_rank"] + l["mixer"]["rot_dim"]) * npos for l in raw["layers"])
