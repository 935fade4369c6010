"""Small Perezen configurations with random weights for the tests (nothing of a published model)."""
import numpy as np

from stack_common import bf16_round, tokens, write_folder  # noqa: F401


def attention(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.45, rot=16, base=300.0, chunk=53, diff=0.3, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, rot=dict(base=base, dims=rot))
    if chunk:
        m["mask"] = dict(size=chunk)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def mlstm(heads=3, dim=20, vdim=48, cap=6.0):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def config(layers, width=104, vocab=211, eps=0.02, positions=700, logit_scale=0.7):
    """layers: list of ((type, mixer), ff or None).  (The rms norms would hide the size of what they norm: eps is large enough to show it.)"""
    return dict(architecture="Perezen", norm=dict(eps=eps), vocab=vocab, width=width, max_positions=positions, logit_scale=logit_scale,
                layers=[dict(type=t, mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None) for (t, m), ff in layers])


def weights(cfg, seed, pos=0.3):
    """Random weights; pos: size of the position vectors."""
    rng = np.random.default_rng(seed)
    D, V, w = cfg["width"], cfg["vocab"], {}

    def mat(name, out, inn, gain=1.0):
        w[name] = bf16_round(rng.standard_normal((out, inn)) * gain / np.sqrt(inn))

    def vec(name, n, mean, spread):
        w[name] = bf16_round(mean + spread * rng.standard_normal(n))
    w["embed"] = bf16_round(rng.standard_normal((V, D)))
    w["pos"] = bf16_round(pos * rng.standard_normal((cfg["max_positions"], D)))
    mat("head", V, D)
    vec("final.norm", D, 1.0, 0.3)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        vec(p + "norm1", D, 1.0, 0.3)
        vec(p + "norm1b", D, 0.6, 0.2)
        mat(p + "mix.g", H * dv, D)
        mat(p + "mix.o", D, H * dv, 2.0)
        if l["type"] == "mlstm":
            mat(p + "mix.q", H * d, D, 1.5)
            mat(p + "mix.k", H * d, D)
            mat(p + "mix.v", H * dv, D)
            vec(p + "mix.norm", H * dv, 1.0, 0.3)
            mat(p + "mix.i", H, D, 2.0)
            vec(p + "mix.i.b", H, -0.5, 1.0)
            mat(p + "mix.f", H, D)
            vec(p + "mix.f.b", H, 3.0, 2.0)
        else:
            G = m["kv_heads"]
            mat(p + "mix.q", H * 2 * d, D)
            vec(p + "mix.q.b", H * 2 * d, 0.0, 0.5)
            vec(p + "mix.q.norm", d, 1.2, 0.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(p + "mix." + n, d, 0.0, 0.5 / np.sqrt(d))
            if m.get("kv_from") is None:
                mat(p + "mix.k", G * 2 * d, D)
                vec(p + "mix.k.b", G * 2 * d, 0.0, 0.5)
                vec(p + "mix.k.norm", d, 1.2, 0.3)
                mat(p + "mix.v", G * dv, D)
                vec(p + "mix.v.b", G * dv, 0.0, 0.5)
        if l["mlp"]:
            vec(p + "norm2", D, 1.0, 0.3)
            vec(p + "norm2b", D, 0.6, 0.2)
            mat(p + "mlp.gate", l["mlp"]["ff"], D, 1.5)
            mat(p + "mlp.up", l["mlp"]["ff"], D)
            mat(p + "mlp.down", D, l["mlp"]["ff"])
    return w


A, R = attention, mlstm
CASES = {
    # every branch: both mixers with and without feed-forward, other sizes per layer, shared keys and values under another mask
    "all": config([(A(), 152), (R(), None), (A(scale=0.3, chunk=31, diff=0.6, kv_from=0), 96), (R(heads=5, dim=8, vdim=24, cap=15.0), 64),
                   (A(heads=2, kv_heads=1, dim=8, vdim=72, rot=8, chunk=200), None), (A(heads=4, kv_heads=1, dim=8, vdim=72, rot=8, kv_from=4), 40)]),
    # sizes that are multiples of nothing much; as many key / value heads as heads
    "odd": config([(A(heads=3, kv_heads=3, dim=19, vdim=37, rot=10, chunk=41), 133), (R(heads=3, dim=13, vdim=21), 61), (A(heads=3, kv_heads=3, dim=19, vdim=37, rot=10, kv_from=0), None)],
                  width=93, vocab=207),
    "one_head": config([(A(heads=1, kv_heads=1, dim=2, vdim=8, rot=2, scale=1.0, chunk=1), 8), (R(heads=1, dim=1, vdim=1), None)], width=16, vocab=31),
    "no_chunks": config([(A(heads=4, kv_heads=2, dim=64, vdim=64, rot=32, scale=0.2, chunk=0), 320), (R(heads=2, dim=64, vdim=64), None)], width=160, vocab=300),
    "recurrent_only": config([(R(), 64), (R(heads=2, dim=40, vdim=100), None)]),
    "attention_only": config([(A(chunk=128), None), (A(heads=2, kv_heads=2, dim=32, vdim=32, rot=32, chunk=64), 64)]),
    # more query vectors per key / value head than a block takes; everything rotated
    "many_heads": config([(A(heads=9, kv_heads=1, dim=16, vdim=16, rot=16, scale=0.6, chunk=90), None), (A(heads=20, kv_heads=2, dim=8, vdim=24, rot=4, chunk=300), 72)], width=120),
    # head sizes of real models, and beyond them
    "large_heads": config([(A(heads=4, kv_heads=2, dim=128, vdim=128, rot=64, scale=0.2, chunk=150), 200), (R(heads=2, dim=128, vdim=256), None)], width=128, vocab=130),
    "wide_values": config([(A(heads=2, kv_heads=1, dim=64, vdim=256, rot=16, scale=0.25, chunk=140), None), (R(heads=1, dim=256, vdim=512), None)], width=88, vocab=115),
    "beyond": config([(A(heads=2, kv_heads=1, dim=200, vdim=300, rot=100, scale=0.15, chunk=100), None), (R(heads=1, dim=300, vdim=70), None), (R(heads=1, dim=16, vdim=600), None)],
                     width=96, vocab=115),
}
