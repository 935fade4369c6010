"""Small Savozen configurations with random weights for the tests (nothing of a published model)."""
import numpy as np

from stack_common import bf16_round, tokens, write_folder  # noqa: F401


def mixer(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=56, scale=0.4, base=10000.0):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))


def config(layers, width=104, vocab=211, loop=None, side=None, emb=1.3, eps=1e-4):
    """layers: list of (mixer, ff or None)."""
    c = dict(architecture="Savozen", embedding=dict(scale=emb), norm=dict(eps=eps), vocab=vocab, width=width,
             layers=[dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None) for m, ff in layers])
    if loop:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    if side:
        c["token_side"] = dict(dim=side)
    return c


def weights(cfg, seed, sharp=3.0):
    """Random weights; `sharp` scales the queries so that single scores stand out of the softmax."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inn, gain=1.0):
        w[name] = bf16_round(rng.standard_normal((out, inn)) * gain / np.sqrt(inn))

    def norm(name):
        w[name] = bf16_round(1.0 + 0.3 * rng.standard_normal(D))
        w[name + ".b"] = bf16_round(0.2 * rng.standard_normal(D))
        w[name + ".alpha"] = bf16_round(np.float32(0.6 + 0.3 * rng.random()))
    w["embed"] = bf16_round(rng.standard_normal((V, D)))
    mat("head", V, D)
    norm("final.norm")
    if cfg.get("loop"):
        w["loop.step"] = bf16_round(0.5 * rng.standard_normal((cfg["loop"]["times"], D)))
    side = cfg.get("token_side")
    if side:
        w["side.embed"] = bf16_round(rng.standard_normal((V, side["dim"] * len(cfg["layers"]))))
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        norm(p + "norm1")
        mat(p + "mix.q", H * (d + r), D, sharp)
        mat(p + "mix.dkv", R + r, D)
        w[p + "mix.dkv.norm"] = bf16_round(1.0 + 0.3 * rng.standard_normal(R))
        mat(p + "mix.uk", H * d, R)
        mat(p + "mix.uv", H * dv, R)
        w[p + "mix.sink"] = bf16_round(1.0 + 2.0 * rng.standard_normal(H))
        mat(p + "mix.g", H * dv, D)
        mat(p + "mix.o", D, H * dv, 2.0)
        if l["mlp"]:
            norm(p + "norm2")
            mat(p + "mlp.gate", l["mlp"]["ff"], D)
            mat(p + "mlp.up", l["mlp"]["ff"], D)
            mat(p + "mlp.down", D, l["mlp"]["ff"])
        if side:
            mat(p + "side.gate", side["dim"], D)
            mat(p + "side.proj", D, side["dim"])
            w[p + "side.norm"] = bf16_round(0.5 + 0.2 * rng.standard_normal(D))
    return w


M = mixer
CASES = {
    # every branch at once: different mixers, a layer without feed-forward, a loop inside the stack, a per-layer token input
    "all": config([(M(), 152), (M(heads=5, dim=8, rot_dim=24, vdim=16, kv_rank=32, scale=0.3, base=500.0), None), (M(heads=2, vdim=72), 96)],
                  loop=(1, 3, 2), side=12),
    # sizes that are multiples of nothing much
    "odd": config([(M(heads=3, dim=19, rot_dim=10, vdim=37, kv_rank=51), 133), (M(heads=1, dim=7, rot_dim=6, vdim=9, kv_rank=13), 61)],
                  width=93, vocab=207, loop=(0, 1, 3), side=7),
    "one_head_one_layer": config([(M(heads=1, dim=16, rot_dim=2, vdim=8, kv_rank=8, scale=1.0), 8)], width=16, vocab=31, emb=1.0),
    "no_loop_no_side": config([(M(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, scale=0.12), 320), (M(), None)], width=160, vocab=300),
    "loop_everything": config([(M(), 64), (M(), 64)], loop=(0, 2, 4), side=16),
    # latents that spread over two, three and four pieces of a cache row; head sizes beyond one operand tile
    "rank_300": config([(M(heads=2, dim=72, rot_dim=40, vdim=144, kv_rank=300, scale=0.1), 96)], width=136, vocab=151, side=8),
    "rank_512": config([(M(heads=9, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=0.08), 200)], width=256, vocab=400),
    "wide_values": config([(M(heads=2, dim=40, rot_dim=24, vdim=272, kv_rank=120, scale=0.15), None)], width=88, vocab=115),
    "rank_900": config([(M(heads=2, dim=32, rot_dim=96, vdim=200, kv_rank=900, scale=0.1), None)], width=120, vocab=130, side=20),
}
