"""Perezen: configuration, what the test models can show (CPU), and the library against the plain oracle (GPU)."""
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

import perezen_cases as pc
import perezen_oracle as po
from stack_common import COMPUTE, bf16, build, check, err, feed

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def expected(cfg, w, toks):
    want = po.forward(cfg, w, toks)
    return want, err(po.forward(cfg, w, toks, operand=bf16), want)


# ---- CPU -------------------------------------------------------------------------------------------
def create(pkg, raw):
    from llama2_jl_b200 import _lib as L
    h = C.c_void_p()
    st = L.lib().l2b_model_create_stack(json.dumps(raw).encode(), 16, L.TYPE_BF16, -1, None, C.byref(h))
    msg = L.lib().l2b_last_error_string().decode()
    if h:
        L.lib().l2b_model_destroy(h)
    return st, msg


def test_configurations_are_checked(pkg):
    from llama2_jl_b200 import _lib as L, load_stack
    good = pc.CASES["all"]
    assert "Perezen" in load_stack.ARCHITECTURES
    for case in pc.CASES.values():
        assert create(pkg, case)[0] in (L.OK, L.ERR_NO_DEVICE)

    def mixer(i):
        return lambda r: r["layers"][i]["mixer"]
    for pick, change, word in [(lambda r: r, lambda r: r.pop("max_positions"), "max_positions"), (lambda r: r, lambda r: r.pop("logit_scale"), "logit_scale"),
                               (lambda r: r["layers"][1], lambda l: l.update(type="latent_attention"), "latent_attention"),
                               (mixer(0), lambda m: m.pop("diff"), "diff"), (mixer(0), lambda m: m.update(kv_heads=4), "kv_heads"), (mixer(0), lambda m: m["rot"].update(dims=26), "rot"),
                               (mixer(0), lambda m: m["mask"].update(size=0), "size"), (mixer(1), lambda m: m.update(gate_cap=0), "gate_cap"),
                               (mixer(2), lambda m: m.update(kv_from=1), "kv_from"), (mixer(2), lambda m: m.update(kv_from=2), "kv_from"), (mixer(5), lambda m: m.update(kv_from=2), "kv_from"),
                               (mixer(2), lambda m: m.update(vdim=41), "kv_from"), (lambda r: r["layers"][0]["mlp"], lambda m: m.update(kind="experts"), "experts")]:
        raw = json.loads(json.dumps(good))
        change(pick(raw))
        st, msg = create(pkg, raw)
        assert st == L.ERR_BAD_ARG and word in msg, (word, st, msg)
    assert pkg.StackConfig(good, 5000).seq_len == good["max_positions"] and pkg.StackConfig(good, 50).seq_len == 50


def test_rotation_turns_halves():
    v = np.arange(14, dtype=np.float64).reshape(1, 2, 7)
    r = po.rotate_half(v, np.array([0.0, 3.0]), 100.0, 4)
    assert np.array_equal(r[0, 0], v[0, 0]) and np.array_equal(r[0, 1, 4:], v[0, 1, 4:])
    for i, f in enumerate((1.0, 0.1)):
        z = complex(v[0, 1, i], v[0, 1, i + 2]) * np.exp(1j * 3.0 * f)
        assert np.allclose([r[0, 1, i], r[0, 1, i + 2]], [z.real, z.imag])


def test_recurrence_is_the_weighted_sum_over_earlier_tokens():
    """The step-by-step recurrence against its closed form: every earlier token weighted by the gates between."""
    rng = np.random.default_rng(3)
    q, k, v = rng.standard_normal((9, 4)), rng.standard_normal((9, 4)), rng.standard_normal((9, 5))
    i, f = 2 * rng.standard_normal(9), po.log_sigmoid(rng.standard_normal(9))
    got = po.mlstm_recurrence(q, k, v, i, f)
    for t in range(9):
        w = np.exp([i[s] + f[s + 1:t + 1].sum() for s in range(t + 1)])
        m = max([i[s] + f[s + 1:t + 1].sum() for s in range(t + 1)] + [f[:t + 1].sum()])
        a = w * (k[:t + 1] @ q[t])
        assert np.allclose(got[t], (a @ v[:t + 1]) * np.exp(-m) / (max(abs(a.sum()) * np.exp(-m), np.exp(-m)) + 1e-6))


def chunks_shifted(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (((i + 1) // size == (j + 1) // size) if size else True)


MISTAKES = {
    "no chunks": lambda mp: mp.setattr(po, "visible", lambda T, s, f=po.visible: f(T, 0)),
    "chunks one off": lambda mp: mp.setattr(po, "visible", chunks_shifted),
    "positions from 1": lambda mp: mp.setattr(po, "embedding", lambda W, t: W["embed"][t] + W["pos"][1:len(t) + 1]),
    "rotation from 1": lambda mp: mp.setattr(po, "rotate_half", lambda v, p, b, d, f=po.rotate_half: f(v, p + (v.shape[0] == 6), b, d)),
    "neighbours rotated": lambda mp: mp.setattr(po, "rotate_half", lambda v, p, b, d, f=po.rotate_half: f(v[..., list(range(0, d, 2)) + list(range(1, d, 2)) + list(range(d, v.shape[-1]))], p, b, d)),
    "constant part of the map weight left out": lambda mp: mp.setattr(po, "differential_weight", lambda w, d, f=po.differential_weight: f(w, 0.0)),
    "no gates": lambda mp: mp.setattr(po, "sigmoid", lambda z: np.ones_like(z)),
    "no result norm": lambda mp: mp.setattr(po, "rms_norm", lambda x, w, e, f=po.rms_norm: x * w if x.shape[-1] == 104 and abs(w.mean() - 0.6) < 0.1 else f(x, w, e)),
    "eps outside the root": lambda mp: mp.setattr(po, "unit_rms", lambda x, e: x / (np.sqrt((x * x).mean(-1, keepdims=True)) + e)),
    "state forgotten": lambda mp: mp.setattr(po, "mlstm_recurrence", lambda q, k, v, i, f, g=po.mlstm_recurrence: np.concatenate([g(*(x[a:a + 33] for x in (q, k, v, i, f))) for a in range(0, len(q), 33)])),
    "no floor of the denominator": lambda mp: mp.setattr(po, "mlstm_denominator", lambda nq, m: abs(nq) + 1e-6),
    "denominator keeps its sign": lambda mp: mp.setattr(po, "mlstm_denominator", lambda nq, m: max(nq, np.exp(-m)) + 1e-6),
    "forget gate after its log": lambda mp: mp.setattr(po, "log_sigmoid", lambda z: -np.log1p(np.exp(z))),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_the_models_show_mistakes(mistake, monkeypatch):
    """A mistake planted in the oracle moves the logits of the test model far beyond the limits of the 32-bit comparison, and (small
    ones, behind a norm that hides most of them, apart) also beyond those of the 16-bit comparison."""
    cfg = pc.CASES["all"]
    w, t = pc.weights(cfg, 1), pc.tokens(cfg, 110, 2)
    want, rounding = expected(cfg, w, t)
    MISTAKES[mistake](monkeypatch)
    e = err(po.forward(cfg, w, t), want)
    assert e.max() > 300 * 3e-5
    if mistake not in ("eps outside the root", "no floor of the denominator", "denominator keeps its sign"):
        assert np.sort(e)[-10] > 4 * rounding.max()


# ---- GPU -------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("case", list(pc.CASES))
def test_prompt_decode_and_portions(pkg, case, compute):
    """Whole prompt, token by token, a prompt then single tokens, and portions of several sizes, all against the oracle; sizes around
    the tiles of the prompt kernels, the switch between their forms, and portions of two tokens."""
    cfg = pc.CASES[case]
    w, t = pc.weights(cfg, 11), pc.tokens(cfg, 301, 12)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 301, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [301]), want, compute)
    for sizes in ([1], [200, 1], [2], [3, 50, 2, 128, 1, 47, 48, 64], [129, 127, 2], [17], [31, 33, 100]):
        state.reset()
        n = 140 if sizes in ([1], [2]) else 301
        check(feed(pkg, state, t[:n], sizes), want, compute, slice(n))
    model.close()


def only(cfg, w, keep):
    """Weights whose other mechanisms are silent: what is not named in `keep` adds zero to the residual stream."""
    w = {k: v.copy() for k, v in w.items()}
    for i, l in enumerate(cfg["layers"]):
        kind = "shared" if l["mixer"].get("kv_from") is not None else l["type"]
        if kind not in keep:
            w[f"l{i}.norm1b"][:] = 0
        if l["mlp"] and "mlp" not in keep:
            w[f"l{i}.norm2b"][:] = 0
    if "positions" not in keep:
        w["pos"][:] = 0
    return w


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("keep", ["", "positions", "attention", "shared", "mlstm", "mlp", "attention shared positions"])
def test_mechanisms_alone(pkg, keep, compute):
    """Embedding, norm and head alone; then one mechanism at a time on top."""
    cfg = pc.CASES["all"]
    w, t = only(cfg, pc.weights(cfg, 21), keep.split()), pc.tokens(cfg, 150, 22)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 150, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [150]), want, compute)
    state.reset()
    check(feed(pkg, state, t, [30, 60, 1]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("size", [100, 128, 1000])
def test_one_key_stands_out(pkg, size, compute):
    """One token's key is what every query asks for in the first map: who comes later in its chunk has its value, the next chunk has
    not.  Places at chunk borders and around tile borders, seen from prompts and from single decode steps."""
    cfg = pc.config([(pc.attention(heads=2, kv_heads=1, dim=32, vdim=32, rot=8, scale=1.0, chunk=size, diff=0.2), None)], vocab=97, eps=1e-4)
    n = 330
    base, toks = pc.weights(cfg, 41, pos=0.02), pc.tokens(cfg, n, 42)
    toks[toks == 5] = 6
    u = np.zeros((2, 32))
    u[0, 8:] = np.random.default_rng(43).choice([-1.0, 1.0], 24)  # (map 1, the dimensions that are not rotated)
    w = {k: v.copy() for k, v in base.items()}
    w["l0.mix.q.b"][:] = pc.bf16_round(np.tile(12 * u.ravel(), 2))
    w["l0.mix.q.norm"][:] = w["l0.mix.k.norm"][:] = 1.0
    e5 = w["embed"][5] / np.sqrt((w["embed"][5] ** 2).mean()) * w["l0.norm1"]
    w["l0.mix.k"] = pc.bf16_round(w["l0.mix.k"] + np.outer(12 * u.ravel(), e5) / (e5 @ e5))
    model = build(pkg, cfg, w, n, compute)
    for place in (0, 1, 63, 99, 100, 101, 127, 128, 129, 199, 200, 255, 256):
        t = toks.copy()
        t[place] = 5
        want = expected(cfg, w, t)
        end = min(n, (place // size + 1) * size)
        moved = err(po.forward(cfg, w, toks), want[0])
        assert moved[place + 1:end].size == 0 or np.median(moved[place + 1:end]) > 5 * np.quantile(want[1], 0.95)
        assert end == n or moved[end:].max() < 1e-9
        state = pkg.RunState(model)
        check(feed(pkg, state, t, [n]), want, compute)
        state.reset()
        cut = max(2, min(place, 190))
        check(feed(pkg, state, t, [cut, 12, 1, 1, 1, 1, 60, 2, 1, 49, 1]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_one_token_stays_in_the_state(pkg, compute):
    """A token whose input gate is wide open, in heads that forget nothing or little: all later tokens carry its value.  Places around the
    chunks of the prompt kernels and the cuts of portions."""
    cfg = pc.config([(pc.mlstm(heads=2, dim=16, vdim=32, cap=9.0), None)], vocab=97, eps=1e-4)
    n = 290
    w, toks = pc.weights(cfg, 51, pos=0.02), pc.tokens(cfg, n, 52)
    toks[toks == 5] = 6
    e5 = w["embed"][5] / np.sqrt((w["embed"][5] ** 2).mean()) * w["l0.norm1"]
    w["l0.mix.i"] = pc.bf16_round(0.3 * w["l0.mix.i"] + np.outer([14.0, 14.0], e5) / (e5 @ e5))
    w["l0.mix.i.b"][:] = -4.0
    w["l0.mix.f"] = pc.bf16_round(0.1 * w["l0.mix.f"])
    w["l0.mix.f.b"][:] = [30.0, 6.0]
    model = build(pkg, cfg, w, n, compute)
    for place in (0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 129, 199, 255, 256):
        t = toks.copy()
        t[place] = 5
        want = expected(cfg, w, t)
        moved = err(po.forward(cfg, w, toks), want[0])
        assert np.median(moved[place:]) > 5 * np.quantile(want[1], 0.95) and (place == 0 or moved[:place].max() < 1e-9)
        state = pkg.RunState(model)
        check(feed(pkg, state, t, [n]), want, compute)
        state.reset()
        check(feed(pkg, state, t, [max(1, place), 40, 1, 2, 128, 1]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_gates_at_their_limits(pkg, compute):
    """Input and forget gates from wide open to shut: the running maximum follows the gates, rises, falls or stays at its start."""
    cfg = pc.config([(pc.mlstm(heads=5, dim=12, vdim=20, cap=15.0), None)])
    w, t = pc.weights(cfg, 61), pc.tokens(cfg, 200, 62)
    w["l0.mix.i.b"][:] = [-80, -80, 80, 0, 80]
    w["l0.mix.f.b"][:] = [-80, 80, 80, -80, -80]
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 200, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [200]), want, compute)
    state.reset()
    check(feed(pkg, state, t, [70, 3, 1, 1, 40]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_prompts_of_several_passes(pkg, compute):
    """A prompt longer than one many-token pass, logits wanted on both sides of the cut, then decode steps with long chunks."""
    cfg = pc.config([(pc.attention(heads=2, kv_heads=1, dim=16, vdim=16, rot=8, scale=0.6, chunk=1100), 40), (pc.mlstm(heads=2, dim=8, vdim=16), None)], width=40, vocab=64, positions=2230)
    n = 2230
    w, t = pc.weights(cfg, 45), pc.tokens(cfg, n, 46)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 5000, compute)  # (more than there are position vectors: the library holds what there are)
    from llama2_jl_b200 import _lib as L
    state = pkg.RunState(model)
    places = [0, 1, 500, 1099, 1100, 2046, 2047, 2048, 2049, 2176]
    check(pkg.extend(state, t[:2177], 0, places), want, compute, places)
    check(np.concatenate([pkg.extend(state, t[p:p + 1], p, [0]) for p in range(2177, n)]), want, compute, slice(2177, n))
    with pytest.raises(L.L2BError):
        pkg.extend(state, t[:1], n, [0])
    assert pkg.prefill(state, t[:2150]) == int(np.argmax(state.logits))
    check(state.logits[None], want, compute, slice(2149, 2150))
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_sessions_are_used_again(pkg, compute):
    """A session keeps nothing of the sequence before, with or without a reset; two sessions do not see one another; a recurrent
    state is not asked for a position it does not stand at."""
    from llama2_jl_b200 import _lib as L
    cfg = pc.CASES["all"]
    w = pc.weights(cfg, 51)
    model = build(pkg, cfg, w, 200, compute)
    a, b = pc.tokens(cfg, 200, 52), pc.tokens(cfg, 77, 53)
    wa, wb = expected(cfg, w, a), expected(cfg, w, b)
    state = pkg.RunState(model)
    first = feed(pkg, state, b, [77])
    check(first, wb, compute)
    feed(pkg, state, a, [200])
    assert np.array_equal(feed(pkg, state, b, [77]), first)  # no reset in between
    feed(pkg, state, a, [3, 1])
    check(feed(pkg, state, b, [1]), wb, compute)
    check(feed(pkg, state, a[:9], [9]), wa, compute, slice(9))
    h = C.c_void_p()
    L.check(L.lib().l2b_session_create(model.device_model().model, None, C.byref(h)))
    other = pkg.RunState(model, h)
    state.reset()
    got_a, got_b, at = [], [], 0
    for n in (40, 30, 1, 1, 5):  # alternating
        got_a.append(pkg.extend(state, a[at:at + n], at, range(n)))
        got_b.append(pkg.extend(other, b[at:at + n], at, range(n)))
        at += n
    check(np.concatenate(got_a), wa, compute, slice(at))
    check(np.concatenate(got_b), wb, compute, slice(at))
    for pos in (at + 1, at - 1):
        for call in (lambda: pkg.extend(state, a[:2], pos), lambda: pkg.extend(state, a[:1], pos), lambda: pkg.transformer_(1, pos, model.config, state)):
            with pytest.raises(L.L2BError, match="recurrent"):
                call()
    check(pkg.extend(state, a[at:at + 5], at, range(5)), wa, compute, slice(at, at + 5))  # (refusals change nothing)
    L.lib().l2b_session_destroy(h)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_batches_of_unequal_sequences(pkg, compute):
    """Sequences of unequal lengths in lock step; a slot whose sequence has ended takes the next one from position 0."""
    from llama2_jl_b200 import _lib as L
    cfg = pc.CASES["all"]
    w = pc.weights(cfg, 61)
    queue = [pc.tokens(cfg, n, 62 + n) for n in (3, 64, 33, 20, 41, 1, 18, 25)]
    want = [expected(cfg, w, s) for s in queue]
    rounding = np.full(80, want[1][1].max())
    model = build(pkg, cfg, w, 80, compute)
    batch = pkg.BatchRunState(model, 3)
    slots, nxt, done = [[i, 0] for i in range(3)], 3, 0
    while done < len(queue):
        got = batch.decode_next([queue[q][p] for q, p in slots], [p for q, p in slots], want_logits=True)
        for i, s in enumerate(slots):
            check(batch.logits[i:i + 1], (want[s[0]][0], rounding), compute, slice(s[1], s[1] + 1))
            assert got[i] == int(np.argmax(batch.logits[i]))
            s[1] += 1
            if s[1] == len(queue[s[0]]):
                done += 1
                s[0], s[1], nxt = (nxt, 0, nxt + 1) if nxt < len(queue) else (1, 0, nxt)
    with pytest.raises(L.L2BError, match="recurrent"):
        batch.decode_next([1, 1, 1], [0, 79, 0])
    batch.reset()
    batch.decode_next([int(queue[0][0])] * 3, [0, 0, 0], want_logits=True)
    check(batch.logits, (np.repeat(want[0][0][:1], 3, 0), rounding[:3]), compute)
    batch.close()
    model.close()


@pytest.mark.gpu
def test_greedy_generation_and_long_decoding(pkg):
    """generate() in 32-bit gives the oracle's greedy stream (500 decoded tokens); sampling is reproducible; the 16-bit stream is
    the argmax of its own logits."""
    cfg = pc.CASES["odd"]
    w, prompt, n = pc.weights(cfg, 71), pc.tokens(cfg, 37, 72), 537
    model = build(pkg, cfg, w, n, "float32")
    got, _ = pkg.generate(model, prompt, n)
    assert np.array_equal(got[:36], prompt[1:])
    fed = np.concatenate([prompt[:1], got[:-1]])
    want = po.forward(cfg, w, fed)
    top = np.sort(want, -1)
    clear = (top[:, -1] - top[:, -2] > 1e-3 * np.abs(want).max()) & (np.arange(n) >= 36)
    assert clear.sum() > 450 and np.array_equal(got[clear], want.argmax(-1)[clear])
    a, _ = pkg.generate(model, prompt, 80, temperature=0.8, seed=5)
    b, _ = pkg.generate(model, prompt, 80, temperature=0.8, seed=5)
    c, _ = pkg.generate(model, prompt, 80, temperature=0.8, seed=6)
    assert np.array_equal(a, b) and not np.array_equal(a, c)
    state = pkg.RunState(model)
    assert pkg.prefill(state, prompt) == got[36]
    check(state.logits[None], (want, None), "float32", slice(36, 37))
    pkg.transformer_(int(got[36]), 37, model.config, state)
    check(state.logits[None], (want, None), "float32", slice(37, 38))
    model.close()
    model = build(pkg, cfg, w, 200, "bfloat16")
    got, _ = pkg.generate(model, prompt, 200)
    state = pkg.RunState(model)
    logits = feed(pkg, state, np.concatenate([prompt[:1], got[:-1]]), [36, 1])
    assert np.array_equal(logits[36:].argmax(-1), got[36:])
    model.close()


@pytest.mark.gpu
def test_folder_and_arguments(pkg, tmp_path):
    from llama2_jl_b200 import _lib as L
    cfg = pc.CASES["all"]
    w, t = pc.weights(cfg, 81), pc.tokens(cfg, 50, 82)
    pc.write_folder(tmp_path, cfg, w)
    model = pkg.load_model(str(tmp_path), seq_len=50, compute="float32")
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [50]), expected(cfg, w, t), "float32")
    assert model.weight_bytes_per_token() > 0 and model.kernels_per_token() > 0
    model.close()
    for change in (lambda x: x.pop("l2.mix.q.b"), lambda x: x.pop("pos"), lambda x: x.update({"l1.mix.f.b": x["l1.mix.f.b"][:-1]})):
        bad = dict(w)
        change(bad)
        pc.write_folder(tmp_path, cfg, bad)
        with pytest.raises(L.L2BError):
            pkg.load_model(str(tmp_path), seq_len=50)
    for layer in (pc.attention(dim=300, vdim=500, heads=1, kv_heads=1), pc.mlstm(dim=1025), pc.mlstm(vdim=1025)):
        with pytest.raises(L.L2BError):
            build(pkg, pc.config([(layer, None)]), {}, 8, "bfloat16").device_model()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_trace_run(pkg, tmp_path, compute):
    """The replay program: requests one after the other, a name used again, wanted places in any order, steps that want nothing."""
    cfg = pc.CASES["odd"]
    w = pc.weights(cfg, 91)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    pc.write_folder(folder, cfg, w)
    a, b = pc.tokens(cfg, 90, 92), pc.tokens(cfg, 21, 93)
    plan = [("x", a, 0, 70, [69, 3]), ("x", a, 70, 88, []), ("x", a, 88, 89, [0]), ("x", a, 89, 90, [0]), ("y", b, 0, 21, [20]), ("x", b, 0, 20, [19])]
    ends = {3: ["x"], 4: ["y"], 5: ["x"]}
    lines = [json.dumps(dict(step=i, entries=[dict(id=n, tokens=[int(v) for v in s[lo:hi]], want=want)], end=ends.get(i, []))) for i, (n, s, lo, hi, want) in enumerate(plan)]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", compute, "--out", str(out), "--max-tokens", "90"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    for i, (n, s, lo, hi, want) in enumerate(plan):
        path = out / f"{i}.f32"
        assert path.exists() == bool(want)
        if want:
            check(np.fromfile(path, "<f4").reshape(len(want), -1), expected(cfg, w, s), compute, [lo + k for k in want])
