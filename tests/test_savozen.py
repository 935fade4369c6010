"""Savozen: configuration and registry, what the test models can show (CPU), and the library against the plain oracle (GPU)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import savozen_cases as sc
import savozen_oracle as so
from stack_common import COMPUTE, bf16, build, check, err, feed

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def expected(cfg, w, toks):
    """(exact logits, error of every position when operands are rounded to bf16)."""
    want = so.forward(cfg, w, toks)
    return want, err(so.forward(cfg, w, toks, operand=bf16), want)


# ---- CPU -------------------------------------------------------------------------------------------
def create(pkg, raw, compute=None):
    from llama2_jl_b200 import _lib as L
    h = C.c_void_p()
    st = L.lib().l2b_model_create_stack(json.dumps(raw).encode(), 16, L.TYPE_F32 if compute is None else compute, -1, None, C.byref(h))
    msg = L.lib().l2b_last_error_string().decode()
    if h:
        L.lib().l2b_model_destroy(h)
    return st, msg


def test_configurations_are_checked(pkg):
    from llama2_jl_b200 import _lib as L
    good = sc.CASES["all"]
    assert create(pkg, good)[0] in (L.OK, L.ERR_NO_DEVICE)
    assert create(pkg, dict(good, loop=None, token_side=None))[0] in (L.OK, L.ERR_NO_DEVICE)

    def broken(change):
        raw = json.loads(json.dumps(good))
        change(raw)
        return create(pkg, raw)
    for change, word in [(lambda r: r.update(architecture="Other"), "Other"), (lambda r: r.pop("vocab"), "vocab"),
                         (lambda r: r["layers"][1].update(type="convolution"), "convolution"), (lambda r: r["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
                         (lambda r: r["layers"][0]["mixer"].update(heads=1.5), "heads"), (lambda r: r["layers"][0]["mlp"].update(kind="experts"), "experts"),
                         (lambda r: r["loop"].update(stop=9), "loop"), (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=64), "rot"),
                         (lambda r: r.update(layers=[]), "layers"), (lambda r: r["norm"].pop("eps"), "eps")]:
        st, msg = broken(change)
        assert st == L.ERR_BAD_ARG and word in msg, (st, msg)
    assert create(pkg, good, L.TYPE_Q4_K)[0] == L.ERR_UNSUPPORTED_TYPE
    assert L.lib().l2b_model_create_stack(b"{not json", 16, L.TYPE_F32, -1, None, C.byref(C.c_void_p())) == L.ERR_BAD_ARG


def test_registry_and_layer_order(pkg, tmp_path):
    from llama2_jl_b200 import load_stack
    sc.write_folder(tmp_path, dict(sc.CASES["all"], architecture="Unheard"), {})
    with pytest.raises(ValueError, match="Unheard"):
        pkg.load_model(str(tmp_path), seq_len=8)
    assert "Savozen" in load_stack.ARCHITECTURES
    with pytest.raises(ValueError):
        pkg.StackConfig(sc.CASES["all"], 8, "float16").compute_type()
    assert so.layer_runs(sc.CASES["all"]) == [(0, None), (1, 0), (2, None), (1, 1), (2, None)]
    assert so.layer_runs(sc.CASES["no_loop_no_side"]) == [(0, None), (1, None)]


def test_bf16_bits(pkg):
    from llama2_jl_b200.model import bf16_bits
    a = np.random.default_rng(0).standard_normal(1000).astype(np.float32)
    r = sc.bf16_round(a)
    assert np.array_equal((bf16_bits(a).astype(np.uint32) << 16).view(np.float32), r)
    assert np.array_equal(bf16_bits(r).astype(np.uint32) << 16, r.view(np.uint32))


def test_rotation_turns_pairs():
    v = np.arange(12, dtype=np.float64).reshape(1, 2, 6)
    r = so.rotate_interleaved(v, np.array([0.0, 3.0]), 100.0, 4)
    assert np.array_equal(r[0, 0], v[0, 0]) and np.array_equal(r[0, 1, 4:], v[0, 1, 4:])
    for i, f in enumerate((1.0, 0.1)):
        z = complex(v[0, 1, 2 * i], v[0, 1, 2 * i + 1]) * np.exp(1j * 3.0 * f)
        assert np.allclose(r[0, 1, 2 * i:2 * i + 2], [z.real, z.imag])


MISTAKES = {
    "no sink": lambda mp: mp.setattr(so, "sink_softmax", lambda s, k: np.exp(s - s.max(-1, keepdims=True)) / np.exp(s - s.max(-1, keepdims=True)).sum(-1, keepdims=True)),
    "positions from 1": lambda mp: mp.setattr(so, "rotate_interleaved", lambda v, p, b, d, f=so.rotate_interleaved: f(v, p + (v.ndim == 3), b, d)),
    "no gate": lambda mp: mp.setattr(so, "sigmoid", lambda z: np.ones_like(z)),
    "last key hidden": lambda mp: mp.setattr(np, "tril", lambda m, f=np.tril: f(m, -1) | (np.arange(m.shape[0])[None] == 0)),
    "plain gelu": lambda mp: mp.setattr(so, "gelu_tanh", lambda z: z * (z > 0)),
    "no norm of the token input": lambda mp: mp.setattr(so, "token_side", lambda x, e, g, p, n, eps, operand=None: x + ((so.gelu_tanh(x @ g.T) * e) @ p.T) * n),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_the_models_show_mistakes(mistake, monkeypatch):
    """A mistake planted in the oracle moves the logits of the test model far beyond the limits of the 16-bit comparison."""
    cfg = sc.CASES["all"]
    w, t = sc.weights(cfg, 1), sc.tokens(cfg, 70, 2)
    want, rounding = expected(cfg, w, t)
    MISTAKES[mistake](monkeypatch)
    assert np.median(err(so.forward(cfg, w, t), want)) > 5 * np.median(rounding)


def test_trace_run_says_what_it_takes():
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--help"], capture_output=True, text=True)
    assert r.returncode == 0 and "--max-tokens" in r.stdout
    assert os.access(os.path.join(ROOT, "bin", "trace_run"), os.X_OK)


# ---- GPU -------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("case", list(sc.CASES))
def test_prompt_decode_and_portions(pkg, case, compute):
    """Whole prompt, token by token, a prompt then single tokens, and portions of several sizes, all against the oracle; sizes around
    the tile of the prompt kernels (128), the switch between its two forms of attention, and portions of two tokens."""
    cfg = sc.CASES[case]
    w, t = sc.weights(cfg, 11), sc.tokens(cfg, 301, 12)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 301, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [301]), want, compute)
    for sizes in ([1], [200, 1], [2], [3, 50, 2, 128, 1, 47, 48, 64], [129, 127, 2], [17]):
        state.reset()
        n = 140 if sizes in ([1], [2]) else 301
        check(feed(pkg, state, t[:n], sizes), want, compute, slice(n))
    model.close()


def only(cfg, w, keep):
    """Weights whose other mechanisms are silent: residual contributions not named in `keep` are zero."""
    w = {k: v.copy() for k, v in w.items()}
    for k in w:
        part = {".mix.o": "mix", ".mlp.down": "mlp", ".side.norm": "side", "loop.step": "step"}
        for suffix, name in part.items():
            if k.endswith(suffix) and name not in keep:
                w[k][:] = 0
    return w


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("keep", ["", "mix", "mlp", "side", "step", "mix step", "mlp side"])
def test_mechanisms_alone(pkg, keep, compute):
    """Embedding scale, norm and head alone; then one mechanism at a time on top."""
    cfg = sc.CASES["all"]
    w, t = only(cfg, sc.weights(cfg, 21), keep.split()), sc.tokens(cfg, 90, 22)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 90, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [90]), want, compute)
    state.reset()
    check(feed(pkg, state, t, [30, 1]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
@pytest.mark.parametrize("sink", [-40.0, 0.0, 6.0, 60.0])
def test_sinks(pkg, sink, compute):
    """From a sink that weighs nothing to one that takes everything."""
    cfg = sc.config([(sc.mixer(heads=2, scale=0.3), None)])
    w, t = sc.weights(cfg, 31), sc.tokens(cfg, 150, 32)
    w["l0.mix.sink"][:] = [sink, sink / 2]
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, 150, compute)
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [150]), want, compute)
    state.reset()
    check(feed(pkg, state, t, [5, 60, 2, 1]), want, compute)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_one_far_key_stands_out(pkg, compute):
    """One early token's key is aligned with what a late token asks for: the late logits are those of the value at that place, and
    follow the place.  Places at and around tile borders, asked for from a prompt and from single decode steps."""
    cfg = sc.config([(sc.mixer(heads=2, dim=32, rot_dim=16, vdim=32, kv_rank=64, scale=1.0), None)], vocab=97)
    n = 420
    for place in (0, 1, 63, 127, 128, 129, 255, 256, 300):
        w, t = sc.weights(cfg, 41, sharp=1.0), sc.tokens(cfg, n, 42)
        t[t == 5] = 6
        t[t == 9] = 10
        t[place] = 5                      # the key
        t[[310, 383, 384, 400, n - 1]] = 9  # who asks for it
        W = {k: np.asarray(v, np.float64) for k, v in w.items()}

        def h(tok):
            return so.dynamic_tanh(W["embed"][tok] * cfg["embedding"]["scale"], W["l0.norm1.alpha"], W["l0.norm1"], W["l0.norm1.b"])
        c = so.rms_norm((W["l0.mix.dkv"] @ h(5))[:64], W["l0.mix.dkv.norm"], cfg["norm"]["eps"])
        q = w["l0.mix.q"].reshape(2, 48, -1)
        ask = h(9)
        for head in range(2):  # unrotated query of token 9 = a multiple of the unrotated key of token 5
            key = W["l0.mix.uk"].reshape(2, 32, 64)[head] @ c
            q[head, :32] += np.outer(key * 40 / (key @ key) - q[head, :32] @ ask, ask) / (ask @ ask)
        w["l0.mix.q"] = sc.bf16_round(q.reshape(96, -1))
        want = expected(cfg, w, t)
        late = [310, 383, 384, 400, n - 1]
        moved = so.forward(cfg, w, np.where(np.arange(n) == place, 6, t))
        assert np.median(err(moved[late], want[0][late])) > 5 * want[1].max()  # without the key the late logits are others
        model = build(pkg, cfg, w, n, compute)
        state = pkg.RunState(model)
        check(feed(pkg, state, t, [n])[late], want, compute, late)
        state.reset()
        check(feed(pkg, state, t, [300, 10, 1])[late], want, compute, late)
        model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_prompts_of_several_passes(pkg, compute):
    """A prompt longer than one many-token pass, logits wanted on both sides of the cut, then decode steps whose ranges of positions
    are longer than the shortest one."""
    cfg = sc.config([(sc.mixer(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=24, scale=0.5), 40)], width=40, vocab=64, side=8)
    n = 2230
    w, t = sc.weights(cfg, 45), sc.tokens(cfg, n, 46)
    want = expected(cfg, w, t)
    model = build(pkg, cfg, w, n, compute)
    state = pkg.RunState(model)
    places = [0, 1, 500, 2046, 2047, 2048, 2049, 2199]
    check(pkg.extend(state, t[:2200], 0, places), want, compute, places)
    got = [pkg.extend(state, t[p:p + 1], p, [0]) for p in range(2200, n)]
    check(np.concatenate(got), want, compute, slice(2200, n))
    assert pkg.prefill(state, t[:2150]) == int(np.argmax(state.logits))
    check(state.logits[None], want, compute, slice(2149, 2150))
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_sessions_are_used_again(pkg, compute):
    """A session's cache holds nothing of the sequence before, with or without a reset; two sessions do not see one another."""
    from llama2_jl_b200 import _lib as L
    cfg = sc.CASES["all"]
    w = sc.weights(cfg, 51)
    model = build(pkg, cfg, w, 200, compute)
    a, b = sc.tokens(cfg, 200, 52), sc.tokens(cfg, 77, 53)
    wa, wb = expected(cfg, w, a), expected(cfg, w, b)
    state = pkg.RunState(model)
    first = feed(pkg, state, b, [77])
    check(first, wb, compute)
    feed(pkg, state, a, [200])
    assert np.array_equal(feed(pkg, state, b, [77]), first)  # no reset in between
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
    L.lib().l2b_session_destroy(h)
    model.close()


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_batches_of_unequal_sequences(pkg, compute):
    cfg = sc.CASES["all"]
    w = sc.weights(cfg, 61)
    lens = [1, 9, 33, 20]
    seqs = [sc.tokens(cfg, n, 62 + n) for n in lens]
    want = [expected(cfg, w, s) for s in seqs]
    model = build(pkg, cfg, w, 40, compute)
    batch = pkg.BatchRunState(model, len(seqs))
    for rounds in range(2):  # the second time on caches that were used before
        for p in range(max(lens)):
            toks = [s[min(p, len(s) - 1)] for s in seqs]
            nxt = batch.decode_next(toks, [min(p, len(s) - 1) for s in seqs], want_logits=True)
            for i, s in enumerate(seqs):
                if p < len(s):
                    check(batch.logits[i:i + 1], (want[i][0], want[2][1]), compute, slice(p, p + 1))
                    assert nxt[i] == int(np.argmax(batch.logits[i]))
        batch.reset()
    batch.close()
    model.close()


@pytest.mark.gpu
def test_greedy_generation_and_long_decoding(pkg):
    """generate() in 32-bit gives the oracle's greedy stream (500 decoded tokens); sampling is reproducible; the 16-bit stream is
    the argmax of its own logits."""
    cfg = sc.CASES["odd"]
    w, prompt, n = sc.weights(cfg, 71), sc.tokens(cfg, 37, 72), 537
    model = build(pkg, cfg, w, n, "float32")
    got, _ = pkg.generate(model, prompt, n)
    assert np.array_equal(got[:36], prompt[1:])
    fed = np.concatenate([prompt[:1], got[:-1]])
    want = so.forward(cfg, w, fed)
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
    cfg = sc.CASES["all"]
    w, t = sc.weights(cfg, 81), sc.tokens(cfg, 50, 82)
    sc.write_folder(tmp_path, cfg, w)
    model = pkg.load_model(str(tmp_path), seq_len=50, compute="float32")
    state = pkg.RunState(model)
    check(feed(pkg, state, t, [50]), expected(cfg, w, t), "float32")
    assert model.weight_bytes_per_token() > 0 and model.kernels_per_token() > 0
    with pytest.raises(L.L2BError):
        pkg.extend(state, t[:2], 49, [0])       # beyond seq_len
    with pytest.raises(L.L2BError):
        pkg.extend(state, t[:4], 0, [2, 1])     # places must ascend
    with pytest.raises(L.L2BError):
        pkg.extend(state, [cfg["vocab"]], 0, [])
    model.close()
    for change in (lambda x: x.pop("l1.mix.sink"), lambda x: x.update({"head": x["head"][:-1]})):
        bad = dict(w)
        change(bad)
        sc.write_folder(tmp_path, cfg, bad)
        with pytest.raises(L.L2BError):
            pkg.load_model(str(tmp_path), seq_len=50)
    (tmp_path / "model.safetensors").write_bytes(b"\x10" * 40)
    with pytest.raises(L.L2BError):
        pkg.load_model(str(tmp_path), seq_len=50)


@pytest.mark.gpu
@pytest.mark.parametrize("compute", COMPUTE)
def test_trace_run(pkg, tmp_path, compute):
    """The replay program: requests one after the other, a name used again, wanted places in any order, steps that want nothing."""
    cfg = sc.CASES["odd"]
    w = sc.weights(cfg, 91)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    sc.write_folder(folder, cfg, w)
    a, b = sc.tokens(cfg, 60, 92), sc.tokens(cfg, 21, 93)
    plan = [("x", a, 0, 40, [39, 3]), ("x", a, 40, 58, []), ("x", a, 58, 59, [0]), ("x", a, 59, 60, [0]), ("y", b, 0, 21, [20]), ("x", b, 0, 20, [19])]
    ends = {3: ["x"], 4: ["y"], 5: ["x"]}
    lines = [json.dumps(dict(step=i, entries=[dict(id=n, tokens=[int(v) for v in s[lo:hi]], want=want)], end=ends.get(i, []))) for i, (n, s, lo, hi, want) in enumerate(plan)]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", compute, "--out", str(out), "--max-tokens", "60"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    for i, (n, s, lo, hi, want) in enumerate(plan):
        path = out / f"{i}.f32"
        assert path.exists() == bool(want)
        if want:
            check(np.fromfile(path, "<f4").reshape(len(want), -1), expected(cfg, w, s), compute, [lo + k for k in want])


@pytest.mark.gpu
def test_extend_on_a_llama_model(pkg, synth):
    """The portion entry point serves the other models too: the same logits as one transformer_ call per position."""
    spec = synth.scaled(synth.LLAMA3_8B_Q4_K_S, n_layers=1, vocab_size=1024, seq_len=64)
    cfg = spec["config"]
    model = pkg.LanguageModel(cfg, None, synth.model_weights(cfg, spec["types"], seed=9))
    t = synth.tokens(40, 6, 3, 1024)
    state = pkg.RunState(model)
    want = []
    for p in range(40):
        pkg.transformer_(int(t[p]), p, cfg, state)
        want.append(state.logits.copy())
    state = pkg.RunState(model)
    got = np.concatenate([pkg.extend(state, t[:30], 0, [0, 7, 29]), pkg.extend(state, t[30:39], 30), pkg.extend(state, t[39:], 39, [0])])
    assert err(got, np.stack([want[i] for i in (0, 7, 29, 39)]).astype(np.float64)).max() < 2e-5
    model.close()
