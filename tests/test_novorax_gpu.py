"""Whole Novorax models on the GPU through the framework's own entry points, against the plain float64 restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import novorax_models as vm
from oracle import plain_novorax as pn

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CONFIGS = {
    # layer orders, repeated groups, windows, experts, gate caps and sizes all differ; some layers have no feed-forward
    "a": vm.config([vm.latent(3, 24, 8, 16, 20, 28, 11, vm.moe(5, 2, 24)), vm.mlstm(2, 20, 12, 6.0, vm.dense(40)),
                    vm.latent(2, 16, 16, 24, 33, 40, 7, vm.dense(56), name="latent_attention_2", rotation=vm.rot(16, 500.0, (2.0, 32, 4.0, 1.0)))],
                   width=72, vocab=101, loop=(1, 3, 3)),
    "b": vm.config([vm.mlstm(3, 12, 20, 9.0, None), vm.latent(4, 32, 8, 32, 24, 48, None, vm.dense(33)), vm.mlstm(2, 8, 8, 3.0, vm.dense(17), name="mlstm_2")],
                   width=50, vocab=67, eps=1e-3, logit_scale=1.5),
    "c": vm.config([vm.latent(4, 64, 32, 48, 72, 80, 70, vm.dense(160)), vm.mlstm(2, 64, 96, 14.0, vm.moe(4, 3, 64)), vm.latent(8, 32, 16, 64, 40, 128, 48, vm.moe(12, 1, 40))],
                   width=192, vocab=300, loop=(0, 3, 2), logit_scale=0.8),
    "d": vm.config([vm.latent(1, 8, 2, 8, 8, 8, 1, vm.moe(3, 3, 9)), vm.mlstm(1, 8, 8, 2.0, vm.dense(9))], width=16, vocab=40, loop=(0, 1, 1)),
    "e": vm.config([vm.mlstm(4, 16, 40, 20.0, vm.moe(7, 2, 30)), vm.latent(5, 20, 12, 28, 36, 52, 16, None, rotation=vm.rot(12, 77.0, None))],
                   width=84, vocab=53, loop=(1, 2, 4), eps=1e-6),
}
# Worst position and median.  The models are narrow (down to 16), so bfloat16 rounding averages little, and a norm behind a
# sublayer whose output nearly cancels makes it large at single positions, in whatever portions they come.
TOL = {"float32": 1e-4, "bfloat16": 0.6}
MEDIAN = {"float32": 1e-5, "bfloat16": 0.08}


class Case:
    def __init__(self, folder, name):
        self.cfg = CONFIGS[name]
        self.w = vm.write_model(folder, self.cfg, vm.make_weights(self.cfg, seed=ord(name)))
        self.path, self.models = folder, {}

    def model(self, dtype="float32", context=512):
        from wick_b200.model import load_model_cuda
        if (dtype, context) not in self.models:
            self.models[dtype, context] = load_model_cuda(self.path, context, 0, dtype)
        return self.models[dtype, context]

    def tokens(self, n, seed=0):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], n).tolist()

    def want(self, tokens):
        return pn.forward(self.cfg, self.w, tokens)


@pytest.fixture(scope="module")
def cases(cuda_lib, tmp_path_factory):
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    made = {}

    def get(name):
        if name not in made:
            made[name] = Case(str(tmp_path_factory.mktemp("novorax_" + name)), name)
        return made[name]
    yield get
    for c in made.values():
        for m in c.models.values():
            m.close()


def check(got, want, dtype, what=""):
    err = np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want ** 2))
    assert np.isfinite(got).all() and err.max() < TOL[dtype], f"{what}: {err.max():.2e} at {int(err.argmax())}"
    assert len(err) < 20 or np.median(err) < MEDIAN[dtype], f"{what}: median {np.median(err):.2e}"


def run_portions(m, toks, portions):
    """Logits of every position, fed in portions (single tokens as decode steps)."""
    s, at, out = m.seq_create(), 0, []
    i = 0
    while at < len(toks):
        p = toks[at:at + portions[i % len(portions)]]
        if len(p) == 1 and at:
            out.append(m.decode_batch_logits(p, [s]))
        else:
            out.append(m.seq_prefill_logits(s, p, at, range(len(p))))
        at += len(p)
        i += 1
    assert m.seq_length(s) == len(toks)
    m.seq_destroy(s)
    return np.concatenate(out)


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("dtype", TOL)
def test_prompt(cases, name, dtype):
    c = cases(name)
    toks = c.tokens(180)
    check(run_portions(c.model(dtype), toks, (len(toks),)), c.want(toks), dtype)
    conf = c.model(dtype).config()
    assert conf.block_types == tuple(l["type"] for l in c.cfg["layers"]) and conf.architecture == "Novorax"
    assert [bool(k) for k in conf.kv_heads_per_layer] == [l["type"].startswith("latent") for l in c.cfg["layers"]]


@pytest.mark.parametrize("name,portions", [("a", (1,)), ("b", (1,)), ("c", (100, 1, 1, 1)), ("a", (2,)), ("b", (2, 3, 1, 17)), ("c", (2, 64, 7, 1)),
                                           ("d", (5, 1)), ("c", (9, 8)), ("e", (1,)), ("e", (63, 2, 65, 1)), ("a", (16, 15))])
@pytest.mark.parametrize("dtype", TOL)
def test_portions_and_decoding(cases, name, portions, dtype):
    c = cases(name)
    toks = c.tokens(150, seed=1)
    check(run_portions(c.model(dtype), toks, portions), c.want(toks), dtype)


@pytest.mark.parametrize("dtype", TOL)
def test_internal_chunks(cases, monkeypatch, dtype):
    """A call longer than the scratch is cut into pieces inside the library."""
    monkeypatch.setenv("WICK_CUDA_MAX_CHUNK", "48")
    c = cases("c")
    m = c.model(dtype, 400)
    monkeypatch.delenv("WICK_CUDA_MAX_CHUNK")
    toks = c.tokens(333, seed=2)
    check(run_portions(m, toks, (len(toks),)), c.want(toks), dtype)


@pytest.mark.parametrize("name", ["a", "e"])
@pytest.mark.parametrize("dtype", TOL)
def test_batches_of_unequal_requests(cases, dtype, name):
    """Rows of a batch equal the same sequence alone; slots are freed and used again in between."""
    c = cases(name)
    m = c.model(dtype)
    lens = [1, 90, 13, 40, 2, 64, 7, 30, 5, 18, 77]
    seqs = [c.tokens(n + 25, seed=10 + i) for i, n in enumerate(lens)]
    want = [c.want(s) for s in seqs]
    for used in (m.seq_create(), m.seq_create()):     # leave something behind in the first slots
        m.seq_prefill(used, c.tokens(120, seed=99), 0)
        m.seq_destroy(used)
    ids = []
    for s, n in zip(seqs, lens):
        ids.append(m.seq_create())
        check(m.seq_prefill(ids[-1], s[:n], 0)[None], want[len(ids) - 1][n - 1:n], dtype, "prompt")
    order = np.random.default_rng(4)
    at = list(lens)
    for step in range(20):
        rows = order.permutation(len(ids))[: 1 + step % len(ids)]
        got = m.decode_batch_logits([seqs[r][at[r]] for r in rows], [ids[r] for r in rows])
        for k, r in enumerate(rows):
            check(got[k:k + 1], want[r][at[r]:at[r] + 1], dtype, f"step {step} sequence {r}")
            at[r] += 1
        if step == 9:           # one request ends, another takes its slot
            m.seq_destroy(ids[3])
            again = m.seq_create()
            assert again == ids[3]
            at[3] = 6
            check(m.seq_prefill_logits(again, seqs[3][:6], 0, [5, 0, 5]), want[3][[5, 0, 5]], dtype, "slot used again")
    for s in ids:
        m.seq_destroy(s)


def test_rows_of_a_batch_do_not_depend_on_the_batch(cases):
    """The same sequence in wide batches: neighbours and places change nothing beyond rounding (here, many row groups)."""
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 0.05)):
        c = cases("d")
        m = c.model(dtype)
        ids = [m.seq_create() for _ in range(150)]
        prompts = [c.tokens(3 + i % 5, seed=i % 7) for i in range(150)]
        for s, p in zip(ids, prompts):
            m.seq_prefill(s, p, 0)
        got = m.decode_batch_logits([i % 7 for i in range(150)], ids)
        for i in range(150):
            want = c.want(prompts[i] + [i % 7])[-1]
            assert np.sqrt(np.mean((got[i] - want) ** 2)) < (TOL[dtype] * np.sqrt(np.mean(want ** 2)))
            assert np.abs(got[i] - got[i % 35]).max() <= tol
        for s in ids:
            m.seq_destroy(s)


def greedy(c, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(np.argmax(c.want(toks)[-1])))
    return toks[-n:]


@pytest.mark.parametrize("name", ["a", "b"])
def test_greedy_generation_and_own_sequence(cases, name):
    """forward_prefill, forward, forward_greedy, generate_greedy, decode_batch_steps and sampling give the tokens of the plain
    model, with the model's own sequence and slots side by side."""
    from wick_b200.model import InferenceState
    c = cases(name)
    m = c.model()
    p1, p2 = c.tokens(60, seed=20), c.tokens(9, seed=21)
    g1, g2 = greedy(c, p1, 12), greedy(c, p2, 12)
    st = InferenceState()
    first = int(np.argmax(m.forward_prefill(p1, 0, st)))
    slot = m.seq_create()
    f2 = int(np.argmax(m.seq_prefill(slot, p2, 0)))
    assert [first] + list(m.generate_greedy(first, 11, st)) == g1
    other = m.seq_create()
    m.seq_prefill(other, p1, 0)
    out = m.decode_batch_steps([f2, first], [slot, other], 11)
    assert [f2] + list(out[:, 0]) == g2 and [first] + list(out[:, 1]) == g1
    m.forward_prefill(p1, 0, st)
    tok, got = first, [first]
    for i in range(11):
        pos = len(p1) + i
        if i % 3 == 0:
            tok = int(np.argmax(m.forward([tok], pos, st)))
        elif i % 3 == 1:
            tok = m.forward_greedy([tok], pos, st)
        else:
            tok = m.forward_sample([tok], pos, st, 0.8, 1, 1.0, 0.5)
        got.append(tok)
    assert got == g1
    m.seq_destroy(slot)
    m.seq_destroy(other)


def test_long_decoding(cases):
    """Hundreds of decoded tokens: windows pass over decoded tokens, the states do not drift."""
    for name in ("a", "e"):
        c = cases(name)
        toks = c.tokens(420, seed=30)
        got = run_portions(c.model(), toks, (5,) + (1,) * 600)
        check(got, c.want(toks), "float32", name)


def test_snapshot_and_embedding_input(cases):
    from wick_b200._lib import WickCudaError
    from wick_b200.model import InferenceState
    c = cases("b")
    m = c.model()
    st = InferenceState()
    toks = c.tokens(80, seed=40)
    want = c.want(toks)
    m.forward_prefill(toks[:50], 0, st)
    snap = m.snapshot_state()
    m.forward_prefill(c.tokens(33, seed=41), 0, st)
    m.restore_state(snap, st)
    assert st.seq_len == 50
    check(m.forward_prefill(toks[50:], 50, st)[None], want[-1:], "float32", "after restore")
    frames = c.w["embed"][toks].astype(np.float32)
    check(m.forward_prefill_from_embeddings(frames, len(toks), 0, st)[None], want[-1:], "float32", "frames")
    m.forward_prefill(toks[:-1], 0, st)
    hid = m.forward_embedding([toks[-1]], 79, st)
    check((c.w["head"] @ hid.astype(np.float64) * c.cfg["logit_scale"])[None], want[-1:], "float32", "hidden row")
    # experts are chosen by token id, so rows without ids are refused
    c = cases("a")
    m = c.model()
    with pytest.raises(WickCudaError, match="token id"):
        m.forward_prefill_from_embeddings(np.zeros((3, 72), np.float32), 3, 0, InferenceState())
    # a restored sequence of a model with a repeated group: every pass has its own state
    toks = c.tokens(70, seed=42)
    st = InferenceState()
    m.forward_prefill(toks[:40], 0, st)
    snap = m.snapshot_state()
    m.forward_prefill(toks[:7], 0, st)
    m.restore_state(snap, st)
    check(m.forward_prefill(toks[40:], 40, st)[None], c.want(toks)[-1:], "float32", "restored passes")


def test_misuse(cases):
    from wick_b200._lib import WickCudaError
    from wick_b200.model import InferenceState
    c = cases("d")
    m = c.model("float32", 20)
    s = m.seq_create()
    with pytest.raises(WickCudaError):
        m.seq_prefill(s, [c.cfg["vocab"]], 0)
    m.seq_prefill(s, [1] * 20, 0)
    with pytest.raises(WickCudaError) as e:
        m.decode_batch([1], [s])
    assert e.value.code == -5
    assert not m.supports_kv_shift()
    m.forward_prefill([1, 2, 3], 0, InferenceState())
    with pytest.raises(WickCudaError):
        m.shift_kv(InferenceState(3), 1, 1)
    m.seq_destroy(s)


def mistakes():
    """Plain forwards with one fault each, to show that the comparisons above would notice."""
    def patched(name, fn):
        def run(cfg, w, toks):
            old = getattr(pn, name)
            setattr(pn, name, fn(old))
            try:
                return pn.forward(cfg, w, toks)
            finally:
                setattr(pn, name, old)
        return run

    def edited(key, fn):
        return lambda cfg, w, toks: pn.forward(cfg, {k: (fn(v) if k.endswith(key) else v) for k, v in w.items()}, toks)
    yield "window one longer", patched("visible", lambda f: lambda n, s: f(n, s + 1))
    yield "window one shorter", patched("visible", lambda f: lambda n, s: f(n, max(s - 1, 1)))
    yield "no sink", edited(".sink", lambda v: v - 50.0)
    yield "no size of the rotation", patched("rotary_frequencies", lambda f: lambda d, b, s: (f(d, b, s)[0], 1.0))
    yield "frequencies not scaled", patched("rotary_frequencies", lambda f: lambda d, b, s: (f(d, b, None)[0], f(d, b, s)[1]))
    yield "halves instead of neighbours", patched("rotate", lambda f: lambda x, d, fr, c: np.concatenate(
        [f(x[..., :d].reshape(x.shape[:-1] + (2, d // 2)).swapaxes(-1, -2).reshape(x.shape[:-1] + (d,)), d, fr, c), x[..., d:]], axis=-1))
    yield "passes alike", edited("loop.step", lambda v: 0.0 * v)
    yield "embedding not fed again", edited("loop.in", lambda v: np.concatenate([v[:, :v.shape[0]], 0 * v[:, v.shape[0]:]], 1))
    yield "gains around one", patched("norm", lambda f: lambda x, w, eps: f(x, w - 1.0, eps))
    yield "always the same expert", edited(".table", lambda v: np.sort(np.zeros_like(v) + np.arange(v.shape[1]), axis=1))
    yield "nothing forgotten", patched("matrix_memory", lambda f: lambda q, k, v, i, g: f(q, k, v, i, 0.0 * g))
    yield "gates not clipped", patched("soft_clip", lambda f: lambda z, cap: z)
    yield "logits not scaled", lambda cfg, w, toks: pn.forward({**cfg, "logit_scale": 1.0}, w, toks)


def test_faults_would_show(cases):
    c = cases("a")
    toks = c.tokens(60, seed=50)
    got = run_portions(c.model(), toks, (60,))
    check(got, c.want(toks), "float32")
    for what, fn in mistakes():
        err = np.sqrt(np.mean((got - fn(c.cfg, c.w, toks)) ** 2)) / np.sqrt(np.mean(got ** 2))
        assert err > 20 * TOL["float32"], f"{what} changes the logits by {err:.1e} only"


def test_trace_runner(cases, tmp_path):
    """bin/trace_run in a process of its own: portions, decode steps, interleaved requests, slots given back."""
    c = cases("e")
    a, b = c.tokens(40, seed=60), c.tokens(25, seed=61)
    wa, wb = c.want(a), c.want(b)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[17:18], "want": [0]}, {"id": "b", "tokens": b[2:3], "want": [0]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[18:], "want": [21, 3]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "b", "tokens": b[3:], "want": [20]}], "end": ["b"]},
    ]
    expect = {0: wa[[0, 16]], 2: np.stack([wa[17], wb[2]]), 3: wa[[39, 21]], 4: wb[[23]]}
    for dtype in TOL:
        out = tmp_path / dtype
        out.mkdir()
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", c.path, "--dtype", dtype, "--out", str(out), "--max-tokens", "70"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(5)]
        assert sorted(os.listdir(out)) == [f"{i}.f32" for i in expect]
        for i, want in expect.items():
            check(np.fromfile(out / f"{i}.f32", "<f4").reshape(want.shape), want, dtype, f"step {i}")


def test_command_line(cases):
    c = cases("a")
    prompt = c.tokens(20, seed=70)
    want = greedy(c, prompt, 6)
    p = subprocess.run([sys.executable, "-m", "wick_b200", "generate", "--model", c.path, "--dtype", "float32", "--tokens", ",".join(map(str, prompt)),
                        "--count", "6", "--context", "64"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.split() == [str(t) for t in want]
    p = subprocess.run([sys.executable, "-m", "wick_b200", "info", "--model", c.path], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0 and "architecture Novorax: 3 layers" in p.stdout and "mlstm" in p.stdout
