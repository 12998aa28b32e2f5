"""Each Novorax mechanism alone on the GPU, through the operator entry points, against the plain float64 restatement."""
import numpy as np
import pytest

from oracle import plain_novorax as pn

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def ops(cuda_lib):
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    from wick_b200 import ops
    return ops


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype).cuda()


def host(t):
    return t.detach().double().cpu().numpy()


def error(got, want):
    got, want = host(got) if torch.is_tensor(got) else got, np.asarray(want)
    assert np.isfinite(got).all()
    return np.abs(got - want).max() / (np.sqrt(np.mean(want ** 2)) + 1e-30)


def close(got, want, tol, what=""):
    assert error(got, want) < tol, f"{what}: {error(got, want):.2e} of the rms"


def row_error(got, want):
    """Largest root mean square error of a row, over the rms of everything."""
    got = host(got) if torch.is_tensor(got) else got
    assert np.isfinite(got).all()
    return np.sqrt(np.mean((got - want) ** 2, axis=1)).max() / (np.sqrt(np.mean(want ** 2)) + 1e-30)


TYPES = {"f32": torch.float32, "bf16": torch.bfloat16}


# ── dense matrices ─────────────────────────────────────────────────────────
@pytest.mark.parametrize("path,dtype,n", [("rows", "bf16", 3), ("f32", "f32", 70), ("tensor", "bf16", 150)])
def test_dense_activations(ops, path, dtype, n):
    rng = np.random.default_rng(n)
    m, k = 137, 72
    w, x = dev(rng.standard_normal((m, k)) * k ** -0.5, torch.bfloat16), dev(rng.standard_normal((n, k)), TYPES[dtype])
    z = host(x) @ host(w).T
    close(ops.dense(w, x, activation="relu2", path=path), np.maximum(z, 0) ** 2, 1e-4, "square of relu")
    close(ops.dense(w, x, activation="relu", path=path), np.maximum(z, 0), 1e-4, "relu")
    close(ops.dense(w, x, activation="silu", path=path), pn.silu(z), 1e-4, "silu")
    close(ops.dense(w, x, activation="none", path=path), z, 1e-4, "none")


# ── residual and norms ─────────────────────────────────────────────────────
@pytest.mark.parametrize("width,n", [(24, 3), (33, 5), (320, 2), (1024, 40), (1500, 4), (4096, 3), (8192, 2), (9000, 2)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_residual_norm(ops, width, n, dtype):
    rng = np.random.default_rng(width)
    dt, tol, eps = TYPES[dtype], 2e-2 if dtype == "bf16" else 1e-5, 0.3   # (a large eps, so that its place shows)
    x0 = rng.standard_normal((n, width)) * 2
    x, y = dev(x0), dev(rng.standard_normal((n, width)) * 0.5)
    post, shift, gain = (dev(rng.standard_normal(width) * 0.4 + 1.0) for _ in range(3))
    xh, yh = host(x), host(y)
    h = ops.residual_norm(x, eps, gain=gain, dtype=dt)
    close(h, pn.rms(xh, eps) * host(gain), tol, "norm")
    assert np.array_equal(host(x), xh)
    h = ops.residual_norm(x, eps, gain=gain, y=y, post=post, dtype=dt)
    want = xh + pn.rms(yh, eps) * host(post)
    close(x, want, 1e-5, "residual")
    close(h, pn.rms(want, eps) * host(gain), tol, "norm after it")
    # several rows per token, at other places, averaged; h rows to several places
    parts = 3
    ys, where = dev(rng.standard_normal((n * parts, width))), rng.permutation(n * parts)
    places = rng.permutation(n * 2)
    x = dev(x0)
    h = ops.residual_norm(x, eps, gain=gain, y=ys, post=post, y_rows=dev(where, torch.int32), y_parts=parts, y_scale=1.0 / parts,
                          h_rows=dev(places, torch.int32), h_parts=2, dtype=dt)
    want = host(dev(x0)) + pn.rms(host(ys)[where].reshape(n, parts, width).mean(1), eps) * host(post)
    close(x, want, 1e-5, "collected residual")
    assert np.array_equal(host(h)[places[0::2]], host(h)[places[1::2]])
    close(host(h)[places[0::2]], pn.rms(want, eps) * host(gain), tol, "scattered rows")
    x = dev(x0)
    h = ops.residual_norm(x, eps, gain=gain, y=ys, post=post, y_parts=parts, dtype=dt)
    close(x, host(dev(x0)) + pn.rms(host(ys).reshape(n, parts, width).sum(1), eps) * host(post), 1e-5, "neighbouring rows")
    # the front of a repeated group: [x | x0], and the replacement behind it
    x, first = dev(x0), dev(rng.standard_normal((n, width)))
    h = ops.residual_norm(x, eps, x0=first, y=y, post=post, dtype=dt)
    close(h, np.concatenate([host(x), host(first)], 1), 2.5e-2 if dtype == "bf16" else 1e-6, "pair")
    h = ops.residual_norm(x, eps, gain=gain, y=y, shift=shift, dtype=dt)
    close(x, yh + host(shift), 1e-6, "replaced")
    close(h, pn.rms(yh + host(shift), eps) * host(gain), tol, "norm of the replaced")


# ── latent attention ───────────────────────────────────────────────────────
class Latent:
    """Random inputs of the mechanism between its first and its last projection; far = (key, queries): that key has a long rotated
    part and those queries point right at it."""

    def __init__(self, ops, H, D, R, E, Q, C, size, n, seed=0, dt=torch.float32, dims=None, scaling=True, far=None):
        rng = np.random.default_rng(seed)
        self.ops, self.shape, self.n, self.dt = ops, (H, D, R, E, Q, C, size), n, dt
        self.dims = dims or R
        lin = lambda o, i, s=1.0: dev(rng.standard_normal((o, i)) * s * i ** -0.5, torch.bfloat16)  # noqa: E731
        self.uq, self.uk, self.uv = lin(H * (D + R), Q, 2.0), lin(H * D, C), lin(H * E, C)
        self.qn, self.kn = dev(rng.standard_normal(Q) * 0.3 + 1), dev(rng.standard_normal(C) * 0.3 + 1)
        self.sink = dev(rng.standard_normal(H) * 1.5 + 1.0)
        self.freq, self.factor = pn.rotary_frequencies(self.dims, 100.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0} if scaling else None)
        self.eps, self.scale = 0.02, (D + R) ** -0.5
        p = rng.standard_normal((n, Q + -Q % 8 + C + R))
        p[:, Q:Q + -Q % 8] = 0.0
        if far is not None:
            key, queries = far
            v = p[key, -R:] = 6.0 * p[key, -R:] / np.abs(p[key, -R:]).mean()
            rows = (np.arange(H)[:, None] * (D + R) + D + np.arange(R)).reshape(-1)
            for i in queries:
                a = (key - i) * self.freq
                u = v.copy()
                u[0::2], u[1::2] = v[0::2] * np.cos(a) - v[1::2] * np.sin(a), v[1::2] * np.cos(a) + v[0::2] * np.sin(a)
                p[i, :Q] = np.linalg.lstsq(host(self.uq)[rows], np.tile(u, H), rcond=None)[0] / host(self.qn)
        self.p = dev(p, dt)

    def angles(self, rows):
        a = np.arange(rows)[:, None] * self.freq[None]
        return dev(np.stack([self.factor * np.cos(a), self.factor * np.sin(a)], axis=2).reshape(rows, -1))

    def run(self, portions, form="auto", rows=None):
        H, D, R, E, Q, C, size = self.shape
        up = lambda v: v + -v % 8  # noqa: E731
        rows = rows or self.n + 2
        cache = torch.full((rows, up(C) + up(R)), 7.0, dtype=self.dt, device="cuda")   # stale rows of an earlier sequence
        w = self.ops.latent_weights(self.uq, self.uk, self.uv, H, D, R, E)
        out, at = [], 0
        while at < self.n:
            k = min(portions[len(out) % len(portions)], self.n - at)
            out.append(self.ops.latent_attention(self.p[at:at + k], cache, at, w, self.sink, self.qn, self.kn, self.angles(rows), H, D, R, self.dims, E, Q, C, size or 0,
                                                 self.scale, self.eps, form))
            at += k
        return torch.cat(out)

    def want(self, mask=None, sink=True):
        """What the mechanism gives; with bf16 the same places are rounded as the cache and the queries are."""
        H, D, R, E, Q, C, size = self.shape
        x, n = host(self.p), self.n
        rnd = (lambda a: host(dev(a, torch.bfloat16))) if self.dt == torch.bfloat16 else (lambda a: a)
        q = rnd(rnd(pn.rms(x[:, :Q], self.eps) * host(self.qn)) @ host(self.uq).T).reshape(n, H, D + R)
        both = x[:, Q + -Q % 8:]
        c = rnd(pn.rms(both[:, :C], self.eps) * host(self.kn))
        kr = rnd(pn.rotate(both[:, C:], self.dims, self.freq, self.factor))
        q = np.concatenate([q[:, :, :D], pn.rotate(q[:, :, D:], self.dims, self.freq, self.factor)], axis=2)
        k = np.concatenate([(c @ host(self.uk).T).reshape(n, H, D), np.repeat(kr[:, None], H, axis=1)], axis=2)
        v = (c @ host(self.uv).T).reshape(n, H, E)
        s = host(self.sink) if sink else np.full(H, -1e9)
        return pn.sink_attention(q, k, v, self.scale, s, pn.visible(n, size) if mask is None else mask).reshape(n, -1)


LATENT = [  # heads, dim, rot_dim, vdim, q_rank, kv_rank, window
    (3, 24, 8, 16, 20, 28, 11), (1, 8, 2, 8, 8, 8, 1), (4, 64, 32, 48, 72, 80, 70), (2, 12, 6, 10, 9, 13, 5), (16, 32, 16, 32, 64, 128, 64),
    (20, 16, 8, 24, 40, 136, 33), (5, 40, 72, 72, 100, 200, 100), (2, 130, 64, 128, 48, 64, None), (8, 128, 64, 128, 96, 512, 90), (40, 8, 8, 8, 16, 24, 17),
]
LATENT_TOL = {"f32": 2e-5, "bf16": 6e-2}


@pytest.mark.parametrize("shape", LATENT)
@pytest.mark.parametrize("dtype,form", [("f32", "absorbed"), ("bf16", "absorbed"), ("bf16", "prompt"), ("bf16", "auto")])
def test_latent_attention(ops, shape, dtype, form):
    a = Latent(ops, *shape, n=200, seed=shape[0], dt=TYPES[dtype])
    want = a.want()
    for portions in ((200,), (70, 2, 1, 1, 33)):
        close(a.run(portions, form), want, LATENT_TOL[dtype], f"portions {portions}")
    close(a.run((64, 64, 1), form, rows=400), want, LATENT_TOL[dtype], "longer cache")
    if form == "absorbed":
        close(a.run((1,), form)[:40], want[:40], LATENT_TOL[dtype], "token by token")


@pytest.mark.parametrize("dims,scaling", [(4, True), (16, False), (10, True)])
def test_latent_rotation_of_a_part(ops, dims, scaling):
    """Fewer rotated dimensions than the rotated part has, with and without scaled frequencies."""
    for dtype, form in (("f32", "absorbed"), ("bf16", "absorbed"), ("bf16", "prompt")):
        a = Latent(ops, 4, 24, 16, 32, 40, 48, 30, n=90, seed=dims, dt=TYPES[dtype], dims=dims, scaling=scaling)
        close(a.run((90,), form), a.want(), LATENT_TOL[dtype], form)


@pytest.mark.parametrize("size,far", [(48, 37), (64, 0), (65, 63), (127, 64), (130, 5)])
@pytest.mark.parametrize("dtype,form,portions", [("f32", "absorbed", (200,)), ("bf16", "prompt", (200,)), ("bf16", "prompt", (90, 21)), ("bf16", "absorbed", (7,)),
                                                 ("f32", "absorbed", (150, 1)), ("bf16", "auto", (150, 1))])
def test_latent_window_edges(ops, size, far, dtype, form, portions):
    """A key that stands out is seen up to its last position and not one further, wherever tiles and portions end."""
    last = far + size - 1
    a = Latent(ops, 2, 32, 8, 32, 32, 64, size, n=far + size + 20, seed=size, dt=TYPES[dtype], far=(far, (last, last + 1)))
    want, tol = a.want(), 2e-5 if dtype == "f32" else 0.1
    assert row_error(a.run(portions, form), want) < tol
    for wrong, at in ((size - 1, last), (size + 1, last + 1)):
        other = a.want(mask=pn.visible(a.n, wrong))
        assert row_error(other[at:at + 1], want[at:at + 1]) > 5 * tol, "the key would not show"


def test_latent_sink_counts_once(ops):
    a = Latent(ops, 4, 32, 16, 32, 32, 64, 40, n=100, seed=5)
    assert error(a.run((100,), "absorbed"), a.want(sink=False)) > 0.2
    for shift in (-30.0, 25.0):     # a sink far below and far above every score
        a.sink = a.sink + shift
        for form, dt in (("absorbed", torch.float32), ("absorbed", torch.bfloat16), ("prompt", torch.bfloat16)):
            a.dt, a.p = dt, a.p.to(dt)
            got, want = host(a.run((60, 40), form)), a.want()
            assert np.abs(got - want).max() < (1e-4 if dt == torch.float32 else 5e-2) * max(np.abs(want).max(), 1e-12), (shift, form)
        a.sink, a.p = a.sink - shift, a.p.float()


def test_latent_growing_scores(ops):
    """Scores that grow along the sequence move the running reference of the prompt form again and again."""
    a = Latent(ops, 2, 32, 16, 32, 32, 64, None, n=300, seed=6, dt=torch.bfloat16)
    p = host(a.p)
    p[:, -16:] *= np.linspace(0.1, 15.0, 300)[:, None]
    a.p = dev(p, torch.bfloat16)
    for form in ("prompt", "absorbed"):
        assert row_error(a.run((300,), form), a.want()) < 0.15, form


# ── matrix memory ──────────────────────────────────────────────────────────
class Memory:
    def __init__(self, ops, H, D, E, cap, n, seed=0, dt=torch.float32, gates=2.0):
        rng = np.random.default_rng(seed)
        self.ops, self.shape, self.n = ops, (H, D, E, cap), n
        self.p = dev(rng.standard_normal((n, 2 * H * D + 2 * H * E)), dt)
        self.gates = dev(rng.standard_normal((n, 2 * H)) * gates)
        self.ib, self.fb, self.norm = dev(rng.standard_normal(H)), dev(rng.standard_normal(H) + 3.0), dev(rng.standard_normal(H * E) * 0.3 + 1.0)
        self.eps = 1e-4

    def run(self, portions, step=False):
        H, D, E, cap = self.shape
        state, m = torch.zeros((H, E + 1, D + -D % 32), device="cuda"), torch.zeros(H, device="cuda")
        out, at = [], 0
        while at < self.n:
            k = min(portions[len(out) % len(portions)], self.n - at)
            one = step or (k == 1 and at > 0)
            out.append(self.ops.matrix_memory(self.p[at:at + k], self.gates[at:at + k].contiguous(), self.ib, self.fb, self.norm, H, D, E, cap, self.eps, state, m, one))
            at += k
        self.state, self.m = state, m
        return torch.cat(out)

    def want(self, gates=None):
        H, D, E, cap = self.shape
        x, g, n = host(self.p), host(self.gates) if gates is None else gates, self.n
        q, k = x[:, :H * D].reshape(n, H, D) * D ** -0.5, x[:, H * D:2 * H * D].reshape(n, H, D)
        v, gate = x[:, 2 * H * D:2 * H * D + H * E].reshape(n, H, E), x[:, 2 * H * D + H * E:]
        i = pn.soft_clip(g[:, :H] + host(self.ib), cap)
        f = pn.log_sigmoid(pn.soft_clip(g[:, H:] + host(self.fb), cap))
        return pn.rms(pn.matrix_memory(q, k, v, i, f), self.eps).reshape(n, -1) * host(self.norm) * pn.sigmoid(gate)


MEMORY = [(1, 4, 6, 5.0), (3, 20, 24, 12.5), (2, 64, 96, 15.0), (4, 33, 17, 3.0), (2, 128, 128, 20.0), (1, 160, 200, 8.0), (5, 8, 130, 30.0)]


def memory_tol(dtype):
    return 3e-4 if dtype == "f32" else 6e-2


@pytest.mark.parametrize("shape", MEMORY)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_matrix_memory(ops, shape, dtype):
    a = Memory(ops, *shape, n=230, seed=shape[1], dt=TYPES[dtype])
    want = a.want()
    for portions in ((230,), (64, 64), (65, 2, 1, 1, 3, 63)):
        close(a.run(portions), want, memory_tol(dtype), f"portions {portions}")
    close(a.run((230,), step=True), want, memory_tol(dtype), "token by token")


def test_matrix_memory_prompt_state_equals_stepped_state(ops):
    a = Memory(ops, 3, 40, 50, 10.0, n=150, seed=1)
    a.run((150,))
    s, m = host(a.state), host(a.m)
    a.run((150,), step=True)
    assert np.abs(m - host(a.m)).max() < 1e-5 and np.abs(s - host(a.state)).max() < 1e-4 * np.abs(s).max()
    assert np.abs(s[:, :, 40:]).max() == 0.0


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [(400,), (100, 1), (63, 65)])
def test_matrix_memory_remembers(ops, dtype, portions):
    """One strong write hundreds of tokens back comes back when its key is asked for, across chunks, portions and steps."""
    H, D, E, cap, n, at = 2, 32, 48, 12.0, 400, 3
    a = Memory(ops, H, D, E, cap, n, seed=9, dt=TYPES[dtype], gates=0.5)
    p, g = host(a.p), host(a.gates)
    g[:, :H] -= 2.0
    g[:, H:] += 40.0                           # nothing is forgotten
    g[at, :H] = 6.0
    p[n - 1, :H * D] = p[at, H * D:2 * H * D]  # the last query is that key
    a.p, a.gates = dev(p, TYPES[dtype]), dev(g)
    want, got = a.want(), a.run(portions)
    assert row_error(got, want) < memory_tol(dtype)
    g[at, :H] = -20.0
    assert row_error(a.want(gates=g)[n - 1:], want[n - 1:]) > 0.5


def test_matrix_memory_extreme_gates(ops):
    """Gates at their caps: weights between exp(-30) and exp(30), forgetting at once and never, and a running maximum so large
    that the constant in the denominator counts."""
    for scale in (0.0, 8.0, 60.0):
        a = Memory(ops, 3, 16, 24, 30.0, n=200, seed=int(scale), gates=scale)
        want = a.want()
        close(a.run((200,)), want, 2e-3, f"prompt {scale}")
        close(a.run((50, 1, 1)), want, 2e-3, f"portions {scale}")


def test_matrix_memory_long_decoding(ops):
    """Thousands of steps with a slowly falling running maximum do not drift."""
    a = Memory(ops, 2, 16, 16, 12.0, n=3000, seed=4, gates=0.3)
    g = host(a.gates)
    g[:, :2] -= 1.0
    g[5, :2] = 7.0
    g[:, 2:] += 6.0
    a.gates = dev(g)
    want = a.want()
    for step in (True, False):
        assert row_error(a.run((3000,), step=step), want) < 1e-3
