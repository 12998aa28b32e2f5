"""Each Nositar mechanism alone on the GPU, through the operator entry points, against the plain float64 restatement."""
import numpy as np
import pytest

from oracle import plain_nositar as pn

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


def close(got, want, tol, what=""):
    got, want = host(got) if torch.is_tensor(got) else got, np.asarray(want)
    scale = np.sqrt(np.mean(want ** 2)) + 1e-30
    err = np.abs(got - want).max() / scale
    assert np.isfinite(got).all() and err < tol, f"{what}: {err:.2e} of the rms"


TYPES = {"f32": (torch.float32, 2e-5), "bf16": (torch.bfloat16, 5e-2)}


# ── dense matrices ─────────────────────────────────────────────────────────
@pytest.mark.parametrize("path,dtype,n", [("rows", "f32", 1), ("rows", "bf16", 1), ("rows", "bf16", 2), ("rows", "f32", 3), ("rows", "bf16", 8),
                                          ("f32", "f32", 5), ("f32", "f32", 130), ("f32", "bf16", 70), ("tensor", "bf16", 1), ("tensor", "bf16", 9),
                                          ("tensor", "bf16", 40), ("tensor", "bf16", 129), ("tensor", "bf16", 700), ("auto", "bf16", 300)])
@pytest.mark.parametrize("m,k", [(1, 8), (37, 20), (130, 33), (257, 64), (512, 200), (300, 1030)])
def test_dense(ops, path, dtype, n, m, k):
    rng = np.random.default_rng(m * 1000 + k + n)
    dt, _ = TYPES[dtype]
    w, u, x = (dev(rng.standard_normal(s) * k ** -0.5 * c, t) for s, c, t in (((m, k), 1, torch.bfloat16), ((m, k), 1, torch.bfloat16), ((n, k), k ** 0.5, dt)))
    wh, uh, xh = host(w), host(u), host(x)
    tol = 2e-6 * max(k, 64) ** 0.5 * 4     # f32 sums of k products, largest error over the rms
    close(ops.dense(w, x, path=path), xh @ wh.T, tol, "plain")
    close(ops.dense(w, x, w_up=u, path=path), np.maximum(xh @ wh.T, 0) * (xh @ uh.T), tol, "relu gated")
    close(ops.dense(w, x, w_up=u, activation="silu", path=path), pn.silu(xh @ wh.T) * (xh @ uh.T), tol, "silu gated")
    close(ops.dense(w, x, softcap=0.7, path=path), pn.softcap(xh @ wh.T, 0.7), tol, "soft cap")
    close(ops.dense(w, x, out_f32=False, path=path), xh @ wh.T, 4e-2 if dtype == "bf16" else tol, "stored in the activation type")


# ── hyper-connections + norm ───────────────────────────────────────────────
@pytest.mark.parametrize("streams,width,n", [(1, 24, 3), (2, 30, 5), (3, 320, 2), (4, 96, 40), (5, 52, 4), (8, 200, 3), (16, 33, 2), (4, 5000, 3)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_hyper_norm(ops, streams, width, n, dtype):
    rng = np.random.default_rng(streams)
    dt, _ = TYPES[dtype]
    x, y = dev(rng.standard_normal((n, streams, width)) * 3), dev(rng.standard_normal((n, width)))
    mix, w_out, w_in, gain = dev(rng.standard_normal((streams, streams))), dev(rng.standard_normal(streams)), dev(rng.standard_normal(streams)), dev(np.float64(1.7).reshape(1))
    eps = 0.3   # large, so that its place in the formula shows
    xh = host(x)
    tol = 2e-2 if dtype == "bf16" else 1e-5
    h = ops.hyper_norm(x, gain, eps, w_in=w_in, dtype=dt)
    close(h, pn.rms(pn.hyper_read(xh, host(w_in)), eps) * host(gain)[0], tol, "read")
    assert np.array_equal(host(x), xh)
    h = ops.hyper_norm(x, gain, eps, w_in=w_in, y=y, mix=mix, w_out=w_out, dtype=dt)
    want = pn.hyper_write(xh, host(mix), host(w_out), host(y))
    close(x, want, 1e-5, "write")
    close(h, pn.rms(pn.hyper_read(want, host(w_in)), eps) * host(gain)[0], tol, "read after write")
    h = ops.hyper_norm(x, gain, eps, dtype=dt)
    close(h, pn.rms(host(x).sum(1), eps) * host(gain)[0], tol, "plain sum")


# ── attention ──────────────────────────────────────────────────────────────
ATTN = [  # heads, kv_heads, dim, vdim, size, keep_first
    (4, 2, 32, 32, 16, 3), (3, 1, 20, 12, 7, 0), (6, 3, 40, 24, 1, 5), (1, 1, 8, 16, 0, 0), (8, 8, 64, 48, 33, 40), (2, 2, 96, 128, 50, 1),
    (16, 4, 128, 128, 64, 4), (8, 2, 64, 64, 100, 12), (4, 1, 80, 80, 40, 8), (12, 4, 16, 32, 9, 9),
]


def attn_inputs(shape, n, seed, dt):
    H, G, D, E, size, keep = shape
    rng = np.random.default_rng(seed)
    qkv = dev(rng.standard_normal((n, H * D + G * (D + E))), dt)
    talk, bias = dev(rng.standard_normal((H, H)) * 0.6 + np.eye(H)), dev(rng.standard_normal(H) - 1.0)
    return qkv, talk, bias


def attn_want(shape, qkv, talk, bias, scale, eps, mask=None, rnd=None):
    """rnd: how the normalised q and k are stored (the caches hold the activation type)."""
    H, G, D, E, size, keep = shape
    n, x = qkv.shape[0], host(qkv)
    rnd = rnd or (lambda a: a)
    q = rnd(pn.rms(x[:, :H * D].reshape(n, H, D), eps))
    k = rnd(pn.rms(x[:, H * D:(H + G) * D].reshape(n, G, D), eps))
    v = x[:, (H + G) * D:].reshape(n, G, E)
    return pn.mixed_sigmoid_attention(q, k, v, scale, host(talk), host(bias), pn.visible(n, size, keep) if mask is None else mask).reshape(n, -1)


def run_attn(ops, shape, qkv, talk, bias, scale, eps, portions):
    H, G, D, E, size, keep = shape
    n = qkv.shape[0]
    kc = torch.zeros((n + 3, G * D), dtype=qkv.dtype, device="cuda")
    vc = torch.zeros((n + 3, G * E), dtype=qkv.dtype, device="cuda")
    out, at = [], 0
    while at < n:
        p = portions[len(out) % len(portions)]
        out.append(ops.mix_attention(qkv[at:at + p].contiguous(), kc, vc, at, H, G, D, E, scale, eps, size, keep, talk, bias))
        at += p
    return torch.cat(out)


@pytest.mark.parametrize("shape", ATTN)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [(1000,), (2, 3, 50, 17), (128, 1, 1, 31)])
def test_attention(ops, shape, dtype, portions):
    n = 301
    dt, _ = TYPES[dtype]
    qkv, talk, bias = attn_inputs(shape, n, 3, dt)
    scale, eps = 0.9 / shape[2] ** 0.5, 1e-3
    rnd = (lambda a: host(dev(a, dt))) if dtype == "bf16" else None
    want = attn_want(shape, qkv, talk, bias, scale, eps, rnd=rnd)
    got = run_attn(ops, shape, qkv, talk, bias, scale, eps, portions)
    close(got, want, 3e-2 if dtype == "bf16" else 2e-5)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("shape", [(4, 2, 32, 32, 40, 6), (2, 1, 64, 64, 65, 1), (8, 4, 128, 64, 128, 3)])
def test_attention_edges_stand_out(ops, shape, dtype):
    """One key that only matching queries score: the output at the window's edges and at the kept first tokens jumps when the
    key is seen.  The same comparison against a mask that is off by one, or has no kept tokens, must fail."""
    H, G, D, E, size, keep = shape
    n = 3 * size + 37
    dt, _ = TYPES[dtype]
    rng = np.random.default_rng(8)
    x = rng.standard_normal((n, H * D + G * (D + E))) * 0.05
    d = rng.standard_normal(D)
    special = [0, keep - 1, keep, n // 2, n // 2 - size, n - 1 - size, n - size]   # kept, not kept, and edges seen from n // 2 and n - 1
    for j in special:
        x[j, H * D:(H + G) * D] = np.tile(d, G)
        x[j, (H + G) * D:] += 20.0 * (1 + special.index(j))
    x[:, :H * D] += np.tile(d, H) * 4
    qkv, talk, bias = dev(x, dt), dev(np.eye(H) + 0.1), dev(np.full(H, -9.0))
    scale, eps = 16.0 / D, 1e-6   # the matching key scores about 16, the others about 0
    got = host(run_attn(ops, shape, qkv, talk, bias, scale, eps, (29, 64, 2)))
    rnd = (lambda a: host(dev(a, dt))) if dtype == "bf16" else None
    tol = 3e-2 if dtype == "bf16" else 1e-4
    close(got, attn_want(shape, qkv, talk, bias, scale, eps, rnd=rnd), tol)
    for wrong in (pn.visible(n, size + 1, keep), pn.visible(n, size - 1, keep), pn.visible(n, size, keep + 1), pn.visible(n, size, keep - 1)):
        with pytest.raises(AssertionError):
            close(got, attn_want(shape, qkv, talk, bias, scale, eps, mask=wrong, rnd=rnd), tol)


# ── delta rule ─────────────────────────────────────────────────────────────
DELTA = [  # heads, kv_heads, dim, vdim, taps
    (2, 2, 32, 16, 4), (4, 2, 24, 40, 3), (3, 1, 8, 17, 1), (2, 1, 64, 64, 2), (2, 2, 100, 33, 5), (4, 4, 128, 128, 4), (1, 1, 200, 20, 7), (6, 3, 48, 8, 4),
]


def delta_inputs(shape, n, seed, dt):
    H, G, D, E, T = shape
    C = 2 * G * D + H * E
    rng = np.random.default_rng(seed)
    off = C + -C % 8
    proj = np.zeros((n, off + H + -H % 8))
    proj[:, :C] = rng.standard_normal((n, C))
    proj[:, off:off + H] = rng.standard_normal((n, H)) * 2
    t = {"proj": dev(proj, dt), "decay": dev(rng.standard_normal((n, H * D)) * 2), "gate": dev(rng.standard_normal((n, H * E))),
         "conv_w": dev(rng.standard_normal((C, T)) * 0.7), "a_log": dev(rng.standard_normal(H) - 1), "dt_bias": dev(rng.standard_normal(H * D) - 1.5),
         "norm": dev(rng.standard_normal(E) * 0.3 + 1)}
    return t, off


def delta_want(shape, t, off, eps, conv=pn.causal_conv):
    H, G, D, E, T = shape
    x, n = host(t["proj"]), t["proj"].shape[0]
    C = 2 * G * D + H * E
    c = pn.silu(conv(x[:, :C], host(t["conv_w"])))
    q = np.repeat(pn.unit(c[:, :G * D].reshape(n, G, D)) * D ** -0.5, H // G, 1)
    k = np.repeat(pn.unit(c[:, G * D:2 * G * D].reshape(n, G, D)), H // G, 1)
    v = c[:, 2 * G * D:].reshape(n, H, E)
    g = pn.channel_decay((host(t["decay"]) + host(t["dt_bias"])).reshape(n, H, D), host(t["a_log"]))
    o = pn.delta_rule(q, k, v, pn.sigmoid(x[:, off:off + H]), g)
    return (pn.rms(o, eps) * host(t["norm"]) * pn.sigmoid(host(t["gate"])).reshape(n, H, E)).reshape(n, -1)


def run_delta(ops, shape, t, off, eps, portions):
    H, G, D, E, T = shape
    dp = D + -D % 32
    n = t["proj"].shape[0]
    state = torch.zeros((H, E, dp), device="cuda")
    conv = torch.zeros((max(T - 1, 1), 2 * G * D + H * E), device="cuda")
    out, at = [], 0
    while at < n:
        s = slice(at, at + portions[len(out) % len(portions)])
        out.append(ops.channel_delta(t["proj"][s].contiguous(), off, t["decay"][s].contiguous(), t["gate"][s].contiguous(), t["conv_w"], t["a_log"],
                                     t["dt_bias"], t["norm"], H, G, D, E, eps, state, conv))
        at = s.stop
    return torch.cat(out), state


@pytest.mark.parametrize("shape", DELTA)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("portions", [(1000,), (2, 1, 33, 16, 5), (64, 1)])
def test_delta(ops, shape, dtype, portions):
    dt, _ = TYPES[dtype]
    t, off = delta_inputs(shape, 150, 5, dt)
    got, _ = run_delta(ops, shape, t, off, 1e-4, portions)
    close(got, delta_want(shape, t, off, 1e-4), 4e-2 if dtype == "bf16" else 1e-4)


def test_delta_remembers_a_far_key(ops):
    """A value written once, with no decay and no other write, is read 400 tokens later; with the state lost at any portion
    border in between the read-out would be zero (and the normalised output arbitrary)."""
    shape = (1, 1, 32, 16, 2)
    n, (H, G, D, E, T) = 400, shape
    t, off = delta_inputs(shape, n, 9, torch.float32)
    p = t["proj"]
    p[:, off:] = -40.0                 # beta = 0 ...
    p[7, off:] = 40.0                  # ... except for one write
    p[-1, :D], p[-1, D:2 * D] = p[7, D:2 * D], p[7, D:2 * D]
    p[-2, :2 * D], p[6, :2 * D] = 0.0, 0.0   # the same convolution inputs around both
    t["conv_w"][:D] = t["conv_w"][D:2 * D]
    t["decay"][:] = -60.0              # softplus 0: decay 1
    want = delta_want(shape, t, off, 1e-6)
    for portions in ((1000,), (2, 3), (64, 31)):
        got, state = run_delta(ops, shape, t, off, 1e-6, portions)
        close(got[-1], want[-1], 1e-4)
        assert float(state.abs().max()) > 0.05
