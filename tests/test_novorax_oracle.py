"""The plain Novorax restatement against closed forms, and the folder loader's error paths (no GPU)."""
import ctypes as C
import json
import os

import numpy as np
import pytest

import novorax_models as vm
from oracle import plain_novorax as pn


def test_visible_edges():
    m = pn.visible(9, 3)
    assert [int(r.sum()) for r in m] == [1, 2, 3, 3, 3, 3, 3, 3, 3] and m[8, 6] and not m[8, 5] and not m[4, 5]
    assert np.array_equal(pn.visible(5, None), np.tril(np.ones((5, 5), bool)))


def test_sink_takes_its_share():
    # equal scores s: k visible keys and the sink of score t share the weight
    q, k = np.zeros((4, 1, 2)), np.zeros((4, 1, 2))
    v = np.ones((4, 1, 3))
    o = pn.sink_attention(q, k, v, 1.0, np.array([np.log(2.0)]), pn.visible(4, 3))
    assert np.allclose(o[:, 0, 0], [1 / 3, 2 / 4, 3 / 5, 3 / 5])
    # a sink far below leaves the plain softmax, one far above leaves nothing
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((4, 1, 2)), rng.standard_normal((4, 1, 2)), rng.standard_normal((4, 1, 3))
    s = np.where(pn.visible(4, None), 0.3 * q[:, 0] @ k[:, 0].T, -np.inf)
    p = np.exp(s) / np.exp(s).sum(1, keepdims=True)
    assert np.allclose(pn.sink_attention(q, k, v, 0.3, np.array([-80.0]), pn.visible(4, None))[:, 0], p @ v[:, 0])
    assert np.abs(pn.sink_attention(q, k, v, 0.3, np.array([60.0]), pn.visible(4, None))).max() < 1e-20


def test_rotation_depends_on_distance_only():
    rng = np.random.default_rng(1)
    f, c = pn.rotary_frequencies(6, 50.0, None)
    assert c == 1.0 and np.allclose(f, 50.0 ** (-np.arange(3) / 3.0))
    a, b = rng.standard_normal(8), rng.standard_normal(8)
    x = pn.rotate(np.tile(a, (12, 1)), 6, f, c)
    y = pn.rotate(np.tile(b, (12, 1)), 6, f, c)
    assert np.allclose(x[:, 6:], a[6:]) and np.allclose(x[5] @ y[2], x[9] @ y[6]) and not np.allclose(x[5] @ y[2], x[5] @ y[3])
    assert np.allclose(x[1, :2], [a[0] * np.cos(1) - a[1] * np.sin(1), a[1] * np.cos(1) + a[0] * np.sin(1)])


def test_scaled_frequencies():
    base, dims, s = 1e4, 32, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    plain, _ = pn.rotary_frequencies(dims, base, None)
    f, c = pn.rotary_frequencies(dims, base, s)
    turns = s["original"] * plain / (2 * np.pi)
    assert c == pytest.approx(0.1 * np.log(16.0) + 1.0)
    assert np.allclose(f[turns > 45], plain[turns > 45]) and np.allclose(f[turns < 0.5], plain[turns < 0.5] / 16.0)
    assert np.all(np.diff(plain / f) >= -1e-12) and len(set(np.round(plain / f, 6))) > 3


def test_matrix_memory_reads_what_was_written():
    # one strong write, then nothing is written and nothing forgotten: the value comes back whenever its key is asked for
    n, d = 5, 4
    k = np.zeros((n, 1, d)); k[:, 0, 1] = 1.0
    v = np.arange(n * 3.0).reshape(n, 1, 3)
    i = np.full((n, 1), -50.0); i[0] = 3.0
    f = np.zeros((n, 1))
    o = pn.matrix_memory(k, k, v, i, f)
    assert np.allclose(o[:, 0], v[0, 0], rtol=1e-4)
    # the running maximum starts at 0: a weak first write is divided by exp(-m) = 1, not by itself
    i[0] = -2.0
    o = pn.matrix_memory(k, k, v + 1.0, i, f)
    assert np.allclose(o[0, 0], np.exp(-2.0) * (v[0, 0] + 1.0), rtol=1e-5)
    # what was written is forgotten by exp(f) per token
    o = pn.matrix_memory(k, k, v + 1.0, i, np.full((n, 1), -0.5))
    assert np.allclose(o[2, 0], np.exp(-3.0) * (v[0, 0] + 1.0), rtol=1e-5)


def test_matrix_memory_is_a_weighted_sum():
    rng = np.random.default_rng(2)
    n, H, d, e = 7, 2, 3, 4
    q, k, v = rng.standard_normal((n, H, d)), rng.standard_normal((n, H, d)), rng.standard_normal((n, H, e))
    i, f = rng.standard_normal((n, H)) * 2, pn.log_sigmoid(rng.standard_normal((n, H)))
    o = pn.matrix_memory(q, k, v, i, f)
    for h in range(H):
        m = 0.0
        for t in range(n):
            m = max(f[t, h] + m, i[t, h])
            w = np.array([np.exp(f[j + 1:t + 1, h].sum() + i[j, h]) * (q[t, h] @ k[j, h]) for j in range(t + 1)])
            want = w @ v[:t + 1, h] / (max(abs(w.sum()), 1.0) + 1e-6 * np.exp(m))
            assert np.allclose(o[t, h], want)


def test_experts_average_and_ids_choose():
    cfg = vm.config([vm.mlstm(1, 4, 4, 5.0, vm.moe(4, 2, 6))], width=8, vocab=10)
    w = {k: np.asarray(v, np.float64) if v.dtype.kind == "f" else v for k, v in vm.make_weights(cfg).items()}
    h = np.random.default_rng(3).standard_normal((2, 8))
    y = pn.table_experts_ff(w, "l0.mlp.", 2, [7, 7], h)
    one = lambda e, x: w[f"l0.mlp.e{e}.down"] @ (pn.silu(w[f"l0.mlp.e{e}.gate"] @ x) * (w[f"l0.mlp.e{e}.up"] @ x))  # noqa: E731
    a, b = w["l0.mlp.table"][7]
    assert a != b and np.allclose(y[1], 0.5 * (one(a, h[1]) + one(b, h[1])))


def test_loop_repeats_with_state_of_its_own():
    """Two passes over a layer equal the layer written out twice, with the entry written between."""
    cfg = vm.config([vm.mlstm(2, 4, 6, 6.0, vm.dense(9)), vm.latent(2, 4, 2, 6, 5, 7, 3, None)], width=10, vocab=12, loop=(1, 2, 2))
    w = {k: np.asarray(v, np.float64) for k, v in vm.make_weights(cfg).items()}
    toks = np.arange(9) % 12
    out = []
    pn.forward(cfg, w, toks, out)
    assert len(out) == 3
    x0 = w["embed"][toks]
    x = pn.layer(cfg, w, 0, toks, x0)
    for t in range(2):
        x = pn.layer(cfg, w, 1, toks, np.concatenate([x, x0], 1) @ w["loop.in"].T + w["loop.step"][t])
    assert np.allclose(out[-1], x)


# ── loader ─────────────────────────────────────────────────────────────────
SMALL = dict(width=16, vocab=20)


def _try(lib, tmp_path, cfg, drop=(), edit=None):
    from wick_b200 import _lib
    w = vm.make_weights(cfg)
    for d in drop:
        w.pop(d)
    if edit:
        edit(w)
    vm.write_model(str(tmp_path), cfg, w)
    h = C.c_void_p()
    code = lib.wick_cuda_model_create_from_path(str(tmp_path).encode(), 32, 0, 0, C.byref(h))
    if code == _lib.OK:
        lib.wick_cuda_model_destroy(h)
    return code, lib.wick_cuda_last_error().decode()


def test_registry_and_config(tmp_path):
    from wick_b200 import model
    cfg = vm.config([vm.mlstm(1, 4, 4, 5.0, None)], **SMALL)
    vm.write_model(str(tmp_path), cfg, vm.make_weights(cfg))
    assert model.model_architecture(str(tmp_path)) == "Novorax"
    assert model.MODEL_CLASSES["Novorax"] is model.CudaNovoraxModel


def test_truncated_and_broken_files(cuda_lib, tmp_path):
    from wick_b200 import _lib
    cfg = vm.config([vm.mlstm(1, 4, 4, 5.0, None)], **SMALL)
    vm.write_model(str(tmp_path), cfg, vm.make_weights(cfg))
    f = os.path.join(tmp_path, "model.safetensors")
    blob = open(f, "rb").read()
    h = C.c_void_p()
    for bad in (blob[:4], blob[:40], blob[:-6]):
        open(f, "wb").write(bad)
        assert cuda_lib.wick_cuda_model_create_from_path(str(tmp_path).encode(), 32, 0, 0, C.byref(h)) == _lib.ERR_BAD_MODEL
    open(f, "wb").write(blob)
    open(os.path.join(tmp_path, "config.json"), "w").write(json.dumps(cfg)[:-2])
    assert cuda_lib.wick_cuda_model_create_from_path(str(tmp_path).encode(), 32, 0, 0, C.byref(h)) == _lib.ERR_BAD_MODEL


@pytest.mark.gpu
def test_loader_names_what_is_wrong(cuda_lib, tmp_path):
    from wick_b200 import _lib
    ok = vm.config([vm.latent(2, 4, 2, 6, 5, 7, 3, vm.moe(3, 2, 5)), vm.mlstm(1, 4, 4, 5.0, vm.dense(7))], loop=(0, 1, 2), **SMALL)
    assert _try(cuda_lib, tmp_path, ok)[0] == _lib.OK

    def edited(fn):
        cfg = json.loads(json.dumps(ok))
        fn(cfg)
        return cfg
    for name in ("l0.mix.sink", "l0.mix.dkv.norm", "l0.mlp.e2.up", "l0.mlp.table", "l1.mix.f.b", "l1.norm2b", "loop.in", "loop.step"):
        code, msg = _try(cuda_lib, tmp_path, ok, drop=[name])
        assert code == _lib.ERR_BAD_MODEL and name in msg, (name, msg)

    def far(w):
        w["l0.mlp.table"] = w["l0.mlp.table"].copy()
        w["l0.mlp.table"][4, 1] = 3
    assert "no expert 3" in _try(cuda_lib, tmp_path, ok, edit=far)[1]
    assert "unknown mixer" in _try(cuda_lib, tmp_path, edited(lambda c: c["layers"][1].update(type="mlstms")))[1]
    base = vm.make_weights(ok)
    for fn, word in ((lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "unknown feed-forward"), (lambda c: c["loop"].update(stop=3), "loop"), (lambda c: c["loop"].update(start=1), "loop"),
                     (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), "rotated"), (lambda c: c["layers"][1]["mixer"].update(gate_cap=0), "gate_cap")):
        cfg = edited(fn)
        vm.write_model(str(tmp_path), cfg, base)
        h = C.c_void_p()
        assert cuda_lib.wick_cuda_model_create_from_path(str(tmp_path).encode(), 32, 0, 0, C.byref(h)) == _lib.ERR_BAD_MODEL
        assert word in cuda_lib.wick_cuda_last_error().decode()


def test_operator_argument_checks(cuda_lib):
    from wick_b200 import _lib
    bad = _lib.ERR_BAD_ARG
    assert cuda_lib.wick_cuda_residual_norm(1, 16, 1, 8, None, 1, None, 1.0, None, None, None, None, 1e-5, 16, 8, 1, None, None) == bad    # no gain, no x0
    assert cuda_lib.wick_cuda_residual_norm(1, 16, 1, 8, 16, 1, None, 1.0, 16, 16, 16, None, 1e-5, 16, 8, 1, None, None) == bad            # post and shift
    assert cuda_lib.wick_cuda_residual_norm(1, 16, 1, 8, None, 1, None, 1.0, None, None, None, 16, 1e-5, 16, 8, 1, None, None) == bad      # [x | x0] too wide
    lat = [1, 16, 32, 1, 0, 16, 8, 16, 16, 16, None, 16, 16, 16, 16, 2, 4, 2, 2, 4, 8, 8, 0, 1.0, 1e-5, 0, 16, 8, None]
    for at, v in ((2, 20), (4, 8), (18, 3), (18, 4), (25, 3), (25, 2), (27, 4)):
        args = list(lat)
        args[at] = v
        assert cuda_lib.wick_cuda_latent_attention(*args) == bad, (at, v)
    mem = [1, 16, 16, 16, 2, 1, 1, 4, 4, 5.0, 1e-5, 16, 16, 16, 16, 16, 0, 16, 8, None]
    for at, v in ((2, 8), (4, 1), (7, 5000), (9, 0.0), (18, 3)):
        args = list(mem)
        args[at] = v
        assert cuda_lib.wick_cuda_matrix_memory(*args) == bad, (at, v)
