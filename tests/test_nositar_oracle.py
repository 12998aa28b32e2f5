"""The plain Nositar restatement against closed forms, and the folder loader's error paths (no GPU)."""
import ctypes as C
import json
import os

import numpy as np
import pytest

import nositar_models as nm
from oracle import plain_nositar as pn


def test_visible_edges():
    m = pn.visible(12, 4, 2)
    for i in range(12):
        for j in range(12):
            want = j <= i and (i - j <= 3 or j <= 1)
            assert m[i, j] == want, (i, j)
    assert np.array_equal(pn.visible(5, 0, 0), np.tril(np.ones((5, 5), bool)))


def test_attention_is_unnormalised_and_blends_heads():
    # scores are zero everywhere: every visible key counts sigmoid(bias) = 1/2, so the output is half the sum of the values
    q, k = np.zeros((6, 2, 4)), np.zeros((6, 1, 4))
    v = np.arange(6.0)[:, None, None] * np.ones((6, 1, 3))
    o = pn.mixed_sigmoid_attention(q, k, v, 1.0, np.eye(2), np.zeros(2), pn.visible(6, 3, 1))
    assert np.allclose(o[5, 0], 0.5 * (0 + 3 + 4 + 5))
    # swapping the heads through `talk` is the same as swapping the queries
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 2, 3))
    a = pn.mixed_sigmoid_attention(q, k, v, 0.7, np.array([[0.0, 1.0], [1.0, 0.0]]), np.zeros(2), pn.visible(6, 0, 0))
    w01 = pn.sigmoid(0.7 * np.einsum("id,jd->ij", q[:, 1], k[:, 1])) * pn.visible(6, 0, 0)
    assert np.allclose(a[:, 0], w01 @ v[:, 0])


def test_delta_rule_writes_and_overwrites():
    # a unit key written with beta = 1 is read back exactly; writing it again replaces the value
    k = np.zeros((3, 1, 4)); k[:, 0, 2] = 1.0
    v = np.array([[5.0, 6.0], [7.0, 8.0], [0.5, -1.0]])[:, None, :]
    o = pn.delta_rule(k, k, v, np.ones((3, 1)), np.ones((3, 1, 4)))
    assert np.allclose(o, v)
    # with beta = 0 from then on the stored value decays per key channel
    g = np.ones((3, 1, 4)); g[1:, 0, 2] = 0.5
    o = pn.delta_rule(k, k, v, np.array([[1.0], [0.0], [0.0]]), g)
    assert np.allclose(o[2, 0], 0.25 * v[0, 0])


def test_causal_conv_and_hyper():
    x = np.arange(8.0).reshape(4, 2)
    t = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    y = pn.causal_conv(x, t)
    assert np.allclose(y[0], [0, 1]) and np.allclose(y[3], [2 * 1 + 4 * 10 + 6 * 100, 7])
    s = np.stack([np.ones((2, 3)), 2 * np.ones((2, 3))], 1)
    out = pn.hyper_write(s, np.array([[1.0, 2.0], [10.0, 20.0]]), np.array([0.0, 1.0]), np.full((2, 3), 0.5))
    assert np.allclose(out[:, 0], 1 + 20) and np.allclose(out[:, 1], 2 + 40 + 0.5)


def _folder(tmp_path, cfg, drop=(), edit=None):
    w = nm.make_weights(cfg)
    for d in drop:
        del w[d]
    if edit:
        edit(w)
    nm.write_model(str(tmp_path), cfg, w)
    return str(tmp_path)


SMALL = dict(width=24, vocab=31, streams=2)


@pytest.mark.parametrize("what", ["missing", "shape", "mixer", "arch", "header", "kind", "json"])
def test_bad_folders_are_refused(cuda_lib, tmp_path, what):
    """A folder that cannot be used is an error that names the reason, before any device work where there is no device."""
    from wick_b200 import _lib
    cfg = nm.config([nm.attention(2, 1, 8, 8, 4, 1, 16), nm.delta(2, 1, 8, 8, 3, 0)], **SMALL)
    drop, edit, expect = (), None, b""
    if what == "missing":
        drop, expect = ("l1.mix.dt_bias",), b"l1.mix.dt_bias"
    if what == "shape":
        edit, expect = lambda w: w.update({"l0.mix.talk": np.ones((2, 3), np.float32)}), b"l0.mix.talk"
    p = _folder(tmp_path, cfg, drop, edit)
    if what in ("mixer", "arch", "kind"):
        c = json.load(open(os.path.join(p, "config.json")))
        if what == "mixer":
            c["layers"][1]["type"], expect = "nothing_known", b"nothing_known"
        elif what == "kind":
            c["layers"][0]["mlp"]["kind"], expect = "sparse", b"sparse"
        else:
            c["architecture"], expect = "Unheard", b"Unheard"
        json.dump(c, open(os.path.join(p, "config.json"), "w"))
    if what == "header":
        f = os.path.join(p, "model.safetensors")
        raw = open(f, "rb").read()
        open(f, "wb").write(raw[:len(raw) - 64])
        expect = b"beyond the end"
    if what == "json":
        open(os.path.join(p, "config.json"), "w").write("{\"architecture\": \"Nositar\", ")
        expect = b"JSON"
    h = C.c_void_p()
    r = cuda_lib.wick_cuda_model_create_from_path(p.encode(), 64, 0, 0, C.byref(h))
    msg = cuda_lib.wick_cuda_last_error()
    assert not h.value
    import torch
    if what in ("header", "json") or torch.cuda.is_available():
        assert r == _lib.ERR_BAD_MODEL and expect in msg, msg
    else:
        assert r in (_lib.ERR_CUDA, _lib.ERR_BAD_ARG)     # no device: the weights are not looked at


def test_architecture_registry(tmp_path):
    from wick_b200 import model
    cfg = nm.config([nm.delta(2, 1, 8, 8, 3, 0)], **SMALL)
    p = _folder(tmp_path, cfg)
    assert model.model_architecture(p) == "Nositar"
    assert set(model.MODEL_CLASSES) == {"lfm2", "Nositar", "Novorax"}
    assert model.MODEL_CLASSES["Nositar"] is model.CudaNositarModel
    json.dump({"architecture": "Unheard"}, open(os.path.join(p, "config.json"), "w"))
    with pytest.raises(ValueError, match="Unheard"):
        model.load_model_cuda(p)


def test_operator_argument_checks(cuda_lib):
    from wick_b200 import _lib
    assert cuda_lib.wick_cuda_dense(1, None, None, 1, 8, 8, None, 8, 1, None, 1, 1, 0, 0.0, 0, None) == _lib.ERR_BAD_ARG
    assert cuda_lib.wick_cuda_dense(1, 16, None, 4, 12, 12, 16, 16, 1, 16, 4, 1, 0, 0.0, 0, None) == _lib.ERR_BAD_ARG   # pitch not padded
    assert cuda_lib.wick_cuda_hyper_norm(1, 16, 1, 17, 8, None, None, None, None, 16, 1e-5, 16, 8, None) == _lib.ERR_BAD_ARG
    assert cuda_lib.wick_cuda_mix_attention(1, 16, 32, 4, 0, 16, 16, 8, None, None, 3, 2, 4, 4, 1.0, 1e-5, 0, 0, 16, 16, None) == _lib.ERR_BAD_ARG
    assert cuda_lib.wick_cuda_channel_delta(1, 16, 64, 4, 16, 16, 16, 16, 16, 16, 1, 2, 1, 8, 8, 3, 1e-5, 16, 16, 16, 16, None) == _lib.ERR_BAD_ARG
