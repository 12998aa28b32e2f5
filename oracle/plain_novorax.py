"""Plain, slow restatement of the Novorax decoder in numpy float64, one function per mechanism.

Test infrastructure only: it shares no code with the product path.  A sequence is evaluated whole, token by token where a
state is carried, with no cache, no batch and no portion.  Matrices are [out, in]; `x` arrays are [tokens, ...].
"""
from __future__ import annotations

import numpy as np

from oracle.plain_nositar import F, load, rms, sigmoid, silu  # noqa: F401  (load: re-exported)


# ── elementwise ────────────────────────────────────────────────────────────────────────────────────────
def norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def soft_clip(z, cap):
    return cap * np.tanh(z / cap)


# ── positions ──────────────────────────────────────────────────────────────────────────────────────────
def rotary_frequencies(dims, base, scaling):
    """Angle per position of every pair, and the factor on cos and sin.  With `scaling` (factor, original, fast, slow) the
    pairs that turn more than `fast` times within `original` positions keep their frequency, those that turn less than `slow`
    times are slowed by `factor`, with a linear ramp in between."""
    i = np.arange(dims // 2, dtype=F)
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0

    def pair_that_turns(times):
        return dims * np.log(scaling["original"] / (2.0 * np.pi * times)) / (2.0 * np.log(base))
    lo = max(np.floor(pair_that_turns(scaling["fast"])), 0.0)
    hi = min(np.ceil(pair_that_turns(scaling["slow"])), dims - 1.0)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate(x, dims, freq, factor):
    """x [n, ..., d]: the first `dims` dimensions in neighbouring pairs, by position (first axis)."""
    n = x.shape[0]
    a = np.arange(n, dtype=F)[:, None] * freq[None, :]
    a = a.reshape((n,) + (1,) * (x.ndim - 2) + (-1,))
    c, s = factor * np.cos(a), factor * np.sin(a)
    y = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


# ── mechanisms ─────────────────────────────────────────────────────────────────────────────────────────
def visible(n, size):
    """[n, n] bool: may query i (row) look at key j (column)?  size None or 0: every earlier token."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


def sink_attention(q, k, v, scale, sink, mask):
    """q, k [n, H, d], v [n, H, e], sink [H] -> [n, H, e].  Softmax over the visible keys and one more entry of score `sink`
    that carries no value."""
    n, H, _ = q.shape
    out = np.zeros((n, H, v.shape[2]), F)
    for h in range(H):
        s = np.where(mask, (q[:, h] @ k[:, h].T) * scale, -np.inf)
        top = np.maximum(s.max(axis=1), sink[h])
        w = np.exp(s - top[:, None])
        out[:, h] = (w @ v[:, h]) / (w.sum(axis=1) + np.exp(sink[h] - top))[:, None]
    return out


def matrix_memory(q, k, v, i_log, f_log):
    """q, k [n, H, d] (q scaled), v [n, H, e], log gates [n, H] -> read-outs [n, H, e]."""
    n, H, d = q.shape
    out = np.zeros((n, H, v.shape[2]), F)
    for h in range(H):
        S, z, m = np.zeros((d, v.shape[2]), F), np.zeros(d, F), 0.0
        for t in range(n):
            m_new = max(f_log[t, h] + m, i_log[t, h])
            keep, write = np.exp(f_log[t, h] + m - m_new), np.exp(i_log[t, h] - m_new)
            S = keep * S + write * np.outer(k[t, h], v[t, h])
            z = keep * z + write * k[t, h]
            m = m_new
            out[t, h] = (S.T @ q[t, h]) / (max(abs(z @ q[t, h]), np.exp(-m)) + 1e-6)
    return out


# ── layers ─────────────────────────────────────────────────────────────────────────────────────────────
def latent_attention_mixer(w, p, mc, eps, h):
    n, H, d, r, e, c_n = h.shape[0], mc["heads"], mc["dim"], mc["rot_dim"], mc["vdim"], mc["kv_rank"]
    freq, factor = rotary_frequencies(mc["rot"]["dims"], mc["rot"]["base"], mc["rot"].get("scaling"))
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(n, H, d + r)
    both = h @ w[p + "dkv"].T
    c = rms(both[:, :c_n], eps) * w[p + "dkv.norm"]
    k_rot = rotate(both[:, c_n:], mc["rot"]["dims"], freq, factor)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(n, H, d), np.repeat(k_rot[:, None, :], H, axis=1)], axis=2)
    q = np.concatenate([q[:, :, :d], rotate(q[:, :, d:], mc["rot"]["dims"], freq, factor)], axis=2)
    v = (c @ w[p + "uv"].T).reshape(n, H, e)
    mask = visible(n, (mc.get("mask") or {}).get("size"))
    return sink_attention(q, k, v, mc["scale"], w[p + "sink"], mask).reshape(n, -1) @ w[p + "o"].T


def mlstm_mixer(w, p, mc, eps, h):
    n, H, d, e, cap = h.shape[0], mc["heads"], mc["dim"], mc["vdim"], mc["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(n, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, H, d)
    v = (h @ w[p + "v"].T).reshape(n, H, e)
    i_log = soft_clip(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f_log = log_sigmoid(soft_clip(h @ w[p + "f"].T + w[p + "f.b"], cap))
    o = rms(matrix_memory(q, k, v, i_log, f_log), eps).reshape(n, -1) * w[p + "norm"]
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_ff(w, p, h):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def table_experts_ff(w, p, top, tokens, h):
    """Every token id has its experts; their outputs are averaged."""
    y = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in w[p + "table"][tok]:
            q = f"{p}e{e}."
            y[t] += w[q + "down"] @ (silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t])) / top
    return y


MIXERS = {"latent_attention": latent_attention_mixer, "mlstm": mlstm_mixer}


def mixer_of(kind):
    """A mixer's name may carry a number that tells several sizes apart."""
    head, _, tail = kind.rpartition("_")
    return MIXERS[head if head and tail.isdigit() else kind]


def layer(cfg, w, i, tokens, x):
    eps, lc, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    y = mixer_of(lc["type"])(w, p + "mix.", lc["mixer"], eps, norm(x, w[p + "norm1"], eps))
    x = x + norm(y, w[p + "norm1b"], eps)
    if lc.get("mlp"):
        h = norm(x, w[p + "norm2"], eps)
        if lc["mlp"]["kind"] == "dense":
            y = dense_ff(w, p + "mlp.", h)
        else:
            y = table_experts_ff(w, p + "mlp.", lc["mlp"]["router"]["top"], tokens, h)
        x = x + norm(y, w[p + "norm2b"], eps)
    return x


def enter_pass(w, t, x, x0):
    return np.concatenate([x, x0], axis=1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [n, vocab] of every position.  layers_out: list that receives the residual after every layer run."""
    tokens = np.asarray(tokens)
    x0 = w["embed"][tokens]
    x, loop, n = x0, cfg.get("loop"), len(cfg["layers"])

    def run(a, b, x):
        for i in range(a, b):
            x = layer(cfg, w, i, tokens, x)
            if layers_out is not None:
                layers_out.append(x)
        return x
    if loop:
        x = run(0, loop["start"], x)
        for t in range(loop["times"]):
            x = run(loop["start"], loop["stop"], enter_pass(w, t, x, x0))
        x = run(loop["stop"], n, x)
    else:
        x = run(0, n, x)
    return (norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T) * cfg["logit_scale"]
