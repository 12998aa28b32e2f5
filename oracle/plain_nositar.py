"""Plain, slow restatement of the Nositar decoder in numpy float64, one function per mechanism.

Test infrastructure only: it shares no code with the product path.  A sequence is evaluated whole, token by token where a
state is carried, with no cache, no batch and no portion.  Matrices are [out, in]; `x` arrays are [tokens, ...].
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np

F = np.float64


# ── files ──────────────────────────────────────────────────────────────────────────────────────────────
def read_safetensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        raw = blob[t["data_offsets"][0]:t["data_offsets"][1]]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(raw, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(F)
        elif t["dtype"] == "F32":
            a = np.frombuffer(raw, np.float32).astype(F)
        elif t["dtype"] == "I32":
            a = np.frombuffer(raw, np.int32)
        else:
            raise ValueError(t["dtype"])
        out[name] = a.reshape(t["shape"])
    return out


def load(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ── elementwise ────────────────────────────────────────────────────────────────────────────────────────
def sigmoid(z):
    z = np.asarray(z, F)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms(x, eps):
    """Divide the last axis by its root mean square."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ── mechanisms ─────────────────────────────────────────────────────────────────────────────────────────
def visible(n, size, keep_first):
    """[n, n] bool: may query i (row) look at key j (column)?  size None or 0 = no window."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    if not size:
        return j <= i
    return (j <= i) & ((i - j < size) | (j < keep_first))


def mixed_sigmoid_attention(q, k, v, scale, talk, head_bias, mask):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e].  Heads' scores are blended by talk [H, H], every visible key
    gets sigmoid(score + bias of the head), nothing is normalised over the keys."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    raw = np.stack([q[:, h] @ k[:, h // rep].T for h in range(H)]) * scale
    mixed = np.zeros_like(raw)
    for h in range(H):
        for g in range(H):
            mixed[h] += talk[h, g] * raw[g]
    w = np.where(mask[None], sigmoid(mixed + head_bias[:, None, None]), 0.0)
    return np.stack([w[h] @ v[:, h // rep] for h in range(H)], axis=1)


def causal_conv(x, taps):
    """x [n, c], taps [c, t], last tap = the current token, zeros before the start."""
    n, t = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for j in range(n):
        for i in range(t):
            src = j - (t - 1 - i)
            if src >= 0:
                y[j] += taps[:, i] * x[src]
    return y


def channel_decay(a, A_log):
    """a [n, H, d] (already with its bias) -> decay factors in (0, 1)."""
    return np.exp(-np.exp(A_log)[None, :, None] * softplus(a))


def delta_rule(q, k, v, beta, g):
    """q, k [n, H, d] (already repeated to all heads), v [n, H, e], beta [n, H], g [n, H, d] -> [n, H, e]."""
    n, H, d = k.shape
    out = np.zeros_like(v)
    for h in range(H):
        S = np.zeros((d, v.shape[2]), F)
        for j in range(n):
            S = g[j, h][:, None] * S
            u = beta[j, h] * (v[j, h] - S.T @ k[j, h])
            S = S + np.outer(k[j, h], u)
            out[j, h] = S.T @ q[j, h]
    return out


def hyper_read(streams, w_in):
    return np.einsum("s,nsw->nw", w_in, streams)


def hyper_write(streams, mix, w_out, y):
    return np.einsum("st,nsw->ntw", mix, streams) + w_out[None, :, None] * y[:, None, :]


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ── layers ─────────────────────────────────────────────────────────────────────────────────────────────
def attention_mixer(w, p, mc, eps, h):
    n, H, G = h.shape[0], mc["heads"], mc["kv_heads"]
    q = rms((h @ w[p + "q"].T).reshape(n, H, mc["dim"]), eps)
    k = rms((h @ w[p + "k"].T).reshape(n, G, mc["dim"]), eps)
    v = (h @ w[p + "v"].T).reshape(n, G, mc["vdim"])
    mask = visible(n, mc["mask"]["size"], mc["mask"]["keep_first"])
    o = mixed_sigmoid_attention(q, k, v, mc["scale"], w[p + "talk"], w[p + "pb"], mask)
    return o.reshape(n, -1) @ w[p + "o"].T


def delta_mixer(w, p, mc, eps, h):
    n, H, G, d, e = h.shape[0], mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + t].T, w[p + t + ".conv"])) for t in "qkv")
    q = unit(q.reshape(n, G, d)) * d ** -0.5
    k = unit(k.reshape(n, G, d))
    q, k = (np.repeat(t, H // G, axis=1) for t in (q, k))
    beta = sigmoid(h @ w[p + "b"].T)
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = channel_decay(a.reshape(n, H, d), w[p + "A_log"])
    o = rms(delta_rule(q, k, v.reshape(n, H, e), beta, g), eps) * w[p + "norm"]
    o = o * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(n, H, e)
    return o.reshape(n, -1) @ w[p + "o"].T


def dense_ff(w, p, h):
    return (np.maximum(h @ w[p + "gate"].T, 0.0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"attention": attention_mixer, "channel_delta": delta_mixer, "channel_delta_2": delta_mixer}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [n, vocab] of every position.  layers_out: list that receives the summed streams after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    streams = np.repeat(x[:, None, :], cfg["streams"], axis=1)
    for i, layer in enumerate(cfg["layers"]):
        subs = [(1, lambda h: MIXERS[layer["type"]](w, f"l{i}.mix.", layer["mixer"], eps, h))]
        if layer["mlp"] is not None:
            subs.append((2, lambda h: dense_ff(w, f"l{i}.mlp.", h)))
        for s, fn in subs:
            hc = f"l{i}.hc{s}."
            y = fn(rms(hyper_read(streams, w[hc + "in"]), eps) * w[f"l{i}.norm{s}"])
            streams = hyper_write(streams, w[hc + "mix"], w[hc + "out"], y)
        if layers_out is not None:
            layers_out.append(streams.sum(axis=1))
    h = rms(streams.sum(axis=1), eps) * w["final.norm"]
    return softcap(h @ w["head"].T, cfg.get("logit_softcap"))
