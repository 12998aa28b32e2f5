"""Small random Nositar models for the tests: config.json + model.safetensors in a folder, weights rounded to bfloat16."""
import json
import os
import struct

import numpy as np


def attention(heads, kv_heads, dim, vdim, size, keep_first, ff, scale=None):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                      "mask": {"size": size, "keep_first": keep_first}}}


def delta(heads, kv_heads, dim, vdim, conv, ff, name="channel_delta"):
    return {"type": name, "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, width, vocab, streams=3, eps=2e-5, embed_scale=0.75, softcap=9.0):
    return {"architecture": "Nositar", "embedding": {"scale": embed_scale}, "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps},
            "streams": streams, "vocab": vocab, "width": width}


def to_bf16(a):
    """f32 -> the nearest bfloat16, as uint16 bits."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_f64(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def make_weights(cfg, seed=0, rank=10):
    """name -> f32 array.  Spread so that every mechanism matters: scores of either sign, decays between nearly 0 and nearly 1,
    streams that differ, gains away from 1."""
    rng = np.random.default_rng(seed)
    n = lambda *s, std=1.0, mean=0.0: (rng.standard_normal(s) * std + mean).astype(np.float32)  # noqa: E731
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    lin = lambda o, i: n(o, i, std=i ** -0.5)  # noqa: E731
    w = {"embed": n(V, W), "head": n(V, W, std=2.0 * W ** -0.5), "final.norm": n(mean=1.3, std=0.1)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            w.update({p + "q": lin(H * D, W), p + "k": lin(G * D, W), p + "v": lin(G * E, W), p + "o": lin(W, H * E),
                      p + "talk": n(H, H, std=0.5) + 1.5 * np.eye(H, dtype=np.float32), p + "pb": n(H, mean=-3.0, std=0.7)})
        else:
            w.update({p + "q": lin(G * D, W), p + "k": lin(G * D, W), p + "v": lin(H * E, W), p + "o": lin(W, H * E),
                      p + "q.conv": n(G * D, m["conv"], std=0.7), p + "k.conv": n(G * D, m["conv"], std=0.7),
                      p + "v.conv": n(H * E, m["conv"], std=0.7), p + "b": lin(H, W), p + "A_log": n(H, std=0.8, mean=-1.0), p + "norm": n(E, mean=1.0, std=0.3),
                      p + "a1": lin(rank, W), p + "a2": lin(H * D, rank), p + "dt_bias": n(H * D, mean=-1.0), p + "g1": lin(rank + 3, W),
                      p + "g2": lin(H * E, rank + 3)})
        subs = [1]
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            w.update({f"l{i}.mlp.gate": lin(F, W), f"l{i}.mlp.up": lin(F, W), f"l{i}.mlp.down": lin(W, F)})
            subs.append(2)
        for s in subs:
            w.update({f"l{i}.norm{s}": n(mean=1.0, std=0.2), f"l{i}.hc{s}.in": n(S, mean=1.0 / S, std=0.3), f"l{i}.hc{s}.out": n(S, mean=0.7, std=0.3),
                      f"l{i}.hc{s}.mix": n(S, S, std=0.2) + 0.8 * np.eye(S, dtype=np.float32)})
    return w


def write_model(folder, cfg, weights):
    """Writes the folder; returns the weights as the file holds them (f64 of the bfloat16 values; integer tables as they are)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at, back = {}, [], 0, {}
    for name, a in weights.items():
        a = np.asarray(a)
        if a.dtype.kind == "i":
            back[name], raw, kind = a, a.astype("<i4").tobytes(), "I32"
        else:
            bits = to_bf16(a).reshape(a.shape)
            back[name] = bf16_f64(bits.reshape(-1)).reshape(a.shape)
            raw, kind = bits.tobytes(), "BF16"
        head[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return back
