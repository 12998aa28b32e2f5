"""Small random Novorax models for the tests: config.json + model.safetensors in a folder, weights rounded to bfloat16."""
import numpy as np

from nositar_models import bf16_f64, to_bf16, write_model  # noqa: F401


def rot(dims, base=100.0, scaling=(4.0, 64, 8.0, 1.0)):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, size, mlp, scale=None, name="latent_attention", rotation=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": rotation or rot(rot_dim)}
    if size:
        mixer["mask"] = {"size": size}
    return {"type": name, "mixer": mixer, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp, name="mlstm"):
    return {"type": name, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width, vocab, loop=None, eps=2e-5, logit_scale=0.6):
    cfg = {"architecture": "Novorax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def make_weights(cfg, seed=0):
    """name -> array.  Spread so that every mechanism matters: scores that differ, sinks of either sign, gates that open and
    close, gains away from 1, passes that differ."""
    rng = np.random.default_rng(seed)
    n = lambda *s, std=1.0, mean=0.0: (rng.standard_normal(s) * std + mean).astype(np.float32)  # noqa: E731
    lin = lambda o, i, std=1.0: n(o, i, std=std * i ** -0.5)  # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": n(V, W), "head": n(V, W, std=2.0 * W ** -0.5), "final.norm": n(W, std=0.3)}
    if cfg.get("loop"):
        w.update({"loop.in": lin(W, 2 * W), "loop.step": n(cfg["loop"]["times"], W, std=0.5)})
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        H, D, E = m["heads"], m["dim"], m["vdim"]
        if layer["type"].startswith("latent_attention"):
            R, Q, C = m["rot_dim"], m["q_rank"], m["kv_rank"]
            w.update({p + "dq": lin(Q, W), p + "dq.norm": n(Q, mean=1.0, std=0.3), p + "uq": lin(H * (D + R), Q, 2.0), p + "dkv": lin(C + R, W),
                      p + "dkv.norm": n(C, mean=1.0, std=0.3), p + "uk": lin(H * D, C), p + "uv": lin(H * E, C), p + "sink": n(H, std=1.5, mean=1.0),
                      p + "o": lin(W, H * E)})
        else:
            w.update({p + "q": lin(H * D, W), p + "k": lin(H * D, W), p + "v": lin(H * E, W), p + "g": lin(H * E, W), p + "o": lin(W, H * E),
                      p + "norm": n(H * E, mean=1.0, std=0.3), p + "i": lin(H, W, 2.0), p + "i.b": n(H), p + "f": lin(H, W, 2.0), p + "f.b": n(H, mean=2.5)})
        subs, f = [1], f"l{i}.mlp."
        if layer["mlp"]:
            subs.append(2)
            if layer["mlp"]["kind"] == "dense":
                F = layer["mlp"]["ff"]
                w.update({f + "up": lin(F, W), f + "down": lin(W, F)})
            else:
                X, F, top = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["top"]
                for e in range(X):
                    w.update({f"{f}e{e}.gate": lin(F, W), f"{f}e{e}.up": lin(F, W), f"{f}e{e}.down": lin(W, F)})
                w[f + "table"] = np.argsort(rng.random((V, X)), axis=1)[:, :top].astype(np.int32)
        for s in subs:
            w.update({f"l{i}.norm{s}": n(W, std=0.3), f"l{i}.norm{s}b": n(W, std=0.3)})
    return w
