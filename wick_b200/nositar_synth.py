"""Seeded random-weight Nositar model folders (config.json + model.safetensors) for benchmarks.

The weights are drawn on the GPU with torch and rounded to bfloat16; they mean nothing, only the shapes resemble a real
model's layers.
"""
from __future__ import annotations

import dataclasses
import json
import os
import struct
from typing import Dict, Tuple

from .gguf_synth import Lfm2Spec


@dataclasses.dataclass(frozen=True)
class NositarSpec:
    """`attn_layers` carry windowed attention, the others the delta rule; every layer has a feed-forward."""
    name: str
    width: int
    n_layers: int
    attn_layers: Tuple[int, ...]
    ffn: int
    vocab: int
    heads: int              # attention: head size width / heads for keys and values
    kv_heads: int
    window: int
    keep_first: int
    delta_heads: int        # delta rule: key and value size width / delta_heads
    delta_rank: int
    conv: int = 4
    streams: int = 4

    def config(self) -> dict:
        d, e = self.width // self.heads, self.width // self.delta_heads
        ff = {"kind": "dense", "ff": self.ffn}
        attn = {"type": "attention", "mlp": ff, "mixer": {"heads": self.heads, "kv_heads": self.kv_heads, "dim": d, "vdim": d, "scale": d ** -0.5,
                                                          "mask": {"size": self.window, "keep_first": self.keep_first}}}
        delta = {"type": "channel_delta", "mlp": ff, "mixer": {"heads": self.delta_heads, "kv_heads": self.delta_heads, "dim": e, "vdim": e, "conv": self.conv}}
        return {"architecture": "Nositar", "embedding": {"scale": 1.0}, "layers": [attn if i in self.attn_layers else delta for i in range(self.n_layers)],
                "logit_softcap": 30.0, "norm": {"eps": 1e-5}, "streams": self.streams, "vocab": self.vocab, "width": self.width}

    def shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, S, out = self.width, self.streams, {}
        out["embed"] = (self.vocab, W)
        for i in range(self.n_layers):
            p = f"l{i}.mix."
            if i in self.attn_layers:
                kv = self.kv_heads * (W // self.heads)
                out.update({p + "q": (W, W), p + "k": (kv, W), p + "v": (kv, W), p + "talk": (self.heads,) * 2, p + "pb": (self.heads,), p + "o": (W, W)})
            else:
                H, e, r = self.delta_heads, W // self.delta_heads, self.delta_rank
                for t in "qkv":
                    out.update({p + t: (W, W), p + t + ".conv": (W, self.conv)})
                out.update({p + "b": (H, W), p + "A_log": (H,), p + "norm": (e,), p + "a1": (r, W), p + "a2": (W, r), p + "dt_bias": (W,),
                            p + "g1": (r, W), p + "g2": (W, r), p + "o": (W, W)})
            out.update({f"l{i}.mlp.gate": (self.ffn, W), f"l{i}.mlp.up": (self.ffn, W), f"l{i}.mlp.down": (W, self.ffn)})
            for s in (1, 2):
                out.update({f"l{i}.norm{s}": (), f"l{i}.hc{s}.in": (S,), f"l{i}.hc{s}.out": (S,), f"l{i}.hc{s}.mix": (S, S)})
        out.update({"final.norm": (), "head": (self.vocab, W)})
        return out

    def matrix_params_per_layer(self) -> int:
        """Parameters of the layers' matrices: the multiply-adds one token costs in the GEMMs outside the head."""
        return sum(s[0] * s[1] for n, s in self.shapes().items() if len(s) == 2 and n[0] == "l" and n.split(".")[-1] not in ("talk", "mix", "conv"))

    def decode_bytes_per_token(self, position: int) -> int:
        """Algorithmic HBM bytes of one decode step at batch 1: every matrix once in bfloat16, one embedding row, the cached
        rows the windows see, and the recurrent states read and written."""
        b = 2 * (self.matrix_params_per_layer() + self.vocab * self.width + self.width)
        seen = min(position + 1, self.window + self.keep_first)
        for i in range(self.n_layers):
            if i in self.attn_layers:
                b += 2 * seen * 2 * self.kv_heads * (self.width // self.heads)
            else:
                b += 2 * 4 * self.width * (self.width // self.delta_heads)
        return b

    def lfm2(self) -> Lfm2Spec:
        """The closest other model of this library at equal size: convolution layers instead of the delta rule, plain causal
        attention with the same width of queries, same feed-forward and vocabulary."""
        return Lfm2Spec(self.name.replace("nositar", "lfm2"), self.width, self.n_layers, self.attn_layers, self.width // 64,
                        max(1, self.kv_heads * (self.width // self.heads) // 64), self.ffn, self.vocab, 8192)


SPECS: Dict[str, NositarSpec] = {
    "nositar-w1024": NositarSpec("nositar-w1024", 1024, 6, (2, 5), 4608, 32768, 8, 4, 1024, 16, 8, 64),
    "nositar-w2048": NositarSpec("nositar-w2048", 2048, 6, (2, 5), 6912, 32768, 16, 4, 1024, 16, 16, 128),
}


def write_folder(folder: str, config: dict, shapes: Dict[str, Tuple[int, ...]], draw, seed: int = 0) -> str:
    """config.json and model.safetensors with the tensors that draw(name, shape, generator) returns: int32 ones as such, the rest
    rounded to bfloat16."""
    import torch
    gen = torch.Generator("cuda").manual_seed(seed)
    os.makedirs(folder, exist_ok=True)
    is_int = {name: name.endswith(".table") for name in shapes}
    head, at = {}, 0
    for name, s in shapes.items():
        n = 4 if is_int[name] else 2
        for d in s:
            n *= d
        head[name] = {"dtype": "I32" if is_int[name] else "BF16", "shape": list(s), "data_offsets": [at, at + n]}
        at += n
    h = json.dumps(head).encode()
    tmp = os.path.join(folder, f"model.{os.getpid()}.part")
    with open(tmp, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for name, s in shapes.items():
            t = draw(name, s, gen)
            f.write((t.to(torch.int32).cpu() if is_int[name] else t.to(torch.bfloat16).cpu().view(torch.int16)).numpy().tobytes())
    os.replace(tmp, os.path.join(folder, "model.safetensors"))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    return folder


def draw_weight(name, s, gen):
    import torch
    t = torch.randn(s, generator=gen, device="cuda")
    last = name.split(".")[-1]
    if len(s) == 2 and last not in ("talk", "mix", "conv"):
        t *= s[1] ** -0.5
    elif last in ("talk", "mix"):
        t = 0.2 * t / s[0] ** 0.5 + torch.eye(s[0], device="cuda")
    elif last == "in":
        t = 0.1 * t + 1.0 / s[0]
    elif last == "pb":
        t = 0.3 * t - 5.0
    elif last in ("A_log", "dt_bias"):
        t = 0.5 * t - 2.0
    elif last != "conv" and name != "embed":
        t = 0.1 * t + 1.0
    return t


def write_model(folder: str, spec: NositarSpec, seed: int = 0) -> str:
    return write_folder(folder, spec.config(), spec.shapes(), draw_weight, seed)


def cached_model(name: str, seed: int = 0) -> str:
    """Folder of the seeded model, written on first use."""
    folder = os.path.join(os.environ.get("WICK_SYNTH_CACHE", "/tmp/wick_b200_models"), f"{name}-s{seed}")
    if not os.path.exists(os.path.join(folder, "config.json")):
        write_model(folder, SPECS[name], seed)
    return folder
