"""Seeded random-weight Novorax model folders (config.json + model.safetensors) for benchmarks.

The weights are drawn on the GPU with torch and rounded to bfloat16; they mean nothing, only the shapes resemble a real
model's layers.
"""
from __future__ import annotations

import dataclasses
import os
from typing import Dict, Tuple

from .nositar_synth import write_folder


@dataclasses.dataclass(frozen=True)
class NovoraxSpec:
    """`attn_layers` carry latent attention, the others the matrix memory; `moe_layers` have experts, the others a dense
    feed-forward.  Layers loop_start .. loop_stop - 1 run loop_times times."""
    name: str
    width: int
    n_layers: int
    attn_layers: Tuple[int, ...]
    moe_layers: Tuple[int, ...]
    ffn: int                # of a dense layer (two matrices)
    expert_ffn: int         # of an expert (three matrices)
    experts: int
    top: int
    vocab: int
    heads: int              # latent attention
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    window: int
    mem_heads: int          # matrix memory
    mem_dim: int
    mem_vdim: int
    loop_start: int
    loop_stop: int
    loop_times: int

    def runs(self) -> list:
        """Layers in the order they run."""
        once = list(range(self.loop_start, self.loop_stop))
        return list(range(self.loop_start)) + once * self.loop_times + list(range(self.loop_stop, self.n_layers))

    def config(self) -> dict:
        latent = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank, "kv_rank": self.kv_rank,
                  "scale": (self.dim + self.rot_dim) ** -0.5, "mask": {"size": self.window},
                  "rot": {"dims": self.rot_dim, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        memory = {"heads": self.mem_heads, "dim": self.mem_dim, "vdim": self.mem_vdim, "gate_cap": 15.0}
        dense = {"kind": "dense", "ff": self.ffn}
        moe = {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.expert_ffn}}
        layers = [{"type": "latent_attention" if i in self.attn_layers else "mlstm", "mixer": latent if i in self.attn_layers else memory,
                   "mlp": moe if i in self.moe_layers else dense} for i in range(self.n_layers)]
        return {"architecture": "Novorax", "layers": layers, "logit_scale": 0.25, "norm": {"eps": 1e-6}, "vocab": self.vocab, "width": self.width,
                "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}}

    def mixer_shapes(self, i: int) -> Dict[str, Tuple[int, ...]]:
        W = self.width
        if i in self.attn_layers:
            H, C = self.heads, self.kv_rank
            return {"dq": (self.q_rank, W), "dq.norm": (self.q_rank,), "uq": (H * (self.dim + self.rot_dim), self.q_rank), "dkv": (C + self.rot_dim, W),
                    "dkv.norm": (C,), "uk": (H * self.dim, C), "uv": (H * self.vdim, C), "sink": (H,), "o": (W, H * self.vdim)}
        H, qk, v = self.mem_heads, self.mem_heads * self.mem_dim, self.mem_heads * self.mem_vdim
        return {"q": (qk, W), "k": (qk, W), "v": (v, W), "g": (v, W), "o": (W, v), "norm": (v,), "i": (H, W), "i.b": (H,), "f": (H, W), "f.b": (H,)}

    def shapes(self) -> Dict[str, Tuple[int, ...]]:
        W, out = self.width, {}
        out["embed"] = (self.vocab, W)
        out.update({"loop.in": (W, 2 * W), "loop.step": (self.loop_times, W)})
        for i in range(self.n_layers):
            p = f"l{i}."
            out.update({p + n: (W,) for n in ("norm1", "norm1b", "norm2", "norm2b")})
            out.update({p + "mix." + n: s for n, s in self.mixer_shapes(i).items()})
            if i in self.moe_layers:
                for e in range(self.experts):
                    q = f"{p}mlp.e{e}."
                    out.update({q + "gate": (self.expert_ffn, W), q + "up": (self.expert_ffn, W), q + "down": (W, self.expert_ffn)})
                out[p + "mlp.table"] = (self.vocab, self.top)
            else:
                out.update({p + "mlp.up": (self.ffn, W), p + "mlp.down": (W, self.ffn)})
        out.update({"final.norm": (W,), "head": (self.vocab, W)})
        return out

    def draw(self, name, s, gen):
        import torch
        if name.endswith(".table"):
            return torch.rand((s[0], self.experts), generator=gen, device="cuda").argsort(dim=1)[:, :s[1]]
        t = torch.randn(s, generator=gen, device="cuda")
        if len(s) == 2 and name not in ("embed", "loop.step"):
            return t * s[1] ** -0.5
        last = name.split(".")[-1]
        if name.endswith(".f.b"):
            return t + 4.0
        if last.startswith("norm") and not name.endswith("mix.norm") and not name.endswith("dq.norm") and not name.endswith("dkv.norm"):
            return 0.1 * t                     # stored around zero
        return 0.1 * t + 1.0 if last == "norm" and name != "final.norm" else 0.1 * t if name in ("final.norm", "loop.step") else t

    def matrix_params_per_run(self) -> int:
        """Multiply-adds one token costs in the matrix products outside the head (chosen experts only), as the prompt form does
        them: keys and values of latent attention are computed per position."""
        W, total = self.width, self.loop_times * 2 * self.width * self.width
        for i in self.runs():
            total += sum(s[0] * s[1] for s in self.mixer_shapes(i).values() if len(s) == 2)
            total += 3 * self.top * self.expert_ffn * W if i in self.moe_layers else 2 * self.ffn * W
        return total

    def decode_bytes_per_token(self, position: int) -> int:
        """Algorithmic HBM bytes of one decode step at batch 1: every matrix of every run once in bfloat16 (chosen experts only),
        one embedding row, the cached rows the windows see, and the recurrent states read and written."""
        b = 2 * (self.matrix_params_per_run() + self.vocab * self.width + self.width)
        seen = min(position + 1, self.window)
        for i in self.runs():
            if i in self.attn_layers:
                b += 2 * seen * (self.kv_rank + self.rot_dim)
            else:
                b += 2 * 4 * self.mem_heads * self.mem_dim * (self.mem_vdim + 1)
        return b


SPECS: Dict[str, NovoraxSpec] = {
    "novorax-w1024": NovoraxSpec("novorax-w1024", 1024, 6, (2, 5), (1, 4), 6912, 2304, 16, 2, 32768, 8, 128, 64, 128, 512, 256, 1024, 4, 128, 256, 1, 5, 1),
    "novorax-w2048": NovoraxSpec("novorax-w2048", 2048, 6, (2, 5), (1, 4), 10368, 3456, 16, 2, 32768, 16, 128, 64, 128, 768, 512, 1024, 8, 128, 256, 1, 5, 1),
}


def cached_model(name: str, seed: int = 0) -> str:
    """Folder of the seeded model, written on first use."""
    folder = os.path.join(os.environ.get("WICK_SYNTH_CACHE", "/tmp/wick_b200_models"), f"{name}-s{seed}")
    if not os.path.exists(os.path.join(folder, "config.json")):
        spec = SPECS[name]
        write_folder(folder, spec.config(), spec.shapes(), spec.draw, seed)
    return folder
