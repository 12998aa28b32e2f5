"""Operator-level entry points of libwick_cuda on torch CUDA tensors.

torch is only the device allocator here: every function hands raw device pointers to the
C ABI and launches on torch's current stream.  Names follow the wick functions they stand
in for (wick/src/backend/simd.rs, cpu.rs).
"""
from __future__ import annotations

import ctypes as C
from typing import Tuple

import numpy as np
import torch

from . import _lib
from ._lib import check

DT_Q4_0, DT_Q8_0 = 2, 8
QTYPE_ID = {"q4_0": DT_Q4_0, "q8_0": DT_Q8_0}


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: torch.Tensor) -> int:
    assert t.is_cuda and t.is_contiguous()
    return t.data_ptr()


class QuantWeight:
    """A quantised [m, k] matrix resident on the GPU in the library's layout (WeightRef, lfm2.rs:19-25)."""

    def __init__(self, dtype: int, raw: np.ndarray, m: int, k: int):
        raw = np.ascontiguousarray(raw, dtype=np.uint8)
        bb = 18 if dtype == DT_Q4_0 else 34
        assert raw.size == m * (k // 32) * bb, "raw block bytes do not match m x k"
        self._lib = _lib.load()
        self._h = C.c_void_p()
        self.dtype, self.m, self.k = dtype, m, k
        torch.cuda.init()
        check(self._lib.wick_cuda_weight_create(dtype, raw.ctypes.data, m, k, C.byref(self._h)))

    def close(self):
        if self._h.value:
            self._lib.wick_cuda_weight_destroy(self._h)
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


def quantize_f32_to_q8_0(x: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """simd.rs:255-323 over the rows of x [n, k] -> (scales [n, k/32] f32, quants [n, k] i8)."""
    x = x.contiguous()
    n, k = (1, x.shape[0]) if x.dim() == 1 else x.shape
    s = torch.empty((n, k // 32), dtype=torch.float32, device=x.device)
    q = torch.empty((n, k), dtype=torch.int8, device=x.device)
    check(_lib.load().wick_cuda_quantize_q8_0(_ptr(x), n, k, _ptr(s), _ptr(q), _stream()))
    return s, q


def gemv_q8(w: QuantWeight, xs: torch.Tensor, xq: torch.Tensor) -> torch.Tensor:
    """gemv_q4_0_q8_0_neon / gemv_q8_0_q8_0_neon (simd.rs:328-415, :440-524)."""
    y = torch.empty(w.m, dtype=torch.float32, device=xq.device)
    check(_lib.load().wick_cuda_gemv_q8(w._h, _ptr(xs), _ptr(xq), _ptr(y), _stream()))
    return y


def gemm_q8(w: QuantWeight, bs: torch.Tensor, bq: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """gemm_q*_q8_0_neon (simd.rs:696-1019) over the n rows of bq; returns token-major [n, m]."""
    n = bq.shape[0]
    if out is None:
        out = torch.empty((n, w.m), dtype=torch.float32, device=bq.device)
    check(_lib.load().wick_cuda_gemm_q8(w._h, _ptr(bs), _ptr(bq), n, _ptr(out), _stream()))
    return out


def gemm_q8_tc(w: QuantWeight, bs: torch.Tensor, bq: torch.Tensor, want_sums: bool = False):
    """The tensor-core (tcgen05) form of gemm_q8: exact int32 block sums, one fused f32 chain per output
    in block order.  Returns out [n, m] (and the block sums [n, m, k/32] when asked).  Synchronises."""
    n = bq.shape[0]
    out = torch.empty((n, w.m), dtype=torch.float32, device=bq.device)
    sums = torch.empty((n, w.m, w.k // 32), dtype=torch.int32, device=bq.device) if want_sums else None
    check(_lib.load().wick_cuda_gemm_q8_tc(w._h, _ptr(bs), _ptr(bq), n, _ptr(out), _ptr(sums) if want_sums else None,
                                           _stream()))
    return (out, sums) if want_sums else out


def gemm_q8_tc_exact(w: QuantWeight, bs: torch.Tensor, bq: torch.Tensor) -> torch.Tensor:
    """gemm_q8 on the tensor cores with the reference's accumulation order: bit-identical to gemm_q8."""
    n = bq.shape[0]
    out = torch.empty((n, w.m), dtype=torch.float32, device=bq.device)
    check(_lib.load().wick_cuda_gemm_q8_tc_exact(w._h, _ptr(bs), _ptr(bq), n, _ptr(out), _stream()))
    return out


def block_sums(w: QuantWeight, xq: torch.Tensor) -> torch.Tensor:
    s = torch.empty((w.m, w.k // 32), dtype=torch.int32, device=xq.device)
    check(_lib.load().wick_cuda_block_sums(w._h, _ptr(xq), _ptr(s), _stream()))
    return s


def rmsnorm_(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """cpu::rmsnorm (cpu.rs:577-594) on each row of x, in place."""
    n, dim = (1, x.shape[0]) if x.dim() == 1 else x.shape
    check(_lib.load().wick_cuda_rmsnorm(_ptr(x), _ptr(weight), n, dim, eps, _stream()))
    return x


def silu_mul_(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    check(_lib.load().wick_cuda_silu_mul(_ptr(gate), _ptr(up), gate.numel(), _stream()))
    return gate


def ggml_expf(x: torch.Tensor) -> torch.Tensor:
    y = torch.empty_like(x)
    check(_lib.load().wick_cuda_expf(_ptr(x), _ptr(y), x.numel(), _stream()))
    return y


def rope_(q: torch.Tensor, k: torch.Tensor, pos: int, n_heads: int, n_kv_heads: int, head_dim: int, freq_base: float):
    check(_lib.load().wick_cuda_rope(_ptr(q), _ptr(k), pos, n_heads, n_kv_heads, head_dim, freq_base, _stream()))
    return q, k


def qknorm_rope_kv_(q, k, v, q_norm, k_norm, eps: float, rope_cos, rope_sin, k_cache, v_cache, start_pos: int, n_heads: int,
                    n_kv_heads: int, head_dim: int):
    """Per-head RMSNorm of Q and K, RoPE from a (position, pair) cos / sin table, and the append of the rotated K rows
    and the V rows to the caches at rows start_pos.. (lfm2.rs:783-855) for the n rows of q [n, n_heads * head_dim]."""
    n = q.shape[0]
    check(_lib.load().wick_cuda_qknorm_rope_kv(_ptr(q), _ptr(k), _ptr(v), _ptr(q_norm), _ptr(k_norm), eps, _ptr(rope_cos), _ptr(rope_sin),
                                               _ptr(k_cache), _ptr(v_cache), n, start_pos, n_heads, n_kv_heads, head_dim, _stream()))
    return q


def attention_decode(q, k_cache, v_cache, n_heads, n_kv_heads, head_dim, seq) -> torch.Tensor:
    out = torch.empty(n_heads * head_dim, dtype=torch.float32, device=q.device)
    check(_lib.load().wick_cuda_attention_decode(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), n_heads, n_kv_heads,
                                                 head_dim, seq, _stream()))
    return out


def attention_decode_splitk(q, k_cache, v_cache, n_heads, n_kv_heads, head_dim, seq) -> torch.Tensor:
    """Opt-in split-K single-query attention (runs of 256 keys + merge); agrees with attention_decode within rounding."""
    out = torch.empty(n_heads * head_dim, dtype=torch.float32, device=q.device)
    check(_lib.load().wick_cuda_attention_decode_splitk(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), n_heads, n_kv_heads,
                                                        head_dim, seq, _stream()))
    return out


def attention_prefill(q, k_cache, v_cache, n, start_pos, n_heads, n_kv_heads, head_dim, flash: bool) -> torch.Tensor:
    out = torch.empty((n, n_heads * head_dim), dtype=torch.float32, device=q.device)
    check(_lib.load().wick_cuda_attention_prefill(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), n, start_pos, n_heads,
                                                  n_kv_heads, head_dim, int(flash), _stream()))
    return out


def shortconv(proj: torch.Tensor, conv_w: torch.Tensor, state: torch.Tensor, kernel_size: int) -> torch.Tensor:
    n, three_hs = proj.shape
    hs = three_hs // 3
    out = torch.empty((n, hs), dtype=torch.float32, device=proj.device)
    check(_lib.load().wick_cuda_shortconv(_ptr(proj), _ptr(conv_w), _ptr(state), _ptr(out), n, hs, kernel_size, _stream()))
    return out


# ── operators of the config.json models; the activation type is that of the tensors ────────────────────
_DENSE_PATHS = {"auto": 0, "rows": 1, "f32": 2, "tensor": 3}
_ACTIVATIONS = {"relu": 0, "silu": 1, "relu2": 2, "none": 3}


def _compute(t: torch.Tensor) -> int:
    return {torch.bfloat16: 1, torch.float32: 2}[t.dtype]


def _opt(t) -> int | None:
    return None if t is None else _ptr(t)


def pad8(t: torch.Tensor) -> torch.Tensor:
    """Rows of a matrix zero-padded to a multiple of 8 columns."""
    return torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)).contiguous()


def dense(w: torch.Tensor, x: torch.Tensor, w_up: torch.Tensor | None = None, activation: str | None = None, softcap: float = 0.0,
          out_f32: bool = True, path: str = "auto") -> torch.Tensor:
    """activation(x [n, k] (bf16 or f32) times bf16 w [m, k] transposed); with w_up: activation(w x) * (w_up x).  The activation is
    none by default, with w_up relu."""
    activation = activation or ("none" if w_up is None else "relu")
    (m, k), n = w.shape, x.shape[0]
    w8, u8, x8 = pad8(w), None if w_up is None else pad8(w_up), pad8(x)
    y = torch.empty((n, m), dtype=torch.float32 if out_f32 else x.dtype, device=x.device)
    check(_lib.load().wick_cuda_dense(_compute(x), _ptr(w8), _opt(u8), m, k, w8.shape[1], _ptr(x8), x8.shape[1], n, _ptr(y), m, int(out_f32),
                                      _ACTIVATIONS[activation], softcap, _DENSE_PATHS[path], _stream()))
    return y


def hyper_norm(x: torch.Tensor, gain: torch.Tensor, eps: float, w_in=None, y=None, mix=None, w_out=None, dtype=torch.float32) -> torch.Tensor:
    """Hyper-connection write (in place on x [n, streams, width]), read and RMS norm; returns h [n, width] of `dtype`."""
    n, s, w = x.shape
    h = torch.zeros((n, w + -w % 8), dtype=dtype, device=x.device)
    check(_lib.load().wick_cuda_hyper_norm(_compute(h), _ptr(x), n, s, w, _opt(y), _opt(mix), _opt(w_out), _opt(w_in), _ptr(gain), eps, _ptr(h),
                                           h.shape[1], _stream()))
    return h[:, :w]


def mix_attention(qkv: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, start_pos: int, heads: int, kv_heads: int, dim: int, vdim: int,
                  scale: float, eps: float, size: int, keep_first: int, talk=None, bias=None) -> torch.Tensor:
    """Windowed attention with head-blended sigmoid scores; appends to the caches [max_seq, kv_heads * dim | vdim]."""
    n = qkv.shape[0]
    q8 = pad8(qkv)
    out = torch.zeros((n, heads * vdim + -(heads * vdim) % 8), dtype=qkv.dtype, device=qkv.device)
    check(_lib.load().wick_cuda_mix_attention(_compute(qkv), _ptr(q8), q8.shape[1], n, start_pos, _ptr(k_cache), _ptr(v_cache), k_cache.shape[0],
                                              _opt(talk), _opt(bias), heads, kv_heads, dim, vdim, scale, eps, size, keep_first, _ptr(out),
                                              out.shape[1], _stream()))
    return out[:, :heads * vdim]


def channel_delta(proj: torch.Tensor, off_beta: int, decay: torch.Tensor, gate: torch.Tensor, conv_w: torch.Tensor, a_log: torch.Tensor,
                  dt_bias: torch.Tensor, norm: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int, eps: float, state: torch.Tensor,
                  conv_state: torch.Tensor) -> torch.Tensor:
    """Short convolutions, channel-decay delta rule and gated output norm; state and conv_state are updated."""
    n = proj.shape[0]
    out = torch.zeros((n, heads * vdim), dtype=proj.dtype, device=proj.device)
    check(_lib.load().wick_cuda_channel_delta(_compute(proj), _ptr(proj), proj.shape[1], off_beta, _ptr(decay), _ptr(gate), _ptr(conv_w), _ptr(a_log),
                                              _ptr(dt_bias), _ptr(norm), n, heads, kv_heads, dim, vdim, conv_w.shape[1], eps, _ptr(state),
                                              _ptr(conv_state), _ptr(out), heads * vdim, _stream()))
    return out


def residual_norm(x: torch.Tensor, eps: float, gain=None, x0=None, y=None, post=None, shift=None, y_rows=None, y_parts: int = 1, y_scale: float = 1.0,
                  h_rows=None, h_parts: int = 1, dtype=torch.float32) -> torch.Tensor:
    """Residual update (in place on x [n, width] f32) and the next sublayer's input: [n, width], or [n, 2 width] with x0."""
    n, w = x.shape
    wide = w if gain is not None else 2 * w
    h = torch.zeros((n * h_parts if h_rows is not None else n, wide + -wide % 8), dtype=dtype, device=x.device)
    check(_lib.load().wick_cuda_residual_norm(_compute(h), _ptr(x), n, w, _opt(y), y_parts, _opt(y_rows), y_scale, _opt(post), _opt(shift), _opt(gain), _opt(x0),
                                              eps, _ptr(h), h.shape[1], h_parts, _opt(h_rows), _stream()))
    return h[:, :wide]


def _up8(n: int) -> int:
    return n + -n % 8


def latent_weights(uq: torch.Tensor, uk: torch.Tensor, uv: torch.Tensor, heads: int, dim: int, rot_dim: int, vdim: int):
    """The layouts that latent_attention takes, from uq [heads * (dim + rot_dim), q_rank], uk [heads * dim, kv_rank] and
    uv [heads * vdim, kv_rank] (bfloat16)."""
    d8, r8, v8, c = _up8(dim), _up8(rot_dim), _up8(vdim), uk.shape[1]
    q = uq.new_zeros((heads, d8 + r8, _up8(uq.shape[1])))
    u = uq.view(heads, dim + rot_dim, -1)
    q[:, :dim, :uq.shape[1]] = u[:, :dim]
    q[:, d8:d8 + rot_dim, :uq.shape[1]] = u[:, dim:]
    k_t = pad8(uk.view(heads, dim, c).transpose(1, 2))
    kv = uk.new_zeros((heads * (d8 + v8), _up8(c)))
    kv[:heads * d8].view(heads, d8, -1)[:, :dim, :c] = uk.view(heads, dim, c)
    kv[heads * d8:].view(heads, v8, -1)[:, :vdim, :c] = uv.view(heads, vdim, c)
    return q, k_t, pad8(uv), kv


_LATENT_FORMS = {"auto": 0, "absorbed": 1, "prompt": 2}


def latent_attention(p: torch.Tensor, cache: torch.Tensor, start_pos: int, weights, sink, q_norm, kv_norm, rope, heads: int, dim: int, rot_dim: int,
                     rot_dims: int, vdim: int, q_rank: int, kv_rank: int, size: int, scale: float, eps: float, form: str = "auto") -> torch.Tensor:
    """Latent attention with a sink; p [n, q_rank up to 8 | kv_rank | rot_dim] (its query latent is normalised in place in a copy),
    weights from latent_weights(); appends to cache [max_seq, kv_rank up to 8 | rot_dim up to 8]."""
    p8, n = pad8(p), p.shape[0]
    if p8.data_ptr() == p.data_ptr():
        p8 = p8.clone()
    uq, uk_t, uv, ukv = weights
    out = torch.zeros((n, _up8(heads * vdim)), dtype=p.dtype, device=p.device)
    check(_lib.load().wick_cuda_latent_attention(_compute(p), _ptr(p8), p8.shape[1], n, start_pos, _ptr(cache), cache.shape[0], _ptr(uq), _ptr(uk_t), _ptr(uv),
                                                 _ptr(ukv) if p.dtype == torch.bfloat16 else None, _ptr(sink), _ptr(q_norm), _ptr(kv_norm), _ptr(rope), heads, dim,
                                                 rot_dim, rot_dims, vdim, q_rank, kv_rank, size, scale, eps, _LATENT_FORMS[form], _ptr(out), out.shape[1], _stream()))
    return out[:, :heads * vdim]


def matrix_memory(p: torch.Tensor, gates: torch.Tensor, i_bias, f_bias, norm, heads: int, dim: int, vdim: int, cap: float, eps: float,
                  state: torch.Tensor, m: torch.Tensor, step: bool = False) -> torch.Tensor:
    """Matrix memory with exponential gates, gated output norm; state [heads, vdim + 1, dim up to 32] and m [heads] are updated."""
    n, p8 = p.shape[0], pad8(p)
    out = torch.zeros((n, _up8(heads * vdim)), dtype=p.dtype, device=p.device)
    check(_lib.load().wick_cuda_matrix_memory(_compute(p), _ptr(p8), p8.shape[1], _ptr(gates), gates.shape[1], n, heads, dim, vdim, cap, eps, _ptr(i_bias),
                                              _ptr(f_bias), _ptr(norm), _ptr(state), _ptr(m), int(step), _ptr(out), out.shape[1], _stream()))
    return out[:, :heads * vdim]


def argmax(logits: torch.Tensor) -> torch.Tensor:
    out = torch.empty(1, dtype=torch.int32, device=logits.device)
    check(_lib.load().wick_cuda_argmax(_ptr(logits), logits.numel(), _ptr(out), _stream()))
    return out


def sample_logits(logits: torch.Tensor, temperature: float, top_k: int, top_p: float, r: float) -> int:
    """Sampler::sample (sampler.rs:64-158) on device logits with the caller's uniform draw r."""
    out = torch.empty(1, dtype=torch.int32, device=logits.device)
    check(_lib.load().wick_cuda_sample_logits(_ptr(logits), logits.numel(), temperature, top_k, top_p, r, _ptr(out), _stream()))
    return int(out.item())


ARGMAX_NOALLOC_MAX = 4096 * 1024


def argmax_noalloc(logits: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Same result as argmax() for callers that may not allocate: the scratch is a fixed array inside
    the library and the caller supplies `out` (one int32 on the device).  At most ARGMAX_NOALLOC_MAX
    logits.  Calls share that array, so keep them on one stream."""
    lib = _lib.load()
    code = lib.wick_cuda_argmax_noalloc(_ptr(logits), logits.numel(), _ptr(out), _stream())
    if code != 0:
        raise _lib.WickCudaError(code, lib.wick_cuda_argmax_noalloc_last_error().decode())
    return out
