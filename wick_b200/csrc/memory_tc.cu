// Prompt form of the matrix memory (kernels_memory.cu has the equations) on tcgen05, for bfloat16 models: chunks of
// MEMORY_TC_CHUNK tokens.  q, k and v are bfloat16 as the projections leave them; everything that is f32 in the recurrence -
// the write weights times k, the states, the weights inside a chunk - enters a product as two bfloat16 terms, x = hi + lo, so that
// products keep about 16 bits and sums are f32.
//   k_memory_states_tc  CTA (chunk, head, 128 value channels): S^T [v, d] = V^T (w k)
//   k_memory_scan_tc    states at the chunks' starts, split into hi and lo; the final one in f32
//   k_memory_out_tc     CTA (chunk, head, VT value channels): S1 = q k^T, O2 = q S_0, z q; then P = S1 weighted, O1 = P V
// CTAs run one chunk each; there is no ring to keep full, other CTAs of the SM fill the gaps.  Every wait is bounded.
// Bound: HBM / L2 (the states once in each direction).
#include "memory_kernels.cuh"
#include "tc_common.cuh"

namespace wick {

namespace {

constexpr int TC = MEMORY_TC_CHUNK, BOX = 128 * TC;  // bytes of a box of 64 columns
constexpr int SMEM_MAX = 226 * 1024, OUT_SMEM_MAX = SMEM_MAX - 4096;  // (beside static shared memory)
static_assert(TC == 128, "rows of a chunk are the MMA's M");

__device__ __forceinline__ bool all_wait(const void* bar, uint32_t parity, volatile uint32_t* abort, uint32_t* err, uint32_t code) {
    return __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(bar), parity, abort, err, code));
}
// Two bfloat16 pairs: a = hi + lo.
__device__ __forceinline__ void split2(float a, float b, uint32_t* hi, uint32_t* lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
    *hi = *reinterpret_cast<const uint32_t*>(&h);
    *lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct TcTail {  // behind the tiles in shared memory
    unsigned long long bars[6];
    uint32_t tmem, abort;
};
__device__ __forceinline__ void tc_begin(TcTail* t, int bars, int warp, int tid, uint32_t cols) {
    if (tid == 0) {
        for (int i = 0; i < bars; i++) mbar_init(smem_u32(&t->bars[i]), 1);
        t->abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&t->tmem)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
}
__device__ __forceinline__ void tc_end(TcTail* t, int warp, uint32_t cols) {
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        if (*(volatile uint32_t*)&t->abort)
            for (int i = 0; i < 64; i++) __nanosleep(1000);  // copies issued before the failure may still be landing
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(t->tmem), "r"(cols) : "memory");
    }
}

// ── chunk sums ─────────────────────────────────────────────────────────────
struct StatesParams {
    CUtensorMap map_k, map_v;
    int n, cd, npad;  // boxes and MMA columns of the key channels
    uint32_t tmem_cols;
};

__global__ void __launch_bounds__(128) k_memory_states_tc(const __grid_constant__ StatesParams p, const __grid_constant__ MemoryShape s, const __grid_constant__ MemoryWork w) {
    extern __shared__ uint8_t st_raw[];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(st_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t *hi = sm, *lo = hi + p.cd * BOX, *sv = lo + p.cd * BOX;
    TcTail* tail = reinterpret_cast<TcTail*>(sv + 2 * BOX);
    const int tid = threadIdx.x, warp = tid >> 5, chunk = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 128, t0 = chunk * TC;
    const int H = s.heads, E = s.vdim, DP = s.dimp(), R = s.rows();
    tc_begin(tail, 2, warp, tid, p.tmem_cols);
    const uint32_t tmem = tail->tmem;
    if (tid == 0) {
        const uint32_t bar = smem_u32(&tail->bars[0]);
        mbar_arrive_expect_tx(bar, (p.cd + 2) * BOX);
        for (int c = 0; c < p.cd; c++) tma_load_3d(smem_u32(hi + c * BOX), &p.map_k, bar, c * 64, h, t0);
        for (int c = 0; c < 2; c++) tma_load_3d(smem_u32(sv + c * BOX), &p.map_v, bar, v0 + c * 64, h, t0);
    }
    const float weight = t0 + tid < p.n ? w.write[(size_t)h * p.n + t0 + tid] : 0.0f;
    bool ok = all_wait(&tail->bars[0], 0, &tail->abort, w.err, 71);
    if (ok)  // row tid of the key tile: k -> hi and lo of w k
        for (int c = 0; c < p.cd; c++)
#pragma unroll
            for (int q = 0; q < 8; q++) {
                uint4* at = reinterpret_cast<uint4*>(hi + c * BOX + tid * 128 + ((q ^ (tid & 7)) << 4));
                float f[8];
                bf16x8_f(*at, f);
                uint4 a, b;
                split2(f[0] * weight, f[1] * weight, &a.x, &b.x);
                split2(f[2] * weight, f[3] * weight, &a.y, &b.y);
                split2(f[4] * weight, f[5] * weight, &a.z, &b.z);
                split2(f[6] * weight, f[7] * weight, &a.w, &b.w);
                *at = a;
                *reinterpret_cast<uint4*>(lo + c * BOX + tid * 128 + ((q ^ (tid & 7)) << 4)) = b;
            }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    __syncthreads();
    if (tid == 0 && ok) {
        const uint32_t idesc = umma_bf16_idesc(128, p.npad) | UMMA_A_MN | UMMA_B_MN;
        for (int part = 0; part < 2; part++) {
            const unsigned long long da = umma_desc_mn_sw128(smem_u32(sv), BOX), db = umma_desc_mn_sw128(smem_u32(part ? lo : hi), BOX);
#pragma unroll
            for (int kk = 0; kk < TC / 16; kk++) umma_bf16(tmem, da + kk * (2048 >> 4), db + kk * (2048 >> 4), idesc, part > 0 || kk > 0);
        }
        umma_commit(smem_u32(&tail->bars[1]));
    }
    float* out = w.S + ((size_t)chunk * H + h) * R * DP;
    if (ok && blockIdx.x == 0)  // z: the sum of w k
        for (int d = tid; d < DP; d += 128) {
            float z = 0.0f;
            if (d < s.dim) {
                const uint8_t* col = hi + d / 64 * BOX + d % 8 * 2;
                const int piece = d % 64 / 8;
                const size_t to_lo = (size_t)p.cd * BOX;
#pragma unroll 8
                for (int j = 0; j < TC; j++) {
                    const uint8_t* at = col + j * 128 + ((piece ^ (j & 7)) << 4);
                    z += __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(at)) + __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(at + to_lo));
                }
            }
            out[(size_t)E * DP + d] = z;
        }
    if (ok) ok = all_wait(&tail->bars[1], 0, &tail->abort, w.err, 72);
    if (ok) {
        tc_fence_after();
        const int v = v0 + tid;  // tensor-memory lane
        float* row = out + (size_t)v * DP;
        for (int c = 0; c < DP; c += 16) {
            int32_t x[16];
            if (c < p.npad) {
                tmem_ld16(tmem + ((uint32_t)(warp * 32) << 16) + c, x);
                tmem_ld_wait();
            } else {
#pragma unroll
                for (int i = 0; i < 16; i++) x[i] = 0;
            }
            if (v < E)
#pragma unroll
                for (int i = 0; i < 16; i += 4) *reinterpret_cast<int4*>(row + c + i) = make_int4(x[i], x[i + 1], x[i + 2], x[i + 3]);
        }
    }
    tc_end(tail, warp, p.tmem_cols);
}

// ── states at the chunks' starts ───────────────────────────────────────────
// A thread per two elements, SB chunks in flight.
constexpr int SB = 8;
__global__ void __launch_bounds__(128) k_memory_scan_tc(int chunks, const __grid_constant__ MemoryShape s, float* __restrict__ state, const __grid_constant__ MemoryWork w) {
    const int h = blockIdx.y, per2 = s.rows() * s.dimp() / 2, i = blockIdx.x * 128 + threadIdx.x;
    if (i >= per2) return;
    float2* st = reinterpret_cast<float2*>(state) + (size_t)h * per2 + i;
    const float2* S = reinterpret_cast<const float2*>(w.S) + (size_t)h * per2 + i;
    uint32_t* hi = reinterpret_cast<uint32_t*>(w.S_hi) + (size_t)h * per2 + i;
    uint32_t* lo = reinterpret_cast<uint32_t*>(w.S_lo) + (size_t)h * per2 + i;
    const size_t step = (size_t)s.heads * per2;
    const float* keep = w.keep + (size_t)h * chunks;
    float2 cur = *st;
    for (int c0 = 0; c0 < chunks; c0 += SB) {
        float2 d[SB];
        float k[SB];
#pragma unroll
        for (int c = 0; c < SB; c++)
            if (c0 + c < chunks) {
                d[c] = S[(c0 + c) * step];
                k[c] = keep[c0 + c];
            }
#pragma unroll
        for (int c = 0; c < SB; c++)
            if (c0 + c < chunks) {
                split2(cur.x, cur.y, hi + (c0 + c) * step, lo + (c0 + c) * step);
                cur = make_float2(fmaf(cur.x, k[c], d[c].x), fmaf(cur.y, k[c], d[c].y));
            }
    }
    *st = cur;
}

// ── read-outs ──────────────────────────────────────────────────────────────
struct OutParams {
    CUtensorMap map_q, map_k, map_v, map_hi, map_lo, map_zhi, map_zlo;
    int n, cd, dim;
    int p_bytes;  // shared memory of k (then P hi) and of S hi (then P lo)
    int s_bytes;
};
constexpr int OUT_THREADS = 256;

// VT value channels per CTA.  Tensor memory: S1 [128] | O2 [VT] | O1 [VT] | z q [16].
template <int VT>
__global__ void __launch_bounds__(OUT_THREADS) k_memory_out_tc(const __grid_constant__ OutParams p, const __grid_constant__ MemoryShape s, const __grid_constant__ MemoryWork w) {
    extern __shared__ uint8_t out_raw[];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(out_raw) + 1023) & ~(uintptr_t)1023);
    constexpr int SBOX = VT * 128, ZBOX = 16 * 128, VB = VT / 64;
    constexpr uint32_t COLS = 512, O2 = 128, O1 = O2 + VT, ZQ = O1 + VT;
    uint8_t *sq = sm, *sk = sq + p.cd * BOX, *shi = sk + p.p_bytes, *slo = shi + p.s_bytes, *sv = slo + p.cd * SBOX, *sz = sv + VB * BOX;
    TcTail* tail = reinterpret_cast<TcTail*>(sz + 2 * p.cd * ZBOX);
    __shared__ double gs[TC];
    __shared__ float sums[2][TC];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, chunk = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VT, t0 = chunk * TC;
    const int H = s.heads, E = s.vdim, R = s.rows();
    tc_begin(tail, 6, warp, tid, COLS);
    const uint32_t tmem = tail->tmem;
    unsigned long long* bars = tail->bars;  // 0 q k, 1 states, 2 values; 3 S1 done, 4 O2 and z q done, 5 O1 done
    volatile uint32_t* abort = &tail->abort;
    if (tid == 0) {
        uint32_t bar = smem_u32(&bars[0]);
        mbar_arrive_expect_tx(bar, 2 * p.cd * BOX);
        for (int c = 0; c < p.cd; c++) {
            tma_load_3d(smem_u32(sq + c * BOX), &p.map_q, bar, c * 64, h, t0);
            tma_load_3d(smem_u32(sk + c * BOX), &p.map_k, bar, c * 64, h, t0);
        }
        const int row = (chunk * H + h) * R;
        bar = smem_u32(&bars[1]);
        mbar_arrive_expect_tx(bar, p.cd * (2 * SBOX + 2 * ZBOX));
        for (int c = 0; c < p.cd; c++) {
            tma_load_2d(smem_u32(shi + c * SBOX), &p.map_hi, bar, c * 64, row + v0);
            tma_load_2d(smem_u32(slo + c * SBOX), &p.map_lo, bar, c * 64, row + v0);
            tma_load_2d(smem_u32(sz + c * ZBOX), &p.map_zhi, bar, c * 64, row + E);
            tma_load_2d(smem_u32(sz + (p.cd + c) * ZBOX), &p.map_zlo, bar, c * 64, row + E);
        }
        bar = smem_u32(&bars[2]);
        mbar_arrive_expect_tx(bar, VB * BOX);
        for (int c = 0; c < VB; c++) tma_load_3d(smem_u32(sv + c * BOX), &p.map_v, bar, v0 + c * 64, h, t0);
        // S1 = q k^T, then O2 = q (hi + lo) and z q
        if (mbar_wait_bounded(smem_u32(&bars[0]), 0, abort, w.err, 73)) {
            tc_fence_after();
            for (int c = 0; c < p.cd; c++) {
                const unsigned long long da = umma_desc_sw128(smem_u32(sq + c * BOX)), db = umma_desc_sw128(smem_u32(sk + c * BOX));
                const int steps = min(4, (p.dim - c * 64 + 15) / 16);
                for (int kk = 0; kk < steps; kk++) umma_bf16(tmem, da + kk * 2, db + kk * 2, umma_bf16_idesc(128, TC), c > 0 || kk > 0);
            }
            umma_commit(smem_u32(&bars[3]));
        }
        if (mbar_wait_bounded(smem_u32(&bars[1]), 0, abort, w.err, 74)) {
            tc_fence_after();
            for (int part = 0; part < 2; part++)
                for (int c = 0; c < p.cd; c++) {
                    const unsigned long long da = umma_desc_sw128(smem_u32(sq + c * BOX)), db = umma_desc_sw128(smem_u32((part ? slo : shi) + c * SBOX)),
                                             dz = umma_desc_sw128(smem_u32(sz + (part * p.cd + c) * ZBOX));
                    const int steps = min(4, (p.dim - c * 64 + 15) / 16);
                    for (int kk = 0; kk < steps; kk++) {
                        const bool acc = part > 0 || c > 0 || kk > 0;
                        umma_bf16(tmem + O2, da + kk * 2, db + kk * 2, umma_bf16_idesc(128, VT), acc);
                        umma_bf16(tmem + ZQ, da + kk * 2, dz + kk * 2, umma_bf16_idesc(128, 16), acc);
                    }
                }
            umma_commit(smem_u32(&bars[4]));
        }
    }
    const int row = (warp & 3) * 32 + lane, half = warp >> 2, t = t0 + row;  // token of this thread's tensor-memory lane
    const bool live = t < p.n;
    const size_t at = (size_t)h * p.n + t;
    const double a = live ? w.a[at] : 0.0;
    const float carry = live ? w.carry[at] : 0.0f, floor_ = live ? expf(-w.m[at]) : 1.0f, qscale = 1.0f / sqrtf((float)p.dim);
    if (tid < TC) gs[tid] = t0 + tid < p.n ? w.g[(size_t)h * p.n + t0 + tid] : 0.0;
    __syncthreads();
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    // k and S hi are read until here and become P hi and P lo
    bool ok = all_wait(&bars[3], 0, abort, w.err, 75) && all_wait(&bars[4], 0, abort, w.err, 76);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    if (ok) {
        float sum = 0.0f;
        uint8_t *phi = sk + half * BOX + row * 128, *plo = shi + half * BOX + row * 128;
#pragma unroll 1
        for (int c0 = 0; c0 < 64; c0 += 16) {
            int32_t x[16];
            tmem_ld16(tmem + lane_base + half * 64 + c0, x);
            tmem_ld_wait();
            uint32_t hi[8], lo[8];
#pragma unroll
            for (int c = 0; c < 16; c += 2) {
                float f[2];
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int j = half * 64 + c0 + c + e;
                    f[e] = j <= row && live ? __int_as_float(x[c + e]) * qscale * __expf((float)(a + gs[j])) : 0.0f;
                    sum += f[e];
                }
                split2(f[0], f[1], &hi[c / 2], &lo[c / 2]);
            }
#pragma unroll
            for (int q = 0; q < 2; q++) {
                const int off = ((c0 / 8 + q) ^ (row & 7)) << 4;
                *reinterpret_cast<uint4*>(phi + off) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
                *reinterpret_cast<uint4*>(plo + off) = make_uint4(lo[4 * q], lo[4 * q + 1], lo[4 * q + 2], lo[4 * q + 3]);
            }
        }
        sums[half][row] = sum;
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (tid == 0 && ok && mbar_wait_bounded(smem_u32(&bars[2]), 0, abort, w.err, 77)) {
        tc_fence_after();
        const uint32_t idesc = umma_bf16_idesc(128, VT) | UMMA_B_MN;
        for (int part = 0; part < 2; part++)
            for (int c = 0; c < 2; c++) {
                const unsigned long long da = umma_desc_sw128(smem_u32((part ? shi : sk) + c * BOX));
                const unsigned long long db = umma_desc_mn_sw128(smem_u32(sv), BOX) + c * (64 * 128 >> 4);
#pragma unroll
                for (int kk = 0; kk < 4; kk++) umma_bf16(tmem + O1, da + kk * 2, db + kk * (2048 >> 4), idesc, part > 0 || c > 0 || kk > 0);
            }
        umma_commit(smem_u32(&bars[5]));
    }
    __syncwarp();
    if (ok) ok = all_wait(&bars[5], 0, abort, w.err, 78);
    if (ok) {
        tc_fence_after();
        int32_t z[8];
        tmem_ld8(tmem + lane_base + ZQ, z);
        tmem_ld_wait();
        const float den = fmaxf(fabsf(fmaf(carry * qscale, __int_as_float(z[0]), sums[0][row] + sums[1][row])), floor_) + 1e-6f, inv = 1.0f / den;
        const float old = carry * qscale;
        float* o = w.o + (size_t)t * H * E + (size_t)h * E + v0;
#pragma unroll 1
        for (int c0 = half * (VT / 2); c0 < (half + 1) * (VT / 2); c0 += 16) {
            int32_t x[16], y[16];
            tmem_ld16(tmem + lane_base + O1 + c0, x);
            tmem_ld16(tmem + lane_base + O2 + c0, y);
            tmem_ld_wait();
            if (live)
#pragma unroll
                for (int c = 0; c < 16; c += 4)
                    if (v0 + c0 + c < E) {  // vdim is a multiple of 8
                        float4 r;
                        r.x = fmaf(old, __int_as_float(y[c]), __int_as_float(x[c])) * inv;
                        r.y = fmaf(old, __int_as_float(y[c + 1]), __int_as_float(x[c + 1])) * inv;
                        r.z = fmaf(old, __int_as_float(y[c + 2]), __int_as_float(x[c + 2])) * inv;
                        r.w = fmaf(old, __int_as_float(y[c + 3]), __int_as_float(x[c + 3])) * inv;
                        *reinterpret_cast<float4*>(o + c0 + c) = r;
                    }
        }
    }
    tc_end(tail, warp, COLS);
}

size_t out_plan(const MemoryShape& s, int vt, OutParams* p) {
    p->cd = (s.dim + 63) / 64;
    p->dim = s.dim;
    p->p_bytes = std::max(p->cd, 2) * BOX;
    p->s_bytes = std::max(p->cd * vt * 128, 2 * BOX);
    return (size_t)p->cd * BOX + p->p_bytes + p->s_bytes + (size_t)p->cd * vt * 128 + (size_t)vt / 64 * BOX + 2 * (size_t)p->cd * 16 * 128 + 1024 + sizeof(TcTail);
}
int out_tile(const MemoryShape& s) {  // value channels per CTA, 0 if nothing fits
    OutParams p{};
    for (int vt : {128, 64})
        if ((vt == 64 || s.vdim > 64) && out_plan(s, vt, &p) <= (size_t)OUT_SMEM_MAX) return vt;
    return 0;
}

}  // namespace

bool memory_tc_supported(const MemoryShape& s) { return s.dim % 8 == 0 && s.vdim % 8 == 0 && s.dim <= 256 && out_tile(s) > 0; }

cudaError_t launch_memory_tc(cudaStream_t st, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, const MemoryWork& w) {
    using B = __nv_bfloat16;
    if (!memory_tc_supported(s) || !w.err || !w.S_hi) return cudaErrorInvalidValue;
    const int H = s.heads, D = s.dim, E = s.vdim, DP = s.dimp(), R = s.rows(), chunks = (a.n + TC - 1) / TC, vt = out_tile(s);
    const B* p = (const B*)a.p;
    StatesParams sp{};
    sp.n = a.n;
    sp.cd = (D + 63) / 64;
    sp.npad = round_up(D, 16);
    sp.tmem_cols = sp.npad <= 32 ? 32 : sp.npad <= 64 ? 64 : sp.npad <= 128 ? 128 : 256;
    OutParams op{};
    const size_t out_smem = out_plan(s, vt, &op), states_smem = (size_t)(2 * sp.cd + 2) * BOX + 1024 + sizeof(TcTail);
    op.n = a.n;
    cudaError_t e = encode_bf16_map3(p, a.n, H, D, D, a.ldp, TC, &op.map_q);
    if (e == cudaSuccess) e = encode_bf16_map3(p + H * D, a.n, H, D, D, a.ldp, TC, &op.map_k);
    if (e == cudaSuccess) e = encode_bf16_map3(p + 2 * H * D, a.n, H, E, E, a.ldp, TC, &op.map_v);
    if (e == cudaSuccess) e = encode_bf16_map(w.S_hi, chunks * H * R, DP, DP, vt, &op.map_hi);
    if (e == cudaSuccess) e = encode_bf16_map(w.S_lo, chunks * H * R, DP, DP, vt, &op.map_lo);
    if (e == cudaSuccess) e = encode_bf16_map(w.S_hi, chunks * H * R, DP, DP, 16, &op.map_zhi);
    if (e == cudaSuccess) e = encode_bf16_map(w.S_lo, chunks * H * R, DP, DP, 16, &op.map_zlo);
    if (e != cudaSuccess) return e;
    sp.map_k = op.map_k;
    sp.map_v = op.map_v;
    auto out_kernel = vt == 128 ? k_memory_out_tc<128> : k_memory_out_tc<64>;
    static cudaError_t configured[3] = {cudaFuncSetAttribute(k_memory_states_tc, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX),
                                        cudaFuncSetAttribute(k_memory_out_tc<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT_SMEM_MAX),
                                        cudaFuncSetAttribute(k_memory_out_tc<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT_SMEM_MAX)};
    for (cudaError_t c : configured)
        if (c != cudaSuccess) return c;
    g_kernel_launches += 3;
    k_memory_states_tc<<<dim3((E + 127) / 128, H, chunks), 128, states_smem, st>>>(sp, s, w);
    k_memory_scan_tc<<<dim3((R * DP / 2 + 127) / 128, H), 128, 0, st>>>(chunks, s, (float*)rs.s0, w);
    out_kernel<<<dim3((E + vt - 1) / vt, H, chunks), OUT_THREADS, out_smem, st>>>(op, s, w);
    return cudaGetLastError();
}

}  // namespace wick
