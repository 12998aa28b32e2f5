// Decode form of the latent attention (kernels_latent.cu) on tcgen05, for bfloat16 models: one token per row (or a few
// consecutive ones), queries already taken to the latent's side.
//
// All heads of a token read the same cache rows, so the rows are the wide side of both products and the heads the narrow one.
// A CTA of four warps owns 64 consecutive keys of one row and up to LS_HEADS heads:
//   S^T [keys, heads] = K q^T      A: the cache rows as they lie, brought into the 128B-swizzled layout by cp.async
//   P^T = exp(S^T - max)           a thread per key; the split's maximum and sum of every head go to the partial record
//   O^T [latent, heads] = K^T P^T  A: the same tile again, read down its columns; 128 latent columns per MMA
// and leaves the sums to k_latent_sum.  A's rows 64..127 in the first product are whatever follows in shared memory; the
// accumulator rows that come of them are not read.  Every wait is bounded.  Bound: HBM (the cache rows once).
#include "latent_kernels.cuh"
#include "tc_common.cuh"

namespace wick {

namespace {

constexpr int LS_KEYS = LATENT_STEP_KEYS, LS_THREADS = 128, LS_HEADS = 32, LS_CHUNK = LS_KEYS * 128;
constexpr int LS_SMEM_MAX = 200 * 1024;

struct LsParams {
    const __nv_bfloat16 *qc, *q;
    int ldq, heads, groups, npad;  // npad: heads of a group up to a multiple of 16
    int chunks, mtiles;
    uint32_t tmem_cols;
    float* partial;
    uint32_t* err;
};

__device__ __forceinline__ void cp16_zfill(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ bool step_wait(const void* bar, uint32_t parity, volatile uint32_t* abort, uint32_t* err, uint32_t code) {
    return __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(bar), parity, abort, err, code));
}

// NP heads (padded) per group.
template <int NP>
__global__ void __launch_bounds__(LS_THREADS) k_latent_step(const __grid_constant__ LsParams p, const __grid_constant__ LatentShape s, const __grid_constant__ RowState rs) {
    extern __shared__ uint8_t ls_raw[];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ls_raw) + 1023) & ~(uintptr_t)1023);
    constexpr int QCHUNK = NP * 128;
    uint8_t* sk = sm;                                    // [chunks][64 keys][128 bytes], then 8 KB that the first product may read
    uint8_t* sq = sk + (p.chunks + 1) * LS_CHUNK;        // [chunks][NP][128 bytes]
    uint8_t* sp = sq + p.chunks * QCHUNK;                // [NP][128 bytes]
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(sp + QCHUNK);
    uint32_t* tmem_word = reinterpret_cast<uint32_t*>(bars + 2);
    volatile uint32_t* abort = tmem_word + 1;
    __shared__ float red[2][2][NP];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int j = blockIdx.y, h0 = blockIdx.z * LS_HEADS, hn = min(LS_HEADS, p.heads - h0), D = s.ldc(), pieces = p.chunks * 8;
    pdl_launch_next();
    pdl_wait();
    const int pos = rs.pos(j), lo = s.size > 0 ? max(0, pos - s.size + 1) : 0, keys = pos - lo + 1, t0 = blockIdx.x * LS_KEYS;
    if (t0 >= keys) return;
    const int cnt = min(LS_KEYS, keys - t0);
    {
        const __nv_bfloat16* cache = (const __nv_bfloat16*)rs.st0(j) + (size_t)(lo + t0) * D;
        for (int i = tid; i < LS_KEYS * pieces; i += LS_THREADS) {
            const int r = i / pieces, c = i % pieces;
            const bool ok = r < cnt && c * 8 < D;
            cp16_zfill(smem_u32(sk + (c >> 3) * LS_CHUNK + r * 128 + (((c & 7) ^ (r & 7)) << 4)), ok ? cache + (size_t)r * D + c * 8 : cache, ok);
        }
        const __nv_bfloat16* qc = p.qc + ((size_t)j * p.heads + h0) * D;
        const int rot_piece = s.off_rot() / 8;
        for (int i = tid; i < NP * pieces; i += LS_THREADS) {
            const int r = i / pieces, c = i % pieces;
            const bool ok = r < hn && c < rot_piece;
            const uint32_t dst = smem_u32(sq + (c >> 3) * QCHUNK + r * 128 + (((c & 7) ^ (r & 7)) << 4));
            if (r < hn && c >= rot_piece && c * 8 < D) continue;  // written below
            cp16_zfill(dst, ok ? qc + (size_t)r * D + c * 8 : qc, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        const int rot_pieces = (D - s.off_rot()) / 8;
        const float2* cs = s.rope + (size_t)pos * (s.rot_dims / 2);
        for (int i = tid; i < hn * rot_pieces; i += LS_THREADS) {
            const int r = i / rot_pieces, d0 = i % rot_pieces * 8, c = rot_piece + d0 / 8;
            uint4 v = *reinterpret_cast<const uint4*>(p.q + (size_t)j * p.ldq + (size_t)(h0 + r) * s.q_pitch() + s.q_off_rot() + d0);
            uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (d0 + 2 * e < s.rot_dims) {
                    const float2 t = cs[d0 / 2 + e];
                    const float a = __uint_as_float(w[e] << 16), b = __uint_as_float(w[e] & 0xffff0000u);
                    const __nv_bfloat162 x = __floats2bfloat162_rn(a * t.x - b * t.y, b * t.x + a * t.y);
                    w[e] = *reinterpret_cast<const uint32_t*>(&x);
                }
            *reinterpret_cast<uint4*>(sq + (c >> 3) * QCHUNK + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
        }
    }
    if (tid == 0) {
        mbar_init(smem_u32(&bars[0]), 1);
        mbar_init(smem_u32(&bars[1]), 1);
        *abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_word)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_word, lane_base = (uint32_t)(warp * 32) << 16;
    if (tid == 0) {
        const uint32_t idesc = umma_bf16_idesc(128, NP);
        for (int c = 0; c < p.chunks; c++) {
            const unsigned long long da = umma_desc_sw128(smem_u32(sk + c * LS_CHUNK)), db = umma_desc_sw128(smem_u32(sq + c * QCHUNK));
            const int steps = min(4, (D - c * 64 + 15) / 16);
            for (int kk = 0; kk < steps; kk++) umma_bf16(tmem, da + kk * 2, db + kk * 2, idesc, c > 0 || kk > 0);
        }
        umma_commit(smem_u32(&bars[0]));
    }
    bool ok = step_wait(&bars[0], 0, abort, p.err, 61);
    tc_fence_after();
    float v[NP], top[NP];
    constexpr float LOG2E = 1.4426950408889634f;
    const float scale = s.scale * LOG2E;
    if (warp < 2) {  // key tid of the tile
        if (ok) {
            int32_t raw[NP];
#pragma unroll
            for (int c = 0; c < NP; c += 16) tmem_ld16(tmem + lane_base + c, raw + c);
            tmem_ld_wait();
#pragma unroll
            for (int h = 0; h < NP; h++) v[h] = tid < cnt ? __int_as_float(raw[h]) * scale : -INFINITY;
        }
#pragma unroll
        for (int h = 0; h < NP; h++) {
            float m = ok ? v[h] : 0.0f;
#pragma unroll
            for (int x = 16; x > 0; x >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, x));
            if (lane == 0) red[0][warp][h] = m;
        }
    }
    __syncthreads();
    if (warp < 2) {
#pragma unroll
        for (int h = 0; h < NP; h++) {
            top[h] = fmaxf(red[0][0][h], red[0][1][h]);
            float e = ok ? exp2f(v[h] - top[h]) : 0.0f;
            *reinterpret_cast<__nv_bfloat16*>(sp + h * 128 + (((tid >> 3) ^ (h & 7)) << 4) + (tid & 7) * 2) = __float2bfloat16_rn(e);
#pragma unroll
            for (int x = 16; x > 0; x >>= 1) e += __shfl_xor_sync(0xffffffffu, e, x);
            if (lane == 0) red[1][warp][h] = e;
        }
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (tid == 0 && ok) {
        const uint32_t idesc = umma_bf16_idesc(128, NP) | UMMA_A_MN;
        for (int m = 0; m < p.mtiles; m++) {
            const unsigned long long da = umma_desc_mn_sw128(smem_u32(sk + 2 * m * LS_CHUNK), LS_CHUNK), db = umma_desc_sw128(smem_u32(sp));
#pragma unroll
            for (int kk = 0; kk < 4; kk++) umma_bf16(tmem + (m + 1) * NP, da + kk * (2048 >> 4), db + kk * 2, idesc, kk > 0);
        }
        umma_commit(smem_u32(&bars[1]));
    }
    const int C = s.kv_rank;
    float* out = p.partial + (((size_t)j * p.heads + h0) * gridDim.x + blockIdx.x) * (C + 2);
    const size_t head = (size_t)gridDim.x * (C + 2);
    if (tid < hn) {
        out[tid * head + C] = fmaxf(red[0][0][tid], red[0][1][tid]);
        out[tid * head + C + 1] = red[1][0][tid] + red[1][1][tid];
    }
    if (ok) ok = step_wait(&bars[1], 0, abort, p.err, 62);
    if (ok) {
        tc_fence_after();
        for (int m = 0; m < p.mtiles; m++) {
            int32_t raw[NP];
#pragma unroll
            for (int c = 0; c < NP; c += 16) tmem_ld16(tmem + lane_base + (m + 1) * NP + c, raw + c);
            tmem_ld_wait();
            const int c = m * 128 + tid;
            if (c < C)
#pragma unroll
                for (int h = 0; h < NP; h++)
                    if (h < hn) out[h * head + c] = __int_as_float(raw[h]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

size_t ls_plan(const LatentShape& s, LsParams* p) {
    p->heads = s.heads;
    p->groups = (s.heads + LS_HEADS - 1) / LS_HEADS;
    p->npad = s.heads <= 16 ? 16 : 32;
    p->chunks = (s.ldc() + 63) / 64;
    p->mtiles = (s.kv_rank + 127) / 128;
    const int cols = (1 + p->mtiles) * p->npad;
    p->tmem_cols = cols <= 64 ? 64 : cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
    if (cols > 512) return 0;
    // the second product reads chunks in pairs: the last one may be followed by the 8 KB of slack
    const size_t smem = (size_t)(p->chunks + 1) * LS_CHUNK + (size_t)(p->chunks + 1) * p->npad * 128 + 1024 + 256;
    return smem <= (size_t)LS_SMEM_MAX ? smem : 0;
}

}  // namespace

bool latent_step_supported(const LatentShape& s, int max_seq) {
    LsParams p{};
    return s.scale > 0.0f && (s.seen(max_seq) + LS_KEYS - 1) / LS_KEYS <= LATENT_MAX_SPLIT && ls_plan(s, &p) > 0;
}

cudaError_t launch_latent_step(cudaStream_t st, const void* qc, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs, float* partial,
                               int splits, uint32_t* err) {
    LsParams p{};
    const size_t smem = ls_plan(s, &p);
    if (!smem || !err) return cudaErrorInvalidValue;
    p.qc = (const __nv_bfloat16*)qc;
    p.q = (const __nv_bfloat16*)q;
    p.ldq = ldq;
    p.partial = partial;
    p.err = err;
    auto kernel = p.npad == 16 ? k_latent_step<16> : k_latent_step<32>;
    static cudaError_t configured[2] = {cudaFuncSetAttribute(k_latent_step<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, LS_SMEM_MAX),
                                        cudaFuncSetAttribute(k_latent_step<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, LS_SMEM_MAX)};
    for (cudaError_t e : configured)
        if (e != cudaSuccess) return e;
    g_kernel_launches++;
    return launch_pdl(kernel, dim3(splits, n, p.groups), dim3(LS_THREADS), smem, st, p, s, rs);
}

}  // namespace wick
