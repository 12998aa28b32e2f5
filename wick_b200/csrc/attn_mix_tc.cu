// Prompt form of the windowed attention with blended sigmoid scores (kernels_mixattn.cu) on tcgen05, for bfloat16 models.
//
// The blend of the heads' scores is linear, so it moves to the query side: with head h's folded query
//     q'_h = concat over kv heads j of  scale * sum over the heads g that use j of talk[h][g] q_g          (length G * dim)
// the blended score is one dot product, sum_g talk[h][g] scale q_g . k_{kv(g)} = q'_h . concat_j(k_j), against a whole cached K
// row.  k_qk_fold_append computes q' in f32 from the f32 normalised queries and rounds once, where the unfused form rounds q;
// after that the output heads are independent of each other.
//
// k_mix_attn_tc: a CTA owns 128 queries of one head and walks over tiles of 64 keys (the kept first keys, then the window):
//   warp 0  lane 0: TMA - q' once (or chunk by chunk when it does not fit), K in chunks of 64 columns, V
//   warp 1  lane 0: S = q' K^T into one of two tensor-memory buffers, then O += P V of the tile before
//   warps 2..17   : P = sigmoid(S + bias) masked to the visible keys, rounded to bf16 into shared memory in the 128B-swizzled
//                   layout of the MMA's A operand; at the end O -> out
// There is no normaliser and no running maximum, so O is accumulated in tensor memory from the first tile to the last.
// Every wait is bounded.  Bound: tensor pipe (G-fold redundant score products) and the special-function unit (exp and
// reciprocal per query, key and head).
#include "hybrid_kernels.cuh"
#include "tc_common.cuh"

namespace wick {

namespace {

constexpr int MT_Q = 128, MT_K = 64, MT_EPI_WARPS = 16, MT_THREADS = 32 * (2 + MT_EPI_WARPS);
constexpr int MT_QCHUNK = MT_Q * 64 * 2, MT_KCHUNK = MT_K * 64 * 2, MT_P = MT_Q * MT_K * 2;
constexpr int MT_SMEM_MAX = 226 * 1024;

struct MtParams {
    CUtensorMap map_q, map_k, map_v;
    __nv_bfloat16* out;
    const float* bias;
    int ldo, n, start_pos;
    int kd, chunks, vdim, vboxes, rep;   // kd = G * dim columns of a K row, in chunks of 64; vboxes of 64 V columns
    int size, keep;
    int q_resident, k_stages, v_stages, p_bufs;
    uint32_t tmem_cols;
    uint32_t* err;
};

__global__ void __launch_bounds__(MT_THREADS, 1) k_mix_attn_tc(const __grid_constant__ MtParams p) {
    extern __shared__ uint8_t mt_raw[];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(mt_raw) + 1023) & ~(uintptr_t)1023);
    const int k_stage = MT_KCHUNK + (p.q_resident ? 0 : MT_QCHUNK), v_stage = p.vboxes * MT_KCHUNK;
    uint8_t* sq = sm;
    uint8_t* sk = sq + (p.q_resident ? p.chunks * MT_QCHUNK : 0);
    uint8_t* sv = sk + p.k_stages * k_stage;
    uint8_t* sp = sv + p.v_stages * v_stage;
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(sp + p.p_bufs * MT_P);
    unsigned long long *q_full = bars, *o_full = bars + 1, *k_full = bars + 2, *k_empty = k_full + 8, *v_full = k_empty + 8, *v_empty = v_full + 2,
                       *s_full = v_empty + 2, *s_empty = s_full + 2, *p_full = s_empty + 2, *p_empty = p_full + 2;
    uint32_t* tmem_word = reinterpret_cast<uint32_t*>(p_empty + 2);
    volatile uint32_t* abort = tmem_word + 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, row0 = (gridDim.y - 1 - blockIdx.y) * MT_Q;  // the longest walks start first
    const int nq = min(MT_Q, p.n - row0), p0 = p.start_pos + row0, p1 = p0 + nq - 1;
    const int lo = p.size > 0 ? max(0, p0 - p.size + 1) : 0, ns = min(p.keep, lo);
    const int kept_tiles = (ns + MT_K - 1) / MT_K, tiles = kept_tiles + (p1 - lo + MT_K) / MT_K;

    if (threadIdx.x == 0) {
        mbar_init(smem_u32(q_full), 1);
        mbar_init(smem_u32(o_full), 1);
        for (int i = 0; i < p.k_stages; i++) {
            mbar_init(smem_u32(&k_full[i]), 1);
            mbar_init(smem_u32(&k_empty[i]), 1);
        }
        for (int i = 0; i < 2; i++) {
            mbar_init(smem_u32(&v_full[i]), 1);
            mbar_init(smem_u32(&v_empty[i]), 1);
            mbar_init(smem_u32(&s_full[i]), 1);
            mbar_init(smem_u32(&s_empty[i]), MT_EPI_WARPS);
            mbar_init(smem_u32(&p_full[i]), MT_EPI_WARPS);
            mbar_init(smem_u32(&p_empty[i]), 1);
        }
        *abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_word)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_word, tmem_o = tmem + 2 * MT_K;

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            if (p.q_resident) {
                mbar_arrive_expect_tx(smem_u32(q_full), p.chunks * MT_QCHUNK);
                for (int c = 0; c < p.chunks; c++) tma_load_2d(smem_u32(sq + c * MT_QCHUNK), &p.map_q, smem_u32(q_full), h * p.kd + c * 64, row0);
            }
            uint32_t g = 0;
            const int vcol = h / p.rep * p.vdim;
            for (int t = 0; t < tiles && ok; t++) {
                const int key0 = t < kept_tiles ? t * MT_K : lo + (t - kept_tiles) * MT_K;
                for (int c = 0; c < p.chunks; c++, g++) {
                    const int s = g % p.k_stages;
                    ok = mbar_wait_bounded(smem_u32(&k_empty[s]), ((g / p.k_stages) & 1) ^ 1, abort, p.err, 21);
                    if (!ok) break;
                    const uint32_t bar = smem_u32(&k_full[s]), dst = smem_u32(sk + s * k_stage);
                    mbar_arrive_expect_tx(bar, k_stage);
                    tma_load_2d(dst, &p.map_k, bar, c * 64, key0);
                    if (!p.q_resident) tma_load_2d(dst + MT_KCHUNK, &p.map_q, bar, h * p.kd + c * 64, row0);
                }
                if (!ok) break;
                const int s = t % p.v_stages;
                ok = mbar_wait_bounded(smem_u32(&v_empty[s]), ((t / p.v_stages) & 1) ^ 1, abort, p.err, 22);
                if (!ok) break;
                mbar_arrive_expect_tx(smem_u32(&v_full[s]), v_stage);
                for (int b = 0; b < p.vboxes; b++)
                    tma_load_2d(smem_u32(sv + s * v_stage + b * MT_KCHUNK), &p.map_v, smem_u32(&v_full[s]), vcol + b * 64, key0);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_bf16_idesc(MT_Q, MT_K);
            const uint32_t idesc_o = umma_bf16_idesc(MT_Q, round_up(p.vdim, 16)) | UMMA_B_MN;  // V
            uint32_t g = 0;
            bool ok = !p.q_resident || mbar_wait_bounded(smem_u32(q_full), 0, abort, p.err, 23);
            for (int t = 0; t <= tiles && ok; t++) {
                if (t < tiles) {
                    const int b = t & 1;
                    ok = mbar_wait_bounded(smem_u32(&s_empty[b]), ((t >> 1) & 1) ^ 1, abort, p.err, 24);
                    if (!ok) break;
                    tc_fence_after();
                    for (int c = 0; c < p.chunks; c++, g++) {
                        const int s = g % p.k_stages;
                        ok = mbar_wait_bounded(smem_u32(&k_full[s]), (g / p.k_stages) & 1, abort, p.err, 25);
                        if (!ok) break;
                        tc_fence_after();
                        const uint32_t ka = smem_u32(sk + s * k_stage);
                        const unsigned long long db = umma_desc_sw128(ka);
                        const unsigned long long da = umma_desc_sw128(p.q_resident ? smem_u32(sq + c * MT_QCHUNK) : ka + MT_KCHUNK);
#pragma unroll
                        for (int kk = 0; kk < 4; kk++) umma_bf16(tmem + b * MT_K, da + kk * 2, db + kk * 2, idesc_s, c > 0 || kk > 0);
                        umma_commit(smem_u32(&k_empty[s]));
                    }
                    if (!ok) break;
                    umma_commit(smem_u32(&s_full[b]));
                }
                if (t > 0) {
                    const int u = t - 1, pb = u % p.p_bufs, vs = u % p.v_stages;
                    ok = mbar_wait_bounded(smem_u32(&p_full[pb]), (u / p.p_bufs) & 1, abort, p.err, 26) &&
                         mbar_wait_bounded(smem_u32(&v_full[vs]), (u / p.v_stages) & 1, abort, p.err, 27);
                    if (!ok) break;
                    tc_fence_after();
                    const unsigned long long da = umma_desc_sw128(smem_u32(sp + pb * MT_P));
                    const unsigned long long db = umma_desc_mn_sw128(smem_u32(sv + vs * v_stage), MT_KCHUNK);
#pragma unroll
                    for (int kk = 0; kk < 4; kk++) umma_bf16(tmem_o, da + kk * 2, db + kk * (2048 >> 4), idesc_o, u > 0 || kk > 0);
                    umma_commit(smem_u32(&v_empty[vs]));
                    umma_commit(smem_u32(&p_empty[pb]));
                }
            }
            if (ok) umma_commit(smem_u32(o_full));
        }
    } else {
        // lanes 32 (warp % 4).. and 16 of the 64 key columns
        const int quarter = warp & 3, part = (warp - 2) >> 2, r = quarter * 32 + lane, qi = p0 + r;
        constexpr float LOG2E = 1.4426950408889634f;
        const float bias = p.bias ? p.bias[h] * -LOG2E : 0.0f;
        const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
        bool ok = true;
        for (int t = 0; t < tiles; t++) {
            const int b = t & 1;
            ok = mbar_wait_bounded(smem_u32(&s_full[b]), (t >> 1) & 1, abort, p.err, 28);
            if (!ok) break;
            tc_fence_after();
            int32_t v[16];
            tmem_ld16(tmem + lane_base + b * MT_K + part * 16, v);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s_empty[b]));
            const bool kept = t < kept_tiles;
            const int key0 = (kept ? t * MT_K : lo + (t - kept_tiles) * MT_K);
            const bool all = kept ? key0 + MT_K <= ns : key0 + MT_K - 1 <= p0 && (p.size <= 0 || p1 - key0 < p.size);
            // sigmoid(z) = 1 / (1 + 2^(-z log2 e))
            float f[16];
#pragma unroll
            for (int c = 0; c < 16; c++) {
                float e;
                asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fmaf(__int_as_float(v[c]), -LOG2E, bias)));
                asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(f[c]) : "f"(1.0f + e));
            }
            if (!all) {
#pragma unroll
                for (int c = 0; c < 16; c++) {
                    const int j = key0 + part * 16 + c;
                    const bool vis = kept ? j < ns : j <= qi && (p.size <= 0 || qi - j < p.size || j < p.keep);
                    f[c] = vis ? f[c] : 0.0f;
                }
            }
            uint32_t w[8];
#pragma unroll
            for (int c = 0; c < 8; c++) {
                const __nv_bfloat162 q = __floats2bfloat162_rn(f[2 * c], f[2 * c + 1]);
                w[c] = *reinterpret_cast<const uint32_t*>(&q);
            }
            const int pb = t % p.p_bufs;
            ok = mbar_wait_bounded(smem_u32(&p_empty[pb]), ((t / p.p_bufs) & 1) ^ 1, abort, p.err, 29);
            if (!ok) break;
            uint8_t* prow = sp + pb * MT_P + r * 128;
#pragma unroll
            for (int c = 0; c < 2; c++)
                *reinterpret_cast<uint4*>(prow + (((part * 2 + c) ^ (r & 7)) << 4)) = make_uint4(w[4 * c], w[4 * c + 1], w[4 * c + 2], w[4 * c + 3]);
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&p_full[pb]));
        }
        if (ok && mbar_wait_bounded(smem_u32(o_full), 0, abort, p.err, 30)) {
            tc_fence_after();
            __nv_bfloat16* dst = p.out + (size_t)(row0 + r) * p.ldo + h * p.vdim;
            for (int c0 = part * 16; c0 < p.vdim; c0 += 64) {
                int32_t v[16];
                tmem_ld16(tmem_o + lane_base + c0, v);
                tmem_ld_wait();
                if (r < nq) {
#pragma unroll
                    for (int q = 0; q < 2; q++)
                        if (c0 + q * 8 < p.vdim) {  // vdim is a multiple of 8
                            uint32_t w[4];
#pragma unroll
                            for (int e = 0; e < 4; e++) {
                                const __nv_bfloat162 x = __floats2bfloat162_rn(__int_as_float(v[q * 8 + 2 * e]), __int_as_float(v[q * 8 + 2 * e + 1]));
                                w[e] = *reinterpret_cast<const uint32_t*>(&x);
                            }
                            *reinterpret_cast<uint4*>(dst + c0 + q * 8) = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        if (*abort)
            for (int i = 0; i < 64; i++) __nanosleep(1000);  // copies issued before the failure may still be landing
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

// Per row: q heads divided by their root mean square and folded (see above), k heads normalised into the cache, v into the cache.
__global__ void __launch_bounds__(256) k_qk_fold_append(const __nv_bfloat16* __restrict__ qkv, int ld, const __grid_constant__ MixAttnShape s,
                                                        const __grid_constant__ RowState rs, __nv_bfloat16* __restrict__ fold) {
    extern __shared__ float qn[];  // [H*D] f32
    const int H = s.heads, G = s.kv_heads, D = s.dim, E = s.vdim, rep = H / G, j = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const __nv_bfloat16* row = qkv + (size_t)j * ld;
    const int pos = rs.pos(j);
    __nv_bfloat16* kc = (__nv_bfloat16*)rs.st0(j) + (size_t)pos * G * D;
    __nv_bfloat16* vc = (__nv_bfloat16*)rs.st1(j) + (size_t)pos * G * E;
    for (int seg = warp; seg < H + G; seg += 8) {
        const __nv_bfloat16* src = row + seg * D;
        float ss = 0.0f;
        for (int i = lane; i < D; i += 32) {
            const float v = act_f(src[i]);
            ss = fmaf(v, v, ss);
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)D + s.eps);
        for (int i = lane; i < D; i += 32) {
            const float v = act_f(src[i]) * r;
            if (seg < H) qn[seg * D + i] = v;
            else kc[(seg - H) * D + i] = __float2bfloat16_rn(v);
        }
    }
    for (int i = threadIdx.x; i < G * E; i += 256) vc[i] = row[(H + G) * D + i];
    __syncthreads();
    const int KD = G * D, half = KD / 2;  // KD is a multiple of 8: two columns per step
    __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(fold + (size_t)j * H * KD);
    for (int i = threadIdx.x; i < H * half; i += 256) {
        const int h = i / half;
        float f[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int c = (i % half) * 2 + e, g0 = c / D * rep, d = c % D;
            float a = 0.0f;
            for (int r = 0; r < rep; r++) a = fmaf(s.talk ? s.talk[h * H + g0 + r] : (h == g0 + r ? 1.0f : 0.0f), qn[(g0 + r) * D + d], a);
            f[e] = a * s.scale;
        }
        dst[i] = __floats2bfloat162_rn(f[0], f[1]);
    }
}

// Shared memory plan: false if the shape does not fit.
bool mt_plan(const MixAttnShape& s, MtParams* p, size_t* smem) {
    if (s.vdim % 8 || (s.kv_heads * s.dim) % 8 || s.vdim > 256 || (size_t)s.heads * s.dim * 4 > 160 * 1024) return false;
    p->kd = s.kv_heads * s.dim;
    p->chunks = (p->kd + 63) / 64;
    p->vdim = s.vdim;
    p->vboxes = (s.vdim + 63) / 64;
    p->rep = s.heads / s.kv_heads;
    p->tmem_cols = s.vdim <= 128 ? 256 : 512;
    const int bars = 1024 + 256;
    for (int resident = 1; resident >= 0; resident--) {
        p->q_resident = resident;
        const int q = resident ? p->chunks * MT_QCHUNK : 0, ks = MT_KCHUNK + (resident ? 0 : MT_QCHUNK), v = p->vboxes * MT_KCHUNK;
        const int tries[4][2] = {{2, 2}, {2, 1}, {1, 2}, {1, 1}};  // V stages, P buffers
        // enough K chunks in flight to cover a trip to L2 matter more than second V and P buffers
        for (int want : {6, 3})
            for (const auto& t : tries) {
                const int left = MT_SMEM_MAX - bars - q - t[0] * v - t[1] * MT_P;
                if (left < want * ks) continue;
                p->v_stages = t[0];
                p->p_bufs = t[1];
                p->k_stages = std::min(left / ks, 8);
                *smem = (size_t)q + t[0] * v + t[1] * MT_P + p->k_stages * ks + bars;
                return true;
            }
    }
    return false;
}

}  // namespace

bool mix_attn_tc_supported(const MixAttnShape& s) {
    MtParams p{};
    size_t smem = 0;
    return mt_plan(s, &p, &smem);
}

void launch_qk_fold_append(cudaStream_t st, const void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, void* fold) {
    const size_t smem = (size_t)s.heads * s.dim * 4;
    if (smem > 48 * 1024) cudaFuncSetAttribute(k_qk_fold_append, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    g_kernel_launches++;
    k_qk_fold_append<<<n, 256, smem, st>>>((const __nv_bfloat16*)qkv, ld, s, rs, (__nv_bfloat16*)fold);
}

cudaError_t launch_mix_attn_tc(cudaStream_t st, const void* fold, int n, const MixAttnShape& s, const RowState& rs, void* out, int ldo, uint32_t* err) {
    MtParams p{};
    size_t smem = 0;
    if (!mt_plan(s, &p, &smem) || !err || rs.separate()) return cudaErrorInvalidValue;
    p.out = (__nv_bfloat16*)out;
    p.bias = s.bias;
    p.ldo = ldo;
    p.n = n;
    p.start_pos = rs.start_pos;
    p.size = s.size;
    p.keep = s.keep_first;
    p.err = err;
    const int rows = rs.start_pos + n, gv = s.kv_heads * s.vdim;  // rows past the last token read as zeros
    cudaError_t e = encode_bf16_map(fold, n, s.heads * p.kd, s.heads * p.kd, MT_Q, &p.map_q);
    if (e == cudaSuccess) e = encode_bf16_map(rs.s0, rows, p.kd, p.kd, MT_K, &p.map_k);
    if (e == cudaSuccess) e = encode_bf16_map(rs.s1, rows, gv, gv, MT_K, &p.map_v);
    if (e != cudaSuccess) return e;
    static cudaError_t configured = cudaFuncSetAttribute(k_mix_attn_tc, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM_MAX);
    if (configured != cudaSuccess) return configured;
    g_kernel_launches++;
    k_mix_attn_tc<<<dim3(s.heads, (n + MT_Q - 1) / MT_Q), MT_THREADS, smem, st>>>(p);
    return cudaGetLastError();
}

}  // namespace wick
