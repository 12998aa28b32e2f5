// Prompt form of the latent attention (kernels_latent.cu) on tcgen05, for bfloat16 models.
//
// Keys and values of the positions that the portion sees come from the cached latents by one GEMM (gemm_bf16.cu); the rotated
// key part is read from the cache by every head.  A CTA owns 128 queries of one head and walks over tiles of 64 keys:
//   warp 0  lane 0: TMA - queries once, keys [W_uk c | rotated part] in chunks of 64 columns, values
//   warp 1  lane 0: S = q K^T into one of two tensor-memory buffers, then O += P V of the tile before
//   warps 2..5    : one query row per thread.  First the rotated columns of q are turned in shared memory; then per tile the
//                   softmax weights, rounded to bf16 into shared memory in the 128B-swizzled layout of the MMA's A operand
// The running reference of a row starts at its sink and moves only when a score exceeds it by more than 2^8, so O in tensor
// memory is rarely rescaled; sums stay in f32.  The sink enters the denominator at the end.
// Every wait is bounded.  Bound: tensor pipe and the special-function unit (one exponential per query, key and head).
#include "latent_kernels.cuh"
#include "tc_common.cuh"

namespace wick {

namespace {

constexpr int LT_Q = 128, LT_K = 64, LT_EPI_WARPS = 4, LT_THREADS = 32 * (2 + LT_EPI_WARPS);
constexpr int LT_QCHUNK = LT_Q * 64 * 2, LT_KCHUNK = LT_K * 64 * 2, LT_P = LT_Q * LT_K * 2;
constexpr int LT_SMEM_MAX = 226 * 1024, LT_SMEM_HALF = 113 * 1024;  // one or two CTAs per SM
constexpr int LT_BARS = 1024 + 256;                                 // alignment, barriers
constexpr float LT_SLACK = 8.0f;                                    // log2 of how far weights may exceed 1

struct LtParams {
    CUtensorMap map_q, map_qr, map_k, map_kr, map_v;
    __nv_bfloat16* out;
    const float* sink;
    const float2* rope;
    int ldo, n, start_pos, key0;        // key0: position of the maps' first key
    int kd, kr, rot_dims, vdim;         // columns: unrotated, rotated part; rotated pairs; values
    int dc, rc, vboxes;                 // chunks of 64 of the above
    int size, k_stages, v_stages, p_bufs;
    float scale;
    uint32_t tmem_cols;
    uint32_t* err;
};

// A wait of a whole warp: every lane gets the same answer.
__device__ __forceinline__ bool warp_wait(const void* bar, uint32_t parity, volatile uint32_t* abort, uint32_t* err, uint32_t code) {
    return __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(bar), parity, abort, err, code));
}

__global__ void __launch_bounds__(LT_THREADS) k_latent_attn_tc(const __grid_constant__ LtParams p) {
    extern __shared__ uint8_t lt_raw[];
    uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~(uintptr_t)1023);
    const int chunks = p.dc + p.rc, k_stage = chunks * LT_KCHUNK, v_stage = p.vboxes * LT_KCHUNK;
    uint8_t* sq = sm;
    uint8_t* sk = sq + chunks * LT_QCHUNK;
    uint8_t* sv = sk + p.k_stages * k_stage;
    uint8_t* sp = sv + p.v_stages * v_stage;
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(sp + p.p_bufs * LT_P);
    unsigned long long *q_full = bars, *q_ready = bars + 1, *o_full = bars + 2, *k_full = bars + 3, *k_empty = k_full + 2, *v_full = k_empty + 2,
                       *v_empty = v_full + 2, *s_full = v_empty + 2, *s_empty = s_full + 2, *p_full = s_empty + 2, *p_empty = p_full + 2;
    uint32_t* tmem_word = reinterpret_cast<uint32_t*>(p_empty + 2);
    volatile uint32_t* abort = tmem_word + 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, row0 = (gridDim.y - 1 - blockIdx.y) * LT_Q;  // the longest walks start first
    const int nq = min(LT_Q, p.n - row0), p0 = p.start_pos + row0, p1 = p0 + nq - 1;
    const int lo = p.size > 0 ? max(0, p0 - p.size + 1) : 0, tiles = (p1 - lo + LT_K) / LT_K;

    if (threadIdx.x == 0) {
        mbar_init(smem_u32(q_full), 1);
        mbar_init(smem_u32(q_ready), LT_EPI_WARPS);
        mbar_init(smem_u32(o_full), 1);
        for (int i = 0; i < 2; i++) {
            mbar_init(smem_u32(&k_full[i]), 1);
            mbar_init(smem_u32(&k_empty[i]), 1);
            mbar_init(smem_u32(&v_full[i]), 1);
            mbar_init(smem_u32(&v_empty[i]), 1);
            mbar_init(smem_u32(&s_full[i]), 1);
            mbar_init(smem_u32(&s_empty[i]), LT_EPI_WARPS);
            mbar_init(smem_u32(&p_full[i]), LT_EPI_WARPS);
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
    const uint32_t tmem = *tmem_word, tmem_o = tmem + 2 * LT_K;

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            mbar_arrive_expect_tx(smem_u32(q_full), chunks * LT_QCHUNK);
            for (int c = 0; c < chunks; c++) {
                if (c < p.dc) tma_load_3d(smem_u32(sq + c * LT_QCHUNK), &p.map_q, smem_u32(q_full), c * 64, h, row0);
                else tma_load_3d(smem_u32(sq + c * LT_QCHUNK), &p.map_qr, smem_u32(q_full), (c - p.dc) * 64, h, row0);
            }
            for (int t = 0; t < tiles && ok; t++) {
                const int key = lo - p.key0 + t * LT_K, ks = t % p.k_stages, vs = t % p.v_stages;
                ok = mbar_wait_bounded(smem_u32(&k_empty[ks]), ((t / p.k_stages) & 1) ^ 1, abort, p.err, 41);
                if (!ok) break;
                uint32_t bar = smem_u32(&k_full[ks]), dst = smem_u32(sk + ks * k_stage);
                mbar_arrive_expect_tx(bar, k_stage);
                for (int c = 0; c < chunks; c++) {
                    if (c < p.dc) tma_load_3d(dst + c * LT_KCHUNK, &p.map_k, bar, c * 64, h, key);
                    else tma_load_2d(dst + c * LT_KCHUNK, &p.map_kr, bar, (c - p.dc) * 64, key);
                }
                ok = mbar_wait_bounded(smem_u32(&v_empty[vs]), ((t / p.v_stages) & 1) ^ 1, abort, p.err, 42);
                if (!ok) break;
                bar = smem_u32(&v_full[vs]);
                dst = smem_u32(sv + vs * v_stage);
                mbar_arrive_expect_tx(bar, v_stage);
                for (int b = 0; b < p.vboxes; b++) tma_load_3d(dst + b * LT_KCHUNK, &p.map_v, bar, b * 64, h, key);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_bf16_idesc(LT_Q, LT_K);
            const uint32_t idesc_o = umma_bf16_idesc(LT_Q, round_up(p.vdim, 16)) | UMMA_B_MN;
            bool ok = mbar_wait_bounded(smem_u32(q_full), 0, abort, p.err, 43) && mbar_wait_bounded(smem_u32(q_ready), 0, abort, p.err, 44);
            tc_fence_after();
            for (int t = 0; t <= tiles && ok; t++) {
                if (t < tiles) {
                    const int b = t & 1, ks = t % p.k_stages;
                    ok = mbar_wait_bounded(smem_u32(&s_empty[b]), ((t >> 1) & 1) ^ 1, abort, p.err, 45) &&
                         mbar_wait_bounded(smem_u32(&k_full[ks]), (t / p.k_stages) & 1, abort, p.err, 46);
                    if (!ok) break;
                    tc_fence_after();
                    for (int c = 0; c < chunks; c++) {
                        const int cols = c < p.dc ? min(64, p.kd - c * 64) : min(64, p.kr - (c - p.dc) * 64), steps = (cols + 15) / 16;
                        const unsigned long long da = umma_desc_sw128(smem_u32(sq + c * LT_QCHUNK)), db = umma_desc_sw128(smem_u32(sk + ks * k_stage + c * LT_KCHUNK));
                        for (int kk = 0; kk < steps; kk++) umma_bf16(tmem + b * LT_K, da + kk * 2, db + kk * 2, idesc_s, c > 0 || kk > 0);
                    }
                    umma_commit(smem_u32(&k_empty[ks]));
                    umma_commit(smem_u32(&s_full[b]));
                }
                if (t > 0) {
                    const int u = t - 1, pb = u % p.p_bufs, vs = u % p.v_stages;
                    ok = mbar_wait_bounded(smem_u32(&p_full[pb]), (u / p.p_bufs) & 1, abort, p.err, 47) &&
                         mbar_wait_bounded(smem_u32(&v_full[vs]), (u / p.v_stages) & 1, abort, p.err, 48);
                    if (!ok) break;
                    tc_fence_after();
                    const unsigned long long da = umma_desc_sw128(smem_u32(sp + pb * LT_P));
                    const unsigned long long db = umma_desc_mn_sw128(smem_u32(sv + vs * v_stage), LT_KCHUNK);
#pragma unroll
                    for (int kk = 0; kk < 4; kk++) umma_bf16(tmem_o, da + kk * 2, db + kk * (2048 >> 4), idesc_o, u > 0 || kk > 0);
                    umma_commit(smem_u32(&v_empty[vs]));
                    umma_commit(smem_u32(&p_empty[pb]));
                }
            }
            if (ok) umma_commit(smem_u32(o_full));
        }
    } else {
        const int quarter = warp & 3, r = quarter * 32 + lane, qi = p0 + r;  // tensor-memory lanes 32 (warp % 4)..
        constexpr float LOG2E = 1.4426950408889634f;
        const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
        const float scale = p.scale * LOG2E, sink = p.sink[h] * LOG2E;
        bool ok = warp_wait(q_full, 0, abort, p.err, 49);
        if (ok) {  // turn the rotated columns of this row
            if (r < nq) {
                const float2* cs = p.rope + (size_t)qi * (p.rot_dims / 2);
                for (int d = 0; d < p.rot_dims; d += 8) {
                    uint4* at = reinterpret_cast<uint4*>(sq + (p.dc + d / 64) * LT_QCHUNK + r * 128 + (((d % 64 / 8) ^ (r & 7)) << 4));
                    uint4 v = *at;
                    uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                    for (int e = 0; e < 4; e++)
                        if (d + 2 * e < p.rot_dims) {
                            const float2 t = cs[d / 2 + e];
                            const float a = __uint_as_float(w[e] << 16), b = __uint_as_float(w[e] & 0xffff0000u);
                            const __nv_bfloat162 q = __floats2bfloat162_rn(a * t.x - b * t.y, b * t.x + a * t.y);
                            w[e] = *reinterpret_cast<const uint32_t*>(&q);
                        }
                    *at = v;
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(q_ready));
        }
        float ref = sink, sum = 0.0f;
        for (int t = 0; t < tiles && ok; t++) {
            const int b = t & 1, key0 = lo + t * LT_K;
            ok = warp_wait(&s_full[b], (t >> 1) & 1, abort, p.err, 50);
            if (!ok) break;
            tc_fence_after();
            int32_t v[LT_K];
            tmem_ld32(tmem + lane_base + b * LT_K, v);
            tmem_ld32(tmem + lane_base + b * LT_K + 32, v + 32);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s_empty[b]));
            if (key0 + LT_K - 1 > p0 || (p.size > 0 && p1 - key0 >= p.size)) {  // some row does not see some key
#pragma unroll
                for (int c = 0; c < LT_K; c++) {
                    const int j = key0 + c;
                    if (j > qi || (p.size > 0 && qi - j >= p.size)) v[c] = __float_as_int(-INFINITY);
                }
            }
            float top = __int_as_float(v[0]);
#pragma unroll
            for (int c = 1; c < LT_K; c++) top = fmaxf(top, __int_as_float(v[c]));
            top *= scale;  // (a scale of 0 or below is refused on the host)
            if (t == 0) {
                ref = fmaxf(ref, top);
            } else if (__any_sync(0xffffffffu, top > ref + LT_SLACK)) {
                const int u = t - 1;  // O must be complete up to the tile before
                ok = warp_wait(&p_empty[u % p.p_bufs], (u / p.p_bufs) & 1, abort, p.err, 51);
                if (!ok) break;
                tc_fence_after();
                const float next = top > ref + LT_SLACK ? top : ref, f = exp2f(ref - next);
                ref = next;
                sum *= f;
                for (int c0 = 0; c0 < p.vdim; c0 += 16) {
                    int32_t o[16];
                    tmem_ld16(tmem_o + lane_base + c0, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int c = 0; c < 16; c++) o[c] = __float_as_int(__int_as_float(o[c]) * f);
                    tmem_st16(tmem_o + lane_base + c0, o);
                }
                tmem_st_wait();
                tc_fence_before();
            }
            uint32_t w[LT_K / 2];
            float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
            for (int c = 0; c < LT_K / 2; c++) {
                float e0, e1;
                asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e0) : "f"(fmaf(__int_as_float(v[2 * c]), scale, -ref)));
                asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e1) : "f"(fmaf(__int_as_float(v[2 * c + 1]), scale, -ref)));
                s0 += e0;
                s1 += e1;
                const __nv_bfloat162 q = __floats2bfloat162_rn(e0, e1);
                w[c] = *reinterpret_cast<const uint32_t*>(&q);
            }
            sum += s0 + s1;
            const int pb = t % p.p_bufs;
            ok = warp_wait(&p_empty[pb], ((t / p.p_bufs) & 1) ^ 1, abort, p.err, 52);
            if (!ok) break;
            uint8_t* prow = sp + pb * LT_P + r * 128;
#pragma unroll
            for (int c = 0; c < 8; c++) *reinterpret_cast<uint4*>(prow + ((c ^ (r & 7)) << 4)) = make_uint4(w[4 * c], w[4 * c + 1], w[4 * c + 2], w[4 * c + 3]);
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&p_full[pb]));
        }
        if (ok && warp_wait(o_full, 0, abort, p.err, 53)) {
            tc_fence_after();
            const float f = 1.0f / (sum + exp2f(sink - ref));
            __nv_bfloat16* dst = p.out + (size_t)(row0 + r) * p.ldo + h * p.vdim;
            const bool wide = p.vdim % 8 == 0;  // rows of 16-byte pieces
            for (int c0 = 0; c0 < p.vdim; c0 += 16) {
                int32_t v[16];
                tmem_ld16(tmem_o + lane_base + c0, v);
                tmem_ld_wait();
                if (r < nq) {
#pragma unroll
                    for (int q = 0; q < 2; q++) {
                        if (wide && c0 + q * 8 < p.vdim) {
                            uint32_t w[4];
#pragma unroll
                            for (int e = 0; e < 4; e++) {
                                const __nv_bfloat162 x = __floats2bfloat162_rn(__int_as_float(v[q * 8 + 2 * e]) * f, __int_as_float(v[q * 8 + 2 * e + 1]) * f);
                                w[e] = *reinterpret_cast<const uint32_t*>(&x);
                            }
                            *reinterpret_cast<uint4*>(dst + c0 + q * 8) = make_uint4(w[0], w[1], w[2], w[3]);
                        } else if (!wide) {
#pragma unroll
                            for (int e = 0; e < 8; e++)
                                if (c0 + q * 8 + e < p.vdim) dst[c0 + q * 8 + e] = __float2bfloat16_rn(__int_as_float(v[q * 8 + e]) * f);
                        }
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

// Shared memory plan: two CTAs per SM where that leaves at least one stage of everything.  False if the shape does not fit.
bool lt_plan(const LatentShape& s, LtParams* p, size_t* smem) {
    if (s.vdim > 256 || s.scale <= 0.0f) return false;
    p->kd = s.dim;
    p->kr = s.rot_dim;
    p->dc = (s.dim + 63) / 64;
    p->rc = (s.rot_dim + 63) / 64;
    p->vdim = s.vdim;
    p->vboxes = (s.vdim + 63) / 64;
    p->tmem_cols = round_up(s.vdim, 16) <= 128 ? 256 : 512;
    const int chunks = p->dc + p->rc, q = chunks * LT_QCHUNK, k = chunks * LT_KCHUNK, v = p->vboxes * LT_KCHUNK;
    for (int budget : {LT_SMEM_HALF, LT_SMEM_MAX}) {
        if (budget == LT_SMEM_HALF && p->tmem_cols > 256) continue;
        p->k_stages = p->v_stages = p->p_bufs = 1;
        auto need = [&]() { return q + p->k_stages * k + p->v_stages * v + p->p_bufs * LT_P + LT_BARS; };
        if (need() > budget) continue;
        for (int* grow : {&p->k_stages, &p->v_stages, &p->p_bufs}) {
            *grow = 2;
            if (need() > budget) *grow = 1;
        }
        *smem = (size_t)need();
        return true;
    }
    return false;
}

}  // namespace

bool latent_tc_supported(const LatentShape& s) {
    LtParams p{};
    size_t smem = 0;
    return lt_plan(s, &p, &smem);
}

static int first_visible(const LatentShape& s, const RowState& rs) { return s.size > 0 ? std::max(0, rs.start_pos - s.size + 1) : 0; }

cudaError_t launch_latent_kv(cudaStream_t st, int n, const LatentShape& s, const RowState& rs, const DenseWeight& ukv, void* kv, uint32_t* err) {
    const int key0 = first_visible(s, rs);
    DenseCall c;
    c.job[0].w = ukv; c.job[0].x = (const __nv_bfloat16*)rs.s0 + (size_t)key0 * s.ldc(); c.job[0].ldx = s.ldc(); c.job[0].y = kv; c.job[0].ldy = latent_tc_cols(s);
    c.n = rs.start_pos + n - key0;
    c.err = err;
    return launch_dense_tc(st, c);
}

cudaError_t launch_latent_attn_tc(cudaStream_t st, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs, const void* kv, void* out,
                                  int ldo, uint32_t* err) {
    LtParams p{};
    size_t smem = 0;
    if (!lt_plan(s, &p, &smem) || !err || rs.separate()) return cudaErrorInvalidValue;
    using B = __nv_bfloat16;
    const int ldc = s.ldc(), ldkv = latent_tc_cols(s), d8 = round_up(s.dim, 8), v8 = round_up(s.vdim, 8);
    p.key0 = first_visible(s, rs);
    const int keys = rs.start_pos + n - p.key0;
    const B* cache = (const B*)rs.s0 + (size_t)p.key0 * ldc;
    p.out = (B*)out;
    p.sink = s.sink;
    p.rope = s.rope;
    p.ldo = ldo;
    p.n = n;
    p.start_pos = rs.start_pos;
    p.rot_dims = s.rot_dims;
    p.size = s.size;
    p.scale = s.scale;
    p.err = err;
    cudaError_t e = encode_bf16_map3(q, n, s.heads, s.dim, s.q_pitch(), ldq, LT_Q, &p.map_q);
    if (e == cudaSuccess) e = encode_bf16_map3((const B*)q + s.q_off_rot(), n, s.heads, s.rot_dim, s.q_pitch(), ldq, LT_Q, &p.map_qr);
    if (e == cudaSuccess) e = encode_bf16_map3(kv, keys, s.heads, s.dim, d8, ldkv, LT_K, &p.map_k);
    if (e == cudaSuccess) e = encode_bf16_map(cache + s.off_rot(), keys, s.rot_dim, ldc, LT_K, &p.map_kr);
    if (e == cudaSuccess) e = encode_bf16_map3((const B*)kv + s.heads * d8, keys, s.heads, s.vdim, v8, ldkv, LT_K, &p.map_v);
    if (e != cudaSuccess) return e;
    static cudaError_t configured = cudaFuncSetAttribute(k_latent_attn_tc, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM_MAX);
    if (configured != cudaSuccess) return configured;
    g_kernel_launches++;
    k_latent_attn_tc<<<dim3(s.heads, (n + LT_Q - 1) / LT_Q), LT_THREADS, smem, st>>>(p);
    return cudaGetLastError();
}

}  // namespace wick
