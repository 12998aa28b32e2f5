// Dense bf16 GEMM on tcgen05: Y[n tokens][m] = X[n][k] W[m][k]^T with f32 accumulators in tensor memory.
//
// A tile is 128 weight rows (the MMA's M, tensor-memory lanes) x BN tokens (its N, tensor-memory columns), so that a few
// tokens only shorten the N side; gated tiles hold 128 gate rows and 128 up rows and the epilogue combines them.  One
// persistent CTA per SM:
//   warp 0  lane 0: TMA producer, stages of 64 k-columns (128-byte rows, 128B swizzle)
//   warp 1  lane 0: issues tcgen05.mma (K = 16 each) and commits; the warp owns the 512 tensor-memory columns
//   warps 2..9    : epilogue; warp w reads lanes 32 (w % 4).. and one half of the columns; the accumulator of the next tile
//                   fills the other half of tensor memory meanwhile
// Out-of-range rows and columns arrive as zeros from TMA, so any m, n, k works (row pitches are multiples of 8).
// With experts, X is sorted by expert and every expert's rows make tiles of their own against its own matrix; the tiles are
// counted on the device.
// Every wait is bounded: on expiry the error word is set, all roles leave, tensor memory is freed.
// Bound: tensor pipe for many tokens, HBM (weight bytes) for few.
#include "hybrid_kernels.cuh"
#include "tc_common.cuh"

namespace wick {

namespace {

constexpr int GB_M = 128, GB_K = 64;
constexpr int GB_EPI_WARPS = 8, GB_THREADS = 32 * (2 + GB_EPI_WARPS);

struct GbParams {
    CUtensorMap map_w[2], map_x[2];
    void* y[2];
    int ldy[2], m[2], k[2];
    int tile_start[3];  // tiles of job 0 from 0, of job 1 from tile_start[1], end tile_start[2]
    bool f32[2];
    int n;
    int act;
    float scale, softcap;
    int block_rows, x_step, y_step;  // > 0: block-diagonal (DenseBlocks)
    int experts;               // > 0: one matrix of m rows per expert, rows of X sorted by expert
    const int* expert_start;   // [experts + 1]
    uint32_t* err;
};

template <int BN, bool DUAL>
struct GbShape {
    static constexpr int A_BYTES = (DUAL ? 2 : 1) * GB_M * GB_K * 2, B_BYTES = BN * GB_K * 2;
    static constexpr int STAGE = A_BYTES + B_BYTES;
    static constexpr int STAGES = 200 * 1024 / STAGE < 8 ? 200 * 1024 / STAGE : 8;
    static constexpr int ACC = (DUAL ? 2 : 1) * BN;  // tensor-memory columns of one tile
    static constexpr size_t SMEM = (size_t)STAGES * STAGE + 1024 + 256;
    static_assert(ACC <= 256, "two tiles in tensor memory");
};

struct GbTile {
    int job, m0, m_end, n0, n_end;
    int w_row, x_col, y_col;  // where the tile's rows are in the weight map, its first column of X, and rows' places in Y
};
// Experts: expert_tiles[e] = tiles before those of expert e.
template <bool EXPERTS>
__device__ __forceinline__ GbTile gb_tile(const GbParams& p, int t, int tiles_n, int bn, const int* expert_tiles) {
    GbTile r;
    if constexpr (EXPERTS) {
        int lo = 0, hi = p.experts;  // the last e with expert_tiles[e] <= t
        while (hi - lo > 1) {
            const int mid = (lo + hi) / 2;
            if (expert_tiles[mid] <= t) lo = mid;
            else hi = mid;
        }
        const int s0 = p.expert_start[lo], local = t - expert_tiles[lo];
        r.n_end = p.expert_start[lo + 1];
        tiles_n = (r.n_end - s0 + bn - 1) / bn;
        r.job = 0;
        r.m0 = local / tiles_n * GB_M;
        r.n0 = s0 + local % tiles_n * bn;
        r.w_row = lo * p.m[0] + r.m0;
        r.m_end = p.m[0];
        r.x_col = 0;
        r.y_col = r.m0;
    } else {
        r.job = t >= p.tile_start[1] ? 1 : 0;
        const int local = t - p.tile_start[r.job];
        r.n0 = local % tiles_n * bn;
        r.n_end = p.n;
        const int mt = local / tiles_n;
        if (p.block_rows > 0) {
            const int per = (p.block_rows + GB_M - 1) / GB_M, b = mt / per;
            r.m0 = mt % per * GB_M;
            r.m_end = p.block_rows;
            r.w_row = b * p.block_rows + r.m0;
            r.x_col = b * p.x_step;
            r.y_col = b * p.y_step + r.m0;
        } else {
            r.m0 = r.w_row = r.y_col = mt * GB_M;
            r.m_end = p.m[r.job];
            r.x_col = 0;
        }
    }
    return r;
}

template <int COLS>
__device__ __forceinline__ void gb_ld(uint32_t taddr, int32_t* r) {
    if constexpr (COLS == 16) tmem_ld16(taddr, r);
    else tmem_ld32(taddr, r);
}

template <int BN, bool DUAL, bool EXPERTS>
__global__ void __launch_bounds__(GB_THREADS, 1) k_gemm_bf16(const __grid_constant__ GbParams p) {
    using Sh = GbShape<BN, DUAL>;
    extern __shared__ uint8_t gb_raw[];
    uint8_t* stages = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gb_raw) + 1023) & ~(uintptr_t)1023);
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(stages + (size_t)Sh::STAGES * Sh::STAGE);
    unsigned long long *full = bars, *empty = bars + Sh::STAGES, *acc_full = empty + Sh::STAGES, *acc_empty = acc_full + 2;
    uint32_t* tmem_word = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile uint32_t* abort = tmem_word + 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int tiles_n = (p.n + BN - 1) / BN;
    const int* expert_tiles = nullptr;
    if constexpr (EXPERTS) {
        __shared__ int pre[MAX_EXPERTS + 1];
        const int tiles_m = (p.m[0] + GB_M - 1) / GB_M;
        if (warp == 1) {  // running sum over the experts, 32 at a time
            int base = 0;
            for (int e0 = 0; e0 < p.experts; e0 += 32) {
                const int e = e0 + lane;
                int v = e < p.experts ? (p.expert_start[e + 1] - p.expert_start[e] + BN - 1) / BN * tiles_m : 0;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const int u = __shfl_up_sync(0xffffffffu, v, o);
                    if (lane >= o) v += u;
                }
                if (e < p.experts) pre[e + 1] = base + v;
                base += __shfl_sync(0xffffffffu, v, 31);
            }
            if (lane == 0) pre[0] = 0;
        }
        expert_tiles = pre;
    }
    if (threadIdx.x == 0) {
        for (int s = 0; s < Sh::STAGES; s++) {
            mbar_init(smem_u32(&full[s]), 1);
            mbar_init(smem_u32(&empty[s]), 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(smem_u32(&acc_full[b]), 1);
            mbar_init(smem_u32(&acc_empty[b]), GB_EPI_WARPS);
        }
        *abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_word)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_word;
    const int tiles = EXPERTS ? expert_tiles[p.experts] : p.tile_start[2];

    if (warp == 0) {
        if (lane == 0) {
            uint32_t g = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const GbTile tl = gb_tile<EXPERTS>(p, t, tiles_n, BN, expert_tiles);
                const int ks = (p.k[tl.job] + GB_K - 1) / GB_K;
                for (int i = 0; i < ks; i++, g++) {
                    const int s = g % Sh::STAGES;
                    ok = mbar_wait_bounded(smem_u32(&empty[s]), ((g / Sh::STAGES) & 1) ^ 1, abort, p.err, 11);
                    if (!ok) break;
                    const uint32_t bar = smem_u32(&full[s]), dst = smem_u32(stages + (size_t)s * Sh::STAGE);
                    mbar_arrive_expect_tx(bar, Sh::STAGE);
                    tma_load_2d(dst, &p.map_w[tl.job], bar, i * GB_K, tl.w_row);
                    if (DUAL) tma_load_2d(dst + GB_M * GB_K * 2, &p.map_w[1], bar, i * GB_K, tl.w_row);
                    tma_load_2d(dst + Sh::A_BYTES, &p.map_x[tl.job], bar, tl.x_col + i * GB_K, tl.n0);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_bf16_idesc(GB_M, BN);
            uint32_t g = 0, it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, it++) {
                const GbTile tl = gb_tile<EXPERTS>(p, t, tiles_n, BN, expert_tiles);
                const int ks = (p.k[tl.job] + GB_K - 1) / GB_K;
                const uint32_t buf = it & 1, d = tmem + buf * 256;
                ok = mbar_wait_bounded(smem_u32(&acc_empty[buf]), ((it >> 1) & 1) ^ 1, abort, p.err, 12);
                if (!ok) break;
                tc_fence_after();
                for (int i = 0; i < ks; i++, g++) {
                    const int s = g % Sh::STAGES;
                    ok = mbar_wait_bounded(smem_u32(&full[s]), (g / Sh::STAGES) & 1, abort, p.err, 13);
                    if (!ok) break;
                    tc_fence_after();
                    const uint32_t a = smem_u32(stages + (size_t)s * Sh::STAGE);
                    const unsigned long long da = umma_desc_sw128(a), db = umma_desc_sw128(a + Sh::A_BYTES);
#pragma unroll
                    for (int kk = 0; kk < GB_K / 16; kk++) {
                        const bool acc = i > 0 || kk > 0;
                        umma_bf16(d, da + kk * 2, db + kk * 2, idesc, acc);  // 16 bf16 = 32 bytes further inside the swizzle atom
                        if (DUAL) umma_bf16(d + BN, umma_desc_sw128(a + GB_M * GB_K * 2) + kk * 2, db + kk * 2, idesc, acc);
                    }
                    umma_commit(smem_u32(&empty[s]));
                }
                if (ok) umma_commit(smem_u32(&acc_full[buf]));
            }
        }
    } else {
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        constexpr int HALF = BN / 2, COLS = HALF < 32 ? HALF : 32;
        uint32_t it = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x, it++) {
            const GbTile tl = gb_tile<EXPERTS>(p, t, tiles_n, BN, expert_tiles);
            const uint32_t buf = it & 1;
            if (!mbar_wait_bounded(smem_u32(&acc_full[buf]), (it >> 1) & 1, abort, p.err, 14)) break;
            tc_fence_after();
            const int row = tl.y_col + quarter * 32 + lane;
            const bool row_ok = tl.m0 + quarter * 32 + lane < tl.m_end;
            const uint32_t base = tmem + buf * 256 + ((uint32_t)(quarter * 32) << 16) + half * HALF;
            const bool f32 = p.f32[tl.job];
            const int ldy = p.ldy[tl.job];
#pragma unroll 1
            for (int c0 = 0; c0 < HALF; c0 += COLS) {
                int32_t v[COLS], u[DUAL ? COLS : 1];
                gb_ld<COLS>(base + c0, v);
                if constexpr (DUAL) gb_ld<COLS>(base + BN + c0, u);
                tmem_ld_wait();
                if (c0 + COLS == HALF) {
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(smem_u32(&acc_empty[buf]));
                }
                const int tok0 = tl.n0 + half * HALF + c0;
                if (row_ok && tok0 < tl.n_end) {
#pragma unroll
                    for (int c = 0; c < COLS; c++) {
                        float f = activate(__int_as_float(v[c]), (Activation)p.act);
                        if constexpr (DUAL) f *= __int_as_float(u[c]);
                        f *= p.scale;
                        if (p.softcap > 0.0f) f = p.softcap * tanhf(f / p.softcap);
                        v[c] = __float_as_int(f);
                    }
                    if (f32) {
                        float* dst = (float*)p.y[tl.job] + (size_t)tok0 * ldy + row;
#pragma unroll
                        for (int c = 0; c < COLS; c++)
                            if (tok0 + c < tl.n_end) dst[(size_t)c * ldy] = __int_as_float(v[c]);
                    } else {
                        __nv_bfloat16* dst = (__nv_bfloat16*)p.y[tl.job] + (size_t)tok0 * ldy + row;
#pragma unroll
                        for (int c = 0; c < COLS; c++)
                            if (tok0 + c < tl.n_end) dst[(size_t)c * ldy] = __float2bfloat16_rn(__int_as_float(v[c]));
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
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

int gb_tiles_m(const DenseCall& c, int job) {
    if (c.blocks) return c.job[job].w.m / c.blocks.rows * ((c.blocks.rows + GB_M - 1) / GB_M);
    return (c.job[job].w.m + GB_M - 1) / GB_M;
}

template <int BN, bool DUAL, bool EXPERTS>
cudaError_t gb_launch(cudaStream_t st, GbParams& p, int jobs, const DenseCall& c, int sms) {
    using Sh = GbShape<BN, DUAL>;
    const int tiles_n = (c.n + BN - 1) / BN, copies = EXPERTS ? c.experts.count : 1;
    int t = 0;
    for (int i = 0; i < 2; i++) {
        p.tile_start[i] = t;
        if (i < jobs) t += gb_tiles_m(c, i) * tiles_n;
    }
    p.tile_start[2] = t;
    if (EXPERTS) t = (c.job[0].w.m + GB_M - 1) / GB_M * (c.n / BN + std::min(c.n, copies));  // no more than this many
    for (int i = 0; i < c.count; i++) {
        cudaError_t e = encode_bf16_map(c.job[i].w.w, c.job[i].w.m * copies, c.job[i].w.k, c.job[i].w.ld, GB_M, &p.map_w[i]);
        // (blocks: columns of X beyond a block's k belong to others and meet zeros of W)
        const int x_cols = c.blocks ? (c.job[i].w.m / c.blocks.rows - 1) * c.blocks.x_step + c.job[i].w.k : c.job[i].w.k;
        if (e == cudaSuccess && i < jobs) e = encode_bf16_map(c.job[i].x, c.n, x_cols, c.job[i].ldx, BN, &p.map_x[i]);
        if (e != cudaSuccess) return e;
    }
    static cudaError_t configured = cudaFuncSetAttribute(k_gemm_bf16<BN, DUAL, EXPERTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::SMEM);
    if (configured != cudaSuccess) return configured;
    g_kernel_launches++;
    k_gemm_bf16<BN, DUAL, EXPERTS><<<t < sms ? t : sms, GB_THREADS, Sh::SMEM, st>>>(p);
    return cudaGetLastError();
}

template <bool DUAL, bool EXPERTS>
cudaError_t gb_bn(cudaStream_t st, GbParams& p, int jobs, const DenseCall& c, int sms) {
    // Tile width: fewest (waves x time per k step), a step being bound by the MMA (BN / 2 cycles per 16 columns) or by the
    // operands it reads from shared memory (32 + BN / 4 cycles).
    int best = 0;
    double best_cost = 0.0;
    for (int bn : {256, 128, 64, 32}) {
        if (DUAL && bn == 256) continue;
        long tiles = 0;
        if (EXPERTS) {  // rows spread evenly over the experts, each with a last tile that is half full on average
            const int used = std::min(c.n, c.experts.count);
            tiles = (long)((c.job[0].w.m + GB_M - 1) / GB_M) * std::max<long>(used, (long)(c.n / (double)bn + 0.5 * used));
        } else {
            for (int i = 0; i < jobs; i++) tiles += (long)gb_tiles_m(c, i) * ((c.n + bn - 1) / bn);
        }
        const double step = std::max(bn / 2.0, 32 + bn / 4.0) + 4.0;
        const double cost = (double)((tiles + sms - 1) / sms) * step;
        if (!best || cost < best_cost) {
            best = bn;
            best_cost = cost;
        }
    }
    switch (best) {
        case 256: if constexpr (!DUAL) return gb_launch<256, DUAL, EXPERTS>(st, p, jobs, c, sms);
        case 128: return gb_launch<128, DUAL, EXPERTS>(st, p, jobs, c, sms);
        case 64: return gb_launch<64, DUAL, EXPERTS>(st, p, jobs, c, sms);
        default: return gb_launch<32, DUAL, EXPERTS>(st, p, jobs, c, sms);
    }
}

}  // namespace

cudaError_t launch_dense_tc(cudaStream_t st, const DenseCall& c) {
    if (c.n <= 0) return cudaSuccess;
    if (!c.err || (c.blocks && (c.count != 1 || c.blocks.x_step % 8 || c.experts)) || (c.experts && (!c.experts.start || c.experts.count > MAX_EXPERTS || (c.count == 2 && !c.gated)))) return cudaErrorInvalidValue;
    static int sms = 0;
    if (!sms) {
        int dev = 0, v = 0;
        cudaError_t e = cudaGetDevice(&dev);
        if (e == cudaSuccess) e = cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
        if (e != cudaSuccess) return e;
        sms = v;
    }
    GbParams p{};
    p.n = c.n;
    p.act = c.act;
    p.scale = c.scale;
    p.softcap = c.softcap;
    p.err = c.err;
    p.block_rows = c.blocks.rows;
    p.x_step = c.blocks.x_step;
    p.y_step = c.blocks.y_step;
    p.experts = c.experts.count;
    p.expert_start = c.experts.start;
    const int jobs = c.gated ? 1 : c.count;
    for (int i = 0; i < jobs; i++) {
        p.y[i] = c.job[i].y;
        p.ldy[i] = c.job[i].ldy;
        p.m[i] = c.job[i].w.m;
        p.k[i] = c.job[i].w.k;
        p.f32[i] = c.job[i].f32;
    }
    if (c.experts) return c.gated ? gb_bn<true, true>(st, p, jobs, c, sms) : gb_bn<false, true>(st, p, jobs, c, sms);
    return c.gated ? gb_bn<true, false>(st, p, jobs, c, sms) : gb_bn<false, false>(st, p, jobs, c, sms);
}

}  // namespace wick
