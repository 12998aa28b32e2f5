// Dense bfloat16 matrices times f32 or bfloat16 activation rows.
//   k_dense_rows  up to DENSE_ROWS_MAX rows (decode): a warp (or several, over parts of k) streams R weight rows with 16-byte
//                 loads, every loaded weight feeds all the activation rows.  HBM-bound: the weight bytes once.  Also the
//                 block-diagonal matrices (any number of rows, DENSE_ROWS_MAX at a time) and, row by row, the matrices of
//                 experts that a table gives.
//   k_dense_simt  any number of rows, f32 multiply-adds on the CUDA cores: prompts of f32 models (bf16 models use gemm_bf16.cu).
// Both accumulate in f32 and share the epilogues: activation, activation(gate) * up, scale, soft cap.
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

template <class T>
__device__ __forceinline__ void dense_store(const DenseCall& c, const DenseJob& j, int row, int col, float v, float up) {
    v = activate(v, c.act);
    if (c.gated) v *= up;
    v *= c.scale;
    if (c.softcap > 0.0f) v = c.softcap * tanhf(v / c.softcap);
    const size_t at = (size_t)row * j.ldy + col;
    if (j.f32) ((float*)j.y)[at] = v;
    else ((T*)j.y)[at] = f_act<T>(v);
}

constexpr int ROWS_WARPS = 4;
constexpr int ROWS_TARGET_WARPS = 148 * 20;

enum RowsMode { ROWS_PLAIN, ROWS_BLOCKS, ROWS_EXPERTS };

// NB activation rows, R weight rows (of each matrix when gated) per unit of WK warps, which split the columns of k.
template <class T, int NB, int R, bool GATED, int WK, int MODE>
__global__ void __launch_bounds__(ROWS_WARPS * 32) k_dense_rows(const __grid_constant__ DenseCall c) {
    constexpr int M = GATED ? 2 : 1;
    __shared__ float red[ROWS_WARPS][M * R * NB];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, part = warp % WK;
    int unit = (blockIdx.x * ROWS_WARPS + warp) / WK;
    int ji = 0;
    if (!GATED && c.count == 2) {
        const int units0 = (c.job[0].w.m + R - 1) / R;
        if (unit >= units0) {
            ji = 1;
            unit -= units0;
        }
    }
    const DenseJob& j = c.job[ji];
    const int m = j.w.m, ld = j.w.ld, row0 = unit * R, k0 = (part * 32 + lane) * 8;
    const int b0 = MODE == ROWS_PLAIN ? 0 : blockIdx.y * NB;  // first activation row
    size_t wrow = 0;                                          // first row of the expert's matrix
    if constexpr (MODE == ROWS_EXPERTS) {
        pdl_launch_next();
        pdl_wait();
        const DenseExperts& e = c.experts;
        const uint32_t tok = e.tokens ? e.tokens[b0 / e.top] : e.ctl->token;
        wrow = (size_t)e.table[(size_t)tok * e.top + b0 % e.top] * m;
    }
    const __nv_bfloat16* wp[M][R];
#pragma unroll
    for (int q = 0; q < M; q++)
#pragma unroll
        for (int r = 0; r < R; r++) {  // a row past the end repeats the last one and is not stored
            wp[q][r] = c.job[ji + q].w.w + (wrow + min(row0 + r, m - 1)) * ld;
            if constexpr (MODE != ROWS_EXPERTS)
                for (int k = k0; k < ld; k += WK * 256)
                    if ((lane & 7) == 0) prefetch_l2(wp[q][r] + k);  // a 128-byte line per eight lanes
        }
    if constexpr (MODE != ROWS_EXPERTS) {
        pdl_launch_next();
        pdl_wait();
    }
    float acc[M][R][NB];
#pragma unroll
    for (int q = 0; q < M; q++)
#pragma unroll
        for (int r = 0; r < R; r++)
#pragma unroll
            for (int b = 0; b < NB; b++) acc[q][r][b] = 0.0f;
    const T* x = (const T*)j.x;
    int ycol = row0;
    if constexpr (MODE == ROWS_BLOCKS) {  // R divides the block's rows
        const int blk = row0 / c.blocks.rows;
        x += blk * c.blocks.x_step;
        ycol = blk * c.blocks.y_step + row0 % c.blocks.rows;
    }
    const int xdiv = MODE == ROWS_EXPERTS && c.experts.x_per_token ? c.experts.top : 1;
#pragma unroll 4
    for (int k = k0; k < ld; k += WK * 256) {
        uint4 wv[M][R];
#pragma unroll
        for (int q = 0; q < M; q++)
#pragma unroll
            for (int r = 0; r < R; r++) wv[q][r] = __ldg(reinterpret_cast<const uint4*>(wp[q][r] + k));
#pragma unroll
        for (int b = 0; b < NB; b++) {
            float xv[8];
            load8(x + (size_t)(min(b0 + b, c.n - 1) / xdiv) * j.ldx + k, xv);
#pragma unroll
            for (int q = 0; q < M; q++)
#pragma unroll
                for (int r = 0; r < R; r++) {
                    float w[8];
                    bf16x8_f(wv[q][r], w);
#pragma unroll
                    for (int i = 0; i < 8; i++) acc[q][r][b] = fmaf(w[i], xv[i], acc[q][r][b]);
                }
        }
    }
#pragma unroll
    for (int q = 0; q < M; q++)
#pragma unroll
        for (int r = 0; r < R; r++)
#pragma unroll
            for (int b = 0; b < NB; b++) {
                const float v = warp_sum(acc[q][r][b]);
                if (lane == 0) red[warp][(q * R + r) * NB + b] = v;
            }
    if constexpr (WK > 1) __syncthreads();
    else __syncwarp();
    if (part == 0)
        for (int i = lane; i < R * NB; i += 32) {
            const int r = i / NB, b = i % NB;
            float v = 0.0f, u = 0.0f;
#pragma unroll
            for (int p = 0; p < WK; p++) {
                v += red[warp + p][i];
                if (GATED) u += red[warp + p][R * NB + i];
            }
            if (row0 + r < m && b0 + b < c.n) dense_store<T>(c, j, b0 + b, ycol + r, v, u);
        }
}

template <class T, int NB, int R, bool GATED, int MODE>
void dense_rows_wk(cudaStream_t st, const DenseCall& c) {
    int units = (c.job[0].w.m + R - 1) / R, ld = c.job[0].w.ld;
    if (!GATED && c.count == 2) {
        units += (c.job[1].w.m + R - 1) / R;
        ld = std::max(ld, c.job[1].w.ld);
    }
    const int groups = MODE == ROWS_PLAIN ? 1 : (c.n + NB - 1) / NB, all = units * groups;
    const int wk = all >= ROWS_TARGET_WARPS || ld <= 256 ? 1 : all * 2 >= ROWS_TARGET_WARPS || ld <= 512 ? 2 : 4;
    const dim3 grid((unsigned)((units * wk + ROWS_WARPS - 1) / ROWS_WARPS), (unsigned)groups), block(ROWS_WARPS * 32);
    if (wk == 1) launch_pdl(k_dense_rows<T, NB, R, GATED, 1, MODE>, grid, block, 0, st, c);
    else if (wk == 2) launch_pdl(k_dense_rows<T, NB, R, GATED, 2, MODE>, grid, block, 0, st, c);
    else launch_pdl(k_dense_rows<T, NB, R, GATED, 4, MODE>, grid, block, 0, st, c);
}

template <class T, int NB>
void dense_rows_go(cudaStream_t st, const DenseCall& c) {
    if (c.blocks) {
        if (c.blocks.rows % 2 == 0) dense_rows_wk<T, NB, 2, false, ROWS_BLOCKS>(st, c);
        else dense_rows_wk<T, NB, 1, false, ROWS_BLOCKS>(st, c);
    } else if (c.gated) {
        dense_rows_wk<T, NB, 1, true, ROWS_PLAIN>(st, c);
    } else {
        dense_rows_wk<T, NB, 2, false, ROWS_PLAIN>(st, c);
    }
}

template <class T>
void dense_rows_n(cudaStream_t st, const DenseCall& c) {
    if (c.experts) {
        if (c.gated) dense_rows_wk<T, 1, 1, true, ROWS_EXPERTS>(st, c);
        else dense_rows_wk<T, 1, 2, false, ROWS_EXPERTS>(st, c);
    } else if (c.n == 1) {
        dense_rows_go<T, 1>(st, c);
    } else if (c.n == 2) {
        dense_rows_go<T, 2>(st, c);
    } else if (c.n <= 4) {
        dense_rows_go<T, 4>(st, c);
    } else {
        dense_rows_go<T, 8>(st, c);
    }
}

// ── f32 tile kernel ────────────────────────────────────────────────────────
constexpr int ST = 64, SK = 16;  // 64 x 64 outputs per CTA, 16 columns of k per step; 256 threads, 4 x 4 outputs each

template <class T, bool GATED>
__global__ void __launch_bounds__(256) k_dense_simt(const __grid_constant__ DenseCall c) {
    constexpr int M = GATED ? 2 : 1;
    __shared__ float xs[SK][ST + 4], ws[M][SK][ST + 4];
    const DenseJob& j = c.job[GATED ? 0 : blockIdx.z];
    const int m0 = blockIdx.x * ST;
    if (m0 >= j.w.m) return;
    int n0 = blockIdx.y * ST, n_end = c.n;
    size_t wrow = 0;  // first row of the expert's matrix
    if (c.experts) {  // the expert whose tiles of sorted rows include number blockIdx.y
        int tile = blockIdx.y, e = 0;
        for (; e < c.experts.count; e++) {
            const int s0 = c.experts.start[e], s1 = c.experts.start[e + 1], t = (s1 - s0 + ST - 1) / ST;
            if (tile < t) {
                n0 = s0 + tile * ST;
                n_end = s1;
                break;
            }
            tile -= t;
        }
        if (e == c.experts.count) return;
        wrow = (size_t)e * j.w.m;
    }
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float acc[M][4][4] = {};
    const int lr = tid >> 2, lk = (tid & 3) * 4;  // the element this thread stages: row lr, four k from lk
    const bool x_ok = n0 + lr < n_end, w_ok = m0 + lr < j.w.m;
    const T* xp = (const T*)j.x + (size_t)(x_ok ? n0 + lr : 0) * j.ldx;
    for (int k0 = 0; k0 < j.w.k; k0 += SK) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int k = k0 + lk + i;
            xs[lk + i][lr] = x_ok && k < j.w.k ? act_f(xp[k]) : 0.0f;
#pragma unroll
            for (int q = 0; q < M; q++)
                ws[q][lk + i][lr] = w_ok && k < j.w.k ? __bfloat162float(c.job[GATED ? q : blockIdx.z].w.w[(wrow + m0 + lr) * j.w.ld + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < SK; k++) {
            const float4 xv = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
            const float xa[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
            for (int q = 0; q < M; q++) {
                const float4 wv = *reinterpret_cast<const float4*>(&ws[q][k][tx * 4]);
                const float wa[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
                for (int a = 0; a < 4; a++)
#pragma unroll
                    for (int b = 0; b < 4; b++) acc[q][a][b] = fmaf(xa[a], wa[b], acc[q][a][b]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int a = 0; a < 4; a++)
#pragma unroll
        for (int b = 0; b < 4; b++) {
            const int row = n0 + ty * 4 + a, col = m0 + tx * 4 + b;
            if (row < n_end && col < j.w.m) dense_store<T>(c, j, row, col, acc[0][a][b], acc[M - 1][a][b]);
        }
}

template <class T>
void dense_simt_go(cudaStream_t st, const DenseCall& c) {
    const int m = c.gated || c.count == 1 ? c.job[0].w.m : max(c.job[0].w.m, c.job[1].w.m);
    const int tiles = c.experts ? c.n / ST + std::min(c.n, c.experts.count) : (c.n + ST - 1) / ST;
    const dim3 grid((m + ST - 1) / ST, tiles, c.gated ? 1 : c.count);
    if (c.gated) k_dense_simt<T, true><<<grid, 256, 0, st>>>(c);
    else k_dense_simt<T, false><<<grid, 256, 0, st>>>(c);
}

}  // namespace

void launch_dense_rows(cudaStream_t st, bool bf16, const DenseCall& c) {
    if (c.n <= 0) return;
    g_kernel_launches++;
    if (bf16) dense_rows_n<__nv_bfloat16>(st, c);
    else dense_rows_n<float>(st, c);
}

void launch_dense_simt(cudaStream_t st, bool bf16, const DenseCall& c) {
    if (c.n <= 0) return;
    g_kernel_launches++;
    if (bf16) dense_simt_go<__nv_bfloat16>(st, c);
    else dense_simt_go<float>(st, c);
}

cudaError_t launch_dense(cudaStream_t st, bool bf16, const DenseCall& c) {
    const bool few = c.experts ? !c.experts.start : c.n <= DENSE_ROWS_MAX;
    if (few || (c.blocks && (!bf16 || c.blocks.x_step % 8))) launch_dense_rows(st, bf16, c);  // (blocks of f32 models: a few rows at a time)
    else if (bf16) return launch_dense_tc(st, c);
    else launch_dense_simt(st, bf16, c);
    return cudaGetLastError();
}

}  // namespace wick
