// Latent attention (launchers' header: LatentShape): the cache rows, and attention with queries taken to the latent's side.
//
// k_latent_append  a CTA per row: c_q and c divided by their root mean square and weighted, the rotated key part turned by the
//                  row's position; c and the rotated part go to the cache.
// k_latent_attn    CTA (key split, row, group of heads): scores of a tile of cache rows, running softmax, weighted sum of the
//                  tile's latents; f32 on the CUDA cores, any sizes.  A group's heads share every cache row that is read.
// k_latent_sum     merges the key splits of a row and adds the sink's share of the denominator.
// bfloat16 models take attn_latent_step.cu for the splits of a few tokens and attn_latent_tc.cu for prompts.
#include "latent_kernels.cuh"

namespace wick {

namespace {

constexpr int LA_THREADS = 256, LA_KT = 32, LA_HEADS = 8;
constexpr int LA_TARGET_CTAS = 296, LA_MAX_SPLIT = 64;
constexpr int LA_STEP_ROWS = 128;  // rows per launch of the tensor-core form, for the size of its partial records
constexpr size_t LA_SMEM_MAX = 200 * 1024;

constexpr int AP_THREADS = 256;

template <class T>
__global__ void __launch_bounds__(AP_THREADS) k_latent_append(T* __restrict__ p, int ldp, const __grid_constant__ LatentShape s, const __grid_constant__ RowState rs) {
    extern __shared__ float row[];  // c_q | c | rotated part
    __shared__ float red[2][AP_THREADS / 32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, j = blockIdx.x, Q = s.q_rank, C = s.kv_rank, skip = s.off_kv() - Q;
    pdl_launch_next();
    pdl_wait();
    const int pos = rs.pos(j);
    T* cq = p + (size_t)j * ldp;
    T* dst = (T*)rs.st0(j) + (size_t)pos * s.ldc();
    float qq = 0.0f, cc = 0.0f;
#pragma unroll 4
    for (int i = tid; i < Q + C + s.rot_dim; i += AP_THREADS) {
        const float v = act_f(cq[i < Q ? i : i + skip]);
        row[i] = v;
        if (i < Q) qq = fmaf(v, v, qq);
        else if (i < Q + C) cc = fmaf(v, v, cc);
    }
    qq = warp_sum(qq);
    cc = warp_sum(cc);
    if (lane == 0) {
        red[0][warp] = qq;
        red[1][warp] = cc;
    }
    __syncthreads();
    qq = cc = 0.0f;
#pragma unroll
    for (int i = 0; i < AP_THREADS / 32; i++) {
        qq += red[0][i];
        cc += red[1][i];
    }
    const float rq = 1.0f / sqrtf(qq / (float)Q + s.eps), rc = 1.0f / sqrtf(cc / (float)C + s.eps);
#pragma unroll 4
    for (int i = tid; i < Q; i += AP_THREADS) cq[i] = f_act<T>(row[i] * rq * s.q_norm[i]);
    const int off = s.off_rot(), ldc = s.ldc();
    const float* r = row + Q + C;
#pragma unroll 4
    for (int i = tid; i < ldc; i += AP_THREADS) {
        float v = 0.0f;
        if (i < C) {
            v = row[Q + i] * rc * s.kv_norm[i];
        } else if (i >= off && i - off < s.rot_dim) {
            const int d = i - off;
            v = r[d];
            if (d < s.rot_dims) {
                const float2 cs = s.rope[(size_t)pos * (s.rot_dims / 2) + d / 2];
                v = d % 2 == 0 ? v * cs.x - r[d + 1] * cs.y : v * cs.x + r[d - 1] * cs.y;
            }
        }
        dst[i] = f_act<T>(v);
    }
}

__device__ __forceinline__ int first_key(const LatentShape& s, int pos) { return s.size > 0 ? max(0, pos - s.size + 1) : 0; }

template <class T>
__global__ void __launch_bounds__(LA_THREADS) k_latent_attn(const T* __restrict__ qc, const T* __restrict__ q, int ldq, const __grid_constant__ LatentShape s,
                                                            const __grid_constant__ RowState rs, T* __restrict__ o, int ldo_h, float* __restrict__ partial) {
    extern __shared__ __align__(16) float sm[];
    const int H = s.heads, D = s.ldc(), C = s.kv_rank, Cp = s.off_rot(), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int j = blockIdx.y, h0 = blockIdx.z * LA_HEADS, hn = min(LA_HEADS, H - h0);
    float* qs = sm;                       // [LA_HEADS][D] queries, scaled
    float* acc = qs + LA_HEADS * D;       // [LA_HEADS][Cp]
    float* wt = acc + LA_HEADS * Cp;      // [LA_HEADS][KT]
    __shared__ float top[LA_HEADS], sum[LA_HEADS], fix[LA_HEADS];
    pdl_launch_next();
    pdl_wait();
    const int pos = rs.pos(j), lo = first_key(s, pos), keys = pos - lo + 1;
    const T* cache = (const T*)rs.st0(j);
    const float2* cs = s.rope + (size_t)pos * (s.rot_dims / 2);
    for (int i = tid; i < hn * D; i += LA_THREADS) {
        const int h = h0 + i / D, d = i % D;
        float v = 0.0f;
        if (d < C) {
            v = act_f(qc[((size_t)j * H + h) * D + d]);
        } else if (d >= Cp && d - Cp < s.rot_dim) {
            const int r = d - Cp;
            const T* p = q + (size_t)j * ldq + (size_t)h * s.q_pitch() + s.q_off_rot();
            v = act_f(p[r]);
            if (r < s.rot_dims) v = r % 2 == 0 ? v * cs[r / 2].x - act_f(p[r + 1]) * cs[r / 2].y : v * cs[r / 2].x + act_f(p[r - 1]) * cs[r / 2].y;
        }
        qs[i] = v * s.scale;
    }
    for (int i = tid; i < LA_HEADS * Cp; i += LA_THREADS) acc[i] = 0.0f;
    if (tid < LA_HEADS) {
        top[tid] = -INFINITY;
        sum[tid] = 0.0f;
    }
    __syncthreads();
    for (int t0 = blockIdx.x * LA_KT; t0 < keys; t0 += gridDim.x * LA_KT) {
        const int cnt = min(LA_KT, keys - t0);
        // scores: a warp per key, lanes split the columns
        for (int key = warp; key < LA_KT; key += LA_THREADS / 32) {
            float a[LA_HEADS] = {};
            if (key < cnt) {
                const T* row = cache + (size_t)(lo + t0 + key) * D;
                for (int d = lane * 8; d < D; d += 256) {
                    float kv[8];
                    load8(row + d, kv);
#pragma unroll
                    for (int h = 0; h < LA_HEADS; h++)
                        if (h < hn)
#pragma unroll
                            for (int x = 0; x < 8; x++) a[h] = fmaf(qs[h * D + d + x], kv[x], a[h]);
                }
            }
#pragma unroll
            for (int h = 0; h < LA_HEADS; h++) {
                const float v = warp_sum(a[h]);
                if (lane == 0) wt[h * LA_KT + key] = key < cnt ? v : -INFINITY;
            }
        }
        __syncthreads();
        for (int h = warp; h < hn; h += LA_THREADS / 32) {
            const float v = wt[h * LA_KT + lane];
            float mx = v;
#pragma unroll
            for (int x = 16; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            mx = fmaxf(mx, top[h]);
            const float e = expf(v - mx), es = warp_sum(e);
            wt[h * LA_KT + lane] = e;
            if (lane == 0) {
                const float f = expf(top[h] - mx);
                fix[h] = f;
                sum[h] = fmaf(sum[h], f, es);
                top[h] = mx;
            }
        }
        __syncthreads();
        for (int i = tid; i < hn * C; i += LA_THREADS) {
            const int h = i / C, c = i % C;
            float a = acc[h * Cp + c] * fix[h];
            for (int key = 0; key < cnt; key++) a = fmaf(wt[h * LA_KT + key], act_f(cache[(size_t)(lo + t0 + key) * D + c]), a);
            acc[h * Cp + c] = a;
        }
        __syncthreads();
    }
    if (!partial) {
        for (int i = tid; i < hn * ldo_h; i += LA_THREADS) {
            const int h = i / ldo_h, c = i % ldo_h;
            const float sink = s.sink[h0 + h], mx = fmaxf(top[h], sink);
            const float f = expf(top[h] - mx) / (sum[h] * expf(top[h] - mx) + expf(sink - mx));
            o[((size_t)j * H + h0 + h) * ldo_h + c] = f_act<T>(c < C ? acc[h * Cp + c] * f : 0.0f);
        }
        return;
    }
    // [row][head][split]: C sums, then top and sum
    for (int i = tid; i < hn * (C + 2); i += LA_THREADS) {
        const int h = i / (C + 2), c = i % (C + 2);
        partial[(((size_t)j * H + h0 + h) * gridDim.x + blockIdx.x) * (C + 2) + c] = c < C ? acc[h * Cp + c] : c == C ? top[h] : sum[h];
    }
}

// A CTA per (head, row).  split_keys > 0: split i holds keys i * split_keys .. of the row, those past its last key are not there.
template <class T>
__global__ void __launch_bounds__(256) k_latent_sum(const float* __restrict__ partial, int splits, int split_keys, const __grid_constant__ LatentShape s,
                                                    const __grid_constant__ RowState rs, T* __restrict__ o, int ldo_h) {
    const int C = s.kv_rank, h = blockIdx.x, H = s.heads, j = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    __shared__ float w[LATENT_MAX_SPLIT], red[2][8];
    pdl_launch_next();
    pdl_wait();
    const float* p = partial + ((size_t)j * H + h) * splits * (C + 2);
    int used = splits;
    if (split_keys > 0) {
        const int pos = rs.pos(j);
        used = (pos - first_key(s, pos) + split_keys) / split_keys;
    }
    // (log weights and the sink in units of log2 where the splits were made by the tensor-core form)
    const float unit = split_keys > 0 ? 1.4426950408889634f : 1.0f, sink = s.sink[h] * unit;
    float top = tid < used ? p[(size_t)tid * (C + 2) + C] : -INFINITY, sum = tid < used ? p[(size_t)tid * (C + 2) + C + 1] : 0.0f;
    float mx = fmaxf(top, sink);
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
    if (lane == 0) red[0][warp] = mx;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; i++) mx = fmaxf(mx, red[0][i]);
    const float f = split_keys > 0 ? exp2f(top - mx) : expf(top - mx);
    sum = warp_sum(sum * f);
    if (lane == 0) red[1][warp] = sum;
    if (tid < used) w[tid] = f;
    __syncthreads();
    float den = split_keys > 0 ? exp2f(sink - mx) : expf(sink - mx);
#pragma unroll
    for (int i = 0; i < 8; i++) den += red[1][i];
    const float inv = 1.0f / den;
    for (int c = tid; c < ldo_h; c += 256) {
        float a = 0.0f;
        if (c < C)
#pragma unroll 8
            for (int i = 0; i < used; i++) a = fmaf(w[i], p[(size_t)i * (C + 2) + c], a);
        o[((size_t)j * H + h) * ldo_h + c] = f_act<T>(a * inv);
    }
}

size_t latent_smem(const LatentShape& s) { return (size_t)LA_HEADS * (s.ldc() + s.off_rot() + LA_KT) * 4; }

int latent_splits(const LatentShape& s, int rows, int max_seq) {
    const int groups = (s.heads + LA_HEADS - 1) / LA_HEADS, ctas = rows * groups, tiles = (s.seen(max_seq) + LA_KT - 1) / LA_KT;
    return std::max(1, std::min({LA_TARGET_CTAS / ctas, tiles, LA_MAX_SPLIT}));
}

template <class T>
cudaError_t latent_attn_go(cudaStream_t st, const void* qc, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs, void* o, int ldo_h,
                           float* partial, int max_seq) {
    static_assert(LA_MAX_SPLIT <= LATENT_MAX_SPLIT && LATENT_MAX_SPLIT <= 256, "a thread per split");
    const size_t smem = latent_smem(s);
    if (smem > 40 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(k_latent_attn<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    const int splits = latent_splits(s, n, max_seq);
    g_kernel_launches++;
    launch_pdl(k_latent_attn<T>, dim3(splits, n, (s.heads + LA_HEADS - 1) / LA_HEADS), dim3(LA_THREADS), smem, st, (const T*)qc, (const T*)q, ldq, s, rs, (T*)o,
               ldo_h, splits > 1 ? partial : nullptr);
    if (splits > 1) {
        g_kernel_launches++;
        launch_pdl(k_latent_sum<T>, dim3(s.heads, n), dim3(256), 0, st, partial, splits, 0, s, rs, (T*)o, ldo_h);
    }
    return cudaGetLastError();
}

}  // namespace

bool latent_supported(const LatentShape& s) { return latent_smem(s) <= LA_SMEM_MAX && (size_t)(s.q_rank + s.kv_rank + s.rot_dim) * 4 <= LA_SMEM_MAX; }

static int step_splits(const LatentShape& s, int max_seq) { return (s.seen(max_seq) + LATENT_STEP_KEYS - 1) / LATENT_STEP_KEYS; }

size_t latent_scratch(const LatentShape& s, bool bf16, int max_rows, int max_seq) {
    const int groups = (s.heads + LA_HEADS - 1) / LA_HEADS;
    // rows * splits: splits <= target / (rows * groups), at least one
    size_t records = (size_t)std::max(LA_TARGET_CTAS / groups + 1, max_rows);
    if (bf16 && latent_step_supported(s, max_seq)) records = (size_t)std::min(max_rows, LA_STEP_ROWS) * step_splits(s, max_seq);
    return records * s.heads * (s.kv_rank + 2);
}

void launch_latent_append(cudaStream_t st, bool bf16, void* p, int ldp, int n, const LatentShape& s, const RowState& rs) {
    if (n <= 0) return;
    const size_t smem = (size_t)(s.q_rank + s.kv_rank + s.rot_dim) * 4;
    g_kernel_launches++;
    auto go = [&](auto kernel, auto* rows) {
        if (smem > 40 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_pdl(kernel, dim3(n), dim3(AP_THREADS), smem, st, rows, ldp, s, rs);
    };
    if (bf16) go(k_latent_append<__nv_bfloat16>, (__nv_bfloat16*)p);
    else go(k_latent_append<float>, (float*)p);
}

cudaError_t launch_latent_attn(cudaStream_t st, bool bf16, const void* qc, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs,
                               void* o, int ldo_h, const LatentScratch& sc, int max_seq) {
    if (n <= 0) return cudaSuccess;
    if (!bf16) return latent_attn_go<float>(st, qc, q, ldq, n, s, rs, o, ldo_h, sc.partial, max_seq);
    using B = __nv_bfloat16;
    if (!latent_step_supported(s, max_seq)) return latent_attn_go<B>(st, qc, q, ldq, n, s, rs, o, ldo_h, sc.partial, max_seq);
    const int splits = step_splits(s, max_seq);
    for (int r0 = 0; r0 < n; r0 += LA_STEP_ROWS) {
        const int rows = std::min(LA_STEP_ROWS, n - r0);
        RowState part = rs;
        if (part.p0) part.p0 += r0;
        if (part.positions) part.positions += r0;
        part.start_pos += r0;
        const cudaError_t e = launch_latent_step(st, (const B*)qc + (size_t)r0 * s.heads * s.ldc(), (const B*)q + (size_t)r0 * ldq, ldq, rows, s, part, sc.partial,
                                                 splits, sc.err);
        if (e != cudaSuccess) return e;
        g_kernel_launches++;
        launch_pdl(k_latent_sum<B>, dim3(s.heads, rows), dim3(256), 0, st, sc.partial, splits, LATENT_STEP_KEYS, s, part,
                   (B*)o + (size_t)r0 * s.heads * ldo_h, ldo_h);
    }
    return cudaGetLastError();
}

}  // namespace wick
