// Windowed causal attention whose scores are blended across heads and squashed by a sigmoid:
//     s_g(i, j) = scale q_g(i) . k_g(j)        w_h(i, j) = sigmoid(sum_g talk[h][g] s_g(i, j) + bias[h])
//     out_h(i) = sum over visible j of w_h(i, j) v_h(j)
// with j visible to i when j <= i and (i - j < size or j < keep_first).  The blend needs the scores of every head at a (query,
// key) pair, so a CTA works on all heads of its queries; there is no normaliser, so partial sums over disjoint keys simply
// add up, and the keys of a query tile can be split over CTAs.
//
// k_mix_attn computes in f32 on the CUDA cores and takes any sizes; k_mix_attn_step is the decode form; prompts of bf16 models go to attn_mix_tc.cu.
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

constexpr int MA_THREADS = 256, MA_KT = 32;
constexpr int MA_TARGET_CTAS = 296, MA_MAX_SPLIT = 64;

// q and k RMS norm per head (no weight), k and v rows into the caches: one warp per (row, head of q | k | v).
template <class T>
__global__ void __launch_bounds__(256) k_qk_rms_append(T* __restrict__ qkv, int ld, int n, const __grid_constant__ MixAttnShape s,
                                                       const __grid_constant__ RowState rs) {
    const int lane = threadIdx.x & 31, H = s.heads, G = s.kv_heads, D = s.dim, E = s.vdim;
    const size_t unit = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int seg_n = H + 2 * G;
    if (unit >= (size_t)n * seg_n) return;
    const int j = (int)(unit / seg_n), seg = (int)(unit % seg_n);
    T* row = qkv + (size_t)j * ld;
    if (seg >= H + G) {
        const int g = seg - H - G;
        T* dst = (T*)rs.st1(j) + (size_t)rs.pos(j) * G * E + g * E;
        const T* src = row + (H + G) * D + g * E;
        for (int i = lane; i < E; i += 32) dst[i] = src[i];
        return;
    }
    T* src = row + seg * D;
    float ss = 0.0f;
    for (int i = lane; i < D; i += 32) {
        const float v = act_f(src[i]);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)D + s.eps);
    T* dst = seg < H ? src : (T*)rs.st0(j) + (size_t)rs.pos(j) * G * D + (seg - H) * D;
    for (int i = lane; i < D; i += 32) dst[i] = f_act<T>(act_f(src[i]) * r);
}

// The keys a tile of queries at positions p0 .. p1 may see: the kept first keys that lie before the window of p0, then
// [lo, p1].  Numbered 0 .. count - 1.
struct KeyRange {
    int ns, lo, count;
    __device__ KeyRange(const MixAttnShape& s, int p0, int p1) {
        lo = s.size > 0 ? max(0, p0 - s.size + 1) : 0;
        ns = min(s.keep_first, lo);
        count = ns + p1 - lo + 1;
    }
    __device__ int key(int i) const { return i < ns ? i : lo + i - ns; }
};
__device__ __forceinline__ bool key_visible(const MixAttnShape& s, int i, int j) {
    return j <= i && (s.size <= 0 || i - j < s.size || j < s.keep_first);
}

template <class T>
__device__ __forceinline__ float dot_any(const float* __restrict__ q, const T* __restrict__ k, int d) {
    float a0 = 0.0f, a1 = 0.0f;
    int i = 0;
    if (d % 8 == 0 && (reinterpret_cast<uintptr_t>(k) & 15) == 0)
        for (; i < d; i += 8) {
            float kv[8];
            load8(k + i, kv);
#pragma unroll
            for (int x = 0; x < 8; x += 2) {
                a0 = fmaf(q[i + x], kv[x], a0);
                a1 = fmaf(q[i + x + 1], kv[x + 1], a1);
            }
        }
    for (; i < d; i++) a0 = fmaf(q[i], act_f(k[i]), a0);
    return a0 + a1;
}

// Tile of qt queries (consecutive tokens of one sequence, or one row of its own), the key tiles blockIdx.y, + gridDim.y, ...
template <class T>
__global__ void __launch_bounds__(MA_THREADS) k_mix_attn(const T* __restrict__ q, int ldq, int n, int qt, const __grid_constant__ MixAttnShape s,
                                                         const __grid_constant__ RowState rs, T* __restrict__ out, int ldo,
                                                         float* __restrict__ partial) {
    extern __shared__ __align__(16) float sm[];
    const int H = s.heads, G = s.kv_heads, D = s.dim, E = s.vdim, rep = H / G, tid = threadIdx.x;
    const int j0 = blockIdx.x * qt, nq = min(qt, n - j0);
    float* qs = sm;                                // [qt][H*D]
    float* acc = qs + (size_t)qt * H * D;          // [qt][H*E]
    float* sc = acc + (size_t)qt * H * E;          // [qt][H][KT] scores
    float* wt = sc + (size_t)qt * H * MA_KT;       // [qt][H][KT] weights
    float* tk = wt + (size_t)qt * H * MA_KT;       // [H][H]
    float* bi = tk + H * H;                        // [H]
    for (int i = tid; i < nq * H * D; i += MA_THREADS) qs[i] = act_f(q[(size_t)(j0 + i / (H * D)) * ldq + i % (H * D)]);
    for (int i = tid; i < nq * H * E; i += MA_THREADS) acc[i] = 0.0f;
    for (int i = tid; i < H * H; i += MA_THREADS) tk[i] = s.talk ? s.talk[i] : (i / H == i % H ? 1.0f : 0.0f);
    for (int i = tid; i < H; i += MA_THREADS) bi[i] = s.bias ? s.bias[i] : 0.0f;
    const int p0 = rs.pos(j0), p1 = p0 + nq - 1;
    const KeyRange kr(s, p0, p1);
    const T* kc = (const T*)rs.st0(j0);
    const T* vc = (const T*)rs.st1(j0);
    __syncthreads();
    for (int t0 = blockIdx.y * MA_KT; t0 < kr.count; t0 += gridDim.y * MA_KT) {
        const int cnt = min(MA_KT, kr.count - t0);
        for (int i = tid; i < nq * H * MA_KT; i += MA_THREADS) {
            const int key = i % MA_KT, h = i / MA_KT % H, qi = i / MA_KT / H;
            if (key < cnt) sc[i] = dot_any(qs + (qi * H + h) * D, kc + ((size_t)kr.key(t0 + key) * G + h / rep) * D, D) * s.scale;
        }
        __syncthreads();
        for (int i = tid; i < nq * H * MA_KT; i += MA_THREADS) {
            const int key = i % MA_KT, h = i / MA_KT % H, qi = i / MA_KT / H;
            float w = 0.0f;
            if (key < cnt && key_visible(s, p0 + qi, kr.key(t0 + key))) {
                float z = bi[h];
                for (int g = 0; g < H; g++) z = fmaf(tk[h * H + g], sc[(qi * H + g) * MA_KT + key], z);
                w = sigmoid_f(z);
            }
            wt[i] = w;
        }
        __syncthreads();
        for (int c = tid; c < H * E; c += MA_THREADS) {
            const int h = c / E, g = h / rep;
            for (int qi = 0; qi < nq; qi++) {
                float a = acc[qi * H * E + c];
                for (int key = 0; key < cnt; key++)
                    a = fmaf(wt[(qi * H + h) * MA_KT + key], act_f(vc[((size_t)kr.key(t0 + key) * G + g) * E + c % E]), a);
                acc[qi * H * E + c] = a;
            }
        }
        __syncthreads();
    }
    for (int i = tid; i < nq * H * E; i += MA_THREADS) {
        const int qi = i / (H * E), c = i % (H * E);
        if (partial) partial[((size_t)(j0 + qi) * gridDim.y + blockIdx.y) * H * E + c] = acc[i];
        else out[(size_t)(j0 + qi) * ldo + c] = f_act<T>(acc[i]);
    }
}

// ── one decode token per row ───────────────────────────────────────────────
// CTA (split, row): the key tiles split, + gridDim.x, ... of the row's visible keys, all heads.  Normalises q itself; the CTA
// whose tile holds the row's own position also normalises k and appends the k and v rows first.  Sizes multiples of 8.
constexpr int MS_KT = 16, MS_CHUNKS = 4;  // keys per tile; 8-column pieces of the output per thread

template <class T>
__device__ __forceinline__ void rms_head(const T* __restrict__ src, int d, float eps, int lane, float* dst_f, T* dst_t) {
    float ss = 0.0f;
    for (int i = lane; i < d; i += 32) {
        const float v = act_f(src[i]);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);
    for (int i = lane; i < d; i += 32) {
        const T v = f_act<T>(act_f(src[i]) * r);  // q is rounded like the cached k
        if (dst_t) dst_t[i] = v;
        else dst_f[i] = act_f(v);
    }
}

template <class T>
__global__ void __launch_bounds__(MA_THREADS) k_mix_attn_step(const T* __restrict__ qkv, int ld, const __grid_constant__ MixAttnShape s,
                                                              const __grid_constant__ RowState rs, T* __restrict__ out, int ldo,
                                                              float* __restrict__ partial) {
    extern __shared__ __align__(16) float sm[];
    const int H = s.heads, G = s.kv_heads, D = s.dim, E = s.vdim, rep = H / G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, j = blockIdx.y;
    float* qs = sm;                          // [H*D]
    float* sc = qs + H * D;                  // [H][KT] scores
    float* wt = sc + H * MS_KT;              // [H][KT] weights
    float* tk = wt + H * MS_KT;              // [H][H]
    float* bi = tk + H * H;                  // [H]
    float* red = bi + round_up(H, 4);        // [groups][H*E] at the end
    for (int i = tid; i < H * H; i += MA_THREADS) tk[i] = s.talk ? s.talk[i] : (i / H == i % H ? 1.0f : 0.0f);
    for (int i = tid; i < H; i += MA_THREADS) bi[i] = s.bias ? s.bias[i] : 0.0f;
    pdl_launch_next();
    pdl_wait();
    const int pos = rs.pos(j);
    const KeyRange kr(s, pos, pos);
    T* kc = (T*)rs.st0(j);
    T* vc = (T*)rs.st1(j);
    const T* row = qkv + (size_t)j * ld;
    const int tiles = (kr.count + MS_KT - 1) / MS_KT;
    const bool newest = (tiles - 1) % (int)gridDim.x == (int)blockIdx.x;
    for (int seg = warp; seg < H + (newest ? G : 0); seg += MA_THREADS / 32)
        rms_head<T>(row + seg * D, D, s.eps, lane, qs + seg * D, seg < H ? nullptr : kc + (size_t)pos * G * D + (seg - H) * D);
    if (newest)
        for (int i = tid; i < G * E; i += MA_THREADS) vc[(size_t)pos * G * E + i] = row[(H + G) * D + i];
    __syncthreads();
    const int CH = H * E / 8, groups = CH >= MA_THREADS ? 1 : MA_THREADS / CH;  // key groups of the weighted sum
    float acc[MS_CHUNKS][8] = {};
    for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
        const int t0 = t * MS_KT, cnt = min(MS_KT, kr.count - t0);
        for (int i = tid; i < H * MS_KT; i += MA_THREADS) {
            const int key = i % MS_KT, h = i / MS_KT;
            float a0 = 0.0f, a1 = 0.0f;
            if (key < cnt) {
                const T* kp = kc + ((size_t)kr.key(t0 + key) * G + h / rep) * D;
                const float* qp = qs + h * D;
#pragma unroll 8
                for (int d = 0; d < D; d += 8) {
                    float kv[8];
                    load8(kp + d, kv);
#pragma unroll
                    for (int x = 0; x < 8; x += 2) {
                        a0 = fmaf(qp[d + x], kv[x], a0);
                        a1 = fmaf(qp[d + x + 1], kv[x + 1], a1);
                    }
                }
            }
            sc[i] = (a0 + a1) * s.scale;
        }
        __syncthreads();
        for (int i = tid; i < H * MS_KT; i += MA_THREADS) {
            const int key = i % MS_KT, h = i / MS_KT;
            float z = bi[h];
            for (int g = 0; g < H; g++) z = fmaf(tk[h * H + g], sc[g * MS_KT + key], z);
            wt[i] = key < cnt ? sigmoid_f(z) : 0.0f;  // every key of the range is visible to the row's position
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < MS_CHUNKS; x++) {
            const int c = groups > 1 ? (x == 0 && tid < CH * groups ? tid % CH : CH) : tid + x * MA_THREADS, grp = groups > 1 ? tid / CH : 0;
            if (c < CH) {
                const int h = c * 8 / E;
                const T* vp = vc + (size_t)(h / rep) * E + c * 8 % E;
#pragma unroll 4
                for (int key = grp; key < cnt; key += groups) {
                    float v[8];
                    load8(vp + (size_t)kr.key(t0 + key) * G * E, v);
                    const float w = wt[h * MS_KT + key];
#pragma unroll
                    for (int e = 0; e < 8; e++) acc[x][e] = fmaf(w, v[e], acc[x][e]);
                }
            }
        }
        __syncthreads();
    }
    if (groups > 1) {
        if (tid < CH * groups)
#pragma unroll
            for (int e = 0; e < 8; e++) red[tid * 8 + e] = acc[0][e];
        __syncthreads();
        if (tid < CH)
#pragma unroll
            for (int e = 0; e < 8; e++) {
                float a = red[tid * 8 + e];
                for (int g = 1; g < groups; g++) a += red[(g * CH + tid) * 8 + e];
                acc[0][e] = a;
            }
    }
    const size_t base = ((size_t)j * gridDim.x + blockIdx.x) * H * E;
#pragma unroll
    for (int x = 0; x < MS_CHUNKS; x++) {
        const int c = tid + x * MA_THREADS;
        if (c < CH)
#pragma unroll
            for (int e = 0; e < 8; e++) {
                if (partial) partial[base + c * 8 + e] = acc[x][e];
                else out[(size_t)j * ldo + c * 8 + e] = f_act<T>(acc[x][e]);
            }
    }
}

// Adds the key splits of a row in a fixed order: 32 columns per CTA, eight strided runs of splits, then the runs.
template <class T>
__global__ void __launch_bounds__(256) k_mix_attn_sum(const float* __restrict__ partial, int splits, int width, T* __restrict__ out, int ldo) {
    __shared__ float red[8][32];
    const int lane = threadIdx.x & 31, run = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    pdl_launch_next();
    pdl_wait();
    const float* p = partial + (size_t)blockIdx.y * splits * width + c;
    float a = 0.0f;
    if (c < width)
#pragma unroll 8
        for (int i = run; i < splits; i += 8) a += p[(size_t)i * width];
    red[run][lane] = a;
    __syncthreads();
    if (run == 0 && c < width) {
#pragma unroll
        for (int i = 1; i < 8; i++) a += red[i][lane];
        out[(size_t)blockIdx.y * ldo + c] = f_act<T>(a);
    }
}

size_t mix_attn_smem(const MixAttnShape& s, int qt) {
    return ((size_t)qt * s.heads * (s.dim + s.vdim + 2 * MA_KT) + (size_t)s.heads * s.heads + s.heads) * 4;
}
constexpr size_t MA_SMEM_MAX = 200 * 1024;

int mix_attn_splits(const MixAttnShape& s, int ctas, int max_seq) {
    const int tiles = (s.seen(max_seq) + MA_KT - 1) / MA_KT + 1;
    return std::max(1, std::min({(MA_TARGET_CTAS + ctas - 1) / std::max(ctas, 1), tiles, MA_MAX_SPLIT}));
}

template <class T>
cudaError_t mix_attn_go(cudaStream_t st, const void* q, int ldq, int n, const MixAttnShape& s, const RowState& rs, void* out, int ldo,
                        float* partial, int max_seq) {
    int qt = rs.separate() ? 1 : 4;
    while (qt > 1 && (mix_attn_smem(s, qt) > MA_SMEM_MAX / 2 || qt > n)) qt /= 2;
    const size_t smem = mix_attn_smem(s, qt);
    if (smem > 48 * 1024) cudaFuncSetAttribute(k_mix_attn<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int ctas = (n + qt - 1) / qt, splits = mix_attn_splits(s, ctas, max_seq);
    g_kernel_launches++;
    k_mix_attn<T><<<dim3(ctas, splits), MA_THREADS, smem, st>>>((const T*)q, ldq, n, qt, s, rs, (T*)out, ldo, splits > 1 ? partial : nullptr);
    if (splits > 1) {
        const int width = s.heads * s.vdim;
        g_kernel_launches++;
        launch_pdl(k_mix_attn_sum<T>, dim3((width + 31) / 32, n), dim3(256), 0, st, partial, splits, width, (T*)out, ldo);
    }
    return cudaGetLastError();
}

size_t mix_attn_step_smem(const MixAttnShape& s) {
    const int ch = s.heads * s.vdim / 8, groups = ch >= MA_THREADS || ch == 0 ? 1 : MA_THREADS / ch;
    return ((size_t)s.heads * (s.dim + 2 * MS_KT) + (size_t)s.heads * s.heads + round_up(s.heads, 4) + (groups > 1 ? (size_t)groups * ch * 8 : 0)) * 4;
}
bool mix_attn_step_supported(const MixAttnShape& s) {
    return s.dim % 8 == 0 && s.vdim % 8 == 0 && s.heads * s.vdim <= 8 * MS_CHUNKS * MA_THREADS && mix_attn_step_smem(s) <= MA_SMEM_MAX;
}

template <class T>
cudaError_t mix_attn_step_go(cudaStream_t st, const void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, void* out, int ldo,
                             float* partial, int max_seq) {
    const size_t smem = mix_attn_step_smem(s);
    if (smem > 40 * 1024) cudaFuncSetAttribute(k_mix_attn_step<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int tiles = (s.seen(max_seq) + MS_KT - 1) / MS_KT + 1;
    const int splits = std::max(1, std::min({MA_TARGET_CTAS / n, tiles, 2 * MA_MAX_SPLIT}));
    g_kernel_launches++;
    launch_pdl(k_mix_attn_step<T>, dim3(splits, n), dim3(MA_THREADS), smem, st, (const T*)qkv, ld, s, rs, (T*)out, ldo, splits > 1 ? partial : nullptr);
    if (splits > 1) {
        const int width = s.heads * s.vdim;
        g_kernel_launches++;
        launch_pdl(k_mix_attn_sum<T>, dim3((width + 31) / 32, n), dim3(256), 0, st, partial, splits, width, (T*)out, ldo);
    }
    return cudaGetLastError();
}

}  // namespace

// The form a launch takes: tensor cores for a prompt portion of a bf16 model whose sizes allow it.
static bool mix_attn_use_tc(bool bf16, int n, const MixAttnShape& s, const RowState& rs, const MixAttnScratch& sc) {
    return bf16 && !rs.separate() && n >= MIX_ATTN_TC_MIN_ROWS && sc.fold && mix_attn_tc_supported(s);
}

void launch_qk_rms_append(cudaStream_t st, bool bf16, void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, const MixAttnScratch& sc) {
    if (n <= 0 || (rs.separate() && mix_attn_step_supported(s))) return;  // k_mix_attn_step does it itself
    if (mix_attn_use_tc(bf16, n, s, rs, sc)) return launch_qk_fold_append(st, qkv, ld, n, s, rs, sc.fold);
    const unsigned grid = (unsigned)(((size_t)n * (s.heads + 2 * s.kv_heads) + 7) / 8);
    g_kernel_launches++;
    if (bf16) k_qk_rms_append<__nv_bfloat16><<<grid, 256, 0, st>>>((__nv_bfloat16*)qkv, ld, n, s, rs);
    else k_qk_rms_append<float><<<grid, 256, 0, st>>>((float*)qkv, ld, n, s, rs);
}

bool mix_attn_supported(const MixAttnShape& s) { return mix_attn_smem(s, 1) <= MA_SMEM_MAX; }

void mix_attn_scratch(const MixAttnShape& s, bool bf16, int max_rows, size_t* partial_floats, size_t* fold_bytes) {
    // rows x splits: splits <= (target + CTAs - 1) / CTAs with up to 4 queries per CTA
    *partial_floats = (size_t)4 * (MA_TARGET_CTAS + max_rows) * s.heads * s.vdim;
    *fold_bytes = bf16 && mix_attn_tc_supported(s) ? (size_t)max_rows * s.heads * s.kv_heads * s.dim * 2 : 0;
}

cudaError_t launch_mix_attn(cudaStream_t st, bool bf16, const void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, void* out,
                            int ldo, const MixAttnScratch& sc, int max_seq) {
    if (n <= 0) return cudaSuccess;
    if (rs.separate() && mix_attn_step_supported(s))
        return bf16 ? mix_attn_step_go<__nv_bfloat16>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq)
                    : mix_attn_step_go<float>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq);
    if (mix_attn_use_tc(bf16, n, s, rs, sc)) return launch_mix_attn_tc(st, sc.fold, n, s, rs, out, ldo, sc.err);
    return bf16 ? mix_attn_go<__nv_bfloat16>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq)
                : mix_attn_go<float>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq);
}

}  // namespace wick
