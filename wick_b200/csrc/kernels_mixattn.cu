// Windowed causal attention whose scores are blended across heads and squashed by a sigmoid:
//     s_g(i, j) = scale q_g(i) . k_g(j)        w_h(i, j) = sigmoid(sum_g talk[h][g] s_g(i, j) + bias[h])
//     out_h(i) = sum over visible j of w_h(i, j) v_h(j)
// with j visible to i when j <= i and (i - j < size or j < keep_first).  The blend needs the scores of every head at a (query,
// key) pair, so a CTA works on all heads of its queries; there is no normaliser, so partial sums over disjoint keys simply
// add up, and the keys of a query tile can be split over CTAs.
//
// k_mix_attn computes in f32 on the CUDA cores and takes any sizes; prompts of bf16 models go to attn_mix_tc.cu.
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

// Adds the key splits of a row in split order.
template <class T>
__global__ void __launch_bounds__(256) k_mix_attn_sum(const float* __restrict__ partial, int splits, int width, T* __restrict__ out, int ldo) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= width) return;
    const float* p = partial + (size_t)blockIdx.y * splits * width + c;
    float a = 0.0f;
    for (int i = 0; i < splits; i++) a += p[(size_t)i * width];
    out[(size_t)blockIdx.y * ldo + c] = f_act<T>(a);
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
        k_mix_attn_sum<T><<<dim3((width + 255) / 256, n), 256, 0, st>>>(partial, splits, width, (T*)out, ldo);
    }
    return cudaGetLastError();
}

}  // namespace

// The form a launch takes: tensor cores for a prompt portion of a bf16 model whose sizes allow it.
static bool mix_attn_use_tc(bool bf16, int n, const MixAttnShape& s, const RowState& rs, const MixAttnScratch& sc) {
    return bf16 && !rs.separate() && n >= MIX_ATTN_TC_MIN_ROWS && sc.fold && mix_attn_tc_supported(s);
}

void launch_qk_rms_append(cudaStream_t st, bool bf16, void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, const MixAttnScratch& sc) {
    if (n <= 0) return;
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
    if (mix_attn_use_tc(bf16, n, s, rs, sc)) return launch_mix_attn_tc(st, sc.fold, n, s, rs, out, ldo, sc.err);
    return bf16 ? mix_attn_go<__nv_bfloat16>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq)
                : mix_attn_go<float>(st, qkv, ld, n, s, rs, out, ldo, sc.partial, max_seq);
}

}  // namespace wick
