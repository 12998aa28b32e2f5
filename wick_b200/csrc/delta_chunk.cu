// Prompt form of the channel-decay delta rule (kernels_delta.cu): DC tokens at a time, in f32.
//
// Within a chunk of DC tokens with decays g_1 .. g_DC (per key channel) and state S before it, unrolling
//     S <- diag(g_i) S;  u_i = beta_i (v_i - S^T k_i);  S <- S + k_i u_i^T;  o_i = S^T q_i
// gives, with D(j, i) = diag(g_{j+1} ... g_i) (the decay from token j to token i),
//     u_i = beta_i (v_i - S^T D(0,i) k_i - sum_{j<i} (k_i . D(j,i) k_j) u_j)
//     o_i =               S^T D(0,i) q_i + sum_{j<=i} (q_i . D(j,i) k_j) u_j
//     S'  = D(0,DC) S + sum_j D(j,DC) k_j u_j^T
// so that the state takes part once per chunk: 2 DC dot products that do not wait for each other, a triangular system of size
// DC per value channel, and one update of rank DC.  Every factor is a product of decays in (0, 1]: nothing is divided and
// nothing can overflow.
//
// k_delta_chunk_prep  a warp per (chunk, head): convolutions + silu, unit q and k, decays, and from them the chunk's record
//                     [D(0,i) k_i][D(0,i) q_i][D(j,DC) k_j][D(0,DC)][beta_i k_i . D(j,i) k_j][q_i . D(j,i) k_j][beta]
// k_delta_chunk_scan  a warp owns NC value channels of a head for the whole prompt: 32 lanes split the key channels, state and
//                     accumulators in registers; records arrive by cp.async one chunk ahead.
// Tokens past the end of the prompt have beta = 0, g = 1, k = q = 0 and change nothing.
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

constexpr int DC = DELTA_CHUNK;

// key channel r of lane `lane` in rows of 32 R channels: vectors of up to four where R allows
template <int R>
struct Lanes {
    static constexpr int V = R % 4 == 0 ? 4 : R % 2 == 0 ? 2 : 1;
    __device__ static int channel(int lane, int r) { return (r / V) * 32 * V + lane * V + r % V; }
    __device__ static void load(const float* row, int lane, float* x) {
#pragma unroll
        for (int r = 0; r < R; r += V) {
            const float* p = row + (r / V) * 32 * V + lane * V;
            if constexpr (V == 4) {
                const float4 t = *reinterpret_cast<const float4*>(p);
                x[r] = t.x; x[r + 1] = t.y; x[r + 2] = t.z; x[r + 3] = t.w;
            } else if constexpr (V == 2) {
                const float2 t = *reinterpret_cast<const float2*>(p);
                x[r] = t.x; x[r + 1] = t.y;
            } else {
                x[r] = *p;
            }
        }
    }
    __device__ static void store(float* row, int lane, const float* x) {
#pragma unroll
        for (int r = 0; r < R; r += V) {
            float* p = row + (r / V) * 32 * V + lane * V;
            if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[r], x[r + 1], x[r + 2], x[r + 3]);
            else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(x[r], x[r + 1]);
            else *p = x[r];
        }
    }
};

__host__ __device__ constexpr int rec_floats(int dp) { return (3 * DC + 1) * dp + 2 * DC * DC + DC; }

// silu after a convolution: an activation, so a bfloat16 model takes the fast forms
template <class T>
__device__ __forceinline__ float conv_act(float z) {
    if constexpr (sizeof(T) == 2) return __fdividef(z, 1.0f + __expf(-z));
    else return silu_f(z);
}

// One halving exchange of a transposing sum over the lanes: N values become N / 2, lanes with bit OFF keep the upper half.
template <int N, int OFF>
__device__ __forceinline__ void halve(float* x, int lane) {
    const bool up = lane & OFF;
#pragma unroll
    for (int i = 0; i < N / 2; i++) {
        const float keep = up ? x[i + N / 2] : x[i], send = up ? x[i] : x[i + N / 2];
        x[i] = keep + __shfl_xor_sync(0xffffffffu, send, OFF);
    }
}
// Sums of 16 values over the lanes: lane l returns that of value l / 2.
__device__ __forceinline__ float sum16(float* x, int lane) {
    halve<16, 16>(x, lane);
    halve<8, 8>(x, lane);
    halve<4, 4>(x, lane);
    halve<2, 2>(x, lane);
    return x[0] + __shfl_xor_sync(0xffffffffu, x[0], 1);
}

// Convolution + silu of channel ch for the DC tokens from t0 on (tokens >= n: zero).
template <class T, int TAPS>
__device__ __forceinline__ void conv_run(const DeltaPrepArgs& a, const float* state, int C, int taps, int t0, int n, int ch, float* y) {
    const T* p = (const T*)a.p + ch;
    const float* w = a.conv_w + (size_t)ch * taps;
    if constexpr (TAPS > 0) {
        float wt[TAPS], x[TAPS - 1 + DC];
#pragma unroll
        for (int i = 0; i < TAPS; i++) wt[i] = w[i];
#pragma unroll
        for (int i = 0; i < TAPS - 1 + DC; i++) {
            const int j = t0 - (TAPS - 1) + i;
            x[i] = j >= n ? 0.0f : j >= 0 ? act_f(p[(size_t)j * a.ldp]) : state[(size_t)(TAPS - 1 + j) * C + ch];
        }
#pragma unroll
        for (int i = 0; i < DC; i++) {
            float s = 0.0f;
#pragma unroll
            for (int k = 0; k < TAPS; k++) s = fmaf(wt[k], x[i + k], s);
            y[i] = t0 + i < n ? conv_act<T>(s) : 0.0f;
        }
    } else {
#pragma unroll
        for (int i = 0; i < DC; i++) {
            float s = 0.0f;
            for (int k = 0; k < taps; k++) {
                const int j = t0 + i - (taps - 1) + k;
                s = fmaf(w[k], j >= n ? 0.0f : j >= 0 ? act_f(p[(size_t)j * a.ldp]) : state[(size_t)(taps - 1 + j) * C + ch], s);
            }
            y[i] = t0 + i < n ? conv_act<T>(s) : 0.0f;
        }
    }
}

constexpr int PREP_THREADS = 128;

// blockIdx.y < H: the record of head y; >= H: the value channels of head y - H.
template <class T, int R, int TAPS>
__global__ void __launch_bounds__(PREP_THREADS) k_delta_chunk_prep(const __grid_constant__ DeltaPrepArgs a, const __grid_constant__ DeltaShape s,
                                                                  const float* __restrict__ state, float* __restrict__ rec, float* __restrict__ v) {
    constexpr int DP = 32 * R;
    const int lane = threadIdx.x & 31, chunk = blockIdx.x * (PREP_THREADS / 32) + (threadIdx.x >> 5);
    const int n = a.n, H = s.heads, G = s.kv_heads, D = s.dim, E = s.vdim, C = s.channels(), t0 = chunk * DC;
    if (t0 >= n) return;
    if ((int)blockIdx.y >= H) {
        const int h = blockIdx.y - H;
        for (int i = lane; i < E; i += 32) {
            float y[DC];
            conv_run<T, TAPS>(a, state, C, s.taps, t0, n, 2 * G * D + h * E + i, y);
#pragma unroll
            for (int t = 0; t < DC; t++)
                if (t0 + t < n) v[(size_t)(t0 + t) * H * E + h * E + i] = y[t];
        }
        return;
    }
    const int h = blockIdx.y, kh = h / (H / G);
    float q[DC][R], k[DC][R], g[DC][R];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int c = Lanes<R>::channel(lane, r);
        float y[DC];
        if (c < D) conv_run<T, TAPS>(a, state, C, s.taps, t0, n, kh * D + c, y);
#pragma unroll
        for (int t = 0; t < DC; t++) q[t][r] = c < D ? y[t] : 0.0f;
        if (c < D) conv_run<T, TAPS>(a, state, C, s.taps, t0, n, (G + kh) * D + c, y);
#pragma unroll
        for (int t = 0; t < DC; t++) k[t][r] = c < D ? y[t] : 0.0f;
    }
    const float rate = expf(a.A_log[h]);
    float x[2 * DC];
#pragma unroll
    for (int t = 0; t < DC; t++) {
        x[t] = x[DC + t] = 0.0f;
#pragma unroll
        for (int r = 0; r < R; r++) {
            x[t] = fmaf(q[t][r], q[t][r], x[t]);
            x[DC + t] = fmaf(k[t][r], k[t][r], x[DC + t]);
        }
    }
    // lane 2t: 1 / |q_t| dim^(1/2), lane 2 (DC + t): 1 / |k_t|
    const float unit = (lane < 16 ? 1.0f / sqrtf((float)D) : 1.0f) / sqrtf(sum16(x, lane) + 1e-6f);
    const int my_t = (lane >> 1) & 7;
    const float beta = t0 + my_t < n ? sigmoid_f(act_f(((const T*)a.p)[(size_t)(t0 + my_t) * a.ldp + a.off_b + h])) : 0.0f;
#pragma unroll
    for (int t = 0; t < DC; t++) {
        const float qs = __shfl_sync(0xffffffffu, unit, 2 * t), ks = __shfl_sync(0xffffffffu, unit, 2 * (DC + t));
#pragma unroll
        for (int r = 0; r < R; r++) {
            q[t][r] *= qs;
            k[t][r] *= ks;
            const int c = Lanes<R>::channel(lane, r);
            g[t][r] = 1.0f;
            if (t0 + t < n && c < D) {
                const float z = a.a[(size_t)(t0 + t) * a.lda + h * D + c] + a.dt_bias[h * D + c];
                g[t][r] = expf(-rate * (fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)))));
            }
        }
    }
    float* o = rec + ((size_t)h * ((n + DC - 1) / DC) + chunk) * rec_floats(DP);
    // beta_i k_i . D(j,i) k_j (stored by columns j) and q_i . D(j,i) k_j (by rows i), zero where token i does not see token j
    float* ab = o + (3 * DC + 1) * DP;
#pragma unroll
    for (int j = 0; j < DC; j++) {
        float w[R];
#pragma unroll
        for (int r = 0; r < R; r++) w[r] = k[j][r];
#pragma unroll
        for (int i = 0; i < DC; i++) {
            x[i] = x[DC + i] = 0.0f;
            if (i < j) continue;
#pragma unroll
            for (int r = 0; r < R; r++) {
                if (i > j) {
                    w[r] *= g[i][r];
                    x[i] = fmaf(k[i][r], w[r], x[i]);
                }
                x[DC + i] = fmaf(q[i][r], w[r], x[DC + i]);
            }
        }
        const float sum = sum16(x, lane) * (lane < 16 ? beta : 1.0f);
        if ((lane & 1) == 0) ab[lane < 16 ? j * DC + my_t : DC * DC + my_t * DC + j] = sum;
        Lanes<R>::store(o + (2 * DC + j) * DP, lane, w);  // D(j,DC) k_j
    }
    if (lane < 16 && (lane & 1) == 0) ab[2 * DC * DC + my_t] = beta;
    float cum[R];
#pragma unroll
    for (int r = 0; r < R; r++) cum[r] = 1.0f;
#pragma unroll
    for (int t = 0; t < DC; t++) {
        float ck[R], cq[R];
#pragma unroll
        for (int r = 0; r < R; r++) {
            cum[r] *= g[t][r];
            ck[r] = cum[r] * k[t][r];
            cq[r] = cum[r] * q[t][r];
        }
        Lanes<R>::store(o + t * DP, lane, ck);
        Lanes<R>::store(o + (DC + t) * DP, lane, cq);
    }
    Lanes<R>::store(o + 3 * DC * DP, lane, cum);
}

__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr int SCAN_WARPS = 4, SCAN_RING = 3;

// NC = 4 value channels per warp; lane = 4 * token + channel after the transposing sums.
template <int R>
__global__ void __launch_bounds__(SCAN_WARPS * 32) k_delta_chunk_scan(int n, const __grid_constant__ DeltaShape s, float* __restrict__ state_all,
                                                                     const float* __restrict__ rec, const float* __restrict__ v, float* __restrict__ out) {
    constexpr int DP = 32 * R, REC = rec_floats(DP), NC = 4, COLS = NC * SCAN_WARPS, SLOT = REC + DC * COLS;
    static_assert(DC == 8 && DC * NC == 32 && REC % 4 == 0, "one (token, channel) pair per lane");
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(16) float u_sh[SCAN_WARPS][DC][NC];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, H = s.heads, E = s.vdim;
    const int c0 = blockIdx.x * COLS, my_c = lane & 3, my_t = lane >> 2;
    const int chunks = (n + DC - 1) / DC;
    const float* hrec = rec + (size_t)h * chunks * REC;
    float S[NC][R];
    float* st[NC];
#pragma unroll
    for (int c = 0; c < NC; c++) {
        st[c] = state_all + ((size_t)h * E + min(c0 + warp * NC + c, E - 1)) * DP;
        Lanes<R>::load(st[c], lane, S[c]);
    }
    auto stage = [&](int ch) {
        if (ch < chunks) {
            float* dst = sm + (ch % SCAN_RING) * SLOT;
            const float* src = hrec + (size_t)ch * REC;
            for (int i = tid; i < REC / 4; i += SCAN_WARPS * 32) cp16(dst + 4 * i, src + 4 * i);
            for (int i = tid; i < DC * COLS; i += SCAN_WARPS * 32) {
                const int t = ch * DC + i / COLS, c = c0 + i % COLS;
                if (t < n && c < E) cp4(dst + REC + i, v + (size_t)t * H * E + h * E + c);
                else dst[REC + i] = 0.0f;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0);
    stage(1);
    for (int ch = 0; ch < chunks; ch++) {
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();  // chunk ch has landed, and everyone is past chunk ch - 1
        stage(ch + 2);
        const float* rc = sm + (ch % SCAN_RING) * SLOT;
        float x[2 * DC * NC];  // [k | q][token][channel], partial sums over this lane's key channels
#pragma unroll
        for (int t = 0; t < 2 * DC; t++) {
            float w[R];
            Lanes<R>::load(rc + t * DP, lane, w);
#pragma unroll
            for (int c = 0; c < NC; c++) {
                float a = 0.0f;
#pragma unroll
                for (int r = 0; r < R; r++) a = fmaf(S[c][r], w[r], a);
                x[t * NC + c] = a;
            }
        }
        float *xk = x, *xq = x + DC * NC;
        halve<32, 16>(xk, lane); halve<32, 16>(xq, lane);
        halve<16, 8>(xk, lane);  halve<16, 8>(xq, lane);
        halve<8, 4>(xk, lane);   halve<8, 4>(xq, lane);
        halve<4, 2>(xk, lane);   halve<4, 2>(xq, lane);
        halve<2, 1>(xk, lane);   halve<2, 1>(xq, lane);
        const float* A = rc + (3 * DC + 1) * DP;
        const float* B = A + DC * DC;
        const float rhs = A[2 * DC * DC + my_t] * (rc[REC + my_t * COLS + warp * NC + my_c] - xk[0]);
        float u[DC];
#pragma unroll
        for (int t = 0; t < DC; t++) u[t] = __shfl_sync(0xffffffffu, rhs, t * 4 + my_c);
#pragma unroll
        for (int t = 1; t < DC; t++)
#pragma unroll
            for (int j = 0; j < t; j++) u[t] = fmaf(-A[j * DC + t], u[j], u[t]);
        float o = xq[0], mine = u[0];
#pragma unroll
        for (int j = 0; j < DC; j++) {
            o = fmaf(B[my_t * DC + j], u[j], o);
            mine = my_t == j ? u[j] : mine;
        }
        const int tok = ch * DC + my_t, col = c0 + warp * NC + my_c;
        if (tok < n && col < E) out[(size_t)tok * H * E + h * E + col] = o;
        u_sh[warp][my_t][my_c] = mine;
        __syncwarp();
        float w[R];
        Lanes<R>::load(rc + 3 * DC * DP, lane, w);
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int r = 0; r < R; r++) S[c][r] *= w[r];
#pragma unroll
        for (int j = 0; j < DC; j++) {
            Lanes<R>::load(rc + (2 * DC + j) * DP, lane, w);
            const float4 uj = *reinterpret_cast<const float4*>(u_sh[warp][j]);
            const float ua[NC] = {uj.x, uj.y, uj.z, uj.w};
#pragma unroll
            for (int c = 0; c < NC; c++)
#pragma unroll
                for (int r = 0; r < R; r++) S[c][r] = fmaf(w[r], ua[c], S[c][r]);
        }
        __syncwarp();
    }
#pragma unroll
    for (int c = 0; c < NC; c++)
        if (c0 + warp * NC + c < E) Lanes<R>::store(st[c], lane, S[c]);
}

template <class T, int R>
void prep_go(cudaStream_t st, const DeltaPrepArgs& a, const DeltaShape& s, const float* state, const DeltaWork& w) {
    const dim3 grid(((a.n + DC - 1) / DC + PREP_THREADS / 32 - 1) / (PREP_THREADS / 32), 2 * s.heads);
    switch (s.taps) {
        case 2: k_delta_chunk_prep<T, R, 2><<<grid, PREP_THREADS, 0, st>>>(a, s, state, w.rec, w.v); break;
        case 3: k_delta_chunk_prep<T, R, 3><<<grid, PREP_THREADS, 0, st>>>(a, s, state, w.rec, w.v); break;
        case 4: k_delta_chunk_prep<T, R, 4><<<grid, PREP_THREADS, 0, st>>>(a, s, state, w.rec, w.v); break;
        default: k_delta_chunk_prep<T, R, 0><<<grid, PREP_THREADS, 0, st>>>(a, s, state, w.rec, w.v);
    }
}

template <int R>
void chunk_go(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w, bool prep) {
    g_kernel_launches++;
    if (prep) {
        if (bf16) prep_go<__nv_bfloat16, R>(st, a, s, (const float*)rs.s1, w);
        else prep_go<float, R>(st, a, s, (const float*)rs.s1, w);
        return;
    }
    const size_t smem = (size_t)SCAN_RING * (rec_floats(32 * R) + DC * 4 * SCAN_WARPS) * 4;
    if (smem > 48 * 1024) cudaFuncSetAttribute(k_delta_chunk_scan<R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    k_delta_chunk_scan<R><<<dim3((s.vdim + 4 * SCAN_WARPS - 1) / (4 * SCAN_WARPS), s.heads), SCAN_WARPS * 32, smem, st>>>(a.n, s, (float*)rs.s0, w.rec, w.v, w.o);
}

void chunk_any(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w, bool prep) {
    switch (s.dimp() / 32) {
        case 1: return chunk_go<1>(st, bf16, a, s, rs, w, prep);
        case 2: return chunk_go<2>(st, bf16, a, s, rs, w, prep);
        case 3: return chunk_go<3>(st, bf16, a, s, rs, w, prep);
        case 4: return chunk_go<4>(st, bf16, a, s, rs, w, prep);
        case 5: return chunk_go<5>(st, bf16, a, s, rs, w, prep);
        case 6: return chunk_go<6>(st, bf16, a, s, rs, w, prep);
        case 7: return chunk_go<7>(st, bf16, a, s, rs, w, prep);
        default: return chunk_go<8>(st, bf16, a, s, rs, w, prep);
    }
}

}  // namespace

size_t delta_record_floats(const DeltaShape& s, int n) { return (size_t)s.heads * ((n + DC - 1) / DC) * rec_floats(s.dimp()); }

void launch_delta_chunk_prep(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w) {
    chunk_any(st, bf16, a, s, rs, w, true);
}

void launch_delta_chunk_scan(cudaStream_t st, int n, const DeltaShape& s, const RowState& rs, const DeltaWork& w) {
    DeltaPrepArgs a;
    a.n = n;
    chunk_any(st, true, a, s, rs, w, false);
}

}  // namespace wick
