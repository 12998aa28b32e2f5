// The gated delta rule with one decay per head and key channel (f32 throughout, as the state is):
//     S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// for decode steps and portions of a few tokens (prompts: delta_chunk.cu).  The columns of S (value channels) do not depend on
// each other: eight lanes hold one column, 4 * R4 key channels each.  The read-out is folded into the same pass over the
// column, o = (diag(g) S)^T q + (k . q) u, so that a token costs one round of cross-lane sums.
// k_delta_prep   short causal convolutions + silu, unit q and k, k . q, decays and step sizes of consecutive tokens: one warp
//                per (token, group of channels that is normalised together).
// k_delta_scan   their recurrence; the state stays in registers, q, k, g rows are staged in shared memory with cp.async.
// k_delta_step   one decode token per row: all of it, and the gated norm, in one launch.
// k_gated_head_norm  RMS norm over the value channels of a head, weights, sigmoid gate (also after delta_chunk.cu, kernels_memory.cu).
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

// ── preparation ────────────────────────────────────────────────────────────
constexpr int PREP_WARPS = 8;
constexpr int PREP_REG = DELTA_MAX_DIM / 32;

// Convolution of channel ch at row j followed by silu.
template <class T>
__device__ __forceinline__ float conv_silu(const DeltaPrepArgs& a, const DeltaShape& s, const float* state, int j, int ch) {
    const int t = s.taps, C = s.channels();
    const float* w = a.conv_w + (size_t)ch * t;
    const T* p = (const T*)a.p;
    const float cur = act_f(p[(size_t)j * a.ldp + ch]);
    float sum = 0.0f;
    for (int i = 0; i < t - 1; i++) {
        const int src = j - (t - 1 - i);  // row of the launch; negative: kept from before
        const float v = src >= 0 ? act_f(p[(size_t)src * a.ldp + ch]) : state[(size_t)(t - 1 + src) * C + ch];
        sum = fmaf(w[i], v, sum);
    }
    return silu_f(fmaf(w[t - 1], cur, sum));
}

template <class T>
__global__ void __launch_bounds__(PREP_WARPS * 32) k_delta_prep(const __grid_constant__ DeltaPrepArgs a, const __grid_constant__ DeltaShape s,
                                                               const float* __restrict__ state, const __grid_constant__ DeltaWork w) {
    const int lane = threadIdx.x & 31;
    const int seg_n = s.kv_heads + 2 * s.heads;
    const size_t unit = (size_t)blockIdx.x * PREP_WARPS + (threadIdx.x >> 5);
    if (unit >= (size_t)a.n * seg_n) return;
    const int j = (int)(unit / seg_n), seg = (int)(unit % seg_n);
    const int G = s.kv_heads, H = s.heads, D = s.dim, E = s.vdim, DP = s.dimp();
    if (seg < G) {  // q and k of key head `seg`
        float q[PREP_REG], k[PREP_REG], qq = 0.0f, kk = 0.0f, kq = 0.0f;
#pragma unroll
        for (int r = 0; r < PREP_REG; r++) {
            const int i = r * 32 + lane;
            q[r] = k[r] = 0.0f;
            if (i < D) {
                q[r] = conv_silu<T>(a, s, state, j, seg * D + i);
                k[r] = conv_silu<T>(a, s, state, j, (G + seg) * D + i);
            }
            qq = fmaf(q[r], q[r], qq);
            kk = fmaf(k[r], k[r], kk);
        }
        const float qs = 1.0f / sqrtf((float)D) / sqrtf(warp_sum(qq) + 1e-6f), ks = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
        float* qo = w.q + ((size_t)j * G + seg) * DP;
        float* ko = w.k + ((size_t)j * G + seg) * DP;
#pragma unroll
        for (int r = 0; r < PREP_REG; r++) {
            const int i = r * 32 + lane;
            if (i < DP) {  // the padding channels are zero
                qo[i] = q[r] *= qs;
                ko[i] = k[r] *= ks;
                kq = fmaf(q[r], k[r], kq);
            }
        }
        kq = warp_sum(kq);
        if (lane == 0) w.kq[(size_t)j * G + seg] = kq;
    } else if (seg < G + H) {  // v of head h
        const int h = seg - G;
        for (int i = lane; i < E; i += 32) w.v[(size_t)j * H * E + h * E + i] = conv_silu<T>(a, s, state, j, 2 * G * D + h * E + i);
    } else {  // decays and step size of head h
        const int h = seg - G - H;
        const float rate = expf(a.A_log[h]);
        float* go = w.g + ((size_t)j * H + h) * DP;
        for (int i = lane; i < DP; i += 32) {
            float g = 1.0f;
            if (i < D) {
                const float z = a.a[(size_t)j * a.lda + h * D + i] + a.dt_bias[h * D + i];
                const float sp = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
                g = expf(-rate * sp);
            }
            go[i] = g;
        }
        if (lane == 0) w.beta[(size_t)j * H + h] = sigmoid_f(act_f(((const T*)a.p)[(size_t)j * a.ldp + a.off_b + h]));
    }
}

// The last taps - 1 inputs after n consecutive tokens of one sequence.  A channel's rows are moved in ascending order, so
// that a kept row is read before it is overwritten.
template <class T>
__global__ void __launch_bounds__(256) k_delta_conv_state(const T* __restrict__ p, int ldp, int n, int channels, int taps, float* __restrict__ state) {
    const int ch = blockIdx.x * 256 + threadIdx.x;
    if (ch >= channels) return;
    for (int r = 0; r < taps - 1; r++) {
        const int src = n - (taps - 1) + r;
        state[(size_t)r * channels + ch] = src >= 0 ? act_f(p[(size_t)src * ldp + ch]) : state[(size_t)(taps - 1 + src) * channels + ch];
    }
}

// ── recurrence ─────────────────────────────────────────────────────────────
constexpr int SCAN_THREADS = 128, SCAN_COLS = SCAN_THREADS / 8;  // value channels per CTA
constexpr int SCAN_TB = 16;                                      // tokens staged at a time

__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

__host__ __device__ constexpr int scan_tok_floats(int dp) { return 3 * dp + SCAN_COLS + 4; }  // q k g rows, v, beta, kq (+ pad)

// R4 * 4 key channels per lane: dimp = 32 * R4.  Lane l of a column's eight holds channels 32 r + 4 l .. + 3.
template <int R4>
__global__ void __launch_bounds__(SCAN_THREADS) k_delta_scan(int nt, const __grid_constant__ DeltaShape s, float* __restrict__ state_all,
                                                            const __grid_constant__ DeltaWork w) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = 32 * R4, TOK = scan_tok_floats(DP);
    const int tid = threadIdx.x, l8 = tid & 7, col = tid >> 3;
    const int h = blockIdx.y, G = s.kv_heads, H = s.heads, E = s.vdim;
    const int kh = h / (H / G), c0 = blockIdx.x * SCAN_COLS, c = c0 + col;
    float* state = state_all + ((size_t)h * E + min(c, E - 1)) * DP;
    float S[R4][4];
#pragma unroll
    for (int r = 0; r < R4; r++) {
        const float4 v = *reinterpret_cast<const float4*>(state + 32 * r + 4 * l8);
        S[r][0] = v.x; S[r][1] = v.y; S[r][2] = v.z; S[r][3] = v.w;
    }
    auto stage = [&](int t0, int buf) {  // tokens t0 .. t0 + SCAN_TB - 1 (as many as there are) into buffer `buf`
        const int cnt = min(SCAN_TB, nt - t0);
        float* dst = sm + buf * SCAN_TB * TOK;
        constexpr int V4 = DP / 4;
        for (int i = tid; i < cnt * 3 * V4; i += SCAN_THREADS) {
            const int t = i / (3 * V4), q = i % (3 * V4), which = q / V4, x = q % V4;
            const size_t row = (size_t)(t0 + t);
            const float* src = which == 0 ? w.q + (row * G + kh) * DP : which == 1 ? w.k + (row * G + kh) * DP : w.g + (row * H + h) * DP;
            cp16(dst + t * TOK + which * DP + 4 * x, src + 4 * x);
        }
        for (int i = tid; i < cnt * (SCAN_COLS + 2); i += SCAN_THREADS) {
            const int t = i / (SCAN_COLS + 2), x = i % (SCAN_COLS + 2);
            const size_t row = (size_t)(t0 + t);
            if (x < SCAN_COLS) {
                if (c0 + x < E) cp4(dst + t * TOK + 3 * DP + x, w.v + row * H * E + h * E + c0 + x);
            } else if (x == SCAN_COLS) {
                cp4(dst + t * TOK + 3 * DP + x, w.beta + row * H + h);
            } else {
                cp4(dst + t * TOK + 3 * DP + x, w.kq + row * G + kh);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    int buf = 0;
    for (int t0 = 0; t0 < nt; t0 += SCAN_TB, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the block's rows are there, and everyone has left the other buffer
        if (t0 + SCAN_TB < nt) stage(t0 + SCAN_TB, buf ^ 1);
        const int cnt = min(SCAN_TB, nt - t0);
        const float* tk = sm + buf * SCAN_TB * TOK;
#pragma unroll 2
        for (int t = 0; t < cnt; t++, tk += TOK) {
            float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
            float4 k4[R4];
#pragma unroll
            for (int r = 0; r < R4; r++) {
                const float4 q = *reinterpret_cast<const float4*>(tk + 32 * r + 4 * l8);
                k4[r] = *reinterpret_cast<const float4*>(tk + DP + 32 * r + 4 * l8);
                const float4 g = *reinterpret_cast<const float4*>(tk + 2 * DP + 32 * r + 4 * l8);
                S[r][0] *= g.x; S[r][1] *= g.y; S[r][2] *= g.z; S[r][3] *= g.w;
                r1[0] = fmaf(S[r][0], k4[r].x, r1[0]); r1[1] = fmaf(S[r][1], k4[r].y, r1[1]);
                r2[0] = fmaf(S[r][0], q.x, r2[0]);     r2[1] = fmaf(S[r][1], q.y, r2[1]);
                r1[0] = fmaf(S[r][2], k4[r].z, r1[0]); r1[1] = fmaf(S[r][3], k4[r].w, r1[1]);
                r2[0] = fmaf(S[r][2], q.z, r2[0]);     r2[1] = fmaf(S[r][3], q.w, r2[1]);
            }
            float a = r1[0] + r1[1], b = r2[0] + r2[1];
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) {
                a += __shfl_xor_sync(0xffffffffu, a, o);
                b += __shfl_xor_sync(0xffffffffu, b, o);
            }
            const float u = tk[3 * DP + SCAN_COLS] * (tk[3 * DP + col] - a);
            const float out = fmaf(tk[3 * DP + SCAN_COLS + 1], u, b);
#pragma unroll
            for (int r = 0; r < R4; r++) {
                S[r][0] = fmaf(k4[r].x, u, S[r][0]);
                S[r][1] = fmaf(k4[r].y, u, S[r][1]);
                S[r][2] = fmaf(k4[r].z, u, S[r][2]);
                S[r][3] = fmaf(k4[r].w, u, S[r][3]);
            }
            if (l8 == 0 && c < E) w.o[(size_t)(t0 + t) * H * E + h * E + c] = out;
        }
    }
    if (c < E)
#pragma unroll
        for (int r = 0; r < R4; r++)
            *reinterpret_cast<float4*>(state + 32 * r + 4 * l8) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
}

template <int R4>
void scan_go(cudaStream_t st, int n, const DeltaShape& s, const RowState& rs, const DeltaWork& w) {
    const dim3 grid((s.vdim + SCAN_COLS - 1) / SCAN_COLS, s.heads);
    const size_t smem = (size_t)2 * SCAN_TB * scan_tok_floats(32 * R4) * 4;
    if (smem > 48 * 1024) cudaFuncSetAttribute(k_delta_scan<R4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    k_delta_scan<R4><<<grid, SCAN_THREADS, smem, st>>>(n, s, (float*)rs.s0, w);
}

// ── one decode token per row ───────────────────────────────────────────────
// A CTA owns a key head of a row and the heads that use it: convolutions and decays (a thread per channel), unit q and k (one
// warp), the state's columns (eight lanes each, as above), the gated norm (a warp per head).
template <class T, int R4, int TAPS>
__global__ void __launch_bounds__(1024) k_delta_step(const __grid_constant__ DeltaPrepArgs a, const __grid_constant__ DeltaShape s,
                                                    const __grid_constant__ RowState rs, const float* __restrict__ norm, const float* __restrict__ gate,
                                                    int ldg, T* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = 32 * R4;
    const int G = s.kv_heads, H = s.heads, D = s.dim, E = s.vdim, rep = H / G, kh = blockIdx.x, j = blockIdx.y, h0 = kh * rep;
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, C = s.channels();
    const int taps = TAPS > 0 ? TAPS : s.taps;
    float *q = sm, *k = q + DP, *g = k + DP, *v = g + rep * DP, *o = v + rep * E, *beta = o + rep * E, *kq = beta + rep;
    pdl_launch_next();
    pdl_wait();
    float* state = (float*)rs.st0(j) + (size_t)h0 * E * DP;
    float* cs = (float*)rs.st1(j);
    const T* p = (const T*)a.p + (size_t)j * a.ldp;
    const int convs = 2 * DP + rep * E;
    for (int i = tid; i < convs + rep * DP + rep; i += nt) {
        if (i < convs) {
            int ch = -1;
            if (i < DP) ch = i < D ? kh * D + i : -1;
            else if (i < 2 * DP) ch = i - DP < D ? (G + kh) * D + i - DP : -1;
            else ch = 2 * G * D + h0 * E + i - 2 * DP;
            float y = 0.0f;
            if (ch >= 0) {
                const float* w = a.conv_w + (size_t)ch * taps;
                const float cur = act_f(p[ch]);
                if constexpr (TAPS > 0) {
                    float x[TAPS], wt[TAPS];
#pragma unroll
                    for (int t = 0; t < TAPS; t++) {
                        x[t] = t < TAPS - 1 ? cs[(size_t)t * C + ch] : cur;
                        wt[t] = w[t];
                    }
#pragma unroll
                    for (int t = 0; t < TAPS; t++) y = fmaf(wt[t], x[t], y);
#pragma unroll
                    for (int t = 0; t < TAPS - 1; t++) cs[(size_t)t * C + ch] = x[t + 1];
                } else {
                    for (int t = 0; t < taps; t++) {
                        const float x = t < taps - 1 ? cs[(size_t)t * C + ch] : cur;
                        y = fmaf(w[t], x, y);
                        if (t > 0) cs[(size_t)(t - 1) * C + ch] = x;
                    }
                }
                y = silu_f(y);
            }
            (i < DP ? q[i] : i < 2 * DP ? k[i - DP] : v[i - 2 * DP]) = y;
        } else if (i < convs + rep * DP) {
            const int r = (i - convs) / DP, c = (i - convs) % DP, h = h0 + r;
            float x = 1.0f;
            if (c < D) {
                const float z = a.a[(size_t)j * a.lda + h * D + c] + a.dt_bias[h * D + c];
                x = expf(-expf(a.A_log[h]) * (fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)))));
            }
            g[r * DP + c] = x;
        } else {
            const int r = i - convs - rep * DP;
            beta[r] = sigmoid_f(act_f(p[a.off_b + h0 + r]));
        }
    }
    __syncthreads();
    if (warp == 0) {
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
        for (int r = 0; r < R4; r++) {
            const float a0 = q[r * 32 + lane], b0 = k[r * 32 + lane];
            qq = fmaf(a0, a0, qq);
            kk = fmaf(b0, b0, kk);
            qk = fmaf(a0, b0, qk);
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        qk = warp_sum(qk);
        const float qs = 1.0f / sqrtf((float)D) / sqrtf(qq + 1e-6f), ks = 1.0f / sqrtf(kk + 1e-6f);
#pragma unroll
        for (int r = 0; r < R4; r++) {
            q[r * 32 + lane] *= qs;
            k[r * 32 + lane] *= ks;
        }
        if (lane == 0) *kq = qk * qs * ks;
    }
    __syncthreads();
    const int l8 = tid & 7, cols = rep * E;
    for (int c0 = 0; c0 < cols; c0 += nt / 8) {
        const int c = c0 + (tid >> 3), r_ = min(c, cols - 1) / E;
        float* sp = state + (size_t)min(c, cols - 1) * DP;
        float S[R4][4], r1 = 0.0f, r2 = 0.0f;
        float4 k4[R4];
#pragma unroll
        for (int r = 0; r < R4; r++) {
            const float4 x = *reinterpret_cast<const float4*>(sp + 32 * r + 4 * l8);
            S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
        }
#pragma unroll
        for (int r = 0; r < R4; r++) {
            const float4 q4 = *reinterpret_cast<const float4*>(q + 32 * r + 4 * l8), g4 = *reinterpret_cast<const float4*>(g + r_ * DP + 32 * r + 4 * l8);
            k4[r] = *reinterpret_cast<const float4*>(k + 32 * r + 4 * l8);
            S[r][0] *= g4.x; S[r][1] *= g4.y; S[r][2] *= g4.z; S[r][3] *= g4.w;
            r1 = fmaf(S[r][0], k4[r].x, r1); r2 = fmaf(S[r][0], q4.x, r2);
            r1 = fmaf(S[r][1], k4[r].y, r1); r2 = fmaf(S[r][1], q4.y, r2);
            r1 = fmaf(S[r][2], k4[r].z, r1); r2 = fmaf(S[r][2], q4.z, r2);
            r1 = fmaf(S[r][3], k4[r].w, r1); r2 = fmaf(S[r][3], q4.w, r2);
        }
#pragma unroll
        for (int x = 4; x > 0; x >>= 1) {
            r1 += __shfl_xor_sync(0xffffffffu, r1, x);
            r2 += __shfl_xor_sync(0xffffffffu, r2, x);
        }
        if (c < cols) {
            const float u = beta[r_] * (v[c] - r1);
            if (l8 == 0) o[c] = fmaf(*kq, u, r2);
#pragma unroll
            for (int r = 0; r < R4; r++)
                *reinterpret_cast<float4*>(sp + 32 * r + 4 * l8) = make_float4(fmaf(k4[r].x, u, S[r][0]), fmaf(k4[r].y, u, S[r][1]),
                                                                              fmaf(k4[r].z, u, S[r][2]), fmaf(k4[r].w, u, S[r][3]));
        }
    }
    __syncthreads();
    for (int r = warp; r < rep; r += nt / 32) {
        float ss = 0.0f;
        for (int i = lane; i < E; i += 32) ss = fmaf(o[r * E + i], o[r * E + i], ss);
        const float rr = 1.0f / sqrtf(warp_sum(ss) / (float)E + s.eps);
        for (int i = lane; i < E; i += 32)
            out[(size_t)j * ldo + (h0 + r) * E + i] = f_act<T>(o[r * E + i] * rr * norm[i] * sigmoid_f(gate[(size_t)j * ldg + (h0 + r) * E + i]));
    }
}

template <class T, int R4>
void step_go(cudaStream_t st, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const float* norm, const float* gate, int ldg, T* out,
             int ldo) {
    const int rep = s.heads / s.kv_heads, cols = rep * s.vdim;
    const dim3 grid(s.kv_heads, a.n), block((unsigned)std::min(1024, std::max(128, round_up(cols * 8, 128))));
    const size_t smem = ((size_t)(2 + rep) * 32 * R4 + 2 * cols + rep + 4) * 4;
    auto k = s.taps == 4 ? k_delta_step<T, R4, 4> : k_delta_step<T, R4, 0>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_pdl(k, grid, block, smem, st, a, s, rs, norm, gate, ldg, out, ldo);
}

template <class T>
void step_any(cudaStream_t st, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const float* norm, const float* gate, int ldg, T* out,
              int ldo) {
    switch (s.dimp() / 32) {
        case 1: return step_go<T, 1>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 2: return step_go<T, 2>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 3: return step_go<T, 3>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 4: return step_go<T, 4>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 5: return step_go<T, 5>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 6: return step_go<T, 6>(st, a, s, rs, norm, gate, ldg, out, ldo);
        case 7: return step_go<T, 7>(st, a, s, rs, norm, gate, ldg, out, ldo);
        default: return step_go<T, 8>(st, a, s, rs, norm, gate, ldg, out, ldo);
    }
}

// ── output ─────────────────────────────────────────────────────────────────
template <class T, class TG>
__global__ void __launch_bounds__(256) k_gated_head_norm(int n, int H, int E, float eps, const float* __restrict__ o, const float* __restrict__ norm, int norm_step,
                                                         const TG* __restrict__ gate, int ldg, T* __restrict__ out, int ldo) {
    const int lane = threadIdx.x & 31;
    const size_t unit = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (unit >= (size_t)n * H) return;
    const int j = (int)(unit / H), h = (int)(unit % H);
    const float* src = o + (size_t)j * H * E + h * E;
    float ss = 0.0f;
    for (int i = lane; i < E; i += 32) ss = fmaf(src[i], src[i], ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)E + eps);
    for (int i = lane; i < E; i += 32)
        out[(size_t)j * ldo + h * E + i] = f_act<T>(src[i] * r * norm[h * norm_step + i] * sigmoid_f(act_f(gate[(size_t)j * ldg + h * E + i])));
}

}  // namespace

static bool use_chunks(int n, const DeltaWork& w) { return n >= DELTA_CHUNK_MIN_ROWS && w.rec; }

void launch_delta_prep(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w) {
    if (a.n <= 0) return;
    const size_t units = (size_t)a.n * (s.kv_heads + 2 * s.heads);
    const unsigned grid = (unsigned)((units + PREP_WARPS - 1) / PREP_WARPS);
    if (use_chunks(a.n, w)) launch_delta_chunk_prep(st, bf16, a, s, rs, w);
    else {
        g_kernel_launches++;
        if (bf16) k_delta_prep<__nv_bfloat16><<<grid, PREP_WARPS * 32, 0, st>>>(a, s, (const float*)rs.s1, w);
        else k_delta_prep<float><<<grid, PREP_WARPS * 32, 0, st>>>(a, s, (const float*)rs.s1, w);
    }
    if (s.taps > 1) {
        const int C = s.channels();
        g_kernel_launches++;
        if (bf16) k_delta_conv_state<__nv_bfloat16><<<(C + 255) / 256, 256, 0, st>>>((const __nv_bfloat16*)a.p, a.ldp, a.n, C, s.taps, (float*)rs.s1);
        else k_delta_conv_state<float><<<(C + 255) / 256, 256, 0, st>>>((const float*)a.p, a.ldp, a.n, C, s.taps, (float*)rs.s1);
    }
}

void launch_delta_scan(cudaStream_t st, int n, const DeltaShape& s, const RowState& rs, const DeltaWork& w) {
    if (n <= 0) return;
    if (use_chunks(n, w)) return launch_delta_chunk_scan(st, n, s, rs, w);
    g_kernel_launches++;
    switch (s.dimp() / 32) {
        case 1: return scan_go<1>(st, n, s, rs, w);
        case 2: return scan_go<2>(st, n, s, rs, w);
        case 3: return scan_go<3>(st, n, s, rs, w);
        case 4: return scan_go<4>(st, n, s, rs, w);
        case 5: return scan_go<5>(st, n, s, rs, w);
        case 6: return scan_go<6>(st, n, s, rs, w);
        case 7: return scan_go<7>(st, n, s, rs, w);
        default: return scan_go<8>(st, n, s, rs, w);
    }
}

void launch_delta_step(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const float* norm,
                       const float* gate, int ldg, void* out, int ldo) {
    if (a.n <= 0) return;
    g_kernel_launches++;
    if (bf16) step_any(st, a, s, rs, norm, gate, ldg, (__nv_bfloat16*)out, ldo);
    else step_any(st, a, s, rs, norm, gate, ldg, (float*)out, ldo);
}

void launch_gated_head_norm(cudaStream_t st, bool bf16, int n, int H, int E, float eps, const float* o, const float* norm, int norm_step,
                            const void* gate, bool gate_f32, int ldg, void* out, int ldo) {
    if (n <= 0) return;
    const unsigned grid = (unsigned)(((size_t)n * H + 7) / 8);
    using B = __nv_bfloat16;
    g_kernel_launches++;
    if (!bf16) k_gated_head_norm<float, float><<<grid, 256, 0, st>>>(n, H, E, eps, o, norm, norm_step, (const float*)gate, ldg, (float*)out, ldo);
    else if (gate_f32) k_gated_head_norm<B, float><<<grid, 256, 0, st>>>(n, H, E, eps, o, norm, norm_step, (const float*)gate, ldg, (B*)out, ldo);
    else k_gated_head_norm<B, B><<<grid, 256, 0, st>>>(n, H, E, eps, o, norm, norm_step, (const B*)gate, ldg, (B*)out, ldo);
}

}  // namespace wick
