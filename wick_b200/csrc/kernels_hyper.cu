// Hyper-connections: several residual streams per token, read as a weighted sum before every sublayer and rewritten as a
// small matrix product plus the sublayer's output after it.  The write of one sublayer, the read of the next and the RMS
// norm in front of it touch the same S * W values of a token, so they are one kernel: the streams are read and written
// once per sublayer, in f32.  HBM-bound: 8 S W + 4 W + (2 or 4) W bytes per token.
#include "hybrid_kernels.cuh"

namespace wick {

constexpr int HYPER_THREADS = 256;

// S streams (0: any number up to HYPER_MAX_STREAMS), V consecutive coordinates per thread and step.
template <class T, int S_, int V>
__global__ void __launch_bounds__(HYPER_THREADS) k_hyper_norm(HyperArgs a) {
    extern __shared__ float u_sh[];  // [W]
    __shared__ float red[HYPER_THREADS / 32];
    __shared__ float prm[HYPER_MAX_STREAMS * (HYPER_MAX_STREAMS + 2)];
    constexpr int SM = S_ ? S_ : HYPER_MAX_STREAMS;
    const int S = S_ ? S_ : a.S, W = a.W, tid = threadIdx.x;
    const int row = blockIdx.x;
    const bool init = a.embed != nullptr || a.frames != nullptr;
    pdl_launch_next();
    float* mix = prm;
    float* w_out = prm + S * S;
    float* w_in = w_out + S;
    for (int i = tid; i < S * S + 2 * S; i += HYPER_THREADS)
        prm[i] = i < S * S ? (a.y ? a.mix[i] : 0.0f) : i < S * S + S ? (a.y ? a.out[i - S * S] : 0.0f) : (a.in ? a.in[i - S * S - S] : 1.0f);
    pdl_wait();
    const int src = a.rows ? a.rows[row] : row;
    __syncthreads();
    float* x = a.x + (size_t)src * S * W;
    const __nv_bfloat16* e = nullptr;
    const float* fr = nullptr;
    if (a.embed) e = a.embed + (size_t)(a.tokens ? a.tokens[src] : a.ctl->token) * a.ld_embed;
    else if (a.frames) fr = a.frames + (size_t)src * W;
    float ss = 0.0f;
    for (int c = tid * V; c < W; c += HYPER_THREADS * V) {
        float xs[SM][V], u[V];
        if (init) {
#pragma unroll
            for (int v = 0; v < V; v++) {
                const float val = e ? __bfloat162float(e[c + v]) * a.embed_scale : fr[c + v];
#pragma unroll
                for (int s = 0; s < SM; s++) xs[s][v] = val;
            }
        } else {
#pragma unroll
            for (int s = 0; s < SM; s++)
                if (s < S) {
                    if constexpr (V == 4) {
                        const float4 t = *reinterpret_cast<const float4*>(x + (size_t)s * W + c);
                        xs[s][0] = t.x; xs[s][1] = t.y; xs[s][2] = t.z; xs[s][3] = t.w;
                    } else {
                        xs[s][0] = x[(size_t)s * W + c];
                    }
                }
        }
        if (a.y) {
            float y[V], nx[SM][V];
            if constexpr (V == 4) {
                const float4 t = *reinterpret_cast<const float4*>(a.y + (size_t)src * a.ldy + c);
                y[0] = t.x; y[1] = t.y; y[2] = t.z; y[3] = t.w;
            } else {
                y[0] = a.y[(size_t)src * a.ldy + c];
            }
#pragma unroll
            for (int t = 0; t < SM; t++)
                if (t < S) {
#pragma unroll
                    for (int v = 0; v < V; v++) nx[t][v] = w_out[t] * y[v];
#pragma unroll
                    for (int s = 0; s < SM; s++)
                        if (s < S) {
                            const float m = mix[s * S + t];
#pragma unroll
                            for (int v = 0; v < V; v++) nx[t][v] = fmaf(m, xs[s][v], nx[t][v]);
                        }
                }
#pragma unroll
            for (int t = 0; t < SM; t++)
#pragma unroll
                for (int v = 0; v < V; v++) xs[t][v] = nx[t][v];
        }
        if (a.store_x && (a.y || init)) {
#pragma unroll
            for (int s = 0; s < SM; s++)
                if (s < S) {
                    if constexpr (V == 4) *reinterpret_cast<float4*>(x + (size_t)s * W + c) = make_float4(xs[s][0], xs[s][1], xs[s][2], xs[s][3]);
                    else x[(size_t)s * W + c] = xs[s][0];
                }
        }
#pragma unroll
        for (int v = 0; v < V; v++) {
            u[v] = 0.0f;
#pragma unroll
            for (int s = 0; s < SM; s++)
                if (s < S) u[v] = fmaf(w_in[s], xs[s][v], u[v]);
            ss = fmaf(u[v], u[v], ss);
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(u_sh + c) = make_float4(u[0], u[1], u[2], u[3]);
        else u_sh[c] = u[0];
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < HYPER_THREADS / 32; i++) t += red[i];
    const float r = *a.gain / sqrtf(t / (float)W + a.eps);
    T* h = (T*)a.h + (size_t)row * a.ldh;
    for (int c = tid * V; c < W; c += HYPER_THREADS * V) {  // the coordinates this thread wrote
        if constexpr (V == 4 && sizeof(T) == 2) {
            const float4 q = *reinterpret_cast<const float4*>(u_sh + c);
            const __nv_bfloat162 lo = __floats2bfloat162_rn(q.x * r, q.y * r), hi = __floats2bfloat162_rn(q.z * r, q.w * r);
            uint2 o;
            o.x = *reinterpret_cast<const uint32_t*>(&lo);
            o.y = *reinterpret_cast<const uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(h + c) = o;
        } else {
#pragma unroll
            for (int v = 0; v < V; v++) h[c + v] = f_act<T>(u_sh[c + v] * r);
        }
        if (a.normed && row == a.n - 1)
#pragma unroll
            for (int v = 0; v < V; v++) a.normed[c + v] = u_sh[c + v] * r;
    }
}

template <class T, int S>
static void hyper_v(cudaStream_t st, const HyperArgs& a) {
    const size_t smem = (size_t)round_up(a.W, 4) * 4;
    if (a.W % 4 == 0 && (!a.y || a.ldy % 4 == 0)) {
        if (smem > 40 * 1024) cudaFuncSetAttribute(k_hyper_norm<T, S, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_pdl(k_hyper_norm<T, S, 4>, dim3(a.n), dim3(HYPER_THREADS), smem, st, a);
    } else {
        if (smem > 40 * 1024) cudaFuncSetAttribute(k_hyper_norm<T, S, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_pdl(k_hyper_norm<T, S, 1>, dim3(a.n), dim3(HYPER_THREADS), smem, st, a);
    }
}

template <class T>
static void hyper_s(cudaStream_t st, const HyperArgs& a) {
    switch (a.S) {
        case 1: return hyper_v<T, 1>(st, a);
        case 2: return hyper_v<T, 2>(st, a);
        case 3: return hyper_v<T, 3>(st, a);
        case 4: return hyper_v<T, 4>(st, a);
        case 8: return hyper_v<T, 8>(st, a);
        default: return hyper_v<T, 0>(st, a);
    }
}

void launch_hyper_norm(cudaStream_t st, bool bf16, const HyperArgs& a) {
    if (a.n <= 0) return;
    g_kernel_launches++;
    if (bf16) hyper_s<__nv_bfloat16>(st, a);
    else hyper_s<float>(st, a);
}

}  // namespace wick
