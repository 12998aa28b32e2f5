// One residual stream with norms before and after every sublayer (launchers' header: ResidualArgs): the previous sublayer's
// output is normalised and added, and the next sublayer's input normalised, in one pass over the token; also the embedding
// rows, the [x | x0] rows in front of a repeated group of layers, rows gathered for experts and the average over their outputs.
// HBM-bound: 8 W bytes of x, 4 W per row of y, 2 W or 4 W per row of h.
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

constexpr int RN_THREADS = 256;  // of the form for any width

template <int TH>
__device__ __forceinline__ float block_sum(float v, float* red, int tid) {
    v = warp_sum(v);
    if ((tid & 31) == 0) red[tid >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < TH / 32; i++) t += red[i];
    return t;
}

template <class T>
__device__ __forceinline__ void put4(T* p, const float4& q) {
    if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(q.x, q.y), hi = __floats2bfloat162_rn(q.z, q.w);
        uint2 o;
        o.x = *reinterpret_cast<const uint32_t*>(&lo);
        o.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = o;
    } else {
        *reinterpret_cast<float4*>(p) = q;
    }
}

// TH threads.  NV > 0: NV groups of four coordinates per thread in registers (W a multiple of 4, at most 4 * NV * TH);
// NV == 0: any W, one coordinate at a time through shared memory.
template <class T, int NV, int TH>
__global__ void __launch_bounds__(TH) k_residual_norm(const __grid_constant__ ResidualArgs a) {
    extern __shared__ float row_sh[];  // NV == 0: [W]
    __shared__ float red[2][TH / 32];
    const int tid = threadIdx.x, W = a.W, row = blockIdx.x;
    constexpr int N4 = NV > 0 ? NV : 1;
    constexpr bool EARLY = NV == 1;  // weights are readable before the kernel in front has finished; otherwise registers count more
    const float* post_row = a.post ? a.post : a.shift;
    float4 early_gain = {}, early_post = {};
    if (EARLY && tid * 4 < W) {
        if (a.gain) early_gain = *reinterpret_cast<const float4*>(a.gain + tid * 4);
        if (post_row) early_post = *reinterpret_cast<const float4*>(post_row + tid * 4);
    }
    auto gain_at = [&](int c) { return EARLY ? early_gain : __ldg(reinterpret_cast<const float4*>(a.gain + c)); };
    auto post_at = [&](int c) { return EARLY ? early_post : __ldg(reinterpret_cast<const float4*>(post_row + c)); };
    pdl_launch_next();
    pdl_wait();
    const int src = a.rows ? a.rows[row] : row;
    float* x = a.x + (size_t)src * W;
    const __nv_bfloat16* e = a.embed && (a.init || !a.gain) ? a.embed + (size_t)(a.tokens ? a.tokens[src] : a.ctl->token) * a.ld_embed : nullptr;
    const float* fr = a.frames ? a.frames + (size_t)src * W : nullptr;
    auto start = [&](int c) { return e ? __bfloat162float(e[c]) : fr[c]; };
    auto y_row = [&](int p) { return a.y + (size_t)(a.y_rows ? a.y_rows[src * a.y_parts + p] : src * a.y_parts + p) * a.ldy; };
    const int outs = a.h_rows ? a.h_parts : 1;
    auto h_row = [&](int p) { return (T*)a.h + (size_t)(a.h_rows ? a.h_rows[row * a.h_parts + p] : row) * a.ldh; };
    if constexpr (NV > 0) {
        float4 v[N4];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < N4; i++) {
            const int c = (i * TH + tid) * 4;
            if (c < W) {
                if (a.init) v[i] = make_float4(start(c), start(c + 1), start(c + 2), start(c + 3));
                else if (a.y && !a.post) v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                else v[i] = *reinterpret_cast<const float4*>(x + c);
            }
        }
        if (a.y) {
            float4 u[N4];
            const float* y = y_row(0);
#pragma unroll
            for (int i = 0; i < N4; i++) {
                const int c = (i * TH + tid) * 4;
                if (c < W) u[i] = *reinterpret_cast<const float4*>(y + c);
            }
            for (int p = 1; p < a.y_parts; p++) {
                y = y_row(p);
#pragma unroll
                for (int i = 0; i < N4; i++) {
                    const int c = (i * TH + tid) * 4;
                    if (c < W) {
                        const float4 t = *reinterpret_cast<const float4*>(y + c);
                        u[i].x += t.x; u[i].y += t.y; u[i].z += t.z; u[i].w += t.w;
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < N4; i++) {
                const int c = (i * TH + tid) * 4;
                if (c < W) {
                    u[i].x *= a.y_scale; u[i].y *= a.y_scale; u[i].z *= a.y_scale; u[i].w *= a.y_scale;
                    ss = fmaf(u[i].x, u[i].x, fmaf(u[i].y, u[i].y, fmaf(u[i].z, u[i].z, fmaf(u[i].w, u[i].w, ss))));
                }
            }
            const float r = a.post ? 1.0f / sqrtf(block_sum<TH>(ss, red[0], tid) / (float)W + a.eps) : 1.0f;
#pragma unroll
            for (int i = 0; i < N4; i++) {
                const int c = (i * TH + tid) * 4;
                if (c < W) {
                    const float4 g = post_at(c);
                    if (a.post) {
                        v[i].x = fmaf(u[i].x * r, g.x, v[i].x); v[i].y = fmaf(u[i].y * r, g.y, v[i].y);
                        v[i].z = fmaf(u[i].z * r, g.z, v[i].z); v[i].w = fmaf(u[i].w * r, g.w, v[i].w);
                    } else {
                        v[i].x = u[i].x + g.x; v[i].y = u[i].y + g.y; v[i].z = u[i].z + g.z; v[i].w = u[i].w + g.w;
                    }
                }
            }
        }
        ss = 0.0f;
#pragma unroll
        for (int i = 0; i < N4; i++) {
            const int c = (i * TH + tid) * 4;
            if (c < W) {
                if (a.store_x && (a.y || a.init)) *reinterpret_cast<float4*>(x + c) = v[i];
                ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
            }
        }
        if (a.gain) {
            const float r = 1.0f / sqrtf(block_sum<TH>(ss, red[1], tid) / (float)W + a.eps);
#pragma unroll
            for (int i = 0; i < N4; i++) {
                const int c = (i * TH + tid) * 4;
                if (c < W) {
                    const float4 g = gain_at(c);
                    v[i].x = v[i].x * r * g.x; v[i].y = v[i].y * r * g.y; v[i].z = v[i].z * r * g.z; v[i].w = v[i].w * r * g.w;
                }
            }
        }
        for (int p = 0; p < outs; p++) {
            T* h = h_row(p);
#pragma unroll
            for (int i = 0; i < N4; i++) {
                const int c = (i * TH + tid) * 4;
                if (c < W) {
                    put4(h + c, v[i]);
                    if (!a.gain) put4(h + W + c, make_float4(start(c), start(c + 1), start(c + 2), start(c + 3)));
                    if (a.normed && row == a.n - 1) *reinterpret_cast<float4*>(a.normed + c) = v[i];
                }
            }
        }
    } else {
        float ss = 0.0f, r = 1.0f;
        if (a.y) {
            for (int c = tid; c < W; c += TH) {
                float u = 0.0f;
                for (int p = 0; p < a.y_parts; p++) u += y_row(p)[c];
                u *= a.y_scale;
                row_sh[c] = u;
                ss = fmaf(u, u, ss);
            }
            if (a.post) r = 1.0f / sqrtf(block_sum<TH>(ss, red[0], tid) / (float)W + a.eps);
        }
        ss = 0.0f;
        for (int c = tid; c < W; c += TH) {  // the coordinates this thread wrote
            float v;
            if (a.y && !a.post) v = row_sh[c] + a.shift[c];
            else {
                v = a.init ? start(c) : x[c];
                if (a.y) v = fmaf(row_sh[c] * r, a.post[c], v);
            }
            if (a.store_x && (a.y || a.init)) x[c] = v;
            row_sh[c] = v;
            ss = fmaf(v, v, ss);
        }
        r = a.gain ? 1.0f / sqrtf(block_sum<TH>(ss, red[1], tid) / (float)W + a.eps) : 1.0f;
        for (int c = tid; c < W; c += TH) {
            const float v = a.gain ? row_sh[c] * r * a.gain[c] : row_sh[c];
            for (int p = 0; p < outs; p++) {
                T* h = h_row(p);
                h[c] = f_act<T>(v);
                if (!a.gain) h[W + c] = f_act<T>(start(c));
            }
            if (a.normed && row == a.n - 1) a.normed[c] = v;
        }
    }
}

template <class T, int NV, int TH>
void residual_launch(cudaStream_t st, const ResidualArgs& a, size_t smem = 0) {
    if (smem > 40 * 1024) cudaFuncSetAttribute(k_residual_norm<T, NV, TH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_pdl(k_residual_norm<T, NV, TH>, dim3(a.n), dim3(TH), smem, st, a);
}

template <class T>
void residual_go(cudaStream_t st, const ResidualArgs& a) {
    const int fours = a.W % 4 == 0 && (!a.y || a.ldy % 4 == 0) ? a.W / 4 : 0;
    if (!fours || fours > 4096) return residual_launch<T, 0, RN_THREADS>(st, a, (size_t)a.W * 4);
    if (a.n >= 256) {  // throughput: small CTAs, four loads of x and of y in flight per thread
        if (fours <= 4 * 64) return residual_launch<T, 4, 64>(st, a);
        if (fours <= 4 * 128) return residual_launch<T, 4, 128>(st, a);
        if (fours <= 4 * 256) return residual_launch<T, 4, 256>(st, a);
    } else {           // latency: many threads
        if (fours <= 128) return residual_launch<T, 1, 128>(st, a);
        if (fours <= 256) return residual_launch<T, 1, 256>(st, a);
        if (fours <= 512) return residual_launch<T, 1, 512>(st, a);
    }
    if (fours <= 1024) return residual_launch<T, 2, 512>(st, a);
    if (fours <= 2048) return residual_launch<T, 4, 512>(st, a);
    return residual_launch<T, 8, 512>(st, a);
}

}  // namespace

void launch_residual_norm(cudaStream_t st, bool bf16, const ResidualArgs& a) {
    if (a.n <= 0) return;
    g_kernel_launches++;
    if (bf16) residual_go<__nv_bfloat16>(st, a);
    else residual_go<float>(st, a);
}

}  // namespace wick
