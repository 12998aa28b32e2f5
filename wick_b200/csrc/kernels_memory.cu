// The matrix memory with exponential gates (launchers' header: MemoryShape), in f32 on the CUDA cores:
//     m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  z likewise with v = 1
//     o  = S^T q / (max(|z . q|, exp(-m')) + 1e-6)
//
// A prompt portion goes MEMORY_CHUNK tokens at a time.  With b_t the sum of f from the chunk's start to t and m_0, S_0 at its
// start, unrolling gives
//     m_t = b_t + max(m_0, max_{j <= t} (i_j - b_j))
//     S_t = exp(b_t + m_0 - m_t) S_0 + sum_{j <= t} exp(b_t - b_j + i_j - m_t) k_j v_j^T
// so the chunks' sums do not wait for each other and only the m's and one pass over the states are sequential:
//   k_memory_gates   per head: i, f, the m's, and the weights above.  Sums and differences of log gates are taken in f64: they
//                    cancel, and the weights are exponentials of what is left.
//   k_memory_states  per (chunk, head, tile of value channels): sum_j w_j k_j v_j^T
//   k_memory_scan    per state element: states at the chunks' starts, and the final one
//   k_memory_out     per (chunk, head, tile of value channels): q S_0 and the chunk's own (q k^T) v, divided
// (bfloat16 models: memory_tc.cu does the last three on the tensor cores.)
// The row of z rides along as one more value channel that is 1 for every token.
// k_memory_step is the decode form: everything for one token of a (row, head), with the gated norm.
#include <cooperative_groups.h>

#include <type_traits>

#include "memory_kernels.cuh"

namespace wick {

namespace cg = cooperative_groups;

namespace {

constexpr int MC = MEMORY_CHUNK;

struct Gates {
    float i, f;
};
__device__ __forceinline__ Gates memory_gates(const MemoryShape& s, const float* row, int h) {
    Gates g;
    g.i = s.cap * tanhf((row[h] + s.i_bias[h]) / s.cap);
    const float z = s.cap * tanhf((row[s.heads + h] + s.f_bias[h]) / s.cap);
    g.f = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
    return g;
}

// A CTA per head; a warp per chunk of 32 TPL tokens.
constexpr int GT_THREADS = 512, GT_MAX_CHUNKS = 512;

__device__ __forceinline__ double shfl_up(double v, int o) { return __shfl_up_sync(0xffffffffu, v, o); }

template <int TPL>
__global__ void __launch_bounds__(GT_THREADS) k_memory_gates(const float* __restrict__ gates, int ldi, int n, const __grid_constant__ MemoryShape s,
                                                             float* __restrict__ m_state, const __grid_constant__ MemoryWork w) {
    constexpr int L = 32 * TPL;
    __shared__ double last_b[GT_MAX_CHUNKS], last_g[GT_MAX_CHUNKS];  // b and max(i - b) of whole chunks
    __shared__ float m0[GT_MAX_CHUNKS + 1];
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, chunks = (n + L - 1) / L;
    double* ga = w.a + (size_t)h * n;
    double* gg = w.g + (size_t)h * n;
    for (int c = warp; c < chunks; c += GT_THREADS / 32) {
        double b[TPL], g[TPL], sum = 0.0;
#pragma unroll
        for (int x = 0; x < TPL; x++) {
            const int t = c * L + TPL * lane + x;
            Gates v = {-INFINITY, 0.0f};
            if (t < n) v = memory_gates(s, gates + (size_t)t * ldi, h);
            b[x] = sum += (double)v.f;
            g[x] = v.i;
        }
        double all = sum;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double u = shfl_up(all, o);
            if (lane >= o) all += u;
        }
        double mx = -INFINITY;
#pragma unroll
        for (int x = 0; x < TPL; x++) {
            b[x] += all - sum;
            g[x] -= b[x];
            mx = fmax(mx, g[x]);
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double u = shfl_up(mx, o);
            if (lane >= o) mx = fmax(mx, u);
        }
        if (lane == 31) {
            last_b[c] = b[TPL - 1];
            last_g[c] = mx;
        }
#pragma unroll
        for (int x = 0; x < TPL; x++) {  // a: b for now
            const int t = c * L + TPL * lane + x;
            if (t < n) {
                ga[t] = b[x];
                gg[t] = g[x];
            }
        }
    }
    __syncthreads();
    if (tid == 0) {
        float m = m_state[h];
        for (int c = 0; c < chunks; c++) {
            m0[c] = m;
            m = (float)(last_b[c] + fmax((double)m, last_g[c]));
        }
        m0[chunks] = m;
        m_state[h] = m;
    }
    __syncthreads();
    for (int c = warp; c < chunks; c += GT_THREADS / 32) {
        double b[TPL], g[TPL], mx = -INFINITY;
#pragma unroll
        for (int x = 0; x < TPL; x++) {
            const int t = c * L + TPL * lane + x;
            b[x] = t < n ? ga[t] : 0.0;
            g[x] = t < n ? gg[t] : -INFINITY;
            mx = fmax(mx, g[x]);
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double u = shfl_up(mx, o);
            if (lane >= o) mx = fmax(mx, u);
        }
        double before = shfl_up(mx, 1);
        if (lane == 0) before = -INFINITY;
        const double first = m0[c];
#pragma unroll
        for (int x = 0; x < TPL; x++) {
            const int t = c * L + TPL * lane + x;
            before = fmax(before, g[x]);
            if (t < n) {
                const float m = (float)(b[x] + fmax(first, before));
                ga[t] = b[x] - (double)m;
                w.m[(size_t)h * n + t] = m;
                w.carry[(size_t)h * n + t] = expf((float)(b[x] + first - (double)m));
                w.write[(size_t)h * n + t] = expf((float)(last_b[c] + g[x] - (double)m0[c + 1]));
            }
        }
        if (lane == 0) w.keep[(size_t)h * chunks + c] = expf((float)(last_b[c] + first - (double)m0[c + 1]));
    }
}

// 64 x 64 outputs per CTA of 256 threads, 4 x 4 each.
constexpr int TV = 64, TK = 32;

// S[chunk][h][v][d] = sum over the chunk's tokens j of write_j v_j k_j, for 64 value channels and 64 key channels.
template <class T>
__global__ void __launch_bounds__(256) k_memory_states(const T* __restrict__ p, int ldp, int n, const __grid_constant__ MemoryShape s, const __grid_constant__ MemoryWork w) {
    __shared__ float vs[MC][TV + 4], ks[MC][TV + 4];
    const int H = s.heads, D = s.dim, E = s.vdim, DP = s.dimp(), R = s.rows(), chunk = blockIdx.z, h = blockIdx.y, t0 = chunk * MC, tid = threadIdx.x;
    const int vt = (R + TV - 1) / TV, v0 = blockIdx.x % vt * TV, d0 = blockIdx.x / vt * TV, tx = tid & 15, ty = tid >> 4;
    for (int i = tid; i < MC * TV; i += 256) {
        const int j = i / TV, c = i % TV, t = t0 + j;
        float v = 0.0f, k = 0.0f;
        if (t < n) {
            const T* row = p + (size_t)t * ldp;
            if (v0 + c < E) v = act_f(row[2 * H * D + h * E + v0 + c]);
            else if (v0 + c == E) v = 1.0f;
            if (d0 + c < D) k = act_f(row[H * D + h * D + d0 + c]) * w.write[(size_t)h * n + t];
        }
        vs[j][c] = v;
        ks[j][c] = k;
    }
    __syncthreads();
    float acc[4][4] = {};
#pragma unroll 8
    for (int j = 0; j < MC; j++) {
        const float4 v = *reinterpret_cast<const float4*>(&vs[j][ty * 4]), k = *reinterpret_cast<const float4*>(&ks[j][tx * 4]);
        const float va[4] = {v.x, v.y, v.z, v.w}, ka[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
        for (int a = 0; a < 4; a++)
#pragma unroll
            for (int b = 0; b < 4; b++) acc[a][b] = fmaf(va[a], ka[b], acc[a][b]);
    }
    float* out = w.S + ((size_t)chunk * H + h) * R * DP;
#pragma unroll
    for (int a = 0; a < 4; a++) {
        const int v = v0 + ty * 4 + a, d = d0 + tx * 4;
        if (v < R && d < DP) *reinterpret_cast<float4*>(out + (size_t)v * DP + d) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
    }
}

// Chunk sums -> states at the chunks' starts; the last state goes to the sequence.  A thread per four elements.
__global__ void __launch_bounds__(256) k_memory_scan(int chunks, const __grid_constant__ MemoryShape s, float* __restrict__ state, const __grid_constant__ MemoryWork w) {
    const int h = blockIdx.y, per4 = s.rows() * s.dimp() / 4, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= per4) return;
    float4* st = reinterpret_cast<float4*>(state) + (size_t)h * per4 + i;
    float4* S = reinterpret_cast<float4*>(w.S) + (size_t)h * per4 + i;
    const size_t step = (size_t)s.heads * per4;
    const float* __restrict__ keep = w.keep + (size_t)h * chunks;
    float4 cur = *st;
    constexpr int SB = 4;  // chunks in flight
    for (int c0 = 0; c0 < chunks; c0 += SB) {
        float4 d[SB];
        float k[SB];
#pragma unroll
        for (int c = 0; c < SB; c++)
            if (c0 + c < chunks) {
                d[c] = S[(c0 + c) * step];
                k[c] = keep[c0 + c];
            }
#pragma unroll
        for (int c = 0; c < SB; c++)
            if (c0 + c < chunks) {
                S[(c0 + c) * step] = cur;
                cur = make_float4(fmaf(cur.x, k[c], d[c].x), fmaf(cur.y, k[c], d[c].y), fmaf(cur.z, k[c], d[c].z), fmaf(cur.w, k[c], d[c].w));
            }
    }
    *st = cur;
}

template <class T>
__global__ void __launch_bounds__(256) k_memory_out(const T* __restrict__ p, int ldp, int n, const __grid_constant__ MemoryShape s, const __grid_constant__ MemoryWork w) {
    __shared__ float qs[TK][MC + 4], ks[TK][MC + 4], ss[TK][TV + 4], P[MC][MC + 4];
    __shared__ float zq[MC], den[MC], zs[TK];
    const int H = s.heads, D = s.dim, E = s.vdim, DP = s.dimp(), R = s.rows(), chunk = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * TV, t0 = chunk * MC;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, cnt = min(MC, n - t0);
    const float* S = w.S + ((size_t)chunk * H + h) * R * DP;
    const float qscale = 1.0f / sqrtf((float)D);
    float sc[4][4] = {}, acc[4][4] = {}, z = 0.0f;
    for (int d0 = 0; d0 < D; d0 += TK) {
        for (int i = tid; i < MC * TK; i += 256) {
            const int j = i / TK, d = i % TK;
            const T* row = p + (size_t)(t0 + min(j, cnt - 1)) * ldp + h * D + d0 + d;
            const bool ok = j < cnt && d0 + d < D;
            qs[d][j] = ok ? act_f(row[0]) * qscale : 0.0f;
            ks[d][j] = ok ? act_f(row[H * D]) : 0.0f;
        }
        for (int i = tid; i < TV * TK; i += 256) {
            const int v = i / TK, d = i % TK;
            ss[d][v] = v0 + v < E ? S[(size_t)(v0 + v) * DP + d0 + d] : 0.0f;  // (dimp is a multiple of TK)
        }
        if (tid < TK) zs[tid] = S[(size_t)E * DP + d0 + tid];
        __syncthreads();
#pragma unroll 8
        for (int d = 0; d < TK; d++) {
            const float4 q = *reinterpret_cast<const float4*>(&qs[d][ty * 4]), k = *reinterpret_cast<const float4*>(&ks[d][tx * 4]),
                         v = *reinterpret_cast<const float4*>(&ss[d][tx * 4]);
            const float qa[4] = {q.x, q.y, q.z, q.w}, ka[4] = {k.x, k.y, k.z, k.w}, va[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int a = 0; a < 4; a++)
#pragma unroll
                for (int b = 0; b < 4; b++) {
                    sc[a][b] = fmaf(qa[a], ka[b], sc[a][b]);
                    acc[a][b] = fmaf(qa[a], va[b], acc[a][b]);
                }
        }
        if (tid < MC)
            for (int d = 0; d < TK; d++) z = fmaf(qs[d][tid], zs[d], z);
        __syncthreads();
    }
    if (tid < MC) zq[tid] = z;
    const double* ga = w.a + (size_t)h * n + t0;
    const double* gg = w.g + (size_t)h * n + t0;
#pragma unroll
    for (int a = 0; a < 4; a++) {
        const int t = ty * 4 + a;
#pragma unroll
        for (int b = 0; b < 4; b++) {
            const int j = tx * 4 + b;
            P[j][t] = j <= t && t < cnt ? sc[a][b] * expf((float)(ga[t] + gg[j])) : 0.0f;
        }
    }
    const float* carry = w.carry + (size_t)h * n + t0;
#pragma unroll
    for (int a = 0; a < 4; a++) {
        const float e = ty * 4 + a < cnt ? carry[ty * 4 + a] : 0.0f;
#pragma unroll
        for (int b = 0; b < 4; b++) acc[a][b] *= e;
    }
    __syncthreads();
    if (tid < cnt) {
        float sum = zq[tid] * carry[tid];
        for (int j = 0; j <= tid; j++) sum += P[j][tid];
        den[tid] = fmaxf(fabsf(sum), expf(-w.m[(size_t)h * n + t0 + tid])) + 1e-6f;
    }
    for (int j0 = 0; j0 < cnt; j0 += TK) {
        for (int i = tid; i < TK * TV; i += 256) {
            const int j = j0 + i / TV, v = i % TV;
            ss[i / TV][v] = j < cnt && v0 + v < E ? act_f(p[(size_t)(t0 + j) * ldp + 2 * H * D + h * E + v0 + v]) : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (int j = 0; j < TK; j++) {
            const float4 q = *reinterpret_cast<const float4*>(&P[j0 + j][ty * 4]), v = *reinterpret_cast<const float4*>(&ss[j][tx * 4]);
            const float qa[4] = {q.x, q.y, q.z, q.w}, va[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int a = 0; a < 4; a++)
#pragma unroll
                for (int b = 0; b < 4; b++) acc[a][b] = fmaf(qa[a], va[b], acc[a][b]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int a = 0; a < 4; a++) {
        const int t = ty * 4 + a;
        if (t < cnt)
#pragma unroll
            for (int b = 0; b < 4; b++)
                if (v0 + tx * 4 + b < E) w.o[(size_t)(t0 + t) * H * E + h * E + v0 + tx * 4 + b] = acc[a][b] / den[t];
    }
}

// ── one decode token per row ───────────────────────────────────────────────
// A cluster of CTAs per (head, row), each with a share of the state's rows (value channels, z last): a warp per state row, lanes
// over the key channels.  The CTAs exchange z . q and the sums of squares of their read-outs through distributed shared memory.
constexpr int MS_MAX_CLUSTER = 8;

template <class T>
__global__ void __launch_bounds__(512) k_memory_step(const __grid_constant__ MemoryArgs a, const __grid_constant__ MemoryShape s, const __grid_constant__ RowState rs,
                                                     T* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) float sm[];
    cg::cluster_group cluster = cg::this_cluster();
    const int CL = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
    const int H = s.heads, D = s.dim, E = s.vdim, DP = s.dimp(), h = blockIdx.x / CL, j = blockIdx.y;
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, warps = nt / 32;
    const int share = (E + 1 + CL - 1) / CL, r0 = rank * share, r1 = min(r0 + share, E + 1);
    float *q = sm, *k = q + DP, *o = k + DP;  // o: [share]
    __shared__ float red[16], parts[2];       // parts: sum of squares of this CTA's read-outs, z . q (of the CTA that has z)
    pdl_launch_next();
    pdl_wait();
    const T* p = (const T*)a.p + (size_t)j * a.ldp;
    float* st = (float*)rs.st0(j) + (size_t)h * s.rows() * DP;
    float* ms = (float*)rs.st1(j) + h;
    const Gates g = memory_gates(s, a.gates + (size_t)j * a.ldi, h);
    // (m0 - m is exact where it matters, so that the rounding of f + m0 does not add up over the tokens)
    const float m0 = *ms, m = fmaxf(g.f + m0, g.i), keep = expf(g.f + (m0 - m)), write = expf(g.i - m);
    const float qscale = 1.0f / sqrtf((float)D);
    for (int i = tid; i < DP; i += nt) {
        q[i] = i < D ? act_f(p[h * D + i]) * qscale : 0.0f;
        k[i] = i < D ? act_f(p[H * D + h * D + i]) * write : 0.0f;
    }
    __syncthreads();
    float ss = 0.0f;
#pragma unroll 4
    for (int r = r0 + warp; r < r1; r += warps) {
        const float v = r < E ? act_f(p[2 * H * D + h * E + r]) : 1.0f;
        float* row = st + (size_t)r * DP;
        float acc = 0.0f;
        for (int i = lane * 4; i < DP; i += 128) {
            float4 x = *reinterpret_cast<const float4*>(row + i);
            const float4 kk = *reinterpret_cast<const float4*>(k + i), qq = *reinterpret_cast<const float4*>(q + i);
            x.x = fmaf(x.x, keep, kk.x * v); x.y = fmaf(x.y, keep, kk.y * v); x.z = fmaf(x.z, keep, kk.z * v); x.w = fmaf(x.w, keep, kk.w * v);
            acc = fmaf(x.x, qq.x, fmaf(x.y, qq.y, fmaf(x.z, qq.z, fmaf(x.w, qq.w, acc))));
            *reinterpret_cast<float4*>(row + i) = x;
        }
        acc = warp_sum(acc);
        if (lane == 0) {
            if (r < E) o[r - r0] = acc;
            else parts[1] = acc;
        }
        if (r < E) ss = fmaf(acc, acc, ss);
    }
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (tid == 0) {
        ss = 0.0f;
        for (int i = 0; i < warps; i++) ss += red[i];
        parts[0] = ss;
    }
    cluster.sync();
    if (rank == 0 && tid == 0) *ms = m;  // (everyone has read it)
    ss = 0.0f;
    for (int i = 0; i < CL; i++) ss += *cluster.map_shared_rank(&parts[0], i);
    const float zq = *cluster.map_shared_rank(&parts[1], E / share);
    cluster.sync();  // a CTA's shared memory stays until everyone has read it
    const float den = fmaxf(fabsf(zq), expf(-m)) + 1e-6f, inv = 1.0f / den;
    const float r = inv / sqrtf(ss * inv * inv / (float)E + s.eps);
    for (int i = r0 + tid; i < min(r1, E); i += nt)
        out[(size_t)j * ldo + h * E + i] = f_act<T>(o[i - r0] * r * s.norm[h * E + i] * sigmoid_f(act_f(p[2 * H * D + H * E + h * E + i])));
}

template <class T>
void memory_step_go(cudaStream_t st, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, T* out, int ldo) {
    int cl = 1;  // enough CTAs to keep the memory busy, at least 16 state rows each
    while (cl < MS_MAX_CLUSTER && s.heads * a.n * cl < 148 && s.rows() / (2 * cl) >= 16) cl *= 2;
    const int share = (s.rows() + cl - 1) / cl;
    const int threads = std::min(512, std::max(128, round_up(share * 8, 128)));
    const size_t smem = ((size_t)2 * s.dimp() + share) * 4;
    if (smem > 40 * 1024) cudaFuncSetAttribute(k_memory_step<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(s.heads * cl, a.n);
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cl;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    cudaLaunchKernelEx(&cfg, k_memory_step<T>, a, s, rs, out, ldo);
}

template <class T>
cudaError_t memory_prompt_go(cudaStream_t st, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, const MemoryWork& w) {
    const int chunks = (a.n + MC - 1) / MC;
    if (chunks > GT_MAX_CHUNKS) return cudaErrorInvalidValue;
    g_kernel_launches += 4;
    k_memory_gates<MC / 32><<<s.heads, GT_THREADS, 0, st>>>(a.gates, a.ldi, a.n, s, (float*)rs.s1, w);
    const int vt = (s.rows() + TV - 1) / TV, dt = (s.dimp() + TV - 1) / TV;
    k_memory_states<T><<<dim3(vt * dt, s.heads, chunks), 256, 0, st>>>((const T*)a.p, a.ldp, a.n, s, w);
    k_memory_scan<<<dim3((s.rows() * s.dimp() / 4 + 255) / 256, s.heads), 256, 0, st>>>(chunks, s, (float*)rs.s0, w);
    k_memory_out<T><<<dim3((s.vdim + TV - 1) / TV, s.heads, chunks), 256, 0, st>>>((const T*)a.p, a.ldp, a.n, s, w);
    return cudaGetLastError();
}

}  // namespace

static bool use_tc(const MemoryShape& s, bool bf16, int n) { return bf16 && n >= MEMORY_TC_MIN_ROWS && memory_tc_supported(s); }

// One walk over the parts of the work memory: sizes, or (base given) pointers.
static size_t carve(const MemoryShape& s, bool bf16, int n, uint8_t* base, MemoryWork* w) {
    const bool tc = use_tc(s, bf16, n);
    const size_t N = (size_t)n, H = s.heads, L = tc ? MEMORY_TC_CHUNK : MC, chunks = (N + L - 1) / L;
    size_t at = 0;
    auto take = [&](auto** out, size_t count) {
        *out = (std::remove_reference_t<decltype(*out)>)(base ? base + at : nullptr);
        at += (count * sizeof(**out) + 255) / 256 * 256;
    };
    take(&w->a, N * H);
    take(&w->g, N * H);
    take(&w->carry, N * H);
    take(&w->write, N * H);
    take(&w->m, N * H);
    take(&w->keep, chunks * H);
    take(&w->S, chunks * s.state_floats());
    if (tc) {
        take((__nv_bfloat16**)&w->S_hi, chunks * s.state_floats());
        take((__nv_bfloat16**)&w->S_lo, chunks * s.state_floats());
    }
    take(&w->o, N * H * s.vdim);
    return at;
}
size_t memory_work_bytes(const MemoryShape& s, bool bf16, int n) {
    MemoryWork w;
    size_t bytes = carve(s, bf16, n, nullptr, &w);
    if (use_tc(s, bf16, n)) bytes = std::max(bytes, carve(s, bf16, MEMORY_TC_MIN_ROWS - 1, nullptr, &w));  // shorter portions take the other form
    return bytes;
}
MemoryWork memory_work(const MemoryShape& s, bool bf16, int n, void* base, uint32_t* err) {
    MemoryWork w;
    carve(s, bf16, n, (uint8_t*)base, &w);
    w.err = err;
    return w;
}

cudaError_t launch_memory_prompt(cudaStream_t st, bool bf16, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, const MemoryWork& w,
                                 void* out, int ldo) {
    if (a.n <= 0) return cudaSuccess;
    cudaError_t e;
    if (use_tc(s, bf16, a.n)) {
        if ((a.n + MEMORY_TC_CHUNK - 1) / MEMORY_TC_CHUNK > GT_MAX_CHUNKS) return cudaErrorInvalidValue;
        g_kernel_launches++;
        k_memory_gates<MEMORY_TC_CHUNK / 32><<<s.heads, GT_THREADS, 0, st>>>(a.gates, a.ldi, a.n, s, (float*)rs.s1, w);
        e = launch_memory_tc(st, a, s, rs, w);
    } else {
        e = bf16 ? memory_prompt_go<__nv_bfloat16>(st, a, s, rs, w) : memory_prompt_go<float>(st, a, s, rs, w);
    }
    if (e != cudaSuccess) return e;
    const int off = 2 * s.heads * s.dim + s.heads * s.vdim;
    const void* gate = bf16 ? (const void*)((const __nv_bfloat16*)a.p + off) : (const void*)((const float*)a.p + off);
    launch_gated_head_norm(st, bf16, a.n, s.heads, s.vdim, s.eps, w.o, s.norm, s.vdim, gate, false, a.ldp, out, ldo);
    return cudaGetLastError();
}

void launch_memory_step(cudaStream_t st, bool bf16, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, void* out, int ldo) {
    if (a.n <= 0) return;
    g_kernel_launches++;
    if (bf16) memory_step_go(st, a, s, rs, (__nv_bfloat16*)out, ldo);
    else memory_step_go(st, a, s, rs, (float*)out, ldo);
}

}  // namespace wick
