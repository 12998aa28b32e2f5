// Sorts the routed rows of a portion by expert (launch_route): a counting sort in shared memory, one CTA per table.  The order
// within an expert is left open; a row's result does not depend on its place.
#include "hybrid_kernels.cuh"

namespace wick {

namespace {

constexpr int RT_THREADS = 1024;
struct RouteJobs {
    RouteJob job[MAX_ROUTES];
};

__global__ void __launch_bounds__(RT_THREADS) k_route(const uint32_t* __restrict__ tokens, int n, const __grid_constant__ RouteJobs jobs) {
    const RouteJob& r = jobs.job[blockIdx.x];
    __shared__ int next[MAX_EXPERTS];
    const int tid = threadIdx.x, total = n * r.top;
    for (int e = tid; e < r.experts; e += RT_THREADS) next[e] = 0;
    __syncthreads();
    for (int i = tid; i < total; i += RT_THREADS) atomicAdd(&next[r.table[(size_t)tokens[i / r.top] * r.top + i % r.top]], 1);
    __syncthreads();
    if (tid < 32) {
        int base = 0;
        for (int e0 = 0; e0 < r.experts; e0 += 32) {
            const int e = e0 + tid, own = e < r.experts ? next[e] : 0;
            int v = own;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int u = __shfl_up_sync(0xffffffffu, v, o);
                if (tid >= o) v += u;
            }
            if (e < r.experts) next[e] = r.start[e] = base + v - own;
            base += __shfl_sync(0xffffffffu, v, 31);
        }
        if (tid == 0) r.start[r.experts] = base;
    }
    __syncthreads();
    for (int i = tid; i < total; i += RT_THREADS)
        r.inv[i] = atomicAdd(&next[r.table[(size_t)tokens[i / r.top] * r.top + i % r.top]], 1);
}

}  // namespace

void launch_route(cudaStream_t st, const uint32_t* tokens, int n, const RouteJob* jobs, int count) {
    for (int i = 0; i < count; i += MAX_ROUTES) {
        RouteJobs j;
        const int c = std::min(MAX_ROUTES, count - i);
        std::copy(jobs + i, jobs + i + c, j.job);
        g_kernel_launches++;
        k_route<<<c, RT_THREADS, 0, st>>>(tokens, n, j);
    }
}

}  // namespace wick
