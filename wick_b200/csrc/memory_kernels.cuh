// Launch wrappers of the matrix memory with exponential gates.
#pragma once
#include "hybrid_kernels.cuh"

namespace wick {

// Per head, with log gates i, f and a running maximum m (log domain):
//   m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  z likewise with v = 1
//   o = S^T q / (max(|z . q|, exp(-m')) + 1e-6)
// The state holds S^T and z together: s0 f32 [H][vdim + 1][dimp], z being the last row; s1 f32 [H]: m.
struct MemoryShape {
    int heads = 0, dim = 0, vdim = 0;
    float cap = 1.0f, eps = 0.0f;
    const float *i_bias = nullptr, *f_bias = nullptr, *norm = nullptr;  // [H], [H], [H * vdim]
    __host__ __device__ int dimp() const { return round_up(dim, 32); }
    __host__ __device__ int rows() const { return vdim + 1; }
    size_t state_floats() const { return (size_t)heads * rows() * dimp(); }
};
constexpr int MEMORY_CHUNK = 64;
constexpr int MEMORY_MAX_DIM = 4096;  // of keys and of values
// Work memory for n tokens of one sequence, carved out of one allocation of memory_work_bytes().
struct MemoryWork {
    double *a = nullptr, *g = nullptr;                   // [H][n]: log weight of token j in token t's sum = a[t] + g[j] (same chunk)
    float *carry = nullptr, *write = nullptr, *m = nullptr;  // [H][n]: weight of the chunk's first state; of token j in the next; m
    float* keep = nullptr;                               // [H][chunks]: weight of the chunk's first state in the next
    float* S = nullptr;                                  // [chunks][H][vdim + 1][dimp] chunk sums, then states at the chunks' starts
    void *S_hi = nullptr, *S_lo = nullptr;               // bf16 [chunks][H][vdim + 1][dimp]: the latter of the tensor-core form
    float* o = nullptr;                                  // [n][H * vdim] read-outs
    uint32_t* err = nullptr;                             // device word for expired waits
};
size_t memory_work_bytes(const MemoryShape& s, bool bf16, int n);
MemoryWork memory_work(const MemoryShape& s, bool bf16, int n, void* base, uint32_t* err);
// Projections: q | k | v | g act columns of a row of p (ldp) in this order, gates f32 [n][ldi]: H input, then H forget logits.
struct MemoryArgs {
    const void* p = nullptr;
    int ldp = 0;
    const float* gates = nullptr;
    int ldi = 0, n = 0;
};
// Consecutive tokens of one sequence: read-outs, normalised and gated, to out act [n][ldo].
cudaError_t launch_memory_prompt(cudaStream_t st, bool bf16, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, const MemoryWork& w,
                                 void* out, int ldo);
// Its tensor-core form (memory_tc.cu): everything between the gates and the output norm, bf16, portions of at least
// MEMORY_TC_MIN_ROWS tokens.
constexpr int MEMORY_TC_CHUNK = 128, MEMORY_TC_MIN_ROWS = 65;
bool memory_tc_supported(const MemoryShape& s);
cudaError_t launch_memory_tc(cudaStream_t st, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, const MemoryWork& w);
// One decode token per row.
void launch_memory_step(cudaStream_t st, bool bf16, const MemoryArgs& a, const MemoryShape& s, const RowState& rs, void* out, int ldo);

}  // namespace wick
