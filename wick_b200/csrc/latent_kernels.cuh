// Launch wrappers of latent attention.
#pragma once
#include "hybrid_kernels.cuh"

namespace wick {

// Queries come through a latent of q_rank, keys and values through a latent of kv_rank that all heads share, beside rot_dim
// key columns that carry the position.  Only the normalised latent and the rotated key part are cached, one row per position:
//   [c: kv_rank, up to a multiple of 8 | rotated part: rot_dim, up to a multiple of 8]   (padding zero)
// A query may be taken to the latent's side, q_c = W_uk^T q, so that its score is one product with a cache row and the weighted
// sum of cache rows gives the value through W_uv ("absorbed"; decode, short portions, f32); or keys and values of the visible
// positions are computed from the cache (prompts).  Softmax has one more entry per head, `sink`, without a value.
struct LatentShape {
    int heads = 0, dim = 0, rot_dim = 0, rot_dims = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    int size = 0;                  // sliding window (0: none): key j is seen by i when i - j < size
    float scale = 1.0f, eps = 0.0f;
    const float* sink = nullptr;   // [H]
    const float2* rope = nullptr;  // [positions][rot_dims / 2] cos, sin of the first rot_dims of the rot_dim columns, in pairs
    const float *q_norm = nullptr, *kv_norm = nullptr;
    __host__ __device__ int ldc() const { return round_up(kv_rank, 8) + round_up(rot_dim, 8); }  // cache row
    __host__ __device__ int off_rot() const { return round_up(kv_rank, 8); }
    // a query row: per head [dim, up to a multiple of 8 | rot_dim, up to a multiple of 8]
    __host__ __device__ int q_off_rot() const { return round_up(dim, 8); }
    __host__ __device__ int q_pitch() const { return round_up(dim, 8) + round_up(rot_dim, 8); }
    __host__ __device__ int off_kv() const { return round_up(q_rank, 8); }  // of the projections' row: [c_q | c, rotated part]
    int seen(int max_seq) const { return size > 0 && size < max_seq ? size : max_seq; }
};
// Rows of p act [n][ldp]: c_q normalised in place, c normalised and the rotated part turned into the cache (state s0 / p0).
void launch_latent_append(cudaStream_t st, bool bf16, void* p, int ldp, int n, const LatentShape& s, const RowState& rs);
// Absorbed attention: qc act [n][H][ldc] (q taken to the latent's side in the first kv_rank columns of a head, zero up to
// off_rot), q act [n][ldq] (the rotated columns are read from here, before the rotation).  o act [n][H][ldo_h]: weighted sums of
// latents.
struct LatentScratch {
    float* partial = nullptr;  // key splits: latent_scratch() floats
    uint32_t* err = nullptr;   // device word for expired waits
};
size_t latent_scratch(const LatentShape& s, bool bf16, int max_rows, int max_seq);
bool latent_supported(const LatentShape& s);
cudaError_t launch_latent_attn(cudaStream_t st, bool bf16, const void* qc, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs,
                               void* o, int ldo_h, const LatentScratch& sc, int max_seq);
// Its tensor-core form (attn_latent_step.cu), bf16: a split per LATENT_STEP_KEYS keys.
constexpr int LATENT_STEP_KEYS = 64, LATENT_MAX_SPLIT = 256;
bool latent_step_supported(const LatentShape& s, int max_seq);
cudaError_t launch_latent_step(cudaStream_t st, const void* qc, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs, float* partial,
                               int splits, uint32_t* err);

// The prompt form (attn_latent_tc.cu): consecutive bf16 tokens of one sequence; keys and values of the visible positions come
// from the cache through ukv, whose rows are [H][dim, up to a multiple of 8] keys, then [H][vdim, up to a multiple of 8] values.
constexpr int LATENT_TC_MIN_ROWS = 16;
bool latent_tc_supported(const LatentShape& s);
// kv act [latent_tc_keys()][latent_tc_cols()]: work memory
inline int latent_tc_cols(const LatentShape& s) { return s.heads * (round_up(s.dim, 8) + round_up(s.vdim, 8)); }
inline size_t latent_tc_keys(const LatentShape& s, int max_rows, int max_seq) {
    return s.size > 0 ? std::min<size_t>(max_seq, (size_t)max_rows + s.size) : (size_t)max_seq;
}
// q act [n][ldq] before the rotation; out act [n][ldo] (H * vdim).
cudaError_t launch_latent_kv(cudaStream_t st, int n, const LatentShape& s, const RowState& rs, const DenseWeight& ukv, void* kv, uint32_t* err);
cudaError_t launch_latent_attn_tc(cudaStream_t st, const void* q, int ldq, int n, const LatentShape& s, const RowState& rs, const void* kv, void* out,
                                  int ldo, uint32_t* err);

}  // namespace wick
