// Launch wrappers of the kernels behind models that are described by a config.json layer list (hybrid.cu): dense bfloat16
// matrices (plain, block-diagonal, per expert), hyper-connection streams, a plain residual with norms around the sublayers,
// windowed attention with blended sigmoid scores, latent attention, the channel-decay delta rule and the matrix memory.
// Sizes and constants are arguments, so that another design can use the same kernels.
//
// Activations are token-major.  "act" buffers hold the model's activation type: bfloat16, or f32 for a model created with
// WICK_CUDA_COMPUTE_F32; `bf16` says which.  Row pitches of act buffers are multiples of 8 elements and their padding
// stays zero.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include <algorithm>

#include "kernels.cuh"

namespace wick {

__host__ __device__ constexpr int round_up(int v, int to) { return (v + to - 1) / to * to; }

// ── dense matrices ─────────────────────────────────────────────────────────
// [m][ld] bfloat16, ld = k rounded up to 8, padding zero, base 16-byte aligned.  The weights of the file are bfloat16, so
// this is exact in both activation types.
struct DenseWeight {
    const __nv_bfloat16* w = nullptr;
    int m = 0, k = 0, ld = 0;
};
enum Activation { ACT_RELU = 0, ACT_SILU = 1, ACT_RELU2 = 2, ACT_NONE = 3 };
struct DenseJob {
    DenseWeight w;
    const void* x = nullptr;  // act [n][ldx]
    int ldx = 0;
    void* y = nullptr;        // act or f32 [n][ldy]
    int ldy = 0;
    bool f32 = false;         // y is f32 whatever the activation type
};
// Block-diagonal matrix: `rows` weight rows per block; block b multiplies columns b * x_step .. of x and fills columns
// b * y_step .. of y.
struct DenseBlocks {
    int rows = 0, x_step = 0, y_step = 0;
    __host__ __device__ explicit operator bool() const { return rows > 0; }
};
// One matrix per expert, stacked (job.w.m rows each).  Few tokens: routed row r belongs to choice r % top of token r / top and
// its expert is looked up; many tokens: rows are sorted by expert, expert e has rows start[e] .. start[e + 1] - 1.
struct DenseExperts {
    int count = 0, top = 1;
    const int* table = nullptr;  // [vocab][top]
    const uint32_t* tokens = nullptr;
    const DecodeCtl* ctl = nullptr;  // the single token of a decode step, when tokens == NULL
    bool x_per_token = false;    // (lookup) the input row of routed row r is r / top
    const int* start = nullptr;  // [count + 1]; NULL: lookup
    __host__ __device__ explicit operator bool() const { return count > 0; }
};
// y = act(x W^T) for n rows.  Up to two independent jobs share a launch; or (gated) the two jobs are gate and up matrices of
// the same shape and input and job[0].y = act(gate x) * (up x).
struct DenseCall {
    DenseJob job[2];
    int count = 1, n = 0;
    bool gated = false;
    Activation act = ACT_NONE;
    float scale = 1.0f;     // y times this
    float softcap = 0.0f;   // > 0: then y = softcap * tanh(y / softcap)
    DenseBlocks blocks;     // one ungated job
    DenseExperts experts;   // one job, or gated; n counts routed rows
    uint32_t* err = nullptr;  // device word for expired waits of the tensor-core kernel
};
// Chooses between the row-streaming kernel (few rows, blocks), the tcgen05 kernel (bfloat16) and the f32 kernel.
cudaError_t launch_dense(cudaStream_t st, bool bf16, const DenseCall& call);
// The individual kernels (launch_dense picks one).
void launch_dense_rows(cudaStream_t st, bool bf16, const DenseCall& call);    // n <= DENSE_ROWS_MAX; any n for blocks and looked-up experts
void launch_dense_simt(cudaStream_t st, bool bf16, const DenseCall& call);    // any n
cudaError_t launch_dense_tc(cudaStream_t st, const DenseCall& call);          // bfloat16, tcgen05
constexpr int DENSE_ROWS_MAX = 8;
constexpr int MAX_EXPERTS = 1024;

// Sorts the n * top routed rows of a portion by expert, one table per block of the launch:
// inv[j * top + s] = sorted row of token j's choice s, start[e] = first row of expert e (start[count] = n * top).
struct RouteJob {
    const int* table = nullptr;  // [vocab][top]
    int* inv = nullptr;
    int* start = nullptr;
    int experts = 0, top = 1;
};
constexpr int MAX_ROUTES = 64;  // tables per launch
void launch_route(cudaStream_t st, const uint32_t* tokens, int n, const RouteJob* jobs, int count);

// ── where the rows of a launch live ────────────────────────────────────────
// Either n consecutive tokens of one sequence (positions == NULL: row j is at start_pos + j, state s0 / s1), or one token of
// each of n sequences (positions[j], and p0[j] / p1[j] unless there is a single row with state s0 / s1).
struct RowState {
    void* const* p0 = nullptr;
    void* const* p1 = nullptr;
    void *s0 = nullptr, *s1 = nullptr;
    const uint32_t* positions = nullptr;
    int start_pos = 0;
    __device__ void* st0(int j) const { return p0 ? p0[j] : s0; }
    __device__ void* st1(int j) const { return p1 ? p1[j] : s1; }
    __device__ int pos(int j) const { return positions ? (int)positions[j] : start_pos + j; }
    bool separate() const { return positions != nullptr; }
};

// ── hyper-connections + RMS norm with a scalar gain ────────────────────────
// x [n][S][W] f32 streams.  One launch applies the previous sublayer's write (if any), reads the next sublayer's input and
// normalises it:
//   x_t <- sum_s mix[s][t] x_s + out[t] y        (y != NULL)
//   h   =  g * u / sqrt(mean(u^2) + eps),  u = sum_s in[s] x_s   (in == NULL: plain sum)
struct HyperArgs {
    // first launch of a step: the streams all equal scale * embed[token] (tokens) or the given frame (frames); x is written
    const uint32_t* tokens = nullptr;
    const DecodeCtl* ctl = nullptr;       // the single token of a decode step, when tokens == NULL
    const __nv_bfloat16* embed = nullptr;
    int ld_embed = 0;
    float embed_scale = 1.0f;
    const float* frames = nullptr;        // [n][W]
    float* x = nullptr;
    bool store_x = true;
    const float* y = nullptr;             // [n][ldy] f32 output of the previous sublayer
    int ldy = 0;
    const float *mix = nullptr, *out = nullptr;  // of the previous sublayer: [S][S], [S]
    const float* in = nullptr;            // of the next sublayer: [S]
    const float* gain = nullptr;          // [1]
    float eps = 0.0f;
    const int* rows = nullptr;            // if set, output row i comes from row rows[i] of x and y (x is then not written)
    void* h = nullptr;                    // act [n][ldh]
    int ldh = 0;
    float* normed = nullptr;              // optional f32 copy of the last row's h [W]
    int n = 0, S = 1, W = 0;
};
constexpr int HYPER_MAX_STREAMS = 16;
void launch_hyper_norm(cudaStream_t st, bool bf16, const HyperArgs& a);

// ── one residual stream with norms before and after every sublayer ─────────
// One launch takes the previous sublayer's output into x and makes the next sublayer's input:
//   x <- the embedding row or frame                (embed / frames)
//   x <- x + post * rms(y)                         (post != NULL; y the sum of y_parts rows times y_scale)
//   x <- y + shift                                 (post == NULL, shift != NULL)
//   h  = gain * rms(x), or h = [x | x0] with the embedding output x0 (gain == NULL)
// with rms(z) = z / sqrt(mean(z^2) + eps).
struct ResidualArgs {
    const uint32_t* tokens = nullptr;     // where embedding rows come from, for the start and for x0
    const DecodeCtl* ctl = nullptr;
    const __nv_bfloat16* embed = nullptr;
    int ld_embed = 0;
    const float* frames = nullptr;        // [n][W]
    bool init = false;                    // x starts as the embedding row / frame
    float* x = nullptr;                   // [n][W]
    bool store_x = true;
    const float* y = nullptr;             // [rows][ldy] f32 output of the previous sublayer
    int ldy = 0;
    int y_parts = 1;                      // rows j * y_parts .. of y belong to token j, or (y_rows) rows y_rows[j * y_parts ..]
    const int* y_rows = nullptr;
    float y_scale = 1.0f;
    const float *post = nullptr, *shift = nullptr;  // [W]
    const float* gain = nullptr;          // [W]
    float eps = 0.0f;
    const int* rows = nullptr;            // if set, output row i comes from token rows[i] (x is then not written)
    void* h = nullptr;                    // act [..][ldh]
    int ldh = 0;
    int h_parts = 1;                      // with h_rows: h of token j goes to rows h_rows[j * h_parts ..]
    const int* h_rows = nullptr;
    float* normed = nullptr;              // optional f32 copy of the last row's h [W]
    int n = 0, W = 0;
};
void launch_residual_norm(cudaStream_t st, bool bf16, const ResidualArgs& a);

// ── windowed attention with blended sigmoid scores ─────────────────────────
struct MixAttnShape {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int size = 0;        // sliding window (0: none): key j is seen by i when i - j < size
    int keep_first = 0;  // ... or j < keep_first
    float scale = 1.0f, eps = 0.0f;
    const float* talk = nullptr;  // [H][H] or NULL
    const float* bias = nullptr;  // [H] added to the blended score, or NULL
    int seen(int max_seq) const { return size > 0 && size + keep_first < max_seq ? size + keep_first : max_seq; }
};
// Work memory of one attention layer: mix_attn_scratch() says how much for up to max_rows rows.
struct MixAttnScratch {
    float* partial = nullptr;  // key splits
    void* fold = nullptr;      // folded queries of the tensor-core form (bf16), 16-byte aligned
    uint32_t* err = nullptr;   // device word for expired waits
};
void mix_attn_scratch(const MixAttnShape& s, bool bf16, int max_rows, size_t* partial_floats, size_t* fold_bytes);
bool mix_attn_supported(const MixAttnShape& s);
// Splits qkv [n][ld] (heads*dim q, kv_heads*dim k, kv_heads*vdim v): q and k divided by their root mean square per head, k and
// v rows appended to the caches (act [pos][kv_heads*dim], [pos][kv_heads*vdim]); q back in place or, where the tensor-core form
// follows, folded into sc.fold.
void launch_qk_rms_append(cudaStream_t st, bool bf16, void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, const MixAttnScratch& sc);
// (For separate rows the decode kernel does this itself where the sizes allow it, and this launches nothing.)
// out act [n][ldo] (heads*vdim), after launch_qk_rms_append of the same rows.
cudaError_t launch_mix_attn(cudaStream_t st, bool bf16, const void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, void* out,
                            int ldo, const MixAttnScratch& sc, int max_seq);
// The tensor-core form (attn_mix_tc.cu): consecutive bf16 tokens of one sequence, sizes that are multiples of 8.
constexpr int MIX_ATTN_TC_MIN_ROWS = 16;
bool mix_attn_tc_supported(const MixAttnShape& s);
void launch_qk_fold_append(cudaStream_t st, const void* qkv, int ld, int n, const MixAttnShape& s, const RowState& rs, void* fold);
cudaError_t launch_mix_attn_tc(cudaStream_t st, const void* fold, int n, const MixAttnShape& s, const RowState& rs, void* out, int ldo, uint32_t* err);

// ── channel-decay delta rule ───────────────────────────────────────────────
struct DeltaShape {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1;
    float eps = 0.0f;
    __host__ __device__ int dimp() const { return round_up(dim, 32); }            // key channels per head in f32 work rows and in the state
    __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; }
    size_t state_floats() const { return (size_t)heads * vdim * dimp(); }   // [H][vdim][dimp]
    size_t conv_floats() const { return (size_t)(taps - 1) * channels(); }  // [taps - 1][channels]
};
constexpr int DELTA_MAX_DIM = 256, DELTA_MAX_TAPS = 16;
// f32 work rows of n tokens that the recurrence reads
struct DeltaWork {
    float *q = nullptr, *k = nullptr;  // [n][G][dimp] unit vectors, q times dim^-1/2
    float* v = nullptr;                // [n][H*vdim]
    float* g = nullptr;                // [n][H][dimp] decay factors
    float* beta = nullptr;             // [n][H]
    float* kq = nullptr;               // [n][G] k . q
    float* o = nullptr;                // [n][H*vdim] read-outs
    float* rec = nullptr;              // chunk records of the prompt form, delta_record_floats(); replaces q, k, g, beta, kq
};
// Portions of at least this many tokens of one sequence take the prompt form (delta_chunk.cu), DELTA_CHUNK tokens at a time.
constexpr int DELTA_CHUNK = 8;
constexpr int DELTA_CHUNK_MIN_ROWS = 8;
size_t delta_record_floats(const DeltaShape& s, int n);
struct DeltaPrepArgs {
    const void* p = nullptr;  // act [n][ldp]: the q | k | v channels at 0.., the beta logits at off_b
    int ldp = 0, off_b = 0;
    const float* a = nullptr;  // [n][lda] decay projection H*dim
    int lda = 0;
    const float *conv_w = nullptr, *A_log = nullptr, *dt_bias = nullptr;  // [channels][taps], [H], [H*dim]
    int n = 0;
};
// Consecutive tokens of one sequence: short convolution + silu, unit q and k, decays and step sizes; advances the convolution
// state (s1).
void launch_delta_prep(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w);
// Their recurrence; state in s0.
void launch_delta_scan(cudaStream_t st, int n, const DeltaShape& s, const RowState& rs, const DeltaWork& w);
// The two steps of the prompt form (called by the launchers above).
void launch_delta_chunk_prep(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const DeltaWork& w);
void launch_delta_chunk_scan(cudaStream_t st, int n, const DeltaShape& s, const RowState& rs, const DeltaWork& w);
// out act [n][ldo] = rms(o) * norm * sigmoid(gate) per head of E values: o f32 [n][H * E], head h's weights at norm + h *
// norm_step, gate f32 or act [n][ldg]
void launch_gated_head_norm(cudaStream_t st, bool bf16, int n, int H, int E, float eps, const float* o, const float* norm, int norm_step,
                            const void* gate, bool gate_f32, int ldg, void* out, int ldo);

// One decode token per row: convolutions, decays, the recurrence and the gated norm in one launch (state s0 / p0 and s1 / p1).
void launch_delta_step(cudaStream_t st, bool bf16, const DeltaPrepArgs& a, const DeltaShape& s, const RowState& rs, const float* norm,
                       const float* gate, int ldg, void* out, int ldo);

// ── launches that may start before their predecessor has finished ──────────
// The kernels of a decode step are launched with programmatic stream serialisation: a kernel is brought up while the one before
// it still runs, touches nothing but weights, and calls pdl_wait() before it reads or writes anything else.  Every kernel
// launched this way must call pdl_wait() (it is what keeps the whole chain ordered).
template <class... P, class... A>
inline cudaError_t launch_pdl(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, A&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kernel, P(args)...);
}
__device__ __forceinline__ void pdl_launch_next() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// ── shared device helpers ──────────────────────────────────────────────────
__device__ __forceinline__ float act_f(float v) { return v; }
__device__ __forceinline__ float act_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T>
__device__ __forceinline__ T f_act(float v);
template <>
__device__ __forceinline__ float f_act<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 f_act<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// eight consecutive values from a 16-byte aligned address
__device__ __forceinline__ void bf16x8_f(const uint4 u, float* f) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) { bf16x8_f(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float* f) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float activate(float z, Activation a) {
    if (a == ACT_SILU) return silu_f(z);
    const float r = fmaxf(z, 0.0f);
    return a == ACT_RELU ? r : a == ACT_RELU2 ? r * r : z;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

}  // namespace wick
