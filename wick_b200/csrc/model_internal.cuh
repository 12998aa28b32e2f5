// Internals shared by the host-side files of libwick_cuda: the model handle, its per-layer sequence state, and what an
// architecture has to provide to be served by the drivers of wick_cuda.cu.
#pragma once
#include <algorithm>
#include <cstdio>
#include <memory>
#include <string>
#include <vector>

#include "../../include/wick_cuda.h"
#include "decode_mega.cuh"
#include "gemm_tc.cuh"
#include "kernels.cuh"

namespace wick {

// Last error message of the calling thread (wick_cuda_last_error).
int32_t fail(int32_t code, const std::string& msg);

#define CU_TRY(expr)                                                                              \
    do {                                                                                          \
        cudaError_t e__ = (expr);                                                                 \
        if (e__ != cudaSuccess)                                                                   \
            return fail(e__ == cudaErrorMemoryAllocation ? WICK_CUDA_ERR_OOM : WICK_CUDA_ERR_CUDA, \
                        std::string(#expr) + ": " + cudaGetErrorString(e__));                     \
    } while (0)
#define W_TRY(expr)                  \
    do {                             \
        int32_t r__ = (expr);        \
        if (r__ != WICK_CUDA_OK) return r__; \
    } while (0)

// One buffer of sequence state of a layer.  A buffer either grows with the sequence (bytes per cached position: K and V
// rows) or has a fixed size and starts at zero (rolling convolution inputs, recurrent state).
struct StateDesc {
    size_t per_pos = 0, fixed = 0;
    size_t bytes(size_t positions) const { return per_pos * positions + fixed; }
};

struct Layer {
    bool is_attn = false;
    int n_kv = 0;
    float *attn_norm = nullptr, *ffn_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr, *conv_w = nullptr;
    DevWeight in_proj, out_proj, q, k, v, o, gate, up, down;
    // int8 copies for the tensor-core prefill GEMM (gemm_tc.cu); q == nullptr when unavailable
    TcWeight tc_in_proj, tc_out_proj, tc_q, tc_k, tc_v, tc_o, tc_gate, tc_up, tc_down;
    // what the layer keeps per sequence (at most two buffers; the model's own sequence is bound here, see SeqSlot)
    StateDesc sd[2];
    void* state[2] = {nullptr, nullptr};
    // lfm2 attention: f32 K and V rows [max_seq][kv_dim]; lfm2 conv: rolling buffer [d_conv][hidden]
    float* k_cache() const { return (float*)state[0]; }
    float* v_cache() const { return (float*)state[1]; }
    float* conv_state() const { return (float*)state[0]; }
};

// Which rows of a prefill chunk get logits: rows[i] of the chunk -> dst + i * vocab.
struct LogitRows {
    const int* rows = nullptr;
    int count = 0;
    float* dst = nullptr;
    bool want_logits = true;  // false: only the output-normed row (m->normed_last) is wanted
};

// An architecture: how its steps are enqueued on m->stream.  Everything around it - sequence slots, state allocation, reset,
// snapshot and restore, graph capture of the decode step, greedy loops, sampling, batching - is common code.
struct ModelFamily {
    // one decode step of the model's own sequence, token and position from m->ctl; captured into a graph
    int32_t (*enqueue_decode)(wick_cuda_model* m, bool greedy);
    // called before a prefill call of n tokens or a batch of n rows: late allocations
    int32_t (*prepare)(wick_cuda_model* m, int n);
    // n <= max_chunk prompt tokens (m->tokens_dev, or frames already in m->hidden) at start_pos..
    int32_t (*enqueue_prefill_chunk)(wick_cuda_model* m, int n, int start_pos, bool flash, bool embed, const LogitRows& out);
    // one token for each of n rows (m->rows_tok, rows_pos, rows_ptrs) -> m->logits_rows
    int32_t (*enqueue_decode_rows)(wick_cuda_model* m, int n);
    bool kv_shift;  // rows of the cache can be dropped and moved (wick_cuda_shift_kv)
};

struct HybridModel;  // hybrid.cuh

}  // namespace wick

struct wick_cuda_model {
    // (types of namespace wick, spelled out because the handle itself is a C type)
    const wick::ModelFamily* family = nullptr;  // what the architecture's own code provides (model_internal.cuh)
    std::string arch;                     // architecture name as the model file spells it
    std::unique_ptr<wick::HybridModel> hybrid;  // weights and scratch of a config.json model (hybrid.cu), NULL for lfm2
    int device = 0;
    cudaStream_t stream = nullptr;
    wick_cuda_config cfg{};
    int head_dim = 0;
    std::vector<wick::Layer> layers;
    wick::DevWeight embd;
    wick::TcWeight tc_embd;       // tensor-core copy of the vocabulary matrix, made for the multi-sequence step only
    bool embd_q6k = false;  // token_embd is Q6_K: embd6 is used for the embedding rows and the logits, embd is empty
    wick::DevQ6K embd6;
    float* output_norm = nullptr;
    float *rope_cos = nullptr, *rope_sin = nullptr;
    int max_chunk = 0;  // tokens of scratch
    // tensor-core prefill GEMMs: available when every matrix meets tc_gemm_supported(); prefill_mode
    // picks the bit-exact one (default), the fused-chain one, or the bit-exact CUDA-core kernel
    bool tc_ok = false;     // the model's shapes allow the tensor-core GEMM
    bool tc_built = false;  // its int8 weight copies and buffers exist (made by the first call that needs them)
    int prefill_mode = WICK_CUDA_PREFILL_EXACT;
    CUtensorMap map_x_hs[2], map_x_is[2];  // activations [max_chunk][hs | is], box of 64 / 128 rows
    int8_t* q8m = nullptr;                  // lane-group-masked activations [4 * max_chunk][hs | is] (exact tensor-core GEMM)
    CUtensorMap map_xm_hs, map_xm_is, map_xm_hs32, map_xm_is32;  // boxes of 64 rows (16 tokens) and of 32 rows (8 tokens)
    float* normed_last = nullptr;  // output-normed hidden row of the last prefilled token
    float* rope_delta = nullptr;   // [head_dim]: cos then sin of the n_keep shift rotation
    uint32_t* tc_err = nullptr;
    // scratch, token-major
    float *hidden = nullptr, *block_out = nullptr, *ffn_out = nullptr, *proj = nullptr, *qbuf = nullptr, *kbuf = nullptr,
          *vbuf = nullptr, *attn_out = nullptr, *gate = nullptr, *up = nullptr, *logits = nullptr;
    float* q8s = nullptr;
    int8_t* q8q = nullptr;
    uint32_t* tokens_dev = nullptr;
    wick::DecodeCtl* ctl = nullptr;
    uint32_t* argmax_tok = nullptr;
    uint32_t* ring = nullptr;
    int ring_len = 0;
    // pinned host staging
    uint32_t* h_u32 = nullptr;   // [ring_len] tokens in / out
    float* h_logits = nullptr;   // [vocab]
    cudaGraphExec_t g_logits = nullptr, g_greedy = nullptr;
    uint64_t nodes_logits = 0, nodes_greedy = 0;  // kernels per graph replay
    uint64_t launches = 0;                        // kernels launched so far
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;     // bracket the GPU work of the last call
    // persistent decode kernel (decode_mega.cu); falls back to the captured graphs when the
    // model does not meet its layout requirements or WICK_CUDA_DECODE=graph is set
    bool mega_ok = false;
    int mega_ctas = 0;
    wick::MegaParams mega{};
    wick::MegaPhase* d_phases = nullptr;
    wick::MegaPhase* d_phases_long = nullptr;  // the same list with an MPH_SCORES phase before every MPH_ATTN (long contexts)
    int n_phases_long = 0;
    float* scores_g = nullptr;
    bool last_launch_long = false, long_ok = false;
    wick::MegaLayer* d_mlayers = nullptr;
    unsigned long long* d_sync = nullptr;  // [0] barrier counter, [1..2] argmax accumulators
    unsigned long long* hidden_flagged = nullptr;  // [hs] flagged copy of the hidden row (persistent decode kernel)
    unsigned long long* d_prof = nullptr;  // [n_phases][4] timestamps of the last step
    unsigned long long bar_base = 0;
    wick::DecodeCtl* h_ctl = nullptr;            // pinned copy of the control block
    uint32_t seq_len = 0;
    uint64_t bytes = 0;
    std::vector<void*> allocs;
    // extra sequence slots for wick_cuda_decode_batch (the model's own sequence is not one of them)
    struct SeqSlot {
        bool live = false;
        uint32_t seq_len = 0;
        std::vector<void*> state;  // [n_layers][2]: the slot's copies of Layer::state (NULL where the layer has none)
    };
    std::vector<SeqSlot> seqs;
    // per-category device timers of the prefill pipeline (WICK_CUDA_PROFILE=events or wick_cuda_profile_enable)
    bool prof_on = false;
    std::vector<cudaEvent_t> prof_events;   // pool, reused chunk after chunk
    std::vector<int> prof_marks;            // category that ENDS at event i + 1 of the current chunk
    size_t prof_used = 0;
    double prof_ms[WICK_CUDA_PROFILE_CATEGORIES] = {};
    // opt-in split-K decode attention (graph decode path and the multi-sequence step; the persistent kernel stays exact)
    bool attn_splitk = false;
    float* splitk_scratch = nullptr;
    size_t splitk_floats = 0;
    float* sample_val = nullptr;        // [vocab] work arrays of the on-device sampler, made on first use
    int* sample_idx = nullptr;
    uint32_t* sample_status = nullptr;
    int batch_cap = 0;                  // rows the batch buffers below hold
    float* logits_rows = nullptr;       // [batch_cap][vocab]
    float* logits_want = nullptr;       // [want_cap][vocab] logits of the places asked for in a prefill call, made on first use
    int want_cap = 0;
    uint32_t *rows_tok = nullptr, *rows_next = nullptr, *rows_pos = nullptr, *rows_out = nullptr;  // device; rows_out [steps][rows]
    size_t rows_out_cap = 0;
    void** rows_ptrs = nullptr;         // device [n_layers][2][batch_cap] per-row state pointers
    uint8_t* h_rows = nullptr;          // pinned staging for tokens, positions, pointers and results
    size_t h_rows_bytes = 0;

    wick_cuda_model();
    ~wick_cuda_model();
};

namespace wick {

template <class T>
int32_t dev_alloc(wick_cuda_model* m, T** out, size_t count) {
    void* p = nullptr;
    size_t bytes = std::max<size_t>(count * sizeof(T), 256);
    CU_TRY(cudaMalloc(&p, bytes));
    m->allocs.push_back(p);
    m->bytes += bytes;
    *out = (T*)p;
    return WICK_CUDA_OK;
}

// Per-category device timers of the prefill pipeline: the kernels enqueued since the previous mark belong to `cat`.
enum ProfCat { PC_EMBED = 0, PC_NORM_QUANT, PC_GEMM, PC_SHORTCONV, PC_QK_ROPE_KV, PC_ATTENTION, PC_ACT_QUANT, PC_LOGITS, PC_RECURRENCE };
void prof_begin(wick_cuda_model* m);
void prof_mark(wick_cuda_model* m, int cat);

}  // namespace wick
