// Models described by a folder (config.json + model.safetensors): a list of layers, each with a mixer and an optional
// feed-forward, over hyper-connection streams.  hybrid.cu parses, loads and drives them; wick_cuda.cu serves them like every
// other architecture (slots, batching, sampling, graphs).
#pragma once
#include <string>
#include <vector>

#include "hybrid_kernels.cuh"
#include "model_internal.cuh"
#include "safetensors.hpp"

namespace wick {

// One sublayer's norm gain and hyper-connection weights (device f32).
struct HyperWeights {
    float *in = nullptr, *out = nullptr, *mix = nullptr, *gain = nullptr;
};

enum MixerKind { MIX_ATTENTION, MIX_DELTA };

struct HybridLayer {
    std::string type;  // the mixer's name in config.json
    MixerKind kind = MIX_ATTENTION;
    HyperWeights hc1, hc2;
    // MIX_ATTENTION: proj = q | k | v rows.  MIX_DELTA: proj = q | k | v | beta | decay down | gate down rows, the last
    // three each at a multiple of 8.
    DenseWeight proj, o;
    MixAttnShape attn;
    DeltaShape delta;
    int off_b = 0, off_a1 = 0, off_g1 = 0;
    DenseWeight a2, g2;  // low-rank up projections of the decay and the output gate
    float *conv_w = nullptr, *A_log = nullptr, *dt_bias = nullptr, *out_norm = nullptr;
    bool has_ff = false;
    Activation act = ACT_RELU;
    DenseWeight gate, up, down;
};

struct HybridModel {
    bool bf16 = true;
    int width = 0, streams = 1;
    float eps = 0.0f, embed_scale = 1.0f, softcap = 0.0f;
    std::vector<HybridLayer> layers;
    DenseWeight embed, head;
    float* final_gain = nullptr;
    // scratch for max_chunk rows (row pitches: ld*)
    int ldh = 0, ldp = 0, ldm = 0, ldf = 0, ldw = 0, lda = 0, ldg = 0;
    float* x = nullptr;        // [rows][streams][width]
    void* h = nullptr;         // act [rows][ldh] normed sublayer input
    void* proj = nullptr;      // act [rows][ldp] mixer projections
    void* mixed = nullptr;     // act [rows][ldm] mixer output before W_o
    void* ff = nullptr;        // act [rows][ldf] activated feed-forward
    float* y = nullptr;        // [rows][ldw] sublayer output
    float *a = nullptr, *gate = nullptr;  // [rows][lda] decay projection, [rows][ldg] gate projection
    MixAttnScratch attn;
    DeltaWork work;
    int* rows_dev = nullptr;   // rows of a chunk that get logits
    int* h_rows = nullptr;     // pinned staging of the same
    ~HybridModel();
};

extern const ModelFamily HYBRID_FAMILY;
int32_t nositar_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute);
const char* hybrid_layer_type(const wick_cuda_model* m, int layer);

// wick_cuda.cu
void choose_max_chunk(wick_cuda_model* m);
void enqueue_step_end(wick_cuda_model* m, bool greedy);

}  // namespace wick
