// Models described by a folder (config.json + model.safetensors): a list of layers, each with a mixer and an optional
// feed-forward, over hyper-connection streams or over one residual stream with norms around the sublayers.  hybrid_load.cu
// reads the folder, hybrid.cu drives the steps; wick_cuda.cu serves the models like every other architecture (slots, batching,
// sampling, graphs).
#pragma once
#include <string>
#include <vector>

#include "hybrid_kernels.cuh"
#include "latent_kernels.cuh"
#include "memory_kernels.cuh"
#include "model_internal.cuh"
#include "safetensors.hpp"

namespace wick {

// What stands around one sublayer (device f32).  Streams: scalar gain and hyper-connection weights.  Single residual: the
// gains in front of and behind the sublayer [W].
struct SublayerWeights {
    float *in = nullptr, *out = nullptr, *mix = nullptr, *gain = nullptr, *post = nullptr;
};

enum MixerKind { MIX_ATTENTION, MIX_DELTA, MIX_LATENT, MIX_MEMORY };
enum FeedForwardKind { FF_NONE, FF_GATED, FF_PLAIN, FF_EXPERTS };

struct HybridLayer {
    std::string type;  // the mixer's name in config.json
    MixerKind kind = MIX_ATTENTION;
    SublayerWeights sub1, sub2;
    // MIX_ATTENTION: proj = q | k | v rows.  MIX_DELTA: proj = q | k | v | beta | decay down | gate down rows, the last
    // three each at a multiple of 8.  MIX_LATENT: proj = q down | k/v down rows, the second at off_kv.  MIX_MEMORY: proj = q | k |
    // v | output gate rows, gates = input gate | forget gate rows.
    DenseWeight proj, o;
    MixAttnShape attn;
    DeltaShape delta;
    LatentShape latent;
    MemoryShape memory;
    int off_b = 0, off_a1 = 0, off_g1 = 0;
    DenseWeight a2, g2;  // low-rank up projections of the decay and the output gate
    float *conv_w = nullptr, *A_log = nullptr, *dt_bias = nullptr, *out_norm = nullptr;
    DenseWeight uq, uk_t, uv;  // latent: queries; per head to the latent's side [kv_rank][dim]; values [vdim][kv_rank]
    DenseWeight ukv;           // keys and values of the prompt form (empty where that does not apply)
    DenseWeight gates;
    FeedForwardKind ff = FF_NONE;
    Activation act = ACT_RELU;
    DenseWeight gate, up, down;  // FF_EXPERTS: of all experts, stacked
    int experts = 0, top = 1, route = -1;  // route: index into HybridModel::routes
    const int* table = nullptr;
};

// One execution of a layer within a step.  A layer of a repeated group runs once per pass, with state of its own every time.
struct LayerRun {
    int layer = 0;
    int enter_pass = -1;  // >= 0: the layer opens this pass of the repeated group
};

// Layers start .. stop - 1 run `times` times; in front of every pass x <- in [x; x0] + step[pass], x0 the embedding output.
struct HybridLoop {
    int start = 0, stop = 0, times = 0;
    DenseWeight in;
    float* step = nullptr;  // [times][W]
    explicit operator bool() const { return times > 0; }
};

struct HybridModel {
    bool bf16 = true;
    int width = 0, streams = 0;  // streams: 0 = one residual stream with norms before and after the sublayers
    float eps = 0.0f, embed_scale = 1.0f, logit_scale = 1.0f, softcap = 0.0f;
    std::vector<HybridLayer> layers;
    std::vector<LayerRun> runs;  // wick_cuda_model::layers[r] holds the state of run r
    HybridLoop loop;
    std::vector<RouteJob> routes;  // one per layer with experts
    int max_top = 1;
    DenseWeight embed, head;
    float* final_gain = nullptr;
    std::vector<std::pair<std::vector<double>, float2*>> rope_tables;  // by their parameters
    // scratch for max_chunk rows (row pitches: ld*)
    int ldh = 0, ldp = 0, ldm = 0, ldf = 0, ldw = 0, lda = 0, ldg = 0, ldq = 0, ldc = 0, ldi = 0, ldcat = 0;
    float* x = nullptr;        // [rows][streams][width]
    void* h = nullptr;         // act [rows (x max_top)][ldh] normed sublayer input
    void* cat = nullptr;       // act [rows][ldcat] [x | x0] in front of a pass
    void* proj = nullptr;      // act [rows][ldp] mixer projections
    void* mixed = nullptr;     // act [rows][ldm] mixer output before W_o
    void* ff = nullptr;        // act [rows (x max_top)][ldf] activated feed-forward
    float* y = nullptr;        // [rows (x max_top)][ldw] sublayer output
    float *a = nullptr, *gate = nullptr;  // [rows][lda] decay projection, [rows][ldg] gate projection
    void *q = nullptr, *qc = nullptr, *oc = nullptr;  // act [rows][ldq], [rows][ldc]: latent queries, on the latent's side, read-outs
    void* kv = nullptr;        // act: keys and values that a portion sees
    float* gates = nullptr;    // [rows][ldi] input and forget gate logits
    LatentScratch latent;
    MixAttnScratch attn;
    DeltaWork work;
    void* memory = nullptr;    // work memory of the matrix memory
    int* rows_dev = nullptr;   // rows of a chunk that get logits
    int* h_rows = nullptr;     // pinned staging of the same
    ~HybridModel();
};

extern const ModelFamily HYBRID_FAMILY;
int32_t nositar_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute);
int32_t novorax_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute);
int32_t hybrid_alloc_scratch(wick_cuda_model* m);  // after the layers are known
const char* hybrid_layer_type(const wick_cuda_model* m, int layer);
int hybrid_first_run(const wick_cuda_model* m, int layer);  // the run whose state stands for a layer

// wick_cuda.cu
void choose_max_chunk(wick_cuda_model* m);
void enqueue_step_end(wick_cuda_model* m, bool greedy);

}  // namespace wick
