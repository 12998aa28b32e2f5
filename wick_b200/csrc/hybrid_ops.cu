// Operator entry points of the kernels behind config.json models (include/wick_cuda.h): device pointers in, asynchronous on
// the caller's stream, arguments checked here so that a bad call is an error code and not a fault.
#include "model_internal.cuh"
#include "hybrid_kernels.cuh"
#include "latent_kernels.cuh"
#include "memory_kernels.cuh"

using namespace wick;

namespace {

struct Scratch {  // stream-ordered temporary
    void* p = nullptr;
    cudaStream_t st = nullptr;
    ~Scratch() {
        if (p) cudaFreeAsync(p, st);
    }
    cudaError_t get(cudaStream_t s, size_t bytes) {
        st = s;
        return cudaMallocAsync(&p, std::max<size_t>(bytes, 256), s);
    }
};

bool act_type(int32_t compute, bool* bf16) {
    *bf16 = compute != WICK_CUDA_COMPUTE_F32;
    return compute == WICK_CUDA_COMPUTE_F32 || compute == WICK_CUDA_COMPUTE_BF16;
}
bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

extern "C" {

int32_t wick_cuda_dense(int32_t compute, const void* w_dev, const void* w_up_dev, uint32_t m, uint32_t k, uint32_t ldw, const void* x_dev,
                        uint32_t ldx, uint32_t n, void* y_dev, uint32_t ldy, int32_t y_f32, int32_t activation, float softcap, int32_t path,
                        void* stream) {
    bool bf16;
    if (!w_dev || !x_dev || !y_dev || !act_type(compute, &bf16)) return fail(WICK_CUDA_ERR_BAD_ARG, "dense: NULL argument or unknown compute type");
    const uint32_t k8 = (k + 7) / 8 * 8;
    if (!m || !k || ldw % 8 || ldx % 8 || ldw != k8 || ldx < k8 || ldy < m || !aligned16(w_dev) || !aligned16(x_dev) || (w_up_dev && !aligned16(w_up_dev)))
        return fail(WICK_CUDA_ERR_BAD_ARG, "dense: ldw must be k rounded up to 8, ldx a multiple of 8 and at least that, ldy >= m, 16-byte aligned bases");
    if (activation < ACT_RELU || activation > ACT_NONE) return fail(WICK_CUDA_ERR_BAD_ARG, "dense: unknown activation");
    if (n == 0) return WICK_CUDA_OK;
    if (path < 0 || path > 3 || (path == WICK_CUDA_DENSE_ROWS && n > (uint32_t)DENSE_ROWS_MAX) || (path == WICK_CUDA_DENSE_TENSOR && !bf16))
        return fail(WICK_CUDA_ERR_BAD_ARG, "dense: this path does not take these arguments");
    cudaStream_t st = (cudaStream_t)stream;
    Scratch err;
    CU_TRY(err.get(st, 4));
    CU_TRY(cudaMemsetAsync(err.p, 0, 4, st));
    DenseCall c;
    c.job[0].w.w = (const __nv_bfloat16*)w_dev;
    c.job[0].w.m = (int)m; c.job[0].w.k = (int)k; c.job[0].w.ld = (int)ldw;
    c.job[0].x = x_dev; c.job[0].ldx = (int)ldx; c.job[0].y = y_dev; c.job[0].ldy = (int)ldy;
    c.n = (int)n;
    c.job[0].f32 = y_f32 != 0 || !bf16;
    c.softcap = softcap;
    c.act = (Activation)activation;
    c.err = (uint32_t*)err.p;
    if (w_up_dev) {
        c.count = 2;
        c.gated = true;
        c.job[1] = c.job[0];
        c.job[1].w.w = (const __nv_bfloat16*)w_up_dev;
    }
    if (path == WICK_CUDA_DENSE_ROWS) launch_dense_rows(st, bf16, c);
    else if (path == WICK_CUDA_DENSE_F32) launch_dense_simt(st, bf16, c);
    else if (path == WICK_CUDA_DENSE_TENSOR) CU_TRY(launch_dense_tc(st, c));
    else CU_TRY(launch_dense(st, bf16, c));
    CU_TRY(cudaGetLastError());
    uint32_t h = 0;
    CU_TRY(cudaMemcpyAsync(&h, err.p, 4, cudaMemcpyDeviceToHost, st));
    CU_TRY(cudaStreamSynchronize(st));
    if (h) return fail(WICK_CUDA_ERR_TIMEOUT, "dense: a bounded wait expired (code " + std::to_string(h) + ")");
    return WICK_CUDA_OK;
}

int32_t wick_cuda_hyper_norm(int32_t compute, float* x_dev, uint32_t n, uint32_t streams, uint32_t width, const float* y_dev, const float* mix_dev,
                             const float* out_dev, const float* in_dev, const float* gain_dev, float eps, void* h_dev, uint32_t ldh, void* stream) {
    bool bf16;
    if (!x_dev || !gain_dev || !h_dev || !act_type(compute, &bf16) || (y_dev && (!mix_dev || !out_dev)))
        return fail(WICK_CUDA_ERR_BAD_ARG, "hyper_norm: NULL argument or unknown compute type");
    if (!streams || streams > (uint32_t)HYPER_MAX_STREAMS || !width || width > 48 * 1024 || ldh < width || ldh % 8 || !aligned16(x_dev) || !aligned16(h_dev))
        return fail(WICK_CUDA_ERR_BAD_ARG, "hyper_norm: 1 .. 16 streams, width <= 49152, ldh a multiple of 8 and >= width, 16-byte aligned bases");
    HyperArgs a;
    a.x = x_dev;
    a.y = y_dev; a.ldy = (int)width; a.mix = mix_dev; a.out = out_dev; a.in = in_dev; a.gain = gain_dev;
    a.eps = eps; a.h = h_dev; a.ldh = (int)ldh; a.n = (int)n; a.S = (int)streams; a.W = (int)width;
    launch_hyper_norm((cudaStream_t)stream, bf16, a);
    CU_TRY(cudaGetLastError());
    return WICK_CUDA_OK;
}

int32_t wick_cuda_mix_attention(int32_t compute, void* qkv_dev, uint32_t ld, uint32_t n, uint32_t start_pos, void* k_cache_dev, void* v_cache_dev,
                                uint32_t max_seq, const float* talk_dev, const float* bias_dev, uint32_t heads, uint32_t kv_heads, uint32_t dim,
                                uint32_t vdim, float scale, float eps, uint32_t size, uint32_t keep_first, void* out_dev, uint32_t ldo, void* stream) {
    bool bf16;
    if (!qkv_dev || !k_cache_dev || !v_cache_dev || !out_dev || !act_type(compute, &bf16))
        return fail(WICK_CUDA_ERR_BAD_ARG, "mix_attention: NULL argument or unknown compute type");
    MixAttnShape s;
    s.heads = (int)heads; s.kv_heads = (int)kv_heads; s.dim = (int)dim; s.vdim = (int)vdim; s.scale = scale; s.eps = eps;
    s.size = (int)size; s.keep_first = (int)keep_first; s.talk = talk_dev; s.bias = bias_dev;
    if (!heads || !kv_heads || heads % kv_heads || !dim || !vdim || ld % 8 || ldo % 8 || ld < heads * dim + kv_heads * (dim + vdim) || ldo < heads * vdim ||
        (uint64_t)start_pos + n > max_seq || !aligned16(qkv_dev) || !aligned16(k_cache_dev) || !aligned16(v_cache_dev) || !aligned16(out_dev) ||
        !mix_attn_supported(s))
        return fail(WICK_CUDA_ERR_BAD_ARG, "mix_attention: inconsistent sizes");
    if (n == 0) return WICK_CUDA_OK;
    cudaStream_t st = (cudaStream_t)stream;
    Scratch partial, fold, err;
    size_t pf = 0, fb = 0;
    mix_attn_scratch(s, bf16, (int)n, &pf, &fb);
    CU_TRY(partial.get(st, pf * 4));
    if (fb) CU_TRY(fold.get(st, fb));
    CU_TRY(err.get(st, 4));
    CU_TRY(cudaMemsetAsync(err.p, 0, 4, st));
    RowState rs;
    rs.s0 = k_cache_dev; rs.s1 = v_cache_dev; rs.start_pos = (int)start_pos;
    MixAttnScratch sc;
    sc.partial = (float*)partial.p; sc.fold = fold.p; sc.err = (uint32_t*)err.p;
    launch_qk_rms_append(st, bf16, qkv_dev, (int)ld, (int)n, s, rs, sc);
    CU_TRY(launch_mix_attn(st, bf16, qkv_dev, (int)ld, (int)n, s, rs, out_dev, (int)ldo, sc, (int)max_seq));
    uint32_t h = 0;
    CU_TRY(cudaMemcpyAsync(&h, err.p, 4, cudaMemcpyDeviceToHost, st));
    CU_TRY(cudaStreamSynchronize(st));
    if (h) return fail(WICK_CUDA_ERR_TIMEOUT, "mix_attention: a bounded wait expired (code " + std::to_string(h) + ")");
    return WICK_CUDA_OK;
}

int32_t wick_cuda_channel_delta(int32_t compute, const void* proj_dev, uint32_t ldp, uint32_t off_beta, const float* decay_dev, const float* gate_dev,
                                const float* conv_w_dev, const float* a_log_dev, const float* dt_bias_dev, const float* norm_dev, uint32_t n,
                                uint32_t heads, uint32_t kv_heads, uint32_t dim, uint32_t vdim, uint32_t taps, float eps, float* state_dev,
                                float* conv_state_dev, void* out_dev, uint32_t ldo, void* stream) {
    bool bf16;
    if (!proj_dev || !decay_dev || !gate_dev || !conv_w_dev || !a_log_dev || !dt_bias_dev || !norm_dev || !state_dev || !out_dev ||
        !act_type(compute, &bf16) || (taps > 1 && !conv_state_dev))
        return fail(WICK_CUDA_ERR_BAD_ARG, "channel_delta: NULL argument or unknown compute type");
    DeltaShape s;
    s.heads = (int)heads; s.kv_heads = (int)kv_heads; s.dim = (int)dim; s.vdim = (int)vdim; s.taps = (int)taps; s.eps = eps;
    if (!heads || !kv_heads || heads % kv_heads || !dim || dim > (uint32_t)DELTA_MAX_DIM || !vdim || !taps || taps > (uint32_t)DELTA_MAX_TAPS ||
        off_beta < (uint32_t)s.channels() || ldp < off_beta + heads || ldo < heads * vdim || !aligned16(state_dev))
        return fail(WICK_CUDA_ERR_BAD_ARG, "channel_delta: inconsistent sizes");
    if (n == 0) return WICK_CUDA_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const size_t qf = (size_t)n * kv_heads * s.dimp(), gf = (size_t)n * heads * s.dimp(), vf = round_up((int)(heads * vdim), 4) * (size_t)n;
    const size_t bf = round_up((int)heads, 4) * (size_t)n;
    Scratch work;
    CU_TRY(work.get(st, (2 * qf + gf + 2 * vf + 2 * bf + delta_record_floats(s, (int)n)) * 4));
    DeltaWork w;
    w.q = (float*)work.p; w.k = w.q + qf; w.g = w.k + qf; w.v = w.g + gf; w.o = w.v + vf; w.beta = w.o + vf; w.kq = w.beta + bf; w.rec = w.kq + bf;
    RowState rs;
    rs.s0 = state_dev; rs.s1 = conv_state_dev;
    DeltaPrepArgs a;
    a.p = proj_dev; a.ldp = (int)ldp; a.off_b = (int)off_beta; a.a = decay_dev; a.lda = (int)(heads * dim);
    a.conv_w = conv_w_dev; a.A_log = a_log_dev; a.dt_bias = dt_bias_dev; a.n = (int)n;
    launch_delta_prep(st, bf16, a, s, rs, w);
    launch_delta_scan(st, (int)n, s, rs, w);
    launch_gated_head_norm(st, bf16, (int)n, s.heads, s.vdim, s.eps, w.o, norm_dev, 0, gate_dev, true, (int)(heads * vdim), out_dev, (int)ldo);
    CU_TRY(cudaGetLastError());
    return WICK_CUDA_OK;
}

int32_t wick_cuda_residual_norm(int32_t compute, float* x_dev, uint32_t n, uint32_t width, const float* y_dev, uint32_t y_parts, const int32_t* y_rows_dev,
                                float y_scale, const float* post_dev, const float* shift_dev, const float* gain_dev, const float* x0_dev, float eps,
                                void* h_dev, uint32_t ldh, uint32_t h_parts, const int32_t* h_rows_dev, void* stream) {
    bool bf16;
    if (!x_dev || !h_dev || !act_type(compute, &bf16) || (!gain_dev && !x0_dev) || (y_dev && !post_dev == !shift_dev) || (y_dev && !y_parts) || (h_rows_dev && !h_parts))
        return fail(WICK_CUDA_ERR_BAD_ARG, "residual_norm: missing argument or unknown compute type");
    if (!width || width > 48 * 1024 || ldh < (gain_dev ? 1u : 2u) * width || ldh % 8 || !aligned16(x_dev) || !aligned16(h_dev) || (y_dev && !aligned16(y_dev)))
        return fail(WICK_CUDA_ERR_BAD_ARG, "residual_norm: width <= 49152, ldh a multiple of 8 and at least the row, 16-byte aligned bases");
    ResidualArgs a;
    a.x = x_dev; a.n = (int)n; a.W = (int)width; a.y = y_dev; a.ldy = (int)width; a.y_parts = (int)y_parts; a.y_rows = y_rows_dev; a.y_scale = y_scale;
    a.post = post_dev; a.shift = shift_dev; a.gain = gain_dev; a.frames = x0_dev; a.eps = eps; a.h = h_dev; a.ldh = (int)ldh;
    if (h_rows_dev) {
        a.h_rows = h_rows_dev;
        a.h_parts = (int)h_parts;
    }
    launch_residual_norm((cudaStream_t)stream, bf16, a);
    CU_TRY(cudaGetLastError());
    return WICK_CUDA_OK;
}

int32_t wick_cuda_latent_attention(int32_t compute, void* p_dev, uint32_t ldp, uint32_t n, uint32_t start_pos, void* cache_dev, uint32_t max_seq,
                                   const void* uq_dev, const void* uk_t_dev, const void* uv_dev, const void* ukv_dev, const float* sink_dev,
                                   const float* q_norm_dev, const float* kv_norm_dev, const float* rope_dev, uint32_t heads, uint32_t dim,
                                   uint32_t rot_dim, uint32_t rot_dims, uint32_t vdim, uint32_t q_rank, uint32_t kv_rank, uint32_t size, float scale,
                                   float eps, int32_t form, void* out_dev, uint32_t ldo, void* stream) {
    bool bf16;
    if (!p_dev || !cache_dev || !uq_dev || !uk_t_dev || !uv_dev || !sink_dev || !q_norm_dev || !kv_norm_dev || !rope_dev || !out_dev || !act_type(compute, &bf16))
        return fail(WICK_CUDA_ERR_BAD_ARG, "latent_attention: NULL argument or unknown compute type");
    LatentShape s;
    s.heads = (int)heads; s.dim = (int)dim; s.rot_dim = (int)rot_dim; s.rot_dims = (int)rot_dims; s.vdim = (int)vdim; s.q_rank = (int)q_rank;
    s.kv_rank = (int)kv_rank; s.size = (int)size; s.scale = scale; s.eps = eps; s.sink = sink_dev; s.rope = (const float2*)rope_dev;
    s.q_norm = q_norm_dev; s.kv_norm = kv_norm_dev;
    if (!heads || !dim || !rot_dim || rot_dims % 2 || rot_dims > rot_dim || !vdim || !q_rank || !kv_rank || ldp % 8 || ldo % 8 ||
        ldp < (uint32_t)s.off_kv() + kv_rank + rot_dim || ldo < heads * vdim || (uint64_t)start_pos + n > max_seq || !aligned16(p_dev) || !aligned16(cache_dev) ||
        !aligned16(uq_dev) || !aligned16(uk_t_dev) || !aligned16(uv_dev) || !aligned16(out_dev) || !latent_supported(s))
        return fail(WICK_CUDA_ERR_BAD_ARG, "latent_attention: inconsistent sizes");
    const bool prompt = form == WICK_CUDA_LATENT_PROMPT || (form == WICK_CUDA_LATENT_AUTO && bf16 && ukv_dev && n >= (uint32_t)LATENT_TC_MIN_ROWS && latent_tc_supported(s));
    if (form < WICK_CUDA_LATENT_AUTO || form > WICK_CUDA_LATENT_PROMPT || (prompt && (!bf16 || !ukv_dev || !aligned16(ukv_dev) || !latent_tc_supported(s))))
        return fail(WICK_CUDA_ERR_BAD_ARG, "latent_attention: this form does not take these arguments");
    if (n == 0) return WICK_CUDA_OK;
    cudaStream_t st = (cudaStream_t)stream;
    const size_t ab = bf16 ? 2 : 4, ldq = (size_t)heads * s.q_pitch(), ldc = (size_t)heads * s.ldc(), ldl = (size_t)heads * s.off_rot();
    Scratch q, qc, oc, kv, partial, err;
    CU_TRY(q.get(st, n * ldq * ab));
    CU_TRY(qc.get(st, n * ldc * ab));
    CU_TRY(cudaMemsetAsync(qc.p, 0, n * ldc * ab, st));
    CU_TRY(oc.get(st, n * ldl * ab));
    CU_TRY(partial.get(st, latent_scratch(s, bf16, (int)n, (int)max_seq) * 4));
    CU_TRY(err.get(st, 4));
    CU_TRY(cudaMemsetAsync(err.p, 0, 4, st));
    RowState rs;
    rs.s0 = cache_dev;
    rs.start_pos = (int)start_pos;
    auto weight = [](const void* w, int m, int k) {
        DenseWeight d;
        d.w = (const __nv_bfloat16*)w; d.m = m; d.k = k; d.ld = round_up(k, 8);
        return d;
    };
    auto dense = [&](const DenseWeight& w, const void* x, size_t ldx, void* y, size_t ldy, int block, int x_step, int y_step) {
        DenseCall c;
        c.job[0].w = w; c.job[0].x = x; c.job[0].ldx = (int)ldx; c.job[0].y = y; c.job[0].ldy = (int)ldy;
        c.n = (int)n;
        c.err = (uint32_t*)err.p;
        c.blocks.rows = block; c.blocks.x_step = x_step; c.blocks.y_step = y_step;
        return launch_dense(st, bf16, c);
    };
    launch_latent_append(st, bf16, p_dev, (int)ldp, (int)n, s, rs);
    CU_TRY(dense(weight(uq_dev, (int)ldq, s.q_rank), p_dev, ldp, q.p, ldq, 0, 0, 0));
    if (prompt) {
        CU_TRY(kv.get(st, (size_t)(start_pos + n) * latent_tc_cols(s) * 2));
        CU_TRY(launch_latent_kv(st, (int)n, s, rs, weight(ukv_dev, latent_tc_cols(s), s.kv_rank), kv.p, (uint32_t*)err.p));
        CU_TRY(launch_latent_attn_tc(st, q.p, (int)ldq, (int)n, s, rs, kv.p, out_dev, (int)ldo, (uint32_t*)err.p));
    } else {
        CU_TRY(dense(weight(uk_t_dev, s.heads * s.kv_rank, s.dim), q.p, ldq, qc.p, ldc, s.kv_rank, s.q_pitch(), s.ldc()));
        LatentScratch sc;
        sc.partial = (float*)partial.p;
        sc.err = (uint32_t*)err.p;
        CU_TRY(launch_latent_attn(st, bf16, qc.p, q.p, (int)ldq, (int)n, s, rs, oc.p, s.off_rot(), sc, (int)max_seq));
        CU_TRY(dense(weight(uv_dev, s.heads * s.vdim, s.kv_rank), oc.p, ldl, out_dev, ldo, s.vdim, s.off_rot(), s.vdim));
    }
    uint32_t h = 0;
    CU_TRY(cudaMemcpyAsync(&h, err.p, 4, cudaMemcpyDeviceToHost, st));
    CU_TRY(cudaStreamSynchronize(st));
    if (h) return fail(WICK_CUDA_ERR_TIMEOUT, "latent_attention: a bounded wait expired (code " + std::to_string(h) + ")");
    return WICK_CUDA_OK;
}

int32_t wick_cuda_matrix_memory(int32_t compute, const void* p_dev, uint32_t ldp, const float* gates_dev, uint32_t ldi, uint32_t n, uint32_t heads, uint32_t dim,
                                uint32_t vdim, float cap, float eps, const float* i_bias_dev, const float* f_bias_dev, const float* norm_dev,
                                float* state_dev, float* m_dev, int32_t step, void* out_dev, uint32_t ldo, void* stream) {
    bool bf16;
    if (!p_dev || !gates_dev || !i_bias_dev || !f_bias_dev || !norm_dev || !state_dev || !m_dev || !out_dev || !act_type(compute, &bf16))
        return fail(WICK_CUDA_ERR_BAD_ARG, "matrix_memory: NULL argument or unknown compute type");
    MemoryShape s;
    s.heads = (int)heads; s.dim = (int)dim; s.vdim = (int)vdim; s.cap = cap; s.eps = eps; s.i_bias = i_bias_dev; s.f_bias = f_bias_dev; s.norm = norm_dev;
    if (!heads || !dim || !vdim || dim > (uint32_t)MEMORY_MAX_DIM || vdim > (uint32_t)MEMORY_MAX_DIM || !(cap > 0.0f) || ldp % 8 ||
        ldp < 2 * heads * (dim + vdim) || ldi < 2 * heads || ldo < heads * vdim || !aligned16(p_dev) || !aligned16(state_dev) || n > (1u << 15))
        return fail(WICK_CUDA_ERR_BAD_ARG, "matrix_memory: inconsistent sizes");
    if (n == 0) return WICK_CUDA_OK;
    cudaStream_t st = (cudaStream_t)stream;
    MemoryArgs a;
    a.p = p_dev; a.ldp = (int)ldp; a.gates = gates_dev; a.ldi = (int)ldi;
    RowState rs;
    rs.s0 = state_dev;
    rs.s1 = m_dev;
    if (step) {  // token by token, each a decode step
        a.n = 1;
        for (uint32_t j = 0; j < n; j++) {
            launch_memory_step(st, bf16, a, s, rs, out_dev, (int)ldo);
            a.p = (const uint8_t*)a.p + (size_t)ldp * (bf16 ? 2 : 4);
            a.gates += ldi;
            out_dev = (uint8_t*)out_dev + (size_t)ldo * (bf16 ? 2 : 4);
        }
        CU_TRY(cudaGetLastError());
        return WICK_CUDA_OK;
    }
    a.n = (int)n;
    Scratch work, err;
    CU_TRY(work.get(st, memory_work_bytes(s, bf16, (int)n)));
    CU_TRY(err.get(st, 4));
    CU_TRY(cudaMemsetAsync(err.p, 0, 4, st));
    CU_TRY(launch_memory_prompt(st, bf16, a, s, rs, memory_work(s, bf16, (int)n, work.p, (uint32_t*)err.p), out_dev, (int)ldo));
    uint32_t h = 0;
    CU_TRY(cudaMemcpyAsync(&h, err.p, 4, cudaMemcpyDeviceToHost, st));
    CU_TRY(cudaStreamSynchronize(st));
    if (h) return fail(WICK_CUDA_ERR_TIMEOUT, "matrix_memory: a bounded wait expired (code " + std::to_string(h) + ")");
    return WICK_CUDA_OK;
}

}  // extern "C"
