// Steps of the models described by config.json (hybrid.cuh): enqueueing prompt chunks and decode steps.
//
// A step alternates one kernel that moves the residual (k_hyper_norm over streams, k_residual_norm over a single one) with the
// sublayer's own kernels:
//   attention   proj GEMM -> qk norm + cache append -> attention -> W_o GEMM
//   delta       proj GEMM -> a2 | g2 GEMM -> convolutions, decays -> recurrence -> gated norm -> W_o GEMM
//   latent      proj GEMM -> norms + cache append -> query GEMM -> to the latent's side -> attention -> values -> W_o GEMM
//   memory      proj | gates GEMM -> recurrence -> gated norm -> W_o GEMM
//   feed-forward  gate | up GEMM with the activation in its epilogue -> down GEMM; with experts the rows in front of them are
//               written in the experts' order, and the next residual kernel collects their outputs
// The last kernel of a sublayer leaves y in f32; the next residual kernel folds it in.
#include "hybrid.cuh"

#include <cstring>

namespace wick {

HybridModel::~HybridModel() {
    if (h_rows) cudaFreeHost(h_rows);
}

const char* hybrid_layer_type(const wick_cuda_model* m, int layer) {
    return layer < (int)m->hybrid->layers.size() ? m->hybrid->layers[layer].type.c_str() : "";
}

int hybrid_first_run(const wick_cuda_model* m, int layer) {
    const std::vector<LayerRun>& runs = m->hybrid->runs;
    for (size_t r = 0; r < runs.size(); r++)
        if (runs[r].layer == layer) return (int)r;
    return 0;
}

namespace {

// Where the embedding rows of a step come from.
struct StepInput {
    const uint32_t* tokens = nullptr;
    const DecodeCtl* ctl = nullptr;  // the single token of a decode step
    const float* frames = nullptr;
};

// The output of the sublayer that is not in the residual yet.
struct Pending {
    const SublayerWeights* sub = nullptr;
    const float* shift = nullptr;    // the residual is replaced by y + shift
    const int* rows = nullptr;       // y of token j: the sum of rows[j * parts ..] times scale
    int parts = 1;
    float scale = 1.0f;
};

struct Step {
    wick_cuda_model* m;
    HybridModel& hm;
    int n;
    bool timed;  // prefill: feed the per-category timers
    StepInput in;
    bool first = true, has_pending = false;
    Pending pending;

    Step(wick_cuda_model* m, int n, bool timed) : m(m), hm(*m->hybrid), n(n), timed(timed) {}
    void mark(int cat) {
        if (timed) prof_mark(m, cat);
    }
    bool few() const { return n <= DENSE_ROWS_MAX; }
    void leave(const Pending& p) {
        pending = p;
        has_pending = true;
    }

    HyperArgs stream_args() {
        HyperArgs a;
        if (first) {
            a.tokens = in.tokens;
            a.ctl = in.ctl;
            a.frames = in.frames;
            if (!in.frames) {
                a.embed = hm.embed.w;
                a.ld_embed = hm.embed.ld;
                a.embed_scale = hm.embed_scale;
            }
        }
        a.x = hm.x;
        a.S = hm.streams;
        a.W = hm.width;
        a.eps = hm.eps;
        a.h = hm.h;
        a.ldh = hm.ldh;
        a.n = n;
        if (has_pending) {
            a.y = hm.y;
            a.ldy = hm.ldw;
            a.mix = pending.sub->mix;
            a.out = pending.sub->out;
        }
        return a;
    }
    ResidualArgs residual_args() {
        ResidualArgs a;
        a.tokens = in.tokens;
        a.ctl = in.ctl;
        a.frames = in.frames;
        if (!in.frames) {
            a.embed = hm.embed.w;
            a.ld_embed = hm.embed.ld;
        }
        a.init = first;
        a.x = hm.x;
        a.W = hm.width;
        a.eps = hm.eps;
        a.h = hm.h;
        a.ldh = hm.ldh;
        a.n = n;
        if (has_pending) {
            a.y = hm.y;
            a.ldy = hm.ldw;
            a.y_rows = pending.rows;
            a.y_parts = pending.parts;
            a.y_scale = pending.scale;
            if (pending.shift) a.shift = pending.shift;
            else a.post = pending.sub->post;
        }
        return a;
    }
    // residual <- pending output; h <- norm of the sublayer's input.  With `route` the rows of h are in the experts' order.
    void enter(const SublayerWeights& w, const RouteJob* route = nullptr) {
        if (hm.streams) {
            HyperArgs a = stream_args();
            a.in = w.in;
            a.gain = w.gain;
            launch_hyper_norm(m->stream, hm.bf16, a);
        } else {
            ResidualArgs a = residual_args();
            a.gain = w.gain;
            if (route) {
                a.h_rows = route->inv;
                a.h_parts = route->top;
            }
            launch_residual_norm(m->stream, hm.bf16, a);
        }
        first = has_pending = false;
        mark(PC_NORM_QUANT);
    }
    // x <- in [x; x0] + step[pass]
    int32_t enter_pass(int pass) {
        ResidualArgs a = residual_args();
        a.h = hm.cat;
        a.ldh = hm.ldcat;
        a.store_x = false;  // replaced by what follows
        launch_residual_norm(m->stream, hm.bf16, a);
        first = false;
        mark(PC_NORM_QUANT);
        W_TRY(dense(hm.loop.in, hm.cat, hm.ldcat, hm.y, hm.ldw, true));
        mark(PC_GEMM);
        Pending p;
        p.shift = hm.loop.step + (size_t)pass * hm.width;
        leave(p);
        return WICK_CUDA_OK;
    }
    DenseCall call(const DenseWeight& w, const void* x, int ldx, void* y, int ldy, bool f32) {
        DenseCall c;
        c.job[0].w = w; c.job[0].x = x; c.job[0].ldx = ldx; c.job[0].y = y; c.job[0].ldy = ldy; c.job[0].f32 = f32;
        c.n = n;
        c.err = m->tc_err;
        return c;
    }
    int32_t run(const DenseCall& c) {
        CU_TRY(launch_dense(m->stream, hm.bf16, c));
        return WICK_CUDA_OK;
    }
    int32_t dense(const DenseWeight& w, const void* x, int ldx, void* y, int ldy, bool f32) { return run(call(w, x, ldx, y, ldy, f32)); }
    int32_t blocks(const DenseWeight& w, int rows, const void* x, int ldx, int x_step, void* y, int ldy, int y_step) {
        DenseCall c = call(w, x, ldx, y, ldy, false);
        c.blocks.rows = rows;
        c.blocks.x_step = x_step;
        c.blocks.y_step = y_step;
        return run(c);
    }
    const void* act_at(const void* p, int col) const { return (const uint8_t*)p + (size_t)col * (hm.bf16 ? 2 : 4); }

    int32_t attention(const HybridLayer& L, const RowState& rs) {
        W_TRY(dense(L.proj, hm.h, hm.ldh, hm.proj, hm.ldp, false));
        mark(PC_GEMM);
        launch_qk_rms_append(m->stream, hm.bf16, hm.proj, hm.ldp, n, L.attn, rs, hm.attn);
        mark(PC_QK_ROPE_KV);
        CU_TRY(launch_mix_attn(m->stream, hm.bf16, hm.proj, hm.ldp, n, L.attn, rs, hm.mixed, hm.ldm, hm.attn, (int)m->cfg.max_seq_len));
        mark(PC_ATTENTION);
        return WICK_CUDA_OK;
    }
    int32_t delta(const HybridLayer& L, const RowState& rs) {
        cudaStream_t st = m->stream;
        W_TRY(dense(L.proj, hm.h, hm.ldh, hm.proj, hm.ldp, false));
        DenseCall c = call(L.a2, act_at(hm.proj, L.off_a1), hm.ldp, hm.a, hm.lda, true);
        c.count = 2;
        c.job[1].w = L.g2; c.job[1].x = act_at(hm.proj, L.off_g1); c.job[1].ldx = hm.ldp; c.job[1].y = hm.gate; c.job[1].ldy = hm.ldg; c.job[1].f32 = true;
        W_TRY(run(c));
        mark(PC_GEMM);
        DeltaPrepArgs a;
        a.p = hm.proj; a.ldp = hm.ldp; a.off_b = L.off_b; a.a = hm.a; a.lda = hm.lda;
        a.conv_w = L.conv_w; a.A_log = L.A_log; a.dt_bias = L.dt_bias; a.n = n;
        if (rs.separate()) {
            launch_delta_step(st, hm.bf16, a, L.delta, rs, L.out_norm, hm.gate, hm.ldg, hm.mixed, hm.ldm);
        } else {
            launch_delta_prep(st, hm.bf16, a, L.delta, rs, hm.work);
            mark(PC_SHORTCONV);
            launch_delta_scan(st, n, L.delta, rs, hm.work);
            launch_gated_head_norm(st, hm.bf16, n, L.delta.heads, L.delta.vdim, L.delta.eps, hm.work.o, L.out_norm, 0, hm.gate, true, hm.ldg, hm.mixed, hm.ldm);
        }
        mark(PC_RECURRENCE);
        return WICK_CUDA_OK;
    }
    int32_t latent(const HybridLayer& L, const RowState& rs) {
        const LatentShape& s = L.latent;
        W_TRY(dense(L.proj, hm.h, hm.ldh, hm.proj, hm.ldp, false));
        mark(PC_GEMM);
        launch_latent_append(m->stream, hm.bf16, hm.proj, hm.ldp, n, s, rs);
        mark(PC_QK_ROPE_KV);
        W_TRY(dense(L.uq, hm.proj, hm.ldp, hm.q, hm.ldq, false));
        if (L.ukv.w && !rs.separate() && n >= LATENT_TC_MIN_ROWS) {
            CU_TRY(launch_latent_kv(m->stream, n, s, rs, L.ukv, hm.kv, m->tc_err));
            mark(PC_GEMM);
            CU_TRY(launch_latent_attn_tc(m->stream, hm.q, hm.ldq, n, s, rs, hm.kv, hm.mixed, hm.ldm, m->tc_err));
            mark(PC_ATTENTION);
            return WICK_CUDA_OK;
        }
        W_TRY(blocks(L.uk_t, s.kv_rank, hm.q, hm.ldq, s.q_pitch(), hm.qc, s.heads * s.ldc(), s.ldc()));
        mark(PC_GEMM);
        CU_TRY(launch_latent_attn(m->stream, hm.bf16, hm.qc, hm.q, hm.ldq, n, s, rs, hm.oc, s.off_rot(), hm.latent, (int)m->cfg.max_seq_len));
        mark(PC_ATTENTION);
        W_TRY(blocks(L.uv, s.vdim, hm.oc, s.heads * s.off_rot(), s.off_rot(), hm.mixed, hm.ldm, s.vdim));
        return WICK_CUDA_OK;
    }
    int32_t memory(const HybridLayer& L, const RowState& rs) {
        DenseCall c = call(L.proj, hm.h, hm.ldh, hm.proj, hm.ldp, false);
        c.count = 2;
        c.job[1].w = L.gates; c.job[1].x = hm.h; c.job[1].ldx = hm.ldh; c.job[1].y = hm.gates; c.job[1].ldy = hm.ldi; c.job[1].f32 = true;
        W_TRY(run(c));
        mark(PC_GEMM);
        MemoryArgs a;
        a.p = hm.proj; a.ldp = hm.ldp; a.gates = hm.gates; a.ldi = hm.ldi; a.n = n;
        if (rs.separate()) launch_memory_step(m->stream, hm.bf16, a, L.memory, rs, hm.mixed, hm.ldm);
        else CU_TRY(launch_memory_prompt(m->stream, hm.bf16, a, L.memory, rs, memory_work(L.memory, hm.bf16, n, hm.memory, m->tc_err), hm.mixed, hm.ldm));
        mark(PC_RECURRENCE);
        return WICK_CUDA_OK;
    }
    int32_t feed_forward(const HybridLayer& L) {
        const RouteJob* route = L.ff == FF_EXPERTS && !few() ? &hm.routes[L.route] : nullptr;
        enter(L.sub2, route);
        DenseCall c = call(L.ff == FF_PLAIN ? L.up : L.gate, hm.h, hm.ldh, hm.ff, hm.ldf, false);
        DenseCall d = call(L.down, hm.ff, hm.ldf, hm.y, hm.ldw, true);
        Pending p;
        p.sub = &L.sub2;
        c.act = L.act;
        if (L.ff != FF_PLAIN) {
            c.gated = true;
            c.count = 2;
            c.job[1] = c.job[0];
            c.job[1].w = L.up;
        }
        if (L.ff == FF_EXPERTS) {
            DenseExperts& e = c.experts;
            e.count = L.experts;
            e.top = L.top;
            e.table = L.table;
            e.tokens = in.tokens;
            e.ctl = in.ctl;
            e.x_per_token = true;
            e.start = route ? route->start : nullptr;
            d.experts = e;
            d.experts.x_per_token = false;
            c.n = d.n = n * L.top;
            p.parts = L.top;
            p.scale = 1.0f / (float)L.top;
            p.rows = route ? route->inv : nullptr;
        }
        W_TRY(run(c));
        W_TRY(run(d));
        mark(PC_GEMM);
        leave(p);
        return WICK_CUDA_OK;
    }

    int32_t layer(const HybridLayer& L, const RowState& rs) {
        enter(L.sub1);
        switch (L.kind) {
            case MIX_ATTENTION: W_TRY(attention(L, rs)); break;
            case MIX_DELTA: W_TRY(delta(L, rs)); break;
            case MIX_LATENT: W_TRY(latent(L, rs)); break;
            case MIX_MEMORY: W_TRY(memory(L, rs)); break;
        }
        W_TRY(dense(L.o, hm.mixed, hm.ldm, hm.y, hm.ldw, true));
        mark(PC_GEMM);
        Pending p;
        p.sub = &L.sub1;
        leave(p);
        return L.ff != FF_NONE ? feed_forward(L) : WICK_CUDA_OK;
    }
    // all layers; state_of(run) says where the rows and the state of a run are
    template <class F>
    int32_t layers(F&& state_of) {
        if (!hm.routes.empty()) {
            if (in.frames) return fail(WICK_CUDA_ERR_BAD_ARG, "architecture " + m->arch + ": experts are chosen by token id, so embeddings alone are not an input");
            if (!few()) launch_route(m->stream, in.tokens, n, hm.routes.data(), (int)hm.routes.size());
        }
        for (size_t r = 0; r < hm.runs.size(); r++) {
            if (hm.runs[r].enter_pass >= 0) W_TRY(enter_pass(hm.runs[r].enter_pass));
            W_TRY(layer(hm.layers[hm.runs[r].layer], state_of(r)));
        }
        return WICK_CUDA_OK;
    }
    // final norm of `count` rows (row i: rows_dev[i], or i itself), then logits
    int32_t logits(int count, const int* rows_dev, float* normed, bool want, float* dst) {
        if (hm.streams) {
            HyperArgs a = stream_args();
            a.rows = rows_dev;
            a.store_x = false;
            a.gain = hm.final_gain;
            a.n = count;
            a.normed = normed;
            launch_hyper_norm(m->stream, hm.bf16, a);
        } else {
            ResidualArgs a = residual_args();
            a.rows = rows_dev;
            a.store_x = false;
            a.gain = hm.final_gain;
            a.n = count;
            a.normed = normed;
            launch_residual_norm(m->stream, hm.bf16, a);
        }
        if (want) {
            DenseCall c = call(hm.head, hm.h, hm.ldh, dst, (int)m->cfg.vocab_size, true);
            c.n = count;
            c.scale = hm.logit_scale;
            c.softcap = hm.softcap;
            W_TRY(run(c));
        }
        mark(PC_LOGITS);
        return WICK_CUDA_OK;
    }
};

int32_t hybrid_enqueue_decode(wick_cuda_model* m, bool greedy) {
    Step s(m, 1, false);
    s.in.ctl = m->ctl;
    W_TRY(s.layers([&](size_t r) {
        RowState rs;
        rs.s0 = m->layers[r].state[0];
        rs.s1 = m->layers[r].state[1];
        rs.positions = &m->ctl->pos;
        return rs;
    }));
    W_TRY(s.logits(1, nullptr, nullptr, true, m->logits));
    enqueue_step_end(m, greedy);
    return WICK_CUDA_OK;
}

int32_t hybrid_prepare(wick_cuda_model*, int) { return WICK_CUDA_OK; }

int32_t hybrid_enqueue_prefill_chunk(wick_cuda_model* m, int n, int start_pos, bool, bool embed, const LogitRows& out) {
    prof_begin(m);
    Step s(m, n, true);
    if (embed) s.in.tokens = m->tokens_dev;
    else s.in.frames = m->hidden;
    W_TRY(s.layers([&](size_t r) {
        RowState rs;
        rs.s0 = m->layers[r].state[0];
        rs.s1 = m->layers[r].state[1];
        rs.start_pos = start_pos;
        return rs;
    }));
    if (out.count) {
        memcpy(s.hm.h_rows, out.rows, (size_t)out.count * sizeof(int));
        CU_TRY(cudaMemcpyAsync(s.hm.rows_dev, s.hm.h_rows, (size_t)out.count * sizeof(int), cudaMemcpyHostToDevice, m->stream));
        W_TRY(s.logits(out.count, s.hm.rows_dev, m->normed_last, out.want_logits, out.dst));
    }
    return WICK_CUDA_OK;
}

int32_t hybrid_enqueue_decode_rows(wick_cuda_model* m, int n) {
    Step s(m, n, false);
    s.in.tokens = m->rows_tok;
    W_TRY(s.layers([&](size_t r) {
        RowState rs;
        rs.p0 = m->rows_ptrs + (r * 2) * m->batch_cap;
        rs.p1 = m->rows_ptrs + (r * 2 + 1) * m->batch_cap;
        rs.positions = m->rows_pos;
        return rs;
    }));
    return s.logits(n, nullptr, nullptr, true, m->logits_rows);
}

}  // namespace

const ModelFamily HYBRID_FAMILY = {hybrid_enqueue_decode, hybrid_prepare, hybrid_enqueue_prefill_chunk, hybrid_enqueue_decode_rows, false};

int32_t hybrid_alloc_scratch(wick_cuda_model* m) {
    HybridModel& hm = *m->hybrid;
    wick_cuda_config& c = m->cfg;
    const size_t act_bytes = hm.bf16 ? 2 : 4, N = (size_t)m->max_chunk;
    const int streams = std::max(hm.streams, 1);
    int ldp = 8, ldm = 8, ldf = 8, lda = 0, ldg = 0, ldq = 0, ldc = 0, ldi = 0;
    size_t kv = 0, partial = 0, fold = 0, wq = 0, wv = 0, wg = 0, wb = 0, wk = 0, wr = 0, lp = 0, mem = 0;
    for (const HybridLayer& L : hm.layers) {
        ldp = std::max(ldp, L.proj.m);
        ldm = std::max(ldm, L.o.k);
        if (L.kind == MIX_ATTENTION) {
            size_t pf = 0, fb = 0;
            mix_attn_scratch(L.attn, hm.bf16, m->max_chunk, &pf, &fb);
            partial = std::max(partial, pf);
            fold = std::max(fold, fb);
            c.n_heads = std::max<uint32_t>(c.n_heads, L.attn.heads);
            c.n_kv_heads = std::max<uint32_t>(c.n_kv_heads, L.attn.kv_heads);
        } else if (L.kind == MIX_DELTA) {
            const DeltaShape& s = L.delta;
            lda = std::max(lda, s.heads * s.dim);
            ldg = std::max(ldg, s.heads * s.vdim);
            wq = std::max(wq, (size_t)s.kv_heads * s.dimp());
            wg = std::max(wg, (size_t)s.heads * s.dimp());
            wv = std::max(wv, (size_t)s.heads * s.vdim);
            wb = std::max(wb, (size_t)s.heads);
            wk = std::max(wk, (size_t)s.kv_heads);
            wr = std::max(wr, delta_record_floats(s, m->max_chunk));
            c.n_heads = std::max<uint32_t>(c.n_heads, s.heads);
            c.conv_kernel_size = std::max<uint32_t>(c.conv_kernel_size, s.taps);
        } else if (L.kind == MIX_LATENT) {
            const LatentShape& s = L.latent;
            ldq = std::max(ldq, s.heads * s.q_pitch());
            ldc = std::max(ldc, s.heads * s.ldc());
            lp = std::max(lp, latent_scratch(s, hm.bf16, m->max_chunk, (int)c.max_seq_len));
            if (L.ukv.w) kv = std::max(kv, latent_tc_keys(s, m->max_chunk, (int)c.max_seq_len) * latent_tc_cols(s));
            c.n_heads = std::max<uint32_t>(c.n_heads, s.heads);
            c.n_kv_heads = std::max<uint32_t>(c.n_kv_heads, 1);
        } else {
            const MemoryShape& s = L.memory;
            ldi = std::max(ldi, 2 * s.heads);
            mem = std::max(mem, memory_work_bytes(s, hm.bf16, m->max_chunk));
            c.n_heads = std::max<uint32_t>(c.n_heads, s.heads);
        }
        if (L.ff != FF_NONE) {
            ldf = std::max(ldf, L.down.k);
            c.intermediate_size = std::max<uint32_t>(c.intermediate_size, L.down.k);
        }
    }
    // act buffers are cleared once, their row padding is never written
    hm.ldh = round_up(hm.width, 8);
    hm.ldw = round_up(hm.width, 8);
    hm.ldp = round_up(ldp, 8);
    hm.ldm = round_up(ldm, 8);
    hm.ldf = round_up(ldf, 8);
    hm.lda = round_up(lda, 8);
    hm.ldg = round_up(ldg, 8);
    hm.ldq = ldq;
    hm.ldc = ldc;
    hm.ldi = round_up(ldi, 8);
    auto act = [&](void** out, size_t elems) -> int32_t {
        uint8_t* p = nullptr;
        W_TRY(dev_alloc(m, &p, elems * act_bytes));
        CU_TRY(cudaMemset(p, 0, std::max<size_t>(elems * act_bytes, 256)));
        *out = p;
        return WICK_CUDA_OK;
    };
    const size_t NT = N * hm.max_top;  // rows in the experts' order
    W_TRY(dev_alloc(m, &hm.x, N * streams * hm.width));
    W_TRY(dev_alloc(m, &m->hidden, N * hm.width));  // embedding-input frames
    W_TRY(act(&hm.h, NT * hm.ldh));
    W_TRY(act(&hm.proj, N * hm.ldp));
    W_TRY(act(&hm.mixed, N * hm.ldm));
    W_TRY(act(&hm.ff, NT * hm.ldf));
    W_TRY(dev_alloc(m, &hm.y, NT * hm.ldw));
    if (hm.loop) {
        hm.ldcat = round_up(2 * hm.width, 8);
        W_TRY(act(&hm.cat, N * hm.ldcat));
    }
    if (partial) W_TRY(dev_alloc(m, &hm.attn.partial, partial));
    if (fold) W_TRY(dev_alloc(m, (uint8_t**)&hm.attn.fold, fold));
    if (wv) {
        W_TRY(dev_alloc(m, &hm.a, N * hm.lda));
        W_TRY(dev_alloc(m, &hm.gate, N * hm.ldg));
        W_TRY(dev_alloc(m, &hm.work.q, N * wq));
        W_TRY(dev_alloc(m, &hm.work.k, N * wq));
        W_TRY(dev_alloc(m, &hm.work.v, N * wv));
        W_TRY(dev_alloc(m, &hm.work.g, N * wg));
        W_TRY(dev_alloc(m, &hm.work.beta, N * wb));
        W_TRY(dev_alloc(m, &hm.work.kq, N * wk));
        W_TRY(dev_alloc(m, &hm.work.o, N * wv));
        W_TRY(dev_alloc(m, &hm.work.rec, wr));
    }
    if (ldq) {
        W_TRY(act(&hm.q, N * hm.ldq));
        W_TRY(act(&hm.qc, N * hm.ldc));
        W_TRY(act(&hm.oc, N * hm.ldc));
        W_TRY(dev_alloc(m, &hm.latent.partial, lp));
        if (kv) W_TRY(act(&hm.kv, kv));
    }
    if (mem) {
        W_TRY(dev_alloc(m, &hm.gates, N * hm.ldi));
        W_TRY(dev_alloc(m, (uint8_t**)&hm.memory, mem));
    }
    for (RouteJob& r : hm.routes) {
        W_TRY(dev_alloc(m, &r.inv, N * r.top));
        W_TRY(dev_alloc(m, &r.start, (size_t)r.experts + 1));
    }
    W_TRY(dev_alloc(m, &hm.rows_dev, N));
    W_TRY(dev_alloc(m, &m->tc_err, 1));
    CU_TRY(cudaMemset(m->tc_err, 0, 4));
    hm.attn.err = hm.latent.err = m->tc_err;
    CU_TRY(cudaMallocHost((void**)&hm.h_rows, N * sizeof(int)));
    return WICK_CUDA_OK;
}

}  // namespace wick
