// Host side of the models described by config.json (hybrid.cuh): reading the configuration and the weights, and
// enqueueing prompt chunks and decode steps.
//
// A step alternates one kernel that moves the streams (k_hyper_norm) with the sublayer's own kernels:
//   attention   proj GEMM -> qk norm + cache append -> attention -> W_o GEMM
//   delta       proj GEMM -> a2 | g2 GEMM -> convolutions, decays -> recurrence -> gated norm -> W_o GEMM
//   feed-forward  gate | up GEMM with the activation in its epilogue -> down GEMM
// The last kernel of a sublayer leaves y in f32; the next k_hyper_norm folds it into the streams.
#include "hybrid.cuh"

#include <cstring>

namespace wick {

HybridModel::~HybridModel() {
    if (h_rows) cudaFreeHost(h_rows);
}

const char* hybrid_layer_type(const wick_cuda_model* m, int layer) { return m->hybrid->layers[layer].type.c_str(); }

namespace {

// ── loading ────────────────────────────────────────────────────────────────
float bf16_to_f32(const uint8_t* p) {
    uint16_t u;
    memcpy(&u, p, 2);
    const uint32_t w = (uint32_t)u << 16;
    float f;
    memcpy(&f, &w, 4);
    return f;
}

struct Loader {
    wick_cuda_model* m;
    const SafeTensors& t;

    int32_t vec(const std::string& name, const std::vector<int64_t>& shape, float** out) const {
        // (a single number may be stored with shape [] or [1])
        const SafeTensor* one = shape.empty() ? t.find(name) : nullptr;
        const SafeTensor& s = t.get(name, one && one->shape == std::vector<int64_t>{1} ? one->shape : shape);
        std::vector<float> host(s.elems());
        for (size_t i = 0; i < host.size(); i++) host[i] = bf16_to_f32(s.data + 2 * i);
        return put(host, out);
    }
    int32_t put(const std::vector<float>& host, float** out) const {
        W_TRY(dev_alloc(m, out, host.size()));
        if (!host.empty()) CU_TRY(cudaMemcpy(*out, host.data(), host.size() * 4, cudaMemcpyHostToDevice));
        return WICK_CUDA_OK;
    }
    // Matrices [rows][k] stacked on top of each other, part i at row `at[i]`; rows in between are zero.
    int32_t matrix(const std::vector<std::pair<std::string, int>>& parts, const std::vector<int>& at, int rows, int k, DenseWeight* out) const {
        DenseWeight w;
        w.m = rows;
        w.k = k;
        w.ld = round_up(k, 8);
        std::vector<uint16_t> host((size_t)rows * w.ld, 0);
        for (size_t i = 0; i < parts.size(); i++) {
            const SafeTensor& s = t.get(parts[i].first, {parts[i].second, k});
            for (int r = 0; r < parts[i].second; r++) memcpy(&host[(size_t)(at[i] + r) * w.ld], s.data + (size_t)r * k * 2, (size_t)k * 2);
        }
        uint16_t* dev = nullptr;
        W_TRY(dev_alloc(m, &dev, host.size()));
        CU_TRY(cudaMemcpy(dev, host.data(), host.size() * 2, cudaMemcpyHostToDevice));
        w.w = (const __nv_bfloat16*)dev;
        *out = w;
        return WICK_CUDA_OK;
    }
    int32_t matrix(const std::string& name, int rows, int k, DenseWeight* out) const { return matrix({{name, rows}}, {0}, rows, k, out); }
    int32_t hyper(const std::string& layer, int q, int streams, HyperWeights* out) const {
        const std::string hc = layer + "hc" + std::to_string(q) + ".";
        W_TRY(vec(layer + "norm" + std::to_string(q), {}, &out->gain));
        W_TRY(vec(hc + "in", {streams}, &out->in));
        W_TRY(vec(hc + "out", {streams}, &out->out));
        return vec(hc + "mix", {streams, streams}, &out->mix);
    }
    // rows of a tensor whose second dimension is known (low-rank projections: the rank is the tensor's)
    int rank(const std::string& name) const {
        const SafeTensor* s = t.find(name);
        if (!s) throw std::runtime_error("tensor not found: " + name);
        if (s->shape.size() != 2 || s->shape[0] < 1) throw std::runtime_error("tensor " + name + ": expected a matrix");
        return (int)s->shape[0];
    }
};

// A mixer's mechanism: its name without the number that tells several sizes of one mechanism apart ("name", "name_2").
std::string mechanism(const std::string& type) {
    const size_t u = type.find_last_of('_');
    if (u == std::string::npos || u + 1 == type.size() || type.find_first_not_of("0123456789", u + 1) != std::string::npos) return type;
    return type.substr(0, u);
}

int32_t load_attention(const Loader& ld, const std::string& p, const JsonValue& mc, int width, HybridLayer* L, Layer* st, size_t act_bytes) {
    MixAttnShape& s = L->attn;
    s.heads = mc.count("heads");
    s.kv_heads = mc.count("kv_heads");
    s.dim = mc.count("dim");
    s.vdim = mc.count("vdim");
    s.scale = (float)mc.number("scale");
    s.eps = ld.m->hybrid->eps;
    if (const JsonValue* mask = mc.find("mask"); mask && mask->is_object()) {
        s.size = mask->count_or("size", 0);
        s.keep_first = mask->count_or("keep_first", 0);
    }
    if (s.heads % s.kv_heads) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": heads must be a multiple of kv_heads");
    if (!mix_attn_supported(s)) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": this many heads of this size do not fit the attention kernel");
    const int q = s.heads * s.dim, k = s.kv_heads * s.dim, v = s.kv_heads * s.vdim;
    W_TRY(ld.matrix({{p + "q", q}, {p + "k", k}, {p + "v", v}}, {0, q, q + k}, q + k + v, width, &L->proj));
    W_TRY(ld.matrix(p + "o", width, s.heads * s.vdim, &L->o));
    float *talk = nullptr, *bias = nullptr;
    W_TRY(ld.vec(p + "talk", {s.heads, s.heads}, &talk));
    W_TRY(ld.vec(p + "pb", {s.heads}, &bias));
    s.talk = talk;
    s.bias = bias;
    st->is_attn = true;
    st->n_kv = s.kv_heads;
    st->sd[0].per_pos = (size_t)k * act_bytes;
    st->sd[1].per_pos = (size_t)v * act_bytes;
    return WICK_CUDA_OK;
}

int32_t load_delta(const Loader& ld, const std::string& p, const JsonValue& mc, int width, HybridLayer* L, Layer* st) {
    DeltaShape& s = L->delta;
    s.heads = mc.count("heads");
    s.kv_heads = mc.count("kv_heads");
    s.dim = mc.count("dim");
    s.vdim = mc.count("vdim");
    s.taps = mc.count("conv");
    s.eps = ld.m->hybrid->eps;
    if (s.heads % s.kv_heads) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": heads must be a multiple of kv_heads");
    if (s.dim > DELTA_MAX_DIM || s.taps > DELTA_MAX_TAPS)
        return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": key size up to " + std::to_string(DELTA_MAX_DIM) + " and up to " + std::to_string(DELTA_MAX_TAPS) + " taps");
    const int qk = s.kv_heads * s.dim, v = s.heads * s.vdim, hd = s.heads * s.dim;
    const int ra = ld.rank(p + "a1"), rg = ld.rank(p + "g1");
    L->off_b = round_up(2 * qk + v, 8);
    L->off_a1 = round_up(L->off_b + s.heads, 8);
    L->off_g1 = round_up(L->off_a1 + ra, 8);
    W_TRY(ld.matrix({{p + "q", qk}, {p + "k", qk}, {p + "v", v}, {p + "b", s.heads}, {p + "a1", ra}, {p + "g1", rg}},
                    {0, qk, 2 * qk, L->off_b, L->off_a1, L->off_g1}, round_up(L->off_g1 + rg, 8), width, &L->proj));
    W_TRY(ld.matrix(p + "a2", hd, ra, &L->a2));
    W_TRY(ld.matrix(p + "g2", v, rg, &L->g2));
    W_TRY(ld.matrix(p + "o", width, v, &L->o));
    std::vector<float> conv;
    for (const auto& part : {std::make_pair("q.conv", qk), std::make_pair("k.conv", qk), std::make_pair("v.conv", v)}) {
        const SafeTensor& c = ld.t.get(p + part.first, {part.second, s.taps});
        for (size_t i = 0; i < c.elems(); i++) conv.push_back(bf16_to_f32(c.data + 2 * i));
    }
    W_TRY(ld.put(conv, &L->conv_w));
    W_TRY(ld.vec(p + "A_log", {s.heads}, &L->A_log));
    W_TRY(ld.vec(p + "dt_bias", {hd}, &L->dt_bias));
    W_TRY(ld.vec(p + "norm", {s.vdim}, &L->out_norm));
    st->sd[0].fixed = s.state_floats() * 4;
    st->sd[1].fixed = s.conv_floats() * 4;
    return WICK_CUDA_OK;
}

// ── one step ───────────────────────────────────────────────────────────────
struct Step {
    wick_cuda_model* m;
    HybridModel& hm;
    int n;
    bool timed;                 // prefill: feed the per-category timers
    const HyperWeights* pending = nullptr;  // sublayer whose y is not in the streams yet
    bool first = true;
    HyperArgs src;              // where the first launch takes the embedding from

    Step(wick_cuda_model* m, int n, bool timed) : m(m), hm(*m->hybrid), n(n), timed(timed) {}
    void mark(int cat) {
        if (timed) prof_mark(m, cat);
    }

    HyperArgs stream_args() {
        HyperArgs a = first ? src : HyperArgs();
        a.x = hm.x;
        a.S = hm.streams;
        a.W = hm.width;
        a.eps = hm.eps;
        a.h = hm.h;
        a.ldh = hm.ldh;
        a.n = n;
        if (pending) {
            a.y = hm.y;
            a.ldy = hm.ldw;
            a.mix = pending->mix;
            a.out = pending->out;
        }
        return a;
    }
    // streams <- pending write; h <- norm of the sublayer's read
    void enter(const HyperWeights& w) {
        HyperArgs a = stream_args();
        a.in = w.in;
        a.gain = w.gain;
        launch_hyper_norm(m->stream, hm.bf16, a);
        first = false;
        pending = &w;
        mark(PC_NORM_QUANT);
    }
    int32_t dense(const DenseWeight& w, const void* x, int ldx, void* y, int ldy, bool f32, float softcap = 0.0f, int rows = -1) {
        DenseCall c;
        c.job[0].w = w; c.job[0].x = x; c.job[0].ldx = ldx; c.job[0].y = y; c.job[0].ldy = ldy;
        c.n = rows < 0 ? n : rows;
        c.out_f32 = f32;
        c.softcap = softcap;
        c.err = m->tc_err;
        CU_TRY(launch_dense(m->stream, hm.bf16, c));
        return WICK_CUDA_OK;
    }
    const void* act_at(const void* p, int col) const { return (const uint8_t*)p + (size_t)col * (hm.bf16 ? 2 : 4); }

    int32_t layer(size_t li, const RowState& rs) {
        const HybridLayer& L = hm.layers[li];
        cudaStream_t st = m->stream;
        enter(L.hc1);
        W_TRY(dense(L.proj, hm.h, hm.ldh, hm.proj, hm.ldp, false));
        mark(PC_GEMM);
        if (L.kind == MIX_ATTENTION) {
            launch_qk_rms_append(st, hm.bf16, hm.proj, hm.ldp, n, L.attn, rs, hm.attn);
            mark(PC_QK_ROPE_KV);
            CU_TRY(launch_mix_attn(st, hm.bf16, hm.proj, hm.ldp, n, L.attn, rs, hm.mixed, hm.ldm, hm.attn, (int)m->cfg.max_seq_len));
            mark(PC_ATTENTION);
        } else {
            DenseCall c;
            c.count = 2;
            c.n = n;
            c.out_f32 = true;
            c.err = m->tc_err;
            c.job[0].w = L.a2; c.job[0].x = act_at(hm.proj, L.off_a1); c.job[0].ldx = hm.ldp; c.job[0].y = hm.a;    c.job[0].ldy = hm.lda;
            c.job[1].w = L.g2; c.job[1].x = act_at(hm.proj, L.off_g1); c.job[1].ldx = hm.ldp; c.job[1].y = hm.gate; c.job[1].ldy = hm.ldg;
            CU_TRY(launch_dense(st, hm.bf16, c));
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
                launch_delta_out(st, hm.bf16, n, L.delta, hm.work.o, L.out_norm, hm.gate, hm.ldg, hm.mixed, hm.ldm);
            }
            mark(PC_RECURRENCE);
        }
        W_TRY(dense(L.o, hm.mixed, hm.ldm, hm.y, hm.ldw, true));
        mark(PC_GEMM);
        if (L.has_ff) {
            enter(L.hc2);
            DenseCall c;
            c.count = 2;
            c.n = n;
            c.gated = true;
            c.act = L.act;
            c.err = m->tc_err;
            c.job[0].w = L.gate; c.job[0].x = hm.h; c.job[0].ldx = hm.ldh; c.job[0].y = hm.ff; c.job[0].ldy = hm.ldf;
            c.job[1] = c.job[0];
            c.job[1].w = L.up;
            CU_TRY(launch_dense(st, hm.bf16, c));
            W_TRY(dense(L.down, hm.ff, hm.ldf, hm.y, hm.ldw, true));
            mark(PC_GEMM);
        }
        return WICK_CUDA_OK;
    }
    // final norm of `count` rows (row i: rows_dev[i], or i itself), then logits
    int32_t logits(int count, const int* rows_dev, float* normed, bool want, float* dst) {
        HyperArgs a = stream_args();
        a.rows = rows_dev;
        a.store_x = false;
        a.gain = hm.final_gain;
        a.n = count;
        a.normed = normed;
        launch_hyper_norm(m->stream, hm.bf16, a);
        if (want) W_TRY(dense(hm.head, hm.h, hm.ldh, dst, (int)m->cfg.vocab_size, true, hm.softcap, count));
        mark(PC_LOGITS);
        return WICK_CUDA_OK;
    }
};

int32_t hybrid_enqueue_decode(wick_cuda_model* m, bool greedy) {
    Step s(m, 1, false);
    s.src.ctl = m->ctl;
    s.src.embed = s.hm.embed.w;
    s.src.ld_embed = s.hm.embed.ld;
    s.src.embed_scale = s.hm.embed_scale;
    for (size_t li = 0; li < m->layers.size(); li++) {
        RowState rs;
        rs.s0 = m->layers[li].state[0];
        rs.s1 = m->layers[li].state[1];
        rs.positions = &m->ctl->pos;
        W_TRY(s.layer(li, rs));
    }
    W_TRY(s.logits(1, nullptr, nullptr, true, m->logits));
    enqueue_step_end(m, greedy);
    return WICK_CUDA_OK;
}

int32_t hybrid_prepare(wick_cuda_model*, int) { return WICK_CUDA_OK; }

int32_t hybrid_enqueue_prefill_chunk(wick_cuda_model* m, int n, int start_pos, bool, bool embed, const LogitRows& out) {
    prof_begin(m);
    Step s(m, n, true);
    if (embed) {
        s.src.tokens = m->tokens_dev;
        s.src.embed = s.hm.embed.w;
        s.src.ld_embed = s.hm.embed.ld;
        s.src.embed_scale = s.hm.embed_scale;
    } else {
        s.src.frames = m->hidden;
    }
    for (size_t li = 0; li < m->layers.size(); li++) {
        RowState rs;
        rs.s0 = m->layers[li].state[0];
        rs.s1 = m->layers[li].state[1];
        rs.start_pos = start_pos;
        W_TRY(s.layer(li, rs));
    }
    if (out.count) {
        memcpy(s.hm.h_rows, out.rows, (size_t)out.count * sizeof(int));
        CU_TRY(cudaMemcpyAsync(s.hm.rows_dev, s.hm.h_rows, (size_t)out.count * sizeof(int), cudaMemcpyHostToDevice, m->stream));
        W_TRY(s.logits(out.count, s.hm.rows_dev, m->normed_last, out.want_logits, out.dst));
    }
    return WICK_CUDA_OK;
}

int32_t hybrid_enqueue_decode_rows(wick_cuda_model* m, int n) {
    Step s(m, n, false);
    s.src.tokens = m->rows_tok;
    s.src.embed = s.hm.embed.w;
    s.src.ld_embed = s.hm.embed.ld;
    s.src.embed_scale = s.hm.embed_scale;
    for (size_t li = 0; li < m->layers.size(); li++) {
        RowState rs;
        rs.p0 = m->rows_ptrs + (li * 2) * m->batch_cap;
        rs.p1 = m->rows_ptrs + (li * 2 + 1) * m->batch_cap;
        rs.positions = m->rows_pos;
        W_TRY(s.layer(li, rs));
    }
    return s.logits(n, nullptr, nullptr, true, m->logits_rows);
}

}  // namespace

const ModelFamily HYBRID_FAMILY = {hybrid_enqueue_decode, hybrid_prepare, hybrid_enqueue_prefill_chunk, hybrid_enqueue_decode_rows, false};

int32_t nositar_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute) {
    m->hybrid.reset(new HybridModel());
    HybridModel& hm = *m->hybrid;
    hm.bf16 = compute != WICK_CUDA_COMPUTE_F32;
    hm.width = config.count("width");
    hm.streams = config.count_or("streams", 1);
    hm.eps = (float)config.at("norm").number("eps");
    hm.embed_scale = (float)(config.find("embedding") ? config.at("embedding").number_or("scale", 1.0) : 1.0);
    hm.softcap = (float)config.number_or("logit_softcap", 0.0);
    if (hm.streams < 1 || hm.streams > HYPER_MAX_STREAMS) return fail(WICK_CUDA_ERR_BAD_MODEL, "streams must be 1 .. " + std::to_string(HYPER_MAX_STREAMS));
    if (hm.width > 48 * 1024) return fail(WICK_CUDA_ERR_BAD_MODEL, "width must be at most 49152");
    const JsonValue& list = config.at("layers");
    if (!list.is_array() || list.items.empty()) return fail(WICK_CUDA_ERR_BAD_MODEL, "layers must be a list");
    wick_cuda_config& c = m->cfg;
    c.n_layers = (uint32_t)list.items.size();
    c.hidden_size = (uint32_t)hm.width;
    c.vocab_size = (uint32_t)config.count("vocab");
    c.max_seq_len = context_size;
    c.rms_norm_eps = hm.eps;
    choose_max_chunk(m);
    const size_t act_bytes = hm.bf16 ? 2 : 4;
    const Loader ld{m, tensors};
    W_TRY(ld.matrix("embed", (int)c.vocab_size, hm.width, &hm.embed));
    W_TRY(ld.matrix("head", (int)c.vocab_size, hm.width, &hm.head));
    W_TRY(ld.vec("final.norm", {}, &hm.final_gain));
    hm.layers.resize(c.n_layers);
    m->layers.resize(c.n_layers);
    int ldp = 8, ldm = 8, ldf = 8, lda = 8, ldg = 8;
    size_t partial = 0, fold = 0, wq = 0, wv = 0, wg = 0, wb = 0, wk = 0, wr = 0;
    for (uint32_t i = 0; i < c.n_layers; i++) {
        const JsonValue& lc = list.items[i];
        HybridLayer& L = hm.layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        L.type = lc.at("type").str;
        const JsonValue& mc = lc.at("mixer");
        const std::string kind = mechanism(L.type);
        if (kind == "attention") {
            L.kind = MIX_ATTENTION;
            W_TRY(load_attention(ld, p + "mix.", mc, hm.width, &L, &m->layers[i], act_bytes));
            const MixAttnShape& s = L.attn;
            ldm = std::max(ldm, s.heads * s.vdim);
            size_t pf = 0, fb = 0;
            mix_attn_scratch(s, hm.bf16, m->max_chunk, &pf, &fb);
            partial = std::max(partial, pf);
            fold = std::max(fold, fb);
            c.n_heads = std::max<uint32_t>(c.n_heads, s.heads);
            c.n_kv_heads = std::max<uint32_t>(c.n_kv_heads, s.kv_heads);
        } else if (kind == "channel_delta") {
            L.kind = MIX_DELTA;
            W_TRY(load_delta(ld, p + "mix.", mc, hm.width, &L, &m->layers[i]));
            const DeltaShape& s = L.delta;
            ldm = std::max(ldm, s.heads * s.vdim);
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
        } else {
            return fail(WICK_CUDA_ERR_BAD_MODEL, "layer " + std::to_string(i) + ": unknown mixer type " + L.type);
        }
        ldp = std::max(ldp, L.proj.m);
        W_TRY(ld.hyper(p, 1, hm.streams, &L.hc1));
        const JsonValue* mlp = lc.find("mlp");
        if (mlp && mlp->is_object()) {
            const std::string ff_kind = mlp->at("kind").str;
            if (ff_kind != "dense") return fail(WICK_CUDA_ERR_BAD_MODEL, "layer " + std::to_string(i) + ": unknown feed-forward kind " + ff_kind);
            const int ff = mlp->count("ff");
            L.has_ff = true;
            W_TRY(ld.matrix(p + "mlp.gate", ff, hm.width, &L.gate));
            W_TRY(ld.matrix(p + "mlp.up", ff, hm.width, &L.up));
            W_TRY(ld.matrix(p + "mlp.down", hm.width, ff, &L.down));
            W_TRY(ld.hyper(p, 2, hm.streams, &L.hc2));
            ldf = std::max(ldf, ff);
            c.intermediate_size = std::max<uint32_t>(c.intermediate_size, ff);
        }
    }
    // scratch; act buffers are cleared once, their row padding is never written
    hm.ldh = round_up(hm.width, 8);
    hm.ldw = round_up(hm.width, 8);
    hm.ldp = round_up(ldp, 8);
    hm.ldm = round_up(ldm, 8);
    hm.ldf = round_up(ldf, 8);
    hm.lda = round_up(lda, 8);
    hm.ldg = round_up(ldg, 8);
    const size_t N = (size_t)m->max_chunk;
    auto act = [&](void** out, int ldx) -> int32_t {
        uint8_t* p = nullptr;
        W_TRY(dev_alloc(m, &p, N * ldx * act_bytes));
        CU_TRY(cudaMemset(p, 0, N * ldx * act_bytes));
        *out = p;
        return WICK_CUDA_OK;
    };
    W_TRY(dev_alloc(m, &hm.x, N * hm.streams * hm.width));
    W_TRY(dev_alloc(m, &m->hidden, N * hm.width));  // embedding-input frames
    W_TRY(act(&hm.h, hm.ldh));
    W_TRY(act(&hm.proj, hm.ldp));
    W_TRY(act(&hm.mixed, hm.ldm));
    W_TRY(act(&hm.ff, hm.ldf));
    W_TRY(dev_alloc(m, &hm.y, N * hm.ldw));
    W_TRY(dev_alloc(m, &hm.a, N * hm.lda));
    W_TRY(dev_alloc(m, &hm.gate, N * hm.ldg));
    W_TRY(dev_alloc(m, &hm.attn.partial, partial));
    if (fold) W_TRY(dev_alloc(m, (uint8_t**)&hm.attn.fold, fold));
    W_TRY(dev_alloc(m, &hm.work.q, N * wq));
    W_TRY(dev_alloc(m, &hm.work.k, N * wq));
    W_TRY(dev_alloc(m, &hm.work.v, N * wv));
    W_TRY(dev_alloc(m, &hm.work.g, N * wg));
    W_TRY(dev_alloc(m, &hm.work.beta, N * wb));
    W_TRY(dev_alloc(m, &hm.work.kq, N * wk));
    W_TRY(dev_alloc(m, &hm.work.o, N * wv));
    W_TRY(dev_alloc(m, &hm.work.rec, wr));
    W_TRY(dev_alloc(m, &hm.rows_dev, N));
    W_TRY(dev_alloc(m, &m->tc_err, 1));
    CU_TRY(cudaMemset(m->tc_err, 0, 4));
    hm.attn.err = m->tc_err;
    CU_TRY(cudaMallocHost((void**)&hm.h_rows, N * sizeof(int)));
    return WICK_CUDA_OK;
}

}  // namespace wick
