// Reading a model folder into a HybridModel: one loader per mixer and per kind of feed-forward, shared by the architectures,
// which differ in what stands around the sublayers.
#include <cmath>
#include <cstring>

#include "hybrid.cuh"

namespace wick {

namespace {

float bf16_to_f32(const uint8_t* p) {
    uint16_t u;
    memcpy(&u, p, 2);
    const uint32_t w = (uint32_t)u << 16;
    float f;
    memcpy(&f, &w, 4);
    return f;
}

// Rows of a tensor at a place of a stacked matrix.
struct Part {
    std::string name;
    int rows;
    int at;
};

struct Loader {
    wick_cuda_model* m;
    const SafeTensors& t;

    std::vector<float> host_vec(const std::string& name, const std::vector<int64_t>& shape) const {
        // (a single number may be stored with shape [] or [1])
        const SafeTensor* one = shape.empty() ? t.find(name) : nullptr;
        const SafeTensor& s = t.get(name, one && one->shape == std::vector<int64_t>{1} ? one->shape : shape);
        std::vector<float> host(s.elems());
        for (size_t i = 0; i < host.size(); i++) host[i] = bf16_to_f32(s.data + 2 * i);
        return host;
    }
    int32_t vec(const std::string& name, const std::vector<int64_t>& shape, float** out) const { return put(host_vec(name, shape), out); }
    // a gain that is stored around zero
    int32_t gain(const std::string& name, int n, float** out) const {
        std::vector<float> host = host_vec(name, {n});
        for (float& v : host) v += 1.0f;
        return put(host, out);
    }
    template <class T>
    int32_t put(const std::vector<T>& host, T** out) const {
        W_TRY(dev_alloc(m, out, host.size()));
        if (!host.empty()) CU_TRY(cudaMemcpy(*out, host.data(), host.size() * sizeof(T), cudaMemcpyHostToDevice));
        return WICK_CUDA_OK;
    }
    int32_t put_matrix(const std::vector<uint16_t>& host, int rows, int k, DenseWeight* out) const {
        DenseWeight w;
        w.m = rows;
        w.k = k;
        w.ld = round_up(k, 8);
        uint16_t* dev = nullptr;
        W_TRY(put(host, &dev));
        w.w = (const __nv_bfloat16*)dev;
        *out = w;
        return WICK_CUDA_OK;
    }
    // Matrices [rows][k] stacked on top of each other; rows in between are zero.
    int32_t matrix(const std::vector<Part>& parts, int rows, int k, DenseWeight* out) const {
        const size_t ld = round_up(k, 8);
        std::vector<uint16_t> host(rows * ld, 0);
        for (const Part& p : parts) {
            const SafeTensor& s = t.get(p.name, {p.rows, k});
            for (int r = 0; r < p.rows; r++) memcpy(&host[(p.at + r) * ld], s.data + (size_t)r * k * 2, (size_t)k * 2);
        }
        return put_matrix(host, rows, k, out);
    }
    int32_t matrix(const std::string& name, int rows, int k, DenseWeight* out) const { return matrix({{name, rows, 0}}, rows, k, out); }
    // One matrix per expert, stacked.
    int32_t expert_matrices(const std::string& p, const char* name, int experts, int rows, int k, DenseWeight* out) const {
        std::vector<Part> parts;
        for (int e = 0; e < experts; e++) parts.push_back({p + "e" + std::to_string(e) + "." + name, rows, e * rows});
        W_TRY(matrix(parts, experts * rows, k, out));
        out->m = rows;
        return WICK_CUDA_OK;
    }
    int32_t hyper(const std::string& layer, int q, int streams, SublayerWeights* out) const {
        const std::string hc = layer + "hc" + std::to_string(q) + ".";
        W_TRY(vec(layer + "norm" + std::to_string(q), {}, &out->gain));
        W_TRY(vec(hc + "in", {streams}, &out->in));
        W_TRY(vec(hc + "out", {streams}, &out->out));
        return vec(hc + "mix", {streams, streams}, &out->mix);
    }
    int32_t norms_around(const std::string& layer, int q, int width, SublayerWeights* out) const {
        const std::string name = layer + "norm" + std::to_string(q);
        W_TRY(gain(name, width, &out->gain));
        return gain(name + "b", width, &out->post);
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

// ── mixers ─────────────────────────────────────────────────────────────────
int32_t load_attention(const Loader& ld, const std::string& p, const JsonValue& mc, HybridLayer* L) {
    const HybridModel& hm = *ld.m->hybrid;
    MixAttnShape& s = L->attn;
    L->kind = MIX_ATTENTION;
    s.heads = mc.count("heads");
    s.kv_heads = mc.count("kv_heads");
    s.dim = mc.count("dim");
    s.vdim = mc.count("vdim");
    s.scale = (float)mc.number("scale");
    s.eps = hm.eps;
    if (const JsonValue* mask = mc.find("mask"); mask && mask->is_object()) {
        s.size = mask->count_or("size", 0);
        s.keep_first = mask->count_or("keep_first", 0);
    }
    if (s.heads % s.kv_heads) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": heads must be a multiple of kv_heads");
    if (!mix_attn_supported(s)) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": this many heads of this size do not fit the attention kernel");
    const int q = s.heads * s.dim, k = s.kv_heads * s.dim, v = s.kv_heads * s.vdim;
    W_TRY(ld.matrix({{p + "q", q, 0}, {p + "k", k, q}, {p + "v", v, q + k}}, q + k + v, hm.width, &L->proj));
    W_TRY(ld.matrix(p + "o", hm.width, s.heads * s.vdim, &L->o));
    float *talk = nullptr, *bias = nullptr;
    W_TRY(ld.vec(p + "talk", {s.heads, s.heads}, &talk));
    W_TRY(ld.vec(p + "pb", {s.heads}, &bias));
    s.talk = talk;
    s.bias = bias;
    return WICK_CUDA_OK;
}

int32_t load_delta(const Loader& ld, const std::string& p, const JsonValue& mc, HybridLayer* L) {
    const int width = ld.m->hybrid->width;
    DeltaShape& s = L->delta;
    L->kind = MIX_DELTA;
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
    W_TRY(ld.matrix({{p + "q", qk, 0}, {p + "k", qk, qk}, {p + "v", v, 2 * qk}, {p + "b", s.heads, L->off_b}, {p + "a1", ra, L->off_a1}, {p + "g1", rg, L->off_g1}},
                    round_up(L->off_g1 + rg, 8), width, &L->proj));
    W_TRY(ld.matrix(p + "a2", hd, ra, &L->a2));
    W_TRY(ld.matrix(p + "g2", v, rg, &L->g2));
    W_TRY(ld.matrix(p + "o", width, v, &L->o));
    std::vector<float> conv;
    for (const auto& part : {std::make_pair("q.conv", qk), std::make_pair("k.conv", qk), std::make_pair("v.conv", v)}) {
        const std::vector<float> c = ld.host_vec(p + part.first, {part.second, s.taps});
        conv.insert(conv.end(), c.begin(), c.end());
    }
    W_TRY(ld.put(conv, &L->conv_w));
    W_TRY(ld.vec(p + "A_log", {s.heads}, &L->A_log));
    W_TRY(ld.vec(p + "dt_bias", {hd}, &L->dt_bias));
    return ld.vec(p + "norm", {s.vdim}, &L->out_norm);
}

// cos and sin of every position for the pairs of `dims` rotated dimensions, in f64 up to the rounding to f32.  With a "scaling"
// object, pairs that turn more than `fast` times within `original` positions keep their frequency, pairs that turn less than
// `slow` times are slowed by `factor`, with a linear ramp in between, and cos and sin grow with log(factor).
int32_t rope_table(const Loader& ld, const JsonValue& rot, const float2** out) {
    HybridModel& hm = *ld.m->hybrid;
    const int dims = rot.count("dims"), half = dims / 2, positions = (int)ld.m->cfg.max_seq_len;
    const double base = rot.number("base");
    if (dims % 2 || base <= 0.0 || base == 1.0) return fail(WICK_CUDA_ERR_BAD_MODEL, "rotation: an even number of dimensions and a positive base other than 1");
    std::vector<double> key{(double)dims, base}, freq(half);
    double size = 1.0;
    for (int i = 0; i < half; i++) freq[i] = std::pow(base, -2.0 * i / dims);
    if (const JsonValue* sc = rot.find("scaling"); sc && sc->is_object()) {
        const double factor = sc->number("factor"), original = sc->number("original"), fast = sc->number("fast"), slow = sc->number("slow");
        if (factor <= 0.0 || original <= 0.0 || fast <= 0.0 || slow <= 0.0) return fail(WICK_CUDA_ERR_BAD_MODEL, "rotation: scaling numbers must be positive");
        key.insert(key.end(), {factor, original, fast, slow});
        const double pi = std::acos(-1.0);
        auto pair_that_turns = [&](double times) { return dims * std::log(original / (2.0 * pi * times)) / (2.0 * std::log(base)); };
        const double lo = std::max(std::floor(pair_that_turns(fast)), 0.0), hi = std::min(std::ceil(pair_that_turns(slow)), dims - 1.0);
        for (int i = 0; i < half; i++) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            freq[i] = freq[i] / factor * ramp + freq[i] * (1.0 - ramp);
        }
        size = 0.1 * std::log(factor) + 1.0;
    }
    for (const auto& t : hm.rope_tables)
        if (t.first == key) {
            *out = t.second;
            return WICK_CUDA_OK;
        }
    std::vector<float2> table((size_t)positions * half);
    for (int p = 0; p < positions; p++)
        for (int i = 0; i < half; i++) table[(size_t)p * half + i] = make_float2((float)(size * std::cos(p * freq[i])), (float)(size * std::sin(p * freq[i])));
    float2* dev = nullptr;
    W_TRY(ld.put(table, &dev));
    hm.rope_tables.emplace_back(key, dev);
    *out = dev;
    return WICK_CUDA_OK;
}

int32_t load_latent(const Loader& ld, const std::string& p, const JsonValue& mc, HybridLayer* L) {
    const int width = ld.m->hybrid->width;
    LatentShape& s = L->latent;
    L->kind = MIX_LATENT;
    s.heads = mc.count("heads");
    s.dim = mc.count("dim");
    s.rot_dim = mc.count("rot_dim");
    s.vdim = mc.count("vdim");
    s.kv_rank = mc.count("kv_rank");
    s.q_rank = mc.find("q_rank") ? mc.count("q_rank") : ld.rank(p + "dq");
    s.scale = (float)mc.number("scale");
    s.eps = ld.m->hybrid->eps;
    if (const JsonValue* mask = mc.find("mask"); mask && mask->is_object()) s.size = mask->count_or("size", 0);
    const JsonValue& rot = mc.at("rot");
    s.rot_dims = rot.count("dims");
    if (s.rot_dims > s.rot_dim) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": more rotated dimensions than the rotated part has");
    W_TRY(rope_table(ld, rot, &s.rope));
    if (!latent_supported(s)) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": a latent of this size does not fit the attention kernel");
    const int H = s.heads, C = s.kv_rank, kv = C + s.rot_dim;
    W_TRY(ld.matrix({{p + "dq", s.q_rank, 0}, {p + "dkv", kv, s.off_kv()}}, s.off_kv() + kv, width, &L->proj));
    // queries: a head's rows at the pitch of LatentShape
    {
        const SafeTensor& t = ld.t.get(p + "uq", {H * (s.dim + s.rot_dim), s.q_rank});
        const size_t l = round_up(s.q_rank, 8);
        std::vector<uint16_t> host(H * s.q_pitch() * l, 0);
        for (int r = 0; r < H * (s.dim + s.rot_dim); r++) {
            const int h = r / (s.dim + s.rot_dim), d = r % (s.dim + s.rot_dim);
            const size_t row = h * s.q_pitch() + (d < s.dim ? d : s.q_off_rot() + d - s.dim);
            memcpy(&host[row * l], t.data + (size_t)r * s.q_rank * 2, (size_t)s.q_rank * 2);
        }
        W_TRY(ld.put_matrix(host, H * s.q_pitch(), s.q_rank, &L->uq));
    }
    // keys, transposed per head: [H * kv_rank][dim]
    {
        const SafeTensor& t = ld.t.get(p + "uk", {H * s.dim, C});
        const size_t l = round_up(s.dim, 8);
        std::vector<uint16_t> host((size_t)H * C * l, 0);
        for (int r = 0; r < H * s.dim; r++)
            for (int c = 0; c < C; c++) memcpy(&host[((size_t)(r / s.dim) * C + c) * l + r % s.dim], t.data + ((size_t)r * C + c) * 2, 2);
        W_TRY(ld.put_matrix(host, H * C, s.dim, &L->uk_t));
    }
    W_TRY(ld.matrix(p + "uv", H * s.vdim, C, &L->uv));
    if (ld.m->hybrid->bf16 && latent_tc_supported(s)) {  // keys and values of the prompt form
        const int d8 = round_up(s.dim, 8), v8 = round_up(s.vdim, 8);
        const SafeTensor &tk = ld.t.get(p + "uk", {H * s.dim, C}), &tv = ld.t.get(p + "uv", {H * s.vdim, C});
        const size_t l = round_up(C, 8);
        std::vector<uint16_t> host((size_t)latent_tc_cols(s) * l, 0);
        for (int h = 0; h < H; h++) {
            for (int d = 0; d < s.dim; d++) memcpy(&host[((size_t)h * d8 + d) * l], tk.data + (size_t)(h * s.dim + d) * C * 2, (size_t)C * 2);
            for (int d = 0; d < s.vdim; d++) memcpy(&host[((size_t)H * d8 + h * v8 + d) * l], tv.data + (size_t)(h * s.vdim + d) * C * 2, (size_t)C * 2);
        }
        W_TRY(ld.put_matrix(host, latent_tc_cols(s), C, &L->ukv));
    }
    W_TRY(ld.matrix(p + "o", width, H * s.vdim, &L->o));
    float *sink = nullptr, *qn = nullptr, *kn = nullptr;
    W_TRY(ld.vec(p + "sink", {H}, &sink));
    W_TRY(ld.vec(p + "dq.norm", {s.q_rank}, &qn));
    W_TRY(ld.vec(p + "dkv.norm", {C}, &kn));
    s.sink = sink;
    s.q_norm = qn;
    s.kv_norm = kn;
    return WICK_CUDA_OK;
}

int32_t load_memory(const Loader& ld, const std::string& p, const JsonValue& mc, HybridLayer* L) {
    const int width = ld.m->hybrid->width;
    MemoryShape& s = L->memory;
    L->kind = MIX_MEMORY;
    s.heads = mc.count("heads");
    s.dim = mc.count("dim");
    s.vdim = mc.count("vdim");
    s.cap = (float)mc.number("gate_cap");
    s.eps = ld.m->hybrid->eps;
    if (s.cap <= 0.0f) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": gate_cap must be positive");
    if (s.dim > MEMORY_MAX_DIM || s.vdim > MEMORY_MAX_DIM) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": key and value sizes up to " + std::to_string(MEMORY_MAX_DIM));
    const int qk = s.heads * s.dim, v = s.heads * s.vdim;
    W_TRY(ld.matrix({{p + "q", qk, 0}, {p + "k", qk, qk}, {p + "v", v, 2 * qk}, {p + "g", v, 2 * qk + v}}, 2 * qk + 2 * v, width, &L->proj));
    W_TRY(ld.matrix({{p + "i", s.heads, 0}, {p + "f", s.heads, s.heads}}, 2 * s.heads, width, &L->gates));
    W_TRY(ld.matrix(p + "o", width, v, &L->o));
    float *bi = nullptr, *bf = nullptr, *norm = nullptr;
    W_TRY(ld.vec(p + "i.b", {s.heads}, &bi));
    W_TRY(ld.vec(p + "f.b", {s.heads}, &bf));
    W_TRY(ld.vec(p + "norm", {v}, &norm));
    s.i_bias = bi;
    s.f_bias = bf;
    s.norm = norm;
    return WICK_CUDA_OK;
}

struct MixerEntry {
    const char* name;
    int32_t (*load)(const Loader& ld, const std::string& prefix, const JsonValue& mixer, HybridLayer* L);
};
const MixerEntry MIXERS[] = {
    {"attention", load_attention},
    {"channel_delta", load_delta},
    {"latent_attention", load_latent},
    {"mlstm", load_memory},
};

// What a layer keeps per sequence.
void describe_state(const HybridLayer& L, bool bf16, Layer* st) {
    const size_t act = bf16 ? 2 : 4;
    switch (L.kind) {
        case MIX_ATTENTION:
            st->is_attn = true;
            st->n_kv = L.attn.kv_heads;
            st->sd[0].per_pos = (size_t)L.attn.kv_heads * L.attn.dim * act;
            st->sd[1].per_pos = (size_t)L.attn.kv_heads * L.attn.vdim * act;
            break;
        case MIX_DELTA:
            st->sd[0].fixed = L.delta.state_floats() * 4;
            st->sd[1].fixed = L.delta.conv_floats() * 4;
            break;
        case MIX_LATENT:
            st->is_attn = true;
            st->n_kv = 1;
            st->sd[0].per_pos = (size_t)L.latent.ldc() * act;
            break;
        case MIX_MEMORY:
            st->sd[0].fixed = L.memory.state_floats() * 4;
            st->sd[1].fixed = (size_t)L.memory.heads * 4;
            break;
    }
}

// ── feed-forward ───────────────────────────────────────────────────────────
int32_t load_gated_ff(const Loader& ld, const std::string& p, int ff, Activation act, HybridLayer* L) {
    const int width = ld.m->hybrid->width;
    L->ff = FF_GATED;
    L->act = act;
    W_TRY(ld.matrix(p + "gate", ff, width, &L->gate));
    W_TRY(ld.matrix(p + "up", ff, width, &L->up));
    return ld.matrix(p + "down", width, ff, &L->down);
}

int32_t load_plain_ff(const Loader& ld, const std::string& p, int ff, Activation act, HybridLayer* L) {
    const int width = ld.m->hybrid->width;
    L->ff = FF_PLAIN;
    L->act = act;
    W_TRY(ld.matrix(p + "up", ff, width, &L->up));
    return ld.matrix(p + "down", width, ff, &L->down);
}

// Experts chosen by the token id through a table, with equal weights.
int32_t load_table_experts(const Loader& ld, const std::string& p, const JsonValue& mlp, Activation act, HybridLayer* L) {
    HybridModel& hm = *ld.m->hybrid;
    const int ff = mlp.at("expert").count("ff"), vocab = (int)ld.m->cfg.vocab_size;
    L->ff = FF_EXPERTS;
    L->act = act;
    L->experts = mlp.at("router").count("experts");
    L->top = mlp.at("router").count("top");
    if (L->experts > MAX_EXPERTS) return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": at most " + std::to_string(MAX_EXPERTS) + " experts");
    W_TRY(ld.expert_matrices(p, "gate", L->experts, ff, hm.width, &L->gate));
    W_TRY(ld.expert_matrices(p, "up", L->experts, ff, hm.width, &L->up));
    W_TRY(ld.expert_matrices(p, "down", L->experts, hm.width, ff, &L->down));
    const SafeTensor& t = ld.t.get(p + "table", {vocab, L->top}, "I32");
    std::vector<int> table(t.elems());
    memcpy(table.data(), t.data, t.elems() * 4);
    for (int e : table)
        if (e < 0 || e >= L->experts) return fail(WICK_CUDA_ERR_BAD_MODEL, p + "table: no expert " + std::to_string(e));
    int* dev = nullptr;
    W_TRY(ld.put(table, &dev));
    L->table = dev;
    L->route = (int)hm.routes.size();
    RouteJob r;
    r.table = dev;
    r.experts = L->experts;
    r.top = L->top;
    hm.routes.push_back(r);
    hm.max_top = std::max(hm.max_top, L->top);
    return WICK_CUDA_OK;
}

// ── the parts all architectures share ──────────────────────────────────────
const JsonValue& begin_model(wick_cuda_model* m, const JsonValue& config, uint32_t context_size, int32_t compute) {
    m->hybrid.reset(new HybridModel());
    HybridModel& hm = *m->hybrid;
    hm.bf16 = compute != WICK_CUDA_COMPUTE_F32;
    hm.width = config.count("width");
    hm.eps = (float)config.at("norm").number("eps");
    const JsonValue& list = config.at("layers");
    if (!list.is_array() || list.items.empty()) throw std::runtime_error("layers must be a list");
    if (hm.width > 48 * 1024) throw std::runtime_error("width must be at most 49152");
    wick_cuda_config& c = m->cfg;
    c.n_layers = (uint32_t)list.items.size();
    c.hidden_size = (uint32_t)hm.width;
    c.vocab_size = (uint32_t)config.count("vocab");
    c.max_seq_len = context_size;
    c.rms_norm_eps = hm.eps;
    choose_max_chunk(m);
    hm.layers.resize(c.n_layers);
    return list;
}

int32_t load_mixer(const Loader& ld, const std::string& p, const JsonValue& lc, HybridLayer* L) {
    L->type = lc.at("type").str;
    const std::string kind = mechanism(L->type);
    for (const MixerEntry& e : MIXERS)
        if (kind == e.name) return e.load(ld, p + "mix.", lc.at("mixer"), L);
    return fail(WICK_CUDA_ERR_BAD_MODEL, p + ": unknown mixer type " + L->type);
}

int32_t end_model(wick_cuda_model* m) {
    HybridModel& hm = *m->hybrid;
    const HybridLoop& lp = hm.loop;
    const int n = (int)hm.layers.size();
    for (int i = 0; i < n; i++) {
        if (lp && i == lp.start)
            for (int t = 0; t < lp.times; t++)
                for (int k = lp.start; k < lp.stop; k++) hm.runs.push_back({k, k == lp.start ? t : -1});
        if (!lp || i < lp.start || i >= lp.stop) hm.runs.push_back({i, -1});
    }
    m->layers.resize(hm.runs.size());
    for (size_t r = 0; r < hm.runs.size(); r++) describe_state(hm.layers[hm.runs[r].layer], hm.bf16, &m->layers[r]);
    return hybrid_alloc_scratch(m);
}

}  // namespace

int32_t nositar_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute) {
    const JsonValue& list = begin_model(m, config, context_size, compute);
    HybridModel& hm = *m->hybrid;
    hm.streams = config.count_or("streams", 1);
    hm.embed_scale = (float)(config.find("embedding") ? config.at("embedding").number_or("scale", 1.0) : 1.0);
    hm.softcap = (float)config.number_or("logit_softcap", 0.0);
    if (hm.streams < 1 || hm.streams > HYPER_MAX_STREAMS) return fail(WICK_CUDA_ERR_BAD_MODEL, "streams must be 1 .. " + std::to_string(HYPER_MAX_STREAMS));
    const Loader ld{m, tensors};
    W_TRY(ld.matrix("embed", (int)m->cfg.vocab_size, hm.width, &hm.embed));
    W_TRY(ld.matrix("head", (int)m->cfg.vocab_size, hm.width, &hm.head));
    W_TRY(ld.vec("final.norm", {}, &hm.final_gain));
    for (size_t i = 0; i < hm.layers.size(); i++) {
        const JsonValue& lc = list.items[i];
        HybridLayer& L = hm.layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        W_TRY(load_mixer(ld, p, lc, &L));
        W_TRY(ld.hyper(p, 1, hm.streams, &L.sub1));
        if (const JsonValue* mlp = lc.find("mlp"); mlp && mlp->is_object()) {
            const std::string kind = mlp->at("kind").str;
            if (kind != "dense") return fail(WICK_CUDA_ERR_BAD_MODEL, "layer " + std::to_string(i) + ": unknown feed-forward kind " + kind);
            W_TRY(load_gated_ff(ld, p + "mlp.", mlp->count("ff"), ACT_RELU, &L));
            W_TRY(ld.hyper(p, 2, hm.streams, &L.sub2));
        }
    }
    return end_model(m);
}

int32_t novorax_build(wick_cuda_model* m, const JsonValue& config, const SafeTensors& tensors, uint32_t context_size, int32_t compute) {
    const JsonValue& list = begin_model(m, config, context_size, compute);
    HybridModel& hm = *m->hybrid;
    hm.logit_scale = (float)config.number_or("logit_scale", 1.0);
    const Loader ld{m, tensors};
    const int n = (int)hm.layers.size(), W = hm.width;
    W_TRY(ld.matrix("embed", (int)m->cfg.vocab_size, W, &hm.embed));
    W_TRY(ld.matrix("head", (int)m->cfg.vocab_size, W, &hm.head));
    W_TRY(ld.gain("final.norm", W, &hm.final_gain));
    if (const JsonValue* lp = config.find("loop"); lp && lp->is_object()) {
        hm.loop.start = lp->count_or("start", 0);
        hm.loop.stop = lp->count_or("stop", n);
        hm.loop.times = lp->count("times");
        if (hm.loop.start >= hm.loop.stop || hm.loop.stop > n || hm.loop.times > 4096) return fail(WICK_CUDA_ERR_BAD_MODEL, "loop: no such layers");
        W_TRY(ld.matrix("loop.in", W, 2 * W, &hm.loop.in));
        W_TRY(ld.vec("loop.step", {hm.loop.times, W}, &hm.loop.step));
    }
    for (int i = 0; i < n; i++) {
        const JsonValue& lc = list.items[i];
        HybridLayer& L = hm.layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        W_TRY(load_mixer(ld, p, lc, &L));
        W_TRY(ld.norms_around(p, 1, W, &L.sub1));
        if (const JsonValue* mlp = lc.find("mlp"); mlp && mlp->is_object()) {
            const std::string kind = mlp->at("kind").str;
            if (kind == "dense") W_TRY(load_plain_ff(ld, p + "mlp.", mlp->count("ff"), ACT_RELU2, &L));
            else if (kind == "moe") W_TRY(load_table_experts(ld, p + "mlp.", *mlp, ACT_SILU, &L));
            else return fail(WICK_CUDA_ERR_BAD_MODEL, "layer " + std::to_string(i) + ": unknown feed-forward kind " + kind);
            W_TRY(ld.norms_around(p, 2, W, &L.sub2));
        }
    }
    return end_model(m);
}

}  // namespace wick
