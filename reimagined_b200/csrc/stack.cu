// The step of a layer-stack model: state layout, scratch, and the host routine that enqueues a whole step -- a portion
// of a prompt or one token of several sequences -- on one stream.  No allocation, no synchronisation; positions live on
// the device, so a caller can capture a decode step in a CUDA graph and replay it per token.
#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

size_t elem(int precision) { return precision == TBL_BF16 ? 2 : 4; }

struct StateLayout {
    int32_t* positions;                        // [slots]
    uint8_t* layer[TBL_MAX_STACK_LAYERS];      // delta-rule states fp32, the latent cache, or the attention cache (maybe another layer's)
    size_t slot_bytes[TBL_MAX_STACK_LAYERS];
    size_t bytes;
};

StateLayout carve_state(const tbl_stack_model& m, int precision, int slots, int capacity, void* base) {
    StateLayout L{};
    uint8_t* p = static_cast<uint8_t*>(base);
    size_t off = 0;
    auto take = [&](size_t bytes) { uint8_t* r = p + off; off += round_up(bytes, 256); return r; };
    L.positions = reinterpret_cast<int32_t*>(take(sizeof(int32_t) * slots));
    for (int i = 0; i < m.n_layers; ++i) {
        const tbl_stack_layer& l = m.layers[i];
        if (l.mixer == TBL_MIXER_ATTENTION && l.attention.kv_from >= 0) {
            L.layer[i] = L.layer[l.attention.kv_from];
            L.slot_bytes[i] = L.slot_bytes[l.attention.kv_from];
            continue;
        }
        if (l.mixer == TBL_MIXER_GENERAL_DELTA) L.slot_bytes[i] = sizeof(float) * static_cast<size_t>(l.delta.heads) * l.delta.dim * l.delta.dim;
        else if (l.mixer == TBL_MIXER_LATENT_ATTENTION) L.slot_bytes[i] = elem(precision) * static_cast<size_t>(capacity) * latent_cache_width(l.latent);
        else L.slot_bytes[i] = elem(precision) * static_cast<size_t>(capacity) * l.attention.kv_heads * attention_cache_width(l.attention);
        L.layer[i] = take(L.slot_bytes[i] * slots);
    }
    L.bytes = off;
    return L;
}

struct Scratch {
    float* history;          // [n_layers + 1][rows][width]: embedding output, then every layer's result; or the residual streams
    float* x[2];             // residual stream between averages; with several streams x[0] is a sublayer's result
    float* proj;
    void *h, *mixed, *hidden, *mixer;
    size_t stride, bytes;
};

Scratch carve_scratch(const tbl_stack_model& m, int precision, int n_seq, int n_tok, int context, void* base) {
    Scratch S{};
    uint8_t* p = static_cast<uint8_t*>(base);
    size_t off = 0;
    auto take = [&](size_t bytes) { uint8_t* r = p + off; off += round_up(bytes, 256); return r; };
    const size_t rows = static_cast<size_t>(n_seq) * n_tok, e = elem(precision);
    size_t proj = 1, mixed = 1, ff = 1, mixer = 1;
    auto most = [](size_t& a, size_t b) { if (b > a) a = b; };
    for (int i = 0; i < m.n_layers; ++i) {
        const tbl_stack_layer& l = m.layers[i];
        if (l.mixer == TBL_MIXER_GENERAL_DELTA) {
            most(proj, l.delta.in.outputs);
            most(mixed, static_cast<size_t>(l.delta.heads) * l.delta.dim);
            most(mixer, delta_workspace(l.delta, precision, static_cast<int>(rows)));
        } else if (l.mixer == TBL_MIXER_LATENT_ATTENTION) {
            most(proj, l.latent.in.outputs);
            most(mixed, static_cast<size_t>(l.latent.heads) * l.latent.vdim);
            most(mixer, latent_workspace(l.latent, precision, n_seq, n_tok, context));
        } else {
            most(proj, l.attention.in.outputs);
            most(mixed, static_cast<size_t>(l.attention.heads) * l.attention.vdim);
            most(mixer, attention_workspace(l.attention, precision, n_seq, n_tok, context));
        }
        most(ff, round_up(l.ff, 8));
    }
    S.stride = round_up(rows * m.width, 64);
    S.history = reinterpret_cast<float*>(take(sizeof(float) * S.stride * (m.streams ? m.streams : m.n_layers + 1)));
    S.x[0] = reinterpret_cast<float*>(take(sizeof(float) * rows * m.width));
    S.x[1] = reinterpret_cast<float*>(take(sizeof(float) * rows * m.width));
    S.proj = reinterpret_cast<float*>(take(sizeof(float) * rows * proj));
    S.h = take(e * rows * m.width);
    S.mixed = take(e * rows * mixed);
    S.hidden = take(e * rows * ff);
    S.mixer = take(mixer);
    S.bytes = off;
    return S;
}

bool dense_ok(const tbl_dense_view& v, int inputs, int outputs) {
    return v.weight && !(reinterpret_cast<uintptr_t>(v.weight) & 15) && v.inputs == inputs && v.outputs == outputs;
}

bool hyper_ok(const tbl_hyper& h) { return h.in && h.mix && h.out; }

int check_model(const tbl_stack_model* m, int precision) {
    if (!m || !m->layers || !m->embedding || !m->final_norm) return TBL_ERR_INVALID_ARG;
    if (precision != TBL_F32 && precision != TBL_BF16) return TBL_ERR_INVALID_ARG;
    if (m->width <= 0 || m->vocab <= 0 || m->n_layers <= 0 || m->n_layers > TBL_MAX_STACK_LAYERS) return TBL_ERR_INVALID_ARG;
    if (m->streams < 0 || m->streams > TBL_MAX_STREAMS) return TBL_ERR_UNSUPPORTED;
    const bool tanh_norm = m->norm_kind == TBL_NORM_DYNAMIC_TANH;
    if (!tanh_norm && m->norm_kind != TBL_NORM_RMS) return TBL_ERR_UNSUPPORTED;
    if (tanh_norm && !m->final_tanh.bias) return TBL_ERR_INVALID_ARG;
    for (int i = 0; i < m->n_layers; ++i) {
        const tbl_stack_layer& l = m->layers[i];
        int rc;
        if (l.mixer == TBL_MIXER_GENERAL_DELTA) rc = check_delta(l.delta, m->width);
        else if (l.mixer == TBL_MIXER_LATENT_ATTENTION) rc = check_latent(l.latent, m->width);
        else if (l.mixer == TBL_MIXER_ATTENTION) rc = check_attention(l.attention, m->width);
        else return TBL_ERR_UNSUPPORTED;
        if (rc != TBL_OK) return rc;
        if (l.mixer == TBL_MIXER_ATTENTION && l.attention.kv_from >= 0) {
            if (l.attention.kv_from >= i) return TBL_ERR_INVALID_ARG;
            const tbl_stack_layer& o = m->layers[l.attention.kv_from];
            if (o.mixer != TBL_MIXER_ATTENTION || o.attention.kv_from >= 0) return TBL_ERR_INVALID_ARG;
            if (o.attention.kv_heads != l.attention.kv_heads || o.attention.maps != l.attention.maps || o.attention.dim != l.attention.dim ||
                o.attention.vdim != l.attention.vdim)
                return TBL_ERR_SHAPE;
        }
        if (!l.norm1 || l.ff < 0) return TBL_ERR_INVALID_ARG;
        if ((tanh_norm && !l.tanh1.bias) || (m->streams && (!hyper_ok(l.hyper1) || l.depth_weights))) return TBL_ERR_INVALID_ARG;
        if (l.ff > 0) {
            if (!l.norm2 || (tanh_norm && !l.tanh2.bias) || (m->streams && !hyper_ok(l.hyper2))) return TBL_ERR_INVALID_ARG;
            if (l.activation != TBL_ACT_SILU && l.activation != TBL_ACT_GELU_TANH) return TBL_ERR_UNSUPPORTED;
            if (!dense_ok(l.gate_up, m->width, 2 * static_cast<int>(round_up(l.ff, TBL_PAIR_BLOCK))) || !dense_ok(l.down, l.ff, m->width))
                return TBL_ERR_SHAPE;
        }
    }
    return dense_ok(m->head, m->width, m->vocab) ? TBL_OK : TBL_ERR_SHAPE;
}

}  // namespace
}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" {

size_t tbl_stack_state_bytes(const tbl_stack_model* model, int precision, int slots, int capacity) {
    if (check_model(model, precision) != TBL_OK || slots <= 0 || capacity <= 0) return 0;
    return carve_state(*model, precision, slots, capacity, nullptr).bytes;
}

int tbl_stack_state_reset(const tbl_stack_model* model, int precision, int slots, int capacity, int slot, void* state_dev,
                          size_t state_bytes, void* stream) {
    const int rc = check_model(model, precision);
    if (rc != TBL_OK) return rc;
    if (slots <= 0 || capacity <= 0 || slot >= slots) return TBL_ERR_INVALID_ARG;
    if (!state_dev || state_bytes < tbl_stack_state_bytes(model, precision, slots, capacity)) return TBL_ERR_WORKSPACE;
    const StateLayout L = carve_state(*model, precision, slots, capacity, state_dev);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (slot < 0) return cudaMemsetAsync(state_dev, 0, L.bytes, st) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
    if (cudaMemsetAsync(L.positions + slot, 0, sizeof(int32_t), st) != cudaSuccess) return TBL_ERR_CUDA;
    for (int i = 0; i < model->n_layers; ++i) {
        if (model->layers[i].mixer != TBL_MIXER_GENERAL_DELTA) continue;
        if (cudaMemsetAsync(L.layer[i] + slot * L.slot_bytes[i], 0, L.slot_bytes[i], st) != cudaSuccess) return TBL_ERR_CUDA;
    }
    return TBL_OK;
}

size_t tbl_stack_workspace_bytes(const tbl_stack_model* model, int precision, int n_seq, int n_tok, int context) {
    if (check_model(model, precision) != TBL_OK || n_seq <= 0 || n_tok <= 0 || context <= 0) return 0;
    return carve_scratch(*model, precision, n_seq, n_tok, context, nullptr).bytes;
}

int tbl_stack_step(const tbl_stack_model* model, int precision, int slots, int capacity, void* state_dev, const int32_t* slots_dev,
                   int n_seq, int n_tok, int context, const int32_t* tokens_dev, const int32_t* want_rows_dev, int n_want,
                   float* logits_dev, float* hidden_trace_dev, void* workspace_dev, size_t workspace_bytes, void* stream) {
    int rc = check_model(model, precision);
    if (rc != TBL_OK) return rc;
    if (!state_dev || !slots_dev || !tokens_dev || slots <= 0 || capacity <= 0 || n_seq <= 0 || n_seq > slots || n_tok <= 0 ||
        context < n_tok || context > capacity || n_want < 0 || n_want > n_seq * n_tok || (n_want > 0 && (!want_rows_dev || !logits_dev)))
        return TBL_ERR_INVALID_ARG;
    if (!workspace_dev || workspace_bytes < tbl_stack_workspace_bytes(model, precision, n_seq, n_tok, context)) return TBL_ERR_WORKSPACE;
    if ((reinterpret_cast<uintptr_t>(workspace_dev) & 255) || (reinterpret_cast<uintptr_t>(state_dev) & 255)) return TBL_ERR_ALIGNMENT;
    const tbl_stack_model& m = *model;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const StateLayout state = carve_state(m, precision, slots, capacity, state_dev);
    const Scratch S = carve_scratch(m, precision, n_seq, n_tok, context, workspace_dev);
    const int rows = n_seq * n_tok, W = m.width;

    auto linear = [&](const tbl_dense_view& v, const void* x, int ldx, float* out, const float* residual) {
        DenseCall c{};
        c.x = x; c.w = static_cast<const bf16*>(v.weight); c.bias = v.bias; c.ldx = ldx; c.M = rows; c.K = v.inputs; c.N = v.outputs;
        c.out_f32 = out; c.ldo = v.outputs; c.residual = residual;
        return launch_dense(precision, kDenseAuto, c, st);
    };
    // layer i's mixer on the normed rows S.h: out = result [+ residual]
    auto mixer = [&](int i, float* out, const float* residual) {
        const tbl_stack_layer& l = m.layers[i];
        if (l.mixer == TBL_MIXER_GENERAL_DELTA) {
            int e = linear(l.delta.in, S.h, W, S.proj, nullptr);
            if (e == TBL_OK)
                e = launch_delta(l.delta, precision, 0, m.norm_eps, S.proj, reinterpret_cast<float*>(state.layer[i]), slots_dev, n_seq, n_tok,
                                 S.mixed, S.mixer, st);
            return e == TBL_OK ? linear(l.delta.out, S.mixed, l.delta.heads * l.delta.dim, out, residual) : e;
        }
        if (l.mixer == TBL_MIXER_LATENT_ATTENTION) {
            int e = linear(l.latent.in, S.h, W, S.proj, nullptr);
            if (e == TBL_OK)
                e = launch_latent(l.latent, precision, 0, m.norm_eps, S.proj, state.layer[i], capacity, slots_dev, state.positions, n_seq, n_tok,
                                  context, S.mixed, S.mixer, st);
            return e == TBL_OK ? linear(l.latent.out, S.mixed, l.latent.heads * l.latent.vdim, out, residual) : e;
        }
        int e = linear(l.attention.in, S.h, W, S.proj, nullptr);
        if (e == TBL_OK)
            e = launch_attention(l.attention, precision, 0, m.norm_eps, S.proj, state.layer[i], slots, capacity, slots_dev, state.positions,
                                 n_seq, n_tok, context, S.mixed, S.mixer, st);
        return e == TBL_OK ? linear(l.attention.out, S.mixed, l.attention.heads * l.attention.vdim, out, residual) : e;
    };
    auto feed_forward = [&](int i, float* out, const float* residual) {
        const tbl_stack_layer& l = m.layers[i];
        DenseCall c{};
        const int ldf = static_cast<int>(round_up(l.ff, 8));
        c.x = S.h; c.w = static_cast<const bf16*>(l.gate_up.weight); c.bias = l.gate_up.bias; c.ldx = W; c.M = rows; c.K = W;
        c.N = l.gate_up.outputs; c.ldo = ldf; c.pair_cols = l.ff; c.act = l.activation;
        if (precision == TBL_BF16) c.out_b16 = static_cast<bf16*>(S.hidden); else c.out_f32 = static_cast<float*>(S.hidden);
        const int e = launch_dense(precision, kDenseAuto, c, st);
        return e == TBL_OK ? linear(l.down, S.hidden, ldf, out, residual) : e;
    };
    // the norm that opens a sublayer (the model's last one: sublayer 0), over `count` arrays of the history
    auto norm_of = [&](int layer, int sublayer, int count) {
        DepthNorm p{};
        p.history = S.history; p.stride = S.stride; p.count = count; p.rows = rows; p.width = W; p.eps = m.norm_eps; p.norm_kind = m.norm_kind;
        const bool final = sublayer == 0;
        const tbl_stack_layer& l = m.layers[final ? 0 : layer];
        const tbl_tanh_norm& t = final ? m.final_tanh : (sublayer == 1 ? l.tanh1 : l.tanh2);
        p.norm = final ? m.final_norm : (sublayer == 1 ? l.norm1 : l.norm2);
        p.alpha = t.alpha; p.norm_bias = t.bias; p.h = S.h;
        if (m.streams) {
            p.streams = m.streams; p.stream = S.history; p.store = !final;
            p.weights = final ? nullptr : (sublayer == 1 ? l.hyper1.in : l.hyper2.in);
        }
        return p;
    };
    // with streams: the result S.x[0] of a sublayer goes into them
    auto update_by = [&](DepthNorm& p, const tbl_hyper& h) { p.y = S.x[0]; p.mix = h.mix; p.out_weights = h.out; };

    // the embedding output is the first entry of the history and the first residual stream, or every one of the streams
    DepthNorm first = norm_of(0, 1, 1);
    first.tokens = tokens_dev; first.table = static_cast<const bf16*>(m.embedding); first.vocab = m.vocab; first.embed_scale = m.embedding_scale;
    if (!m.streams) first.x = S.history;
    rc = launch_depth_norm(precision, first, st);
    if (rc != TBL_OK) return rc;

    const int last_layer = m.n_layers - 1;
    const float* x = S.history;
    for (int i = 0; i < m.n_layers; ++i) {
        const tbl_stack_layer& l = m.layers[i];
        const bool last = i == last_layer;
        float* trace = hidden_trace_dev ? hidden_trace_dev + static_cast<size_t>(i) * rows * W : nullptr;
        if (m.streams) {
            rc = mixer(i, S.x[0], nullptr);
            if (rc != TBL_OK) return rc;
            if (l.ff) {
                DepthNorm q = norm_of(i, 2, 1);
                update_by(q, l.hyper1);
                rc = launch_depth_norm(precision, q, st);
                if (rc == TBL_OK) rc = feed_forward(i, S.x[0], nullptr);
                if (rc != TBL_OK) return rc;
            }
            // close the layer; after the last one the sum of the streams is only needed where asked for
            if (!last || trace) {
                DepthNorm q = last ? norm_of(0, 0, 1) : norm_of(i + 1, 1, 1);
                update_by(q, l.ff ? l.hyper2 : l.hyper1);
                q.trace = trace;
                if (last) q.h = nullptr;
                rc = launch_depth_norm(precision, q, st);
                if (rc != TBL_OK) return rc;
            }
            continue;
        }
        float* result = S.history + (i + 1) * S.stride;
        float* after_mixer = l.ff ? S.x[1] : result;
        rc = mixer(i, after_mixer, x);
        if (rc != TBL_OK) return rc;
        if (l.ff) {
            DepthNorm q = norm_of(i, 2, 1);
            q.history = after_mixer;
            rc = launch_depth_norm(precision, q, st);
            if (rc == TBL_OK) rc = feed_forward(i, result, after_mixer);
            if (rc != TBL_OK) return rc;
        }
        // close the layer: learned average over the depth, next layer's norm (the last one is only needed where asked for)
        const float* weights = l.depth_weights;
        if (!last || trace) {
            DepthNorm q = last ? norm_of(0, 0, i + 2) : norm_of(i + 1, 1, i + 2);
            q.weights = weights;
            if (last) q.h = nullptr;
            q.x = weights && !last ? S.x[0] : nullptr;
            q.trace = trace;
            rc = launch_depth_norm(precision, q, st);
            if (rc != TBL_OK) return rc;
            x = weights ? S.x[0] : result;
        }
    }
    DepthNorm f = norm_of(0, 0, m.n_layers + 1);
    if (m.streams) update_by(f, m.layers[last_layer].ff ? m.layers[last_layer].hyper2 : m.layers[last_layer].hyper1);
    else f.weights = m.layers[last_layer].depth_weights;
    f.row_index = want_rows_dev; f.rows = n_want > 0 ? n_want : 1;
    f.positions = state.positions; f.slots = slots_dev; f.n_seq = n_seq; f.n_tok = n_tok;
    if (n_want == 0) { f.row_index = nullptr; f.h = nullptr; }
    rc = launch_depth_norm(precision, f, st);
    if (rc != TBL_OK || n_want == 0) return rc;
    DenseCall c{};
    c.x = S.h; c.w = static_cast<const bf16*>(m.head.weight); c.bias = m.head.bias; c.ldx = W; c.M = n_want; c.K = W; c.N = m.vocab;
    c.out_f32 = logits_dev; c.ldo = m.vocab;
    return launch_dense(precision, kDenseAuto, c, st);
}

}  // extern "C"
