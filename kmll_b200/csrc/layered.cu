// Layered decoders: pre-norm layers from a list of descriptions, bf16 weights.  A layer holds one mixer or two side by side
// (latent attention, grouped attention, linear attention with a fixed decay per head or with a decay per key channel and token)
// and perhaps a feed-forward.  The decode loop, the graph, the pending token, the history and the session-level entry points are
// those of runtime.cu; this file holds the weights, the caches and states, the decode step and the prompt path.
//
// Decode step, per layer (f32 activations, one launch each):
//   norm + stacked projection of every mixer | each mixer | norms / gates / scales + output projection of every mixer + residual
//   | norm + up (gated: act(gate) * up) | (PolyNorm) + down + residual      then norm + lm_head + arg-max + end of the step
// Prompt path: the same in rows, up to kMaxRows tokens at a time; bf16 activations on tcgen05, or f32 throughout.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "decoder.cuh"

namespace kmll {

namespace {

constexpr int kMaxRows = 4096;  // tokens per pass of the prompt path
inline int up8(int v) { return (v + 7) & ~7; }

struct Mat {
    uint16_t* w = nullptr;
    int rows = 0, cols = 0, ld = 0;
};

// A mixer of a layer.  Its projections are rows of the layer's stacked matrix (offsets below), its output is columns
// [o_off, o_off + width()) of the vector that the layer's output projection reads.
struct LMixer {
    kmll_mixer_spec sp;
    int off_q = 0, off_k = 0, off_v = 0, off_g = 0;  // latent: off_k = the latent's; off_g = output gate
    int off_a = 0, off_b = 0, off_gd = 0;            // gated linear: decay and gate factors, write strength
    int o_off = 0;
    uint16_t *mix_norm = nullptr, *dkv_norm = nullptr, *decay_bias = nullptr, *decay_log = nullptr, *conv = nullptr;
    Mat ukv, decay_up, gate_up;
    float2* table = nullptr;   // rotation [max_seq][rot / 2]
    float* powers = nullptr;   // [heads][kLinChunk + 1]
    bool decay_set = false, table_set = false;
    size_t state_off = 0, ring_off = 0;  // within Layered::states
    void* cache = nullptr;
    int pitch = 0, kr_off = 0;
    int width() const { return sp.heads * sp.vdim; }
    int kv_heads() const { return sp.kv_heads > 0 ? sp.kv_heads : sp.heads; }
    int conv_channels() const { return 2 * kv_heads() * sp.dim + width(); }
};

struct LLayer {
    int n_mix = 0, mlp = 0, mlp_act = 0, ff = 0;
    LMixer mix[2];
    uint16_t *norm1 = nullptr, *norm2 = nullptr, *norm1_b = nullptr, *norm2_b = nullptr, *act = nullptr;
    Mat proj, wo, up, down;    // up: gated feed-forward: rows 2 i and 2 i + 1 = row i of gate and up
    int width = 0;             // columns of wo
};

}  // namespace

struct Layered {
    kmll_layered_config cfg;
    bool plain = false;  // plain kernels also where faster forms exist
    std::vector<LLayer> layers;
    uint16_t *pos_table = nullptr, *final_norm_b = nullptr, *embed_norm = nullptr, *embed_norm_b = nullptr;
    Mat embed;  // its rows are the decoder's embedding table
    Mat head;   // tied: the same matrix
    float* logits = nullptr;
    unsigned int* counter = nullptr;
    uint32_t* token_log = nullptr;  // [max_seq] tokens of the sequence by position
    float* states = nullptr;
    size_t state_floats = 0;
    // remembered states (rewind) and the copy held around a warm-up step
    float *saved = nullptr, *saved_logits = nullptr, *held = nullptr;
    int saved_at = -1;
    // one-token scratch
    float *proj1 = nullptr, *o1 = nullptr, *z1 = nullptr, *work = nullptr, *gate1 = nullptr;
    // prompt scratch for `rows` tokens
    int rows = 0;
    std::vector<void*> row_allocs;
    float *x = nullptr, *o = nullptr, *lin = nullptr, *gate = nullptr;
    int ldo = 0, max_gate = 0;
    float* gemm_partial = nullptr;        // scratch of the projections over few rows
    unsigned int* gemm_counters = nullptr;
    void *a = nullptr, *p = nullptr, *z = nullptr;
    int* want = nullptr;
    void* expanded = nullptr;
    size_t expanded_bytes = 0;
    int lda = 0, ldp = 0, ldz = 0;
    float* tap = nullptr;
};

namespace {

int alloc_mat(Decoder* d, Mat* m, int rows, int cols) {
    m->rows = rows;
    m->cols = cols;
    m->ld = up8(cols);
    const size_t n = (size_t)rows * m->ld;
    KMLL_TRY(dalloc(d, &m->w, n));
    KMLL_CUDA(cudaMemset(m->w, 0, n * 2));
    d->weight_bytes += n * 2;
    return KMLL_OK;
}
int alloc_vec(Decoder* d, uint16_t** v, size_t n) {
    KMLL_TRY(dalloc(d, v, n));
    d->weight_bytes += n * 2;
    return KMLL_OK;
}

int validate_mixer(const kmll_mixer_spec& s, int l, bool beside) {
    if (s.mixer < KMLL_MIXER_LATENT_ATTENTION || s.mixer > KMLL_MIXER_GATED_LINEAR) return fail(KMLL_ERR_SHAPE, "layer %d: unknown mixer %d", l, s.mixer);
    if (s.heads <= 0 || s.dim <= 0 || s.vdim <= 0) return fail(KMLL_ERR_SHAPE, "layer %d: head sizes must be positive", l);
    if (beside && s.mixer != KMLL_MIXER_ATTENTION && s.mixer != KMLL_MIXER_GATED_LINEAR)
        return fail(KMLL_ERR_UNSUPPORTED, "layer %d: a second mixer is grouped or gated linear attention", l);
    if (s.rot_dim < 0 || (s.rot_dim & 1)) return fail(KMLL_ERR_SHAPE, "layer %d: rot_dim must be even", l);
    if (s.window < 0 || s.chunk < 0) return fail(KMLL_ERR_SHAPE, "layer %d: bad window or chunk", l);
    if (s.kv_heads < 0 || (s.kv_heads > 0 && s.heads % s.kv_heads != 0)) return fail(KMLL_ERR_SHAPE, "layer %d: %d heads over %d key / value heads", l, s.heads, s.kv_heads);
    switch (s.mixer) {
        case KMLL_MIXER_LATENT_ATTENTION:
            if (s.kv_rank <= 0) return fail(KMLL_ERR_SHAPE, "layer %d: bad latent size", l);
            break;
        case KMLL_MIXER_LINEAR_ATTENTION:
            if (s.rot_dim > s.dim) return fail(KMLL_ERR_SHAPE, "layer %d: rot_dim exceeds the key size", l);
            if (s.dim > 512) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: key size %d above 512", l, s.dim);
            if (s.qkv_act != KMLL_ACT_NONE && s.qkv_act != KMLL_ACT_SILU) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: q, k, v go through SiLU or nothing", l);
            if (s.out_norm != KMLL_OUT_NORM_PER_HEAD && s.out_norm != KMLL_OUT_NORM_JOINT) return fail(KMLL_ERR_SHAPE, "layer %d: bad output norm", l);
            break;
        case KMLL_MIXER_ATTENTION:
            if (s.rot_dim != 0) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: grouped attention has no rotation", l);
            if (s.window > 0 && s.chunk > 0) return fail(KMLL_ERR_SHAPE, "layer %d: a window and a chunk", l);
            break;
        default:
            if (s.rot_dim != 0) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: gated linear attention has no rotation", l);
            if (s.dim > 512) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: key size %d above 512", l, s.dim);
            if (s.decay != KMLL_DECAY_LOGISTIC && s.decay != KMLL_DECAY_SOFTPLUS) return fail(KMLL_ERR_SHAPE, "layer %d: unknown decay %d", l, s.decay);
            if (s.decay == KMLL_DECAY_LOGISTIC && !(s.decay_tau > 0.0f)) return fail(KMLL_ERR_SHAPE, "layer %d: decay_tau must be positive", l);
            if (s.decay_rank <= 0 || s.gate_rank < 0 || s.unit_eps < 0.0f) return fail(KMLL_ERR_SHAPE, "layer %d: bad rank", l);
            if (s.conv < 0 || s.conv > kMaxConvTaps) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: %d taps, at most %d", l, s.conv, kMaxConvTaps);
            if (s.out_norm != KMLL_OUT_NORM_HEAD_WEIGHTED && s.out_norm != KMLL_OUT_NORM_PER_HEAD) return fail(KMLL_ERR_SHAPE, "layer %d: bad output norm", l);
            break;
    }
    return KMLL_OK;
}

int validate(const kmll_layered_config& c, const kmll_layer_spec* specs) {
    if (c.n_layers <= 0 || c.dim <= 0 || c.vocab_size <= 0 || c.max_seq_len <= 0) return fail(KMLL_ERR_SHAPE, "layered decoder: every size must be positive");
    if (c.position_rows > 0 && c.max_seq_len > c.position_rows)
        return fail(KMLL_ERR_SHAPE, "layered decoder: max_seq_len %d exceeds the %d learned positions", c.max_seq_len, c.position_rows);
    if (c.norm != KMLL_NORM_RMS && c.norm != KMLL_NORM_LAYER) return fail(KMLL_ERR_SHAPE, "layered decoder: unknown norm %d", c.norm);
    for (int l = 0; l < c.n_layers; ++l) {
        const kmll_layer_spec& s = specs[l];
        KMLL_TRY(validate_mixer(s.mixers[0], l, false));
        if (s.mixers[1].mixer != KMLL_MIXER_NONE) KMLL_TRY(validate_mixer(s.mixers[1], l, true));
        if (s.mlp < KMLL_MLP_NONE || s.mlp > KMLL_MLP_GATED || (s.mlp != KMLL_MLP_NONE && s.ff <= 0)) return fail(KMLL_ERR_SHAPE, "layer %d: bad feed-forward", l);
        if (s.mlp == KMLL_MLP_GATED && s.mlp_act != KMLL_ACT_SILU && s.mlp_act != KMLL_ACT_GELU_TANH) return fail(KMLL_ERR_SHAPE, "layer %d: unknown activation %d", l, s.mlp_act);
    }
    return KMLL_OK;
}

// where the rows of a mixer's projections lie in the layer's stacked matrix; returns the first row behind them
int place_rows(LMixer* m, int base) {
    const kmll_mixer_spec& s = m->sp;
    const int g = m->kv_heads();
    m->off_q = base;
    switch (s.mixer) {
        case KMLL_MIXER_LATENT_ATTENTION:
            m->off_k = base + s.heads * (s.dim + s.rot_dim);
            return m->off_k + s.kv_rank + s.rot_dim;
        case KMLL_MIXER_LINEAR_ATTENTION:
            m->off_k = base + s.heads * s.dim;
            m->off_v = m->off_k + s.heads * s.dim;
            m->off_g = m->off_v + s.heads * s.vdim;
            return m->off_g + s.heads * s.vdim;
        case KMLL_MIXER_ATTENTION:
            m->off_k = base + up8(s.heads * s.dim);
            m->off_v = m->off_k + up8(g * s.dim);
            m->off_g = m->off_v + up8(g * s.vdim);
            return m->off_g + (s.head_gate ? s.heads : 0);
        default:
            m->off_k = base + up8(g * s.dim);
            m->off_v = m->off_k + up8(g * s.dim);
            m->off_g = m->off_v + up8(s.heads * s.vdim);
            m->off_a = m->off_g + (s.gate_rank == 0 ? up8(s.heads * s.vdim) : 0);
            m->off_gd = m->off_a + up8(s.decay_rank);
            m->off_b = m->off_gd + up8(s.gate_rank);
            return m->off_b + (s.delta ? s.heads : 0);
    }
}

// weights, cache and state of a mixer apart from the stacked matrices
int create_mixer(Decoder* d, LMixer* m, size_t* work) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    const kmll_mixer_spec& s = m->sp;
    auto cache = [&](int pitch) -> int {
        const size_t bytes = (size_t)c.max_seq_len * pitch * (c.compute_f32 ? 4 : 2);
        uint8_t* p = nullptr;
        KMLL_TRY(dalloc(d, &p, bytes));
        KMLL_CUDA(cudaMemset(p, 0, bytes));
        m->cache = p;
        m->pitch = pitch;
        d->kv_bytes += bytes;
        return KMLL_OK;
    };
    auto state = [&](size_t floats) {
        const size_t at = L->state_floats;
        L->state_floats += (floats + 3) & ~(size_t)3;
        return at;
    };
    if (s.rot_dim > 0) KMLL_TRY(dalloc(d, &m->table, (size_t)c.max_seq_len * (s.rot_dim / 2)));
    if (s.mixer == KMLL_MIXER_LATENT_ATTENTION) {
        KMLL_TRY(alloc_vec(d, &m->dkv_norm, s.kv_rank));
        KMLL_TRY(alloc_mat(d, &m->ukv, s.heads * (s.dim + s.vdim), s.kv_rank));
        m->kr_off = up8(s.kv_rank);
        KMLL_TRY(cache(up8(m->kr_off + s.rot_dim)));
        const int span = s.window > 0 && s.window < c.max_seq_len ? s.window : c.max_seq_len;
        *work = std::max(*work, latent_decode_work_floats(s.heads, s.kv_rank, s.rot_dim, span));
    } else if (s.mixer == KMLL_MIXER_ATTENTION) {
        KMLL_TRY(cache(m->kv_heads() * (up8(s.dim) + up8(s.vdim))));
    } else {
        if (s.out_norm == KMLL_OUT_NORM_JOINT) KMLL_TRY(alloc_vec(d, &m->mix_norm, s.heads * s.vdim));
        if (s.out_norm == KMLL_OUT_NORM_HEAD_WEIGHTED) KMLL_TRY(alloc_vec(d, &m->mix_norm, s.vdim));
        m->state_off = state((size_t)s.heads * s.dim * s.vdim);
        if (s.mixer == KMLL_MIXER_LINEAR_ATTENTION) {
            KMLL_TRY(dalloc(d, &m->powers, (size_t)s.heads * (kLinChunk + 1)));
        } else {
            KMLL_TRY(alloc_mat(d, &m->decay_up, s.heads * s.dim, s.decay_rank));
            KMLL_TRY(alloc_vec(d, &m->decay_bias, (size_t)s.heads * s.dim));
            if (s.decay == KMLL_DECAY_SOFTPLUS) KMLL_TRY(alloc_vec(d, &m->decay_log, s.heads));
            if (s.conv > 0) {
                KMLL_TRY(alloc_vec(d, &m->conv, (size_t)m->conv_channels() * s.conv));
                m->ring_off = state((size_t)m->conv_channels() * s.conv);
            }
            if (s.gate_rank > 0) KMLL_TRY(alloc_mat(d, &m->gate_up, s.heads * s.vdim, s.gate_rank));
        }
    }
    return KMLL_OK;
}

int create(Decoder* d, const kmll_layered_config& c, const kmll_layer_spec* specs) {
    Layered* L = d->lay;
    L->cfg = c;
    const char* env = std::getenv("KMLL_LAYERED");
    L->plain = env != nullptr && strcmp(env, "plain") == 0;
    L->layers.resize(c.n_layers);
    const bool layer_norm = c.norm == KMLL_NORM_LAYER;
    KMLL_CUDA(cudaGetDevice(&d->device));
    KMLL_TRY(alloc_mat(d, &L->embed, c.vocab_size, c.dim));
    d->embedding = L->embed.w;
    if (c.position_rows > 0) KMLL_TRY(alloc_vec(d, &L->pos_table, (size_t)c.position_rows * c.dim));
    if (c.embed_norm) KMLL_TRY(alloc_vec(d, &L->embed_norm, c.dim));
    if (c.embed_norm && layer_norm) KMLL_TRY(alloc_vec(d, &L->embed_norm_b, c.dim));
    KMLL_TRY(alloc_vec(d, &d->final_norm, c.dim));
    if (layer_norm) KMLL_TRY(alloc_vec(d, &L->final_norm_b, c.dim));
    if (c.tie_output) L->head = L->embed;
    else KMLL_TRY(alloc_mat(d, &L->head, c.vocab_size, c.dim));
    int max_p = 0, max_o = 0, max_ff = 1;
    size_t work = 1;
    for (int l = 0; l < c.n_layers; ++l) {
        LLayer& y = L->layers[l];
        const kmll_layer_spec& s = specs[l];
        KMLL_TRY(alloc_vec(d, &y.norm1, c.dim));
        if (layer_norm) KMLL_TRY(alloc_vec(d, &y.norm1_b, c.dim));
        y.n_mix = s.mixers[1].mixer != KMLL_MIXER_NONE ? 2 : 1;
        int rows = 0;
        for (int i = 0; i < y.n_mix; ++i) {
            LMixer& m = y.mix[i];
            m.sp = s.mixers[i];
            rows = place_rows(&m, up8(rows));
            m.o_off = up8(y.width);
            y.width = m.o_off + m.width();
            KMLL_TRY(create_mixer(d, &m, &work));
            if (m.sp.mixer == KMLL_MIXER_GATED_LINEAR && m.sp.gate_rank > 0) L->max_gate = std::max(L->max_gate, m.width());
        }
        KMLL_TRY(alloc_mat(d, &y.proj, rows, c.dim));
        KMLL_TRY(alloc_mat(d, &y.wo, c.dim, y.width));
        y.mlp = s.mlp;
        y.mlp_act = s.mlp_act;
        y.ff = s.ff;
        if (s.mlp != KMLL_MLP_NONE) {
            KMLL_TRY(alloc_vec(d, &y.norm2, c.dim));
            if (layer_norm) KMLL_TRY(alloc_vec(d, &y.norm2_b, c.dim));
            KMLL_TRY(alloc_mat(d, &y.up, s.mlp == KMLL_MLP_GATED ? 2 * s.ff : s.ff, c.dim));
            KMLL_TRY(alloc_mat(d, &y.down, c.dim, s.ff));
            if (s.mlp == KMLL_MLP_POLYNORM) KMLL_TRY(alloc_vec(d, &y.act, 4));
            max_ff = std::max(max_ff, s.ff);
        }
        max_p = std::max(max_p, y.proj.rows);
        max_o = std::max(max_o, y.width);
    }
    L->lda = std::max({up8(c.dim), up8(max_o), up8(max_ff)});
    L->ldp = up8(max_p);
    L->ldz = up8(max_ff);
    L->ldo = up8(max_o);
    if (L->state_floats == 0) L->state_floats = 4;
    KMLL_TRY(dalloc(d, &L->states, L->state_floats));
    KMLL_TRY(dalloc(d, &L->saved, L->state_floats));
    KMLL_TRY(dalloc(d, &L->held, L->state_floats));
    KMLL_CUDA(cudaMemset(L->states, 0, L->state_floats * 4));
    d->kv_bytes += L->state_floats * 4;
    if (!c.compute_f32) {
        KMLL_TRY(dalloc(d, &L->gemm_partial, kGemmPartialFloats));
        KMLL_TRY(dalloc(d, &L->gemm_counters, (size_t)74));
        KMLL_CUDA(cudaMemset(L->gemm_counters, 0, 74 * 4));
    }
    KMLL_TRY(dalloc(d, &L->logits, (size_t)c.vocab_size));
    KMLL_TRY(dalloc(d, &L->saved_logits, (size_t)c.vocab_size));
    KMLL_TRY(dalloc(d, &L->counter, (size_t)4));
    KMLL_CUDA(cudaMemset(L->counter, 0, 16));
    KMLL_TRY(dalloc(d, &L->token_log, (size_t)c.max_seq_len));
    KMLL_CUDA(cudaMemset(L->token_log, 0, (size_t)c.max_seq_len * 4));
    KMLL_TRY(dalloc(d, &L->proj1, (size_t)L->ldp));
    KMLL_TRY(dalloc(d, &L->o1, (size_t)L->ldo));
    KMLL_TRY(dalloc(d, &L->z1, (size_t)max_ff));
    KMLL_TRY(dalloc(d, &L->gate1, (size_t)std::max(L->max_gate, 1)));
    KMLL_TRY(dalloc(d, &L->work, work));
    KMLL_TRY(dalloc(d, &d->hidden_a, (size_t)c.dim));
    KMLL_TRY(dalloc(d, &d->part_tok, (size_t)kMatvecMaxBlocks));
    KMLL_TRY(dalloc(d, &d->part_logit, (size_t)kMatvecMaxBlocks));
    KMLL_TRY(dalloc(d, &d->packed_final, (size_t)2));
    KMLL_TRY(dalloc(d, &d->state, (size_t)1));
    KMLL_CUDA(cudaMemset(d->state, 0, sizeof(DecodeState)));
    d->history_cap = c.max_seq_len;
    KMLL_TRY(dalloc(d, &d->history, (size_t)d->history_cap));
    KMLL_CUDA(cudaMallocHost((void**)&d->pinned, 64 * sizeof(uint64_t)));
    return KMLL_OK;
}

int ready(const Decoder* d) {
    if (!d->weights_set) return fail(KMLL_ERR_STATE, "decoder has no weights");
    for (size_t l = 0; l < d->lay->layers.size(); ++l)
        for (int i = 0; i < d->lay->layers[l].n_mix; ++i) {
            const LMixer& m = d->lay->layers[l].mix[i];
            if (m.table != nullptr && !m.table_set) return fail(KMLL_ERR_STATE, "layer %zu: kmll_layered_set_rotation has not been called", l);
            if (m.powers != nullptr && !m.decay_set) return fail(KMLL_ERR_STATE, "layer %zu: kmll_layered_set_decay has not been called", l);
        }
    return KMLL_OK;
}

LinearAttnArgs linear_args(const Layered* L, const LMixer& m) {
    LinearAttnArgs a;
    memset(&a, 0, sizeof(a));
    a.ld = L->ldp;
    a.q_off = m.off_q; a.k_off = m.off_k; a.v_off = m.off_v;
    a.heads = m.sp.heads; a.dk = m.sp.dim; a.dv = m.sp.vdim;
    a.rot = m.sp.rot_dim;
    a.table = m.table;
    a.key_scale = m.sp.key_scale;
    a.powers = m.powers;
    a.state = L->states + m.state_off;
    return a;
}
LatentArgs latent_args(const Layered* L, const LMixer& m) {
    LatentArgs a;
    memset(&a, 0, sizeof(a));
    a.ld = L->ldp;
    a.q_off = m.off_q; a.dkv_off = m.off_k;
    a.heads = m.sp.heads; a.dim = m.sp.dim; a.rot = m.sp.rot_dim; a.vdim = m.sp.vdim; a.rank = m.sp.kv_rank; a.window = m.sp.window;
    a.scale = m.sp.score_scale;
    a.eps = L->cfg.norm_eps;
    a.norm_w = m.dkv_norm;
    a.uk = m.ukv.w;
    a.uv = m.ukv.w + (size_t)m.sp.heads * m.sp.dim * m.ukv.ld;
    a.ldu = m.ukv.ld;
    a.table = m.table;
    a.cache = m.cache; a.cache_f32 = L->cfg.compute_f32; a.pitch = m.pitch; a.kr_off = m.kr_off; a.max_seq = L->cfg.max_seq_len;
    return a;
}
GroupedArgs grouped_args(const Layered* L, const LMixer& m) {
    GroupedArgs a;
    memset(&a, 0, sizeof(a));
    a.ld = L->ldp;
    a.q_off = m.off_q; a.k_off = m.off_k; a.v_off = m.off_v;
    a.heads = m.sp.heads; a.kv_heads = m.kv_heads(); a.dim = m.sp.dim; a.vdim = m.sp.vdim; a.window = m.sp.window; a.chunk = m.sp.chunk;
    a.scale = m.sp.score_scale;
    a.cache = m.cache; a.cache_f32 = L->cfg.compute_f32; a.pitch = m.pitch; a.dimp = up8(m.sp.dim); a.vdimp = up8(m.sp.vdim); a.max_seq = L->cfg.max_seq_len;
    return a;
}
GatedLinearArgs gated_args(const Layered* L, const LMixer& m) {
    GatedLinearArgs a;
    memset(&a, 0, sizeof(a));
    const kmll_mixer_spec& s = m.sp;
    a.ld = L->ldp;
    a.q_off = m.off_q; a.k_off = m.off_k; a.v_off = m.off_v; a.a_off = m.off_a; a.b_off = m.off_b; a.g_off = m.off_gd;
    a.heads = s.heads; a.kv_heads = m.kv_heads(); a.dk = s.dim; a.dv = s.vdim;
    a.decay = s.decay; a.inv_tau = s.decay == KMLL_DECAY_LOGISTIC ? 1.0f / s.decay_tau : 0.0f; a.rank = s.decay_rank;
    a.up = m.decay_up.w; a.ldu = m.decay_up.ld; a.bias = m.decay_bias; a.a_log = m.decay_log;
    a.delta = s.delta;
    a.taps = s.conv; a.conv = m.conv; a.ring = L->states + m.ring_off;
    a.unit_eps = s.unit_eps; a.q_scale = s.q_scale;
    a.gate_rank = s.gate_rank; a.gate_up = m.gate_up.w; a.ldg = m.gate_up.ld;
    a.state = L->states + m.state_off;
    return a;
}
// the mixer's part of what the output projection reads; `gate_base`: the stacked projection's result in f32 or bf16
GateSegment segment(const Layered* L, const LMixer& m, const void* gate_base, int elem, const float* low_rank) {
    const kmll_mixer_spec& s = m.sp;
    GateSegment g;
    memset(&g, 0, sizeof(g));
    g.begin = m.o_off; g.cols = m.width(); g.head_len = s.vdim; g.gate_len = 1;
    g.scale = s.out_scale; g.eps = L->cfg.norm_eps; g.act = s.gate_act; g.norm_w = m.mix_norm;
    g.norm = KMLL_OUT_NORM_NONE;
    const void* rows = static_cast<const uint8_t*>(gate_base) + (size_t)m.off_g * elem;
    if (s.mixer == KMLL_MIXER_ATTENTION) {
        if (s.head_gate) { g.gate = rows; g.gate_len = s.vdim; }
    } else if (s.mixer != KMLL_MIXER_LATENT_ATTENTION) {
        g.norm = s.out_norm;
        g.gate = s.mixer == KMLL_MIXER_GATED_LINEAR && s.gate_rank > 0 ? (const void*)low_rank : rows;
    }
    return g;
}

Bf16Matvec matvec(const Mat& m, const float* x, float* out) {
    Bf16Matvec v;
    memset(&v, 0, sizeof(v));
    v.w = m.w; v.rows = m.rows; v.K = m.cols; v.ldw = m.ld;
    v.x = x; v.y = out;
    v.out_scale = 1.0f;
    return v;
}
NormArgs norm_args(const Layered* L, const uint16_t* w, const uint16_t* b) { return NormArgs{L->cfg.norm, w, b, L->cfg.norm_offset, L->cfg.norm_eps}; }
void normed(Bf16Matvec* v, const Layered* L, const uint16_t* w, const uint16_t* b) {
    v->pro = PRO_NORM;
    v->norm = norm_args(L, w, b);
}
EmbedArgs embed_args(const Decoder* d) {
    const Layered* L = d->lay;
    EmbedArgs e;
    memset(&e, 0, sizeof(e));
    e.table = d->embedding; e.pos_table = L->pos_table; e.vocab = L->cfg.vocab_size; e.dim = L->cfg.dim; e.ld = L->embed.ld;
    e.scale = L->cfg.embed_scale;
    e.norm = norm_args(L, L->embed_norm, L->embed_norm_b);
    return e;
}
// final norm + lm_head of d->hidden_a -> logits and arg-max; with `state` the decode step ends here
int head_top1(Decoder* d, cudaStream_t s, DecodeState* state) {
    Layered* L = d->lay;
    Bf16Matvec v = matvec(L->head, d->hidden_a, L->logits);
    normed(&v, L, d->final_norm, L->final_norm_b);
    v.out_scale = L->cfg.logit_scale;
    v.part_tok = d->part_tok; v.part_logit = d->part_logit; v.counter = L->counter; v.packed = d->packed_final; v.state = state;
    return bf16_matvec(s, v);
}

// scratch of the prompt path for n rows
int ensure_rows(Decoder* d, cudaStream_t s, int n) {
    Layered* L = d->lay;
    if (n <= L->rows) return KMLL_OK;
    int want = 64;
    while (want < n) want *= 2;
    if (want > kMaxRows) want = kMaxRows;
    KMLL_CUDA(cudaStreamSynchronize(s));
    for (void* p : L->row_allocs) cudaFree(p);
    L->row_allocs.clear();
    L->rows = 0;
    const kmll_layered_config& c = L->cfg;
    const size_t e = c.compute_f32 ? 4 : 2;
    size_t total = 0, lin = 4;
    if (!c.compute_f32 && !L->plain)
        for (const LLayer& y : L->layers)
            for (int i = 0; i < y.n_mix; ++i) {
                const kmll_mixer_spec& m = y.mix[i].sp;
                if (m.mixer == KMLL_MIXER_LINEAR_ATTENTION) lin = std::max(lin, linear_attention_scratch_floats(want, m.heads, m.dim, m.vdim));
                if (m.mixer == KMLL_MIXER_GATED_LINEAR) lin = std::max(lin, gated_chunk_scratch_floats(want, m.heads, m.dim, m.vdim, m.delta));
            }
    auto take = [&](void** p, size_t bytes) -> int {
        cudaError_t er = cudaMalloc(p, bytes + 64);
        if (er != cudaSuccess) return fail(KMLL_ERR_CUDA, "prompt scratch (%zu bytes): %s", bytes, cudaGetErrorString(er));
        L->row_allocs.push_back(*p);
        total += bytes;
        return KMLL_OK;
    };
    KMLL_TRY(take((void**)&L->x, (size_t)want * c.dim * 4));
    KMLL_TRY(take((void**)&L->o, (size_t)want * L->ldo * 4));
    if (L->max_gate > 0) KMLL_TRY(take((void**)&L->gate, (size_t)want * L->max_gate * 4));
    KMLL_TRY(take(&L->a, (size_t)want * L->lda * e));
    KMLL_TRY(take(&L->p, (size_t)want * L->ldp * e));
    KMLL_TRY(take(&L->z, (size_t)want * L->ldz * e));
    KMLL_TRY(take((void**)&L->want, (size_t)want * 4));
    KMLL_TRY(take((void**)&L->lin, lin * 4));
    L->rows = want;
    return KMLL_OK;
}
int ensure_expanded(Layered* L, cudaStream_t s, size_t bytes) {
    if (bytes <= L->expanded_bytes) return KMLL_OK;
    KMLL_CUDA(cudaStreamSynchronize(s));
    cudaFree(L->expanded);
    L->expanded = nullptr;
    L->expanded_bytes = 0;
    cudaError_t e = cudaMalloc(&L->expanded, bytes + 64);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "latent expansion (%zu bytes): %s", bytes, cudaGetErrorString(e));
    L->expanded_bytes = bytes;
    return KMLL_OK;
}

Bf16Gemm rows_gemm(const Layered* L, const void* x, int ldx, int T, const Mat& w, void* out, bool out_f32, int ldo) {
    Bf16Gemm g;
    memset(&g, 0, sizeof(g));
    g.x = x; g.x_f32 = L->cfg.compute_f32; g.ldx = ldx; g.T = T; g.K = w.cols;
    g.w = w.w; g.rows = w.rows; g.ldw = w.ld;
    g.out = out; g.out_bf16 = !(out_f32 || L->cfg.compute_f32); g.ldo = ldo;
    g.out_scale = 1.0f;
    g.partial = L->gemm_partial; g.counters = L->gemm_counters;
    return g;
}

// one mixer over T rows of projections in L->p; its output goes to its columns of L->a
int mix_rows(Decoder* d, cudaStream_t s, const LLayer& y, const LMixer& m, int pos0, int T, int end) {
    Layered* L = d->lay;
    const kmll_mixer_spec& sp = m.sp;
    const int f32 = L->cfg.compute_f32, elem = f32 ? 4 : 2;
    if (sp.mixer == KMLL_MIXER_LINEAR_ATTENTION) {
        LinearAttnArgs a = linear_args(L, m);
        a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o + m.o_off; a.scratch = L->lin; a.ldo = L->ldo;
        if (!L->plain && linear_attention_chunked_ok(a)) KMLL_TRY(linear_attention_chunked(s, a));
        else KMLL_TRY(linear_attention_recurrent(s, a));
    } else if (sp.mixer == KMLL_MIXER_LATENT_ATTENTION) {
        LatentArgs a = latent_args(L, m);
        a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o + m.o_off; a.ldo = L->ldo;
        KMLL_TRY(latent_write_cache(s, a));
        if (!L->plain && latent_prefill_ok(a)) {
            a.first = sp.window > 0 ? std::max(0, pos0 - sp.window + 1) : 0;
            a.lde = up8(m.ukv.rows);
            const int rows = pos0 + T - a.first;
            KMLL_TRY(ensure_expanded(L, s, (size_t)rows * a.lde * 2));
            a.expanded = L->expanded;
            KMLL_TRY(bf16_gemm(s, rows_gemm(L, (const uint16_t*)m.cache + (size_t)a.first * m.pitch, m.pitch, rows, m.ukv, L->expanded, false, a.lde)));
            KMLL_TRY(latent_attention_prefill(s, a));
        } else {
            KMLL_TRY(latent_attention_plain(s, a));
        }
    } else if (sp.mixer == KMLL_MIXER_ATTENTION) {
        GroupedArgs a = grouped_args(L, m);
        a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o + m.o_off; a.ldo = L->ldo;
        KMLL_TRY(grouped_write_cache(s, a));
        if (!L->plain && grouped_prefill_ok(a)) KMLL_TRY(grouped_attention_prefill(s, a));
        else KMLL_TRY(grouped_attention_plain(s, a));
    } else {
        GatedLinearArgs a = gated_args(L, m);
        a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o + m.o_off; a.ldo = L->ldo; a.scratch = L->lin; a.gate = L->gate;
        if (!L->plain && gated_linear_chunked_ok(a)) {
            if (sp.gate_rank > 0)
                KMLL_TRY(bf16_gemm(s, rows_gemm(L, (const uint16_t*)L->p + m.off_gd, L->ldp, T, m.gate_up, L->gate, true, m.width())));
            KMLL_TRY(gated_linear_chunked(s, a));
        } else {
            KMLL_TRY(gated_linear_steps(s, a));
        }
    }
    const GateSegment g = segment(L, m, L->p, elem, L->gate);
    const bool low = sp.mixer == KMLL_MIXER_GATED_LINEAR && sp.gate_rank > 0;
    return gated_rows(s, L->o, L->ldo, T, g, f32 || low, low ? m.width() : L->ldp, end, f32, L->a, up8(y.width));
}

// T tokens (already in the token log) through the layers from position pos0; the residual stream ends up in L->x
int forward_rows(Decoder* d, cudaStream_t s, int pos0, int T, float* tap, size_t tap_stride) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    const int f32 = c.compute_f32;
    EmbedArgs e = embed_args(d);
    e.tokens = L->token_log + pos0; e.pos0 = pos0; e.T = T; e.x = L->x;
    KMLL_TRY(embed_rows(s, e));
    const int ldx = up8(c.dim);
    for (size_t l = 0; l < L->layers.size(); ++l) {
        LLayer& y = L->layers[l];
        KMLL_TRY(norm_rows(s, L->x, c.dim, nullptr, T, norm_args(L, y.norm1, y.norm1_b), f32, L->a, ldx));
        Bf16Gemm g = rows_gemm(L, L->a, ldx, T, y.proj, L->p, false, L->ldp);
        if (y.mix[0].sp.mixer == KMLL_MIXER_LINEAR_ATTENTION && y.mix[0].sp.qkv_act == KMLL_ACT_SILU) g.silu_rows = y.mix[0].off_g;
        KMLL_TRY(bf16_gemm(s, g));
        for (int i = 0; i < y.n_mix; ++i) KMLL_TRY(mix_rows(d, s, y, y.mix[i], pos0, T, i + 1 < y.n_mix ? y.mix[i + 1].o_off : y.width));
        g = rows_gemm(L, L->a, up8(y.width), T, y.wo, L->x, true, c.dim);
        g.residual = L->x;
        KMLL_TRY(bf16_gemm(s, g));
        if (y.mlp != KMLL_MLP_NONE) {
            KMLL_TRY(norm_rows(s, L->x, c.dim, nullptr, T, norm_args(L, y.norm2, y.norm2_b), f32, L->a, ldx));
            g = rows_gemm(L, L->a, ldx, T, y.up, L->z, false, L->ldz);
            if (y.mlp == KMLL_MLP_GATED) g.pair_act = y.mlp_act;
            KMLL_TRY(bf16_gemm(s, g));
            if (y.mlp == KMLL_MLP_POLYNORM) KMLL_TRY(polynorm_rows(s, L->z, f32, L->ldz, y.ff, T, y.act, c.norm_eps, L->a, up8(y.ff)));
            g = y.mlp == KMLL_MLP_GATED ? rows_gemm(L, L->z, L->ldz, T, y.down, L->x, true, c.dim) : rows_gemm(L, L->a, up8(y.ff), T, y.down, L->x, true, c.dim);
            g.residual = L->x;
            KMLL_TRY(bf16_gemm(s, g));
        }
        if (tap != nullptr) KMLL_CUDA(cudaMemcpyAsync(tap + l * tap_stride, L->x, (size_t)T * c.dim * 4, cudaMemcpyDeviceToDevice, s));
    }
    return KMLL_OK;
}

// one mixer over the projections of one token in L->proj1; its output goes to its columns of L->o1
int mix_token(Decoder* d, cudaStream_t s, const LMixer& m) {
    Layered* L = d->lay;
    float* const out = L->o1 + m.o_off;
    if (m.sp.mixer == KMLL_MIXER_LINEAR_ATTENTION) {
        LinearAttnArgs a = linear_args(L, m);
        a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = out; a.ldo = L->ldo;
        return linear_attention_recurrent(s, a);
    }
    if (m.sp.mixer == KMLL_MIXER_LATENT_ATTENTION) {
        LatentArgs a = latent_args(L, m);
        a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = out; a.ldo = L->ldo; a.work = L->work;
        if (!L->plain && latent_decode_ok(a)) return latent_attention_decode(s, a);
        KMLL_TRY(latent_write_cache(s, a));
        return latent_attention_plain(s, a);
    }
    if (m.sp.mixer == KMLL_MIXER_ATTENTION) {
        GroupedArgs a = grouped_args(L, m);
        a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = out; a.ldo = L->ldo;
        if (!L->plain && grouped_decode_ok(a)) return grouped_attention_decode(s, a);
        KMLL_TRY(grouped_write_cache(s, a));
        return grouped_attention_plain(s, a);
    }
    GatedLinearArgs a = gated_args(L, m);
    a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = out; a.ldo = L->ldo; a.gate = L->gate1;
    return gated_linear_steps(s, a);
}

}  // namespace

int layered_enqueue_step(Decoder* d, cudaStream_t s, int* launches) {
    Layered* L = d->lay;
    const unsigned long long before = launch_counter();
    KMLL_TRY(ready(d));
    EmbedArgs e = embed_args(d);
    e.T = 1; e.x = d->hidden_a; e.state = d->state; e.history = d->history; e.history_cap = d->history_cap; e.token_log = L->token_log;
    KMLL_TRY(embed_rows(s, e));
    float* const x = d->hidden_a;
    for (LLayer& y : L->layers) {
        Bf16Matvec in = matvec(y.proj, x, L->proj1);
        normed(&in, L, y.norm1, y.norm1_b);
        if (y.mix[0].sp.mixer == KMLL_MIXER_LINEAR_ATTENTION && y.mix[0].sp.qkv_act == KMLL_ACT_SILU) in.silu_rows = y.mix[0].off_g;
        KMLL_TRY(bf16_matvec(s, in));
        Bf16Matvec out = matvec(y.wo, L->o1, x);
        out.residual = x;
        out.n_seg = y.n_mix;
        bool plain = y.n_mix == 1;
        for (int i = 0; i < y.n_mix; ++i) {
            KMLL_TRY(mix_token(d, s, y.mix[i]));
            out.seg[i] = segment(L, y.mix[i], L->proj1, 4, L->gate1);
            plain = plain && out.seg[i].norm == KMLL_OUT_NORM_NONE && out.seg[i].gate == nullptr && out.seg[i].scale == 1.0f;
        }
        out.pro = plain ? PRO_PLAIN : PRO_GATED;
        KMLL_TRY(bf16_matvec(s, out));
        if (y.mlp != KMLL_MLP_NONE) {
            Bf16Matvec up = matvec(y.up, x, L->z1);
            normed(&up, L, y.norm2, y.norm2_b);
            if (y.mlp == KMLL_MLP_GATED) up.pair_act = y.mlp_act;
            KMLL_TRY(bf16_matvec(s, up));
            Bf16Matvec down = matvec(y.down, L->z1, x);
            if (y.mlp == KMLL_MLP_POLYNORM) {
                down.pro = PRO_POLYNORM;
                down.coef = y.act;
                down.eps = L->cfg.norm_eps;
            }
            down.residual = x;
            KMLL_TRY(bf16_matvec(s, down));
        }
    }
    KMLL_TRY(head_top1(d, s, d->state));
    if (launches) *launches = (int)(launch_counter() - before);
    return KMLL_OK;
}

int layered_forward(Decoder* d, cudaStream_t s, const uint32_t* tokens_host, const uint32_t* tokens_device, int n, const int* want, int n_want,
                    float* logits_out, bool top) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    KMLL_TRY(ready(d));
    if (d->host_position + n > c.max_seq_len)
        return fail(KMLL_ERR_CAPACITY, "position %d exceeds max sequence length %d", d->host_position + n, c.max_seq_len);
    int wi = 0;
    for (int t0 = 0; t0 < n; t0 += kMaxRows) {
        const int T = std::min(kMaxRows, n - t0), pos0 = d->host_position;
        KMLL_TRY(ensure_rows(d, s, T));
        if (tokens_host != nullptr)
            KMLL_CUDA(cudaMemcpyAsync(L->token_log + pos0, tokens_host + t0, (size_t)T * 4, cudaMemcpyHostToDevice, s));
        else if (tokens_device != L->token_log + pos0 - t0)
            return fail(KMLL_ERR_STATE, "internal: device tokens are replayed in place");
        KMLL_TRY(forward_rows(d, s, pos0, T, L->tap != nullptr ? L->tap + (size_t)t0 * c.dim : nullptr, (size_t)n * c.dim));
        int w1 = wi;
        while (w1 < n_want && want[w1] < t0 + T) ++w1;
        if (w1 > wi) {
            std::vector<int> rows(w1 - wi);
            for (int i = wi; i < w1; ++i) rows[i - wi] = want[i] - t0;
            KMLL_CUDA(cudaMemcpyAsync(L->want, rows.data(), rows.size() * 4, cudaMemcpyHostToDevice, s));
            KMLL_CUDA(cudaStreamSynchronize(s));  // `rows` lives on this stack frame
            KMLL_TRY(norm_rows(s, L->x, c.dim, L->want, w1 - wi, norm_args(L, d->final_norm, L->final_norm_b), c.compute_f32, L->a, up8(c.dim)));
            Bf16Gemm g = rows_gemm(L, L->a, up8(c.dim), w1 - wi, L->head, logits_out + (size_t)wi * c.vocab_size, true, c.vocab_size);
            g.out_scale = c.logit_scale;
            KMLL_TRY(bf16_gemm(s, g));
            wi = w1;
        }
        d->host_position += T;
        if (t0 + T == n && top) {
            KMLL_CUDA(cudaMemcpyAsync(d->hidden_a, L->x + (size_t)(T - 1) * c.dim, (size_t)c.dim * 4, cudaMemcpyDeviceToDevice, s));
            KMLL_TRY(head_top1(d, s, nullptr));
        }
    }
    return KMLL_OK;
}

int layered_reset(Decoder* d, cudaStream_t s) {
    KMLL_CUDA(cudaMemsetAsync(d->lay->states, 0, d->lay->state_floats * 4, s));
    d->lay->saved_at = -1;
    d->host_position = 0;
    return KMLL_OK;
}

int layered_save_state(Decoder* d, cudaStream_t s) {
    Layered* L = d->lay;
    KMLL_CUDA(cudaMemcpyAsync(L->saved, L->states, L->state_floats * 4, cudaMemcpyDeviceToDevice, s));
    KMLL_CUDA(cudaMemcpyAsync(L->saved_logits, L->logits, (size_t)L->cfg.vocab_size * 4, cudaMemcpyDeviceToDevice, s));
    L->saved_at = d->host_position;
    return KMLL_OK;
}

int layered_rewind(Decoder* d, cudaStream_t s, int position) {
    Layered* L = d->lay;
    if (position == d->host_position) return KMLL_OK;
    if (L->saved_at >= 0 && L->saved_at <= position) {
        KMLL_CUDA(cudaMemcpyAsync(L->states, L->saved, L->state_floats * 4, cudaMemcpyDeviceToDevice, s));
        KMLL_CUDA(cudaMemcpyAsync(L->logits, L->saved_logits, (size_t)L->cfg.vocab_size * 4, cudaMemcpyDeviceToDevice, s));
        d->host_position = L->saved_at;
    } else {
        KMLL_TRY(layered_reset(d, s));
    }
    const int from = d->host_position;
    if (from < position) KMLL_TRY(layered_forward(d, s, nullptr, L->token_log + from, position - from, nullptr, 0, nullptr, true));
    return KMLL_OK;
}

int layered_hold_state(Decoder* d, cudaStream_t s, bool restore) {
    Layered* L = d->lay;
    KMLL_CUDA(cudaMemcpyAsync(restore ? L->states : L->held, restore ? L->held : L->states, L->state_floats * 4, cudaMemcpyDeviceToDevice, s));
    return KMLL_OK;
}

const float* layered_logits(const Decoder* d) { return d->lay->logits; }
bool layered_tapped(const Decoder* d) { return d->lay->tap != nullptr; }

void layered_destroy(Decoder* d) {
    if (d->lay == nullptr) return;
    for (void* p : d->lay->row_allocs) cudaFree(p);
    cudaFree(d->lay->expanded);
    delete d->lay;
    d->lay = nullptr;
}

// ---- tensors -----------------------------------------------------------------------------------------------------------------
namespace {
struct Slot {
    uint16_t* w = nullptr;
    int rows = 1, cols = 0, ld = 0;
};
int find(Decoder* d, int layer, int tensor, Slot* out) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    auto vec = [&](uint16_t* w, int n) { out->w = w; out->rows = 1; out->cols = out->ld = n; };
    auto rows = [&](const Mat& m, int r0, int n, int step = 1) {
        out->w = m.w != nullptr ? m.w + (size_t)r0 * m.ld : nullptr; out->rows = n; out->cols = m.cols; out->ld = m.ld * step;
    };
    const bool second = (tensor & KMLL_T_BESIDE) != 0;
    const int id = tensor & ~KMLL_T_BESIDE;
    if (layer == -1) {
        switch (tensor) {
            case KMLL_T_EMBEDDING: rows(L->embed, 0, c.vocab_size); break;
            case KMLL_T_POSITION: out->w = L->pos_table; out->rows = c.position_rows; out->cols = out->ld = c.dim; break;
            case KMLL_T_FINAL_NORM: vec(d->final_norm, c.dim); break;
            case KMLL_T_FINAL_NORM_BIAS: vec(L->final_norm_b, c.dim); break;
            case KMLL_T_EMBED_NORM: vec(L->embed_norm, c.dim); break;
            case KMLL_T_EMBED_NORM_BIAS: vec(L->embed_norm_b, c.dim); break;
            case KMLL_T_OUTPUT: if (!c.tie_output) rows(L->head, 0, c.vocab_size); break;
            default: break;
        }
    } else {
        if (layer < 0 || layer >= c.n_layers) return fail(KMLL_ERR_SHAPE, "layer %d out of range", layer);
        LLayer& y = L->layers[layer];
        const bool ff = y.mlp != KMLL_MLP_NONE, pair = y.mlp == KMLL_MLP_GATED;
        bool found = !second;
        if (!second) switch (id) {
            case KMLL_T_ATTENTION_NORM: vec(y.norm1, c.dim); break;
            case KMLL_T_ATTENTION_NORM_BIAS: vec(y.norm1_b, c.dim); break;
            case KMLL_T_FFN_NORM: if (ff) vec(y.norm2, c.dim); break;
            case KMLL_T_FFN_NORM_BIAS: if (ff) vec(y.norm2_b, c.dim); break;
            case KMLL_T_W1: if (pair) rows(y.up, 0, y.ff, 2); break;
            case KMLL_T_W3: if (ff) rows(y.up, pair ? 1 : 0, y.ff, pair ? 2 : 1); break;
            case KMLL_T_W2: if (ff) rows(y.down, 0, c.dim); break;
            case KMLL_T_ACT: if (ff) vec(y.act, 4); break;
            default: found = false; break;
        }
        if (!found && (second ? 1 : 0) < y.n_mix) {
            LMixer& m = y.mix[second ? 1 : 0];
            const kmll_mixer_spec& s = m.sp;
            const int g = m.kv_heads(), nk = g * s.dim;
            const bool lat = s.mixer == KMLL_MIXER_LATENT_ATTENTION, att = s.mixer == KMLL_MIXER_ATTENTION, lin = s.mixer == KMLL_MIXER_LINEAR_ATTENTION,
                       gat = s.mixer == KMLL_MIXER_GATED_LINEAR;
            auto conv = [&](int ch, int n) { out->w = m.conv != nullptr ? m.conv + (size_t)ch * s.conv : nullptr; out->rows = n; out->cols = out->ld = s.conv; };
            switch (id) {
                case KMLL_T_WQ: rows(y.proj, m.off_q, lat ? s.heads * (s.dim + s.rot_dim) : gat ? nk : s.heads * s.dim); break;
                case KMLL_T_WK: if (!lat) rows(y.proj, m.off_k, lin ? s.heads * s.dim : nk); break;
                case KMLL_T_WV: if (!lat) rows(y.proj, m.off_v, att ? g * s.vdim : s.heads * s.vdim); break;
                case KMLL_T_GATE:
                    if (att && s.head_gate) rows(y.proj, m.off_g, s.heads);
                    else if (lin || (gat && s.gate_rank == 0)) rows(y.proj, m.off_g, s.heads * s.vdim);
                    break;
                case KMLL_T_MIX_NORM: if (m.mix_norm != nullptr) vec(m.mix_norm, s.out_norm == KMLL_OUT_NORM_HEAD_WEIGHTED ? s.vdim : s.heads * s.vdim); break;
                case KMLL_T_DKV: if (lat) rows(y.proj, m.off_k, s.kv_rank + s.rot_dim); break;
                case KMLL_T_DKV_NORM: if (lat) vec(m.dkv_norm, s.kv_rank); break;
                case KMLL_T_UK: if (lat) rows(m.ukv, 0, s.heads * s.dim); break;
                case KMLL_T_UV: if (lat) rows(m.ukv, s.heads * s.dim, s.heads * s.vdim); break;
                case KMLL_T_DECAY_DOWN: if (gat) rows(y.proj, m.off_a, s.decay_rank); break;
                case KMLL_T_DECAY_UP: if (gat) rows(m.decay_up, 0, s.heads * s.dim); break;
                case KMLL_T_DECAY_BIAS: if (gat) vec(m.decay_bias, s.heads * s.dim); break;
                case KMLL_T_DECAY_LOG: if (gat) vec(m.decay_log, s.heads); break;
                case KMLL_T_BETA: if (gat && s.delta) rows(y.proj, m.off_b, s.heads); break;
                case KMLL_T_Q_CONV: if (gat) conv(0, nk); break;
                case KMLL_T_K_CONV: if (gat) conv(nk, nk); break;
                case KMLL_T_V_CONV: if (gat) conv(2 * nk, s.heads * s.vdim); break;
                case KMLL_T_GATE_DOWN: if (gat && s.gate_rank > 0) rows(y.proj, m.off_gd, s.gate_rank); break;
                case KMLL_T_GATE_UP: if (gat && s.gate_rank > 0) rows(m.gate_up, 0, s.heads * s.vdim); break;
                case KMLL_T_WO: rows(y.wo, 0, c.dim); out->w += m.o_off; out->cols = m.width(); break;
                default: break;
            }
        }
    }
    if (out->w == nullptr) return fail(KMLL_ERR_SHAPE, "tensor %d does not exist in layer %d of this model", tensor, layer);
    return KMLL_OK;
}
}  // namespace

int layered_set_tensor(Decoder* d, int layer, int tensor, const void* values) {
    Slot t;
    KMLL_TRY(find(d, layer, tensor, &t));
    KMLL_CUDA(cudaMemcpy2D(t.w, (size_t)t.ld * 2, values, (size_t)t.cols * 2, (size_t)t.cols * 2, t.rows, cudaMemcpyHostToDevice));
    d->weights_set = true;
    return KMLL_OK;
}
int layered_get_tensor(Decoder* d, int layer, int tensor, void* values) {
    Slot t;
    KMLL_TRY(find(d, layer, tensor, &t));
    KMLL_CUDA(cudaDeviceSynchronize());
    if (values) KMLL_CUDA(cudaMemcpy2D(values, (size_t)t.cols * 2, t.w, (size_t)t.ld * 2, (size_t)t.cols * 2, t.rows, cudaMemcpyDeviceToHost));
    return KMLL_OK;
}

int layered_init_random(Decoder* d, uint64_t seed, float std, int tie_embeddings) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    constexpr size_t kBatch = 1u << 24;
    float* tmp = nullptr;
    KMLL_CUDA(cudaMalloc((void**)&tmp, kBatch * 4));
    uint64_t at = seed * 0x9e3779b97f4a7c15ull;
    auto normal = [&](uint16_t* w, size_t n) -> int {  // (row padding included: the other operand is zero there)
        for (size_t i = 0; i < n; i += kBatch) {
            const size_t m = std::min(kBatch, n - i);
            KMLL_TRY(kmll_fill_normal_f32(nullptr, tmp, m, ++at, std));
            KMLL_TRY(kmll_f32_to_bf16(nullptr, tmp, m, w + i));
        }
        return KMLL_OK;
    };
    auto constant = [&](uint16_t* w, size_t n, float v) -> int {
        uint32_t bits;
        memcpy(&bits, &v, 4);
        std::vector<uint16_t> h(n, (uint16_t)(bits >> 16));
        KMLL_CUDA(cudaMemcpy(w, h.data(), n * 2, cudaMemcpyHostToDevice));
        return KMLL_OK;
    };
    auto mat = [&](Mat& m) { return normal(m.w, (size_t)m.rows * m.ld); };
    const float neutral = 1.0f - c.norm_offset;
    auto body = [&]() -> int {
        KMLL_TRY(mat(L->embed));
        if (L->embed_norm) KMLL_TRY(constant(L->embed_norm, c.dim, neutral));
        if (L->embed_norm_b) KMLL_TRY(constant(L->embed_norm_b, c.dim, 0.0f));
        if (L->final_norm_b) KMLL_TRY(constant(L->final_norm_b, c.dim, 0.0f));
        if (L->pos_table) KMLL_TRY(normal(L->pos_table, (size_t)c.position_rows * c.dim));
        KMLL_TRY(constant(d->final_norm, c.dim, neutral));
        if (c.tie_output) {}
        else if (tie_embeddings) KMLL_CUDA(cudaMemcpy(L->head.w, L->embed.w, (size_t)L->head.rows * L->head.ld * 2, cudaMemcpyDeviceToDevice));
        else KMLL_TRY(mat(L->head));
        for (LLayer& y : L->layers) {
            KMLL_TRY(constant(y.norm1, c.dim, neutral));
            if (y.norm1_b) KMLL_TRY(constant(y.norm1_b, c.dim, 0.0f));
            KMLL_TRY(mat(y.proj));
            KMLL_TRY(mat(y.wo));
            for (int i = 0; i < y.n_mix; ++i) {
                LMixer& m = y.mix[i];
                if (m.ukv.w) KMLL_TRY(mat(m.ukv));
                if (m.dkv_norm) KMLL_TRY(constant(m.dkv_norm, m.sp.kv_rank, 1.0f));
                if (m.mix_norm) KMLL_TRY(constant(m.mix_norm, m.sp.out_norm == KMLL_OUT_NORM_HEAD_WEIGHTED ? m.sp.vdim : m.width(), 1.0f));
                if (m.decay_up.w) KMLL_TRY(mat(m.decay_up));
                if (m.gate_up.w) KMLL_TRY(mat(m.gate_up));
                if (m.decay_bias) KMLL_TRY(constant(m.decay_bias, (size_t)m.sp.heads * m.sp.dim, m.sp.decay == KMLL_DECAY_SOFTPLUS ? -2.0f : 2.0f));
                if (m.decay_log) KMLL_TRY(constant(m.decay_log, m.sp.heads, 0.0f));
                if (m.conv) {  // the current token passes
                    std::vector<uint16_t> taps((size_t)m.conv_channels() * m.sp.conv, 0);
                    for (size_t ch = 1; ch <= (size_t)m.conv_channels(); ++ch) taps[ch * m.sp.conv - 1] = 0x3f80;
                    KMLL_CUDA(cudaMemcpy(m.conv, taps.data(), taps.size() * 2, cudaMemcpyHostToDevice));
                }
            }
            if (y.mlp != KMLL_MLP_NONE) {
                KMLL_TRY(constant(y.norm2, c.dim, neutral));
                if (y.norm2_b) KMLL_TRY(constant(y.norm2_b, c.dim, 0.0f));
                KMLL_TRY(mat(y.up));
                KMLL_TRY(mat(y.down));
                if (y.act) {
                    KMLL_TRY(constant(y.act, 3, 1.0f / 3.0f));
                    KMLL_TRY(constant(y.act + 3, 1, 0.0f));
                }
            }
        }
        KMLL_CUDA(cudaDeviceSynchronize());
        return KMLL_OK;
    };
    const int rc = body();
    cudaFree(tmp);
    if (rc == KMLL_OK) d->weights_set = true;
    return rc;
}

}  // namespace kmll

using namespace kmll;

extern "C" {

size_t kmll_layer_spec_bytes(void) { return sizeof(kmll_layer_spec); }
size_t kmll_layered_config_bytes(void) { return sizeof(kmll_layered_config); }

int kmll_layered_create(const kmll_layered_config* config, const kmll_layer_spec* layers, kmll_decoder_t* out) {
    KMLL_REQUIRE_PTR(config);
    KMLL_REQUIRE_PTR(layers);
    KMLL_REQUIRE_PTR(out);
    KMLL_TRY(validate(*config, layers));
    Decoder* d = new Decoder();
    d->lay = new Layered();
    kmll_decoder_config& c = d->cfg;
    memset(&c, 0, sizeof(c));
    c.n_layers = config->n_layers;
    c.dim = config->dim;
    c.vocab_size = config->vocab_size;
    c.norm_eps = config->norm_eps;
    c.max_seq_len = config->max_seq_len;
    c.format = KMLL_FORMAT_BF16;
    c.fused = 1;
    c.tp_size = 1;
    const int rc = create(d, *config, layers);
    if (rc != KMLL_OK) {
        kmll_decoder_destroy(d);
        return rc;
    }
    *out = d;
    return KMLL_OK;
}

int kmll_layered_set_rotation(kmll_decoder_t dec, int layer, const double* freqs_host, int count, double magnitude) {
    KMLL_REQUIRE_PTR(dec);
    KMLL_REQUIRE_PTR(freqs_host);
    Decoder* d = static_cast<Decoder*>(dec);
    if (d->lay == nullptr) return fail(KMLL_ERR_UNSUPPORTED, "set_rotation: not a layered decoder");
    KMLL_REQUIRE(layer >= 0 && layer < d->cfg.n_layers, "set_rotation: layer %d out of range", layer);
    LMixer& y = d->lay->layers[layer].mix[0];
    KMLL_REQUIRE(y.sp.rot_dim > 0 && count == y.sp.rot_dim / 2, "set_rotation: %d frequencies given, %d expected", count, y.sp.rot_dim / 2);
    double* dev = nullptr;
    KMLL_CUDA(cudaMalloc((void**)&dev, sizeof(double) * count));
    cudaError_t e = cudaMemcpy(dev, freqs_host, sizeof(double) * count, cudaMemcpyHostToDevice);
    int rc = e == cudaSuccess ? rotation_table(nullptr, dev, count, d->cfg.max_seq_len, magnitude, y.table) : fail(KMLL_ERR_CUDA, "set_rotation: %s", cudaGetErrorString(e));
    e = cudaDeviceSynchronize();
    cudaFree(dev);
    if (rc == KMLL_OK && e != cudaSuccess) rc = fail(KMLL_ERR_CUDA, "set_rotation: %s", cudaGetErrorString(e));
    if (rc == KMLL_OK) y.table_set = true;
    return rc;
}

int kmll_layered_set_decay(kmll_decoder_t dec, int layer, const double* decay_host, int count) {
    KMLL_REQUIRE_PTR(dec);
    KMLL_REQUIRE_PTR(decay_host);
    Decoder* d = static_cast<Decoder*>(dec);
    if (d->lay == nullptr) return fail(KMLL_ERR_UNSUPPORTED, "set_decay: not a layered decoder");
    KMLL_REQUIRE(layer >= 0 && layer < d->cfg.n_layers, "set_decay: layer %d out of range", layer);
    LMixer& y = d->lay->layers[layer].mix[0];
    KMLL_REQUIRE(y.powers != nullptr && count == y.sp.heads, "set_decay: %d values given, the layer has %d heads", count, y.powers ? y.sp.heads : 0);
    std::vector<float> pw((size_t)count * (kLinChunk + 1));
    for (int h = 0; h < count; ++h) {
        KMLL_REQUIRE(std::isfinite(decay_host[h]), "set_decay: value %d is not finite", h);
        double v = 1.0;
        for (int i = 0; i <= kLinChunk; ++i, v *= decay_host[h]) pw[(size_t)h * (kLinChunk + 1) + i] = (float)v;
    }
    KMLL_CUDA(cudaDeviceSynchronize());
    KMLL_CUDA(cudaMemcpy(y.powers, pw.data(), pw.size() * 4, cudaMemcpyHostToDevice));
    y.decay_set = true;
    return KMLL_OK;
}

int kmll_layered_tap(kmll_decoder_t dec, float* residual_device) {
    KMLL_REQUIRE_PTR(dec);
    Decoder* d = static_cast<Decoder*>(dec);
    if (d->lay == nullptr) return fail(KMLL_ERR_UNSUPPORTED, "tap: not a layered decoder");
    d->lay->tap = residual_device;
    return KMLL_OK;
}

}  // extern "C"
