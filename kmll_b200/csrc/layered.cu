// Layered decoders: pre-norm layers from a list of descriptions (latent attention, linear attention with a fixed decay per
// head; PolyNorm feed-forward), bf16 weights.  The decode loop, the graph, the pending token, the history and the
// session-level entry points are those of runtime.cu; this file holds the weights, the caches and states, the decode step and
// the prompt path.
//
// Decode step, per layer (f32 activations, one launch each):
//   norm + stacked projection | mixer (linear: state update; latent: absorb, attend, merge) | norm / gate + output projection
//   + residual | norm + up | PolyNorm + down + residual                      then norm + lm_head + arg-max + end of the step
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

struct LLayer {
    kmll_layer_spec sp;
    uint16_t *norm1 = nullptr, *norm2 = nullptr, *mix_norm = nullptr, *dkv_norm = nullptr, *act = nullptr;
    Mat proj;               // linear: q | k | v | gate; latent: q | (latent, rotated part)
    int off_k = 0, off_v = 0, off_g = 0;  // row offsets in proj (latent: off_k = the latent's)
    Mat wo, ukv, up, down;
    float2* table = nullptr;   // rotation [max_seq][rot / 2]
    float* powers = nullptr;   // [heads][kLinChunk + 1]
    bool decay_set = false, table_set = false;
    size_t state_off = 0, state_floats = 0;  // within Layered::states
    void* cache = nullptr;
    int pitch = 0, kr_off = 0;
    int width() const { return sp.heads * sp.vdim; }
};

}  // namespace

struct Layered {
    kmll_layered_config cfg;
    bool plain = false;  // plain kernels also where faster forms exist
    std::vector<LLayer> layers;
    uint16_t* pos_table = nullptr;
    Mat head;
    float* logits = nullptr;
    unsigned int* counter = nullptr;
    uint32_t* token_log = nullptr;  // [max_seq] tokens of the sequence by position
    float* states = nullptr;
    size_t state_floats = 0;
    // remembered states (rewind) and the copy held around a warm-up step
    float *saved = nullptr, *saved_logits = nullptr, *held = nullptr;
    int saved_at = -1;
    // one-token scratch
    float *proj1 = nullptr, *o1 = nullptr, *z1 = nullptr, *latent_work = nullptr;
    // prompt scratch for `rows` tokens
    int rows = 0;
    std::vector<void*> row_allocs;
    float *x = nullptr, *o = nullptr, *lin = nullptr;
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

int validate(const kmll_layered_config& c, const kmll_layer_spec* specs) {
    if (c.n_layers <= 0 || c.dim <= 0 || c.vocab_size <= 0 || c.max_seq_len <= 0) return fail(KMLL_ERR_SHAPE, "layered decoder: every size must be positive");
    if (c.position_rows > 0 && c.max_seq_len > c.position_rows)
        return fail(KMLL_ERR_SHAPE, "layered decoder: max_seq_len %d exceeds the %d learned positions", c.max_seq_len, c.position_rows);
    for (int l = 0; l < c.n_layers; ++l) {
        const kmll_layer_spec& s = specs[l];
        if (s.mixer != KMLL_MIXER_LATENT_ATTENTION && s.mixer != KMLL_MIXER_LINEAR_ATTENTION) return fail(KMLL_ERR_SHAPE, "layer %d: unknown mixer %d", l, s.mixer);
        if (s.heads <= 0 || s.dim <= 0 || s.vdim <= 0) return fail(KMLL_ERR_SHAPE, "layer %d: head sizes must be positive", l);
        if (s.rot_dim < 0 || (s.rot_dim & 1)) return fail(KMLL_ERR_SHAPE, "layer %d: rot_dim must be even", l);
        if (s.mixer == KMLL_MIXER_LATENT_ATTENTION && (s.kv_rank <= 0 || s.window < 0)) return fail(KMLL_ERR_SHAPE, "layer %d: bad latent size or window", l);
        if (s.mixer == KMLL_MIXER_LINEAR_ATTENTION && s.rot_dim > s.dim) return fail(KMLL_ERR_SHAPE, "layer %d: rot_dim exceeds the key size", l);
        if (s.mixer == KMLL_MIXER_LINEAR_ATTENTION && s.dim > 512) return fail(KMLL_ERR_UNSUPPORTED, "layer %d: key size %d above 512", l, s.dim);
        if (s.mixer == KMLL_MIXER_LINEAR_ATTENTION && s.qkv_act != KMLL_ACT_NONE && s.qkv_act != KMLL_ACT_SILU)
            return fail(KMLL_ERR_UNSUPPORTED, "layer %d: q, k, v go through SiLU or nothing", l);
        if (s.mlp != KMLL_MLP_NONE && (s.mlp != KMLL_MLP_POLYNORM || s.ff <= 0)) return fail(KMLL_ERR_SHAPE, "layer %d: bad feed-forward", l);
    }
    return KMLL_OK;
}

int create(Decoder* d, const kmll_layered_config& c, const kmll_layer_spec* specs) {
    Layered* L = d->lay;
    L->cfg = c;
    const char* env = std::getenv("KMLL_LAYERED");
    L->plain = env != nullptr && strcmp(env, "plain") == 0;
    L->layers.resize(c.n_layers);
    KMLL_CUDA(cudaGetDevice(&d->device));
    KMLL_TRY(alloc_vec(d, &d->embedding, (size_t)c.vocab_size * c.dim));
    if (c.position_rows > 0) KMLL_TRY(alloc_vec(d, &L->pos_table, (size_t)c.position_rows * c.dim));
    KMLL_TRY(alloc_vec(d, &d->final_norm, c.dim));
    KMLL_TRY(alloc_mat(d, &L->head, c.vocab_size, c.dim));
    int max_p = 0, max_o = 0, max_ff = 1, max_a = up8(c.dim);
    size_t work = 1;
    for (int l = 0; l < c.n_layers; ++l) {
        LLayer& y = L->layers[l];
        const kmll_layer_spec& s = y.sp = specs[l];
        KMLL_TRY(alloc_vec(d, &y.norm1, c.dim));
        if (s.mixer == KMLL_MIXER_LATENT_ATTENTION) {
            y.off_k = s.heads * (s.dim + s.rot_dim);
            KMLL_TRY(alloc_mat(d, &y.proj, y.off_k + s.kv_rank + s.rot_dim, c.dim));
            KMLL_TRY(alloc_vec(d, &y.dkv_norm, s.kv_rank));
            KMLL_TRY(alloc_mat(d, &y.ukv, s.heads * (s.dim + s.vdim), s.kv_rank));
            y.kr_off = up8(s.kv_rank);
            y.pitch = up8(y.kr_off + s.rot_dim);
            const size_t bytes = (size_t)c.max_seq_len * y.pitch * (c.compute_f32 ? 4 : 2);
            uint8_t* cache = nullptr;
            KMLL_TRY(dalloc(d, &cache, bytes));
            KMLL_CUDA(cudaMemset(cache, 0, bytes));
            y.cache = cache;
            d->kv_bytes += bytes;
            const int span = s.window > 0 && s.window < c.max_seq_len ? s.window : c.max_seq_len;
            work = std::max(work, latent_decode_work_floats(s.heads, s.kv_rank, s.rot_dim, span));
        } else {
            y.off_k = s.heads * s.dim;
            y.off_v = 2 * y.off_k;
            y.off_g = y.off_v + s.heads * s.vdim;
            KMLL_TRY(alloc_mat(d, &y.proj, y.off_g + s.heads * s.vdim, c.dim));
            if (s.out_norm == KMLL_OUT_NORM_JOINT) KMLL_TRY(alloc_vec(d, &y.mix_norm, s.heads * s.vdim));
            KMLL_TRY(dalloc(d, &y.powers, (size_t)s.heads * (kLinChunk + 1)));
            y.state_off = L->state_floats;
            y.state_floats = (size_t)s.heads * s.dim * s.vdim;
            L->state_floats += (y.state_floats + 3) & ~(size_t)3;
        }
        if (s.rot_dim > 0) KMLL_TRY(dalloc(d, &y.table, (size_t)c.max_seq_len * (s.rot_dim / 2)));
        KMLL_TRY(alloc_mat(d, &y.wo, c.dim, y.width()));
        if (s.mlp != KMLL_MLP_NONE) {
            KMLL_TRY(alloc_vec(d, &y.norm2, c.dim));
            KMLL_TRY(alloc_mat(d, &y.up, s.ff, c.dim));
            KMLL_TRY(alloc_mat(d, &y.down, c.dim, s.ff));
            KMLL_TRY(alloc_vec(d, &y.act, 4));
            max_ff = std::max(max_ff, s.ff);
        }
        max_p = std::max(max_p, y.proj.rows);
        max_o = std::max(max_o, y.width());
    }
    L->lda = std::max({max_a, up8(max_o), up8(max_ff)});
    L->ldp = up8(max_p);
    L->ldz = up8(max_ff);
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
    KMLL_TRY(dalloc(d, &L->o1, (size_t)max_o));
    KMLL_TRY(dalloc(d, &L->z1, (size_t)max_ff));
    KMLL_TRY(dalloc(d, &L->latent_work, work));
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
    for (size_t l = 0; l < d->lay->layers.size(); ++l) {
        const LLayer& y = d->lay->layers[l];
        if (y.table != nullptr && !y.table_set) return fail(KMLL_ERR_STATE, "layer %zu: kmll_layered_set_rotation has not been called", l);
        if (y.powers != nullptr && !y.decay_set) return fail(KMLL_ERR_STATE, "layer %zu: kmll_layered_set_decay has not been called", l);
    }
    return KMLL_OK;
}

LinearAttnArgs linear_args(const Layered* L, const LLayer& y) {
    LinearAttnArgs a;
    memset(&a, 0, sizeof(a));
    a.ld = L->ldp;
    a.q_off = 0; a.k_off = y.off_k; a.v_off = y.off_v;
    a.heads = y.sp.heads; a.dk = y.sp.dim; a.dv = y.sp.vdim;
    a.rot = y.sp.rot_dim;
    a.table = y.table;
    a.key_scale = y.sp.key_scale;
    a.powers = y.powers;
    a.state = L->states + y.state_off;
    return a;
}
LatentArgs latent_args(const Layered* L, const LLayer& y) {
    LatentArgs a;
    memset(&a, 0, sizeof(a));
    a.ld = L->ldp;
    a.q_off = 0; a.dkv_off = y.off_k;
    a.heads = y.sp.heads; a.dim = y.sp.dim; a.rot = y.sp.rot_dim; a.vdim = y.sp.vdim; a.rank = y.sp.kv_rank; a.window = y.sp.window;
    a.scale = y.sp.score_scale;
    a.eps = L->cfg.norm_eps;
    a.norm_w = y.dkv_norm;
    a.uk = y.ukv.w;
    a.uv = y.ukv.w + (size_t)y.sp.heads * y.sp.dim * y.ukv.ld;
    a.ldu = y.ukv.ld;
    a.table = y.table;
    a.cache = y.cache; a.cache_f32 = L->cfg.compute_f32; a.pitch = y.pitch; a.kr_off = y.kr_off; a.max_seq = L->cfg.max_seq_len;
    return a;
}

Bf16Matvec matvec(const Mat& m, const float* x, float* out) {
    Bf16Matvec v;
    memset(&v, 0, sizeof(v));
    v.w = m.w; v.rows = m.rows; v.K = m.cols; v.ldw = m.ld;
    v.x = x; v.y = out;
    return v;
}
void normed(Bf16Matvec* v, const Layered* L, const uint16_t* w) {
    v->pro = PRO_RMSNORM;
    v->norm_w = w;
    v->norm_offset = L->cfg.norm_offset;
    v->eps = L->cfg.norm_eps;
}
// final norm + lm_head of d->hidden_a -> logits and arg-max; with `state` the decode step ends here
int head_top1(Decoder* d, cudaStream_t s, DecodeState* state) {
    Layered* L = d->lay;
    Bf16Matvec v = matvec(L->head, d->hidden_a, L->logits);
    normed(&v, L, d->final_norm);
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
    int max_o = 1;
    for (const LLayer& y : L->layers) {
        max_o = std::max(max_o, y.width());
        if (y.sp.mixer == KMLL_MIXER_LINEAR_ATTENTION && !c.compute_f32 && !L->plain)
            lin = std::max(lin, linear_attention_scratch_floats(want, y.sp.heads, y.sp.dim, y.sp.vdim));
    }
    auto take = [&](void** p, size_t bytes) -> int {
        cudaError_t er = cudaMalloc(p, bytes + 64);
        if (er != cudaSuccess) return fail(KMLL_ERR_CUDA, "prompt scratch (%zu bytes): %s", bytes, cudaGetErrorString(er));
        L->row_allocs.push_back(*p);
        total += bytes;
        return KMLL_OK;
    };
    KMLL_TRY(take((void**)&L->x, (size_t)want * c.dim * 4));
    KMLL_TRY(take((void**)&L->o, (size_t)want * max_o * 4));
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

int gemm(const Layered* L, cudaStream_t s, const void* x, int ldx, int T, const uint16_t* w, int rows, int K, int ldw, void* out, bool out_f32, int ldo,
         const float* residual = nullptr, int silu_rows = 0) {
    Bf16Gemm g;
    memset(&g, 0, sizeof(g));
    g.x = x; g.x_f32 = L->cfg.compute_f32; g.ldx = ldx; g.T = T; g.K = K;
    g.w = w; g.rows = rows; g.ldw = ldw;
    g.out = out; g.out_bf16 = !(out_f32 || L->cfg.compute_f32); g.ldo = ldo;
    g.residual = residual; g.silu_rows = silu_rows;
    g.partial = L->gemm_partial; g.counters = L->gemm_counters;
    return bf16_gemm(s, g);
}

// T tokens (already in the token log) through the layers from position pos0; the residual stream ends up in L->x
int forward_rows(Decoder* d, cudaStream_t s, int pos0, int T, float* tap, size_t tap_stride) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    const int f32 = c.compute_f32;
    KMLL_TRY(embed_rows(s, d->embedding, L->pos_table, c.vocab_size, c.dim, L->token_log + pos0, pos0, T, L->x));
    const int ldx = up8(c.dim);
    for (size_t l = 0; l < L->layers.size(); ++l) {
        LLayer& y = L->layers[l];
        const kmll_layer_spec& sp = y.sp;
        const int ldw = up8(y.width());
        KMLL_TRY(norm_rows(s, L->x, c.dim, nullptr, T, y.norm1, c.norm_offset, c.norm_eps, f32, L->a, ldx));
        if (sp.mixer == KMLL_MIXER_LINEAR_ATTENTION) {
            KMLL_TRY(gemm(L, s, L->a, ldx, T, y.proj.w, y.proj.rows, c.dim, y.proj.ld, L->p, false, L->ldp, nullptr,
                          sp.qkv_act == KMLL_ACT_SILU ? y.off_g : 0));
            LinearAttnArgs a = linear_args(L, y);
            a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o; a.scratch = L->lin;
            if (!L->plain && linear_attention_chunked_ok(a)) KMLL_TRY(linear_attention_chunked(s, a));
            else KMLL_TRY(linear_attention_recurrent(s, a));
            const void* gate = f32 ? (const void*)((const float*)L->p + y.off_g) : (const void*)((const uint16_t*)L->p + y.off_g);
            KMLL_TRY(gated_rows(s, L->o, y.width(), y.width(), T, y.mix_norm, sp.vdim, c.norm_eps, gate, f32, L->ldp, sp.gate_act, L->a, ldw));
        } else {
            KMLL_TRY(gemm(L, s, L->a, ldx, T, y.proj.w, y.proj.rows, c.dim, y.proj.ld, L->p, false, L->ldp));
            LatentArgs a = latent_args(L, y);
            a.in = L->p; a.in_f32 = f32; a.T = T; a.pos0 = pos0; a.out = L->o;
            KMLL_TRY(latent_write_cache(s, a));
            if (!L->plain && latent_prefill_ok(a)) {
                a.first = sp.window > 0 ? std::max(0, pos0 - sp.window + 1) : 0;
                a.lde = up8(y.ukv.rows);
                const int rows = pos0 + T - a.first;
                KMLL_TRY(ensure_expanded(L, s, (size_t)rows * a.lde * 2));
                a.expanded = L->expanded;
                KMLL_TRY(gemm(L, s, (const uint16_t*)y.cache + (size_t)a.first * y.pitch, y.pitch, rows, y.ukv.w, y.ukv.rows, sp.kv_rank, y.ukv.ld, L->expanded,
                              false, a.lde));
                KMLL_TRY(latent_attention_prefill(s, a));
            } else {
                KMLL_TRY(latent_attention_plain(s, a));
            }
            KMLL_TRY(convert_rows(s, L->o, y.width(), y.width(), T, f32, L->a, ldw));
        }
        KMLL_TRY(gemm(L, s, L->a, ldw, T, y.wo.w, c.dim, y.width(), y.wo.ld, L->x, true, c.dim, L->x));
        if (sp.mlp != KMLL_MLP_NONE) {
            const int ldf = up8(sp.ff);
            KMLL_TRY(norm_rows(s, L->x, c.dim, nullptr, T, y.norm2, c.norm_offset, c.norm_eps, f32, L->a, ldx));
            KMLL_TRY(gemm(L, s, L->a, ldx, T, y.up.w, sp.ff, c.dim, y.up.ld, L->z, false, L->ldz));
            KMLL_TRY(polynorm_rows(s, L->z, f32, L->ldz, sp.ff, T, y.act, c.norm_eps, L->a, ldf));
            KMLL_TRY(gemm(L, s, L->a, ldf, T, y.down.w, c.dim, sp.ff, y.down.ld, L->x, true, c.dim, L->x));
        }
        if (tap != nullptr) KMLL_CUDA(cudaMemcpyAsync(tap + l * tap_stride, L->x, (size_t)T * c.dim * 4, cudaMemcpyDeviceToDevice, s));
    }
    return KMLL_OK;
}

}  // namespace

int layered_enqueue_step(Decoder* d, cudaStream_t s, int* launches) {
    Layered* L = d->lay;
    const kmll_layered_config& c = L->cfg;
    const unsigned long long before = launch_counter();
    KMLL_TRY(ready(d));
    KMLL_TRY(decode_begin(s, d->embedding, c.vocab_size, c.dim, d->state, d->history, d->history_cap, d->hidden_a, nullptr, L->pos_table, L->token_log));
    float* const x = d->hidden_a;
    for (LLayer& y : L->layers) {
        const kmll_layer_spec& sp = y.sp;
        Bf16Matvec in = matvec(y.proj, x, L->proj1);
        normed(&in, L, y.norm1);
        Bf16Matvec out = matvec(y.wo, L->o1, x);
        out.residual = x;
        if (sp.mixer == KMLL_MIXER_LINEAR_ATTENTION) {
            if (sp.qkv_act == KMLL_ACT_SILU) in.silu_rows = y.off_g;
            KMLL_TRY(bf16_matvec(s, in));
            LinearAttnArgs a = linear_args(L, y);
            a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = L->o1;
            KMLL_TRY(linear_attention_recurrent(s, a));
            out.pro = PRO_GATED;
            out.norm_w = y.mix_norm;
            out.head_len = sp.vdim;
            out.eps = c.norm_eps;
            out.gate = L->proj1 + y.off_g;
            out.gate_act = sp.gate_act;
        } else {
            KMLL_TRY(bf16_matvec(s, in));
            LatentArgs a = latent_args(L, y);
            a.in = L->proj1; a.in_f32 = 1; a.T = 1; a.at = d->state; a.out = L->o1; a.work = L->latent_work;
            if (!L->plain && latent_decode_ok(a)) {
                KMLL_TRY(latent_attention_decode(s, a));
            } else {
                KMLL_TRY(latent_write_cache(s, a));
                KMLL_TRY(latent_attention_plain(s, a));
            }
        }
        KMLL_TRY(bf16_matvec(s, out));
        if (sp.mlp != KMLL_MLP_NONE) {
            Bf16Matvec up = matvec(y.up, x, L->z1);
            normed(&up, L, y.norm2);
            KMLL_TRY(bf16_matvec(s, up));
            Bf16Matvec down = matvec(y.down, L->z1, x);
            down.pro = PRO_POLYNORM;
            down.coef = y.act;
            down.eps = c.norm_eps;
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
            KMLL_TRY(norm_rows(s, L->x, c.dim, L->want, w1 - wi, d->final_norm, c.norm_offset, c.norm_eps, c.compute_f32, L->a, up8(c.dim)));
            KMLL_TRY(gemm(L, s, L->a, up8(c.dim), w1 - wi, L->head.w, L->head.rows, c.dim, L->head.ld, logits_out + (size_t)wi * c.vocab_size, true, c.vocab_size));
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
    auto rows = [&](const Mat& m, int r0, int n) { out->w = m.w != nullptr ? m.w + (size_t)r0 * m.ld : nullptr; out->rows = n; out->cols = m.cols; out->ld = m.ld; };
    if (layer == -1) {
        switch (tensor) {
            case KMLL_T_EMBEDDING: out->w = d->embedding; out->rows = c.vocab_size; out->cols = out->ld = c.dim; break;
            case KMLL_T_POSITION: out->w = L->pos_table; out->rows = c.position_rows; out->cols = out->ld = c.dim; break;
            case KMLL_T_FINAL_NORM: vec(d->final_norm, c.dim); break;
            case KMLL_T_OUTPUT: rows(L->head, 0, c.vocab_size); break;
            default: break;
        }
    } else {
        if (layer < 0 || layer >= c.n_layers) return fail(KMLL_ERR_SHAPE, "layer %d out of range", layer);
        LLayer& y = L->layers[layer];
        const kmll_layer_spec& s = y.sp;
        const bool lin = s.mixer == KMLL_MIXER_LINEAR_ATTENTION, ff = s.mlp != KMLL_MLP_NONE;
        switch (tensor) {
            case KMLL_T_ATTENTION_NORM: vec(y.norm1, c.dim); break;
            case KMLL_T_WQ: rows(y.proj, 0, y.off_k); break;
            case KMLL_T_WK: if (lin) rows(y.proj, y.off_k, s.heads * s.dim); break;
            case KMLL_T_WV: if (lin) rows(y.proj, y.off_v, s.heads * s.vdim); break;
            case KMLL_T_GATE: if (lin) rows(y.proj, y.off_g, s.heads * s.vdim); break;
            case KMLL_T_MIX_NORM: if (lin) vec(y.mix_norm, s.heads * s.vdim); break;
            case KMLL_T_DKV: if (!lin) rows(y.proj, y.off_k, s.kv_rank + s.rot_dim); break;
            case KMLL_T_DKV_NORM: if (!lin) vec(y.dkv_norm, s.kv_rank); break;
            case KMLL_T_UK: if (!lin) rows(y.ukv, 0, s.heads * s.dim); break;
            case KMLL_T_UV: if (!lin) rows(y.ukv, s.heads * s.dim, s.heads * s.vdim); break;
            case KMLL_T_WO: rows(y.wo, 0, c.dim); break;
            case KMLL_T_FFN_NORM: if (ff) vec(y.norm2, c.dim); break;
            case KMLL_T_W3: if (ff) rows(y.up, 0, s.ff); break;
            case KMLL_T_W2: if (ff) rows(y.down, 0, c.dim); break;
            case KMLL_T_ACT: if (ff) vec(y.act, 4); break;
            default: break;
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
        KMLL_TRY(normal(d->embedding, (size_t)c.vocab_size * c.dim));
        if (L->pos_table) KMLL_TRY(normal(L->pos_table, (size_t)c.position_rows * c.dim));
        KMLL_TRY(constant(d->final_norm, c.dim, neutral));
        if (tie_embeddings) KMLL_CUDA(cudaMemcpy2D(L->head.w, (size_t)L->head.ld * 2, d->embedding, (size_t)c.dim * 2, (size_t)c.dim * 2, c.vocab_size, cudaMemcpyDeviceToDevice));
        else KMLL_TRY(mat(L->head));
        for (LLayer& y : L->layers) {
            KMLL_TRY(constant(y.norm1, c.dim, neutral));
            KMLL_TRY(mat(y.proj));
            KMLL_TRY(mat(y.wo));
            if (y.ukv.w) KMLL_TRY(mat(y.ukv));
            if (y.dkv_norm) KMLL_TRY(constant(y.dkv_norm, y.sp.kv_rank, 1.0f));
            if (y.mix_norm) KMLL_TRY(constant(y.mix_norm, y.width(), 1.0f));
            if (y.sp.mlp != KMLL_MLP_NONE) {
                KMLL_TRY(constant(y.norm2, c.dim, neutral));
                KMLL_TRY(mat(y.up));
                KMLL_TRY(mat(y.down));
                KMLL_TRY(constant(y.act, 3, 1.0f / 3.0f));
                KMLL_TRY(constant(y.act + 3, 1, 0.0f));
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
    LLayer& y = d->lay->layers[layer];
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
    LLayer& y = d->lay->layers[layer];
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
