// C ABI of the layered decoders' operators (include/kmll_b200.h): argument checks, then the launches the decoder itself uses.
#include <cstring>

#include "internal.cuh"

using namespace kmll;

namespace {
Bf16Matvec base(const float* x, const uint16_t* w, int pitch, int rows, int cols, const float* residual, float* y) {
    Bf16Matvec v;
    memset(&v, 0, sizeof(v));
    v.x = x; v.w = w; v.ldw = pitch; v.rows = rows; v.K = cols; v.residual = residual; v.y = y; v.out_scale = 1.0f;
    return v;
}
int up8(int v) { return (v + 7) & ~7; }
}  // namespace

extern "C" {

int kmll_linear_bf16(kmll_stream_t s, const float* x, const uint16_t* w, int pitch, int rows, int cols, const uint16_t* norm_weight, float norm_offset,
                     float eps, const float* residual, int silu_rows, float* y) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(y);
    Bf16Matvec v = base(x, w, pitch, rows, cols, residual, y);
    v.silu_rows = silu_rows;
    if (norm_weight != nullptr) { v.pro = PRO_NORM; v.norm = NormArgs{KMLL_NORM_RMS, norm_weight, nullptr, norm_offset, eps}; }
    return bf16_matvec(as_stream(s), v);
}

int kmll_polynorm_linear_bf16(kmll_stream_t s, const float* x, const uint16_t* coef, float eps, const uint16_t* w, int pitch, int rows, int cols,
                              const float* residual, float* y) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(coef); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(y);
    Bf16Matvec v = base(x, w, pitch, rows, cols, residual, y);
    v.pro = PRO_POLYNORM; v.coef = coef; v.eps = eps;
    return bf16_matvec(as_stream(s), v);
}

int kmll_gated_linear_bf16(kmll_stream_t s, const float* x, const uint16_t* norm_weight, int head_len, float eps, const float* gate, int gate_sigmoid,
                           const uint16_t* w, int pitch, int rows, int cols, const float* residual, float* y) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(gate); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(y);
    KMLL_REQUIRE(norm_weight != nullptr || (head_len > 0 && cols > 0 && cols % head_len == 0), "gated_linear_bf16: %d columns are not heads of %d", cols, head_len);
    Bf16Matvec v = base(x, w, pitch, rows, cols, residual, y);
    v.pro = PRO_GATED;
    v.n_seg = 1;
    v.seg[0] = GateSegment{0, cols, norm_weight != nullptr ? cols : head_len, norm_weight != nullptr ? KMLL_OUT_NORM_JOINT : KMLL_OUT_NORM_PER_HEAD, norm_weight, gate, 1,
                           gate_sigmoid ? KMLL_ACT_SIGMOID : KMLL_ACT_SILU, 1.0f, eps};
    return bf16_matvec(as_stream(s), v);
}

size_t kmll_linear_batched_bf16_workspace_bytes(void) { return 512 + kGemmPartialFloats * 4; }

int kmll_linear_batched_bf16(kmll_stream_t s, const void* x, int x_f32, int ldx, int batch, const uint16_t* w, int pitch, int rows, int cols,
                             const float* residual, void* workspace, void* out, int out_bf16) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(out);
    Bf16Gemm g;
    memset(&g, 0, sizeof(g));
    g.x = x; g.x_f32 = x_f32; g.ldx = ldx; g.T = batch; g.K = cols; g.w = w; g.rows = rows; g.ldw = pitch; g.out = out; g.out_bf16 = out_bf16; g.ldo = rows;
    g.residual = residual; g.out_scale = 1.0f;
    if (workspace != nullptr) {
        g.counters = static_cast<unsigned int*>(workspace);
        g.partial = static_cast<float*>(workspace) + 128;
    }
    return bf16_gemm(as_stream(s), g);
}

int kmll_polynorm_rows_bf16(kmll_stream_t s, const uint16_t* x, int batch, int dim, const uint16_t* coef, float eps, uint16_t* out) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(coef); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(batch > 0 && dim > 0, "polynorm_rows: bad shape");
    return polynorm_rows(as_stream(s), x, 0, dim, dim, batch, coef, eps, out, dim);
}

size_t kmll_linear_attention_scratch_floats(int tokens, int heads, int dk, int dv) { return linear_attention_scratch_floats(tokens, heads, dk, dv); }

int kmll_linear_attention(kmll_stream_t s, const void* in, int in_f32, int ld, int q_off, int k_off, int v_off, int tokens, int heads, int dk, int dv,
                          int rot, const float* table, int position, const int* position_device, float key_scale, const float* powers, float* state,
                          float* scratch, float* out) {
    KMLL_REQUIRE_PTR(in); KMLL_REQUIRE_PTR(powers); KMLL_REQUIRE_PTR(state); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(tokens > 0 && heads > 0 && dk > 0 && dv > 0 && rot >= 0 && rot <= dk && (rot & 1) == 0 && position >= 0, "linear_attention: bad shape");
    if (rot > 0) KMLL_REQUIRE_PTR(table);
    LinearAttnArgs a;
    memset(&a, 0, sizeof(a));
    a.in = in; a.in_f32 = in_f32; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.T = tokens; a.heads = heads; a.dk = dk; a.dv = dv; a.rot = rot;
    a.table = reinterpret_cast<const float2*>(table);
    a.at = reinterpret_cast<const DecodeState*>(position_device);  // (the position is its first field)
    a.pos0 = position; a.key_scale = key_scale; a.powers = powers; a.state = state; a.scratch = scratch; a.out = out; a.ldo = heads * dv;
    return scratch != nullptr ? linear_attention_chunked(as_stream(s), a) : linear_attention_recurrent(as_stream(s), a);
}

static LatentArgs latent_base(int heads, int dim, int rot, int vdim, int rank, int window, float scale, const float* table, const uint16_t* cache, int pitch,
                              int max_seq, float* out) {
    LatentArgs a;
    memset(&a, 0, sizeof(a));
    a.dkv_off = heads * (dim + rot);
    a.heads = heads; a.dim = dim; a.rot = rot; a.vdim = vdim; a.rank = rank; a.window = window; a.scale = scale;
    a.table = reinterpret_cast<const float2*>(table);
    a.cache = const_cast<uint16_t*>(cache); a.pitch = pitch; a.kr_off = up8(rank); a.max_seq = max_seq;
    a.out = out; a.ldo = heads * vdim;
    return a;
}

size_t kmll_latent_attention_workspace_floats(int heads, int rank, int rot, int window, int max_seq) {
    return latent_decode_work_floats(heads, rank, rot, window > 0 && window < max_seq ? window : max_seq);
}

int kmll_latent_attention_decode(kmll_stream_t s, const float* in, int heads, int dim, int rot, int vdim, int rank, int window, float scale, float eps,
                                 const uint16_t* latent_norm, const uint16_t* w_uk_uv, int w_pitch, const float* table, const int* position_device,
                                 uint16_t* cache, int pitch, int max_seq, float* workspace, float* out) {
    KMLL_REQUIRE_PTR(in); KMLL_REQUIRE_PTR(latent_norm); KMLL_REQUIRE_PTR(w_uk_uv); KMLL_REQUIRE_PTR(position_device); KMLL_REQUIRE_PTR(cache);
    KMLL_REQUIRE_PTR(workspace); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && rank > 0 && rot >= 0 && (rot & 1) == 0 && (pitch & 7) == 0 && pitch >= up8(rank) + rot && (w_pitch & 7) == 0 &&
                     w_pitch >= rank, "latent_attention_decode: bad shape");
    if (rot > 0) KMLL_REQUIRE_PTR(table);
    LatentArgs a = latent_base(heads, dim, rot, vdim, rank, window, scale, table, cache, pitch, max_seq, out);
    a.in = in; a.in_f32 = 1; a.T = 1; a.eps = eps; a.norm_w = latent_norm; a.uk = w_uk_uv; a.uv = w_uk_uv + (size_t)heads * dim * w_pitch; a.ldu = w_pitch;
    a.at = reinterpret_cast<const DecodeState*>(position_device);
    a.work = workspace;
    if (!latent_decode_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "latent_attention_decode: latent size %d is too large", rank);
    return latent_attention_decode(as_stream(s), a);
}

int kmll_latent_attention_prefill(kmll_stream_t s, const uint16_t* in, int ld, int tokens, int position, int heads, int dim, int rot, int vdim, int rank,
                                  int window, float scale, const float* table, const uint16_t* cache, int pitch, int max_seq, const uint16_t* expanded, int lde,
                                  int first, float* out) {
    KMLL_REQUIRE_PTR(in); KMLL_REQUIRE_PTR(cache); KMLL_REQUIRE_PTR(expanded); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(tokens > 0 && position >= 0 && position + tokens <= max_seq && heads > 0 && dim > 0 && vdim > 0 && rank > 0 && rot >= 0 && (rot & 1) == 0 &&
                     (pitch & 7) == 0 && pitch >= up8(rank) + rot && first >= 0 && first <= (window > 0 && position >= window ? position - window + 1 : 0),
                 "latent_attention_prefill: bad shape");
    if (rot > 0) KMLL_REQUIRE_PTR(table);
    LatentArgs a = latent_base(heads, dim, rot, vdim, rank, window, scale, table, cache, pitch, max_seq, out);
    a.in = in; a.ld = ld; a.T = tokens; a.pos0 = position; a.expanded = const_cast<uint16_t*>(expanded); a.lde = lde; a.first = first;
    return latent_attention_prefill(as_stream(s), a);
}

int kmll_normed_linear_bf16(kmll_stream_t s, const float* x, const uint16_t* w, int pitch, int rows, int cols, int norm, const uint16_t* norm_weight,
                            const uint16_t* norm_bias, float eps, int pair_act, float out_scale, float* y) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(y);
    if (norm == KMLL_NORM_LAYER && norm_weight != nullptr) KMLL_REQUIRE_PTR(norm_bias);
    Bf16Matvec v = base(x, w, pitch, rows, cols, nullptr, y);
    v.pair_act = pair_act;
    v.out_scale = out_scale;
    if (norm_weight != nullptr) { v.pro = PRO_NORM; v.norm = NormArgs{norm, norm_weight, norm_bias, 0.0f, eps}; }
    return bf16_matvec(as_stream(s), v);
}

int kmll_pair_linear_batched_bf16(kmll_stream_t s, const void* x, int x_f32, int ldx, int batch, const uint16_t* w, int pitch, int rows, int cols, int pair_act,
                                  void* workspace, void* out) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(pair_act != KMLL_ACT_NONE, "pair_linear_batched: no activation");
    Bf16Gemm g;
    memset(&g, 0, sizeof(g));
    g.x = x; g.x_f32 = x_f32; g.ldx = ldx; g.T = batch; g.K = cols; g.w = w; g.rows = rows; g.ldw = pitch; g.out = out; g.out_bf16 = !x_f32; g.ldo = rows / 2;
    g.pair_act = pair_act; g.out_scale = 1.0f;
    if (workspace != nullptr) {
        g.counters = static_cast<unsigned int*>(workspace);
        g.partial = static_cast<float*>(workspace) + 128;
    }
    return bf16_gemm(as_stream(s), g);
}

int kmll_norm_rows_bf16(kmll_stream_t s, const float* x, int batch, int dim, int norm, const uint16_t* weight, const uint16_t* bias, float eps, uint16_t* out) {
    KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(weight); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE(batch > 0 && dim > 0, "norm_rows: bad shape");
    if (norm == KMLL_NORM_LAYER) KMLL_REQUIRE_PTR(bias);
    return norm_rows(as_stream(s), x, dim, nullptr, batch, NormArgs{norm, weight, bias, 0.0f, eps}, 0, out, dim);
}

int kmll_mixer_output_linear_bf16(kmll_stream_t s, const kmll_mixer_spec* mixers, int n_mixers, const float* x, const uint16_t* const* norm_weights,
                                  const float* const* gates, float eps, const uint16_t* w, int pitch, int rows, int cols, const float* residual, float* y) {
    KMLL_REQUIRE_PTR(mixers); KMLL_REQUIRE_PTR(x); KMLL_REQUIRE_PTR(norm_weights); KMLL_REQUIRE_PTR(gates); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(y);
    KMLL_REQUIRE(n_mixers == 1 || n_mixers == 2, "mixer_output_linear: %d mixers", n_mixers);
    Bf16Matvec v = base(x, w, pitch, rows, cols, residual, y);
    v.pro = PRO_GATED;
    v.n_seg = n_mixers;
    int at = 0;
    for (int i = 0; i < n_mixers; ++i) {
        const kmll_mixer_spec& m = mixers[i];
        KMLL_REQUIRE(m.heads > 0 && m.vdim > 0, "mixer_output_linear: bad shape");
        const bool att = m.mixer == KMLL_MIXER_ATTENTION;
        v.seg[i] = GateSegment{up8(at), m.heads * m.vdim, m.vdim, att ? KMLL_OUT_NORM_NONE : m.out_norm, norm_weights[i], gates[i], att ? m.vdim : 1, m.gate_act, m.out_scale, eps};
        if (v.seg[i].norm == KMLL_OUT_NORM_JOINT || v.seg[i].norm == KMLL_OUT_NORM_HEAD_WEIGHTED) KMLL_REQUIRE_PTR(norm_weights[i]);
        at = v.seg[i].begin + v.seg[i].cols;
    }
    KMLL_REQUIRE(at == cols, "mixer_output_linear: the mixers give %d columns, not %d", at, cols);
    return bf16_matvec(as_stream(s), v);
}

int kmll_grouped_attention(kmll_stream_t s, const kmll_mixer_spec* m, const void* in, int in_f32, int ld, int q_off, int k_off, int v_off, int tokens, int position,
                           const int* position_device, void* cache, int cache_f32, int pitch, int max_seq, float* out, int ldo) {
    KMLL_REQUIRE_PTR(m); KMLL_REQUIRE_PTR(in); KMLL_REQUIRE_PTR(cache); KMLL_REQUIRE_PTR(out);
    const int g = m->kv_heads > 0 ? m->kv_heads : m->heads;
    KMLL_REQUIRE(m->heads > 0 && m->heads % g == 0 && m->dim > 0 && m->vdim > 0 && m->window >= 0 && m->chunk >= 0 && tokens > 0 && position >= 0 &&
                     (position_device != nullptr || position + tokens <= max_seq) && (pitch & 7) == 0 && pitch >= g * (up8(m->dim) + up8(m->vdim)) && ldo >= m->heads * m->vdim,
                 "grouped_attention: bad shape");
    GroupedArgs a;
    memset(&a, 0, sizeof(a));
    a.in = in; a.in_f32 = in_f32; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off;
    a.T = tokens; a.heads = m->heads; a.kv_heads = g; a.dim = m->dim; a.vdim = m->vdim; a.window = m->window; a.chunk = m->chunk; a.scale = m->score_scale;
    a.at = reinterpret_cast<const DecodeState*>(position_device);  // (the position is its first field)
    a.pos0 = position;
    a.cache = cache; a.cache_f32 = cache_f32; a.pitch = pitch; a.dimp = up8(m->dim); a.vdimp = up8(m->vdim); a.max_seq = max_seq;
    a.out = out; a.ldo = ldo;
    if (grouped_decode_ok(a)) return grouped_attention_decode(as_stream(s), a);
    KMLL_TRY_RC(grouped_write_cache(as_stream(s), a));
    return position_device == nullptr && grouped_prefill_ok(a) ? grouped_attention_prefill(as_stream(s), a) : grouped_attention_plain(as_stream(s), a);
}

size_t kmll_gated_linear_scratch_floats(const kmll_mixer_spec* m, int tokens) {
    return m != nullptr && tokens > 0 ? gated_chunk_scratch_floats(tokens, m->heads, m->dim, m->vdim, m->delta) : 0;
}

int kmll_gated_linear_attention(kmll_stream_t s, const kmll_mixer_spec* m, const kmll_gated_linear_weights* w, const void* in, int in_f32, int ld, const int* offsets,
                                int tokens, int position, const int* position_device, float* state, float* ring, float* scratch, float* gate, float* out, int ldo) {
    KMLL_REQUIRE_PTR(m); KMLL_REQUIRE_PTR(w); KMLL_REQUIRE_PTR(in); KMLL_REQUIRE_PTR(offsets); KMLL_REQUIRE_PTR(state); KMLL_REQUIRE_PTR(out);
    KMLL_REQUIRE_PTR(w->decay_up);
    const int g = m->kv_heads > 0 ? m->kv_heads : m->heads;
    KMLL_REQUIRE(m->heads > 0 && m->heads % g == 0 && m->dim > 0 && m->vdim > 0 && m->decay_rank > 0 && (w->decay_pitch & 7) == 0 && w->decay_pitch >= m->decay_rank &&
                     m->conv >= 0 && m->conv <= kMaxConvTaps && tokens > 0 && position >= 0 && ldo >= m->heads * m->vdim &&
                     (m->decay == KMLL_DECAY_SOFTPLUS || (m->decay == KMLL_DECAY_LOGISTIC && m->decay_tau > 0.0f)),
                 "gated_linear_attention: bad shape");
    KMLL_REQUIRE(position_device == nullptr || tokens == 1, "gated_linear_attention: a position on the device is for one token");
    if (m->decay == KMLL_DECAY_SOFTPLUS) KMLL_REQUIRE_PTR(w->decay_log);
    if (m->conv > 0) { KMLL_REQUIRE_PTR(w->conv); KMLL_REQUIRE_PTR(ring); }
    GatedLinearArgs a;
    memset(&a, 0, sizeof(a));
    a.in = in; a.in_f32 = in_f32; a.ld = ld;
    a.q_off = offsets[0]; a.k_off = offsets[1]; a.v_off = offsets[2]; a.a_off = offsets[3]; a.b_off = offsets[4]; a.g_off = offsets[5];
    a.T = tokens; a.heads = m->heads; a.kv_heads = g; a.dk = m->dim; a.dv = m->vdim;
    a.decay = m->decay; a.inv_tau = m->decay == KMLL_DECAY_LOGISTIC ? 1.0f / m->decay_tau : 0.0f; a.rank = m->decay_rank;
    a.up = w->decay_up; a.ldu = w->decay_pitch; a.bias = w->decay_bias; a.a_log = w->decay_log;
    a.delta = m->delta; a.taps = m->conv; a.conv = w->conv; a.ring = ring; a.unit_eps = m->unit_eps; a.q_scale = m->q_scale;
    a.at = reinterpret_cast<const DecodeState*>(position_device);
    a.pos0 = position; a.state = state; a.out = out; a.ldo = ldo; a.scratch = scratch;
    if (scratch != nullptr) return gated_linear_chunked(as_stream(s), a);
    if (m->gate_rank > 0) {
        KMLL_REQUIRE_PTR(w->gate_up); KMLL_REQUIRE_PTR(gate);
        KMLL_REQUIRE((w->gate_pitch & 7) == 0 && w->gate_pitch >= m->gate_rank, "gated_linear_attention: bad gate pitch");
        a.gate_rank = m->gate_rank; a.gate_up = w->gate_up; a.ldg = w->gate_pitch; a.gate = gate;
    }
    return gated_linear_steps(as_stream(s), a);
}

}  // extern "C"
