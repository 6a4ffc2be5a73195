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

}  // extern "C"
