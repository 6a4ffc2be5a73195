// Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, no softmax and no denominator.
//
//   recurrent form  token after token in f32 with the state in registers: decode steps, and prompts of decoders that compute
//                   in f32
//   chunked form    prompts in bf16: chunks of 64 tokens on the tensor cores (three launches)
//
// Rotated q and k, decays, scaled keys and the state are f32 throughout; where they meet the tensor cores they are split into
// a bf16 head and a bf16 remainder (16 mantissa bits, products exact, f32 accumulation).
#include "internal.cuh"
#include "mma_bf16.cuh"

namespace kmll {

namespace {

template <bool F32>
__device__ inline float in_at(const void* p, size_t i) {
    return F32 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
// element i of a head vector of which the first `rot` entries are rotated (i pairs with i + rot / 2); cs: this position's row
template <bool F32>
__device__ inline float rotated_at(const void* p, size_t base, int i, int rot, const float2* cs) {
    if (i >= rot) return in_at<F32>(p, base + i);
    const int half = rot >> 1, j = i < half ? i : i - half;
    const float u = in_at<F32>(p, base + j), v = in_at<F32>(p, base + j + half);
    const float2 t = cs[j];
    return i < half ? u * t.x - v * t.y : v * t.x + u * t.y;
}

// ---- recurrent form -------------------------------------------------------------------------------------------------------
// Block (head, 32 value columns): thread (part, column quad) keeps RP rows of four state columns in registers for the whole
// call.  The state is fetched before the dependency wait: its last writer lies more than one launch back.
template <bool F32, int RP>
__global__ void __launch_bounds__(256) linear_recurrent_kernel(const LinearAttnArgs a) {
    extern __shared__ float lsm[];  // q [dk] | k [dk] | reduction [8][32]
    float* const sq = lsm;
    float* const sk = lsm + a.dk;
    float* const red = lsm + 2 * a.dk;
    const int h = blockIdx.x, tid = threadIdx.x, part = tid >> 3, cq = tid & 7, lane = tid & 31, warp = tid >> 5;
    const int c0 = blockIdx.y * 32 + cq * 4;
    float* const S = a.state + (size_t)h * a.dk * a.dv;
    const bool vec = (a.dv & 3) == 0;
    float s[RP][4];
#pragma unroll
    for (int r = 0; r < RP; ++r) {
        const int i = part + r * 32;
#pragma unroll
        for (int e = 0; e < 4; ++e) s[r][e] = 0.0f;
        if (i < a.dk && c0 < a.dv) {
            if (vec) {
                const float4 t = *reinterpret_cast<const float4*>(S + (size_t)i * a.dv + c0);
                s[r][0] = t.x; s[r][1] = t.y; s[r][2] = t.z; s[r][3] = t.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (c0 + e < a.dv) s[r][e] = S[(size_t)i * a.dv + c0 + e];
            }
        }
    }
    const float decay = a.powers[(size_t)h * (kLinChunk + 1) + 1];
    pdl_wait();
    const int pos0 = a.at != nullptr ? a.at->position : a.pos0;
    const int half = a.rot >> 1;
    for (int t = 0; t < a.T; ++t) {
        const size_t row = (size_t)t * a.ld;
        const float2* cs = a.rot > 0 ? a.table + (size_t)(pos0 + t) * half : nullptr;
        for (int i = tid; i < 2 * a.dk; i += 256) {
            if (i < a.dk) sq[i] = rotated_at<F32>(a.in, row + a.q_off + (size_t)h * a.dk, i, a.rot, cs);
            else sk[i - a.dk] = rotated_at<F32>(a.in, row + a.k_off + (size_t)h * a.dk, i - a.dk, a.rot, cs) * a.key_scale;
        }
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = c0 + e < a.dv ? in_at<F32>(a.in, row + a.v_off + (size_t)h * a.dv + c0 + e) : 0.0f;
        __syncthreads();
        float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int r = 0; r < RP; ++r) {
            const int i = part + r * 32;
            if (i < a.dk) {
                const float k = sk[i], q = sq[i];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[r][e] = fmaf(decay, s[r][e], k * v[e]);
                    o[e] = fmaf(q, s[r][e], o[e]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
        }
        if (lane < 8)
#pragma unroll
            for (int e = 0; e < 4; ++e) red[warp * 32 + lane * 4 + e] = o[e];
        __syncthreads();
        const int c = blockIdx.y * 32 + tid;
        if (tid < 32 && c < a.dv) {
            float sum = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) sum += red[w * 32 + tid];
            a.out[(size_t)t * a.heads * a.dv + (size_t)h * a.dv + c] = sum;
        }
        // (the next token's q and k overwrite nothing that is still read: all reads of them lie before the barrier above;
        // `red` is rewritten only after the next barrier)
    }
#pragma unroll
    for (int r = 0; r < RP; ++r) {
        const int i = part + r * 32;
        if (i < a.dk && c0 < a.dv) {
            if (vec) {
                *reinterpret_cast<float4*>(S + (size_t)i * a.dv + c0) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (c0 + e < a.dv) S[(size_t)i * a.dv + c0 + e] = s[r][e];
            }
        }
    }
}

// ---- chunked form -----------------------------------------------------------------------------------------------------------
// 64 tokens per chunk, tiles of 64 value columns.  With n tokens in the chunk and S_in the state ahead of it:
//   states   KV = sum_j decay^(n-1-j) k_j v_j^T                     one block per (chunk, head, value tile)
//   scan     S_in of every chunk, and the state behind the last      elementwise, in place over the KV buffer
//   outputs  o_i = decay^(i+1) q_i S_in + sum_{j<=i} decay^(i-j) (q_i . k_j) v_j
constexpr int kC = kLinChunk, kVT = 64, kCThreads = 128;

// eight consecutive bf16 input values as f32; columns at or beyond `n` are zeros
__device__ inline void load8(const uint16_t* p, int i, int n, bool aligned, float (&v)[8]) {
    if (aligned && i + 8 <= n) {
        const uint4 t = *reinterpret_cast<const uint4*>(p + i);
        const uint32_t w[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            v[2 * e] = __uint_as_float(w[e] << 16);
            v[2 * e + 1] = __uint_as_float(w[e] & 0xffff0000u);
        }
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = i + e < n ? bf16_bits_to_f32(p[i + e]) : 0.0f;
    }
}
__device__ inline void store_split8(uint16_t* hi, uint16_t* lo, int at, const float (&v)[8], bool with_lo) {
    uint4 h, l;
    split_bf16x2(v[0], v[1], h.x, l.x);
    split_bf16x2(v[2], v[3], h.y, l.y);
    split_bf16x2(v[4], v[5], h.z, l.z);
    split_bf16x2(v[6], v[7], h.w, l.w);
    *reinterpret_cast<uint4*>(hi + at) = h;
    if (with_lo) *reinterpret_cast<uint4*>(lo + at) = l;
}

struct ChunkCtx {
    const uint16_t* in;
    int t0, n, pos0;  // first token of the chunk (row of `in`), its tokens, position of row 0
    bool al;          // 16-byte rows
};
// q or k tile [64 tokens][DK] of head h -> head (and remainder) tiles; scaled by `scale`
template <int DK, bool ROT>
__device__ inline void load_qk_tile(const LinearAttnArgs& a, const ChunkCtx& c, int off, int h, float scale, uint16_t* hi, uint16_t* lo) {
    constexpr int RUNS = DK / 8, P = DK + 8;
    const int half = a.rot >> 1;
    for (int i = threadIdx.x; i < kC * RUNS; i += kCThreads) {
        const int t = i / RUNS, r = (i - t * RUNS) * 8;
        float v[8] = {};
        if (t < c.n) {
            const uint16_t* p = c.in + (size_t)(c.t0 + t) * a.ld + off + (size_t)h * a.dk;
            if (!ROT || r >= a.rot) {
                load8(p, r, a.dk, c.al, v);
            } else if ((half & 7) == 0) {  // the run and its partner run lie in one half each
                float w[8];
                const bool low = r < half;
                load8(p, r, a.dk, c.al, v);
                load8(p, low ? r + half : r - half, a.dk, c.al, w);
                const float2* cs = a.table + (size_t)(c.pos0 + c.t0 + t) * half + (low ? r : r - half);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float2 f = cs[e];
                    v[e] = low ? v[e] * f.x - w[e] * f.y : v[e] * f.x + w[e] * f.y;
                }
            } else {
                const float2* cs = a.table + (size_t)(c.pos0 + c.t0 + t) * half;
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = r + e < a.dk ? rotated_at<false>(p, 0, r + e, a.rot, cs) : 0.0f;
            }
            if (ROT)
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] *= scale;
        }
        store_split8(hi, lo, t * P + r, v, ROT);
    }
}

template <int DK, bool ROT>
__global__ void __launch_bounds__(kCThreads) linear_chunk_states_kernel(const LinearAttnArgs a) {
    constexpr int P = DK + 8, PV = kVT + 8, MT = (DK / 16 + 3) / 4;
    extern __shared__ __align__(16) uint16_t csm[];
    uint16_t* const kh = csm;
    uint16_t* const kl = kh + kC * P;  // ROT only
    uint16_t* const vh = kh + (ROT ? 2 : 1) * kC * P;
    uint16_t* const vl = vh + kC * PV;
    pdl_wait();
    const int h = blockIdx.y, v0 = blockIdx.z * kVT, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    ChunkCtx c;
    c.in = static_cast<const uint16_t*>(a.in);
    c.t0 = blockIdx.x * kC;
    c.n = min(kC, a.T - c.t0);
    c.pos0 = a.at != nullptr ? a.at->position : a.pos0;
    c.al = ((a.ld | a.q_off | a.k_off | a.v_off | a.dk | a.dv) & 7) == 0;
    const float* pw = a.powers + (size_t)h * (kC + 1);
    load_qk_tile<DK, ROT>(a, c, a.k_off, h, a.key_scale, kh, kl);
    const float vscale = ROT ? 1.0f : a.key_scale;
    for (int i = tid; i < kC * (kVT / 8); i += kCThreads) {
        const int t = i / (kVT / 8), r = (i % (kVT / 8)) * 8;
        float v[8] = {};
        if (t < c.n) {
            load8(c.in + (size_t)(c.t0 + t) * a.ld + a.v_off + (size_t)h * a.dv, v0 + r, a.dv, c.al, v);
            const float w = pw[c.n - 1 - t] * vscale;
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] *= w;
        }
        store_split8(vh, vl, t * PV + r, v, true);
    }
    __syncthreads();
    float* const KV = a.scratch + ((size_t)blockIdx.x * a.heads + h) * a.dk * a.dv;
#pragma unroll
    for (int mi = 0; mi < MT; ++mi) {
        const int m0 = (warp + mi * 4) * 16;
        if (m0 >= a.dk || m0 >= DK) break;
        float acc[kVT / 8][4];
#pragma unroll
        for (int nb = 0; nb < kVT / 8; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nb][e] = 0.0f;
#pragma unroll
        for (int ks = 0; ks < kC / 16; ++ks) {
            const int ao = (ks * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * P + m0 + ((lane >> 3) & 1) * 8;
            uint32_t ah[4], al[4];
            ldmatrix_x4_trans(ah, kh + ao);
            if (ROT) ldmatrix_x4_trans(al, kl + ao);
#pragma unroll
            for (int d2 = 0; d2 < kVT / 16; ++d2) {
                const int bo = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8;
                uint32_t b[4];
                ldmatrix_x4_trans(b, vh + bo);
                mma_bf16(acc[2 * d2], ah, b[0], b[1]);
                mma_bf16(acc[2 * d2 + 1], ah, b[2], b[3]);
                if (ROT) {
                    mma_bf16(acc[2 * d2], al, b[0], b[1]);
                    mma_bf16(acc[2 * d2 + 1], al, b[2], b[3]);
                }
                ldmatrix_x4_trans(b, vl + bo);
                mma_bf16(acc[2 * d2], ah, b[0], b[1]);
                mma_bf16(acc[2 * d2 + 1], ah, b[2], b[3]);
            }
        }
        const int g = lane >> 2, tq = lane & 3;
#pragma unroll
        for (int nb = 0; nb < kVT / 8; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = m0 + g + (e >> 1) * 8, j = v0 + nb * 8 + 2 * tq + (e & 1);
                if (i < a.dk && j < a.dv) KV[(size_t)i * a.dv + j] = acc[nb][e];
            }
    }
}

__global__ void __launch_bounds__(256) linear_chunk_scan_kernel(const LinearAttnArgs a) {
    pdl_wait();
    const size_t per_head = (size_t)a.dk * a.dv, total = per_head * a.heads;
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= total) return;
    const float* pw = a.powers + (i / per_head) * (kC + 1);
    const int chunks = (a.T + kC - 1) / kC;
    float s = a.state[i];
    for (int c0 = 0; c0 < chunks; c0 += 8) {
        float kv[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) kv[j] = c0 + j < chunks ? a.scratch[(size_t)(c0 + j) * total + i] : 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (c0 + j >= chunks) break;
            a.scratch[(size_t)(c0 + j) * total + i] = s;
            s = fmaf(pw[min(kC, a.T - (c0 + j) * kC)], s, kv[j]);
        }
    }
    a.state[i] = s;
}

template <int DK, bool ROT>
__global__ void __launch_bounds__(kCThreads) linear_chunk_outputs_kernel(const LinearAttnArgs a) {
    constexpr int P = DK + 8, PV = kVT + 8, KS = DK / 16;
    extern __shared__ __align__(16) uint16_t csm[];
    uint16_t* const qh = csm;
    uint16_t* const kh = qh + kC * P;
    uint16_t* const ql = kh + kC * P;  // ROT only
    uint16_t* const kl = ql + kC * P;
    uint16_t* const vh = qh + (ROT ? 4 : 2) * kC * P;
    uint16_t* const sh = vh + kC * PV;
    uint16_t* const sl = sh + DK * PV;
    __shared__ float pw[kC + 1];
    pdl_wait();
    const int h = blockIdx.y, v0 = blockIdx.z * kVT, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    ChunkCtx c;
    c.in = static_cast<const uint16_t*>(a.in);
    c.t0 = blockIdx.x * kC;
    c.n = min(kC, a.T - c.t0);
    c.pos0 = a.at != nullptr ? a.at->position : a.pos0;
    c.al = ((a.ld | a.q_off | a.k_off | a.v_off | a.dk | a.dv) & 7) == 0;
    if (tid <= kC) pw[tid] = a.powers[(size_t)h * (kC + 1) + tid];
    load_qk_tile<DK, ROT>(a, c, a.q_off, h, 1.0f, qh, ql);
    load_qk_tile<DK, ROT>(a, c, a.k_off, h, a.key_scale, kh, kl);
    const float sscale = ROT ? 1.0f : a.key_scale;  // without rotation the keys stay exact and the scores carry the factor
    for (int i = tid; i < kC * (kVT / 8); i += kCThreads) {
        const int t = i / (kVT / 8), r = (i % (kVT / 8)) * 8;
        float v[8] = {};
        if (t < c.n) load8(c.in + (size_t)(c.t0 + t) * a.ld + a.v_off + (size_t)h * a.dv, v0 + r, a.dv, c.al, v);
        store_split8(vh, nullptr, t * PV + r, v, false);
    }
    const float* S = a.scratch + ((size_t)blockIdx.x * a.heads + h) * a.dk * a.dv;
    const bool v4 = (a.dv & 3) == 0;
    for (int i = tid; i < DK * (kVT / 8); i += kCThreads) {
        const int d = i / (kVT / 8), r = (i % (kVT / 8)) * 8;
        float v[8] = {};
        if (d < a.dk) {
            const float* p = S + (size_t)d * a.dv + v0 + r;
            if (v4 && v0 + r + 8 <= a.dv) {
                const float4 x = *reinterpret_cast<const float4*>(p), y = *reinterpret_cast<const float4*>(p + 4);
                v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e)
                    if (v0 + r + e < a.dv) v[e] = p[e];
            }
        }
        store_split8(sh, sl, d * PV + r, v, true);
    }
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3, ra = warp * 16 + g, rb = ra + 8;  // this lane's two token rows
    if (warp * 16 >= c.n) return;
    float sc[kC / 8][4], o[kVT / 8][4];
#pragma unroll
    for (int nb = 0; nb < kC / 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[nb][e] = 0.0f;
#pragma unroll
    for (int nb = 0; nb < kVT / 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[nb][e] = 0.0f;
#pragma unroll 2
    for (int ks = 0; ks < KS; ++ks) {
        const int ao = (warp * 16 + (lane & 15)) * P + ks * 16 + (lane >> 4) * 8;
        uint32_t ah[4], al[4], b[4];
        ldmatrix_x4(ah, qh + ao);
        if (ROT) ldmatrix_x4(al, ql + ao);
        // scores against the keys of the chunk (only the blocks at or before this warp's rows)
#pragma unroll
        for (int n2 = 0; n2 < kC / 16; ++n2) {
            if (n2 > warp) break;
            const int bo = (n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * P + ks * 16 + ((lane >> 3) & 1) * 8;
            ldmatrix_x4(b, kh + bo);
            mma_bf16(sc[2 * n2], ah, b[0], b[1]);
            mma_bf16(sc[2 * n2 + 1], ah, b[2], b[3]);
            if (ROT) {
                mma_bf16(sc[2 * n2], al, b[0], b[1]);
                mma_bf16(sc[2 * n2 + 1], al, b[2], b[3]);
                ldmatrix_x4(b, kl + bo);
                mma_bf16(sc[2 * n2], ah, b[0], b[1]);
                mma_bf16(sc[2 * n2 + 1], ah, b[2], b[3]);
            }
        }
        // q S_in
#pragma unroll
        for (int d2 = 0; d2 < kVT / 16; ++d2) {
            const int bo = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8;
            ldmatrix_x4_trans(b, sh + bo);
            mma_bf16(o[2 * d2], ah, b[0], b[1]);
            mma_bf16(o[2 * d2 + 1], ah, b[2], b[3]);
            if (ROT) {
                mma_bf16(o[2 * d2], al, b[0], b[1]);
                mma_bf16(o[2 * d2 + 1], al, b[2], b[3]);
            }
            ldmatrix_x4_trans(b, sl + bo);
            mma_bf16(o[2 * d2], ah, b[0], b[1]);
            mma_bf16(o[2 * d2 + 1], ah, b[2], b[3]);
        }
    }
    const float pa = pw[ra + 1], pb = pw[rb + 1];
#pragma unroll
    for (int nb = 0; nb < kVT / 8; ++nb) { o[nb][0] *= pa; o[nb][1] *= pa; o[nb][2] *= pb; o[nb][3] *= pb; }
#pragma unroll
    for (int nb = 0; nb < kC / 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (e >> 1) ? rb : ra, j = nb * 8 + 2 * tq + (e & 1);
            sc[nb][e] = j <= i ? sc[nb][e] * (pw[i - j] * sscale) : 0.0f;
        }
#pragma unroll
    for (int j = 0; j < kC / 16; ++j) {
        if (j > warp) break;
        uint32_t ph[4], pl[4], b[4];
        split_bf16x2(sc[2 * j][0], sc[2 * j][1], ph[0], pl[0]);
        split_bf16x2(sc[2 * j][2], sc[2 * j][3], ph[1], pl[1]);
        split_bf16x2(sc[2 * j + 1][0], sc[2 * j + 1][1], ph[2], pl[2]);
        split_bf16x2(sc[2 * j + 1][2], sc[2 * j + 1][3], ph[3], pl[3]);
#pragma unroll
        for (int d2 = 0; d2 < kVT / 16; ++d2) {
            ldmatrix_x4_trans(b, vh + (j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8);
            mma_bf16(o[2 * d2], ph, b[0], b[1]);
            mma_bf16(o[2 * d2 + 1], ph, b[2], b[3]);
            mma_bf16(o[2 * d2], pl, b[0], b[1]);
            mma_bf16(o[2 * d2 + 1], pl, b[2], b[3]);
        }
    }
    const size_t ldo = (size_t)a.heads * a.dv;
#pragma unroll
    for (int nb = 0; nb < kVT / 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (e >> 1) ? rb : ra, j = v0 + nb * 8 + 2 * tq + (e & 1);
            if (i < c.n && j < a.dv) a.out[(size_t)(c.t0 + i) * ldo + (size_t)h * a.dv + j] = o[nb][e];
        }
}

template <int DK, bool ROT>
int run_chunked(cudaStream_t stream, const LinearAttnArgs& a) {
    constexpr int P = DK + 8, PV = kVT + 8;
    const int chunks = (a.T + kC - 1) / kC, vt = (a.dv + kVT - 1) / kVT;
    const dim3 grid(chunks, a.heads, vt);
    const size_t s1 = ((size_t)(ROT ? 2 : 1) * kC * P + 2 * kC * PV) * 2, s3 = ((size_t)(ROT ? 4 : 2) * kC * P + (size_t)kC * PV + 2 * (size_t)DK * PV) * 2;
    cudaError_t e = allow_all_dynamic_smem(linear_chunk_states_kernel<DK, ROT>);
    if (e == cudaSuccess) e = allow_all_dynamic_smem(linear_chunk_outputs_kernel<DK, ROT>);
    if (e == cudaSuccess) e = launch(linear_chunk_states_kernel<DK, ROT>, grid, dim3(kCThreads), s1, stream, true, a);
    const size_t total = (size_t)a.heads * a.dk * a.dv;
    if (e == cudaSuccess) e = launch(linear_chunk_scan_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, true, a);
    if (e == cudaSuccess) e = launch(linear_chunk_outputs_kernel<DK, ROT>, grid, dim3(kCThreads), s3, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "linear attention (chunked): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

template <bool F32>
int run_recurrent(cudaStream_t stream, const LinearAttnArgs& a) {
    const int rp = (a.dk + 31) / 32;
    auto k = rp <= 1 ? linear_recurrent_kernel<F32, 1> : rp <= 2 ? linear_recurrent_kernel<F32, 2> : rp <= 4 ? linear_recurrent_kernel<F32, 4>
           : rp <= 8 ? linear_recurrent_kernel<F32, 8> : linear_recurrent_kernel<F32, 16>;
    cudaError_t e = launch(k, dim3(a.heads, (a.dv + 31) / 32), dim3(256), (size_t)(2 * a.dk + 256) * 4, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "linear attention (recurrent): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace

size_t linear_attention_scratch_floats(int T, int heads, int dk, int dv) { return (size_t)((T + kC - 1) / kC) * heads * dk * dv; }

int linear_attention_recurrent(cudaStream_t stream, const LinearAttnArgs& a) {
    if (a.dk > 512) return fail(KMLL_ERR_UNSUPPORTED, "linear attention: key size %d above 512", a.dk);
    return a.in_f32 ? run_recurrent<true>(stream, a) : run_recurrent<false>(stream, a);
}

bool linear_attention_chunked_ok(const LinearAttnArgs& a) { return !a.in_f32 && a.dk <= 256; }

int linear_attention_chunked(cudaStream_t stream, const LinearAttnArgs& a) {
    if (!linear_attention_chunked_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "linear attention: no chunked form for key size %d", a.dk);
    const bool rot = a.rot > 0;
    if (a.dk <= 32) return rot ? run_chunked<32, true>(stream, a) : run_chunked<32, false>(stream, a);
    if (a.dk <= 64) return rot ? run_chunked<64, true>(stream, a) : run_chunked<64, false>(stream, a);
    if (a.dk <= 128) return rot ? run_chunked<128, true>(stream, a) : run_chunked<128, false>(stream, a);
    return rot ? run_chunked<256, true>(stream, a) : run_chunked<256, false>(stream, a);
}

}  // namespace kmll
