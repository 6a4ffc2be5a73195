// Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, no softmax and no denominator.
//
//   recurrent form  token after token in f32 with the state in registers: decode steps, and prompts of decoders that compute
//                   in f32
//   chunked form    prompts in bf16: chunks of 64 tokens on the tensor cores (three launches)
//
// Rotated q and k, decays, scaled keys and the state are f32 throughout; where they meet the tensor cores they are split into
// a bf16 head and a bf16 remainder (16 mantissa bits, products exact, f32 accumulation).
#include <cstring>

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
            a.out[(size_t)t * a.ldo + (size_t)h * a.dv + c] = sum;
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
// Chunks of 128 tokens in blocks of 64, value tiles of VT columns, keys in slices of 64 entries.  With n tokens in the chunk and
// S_in the state ahead of it:
//   prepare  rotated (and, when sizes are not multiples of 8, padded) q and k as bf16 head / remainder planes
//   states   KV = sum_j decay^(n-1-j) k_j v_j^T                     one block per (chunk, head, key slice, value tile)
//   scan     S_in of every chunk as head / remainder planes, and the state behind the last      elementwise
//   outputs  o_i = decay^(i+1) q_i S_in + sum_{j<=i} decay^(i-j) (q_i . k_j) v_j               one block per (64 rows, head, tile)
// Without rotation q, k and v are used as the projection wrote them (bf16, exact); the scale of the keys then goes on the scores
// and on the decay weights instead.
constexpr int kC = kLinChunk, kB = 64, kCThreads = 128, kPS = 64 + 8;  // kPS: pitch of a tile with 64 columns

struct ChunkArgs {
    const uint16_t *qh, *ql, *kh, *kl, *v;  // rows of ldq / ldv elements, heads hq / hv apart; ql, kl null: exact
    int ldq, hq, ldv, hv;
    int T, heads, dk, dv, dvp, chunks, ldo;
    float key_scale;                        // still to be applied (1 once it is in the planes)
    const float* powers;
    float* state;
    float* kv;                              // [chunks][heads][dk][dv]
    uint16_t *sh, *sl;                      // [chunks][heads][dk][dvp]
    float* out;
};

__device__ inline uint32_t sm32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ inline void copy_wait() {
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
}
// tile [64][cols] <- rows r0 .. of src (pitch ld, from column c0), zero beyond `rows` rows and `lim` columns (multiples of 8)
template <int COLS>
__device__ inline void copy_tile(uint16_t* tile, const uint16_t* src, size_t ld, int rows, int c0, int lim) {
    constexpr int RUNS = COLS / 8, P = COLS + 8;
    for (int i = threadIdx.x; i < kB * RUNS; i += kCThreads) {
        const int r = i / RUNS, c = (i - r * RUNS) * 8;
        const bool live = r < rows && c0 + c < lim;
        cp_async16_zfill_to(sm32(tile + r * P + c), live ? src + (size_t)r * ld + c0 + c : src, live ? 16u : 0u);
    }
}

// eight consecutive bf16 values as f32; entries at or beyond n are zeros
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
__device__ inline void store_split8(uint16_t* hi, uint16_t* lo, const float (&v)[8]) {
    uint4 h, l;
    split_bf16x2(v[0], v[1], h.x, l.x);
    split_bf16x2(v[2], v[3], h.y, l.y);
    split_bf16x2(v[4], v[5], h.z, l.z);
    split_bf16x2(v[6], v[7], h.w, l.w);
    *reinterpret_cast<uint4*>(hi) = h;
    if (lo != nullptr) *reinterpret_cast<uint4*>(lo) = l;
}

// planes of q, k (and v, when `vout` is given): one thread per run of eight entries
__global__ void __launch_bounds__(256) linear_prepare_kernel(const LinearAttnArgs a, uint16_t* qh, uint16_t* ql, uint16_t* kh, uint16_t* kl, uint16_t* vout, int dkp,
                                                             int dvp) {
    pdl_wait();
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const int rq = dkp / 8, rv = vout != nullptr ? dvp / 8 : 0, per = a.heads * (2 * rq + rv);
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long long)a.T * per) return;
    const int t = (int)(i / per);
    int j = (int)(i - (long long)t * per);
    const uint16_t* row = in + (size_t)t * a.ld;
    const bool al = ((a.ld | a.q_off | a.k_off | a.v_off | a.dk | a.dv) & 7) == 0;
    float v[8];
    if (j >= a.heads * 2 * rq) {
        j -= a.heads * 2 * rq;
        const int h = j / rv, r = (j - h * rv) * 8;
        load8(row + a.v_off + (size_t)h * a.dv, r, a.dv, al, v);
        store_split8(vout + ((size_t)t * a.heads + h) * dvp + r, nullptr, v);
        return;
    }
    const bool is_k = j >= a.heads * rq;
    if (is_k) j -= a.heads * rq;
    const int h = j / rq, r = (j - h * rq) * 8, half = a.rot >> 1;
    const uint16_t* p = row + (is_k ? a.k_off : a.q_off) + (size_t)h * a.dk;
    if (r >= a.rot) {
        load8(p, r, a.dk, al, v);
    } else {
        const float2* cs = a.table + (size_t)((a.at != nullptr ? a.at->position : a.pos0) + t) * half;
        if (al && (half & 7) == 0) {  // the run and its partner run lie in one half each
            float w[8];
            const bool low = r < half;
            load8(p, r, a.dk, true, v);
            load8(p, low ? r + half : r - half, a.dk, true, w);
            const float4* c4 = reinterpret_cast<const float4*>(cs + (low ? r : r - half));
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float4 f = c4[e];
                v[2 * e] = low ? v[2 * e] * f.x - w[2 * e] * f.y : v[2 * e] * f.x + w[2 * e] * f.y;
                v[2 * e + 1] = low ? v[2 * e + 1] * f.z - w[2 * e + 1] * f.w : v[2 * e + 1] * f.z + w[2 * e + 1] * f.w;
            }
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = r + e < a.dk ? rotated_at<false>(p, 0, r + e, a.rot, cs) : 0.0f;
        }
    }
    if (is_k)
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= a.key_scale;
    const size_t at = ((size_t)t * a.heads + h) * dkp + r;
    store_split8((is_k ? kh : qh) + at, (is_k ? kl : ql) + at, v);
}

template <int VT, bool LO>
__global__ void __launch_bounds__(kCThreads) linear_chunk_states_kernel(const ChunkArgs a) {
    constexpr int PV = VT + 8;
    extern __shared__ __align__(16) uint16_t csm[];
    uint16_t* const vh = csm;
    uint16_t* const vl = vh + kB * PV;
    uint16_t* const kh = vl + kB * PV;
    uint16_t* const kl = kh + kB * kPS;  // LO only
    const int ndv = (a.dv + VT - 1) / VT;
    const int c = blockIdx.x, h = blockIdx.y, k0 = (blockIdx.z / ndv) * 64, v0 = (blockIdx.z % ndv) * VT;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int n = min(kC, a.T - c * kC);
    const float* pw = a.powers + (size_t)h * (kC + 1);
    float acc[VT / 8][4];
#pragma unroll
    for (int i = 0; i < VT / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.0f;
    pdl_wait();
    for (int b = 0; b < n; b += kB) {
        const int t0 = c * kC + b, rows = min(kB, n - b);
        if (b > 0) __syncthreads();
        copy_tile<64>(kh, a.kh + (size_t)t0 * a.ldq + (size_t)h * a.hq, a.ldq, rows, k0, a.hq);
        if (LO) copy_tile<64>(kl, a.kl + (size_t)t0 * a.ldq + (size_t)h * a.hq, a.ldq, rows, k0, a.hq);
        for (int i = tid; i < kB * (VT / 8); i += kCThreads) {
            const int t = i / (VT / 8), r = (i % (VT / 8)) * 8;
            float v[8] = {};
            if (t < rows && v0 + r < a.hv) {
                load8(a.v + (size_t)(t0 + t) * a.ldv + (size_t)h * a.hv, v0 + r, a.hv, true, v);
                const float w = pw[n - 1 - b - t] * a.key_scale;
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] *= w;
            }
            store_split8(vh + t * PV + r, vl + t * PV + r, v);
        }
        copy_wait();
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < kB / 16; ++ks) {
            const int ao = (ks * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * kPS + warp * 16 + ((lane >> 3) & 1) * 8;
            uint32_t ah[4], al[4], x[4];
            ldmatrix_x4_trans(ah, kh + ao);
            if (LO) ldmatrix_x4_trans(al, kl + ao);
#pragma unroll
            for (int d2 = 0; d2 < VT / 16; ++d2) {
                const int bo = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8;
                ldmatrix_x4_trans(x, vh + bo);
                mma_bf16(acc[2 * d2], ah, x[0], x[1]);
                mma_bf16(acc[2 * d2 + 1], ah, x[2], x[3]);
                if (LO) {
                    mma_bf16(acc[2 * d2], al, x[0], x[1]);
                    mma_bf16(acc[2 * d2 + 1], al, x[2], x[3]);
                }
                ldmatrix_x4_trans(x, vl + bo);
                mma_bf16(acc[2 * d2], ah, x[0], x[1]);
                mma_bf16(acc[2 * d2 + 1], ah, x[2], x[3]);
            }
        }
    }
    float* const KV = a.kv + ((size_t)c * a.heads + h) * a.dk * a.dv;
    const bool v2 = (a.dv & 1) == 0;
#pragma unroll
    for (int i = 0; i < VT / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int d = k0 + warp * 16 + g + (e >> 1) * 8, j = v0 + i * 8 + 2 * tq;
            if (d < a.dk && j < a.dv) {
                float* p = KV + (size_t)d * a.dv + j;
                if (v2) {
                    *reinterpret_cast<float2*>(p) = make_float2(acc[i][e], acc[i][e + 1]);
                } else {
                    p[0] = acc[i][e];
                    if (j + 1 < a.dv) p[1] = acc[i][e + 1];
                }
            }
        }
}

// one thread per pair of state columns (dvp is even; the padding columns become zeros)
__global__ void __launch_bounds__(256) linear_chunk_scan_kernel(const ChunkArgs a) {
    pdl_wait();
    const int half = a.dvp >> 1;
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x, rows = (size_t)a.heads * a.dk;
    if (i >= rows * half) return;
    const size_t row = i / half;
    const int j = (int)(i - row * half) * 2;
    const float* pw = a.powers + (row / a.dk) * (kC + 1);
    const bool l0 = j < a.dv, l1 = j + 1 < a.dv, v2 = (a.dv & 1) == 0 && l0;
    const size_t at = row * a.dv + j, plane = row * a.dvp + j, kv_step = rows * a.dv, s_step = rows * a.dvp;
    float s0 = l0 ? a.state[at] : 0.0f, s1 = l1 ? a.state[at + 1] : 0.0f;
    const float full = pw[kC];
    for (int c0 = 0; c0 < a.chunks; c0 += 8) {
        float2 kv[8];
#pragma unroll
        for (int q = 0; q < 8; ++q) {
            kv[q] = make_float2(0.0f, 0.0f);
            if (c0 + q < a.chunks) {
                const float* p = a.kv + (size_t)(c0 + q) * kv_step + at;
                if (v2) kv[q] = *reinterpret_cast<const float2*>(p);
                else if (l0) kv[q] = make_float2(p[0], l1 ? p[1] : 0.0f);
            }
        }
#pragma unroll
        for (int q = 0; q < 8; ++q) {
            const int c = c0 + q;
            if (c >= a.chunks) break;
            uint32_t hi, lo;
            split_bf16x2(s0, s1, hi, lo);
            *reinterpret_cast<uint32_t*>(a.sh + (size_t)c * s_step + plane) = hi;
            *reinterpret_cast<uint32_t*>(a.sl + (size_t)c * s_step + plane) = lo;
            const float f = c + 1 < a.chunks ? full : pw[a.T - c * kC];
            s0 = fmaf(f, s0, kv[q].x);
            s1 = fmaf(f, s1, kv[q].y);
        }
    }
    if (l0) a.state[at] = s0;
    if (l1) a.state[at + 1] = s1;
}

template <int VT, bool LO>
__global__ void __launch_bounds__(kCThreads) linear_chunk_outputs_kernel(const ChunkArgs a) {
    constexpr int PV = VT + 8;
    extern __shared__ __align__(16) uint16_t csm[];
    uint16_t* const sh = csm;               // [64][PV] slice of S_in ...
    uint16_t* const sl = sh + kB * PV;
    uint16_t* const kh = csm;               // ... or, later, [64][72] slice of the keys, and behind it the values
    uint16_t* const kl = kh + kB * kPS;
    uint16_t* const vt = sl + kB * PV;      // [64][PV]
    uint16_t* const qh = vt + kB * PV;
    uint16_t* const ql = qh + kB * kPS;     // LO only
    __shared__ float pw[kC + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int rb = (int)gridDim.x - 1 - (int)blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT;
    const int c = rb / (kC / kB), sub = rb % (kC / kB), t0 = rb * kB, rows = min(kB, a.T - t0);
    const int ra = warp * 16 + g, rbw = ra + 8;  // this lane's two rows within the block
    const int ao0 = (warp * 16 + (lane & 15)) * kPS + (lane >> 4) * 8;
    pdl_wait();
    for (int i = tid; i <= kC; i += kCThreads) pw[i] = a.powers[(size_t)h * (kC + 1) + i];
    const uint16_t* Qh = a.qh + (size_t)t0 * a.ldq + (size_t)h * a.hq;
    const uint16_t* Ql = LO ? a.ql + (size_t)t0 * a.ldq + (size_t)h * a.hq : nullptr;
    float o[VT / 8][4];
#pragma unroll
    for (int i = 0; i < VT / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
    // ---- q S_in
    const size_t S0 = ((size_t)c * a.heads + h) * a.dk * a.dvp;
    for (int k0 = 0; k0 < a.dk; k0 += 64) {
        __syncthreads();
        copy_tile<64>(qh, Qh, a.ldq, rows, k0, a.hq);
        if (LO) copy_tile<64>(ql, Ql, a.ldq, rows, k0, a.hq);
        copy_tile<VT>(sh, a.sh + S0 + (size_t)k0 * a.dvp, a.dvp, a.dk - k0, v0, a.dvp);
        copy_tile<VT>(sl, a.sl + S0 + (size_t)k0 * a.dvp, a.dvp, a.dk - k0, v0, a.dvp);
        copy_wait();
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            if (k0 + ks * 16 >= a.dk) break;
            uint32_t ah[4], al[4], x[4];
            ldmatrix_x4(ah, qh + ao0 + ks * 16);
            if (LO) ldmatrix_x4(al, ql + ao0 + ks * 16);
#pragma unroll
            for (int d2 = 0; d2 < VT / 16; ++d2) {
                const int bo = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8;
                ldmatrix_x4_trans(x, sh + bo);
                mma_bf16(o[2 * d2], ah, x[0], x[1]);
                mma_bf16(o[2 * d2 + 1], ah, x[2], x[3]);
                if (LO) {
                    mma_bf16(o[2 * d2], al, x[0], x[1]);
                    mma_bf16(o[2 * d2 + 1], al, x[2], x[3]);
                }
                ldmatrix_x4_trans(x, sl + bo);
                mma_bf16(o[2 * d2], ah, x[0], x[1]);
                mma_bf16(o[2 * d2 + 1], ah, x[2], x[3]);
            }
        }
    }
    {
        const float pa = pw[sub * kB + ra + 1], pb = pw[sub * kB + rbw + 1];
#pragma unroll
        for (int i = 0; i < VT / 8; ++i) { o[i][0] *= pa; o[i][1] *= pa; o[i][2] *= pb; o[i][3] *= pb; }
    }
    // ---- the tokens of the chunk, 64 at a time
    const bool one_slice = a.dk <= 64;  // q of the loop above is still in place
    for (int kb = 0; kb <= sub; ++kb) {
        const int j0 = c * kC + kb * kB, jrows = min(kB, a.T - j0);
        const bool diag = kb == sub;
        float sc[kB / 8][4];
#pragma unroll
        for (int i = 0; i < kB / 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[i][e] = 0.0f;
        for (int k0 = 0; k0 < a.dk; k0 += 64) {
            __syncthreads();
            if (!one_slice) {
                copy_tile<64>(qh, Qh, a.ldq, rows, k0, a.hq);
                if (LO) copy_tile<64>(ql, Ql, a.ldq, rows, k0, a.hq);
            }
            copy_tile<64>(kh, a.kh + (size_t)j0 * a.ldq + (size_t)h * a.hq, a.ldq, jrows, k0, a.hq);
            if (LO) copy_tile<64>(kl, a.kl + (size_t)j0 * a.ldq + (size_t)h * a.hq, a.ldq, jrows, k0, a.hq);
            if (k0 == 0) copy_tile<VT>(vt, a.v + (size_t)j0 * a.ldv + (size_t)h * a.hv, a.ldv, jrows, v0, a.hv);
            copy_wait();
            __syncthreads();
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                if (k0 + ks * 16 >= a.dk) break;
                uint32_t ah[4], al[4], x[4];
                ldmatrix_x4(ah, qh + ao0 + ks * 16);
                if (LO) ldmatrix_x4(al, ql + ao0 + ks * 16);
#pragma unroll
                for (int n2 = 0; n2 < kB / 16; ++n2) {
                    if (diag && n2 > warp) break;  // keys behind every row of this warp
                    const int bo = (n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * kPS + ks * 16 + ((lane >> 3) & 1) * 8;
                    ldmatrix_x4(x, kh + bo);
                    mma_bf16(sc[2 * n2], ah, x[0], x[1]);
                    mma_bf16(sc[2 * n2 + 1], ah, x[2], x[3]);
                    if (LO) {
                        mma_bf16(sc[2 * n2], al, x[0], x[1]);
                        mma_bf16(sc[2 * n2 + 1], al, x[2], x[3]);
                        ldmatrix_x4(x, kl + bo);
                        mma_bf16(sc[2 * n2], ah, x[0], x[1]);
                        mma_bf16(sc[2 * n2 + 1], ah, x[2], x[3]);
                    }
                }
            }
        }
        const int shift = (sub - kb) * kB;
#pragma unroll
        for (int i = 0; i < kB / 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = shift + ((e >> 1) ? rbw : ra) - (i * 8 + 2 * tq + (e & 1));
                sc[i][e] = d >= 0 ? sc[i][e] * (pw[d] * a.key_scale) : 0.0f;
            }
#pragma unroll
        for (int j = 0; j < kB / 16; ++j) {
            if (diag && j > warp) break;
            uint32_t ph[4], pl[4], x[4];
            split_bf16x2(sc[2 * j][0], sc[2 * j][1], ph[0], pl[0]);
            split_bf16x2(sc[2 * j][2], sc[2 * j][3], ph[1], pl[1]);
            split_bf16x2(sc[2 * j + 1][0], sc[2 * j + 1][1], ph[2], pl[2]);
            split_bf16x2(sc[2 * j + 1][2], sc[2 * j + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int d2 = 0; d2 < VT / 16; ++d2) {
                ldmatrix_x4_trans(x, vt + (j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8);
                mma_bf16(o[2 * d2], ph, x[0], x[1]);
                mma_bf16(o[2 * d2 + 1], ph, x[2], x[3]);
                mma_bf16(o[2 * d2], pl, x[0], x[1]);
                mma_bf16(o[2 * d2 + 1], pl, x[2], x[3]);
            }
        }
    }
    const size_t ldo = (size_t)a.ldo;
    const bool v2 = ((a.dv | a.ldo) & 1) == 0;
#pragma unroll
    for (int i = 0; i < VT / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int r = (e >> 1) ? rbw : ra, j = v0 + i * 8 + 2 * tq;
            if (r < rows && j < a.dv) {
                float* p = a.out + (size_t)(t0 + r) * ldo + (size_t)h * a.dv + j;
                if (v2) {
                    *reinterpret_cast<float2*>(p) = make_float2(o[i][e], o[i][e + 1]);
                } else {
                    p[0] = o[i][e];
                    if (j + 1 < a.dv) p[1] = o[i][e + 1];
                }
            }
        }
}

inline int pad8(int v) { return (v + 7) & ~7; }
// areas of the scratch buffer, in floats (every area starts on a 16-byte boundary)
struct ChunkScratch {
    size_t kv, s_plane, qk_plane, v_plane, total;
};
ChunkScratch chunk_scratch(int T, int heads, int dk, int dv) {
    ChunkScratch c;
    const size_t chunks = (size_t)((T + kC - 1) / kC);
    auto up4 = [](size_t v) { return (v + 3) & ~(size_t)3; };
    c.kv = up4(chunks * heads * dk * dv);
    c.s_plane = up4(chunks * heads * dk * pad8(dv) / 2);
    c.qk_plane = up4((size_t)T * heads * pad8(dk) / 2);
    c.v_plane = up4((size_t)T * heads * pad8(dv) / 2);
    c.total = c.kv + 2 * c.s_plane + 4 * c.qk_plane + c.v_plane;
    return c;
}

template <int VT, bool LO>
int run_chunked(cudaStream_t stream, const ChunkArgs& a) {
    constexpr int PV = VT + 8;
    const int ndk = (a.dk + 63) / 64, ndv = (a.dv + VT - 1) / VT;
    const size_t s1 = ((size_t)2 * kB * PV + (size_t)(LO ? 2 : 1) * kB * kPS) * 2, s3 = ((size_t)3 * kB * PV + (size_t)(LO ? 2 : 1) * kB * kPS) * 2;
    cudaError_t e = allow_all_dynamic_smem(linear_chunk_states_kernel<VT, LO>);
    if (e == cudaSuccess) e = allow_all_dynamic_smem(linear_chunk_outputs_kernel<VT, LO>);
    if (e == cudaSuccess) e = launch(linear_chunk_states_kernel<VT, LO>, dim3(a.chunks, a.heads, ndk * ndv), dim3(kCThreads), s1, stream, true, a);
    const size_t pairs = (size_t)a.heads * a.dk * (a.dvp / 2);
    if (e == cudaSuccess) e = launch(linear_chunk_scan_kernel, dim3((unsigned)((pairs + 255) / 256)), dim3(256), 0, stream, true, a);
    if (e == cudaSuccess) e = launch(linear_chunk_outputs_kernel<VT, LO>, dim3((a.T + kB - 1) / kB, a.heads, ndv), dim3(kCThreads), s3, stream, true, a);
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

size_t linear_attention_scratch_floats(int T, int heads, int dk, int dv) { return chunk_scratch(T, heads, dk, dv).total; }

int linear_attention_recurrent(cudaStream_t stream, const LinearAttnArgs& a) {
    if (a.dk > 512) return fail(KMLL_ERR_UNSUPPORTED, "linear attention: key size %d above 512", a.dk);
    return a.in_f32 ? run_recurrent<true>(stream, a) : run_recurrent<false>(stream, a);
}

bool linear_attention_chunked_ok(const LinearAttnArgs& a) { return !a.in_f32; }

int linear_attention_chunked(cudaStream_t stream, const LinearAttnArgs& a) {
    if (a.in_f32) return fail(KMLL_ERR_UNSUPPORTED, "linear attention: the chunked form takes bf16 q, k and v");
    const ChunkScratch m = chunk_scratch(a.T, a.heads, a.dk, a.dv);
    const int dkp = pad8(a.dk), dvp = pad8(a.dv);
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const bool aligned = ((a.ld | a.q_off | a.k_off | a.v_off | a.dk | a.dv) & 7) == 0 && (reinterpret_cast<uintptr_t>(a.in) & 15u) == 0;
    const bool planes = a.rot > 0 || !aligned;
    ChunkArgs c;
    memset(&c, 0, sizeof(c));
    c.T = a.T; c.heads = a.heads; c.dk = a.dk; c.dv = a.dv; c.dvp = dvp; c.chunks = (a.T + kC - 1) / kC;
    c.powers = a.powers; c.state = a.state; c.out = a.out; c.ldo = a.ldo;
    float* f = a.scratch;
    c.kv = f;
    c.sh = reinterpret_cast<uint16_t*>(f + m.kv);
    c.sl = reinterpret_cast<uint16_t*>(f + m.kv + m.s_plane);
    f += m.kv + 2 * m.s_plane;
    if (planes) {
        uint16_t* pl[4];
        for (int i = 0; i < 4; ++i) pl[i] = reinterpret_cast<uint16_t*>(f + (size_t)i * m.qk_plane);
        uint16_t* v = aligned ? nullptr : reinterpret_cast<uint16_t*>(f + 4 * m.qk_plane);
        const long long items = (long long)a.T * a.heads * (2 * (dkp / 8) + (v != nullptr ? dvp / 8 : 0));
        cudaError_t e = launch(linear_prepare_kernel, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, stream, true, a, pl[0], pl[1], pl[2], pl[3], v, dkp, dvp);
        if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "linear attention (prepare): %s", cudaGetErrorString(e));
        c.qh = pl[0]; c.ql = pl[1]; c.kh = pl[2]; c.kl = pl[3];
        c.ldq = a.heads * dkp; c.hq = dkp;
        c.v = v != nullptr ? v : in + a.v_off;
        c.ldv = v != nullptr ? a.heads * dvp : a.ld;
        c.hv = dvp;
        c.key_scale = 1.0f;
        return a.dv <= 64 ? run_chunked<64, true>(stream, c) : run_chunked<128, true>(stream, c);
    }
    c.qh = in + a.q_off; c.kh = in + a.k_off; c.v = in + a.v_off;
    c.ldq = c.ldv = a.ld; c.hq = a.dk; c.hv = a.dv;
    c.key_scale = a.key_scale;
    return a.dv <= 64 ? run_chunked<64, false>(stream, c) : run_chunked<128, false>(stream, c);
}

}  // namespace kmll
