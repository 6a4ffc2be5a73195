// Linear attention whose decay depends on the token, one value per key channel (optionally with the delta rule):
//   S <- diag(alpha) S + k u^T,  o = S^T q;   u = v, or beta (v - (diag(alpha) S)^T k)
//
//   step form     token after token in f32 with the state in registers; everything between the projections and the recurrence
//                 (short convolutions, unit vectors, decays, write strengths, the low-rank gate) happens in the same launch:
//                 decode steps, prompts of decoders that compute in f32, short portions, sizes the chunked form lacks
//   chunked form  prompts in bf16, chunks of 64 tokens on the tensor cores: one launch prepares every chunk on its own, a second
//                 carries the state through the chunks and writes the outputs
//
// With G the running sum of log2 alpha inside a chunk and S_in the state ahead of it,
//   o_i = (q_i 2^G_i) S_in + sum_{j <= i} A_ij u_j           A_ij = sum_d q_id k_jd 2^(G_id - G_jd)
//   S_out = diag(2^G_n) S_in + sum_j (k_j 2^(G_n - G_j)) u_j^T
// and for the delta rule (I + L) U = beta (V - (K 2^G) S_in) with L_ij = beta_i sum_d k_id k_jd 2^(G_id - G_jd), j < i; so with
// X = (I + L)^-1 each chunk's U = X beta V - W S_in, W = X beta (K 2^G).  Every exponent that is evaluated is a sum of log decays
// over consecutive tokens, hence not positive: blocks of 16 x 16 tokens below the diagonal factor through the row ahead of the
// block, blocks on the diagonal are summed directly.
#include "activations.cuh"
#include "mma_bf16.cuh"

namespace kmll {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

template <bool F32>
__device__ inline float in_at(const void* p, size_t i) {
    return F32 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
__host__ __device__ inline int round_to(int v, int m) { return (v + m - 1) / m * m; }

// log2 of the decay
__device__ inline float log2_decay(const GatedLinearArgs& a, float z, float rate) {
    const float l = a.decay == KMLL_DECAY_LOGISTIC ? -softplus(-z) * a.inv_tau : -rate * softplus(z);
    return fmaxf(l * kLog2e, -150.0f);  // (2^-150 is zero in f32)
}
__device__ inline float decay_rate(const GatedLinearArgs& a, int h) { return a.decay == KMLL_DECAY_SOFTPLUS ? expf(bf16_bits_to_f32(a.a_log[h])) : 0.0f; }

// Input of channel `ch` (column `col` of the projection) `back` tokens before token t of this call (at position pos): from the
// rows of the call, from the ring of earlier positions, or zero before the sequence.
template <bool F32>
__device__ inline float earlier(const GatedLinearArgs& a, int t, int pos, int back, int col, int ch, int channels) {
    if (back <= t) return in_at<F32>(a.in, (size_t)(t - back) * a.ld + col);
    return back <= pos ? a.ring[(size_t)((pos - back) % a.taps) * channels + ch] : 0.0f;
}
// channel through its convolution and SiLU (taps > 0)
template <bool F32>
__device__ inline float convolved(const GatedLinearArgs& a, int t, int pos, int col, int ch, int channels) {
    if (a.taps == 0) return in_at<F32>(a.in, (size_t)t * a.ld + col);
    const uint16_t* w = a.conv + (size_t)ch * a.taps;
    float y = 0.0f;
    for (int j = 0; j < a.taps; ++j) y = fmaf(bf16_bits_to_f32(w[j]), earlier<F32>(a, t, pos, a.taps - 1 - j, col, ch, channels), y);
    return act_silu(y);
}
// dot product of a bf16 row of n (a multiple of 8, 16-byte aligned) with f32 values
__device__ inline float dot_row(const uint16_t* w, const float* x, int n) {
    float s = 0.0f;
    for (int r = 0; r < n; r += 8) {
        const uint4 t = *reinterpret_cast<const uint4*>(w + r);
        const uint32_t ww[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            s = fmaf(__uint_as_float(ww[e] << 16), x[r + 2 * e], s);
            s = fmaf(__uint_as_float(ww[e] & 0xffff0000u), x[r + 2 * e + 1], s);
        }
    }
    return s;
}

// ---- step form ------------------------------------------------------------------------------------------------------------------
// Block (head, 32 value columns): four warps of eight columns; lane (row lane, column quad) keeps rows rl, rl + 16, .. of four
// columns in registers for the whole call, so the sums over keys stay inside a warp.
constexpr int kSThreads = 128, kSCols = 32;

template <bool F32, int RP>
__global__ void __launch_bounds__(kSThreads) gated_step_kernel(const GatedLinearArgs a) {
    extern __shared__ __align__(16) float ssm[];  // q | k | decay, [dk] each | v [32] | a [rank] | g [gate_rank], padded
    const int dkr = round_to(a.dk, 4), rank8 = round_to(a.rank, 8), gate8 = round_to(a.gate_rank, 8);
    float* const sq = ssm;
    float* const sk = sq + dkr;
    float* const sg = sk + dkr;
    float* const sv = sg + dkr;
    float* const sa = sv + kSCols;
    float* const sgr = sa + rank8;
    __shared__ float dots[4];  // q.q, k.k, q.k, beta
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane & 15;
    const int col0 = blockIdx.y * kSCols, lc = warp * 8 + (lane >> 4) * 4, c0 = col0 + lc;
    const int per = a.heads / a.kv_heads, hq = h / per, nq = a.kv_heads * a.dk, channels = 2 * nq + a.heads * a.dv;
    float* const S = a.state + (size_t)h * a.dk * a.dv;
    const bool vec = (a.dv & 3) == 0;
    float s[RP][4];
#pragma unroll
    for (int r = 0; r < RP; ++r) {  // (the state's last writer lies more than one launch back)
        const int i = rl + r * 16;
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
    {   // weights never change: towards L2 ahead of the dependency wait
        const char* up = reinterpret_cast<const char*>(a.up + (size_t)h * a.dk * a.ldu);
        for (int i = tid * 128; i < a.dk * a.ldu * 2; i += kSThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(up + i));
        if (a.gate_rank > 0) {
            const int rows = min(kSCols, a.dv - col0);
            const char* gu = reinterpret_cast<const char*>(a.gate_up + (size_t)(h * a.dv + col0) * a.ldg);
            for (int i = tid * 128; i < rows * a.ldg * 2; i += kSThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(gu + i));
        }
    }
    const float rate = decay_rate(a, h);
    const int pos0 = a.at != nullptr ? a.at->position : a.pos0;  // (written more than one launch ago)
    pdl_wait();
    for (int t = 0; t < a.T; ++t) {
        const int pos = pos0 + t;
        const size_t row = (size_t)t * a.ld;
        // ---- q, k, v, and the inputs of the low-rank maps
        const int n_in = 2 * a.dk + kSCols;
        for (int i = tid; i < n_in + rank8 + gate8; i += kSThreads) {
            if (i < 2 * a.dk) {
                const int d = i < a.dk ? i : i - a.dk, ch = (i < a.dk ? 0 : nq) + hq * a.dk + d, col = (i < a.dk ? a.q_off : a.k_off) + hq * a.dk + d;
                const float y = convolved<F32>(a, t, pos, col, ch, channels);
                if (i < a.dk) sq[d] = y;
                else sk[d] = y;
                if (a.taps > 0 && a.T == 1 && blockIdx.y == 0 && h == hq * per) a.ring[(size_t)(pos % a.taps) * channels + ch] = in_at<F32>(a.in, row + col);
            } else if (i < n_in) {
                const int c = i - 2 * a.dk, ch = 2 * nq + h * a.dv + col0 + c, col = a.v_off + h * a.dv + col0 + c;
                float y = 0.0f;
                if (col0 + c < a.dv) {
                    y = convolved<F32>(a, t, pos, col, ch, channels);
                    if (a.taps > 0 && a.T == 1) a.ring[(size_t)(pos % a.taps) * channels + ch] = in_at<F32>(a.in, row + col);
                }
                sv[c] = y;
            } else if (i < n_in + rank8) {
                const int r = i - n_in;
                sa[r] = r < a.rank ? in_at<F32>(a.in, row + a.a_off + r) : 0.0f;
            } else {
                const int r = i - n_in - rank8;
                sgr[r] = r < a.gate_rank ? in_at<F32>(a.in, row + a.g_off + r) : 0.0f;
            }
        }
        __syncthreads();
        // ---- decays, norms of q and k, gate
        if (warp < 3) {
            const float* x = warp == 1 ? sk : sq;
            const float* y = warp == 0 ? sq : sk;
            float d = 0.0f;
            for (int i = lane; i < a.dk; i += 32) d = fmaf(x[i], y[i], d);
            d = warp_sum(d);
            if (lane == 0) dots[warp] = d;
        } else if (lane == 0) {
            dots[3] = a.delta ? act_sigmoid(in_at<F32>(a.in, row + a.b_off + h)) : 1.0f;
        }
        for (int d = tid; d < a.dk; d += kSThreads) {
            float z = dot_row(a.up + (size_t)(h * a.dk + d) * a.ldu, sa, rank8);
            if (a.bias != nullptr) z += bf16_bits_to_f32(a.bias[h * a.dk + d]);
            sg[d] = exp2f(log2_decay(a, z, rate));
        }
        if (a.gate_rank > 0) {
            const int c = tid >> 2, part = tid & 3;  // four lanes per column
            float g = 0.0f;
            if (col0 + c < a.dv)
                for (int r = part * 8; r < gate8; r += 32) g += dot_row(a.gate_up + (size_t)(h * a.dv + col0 + c) * a.ldg + r, sgr + r, 8);
            g += __shfl_xor_sync(0xffffffffu, g, 1);
            g += __shfl_xor_sync(0xffffffffu, g, 2);
            if (part == 0 && col0 + c < a.dv) a.gate[(size_t)t * a.heads * a.dv + (size_t)h * a.dv + col0 + c] = g;
        }
        __syncthreads();
        // ---- the recurrence
        float fq = a.q_scale, fk = 1.0f;
        if (a.unit_eps > 0.0f) {
            fq *= 1.0f / sqrtf(dots[0] + a.unit_eps);
            fk = 1.0f / sqrtf(dots[1] + a.unit_eps);
        }
        const float qk = dots[2] * fq * fk, beta = dots[3];
        float kv[4] = {}, qs[4] = {};
#pragma unroll
        for (int r = 0; r < RP; ++r) {
            const int i = rl + r * 16;
            if (i < a.dk) {
                const float g = sg[i], k = sk[i] * fk, q = sq[i] * fq;
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[r][e] *= g;
                    kv[e] = fmaf(k, s[r][e], kv[e]);
                    qs[e] = fmaf(q, s[r][e], qs[e]);
                }
            }
        }
#pragma unroll
        for (int off = 1; off < 16; off <<= 1)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                kv[e] += __shfl_xor_sync(0xffffffffu, kv[e], off);
                qs[e] += __shfl_xor_sync(0xffffffffu, qs[e], off);
            }
        float u[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) u[e] = a.delta ? beta * (sv[lc + e] - kv[e]) : sv[lc + e];
#pragma unroll
        for (int r = 0; r < RP; ++r) {
            const int i = rl + r * 16;
            if (i < a.dk) {
                const float k = sk[i] * fk;
#pragma unroll
                for (int e = 0; e < 4; ++e) s[r][e] = fmaf(k, u[e], s[r][e]);
            }
        }
        if (rl < 4) {  // S^T q with the token's own write
            const float o = rl == 0 ? qs[0] + qk * u[0] : rl == 1 ? qs[1] + qk * u[1] : rl == 2 ? qs[2] + qk * u[2] : qs[3] + qk * u[3];
            if (c0 + rl < a.dv) a.out[(size_t)t * a.ldo + (size_t)h * a.dv + c0 + rl] = o;
        }
        if (t + 1 < a.T) __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < RP; ++r) {
        const int i = rl + r * 16;
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

// the last inputs of a call into the ring (calls of more than one token, after every reader of the older entries)
template <bool F32>
__global__ void __launch_bounds__(256) gated_ring_kernel(const GatedLinearArgs a) {
    pdl_wait();
    const int nq = a.kv_heads * a.dk, channels = 2 * nq + a.heads * a.dv, ch = blockIdx.x * 256 + threadIdx.x;
    if (ch >= channels) return;
    const int col = ch < nq ? a.q_off + ch : ch < 2 * nq ? a.k_off + ch - nq : a.v_off + ch - 2 * nq;
    for (int t = max(0, a.T - a.taps); t < a.T; ++t)
        a.ring[(size_t)((a.pos0 + t) % a.taps) * channels + ch] = in_at<F32>(a.in, (size_t)t * a.ld + col);
}
template <bool F32>
int write_ring(cudaStream_t stream, const GatedLinearArgs& a) {
    const int channels = 2 * a.kv_heads * a.dk + a.heads * a.dv;
    cudaError_t e = launch(gated_ring_kernel<F32>, dim3((channels + 255) / 256), dim3(256), 0, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gated linear attention (ring): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

template <bool F32>
int run_steps(cudaStream_t stream, const GatedLinearArgs& a) {
    const int rp = (a.dk + 15) / 16;
    auto k = rp <= 2 ? gated_step_kernel<F32, 2> : rp <= 4 ? gated_step_kernel<F32, 4> : rp <= 8 ? gated_step_kernel<F32, 8>
           : rp <= 16 ? gated_step_kernel<F32, 16> : gated_step_kernel<F32, 32>;
    const size_t smem = ((size_t)3 * round_to(a.dk, 4) + kSCols + round_to(a.rank, 8) + round_to(a.gate_rank, 8)) * 4;
    cudaError_t e = allow_all_dynamic_smem(k);
    if (e == cudaSuccess) e = launch(k, dim3(a.heads, (a.dv + kSCols - 1) / kSCols), dim3(kSThreads), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gated linear attention (steps): %s", cudaGetErrorString(e));
    return a.taps > 0 && a.T > 1 ? write_ring<F32>(stream, a) : KMLL_OK;
}

// ---- chunked form -----------------------------------------------------------------------------------------------------------------
constexpr int kGC = 64, kGThreads = 256, kAP = kGC + 4;  // tokens per chunk; pitch of the token-by-token matrices in f32

// What the preparing launch leaves per (chunk, head): bf16 head / remainder planes [64][DK] of q 2^G, k 2^(G_n - G) and (delta) W,
// [64][64] of A, then 2^G_n [DK] in f32.
struct ChunkLayout {
    int dk;                // DK
    size_t plane, a_plane, floats;  // in floats; `floats` per (chunk, head)
};
__host__ __device__ inline ChunkLayout chunk_layout(int DK, int delta) {
    ChunkLayout l;
    l.dk = DK;
    l.plane = (size_t)kGC * DK / 2;
    l.a_plane = (size_t)kGC * kGC / 2;
    l.floats = (delta ? 6 : 4) * l.plane + 2 * l.a_plane + DK;
    return l;
}
struct ChunkArgs {
    GatedLinearArgs a;
    int chunks, dvp;       // dvp: dv rounded up to 32
    float* planes;         // [chunks][heads][layout.floats]
    float* u0;             // delta: [chunks][heads][64][dvp]
};
inline int padded_keys(int dk) { return dk <= 64 ? 64 : 128; }

// f32 pairs in shared memory -> operand registers (head, remainder)
__device__ inline void split_pair(const float2 v, uint32_t& hi, uint32_t& lo) { split_bf16x2(v.x, v.y, hi, lo); }
// c += (ah + al) (bh + bl) without the product of the remainders
__device__ inline void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    mma_bf16(c, ah, bh0, bh1);
    mma_bf16(c, al, bh0, bh1);
    mma_bf16(c, ah, bl0, bl1);
}

template <int DK, bool DELTA>
__global__ void __launch_bounds__(kGThreads) gated_chunk_prepare_kernel(const ChunkArgs ca) {
    constexpr int P = DK + 4;
    const GatedLinearArgs& a = ca.a;
    extern __shared__ __align__(16) float gsm[];
    float* const Q = gsm;                  // [64][P]
    float* const K = Q + kGC * P;
    float* const G = K + kGC * P;          // log2 decays, then their running sums
    float* const A = G + kGC * P;          // [64][kAP]
    float* const L = A + kGC * kAP;        // DELTA: L, then its inverse
    __shared__ float beta[kGC], total[4 * DK];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int c = blockIdx.x, h = blockIdx.y, t0 = c * kGC, n = min(kGC, a.T - t0);
    const int per = a.heads / a.kv_heads, hq = h / per, nq = a.kv_heads * a.dk, channels = 2 * nq + a.heads * a.dv;
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const ChunkLayout lay = chunk_layout(DK, DELTA ? 1 : 0);
    float* const out = ca.planes + ((size_t)c * a.heads + h) * lay.floats;
    uint16_t* const planes = reinterpret_cast<uint16_t*>(out);
    for (int i = tid; i < kGC * kAP * (DELTA ? 2 : 1); i += kGThreads) A[i] = 0.0f;
    const float rate = decay_rate(a, h);
    pdl_wait();
    // ---- q, k, log decays, write strengths; rows behind the last token change nothing (zeros, decay 1)
    for (int i = tid; i < kGC * DK; i += kGThreads) {
        const int t = i / DK, d = i % DK;
        float q = 0.0f, k = 0.0f;
        if (t < n && d < a.dk) {
            const int ch = hq * a.dk + d;
            q = convolved<false>(a, t0 + t, a.pos0 + t0 + t, a.q_off + ch, ch, channels);
            k = convolved<false>(a, t0 + t, a.pos0 + t0 + t, a.k_off + ch, nq + ch, channels);
            if (a.unit_eps <= 0.0f) q *= a.q_scale;
        }
        Q[t * P + d] = q;
        K[t * P + d] = k;
    }
    if (tid < kGC) beta[tid] = !DELTA ? 1.0f : tid < n ? act_sigmoid(bf16_bits_to_f32(in[(size_t)(t0 + tid) * a.ld + a.b_off + h])) : 0.0f;
    {   // z = W_up a: 64 tokens x DK channels, DK / 8 column blocks over the warps
        constexpr int NB = DK / 64;
        const int rank8 = round_to(a.rank, 8);
        float z[NB][4][4];
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int m = 0; m < 4; ++m)
#pragma unroll
                for (int e = 0; e < 4; ++e) z[b][m][e] = 0.0f;
        for (int k0 = 0; k0 < rank8; k0 += 16) {
            const int ka = k0 + 2 * tq, kb = ka + 8;
            uint32_t w[NB][2];
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const int d = (warp * NB + b) * 8 + g;
                const uint16_t* up = a.up + (size_t)(h * a.dk + d) * a.ldu;
                w[b][0] = d < a.dk && ka < rank8 ? *reinterpret_cast<const uint32_t*>(up + ka) : 0u;
                w[b][1] = d < a.dk && kb < rank8 ? *reinterpret_cast<const uint32_t*>(up + kb) : 0u;
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                const int ra = m * 16 + g, rb = ra + 8;
                const uint16_t* pa = in + (size_t)(t0 + ra) * a.ld + a.a_off;
                const uint16_t* pb = in + (size_t)(t0 + rb) * a.ld + a.a_off;
                uint32_t x[4];
                x[0] = ra < n && ka < rank8 ? *reinterpret_cast<const uint32_t*>(pa + ka) : 0u;
                x[1] = rb < n && ka < rank8 ? *reinterpret_cast<const uint32_t*>(pb + ka) : 0u;
                x[2] = ra < n && kb < rank8 ? *reinterpret_cast<const uint32_t*>(pa + kb) : 0u;
                x[3] = rb < n && kb < rank8 ? *reinterpret_cast<const uint32_t*>(pb + kb) : 0u;
#pragma unroll
                for (int b = 0; b < NB; ++b) mma_bf16(z[b][m], x, w[b][0], w[b][1]);
            }
        }
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int m = 0; m < 4; ++m)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = m * 16 + g + (e >> 1) * 8, d = (warp * NB + b) * 8 + 2 * tq + (e & 1);
                    float l = 0.0f;
                    if (t < n && d < a.dk) l = log2_decay(a, z[b][m][e] + (a.bias != nullptr ? bf16_bits_to_f32(a.bias[h * a.dk + d]) : 0.0f), rate);
                    G[t * P + d] = l;
                }
    }
    __syncthreads();
    // ---- unit vectors; running sums of the log decays
    if (a.unit_eps > 0.0f)
        for (int r = warp; r < 2 * kGC; r += kGThreads / 32) {
            float* x = (r < kGC ? Q : K) + (r & (kGC - 1)) * P;
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < DK / 32; ++i) s += x[lane + i * 32] * x[lane + i * 32];
            const float f = (r < kGC ? a.q_scale : 1.0f) / sqrtf(warp_sum(s) + a.unit_eps);
#pragma unroll
            for (int i = 0; i < DK / 32; ++i) x[lane + i * 32] *= f;
        }
    {
        constexpr int SEG = kGThreads / DK, LEN = kGC / SEG;
        const int d = tid % DK, seg = tid / DK;
        float run = 0.0f;
#pragma unroll
        for (int i = 0; i < LEN; ++i) {
            run += G[(seg * LEN + i) * P + d];
            G[(seg * LEN + i) * P + d] = run;
        }
        total[seg * DK + d] = run;
        __syncthreads();
        float before = 0.0f;
        for (int s = 0; s < seg; ++s) before += total[s * DK + d];
        if (seg > 0)
#pragma unroll
            for (int i = 0; i < LEN; ++i) G[(seg * LEN + i) * P + d] += before;
    }
    __syncthreads();
    // ---- A and L: six 16 x 16 blocks below the diagonal, then the pairs on the diagonal blocks, 32 at a time
    constexpr int kPairs = 136, kUnits = 6 + 4 * kPairs / 32;
    for (int u = warp; u < kUnits; u += kGThreads / 32) {
        if (u < 6) {
            const int I = u < 1 ? 1 : u < 3 ? 2 : 3, J = u - (I * (I - 1)) / 2, ref = I * 16 - 1;
            const int ia = I * 16 + g, ib = ia + 8;
            float ca_[2][4] = {}, cl_[2][4] = {};
#pragma unroll 2
            for (int k0 = 0; k0 < DK; k0 += 16) {
                uint32_t qh[4], ql[4], kh[4], kl[4];
#pragma unroll
                for (int x = 0; x < 2; ++x) {  // channels d, d + 1 of both rows
                    const int d = k0 + x * 8 + 2 * tq;
                    const float2 gr = *reinterpret_cast<const float2*>(G + ref * P + d);
#pragma unroll
                    for (int y = 0; y < 2; ++y) {
                        const int i = y == 0 ? ia : ib;
                        const float2 gi = *reinterpret_cast<const float2*>(G + i * P + d);
                        const float e0 = ex2_approx(gi.x - gr.x), e1 = ex2_approx(gi.y - gr.y);
                        const float2 q = *reinterpret_cast<const float2*>(Q + i * P + d);
                        split_bf16x2(q.x * e0, q.y * e1, qh[x * 2 + y], ql[x * 2 + y]);
                        if (DELTA) {
                            const float2 k = *reinterpret_cast<const float2*>(K + i * P + d);
                            split_bf16x2(k.x * e0, k.y * e1, kh[x * 2 + y], kl[x * 2 + y]);
                        }
                    }
                }
#pragma unroll
                for (int nb = 0; nb < 2; ++nb) {
                    const int j = J * 16 + nb * 8 + g;
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const int d = k0 + x * 8 + 2 * tq;
                        const float2 gr = *reinterpret_cast<const float2*>(G + ref * P + d), gj = *reinterpret_cast<const float2*>(G + j * P + d);
                        const float2 k = *reinterpret_cast<const float2*>(K + j * P + d);
                        split_bf16x2(k.x * ex2_approx(gr.x - gj.x), k.y * ex2_approx(gr.y - gj.y), bh[x], bl[x]);
                    }
                    mma_split(ca_[nb], qh, ql, bh[0], bh[1], bl[0], bl[1]);
                    if (DELTA) mma_split(cl_[nb], kh, kl, bh[0], bh[1], bl[0], bl[1]);
                }
            }
#pragma unroll
            for (int nb = 0; nb < 2; ++nb)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = (e >> 1) ? ib : ia, j = J * 16 + nb * 8 + 2 * tq + (e & 1);
                    A[i * kAP + j] = ca_[nb][e];
                    if (DELTA) L[i * kAP + j] = beta[i] * cl_[nb][e];
                }
        } else {
            const int p = (u - 6) * 32 + lane, B = p / kPairs, r = p - B * kPairs;
            int i = (int)((sqrtf(8.0f * (float)r + 1.0f) - 1.0f) * 0.5f);
            if (i * (i + 1) / 2 > r) --i;
            if ((i + 1) * (i + 2) / 2 <= r) ++i;
            const int j = B * 16 + r - i * (i + 1) / 2;
            i += B * 16;
            float sa = 0.0f, sl = 0.0f;
#pragma unroll 2
            for (int d = 0; d < DK; d += 4) {
                const float4 gi = *reinterpret_cast<const float4*>(G + i * P + d), gj = *reinterpret_cast<const float4*>(G + j * P + d);
                const float4 kj = *reinterpret_cast<const float4*>(K + j * P + d), qi = *reinterpret_cast<const float4*>(Q + i * P + d);
                const float w0 = kj.x * ex2_approx(gi.x - gj.x), w1 = kj.y * ex2_approx(gi.y - gj.y), w2 = kj.z * ex2_approx(gi.z - gj.z),
                            w3 = kj.w * ex2_approx(gi.w - gj.w);
                sa += qi.x * w0 + qi.y * w1 + qi.z * w2 + qi.w * w3;
                if (DELTA) {
                    const float4 ki = *reinterpret_cast<const float4*>(K + i * P + d);
                    sl += ki.x * w0 + ki.y * w1 + ki.z * w2 + ki.w * w3;
                }
            }
            A[i * kAP + j] = sa;
            if (DELTA && j < i) L[i * kAP + j] = beta[i] * sl;
        }
    }
    __syncthreads();
    // ---- planes of q, k and A; the inverse of I + L by forward substitution, one column per thread of the first two warps
    if (!DELTA || warp >= 2) {
        const int first = DELTA ? tid - 64 : tid, step = DELTA ? kGThreads - 64 : kGThreads;
        const size_t pl = lay.plane * 2;
        for (int i = first; i < kGC * DK / 2; i += step) {
            const int t = i / (DK / 2), d = (i % (DK / 2)) * 2;
            const float2 gt = *reinterpret_cast<const float2*>(G + t * P + d), gn = *reinterpret_cast<const float2*>(G + (kGC - 1) * P + d);
            const float2 q = *reinterpret_cast<const float2*>(Q + t * P + d), k = *reinterpret_cast<const float2*>(K + t * P + d);
            uint32_t hi, lo;
            uint32_t* p = reinterpret_cast<uint32_t*>(planes) + i;
            split_bf16x2(q.x * ex2_approx(gt.x), q.y * ex2_approx(gt.y), hi, lo);
            p[0] = hi;
            p[pl / 2] = lo;
            split_bf16x2(k.x * ex2_approx(gn.x - gt.x), k.y * ex2_approx(gn.y - gt.y), hi, lo);
            p[pl] = hi;
            p[3 * (pl / 2)] = lo;
        }
        uint32_t* ap = reinterpret_cast<uint32_t*>(out + (DELTA ? 6 : 4) * lay.plane);
        for (int i = first; i < kGC * kGC / 2; i += step) {
            const float2 v = *reinterpret_cast<const float2*>(A + (i / (kGC / 2)) * kAP + (i % (kGC / 2)) * 2);
            uint32_t hi, lo;
            split_bf16x2(v.x, v.y, hi, lo);
            ap[i] = hi;
            ap[lay.a_plane + i] = lo;
        }
        float* dn = out + (DELTA ? 6 : 4) * lay.plane + 2 * lay.a_plane;
        for (int d = first; d < DK; d += step) dn[d] = ex2_approx(G[(kGC - 1) * P + d]);
    } else if (DELTA) {
        float x[kGC];
#pragma unroll
        for (int i = 0; i < kGC; ++i) {
            float s0 = i == tid ? 1.0f : 0.0f, s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
#pragma unroll
            for (int m = 0; m + 3 < i; m += 4) {
                const float4 l = *reinterpret_cast<const float4*>(L + i * kAP + m);
                s0 = fmaf(-l.x, x[m], s0);
                s1 = fmaf(-l.y, x[m + 1], s1);
                s2 = fmaf(-l.z, x[m + 2], s2);
                s3 = fmaf(-l.w, x[m + 3], s3);
            }
#pragma unroll
            for (int m = i / 4 * 4; m < i; ++m) s0 = fmaf(-L[i * kAP + m], x[m], s0);
            x[i] = (s0 + s1) + (s2 + s3);
        }
        asm volatile("bar.sync 1, 64;" ::: "memory");  // both warps have read L
#pragma unroll
        for (int i = 0; i < kGC; ++i) L[i * kAP + tid] = x[i];
    }
    if (!DELTA) return;
    __syncthreads();
    // ---- W = X (beta k 2^G), U0 = X (beta v): right-hand sides into Q's place, DK columns at a time
    for (int i = tid; i < kGC * DK; i += kGThreads) {
        const int t = i / DK, d = i % DK;
        K[t * P + d] *= beta[t] * ex2_approx(G[t * P + d]);
    }
    const int tiles = (ca.dvp + DK - 1) / DK;
    for (int tile = -1; tile < tiles; ++tile) {
        const float* R = K;
        if (tile >= 0) {
            __syncthreads();
            for (int i = tid; i < kGC * DK; i += kGThreads) {
                const int t = i / DK, col = tile * DK + i % DK;
                float v = 0.0f;
                if (t < n && col < a.dv) v = beta[t] * convolved<false>(a, t0 + t, a.pos0 + t0 + t, a.v_off + h * a.dv + col, 2 * nq + h * a.dv + col, channels);
                Q[t * P + i % DK] = v;
            }
            R = Q;
        }
        __syncthreads();
        constexpr int NB = DK / 64;  // column blocks of 8 per warp
#pragma unroll 1
        for (int m = 0; m < 4; ++m) {
            float acc[NB][4] = {};
            for (int ks = 0; ks <= m; ++ks) {  // X is lower triangular
                uint32_t xh[4], xl[4];
#pragma unroll
                for (int x = 0; x < 2; ++x)
#pragma unroll
                    for (int y = 0; y < 2; ++y)
                        split_pair(*reinterpret_cast<const float2*>(L + (m * 16 + g + y * 8) * kAP + ks * 16 + x * 8 + 2 * tq), xh[x * 2 + y], xl[x * 2 + y]);
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    const int d = (warp * NB + b) * 8 + g;
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const int r = ks * 16 + x * 8 + 2 * tq;
                        split_bf16x2(R[r * P + d], R[(r + 1) * P + d], bh[x], bl[x]);
                    }
                    mma_split(acc[b], xh, xl, bh[0], bh[1], bl[0], bl[1]);
                }
            }
#pragma unroll
            for (int b = 0; b < NB; ++b)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int t = m * 16 + g + (e >> 1) * 8, d = (warp * NB + b) * 8 + 2 * tq;
                    if (tile < 0) {
                        uint32_t hi, lo;
                        split_bf16x2(acc[b][e], acc[b][e + 1], hi, lo);
                        uint32_t* p = reinterpret_cast<uint32_t*>(out + 4 * lay.plane) + (t * DK + d) / 2;
                        p[0] = hi;
                        p[lay.plane] = lo;
                    } else if (tile * DK + d < ca.dvp) {
                        float* p = ca.u0 + (((size_t)c * a.heads + h) * kGC + t) * ca.dvp + tile * DK + d;
                        *reinterpret_cast<float2*>(p) = make_float2(acc[b][e], acc[b][e + 1]);
                    }
                }
        }
    }
}

// Block (head, 32 value columns): the state in registers, chunk after chunk.
template <int DK, bool DELTA>
__global__ void __launch_bounds__(kGThreads) gated_chunk_scan_kernel(const ChunkArgs ca) {
    constexpr int P = DK + 8, PA = kGC + 8, PU = 32 + 8, MT = DK / 16, NT = MT / 2;
    const GatedLinearArgs& a = ca.a;
    extern __shared__ __align__(16) uint16_t rsm[];
    uint16_t* const Qt = rsm;                        // [2][64][P]: heads, remainders
    uint16_t* const Kt = Qt + 2 * kGC * P;
    uint16_t* const At = Kt + 2 * kGC * P;           // [2][64][PA]
    uint16_t* const Ss = At + 2 * kGC * PA;          // [2][DK][PU]
    uint16_t* const Us = Ss + 2 * DK * PU;           // [2][64][PU]
    float* const Dn = reinterpret_cast<float*>(Us + 2 * kGC * PU);  // [DK]
    uint16_t* const Wt = reinterpret_cast<uint16_t*>(Dn + DK);      // DELTA: [2][64][P]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int h = blockIdx.x, v0 = blockIdx.y * 32;
    const int mt = warp % MT, nt0 = (warp / MT) * NT;
    const ChunkLayout lay = chunk_layout(DK, DELTA ? 1 : 0);
    float* const S = a.state + (size_t)h * a.dk * a.dv;
    float s[NT][4];
    auto at = [&](int i, int e, int& d, int& col) { d = mt * 16 + g + (e >> 1) * 8; col = v0 + (nt0 + i) * 8 + 2 * tq + (e & 1); };
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int d, col;
            at(i, e, d, col);
            s[i][e] = d < a.dk && col < a.dv ? S[(size_t)d * a.dv + col] : 0.0f;
        }
    pdl_wait();
    auto copy = [&](uint16_t* tile, const uint16_t* src, int rows, int cols, int pitch) {
        const int runs = cols / 8;
        for (int i = tid; i < rows * runs; i += kGThreads) {
            const int r = i / runs, cc = (i - r * runs) * 8;
            cp_async16_to((uint32_t)__cvta_generic_to_shared(tile + r * pitch + cc), src + (size_t)r * cols + cc);
        }
    };
    auto source = [&](int c) { return ca.planes + ((size_t)c * a.heads + h) * lay.floats; };
    auto load_first = [&](int c) {  // q 2^G, W
        if (c < ca.chunks) {
            const float* p = source(c);
            copy(Qt, reinterpret_cast<const uint16_t*>(p), 2 * kGC, DK, P);
            if (DELTA) copy(Wt, reinterpret_cast<const uint16_t*>(p + 4 * lay.plane), 2 * kGC, DK, P);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto load_second = [&](int c) {  // k 2^(G_n - G), A, 2^G_n
        if (c < ca.chunks) {
            const float* p = source(c);
            copy(Kt, reinterpret_cast<const uint16_t*>(p + 2 * lay.plane), 2 * kGC, DK, P);
            const float* ap = p + (DELTA ? 6 : 4) * lay.plane;
            copy(At, reinterpret_cast<const uint16_t*>(ap), 2 * kGC, kGC, PA);
            if (tid < DK / 4) cp_async16_to((uint32_t)__cvta_generic_to_shared(Dn + tid * 4), ap + 2 * lay.a_plane + tid * 4);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_first(0);
    load_second(0);
    const int wr = (warp & 3) * 16;  // rows of this warp in the products with 64 rows
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    for (int c = 0; c < ca.chunks; ++c) {
        const int t0 = c * kGC, n = min(kGC, a.T - t0);
        // ---- the state as head / remainder planes; U0 (or v) on its way
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                uint32_t hi, lo;
                split_bf16x2(s[i][e], s[i][e + 1], hi, lo);
                const int o = (mt * 16 + g + (e >> 1) * 8) * PU + (nt0 + i) * 8 + 2 * tq;
                *reinterpret_cast<uint32_t*>(Ss + o) = hi;
                *reinterpret_cast<uint32_t*>(Ss + DK * PU + o) = lo;
            }
        float2 u[4][2];
        if (warp < 4) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    const int t = wr + g + y * 8, col = v0 + i * 8 + 2 * tq;
                    if (DELTA) {
                        u[i][y] = *reinterpret_cast<const float2*>(ca.u0 + (((size_t)c * a.heads + h) * kGC + t) * ca.dvp + col);
                    } else {
                        const uint16_t* v = in + (size_t)(t0 + t) * a.ld + a.v_off + (size_t)h * a.dv + col;
                        u[i][y].x = t < n && col < a.dv ? bf16_bits_to_f32(v[0]) : 0.0f;
                        u[i][y].y = t < n && col + 1 < a.dv ? bf16_bits_to_f32(v[1]) : 0.0f;
                    }
                }
        }
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        // ---- first half of the block: U = U0 - W S; second half: q 2^G S
        float o[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
        if (DELTA || warp >= 4) {
            const uint16_t* X = warp < 4 ? Wt : Qt;
#pragma unroll 2
            for (int k = 0; k < DK / 16; ++k) {
                uint32_t xh[4], xl[4], bh[4], bl[4];
                const int ao = (wr + (lane & 15)) * P + k * 16 + (lane >> 4) * 8;
                ldmatrix_x4(xh, X + ao);
                ldmatrix_x4(xl, X + kGC * P + ao);
#pragma unroll
                for (int n2 = 0; n2 < 2; ++n2) {
                    const int bo = (k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PU + n2 * 16 + (lane >> 4) * 8;
                    ldmatrix_x4_trans(bh, Ss + bo);
                    ldmatrix_x4_trans(bl, Ss + DK * PU + bo);
                    mma_split(o[2 * n2], xh, xl, bh[0], bh[1], bl[0], bl[1]);
                    mma_split(o[2 * n2 + 1], xh, xl, bh[2], bh[3], bl[2], bl[3]);
                }
            }
        }
        if (warp < 4) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    uint32_t hi, lo;
                    split_bf16x2(u[i][y].x - o[i][2 * y], u[i][y].y - o[i][2 * y + 1], hi, lo);
                    const int at_ = (wr + g + y * 8) * PU + i * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(Us + at_) = hi;
                    if (DELTA) *reinterpret_cast<uint32_t*>(Us + kGC * PU + at_) = lo;
                }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        load_first(c + 1);
        // ---- outputs: + A U
        if (warp >= 4) {
            for (int k = 0; k <= (warp & 3); ++k) {
                uint32_t xh[4], xl[4], bh[4], bl[4] = {};
                const int ao = (wr + (lane & 15)) * PA + k * 16 + (lane >> 4) * 8;
                ldmatrix_x4(xh, At + ao);
                ldmatrix_x4(xl, At + kGC * PA + ao);
#pragma unroll
                for (int n2 = 0; n2 < 2; ++n2) {
                    const int bo = (k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PU + n2 * 16 + (lane >> 4) * 8;
                    ldmatrix_x4_trans(bh, Us + bo);
                    if (DELTA) {
                        ldmatrix_x4_trans(bl, Us + kGC * PU + bo);
                        mma_split(o[2 * n2], xh, xl, bh[0], bh[1], bl[0], bl[1]);
                        mma_split(o[2 * n2 + 1], xh, xl, bh[2], bh[3], bl[2], bl[3]);
                    } else {
                        mma_bf16(o[2 * n2], xh, bh[0], bh[1]);
                        mma_bf16(o[2 * n2], xl, bh[0], bh[1]);
                        mma_bf16(o[2 * n2 + 1], xh, bh[2], bh[3]);
                        mma_bf16(o[2 * n2 + 1], xl, bh[2], bh[3]);
                    }
                }
            }
            const bool v2 = ((a.ldo | a.dv) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 7u) == 0;
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int t = wr + g + (e >> 1) * 8, col = v0 + i * 8 + 2 * tq;
                    if (t >= n || col >= a.dv) continue;
                    float* p = a.out + (size_t)(t0 + t) * a.ldo + (size_t)h * a.dv + col;
                    if (v2) {
                        *reinterpret_cast<float2*>(p) = make_float2(o[i][e], o[i][e + 1]);
                    } else {
                        p[0] = o[i][e];
                        if (col + 1 < a.dv) p[1] = o[i][e + 1];
                    }
                }
        }
        // ---- the state behind the chunk
        {
            const float da = Dn[mt * 16 + g], db = Dn[mt * 16 + g + 8];
#pragma unroll
            for (int i = 0; i < NT; ++i) { s[i][0] *= da; s[i][1] *= da; s[i][2] *= db; s[i][3] *= db; }
#pragma unroll
            for (int k = 0; k < kGC / 16; ++k) {
                uint32_t xh[4], xl[4], bh[4], bl[4];
                const int ao = (k * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * P + mt * 16 + ((lane >> 3) & 1) * 8;
                ldmatrix_x4_trans(xh, Kt + ao);
                ldmatrix_x4_trans(xl, Kt + kGC * P + ao);
#pragma unroll
                for (int n2 = 0; n2 < NT / 2; ++n2) {
                    const int bo = (k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PU + nt0 * 8 + n2 * 16 + (lane >> 4) * 8;
                    ldmatrix_x4_trans(bh, Us + bo);
                    if (DELTA) {
                        ldmatrix_x4_trans(bl, Us + kGC * PU + bo);
                        mma_split(s[2 * n2], xh, xl, bh[0], bh[1], bl[0], bl[1]);
                        mma_split(s[2 * n2 + 1], xh, xl, bh[2], bh[3], bl[2], bl[3]);
                    } else {
                        mma_bf16(s[2 * n2], xh, bh[0], bh[1]);
                        mma_bf16(s[2 * n2], xl, bh[0], bh[1]);
                        mma_bf16(s[2 * n2 + 1], xh, bh[2], bh[3]);
                        mma_bf16(s[2 * n2 + 1], xl, bh[2], bh[3]);
                    }
                }
            }
        }
        __syncthreads();
        load_second(c + 1);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int d, col;
            at(i, e, d, col);
            if (d < a.dk && col < a.dv) S[(size_t)d * a.dv + col] = s[i][e];
        }
}

template <int DK, bool DELTA>
int run_chunked(cudaStream_t stream, const ChunkArgs& ca) {
    constexpr size_t s1 = ((size_t)3 * kGC * (DK + 4) + (DELTA ? 2 : 1) * kGC * kAP) * 4;
    constexpr size_t s2 = ((size_t)(DELTA ? 6 : 4) * kGC * (DK + 8) + 2 * kGC * (kGC + 8) + 2 * (size_t)DK * 40 + 2 * kGC * 40) * 2 + (size_t)DK * 4;
    cudaError_t e = allow_all_dynamic_smem(gated_chunk_prepare_kernel<DK, DELTA>);
    if (e == cudaSuccess) e = allow_all_dynamic_smem(gated_chunk_scan_kernel<DK, DELTA>);
    if (e == cudaSuccess) e = launch(gated_chunk_prepare_kernel<DK, DELTA>, dim3(ca.chunks, ca.a.heads), dim3(kGThreads), s1, stream, true, ca);
    if (e == cudaSuccess) e = launch(gated_chunk_scan_kernel<DK, DELTA>, dim3(ca.a.heads, ca.dvp / 32), dim3(kGThreads), s2, stream, true, ca);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gated linear attention (chunked): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace

int gated_linear_steps(cudaStream_t stream, const GatedLinearArgs& a) {
    if (a.dk > 512) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: key size %d above 512", a.dk);
    if (a.taps > kMaxConvTaps) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: %d taps", a.taps);
    return a.in_f32 ? run_steps<true>(stream, a) : run_steps<false>(stream, a);
}

bool gated_linear_chunked_ok(const GatedLinearArgs& a) {
    return !a.in_f32 && a.dk <= 128 && a.T >= 4 && a.taps <= kMaxConvTaps && ((a.ld | a.a_off | a.ldu) & 7) == 0;
}
size_t gated_chunk_scratch_floats(int T, int heads, int dk, int dv, int delta) {
    if (dk > 128) return 4;
    const size_t blocks = (size_t)((T + kGC - 1) / kGC) * heads;
    return blocks * chunk_layout(padded_keys(dk), delta).floats + (delta ? blocks * kGC * round_to(dv, 32) : 0);
}
int gated_linear_chunked(cudaStream_t stream, const GatedLinearArgs& a) {
    if (!gated_linear_chunked_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: no chunked form for key size %d", a.dk);
    ChunkArgs ca;
    ca.a = a;
    ca.chunks = (a.T + kGC - 1) / kGC;
    ca.dvp = round_to(a.dv, 32);
    const int DK = padded_keys(a.dk);
    ca.planes = a.scratch;
    ca.u0 = a.scratch + (size_t)ca.chunks * a.heads * chunk_layout(DK, a.delta).floats;
    const int rc = DK == 64 ? (a.delta ? run_chunked<64, true>(stream, ca) : run_chunked<64, false>(stream, ca))
                            : (a.delta ? run_chunked<128, true>(stream, ca) : run_chunked<128, false>(stream, ca));
    if (rc != KMLL_OK) return rc;
    return a.taps > 0 ? write_ring<false>(stream, a) : KMLL_OK;
}

}  // namespace kmll
