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
// X = (I + L)^-1 each chunk's U = X beta V - W S_in, W = X beta (K 2^G).  A and L are made in blocks of 16 x 16 tokens whose
// factors refer to one row's G.  Below the diagonal that is the row ahead of the block, so that both exponents are sums of log
// decays and not positive.  On the diagonal it is the block's first row, and the keys' exponents are positive; a block in which
// some channel decays to less than 2^-90 is summed pair by pair instead.

#include <type_traits>

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
// dot product of eight bf16 weights with eight values (both 16-byte aligned)
__device__ inline float dot8(const uint16_t* w, const float* x) {
    const uint4 t = *reinterpret_cast<const uint4*>(w);
    const float4 u = *reinterpret_cast<const float4*>(x), v = *reinterpret_cast<const float4*>(x + 4);
    float s = __uint_as_float(t.x << 16) * u.x, r = __uint_as_float(t.z << 16) * v.x;
    s = fmaf(__uint_as_float(t.x & 0xffff0000u), u.y, s);
    r = fmaf(__uint_as_float(t.z & 0xffff0000u), v.y, r);
    s = fmaf(__uint_as_float(t.y << 16), u.z, s);
    r = fmaf(__uint_as_float(t.w << 16), v.z, r);
    s = fmaf(__uint_as_float(t.y & 0xffff0000u), u.w, s);
    r = fmaf(__uint_as_float(t.w & 0xffff0000u), v.w, r);
    return s + r;
}

// ---- step form ------------------------------------------------------------------------------------------------------------------
// Block (head, 32 value columns): eight warps of four columns; a lane keeps rows lane, lane + 32, .. of them in registers for the
// whole call, so the sums over keys stay inside a warp.  Of a single token's work, everything that does not read its projections
// (state, low-rank maps, the convolutions over earlier inputs) is done ahead of the dependency wait.
constexpr int kSThreads = 256, kSCols = 32;
struct StepLayout {
    int dkr, rank8, gate8, chans;  // padded sizes; channels a block convolves
    int off_part, off_maps;        // in floats: partial convolutions; in bytes: the staged maps
    bool staged;
    int total;
};
__host__ __device__ inline StepLayout step_layout(int dk, int rank, int gate_rank, int taps) {
    StepLayout l;
    l.dkr = round_to(dk, 4);
    l.rank8 = round_to(rank, 8);
    l.gate8 = round_to(gate_rank, 8);
    l.chans = 2 * dk + kSCols;
    l.off_part = 3 * l.dkr + kSCols + l.rank8 + l.gate8;
    l.off_maps = round_to((l.off_part + (taps > 0 ? 2 * l.chans : 0)) * 4, 16);
    const int maps = (dk * (l.rank8 + 8) + (gate_rank > 0 ? kSCols * (l.gate8 + 8) : 0)) * 2;
    l.staged = maps <= 96 * 1024;
    l.total = l.off_maps + (l.staged ? maps : 0);
    return l;
}

template <bool F32, int RP>
__global__ void __launch_bounds__(kSThreads) gated_step_kernel(const GatedLinearArgs a) {
    extern __shared__ __align__(16) float ssm[];  // q | k | decay, [dk] each | v [32] | decay factor | gate factor | ..
    const StepLayout sl = step_layout(a.dk, a.rank, a.gate_rank, a.taps);
    const int rank8 = sl.rank8, gate8 = sl.gate8;
    float* const sq = ssm;
    float* const sk = sq + sl.dkr;
    float* const sg = sk + sl.dkr;
    float* const sv = sg + sl.dkr;
    float* const sa = sv + kSCols;
    float* const sgr = sa + rank8;
    float* const early = ssm + sl.off_part;       // one token: sum over the earlier taps, then the last tap, per channel
    uint16_t* const maps = reinterpret_cast<uint16_t*>(reinterpret_cast<unsigned char*>(ssm) + sl.off_maps);
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col0 = blockIdx.y * kSCols, lc = warp * 4, c0 = col0 + lc;
    const int per = a.heads / a.kv_heads, hq = h / per, nq = a.kv_heads * a.dk, channels = 2 * nq + a.heads * a.dv;
    float* const S = a.state + (size_t)h * a.dk * a.dv;
    const bool vec = (a.dv & 3) == 0, single = a.T == 1;
    // weights never change; the state's last writer lies more than one launch back, and so does that of the position and the ring
    const int up_pitch = sl.staged ? rank8 + 8 : a.ldu, gate_pitch = sl.staged ? gate8 + 8 : a.ldg;
    const uint16_t* up = a.up + (size_t)h * a.dk * a.ldu;
    const uint16_t* gate_up = a.gate_rank > 0 ? a.gate_up + (size_t)(h * a.dv + col0) * a.ldg : nullptr;
    if (sl.staged) {
        const int runs = rank8 / 8;
        for (int i = tid; i < a.dk * runs; i += kSThreads) {
            const int d = i / runs, r = (i - d * runs) * 8;
            cp_async16_to((uint32_t)__cvta_generic_to_shared(maps + d * up_pitch + r), up + (size_t)d * a.ldu + r);
        }
        uint16_t* const gm = maps + a.dk * up_pitch;
        if (a.gate_rank > 0) {
            const int gruns = gate8 / 8, rows = min(kSCols, a.dv - col0);
            for (int i = tid; i < rows * gruns; i += kSThreads) {
                const int c = i / gruns, r = (i - c * gruns) * 8;
                cp_async16_to((uint32_t)__cvta_generic_to_shared(gm + c * gate_pitch + r), gate_up + (size_t)c * a.ldg + r);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        up = maps;
        gate_up = gm;
    }
    float s[RP][4];
#pragma unroll
    for (int r = 0; r < RP; ++r) {
        const int i = lane + r * 32;
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
    const int pos0 = a.at != nullptr ? a.at->position : a.pos0;
    // column of the projection and channel of entry i of q | k | v (v: of this block's columns); false: no such channel
    auto place = [&](int i, int& col, int& ch) -> bool {
        if (i < 2 * a.dk) {
            const int d = i < a.dk ? i : i - a.dk;
            ch = (i < a.dk ? 0 : nq) + hq * a.dk + d;
            col = (i < a.dk ? a.q_off : a.k_off) + hq * a.dk + d;
            return true;
        }
        const int c = i - 2 * a.dk;
        ch = 2 * nq + h * a.dv + col0 + c;
        col = a.v_off + h * a.dv + col0 + c;
        return col0 + c < a.dv;
    };
    if (single && a.taps > 0)
#pragma unroll 2
        for (int i = tid; i < sl.chans; i += kSThreads) {
            int col, ch;
            float y = 0.0f, last = 0.0f;
            if (place(i, col, ch)) {
                const uint16_t* w = a.conv + (size_t)ch * a.taps;
                for (int j0 = 0; j0 + 1 < a.taps; j0 += 4) {  // four loads in flight
                    float x[4], f[4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const int p = pos0 - (a.taps - 1 - j0 - j);
                        const bool live = j0 + j + 1 < a.taps && p >= 0;
                        x[j] = live ? a.ring[(size_t)(p % a.taps) * channels + ch] : 0.0f;
                        f[j] = live ? bf16_bits_to_f32(w[j0 + j]) : 0.0f;
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j) y = fmaf(f[j], x[j], y);
                }
                last = bf16_bits_to_f32(w[a.taps - 1]);
            }
            early[i] = y;
            early[sl.chans + i] = last;
        }
    const float rate = decay_rate(a, h);
    pdl_wait();
    for (int t = 0; t < a.T; ++t) {
        const int pos = pos0 + t;
        const size_t row = (size_t)t * a.ld;
        // ---- q, k, v; decays (two lanes per channel); gate (eight lanes per column)
        const int entries = sl.chans + rank8 + gate8;
        for (int i0 = tid; i0 < entries; i0 += 4 * kSThreads) {
            float x[4];
            int ch[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {  // four loads in flight
                const int i = i0 + j * kSThreads, r = i - sl.chans;
                int col = -1;
                ch[j] = -1;
                if (i < sl.chans) {
                    if (!place(i, col, ch[j])) col = ch[j] = -1;
                } else if (i < entries) {
                    if (r < rank8) col = r < a.rank ? a.a_off + r : -1;
                    else col = r - rank8 < a.gate_rank ? a.g_off + r - rank8 : -1;
                }
                x[j] = col >= 0 ? in_at<F32>(a.in, row + col) : 0.0f;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int i = i0 + j * kSThreads;
                if (i >= entries) break;
                float y = x[j];
                if (ch[j] >= 0 && a.taps > 0) {
                    if (single) {
                        y = act_silu(fmaf(early[sl.chans + i], x[j], early[i]));
                        if (i >= 2 * a.dk || (blockIdx.y == 0 && h == hq * per)) a.ring[(size_t)(pos % a.taps) * channels + ch[j]] = x[j];
                    } else {
                        int col, unused;
                        place(i, col, unused);
                        y = convolved<F32>(a, t, pos, col, ch[j], channels);
                    }
                }
                (i < a.dk ? sq : i < 2 * a.dk ? sk - a.dk : sv - 2 * a.dk)[i] = y;  // (the factors follow v)
            }
        }
        const float beta = a.delta ? act_sigmoid(in_at<F32>(a.in, row + a.b_off + h)) : 1.0f;
        if (t == 0 && sl.staged) asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i0 = 0; i0 < 2 * a.dk; i0 += kSThreads) {
            const int d = (i0 + tid) >> 1;
            float z = 0.0f;
            if (d < a.dk)
#pragma unroll 4
                for (int r = (tid & 1) * 8; r < rank8; r += 16) z += dot8(up + (size_t)d * up_pitch + r, sa + r);
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            if (d < a.dk && (tid & 1) == 0) {
                if (a.bias != nullptr) z += bf16_bits_to_f32(a.bias[h * a.dk + d]);
                sg[d] = exp2f(log2_decay(a, z, rate));
            }
        }
        if (a.gate_rank > 0) {
            const int c = tid >> 3, part = tid & 7;
            float g = 0.0f;
            if (col0 + c < a.dv)
                for (int r = part * 8; r < gate8; r += 64) g += dot8(gate_up + (size_t)c * gate_pitch + r, sgr + r);
            g += __shfl_xor_sync(0xffffffffu, g, 1);
            g += __shfl_xor_sync(0xffffffffu, g, 2);
            g += __shfl_xor_sync(0xffffffffu, g, 4);
            if (part == 0 && col0 + c < a.dv) a.gate[(size_t)t * a.heads * a.dv + (size_t)h * a.dv + col0 + c] = g;
        }
        __syncthreads();
        // ---- the recurrence
        float sums[16] = {};  // of the decayed state: S^T k, S^T q; then q.q, k.k, q.k
#pragma unroll
        for (int r = 0; r < RP; ++r) {
            const int i = lane + r * 32;
            if (i < a.dk) {
                const float g = sg[i], k = sk[i], q = sq[i];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[r][e] *= g;
                    sums[e] = fmaf(k, s[r][e], sums[e]);
                    sums[4 + e] = fmaf(q, s[r][e], sums[4 + e]);
                }
                sums[8] = fmaf(q, q, sums[8]);
                sums[9] = fmaf(k, k, sums[9]);
                sums[10] = fmaf(q, k, sums[10]);
            }
        }
        // fold the sums over 32 lanes: lanes keep one half of them in each step; lanes 2 j and 2 j + 1 end up with sum j
#pragma unroll
        for (int n = 8, off = 16; n >= 1; n >>= 1, off >>= 1) {
            const bool high = (lane & off) != 0;
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (i < n) {
                    const float keep = high ? sums[i + n] : sums[i], give = high ? sums[i] : sums[i + n];
                    sums[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                }
        }
        const float all = sums[0] + __shfl_xor_sync(0xffffffffu, sums[0], 1);
        float fq = a.q_scale, fk = 1.0f;
        if (a.unit_eps > 0.0f) {
            fq *= 1.0f / sqrtf(__shfl_sync(0xffffffffu, all, 16) + a.unit_eps);
            fk = 1.0f / sqrtf(__shfl_sync(0xffffffffu, all, 18) + a.unit_eps);
        }
        const float qk = __shfl_sync(0xffffffffu, all, 20) * fq * fk;
        float u[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float kv = __shfl_sync(0xffffffffu, all, e * 2);
            u[e] = a.delta ? beta * (sv[lc + e] - fk * kv) : sv[lc + e];
        }
        const float qs = __shfl_sync(0xffffffffu, all, 8 + (lane & 3) * 2);
        if (lane < 4 && c0 + lane < a.dv)  // S^T q with the token's own write
            a.out[(size_t)t * a.ldo + (size_t)h * a.dv + c0 + lane] = fq * qs + qk * (lane == 0 ? u[0] : lane == 1 ? u[1] : lane == 2 ? u[2] : u[3]);
#pragma unroll
        for (int r = 0; r < RP; ++r) {
            const int i = lane + r * 32;
            if (i < a.dk) {
                const float k = sk[i] * fk;
#pragma unroll
                for (int e = 0; e < 4; ++e) s[r][e] = fmaf(k, u[e], s[r][e]);
            }
        }
        if (t + 1 < a.T) __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < RP; ++r) {
        const int i = lane + r * 32;
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
    const int rp = (a.dk + 31) / 32;
    auto k = rp <= 1 ? gated_step_kernel<F32, 1> : rp <= 2 ? gated_step_kernel<F32, 2> : rp <= 4 ? gated_step_kernel<F32, 4>
           : rp <= 8 ? gated_step_kernel<F32, 8> : gated_step_kernel<F32, 16>;
    const size_t smem = (size_t)step_layout(a.dk, a.rank, a.gate_rank, a.taps).total;
    if (smem > 220 * 1024) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: ranks %d, %d are too large", a.rank, a.gate_rank);
    cudaError_t e = allow_all_dynamic_smem(k);
    if (e == cudaSuccess) e = launch(k, dim3(a.heads, (a.dv + kSCols - 1) / kSCols), dim3(kSThreads), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gated linear attention (steps): %s", cudaGetErrorString(e));
    return a.taps > 0 && a.T > 1 ? write_ring<F32>(stream, a) : KMLL_OK;
}

// ---- chunked form -----------------------------------------------------------------------------------------------------------------
constexpr int kGC = 64, kGThreads = 256, kAP = kGC + 8;  // tokens per chunk; pitch of token-by-token matrices

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

// SiLU and log2 of the decay from the hardware's 2^x and log2 (a few ulp)
__device__ inline float fast_silu(float z) { return __fdividef(z, 1.0f + ex2_approx(-z * kLog2e)); }
__device__ inline float fast_softplus(float z) {
    const float t = ex2_approx(-fabsf(z) * kLog2e);
    return fmaxf(z, 0.0f) + (t < 0.015625f ? t * (1.0f - t * (0.5f - t * (1.0f / 3.0f))) : __logf(1.0f + t));
}
__device__ inline float fast_log2_decay(const GatedLinearArgs& a, float z, float rate) {
    const float l = a.decay == KMLL_DECAY_LOGISTIC ? -fast_softplus(-z) * a.inv_tau : -rate * fast_softplus(z);
    return fmaxf(l * kLog2e, -150.0f);
}
// c += (ah + al) (bh + bl) without the product of the remainders
__device__ inline void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    mma_bf16(c, ah, bh0, bh1);
    mma_bf16(c, al, bh0, bh1);
    mma_bf16(c, ah, bl0, bl1);
}

// Shared memory of the preparing launch, in bytes: q, k and log decays of the chunk in f32; ahead of them, in the same places, the
// projected rows they come from.
struct PrepareLayout {
    int P, PR;             // pitches: f32 rows, rows of the decay map
    int off_k, off_g, off_l, off_x, off_v, staged_decay, total;
};
__host__ __device__ inline PrepareLayout prepare_layout(int DK, int delta, int taps, int rank) {
    PrepareLayout l;
    const int rows = kGC + (taps > 0 ? taps - 1 : 0), tile = kGC * (DK + 4) * 4, raw = rows * DK * 2;
    l.P = DK + 4;
    l.PR = round_to(rank, 16) + 8;
    l.off_k = tile;
    l.off_g = 2 * tile;
    l.off_l = l.off_g + (2 * raw > tile ? 2 * raw : tile);
    l.off_x = l.off_l + (delta ? kGC * kAP * 4 : 0);
    l.off_v = l.off_x + (delta ? 2 * kGC * kAP * 2 : 0);
    l.total = l.off_v + (delta ? raw : 0);
    l.staged_decay = (kGC + DK) * l.PR * 2 <= 2 * tile;  // the decay factor and map fit in the places of q and k
    return l;
}

// Rows [t0 - taps + 1, t0 + 64) of `cols` consecutive projected channels (from column `col`, ring channel `ch`) -> bf16 tile
// [..][DK]; zeros where there is no token or channel.
template <int DK, int NT>
__device__ inline void stage_rows(const GatedLinearArgs& a, uint16_t* tile, int t0, int n, int col, int ch, int cols, int channels, bool fast) {
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const int back = a.taps > 0 ? a.taps - 1 : 0, rows = kGC + back;
    constexpr int RUNS = DK / 8;
    for (int i = threadIdx.x; i < rows * RUNS; i += NT) {
        const int r = i / RUNS, c = (i % RUNS) * 8, t = t0 + r - back;
        uint16_t* dst = tile + r * DK + c;
        if (t >= 0 && fast) {
            const bool live = r - back < n && c < cols;
            cp_async16_zfill_to((uint32_t)__cvta_generic_to_shared(dst), live ? in + (size_t)t * a.ld + col + c : in, live ? 16u : 0u);
        } else {
            for (int e = 0; e < 8; ++e) {
                uint16_t v = 0;
                if (c + e < cols && r - back < n) {
                    if (t >= 0) v = in[(size_t)t * a.ld + col + c + e];
                    else if (a.pos0 + t >= 0) v = f32_to_bf16_bits(a.ring[(size_t)((a.pos0 + t) % a.taps) * channels + ch + c + e]);
                }
                dst[e] = v;
            }
        }
    }
}
__device__ inline float2 unpack2(uint32_t x) { return make_float2(__uint_as_float(x << 16), __uint_as_float(x & 0xffff0000u)); }
// taps of channels ch, ch + 1 (odd: of ch alone), up to four of them, the last at index 3
struct PairTaps { float2 w[4]; };
__device__ inline PairTaps load_taps(const GatedLinearArgs& a, int ch, bool live, bool odd) {
    PairTaps p;
    const int lead = 4 - a.taps;
    const uint16_t* w = a.conv + (size_t)ch * a.taps;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const bool on = live && a.taps > 0 && a.taps <= 4 && j >= lead;
        p.w[j] = make_float2(on ? bf16_bits_to_f32(w[j - lead]) : 0.0f, on && !odd ? bf16_bits_to_f32(w[a.taps + j - lead]) : 0.0f);
    }
    return p;
}
// channels d, d + 1 of tokens t .. t + ROWS - 1 from a staged tile, through convolution and SiLU
template <int DK, int ROWS>
__device__ inline void staged_rows(const GatedLinearArgs& a, const uint16_t* tile, int t, int d, const PairTaps& taps, int ch, bool odd, float2 (&y)[ROWS]) {
    auto at = [&](int r) { return unpack2(*reinterpret_cast<const uint32_t*>(tile + r * DK + d)); };
    if (a.taps == 0) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) y[i] = at(t + i);
        return;
    }
    if (a.taps <= 4) {
        const int lead = 4 - a.taps;  // missing taps
        float2 x[4];
#pragma unroll
        for (int j = 0; j < 3; ++j) x[j] = j >= lead ? at(t + j - lead) : make_float2(0.0f, 0.0f);
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            x[3] = at(t + i + 3 - lead);
            float2 s = __fmul2_rn(taps.w[0], x[0]);
            s = __ffma2_rn(taps.w[1], x[1], s);
            s = __ffma2_rn(taps.w[2], x[2], s);
            y[i] = __ffma2_rn(taps.w[3], x[3], s);
            x[0] = x[1];
            x[1] = x[2];
            x[2] = x[3];
        }
    } else {
        const uint16_t* w0 = a.conv + (size_t)ch * a.taps;
        const uint16_t* w1 = odd ? w0 : w0 + a.taps;
#pragma unroll
        for (int i = 0; i < ROWS; ++i) y[i] = make_float2(0.0f, 0.0f);
        for (int j = 0; j < a.taps; ++j) {
            const float2 w = make_float2(bf16_bits_to_f32(w0[j]), bf16_bits_to_f32(w1[j]));
#pragma unroll
            for (int i = 0; i < ROWS; ++i) y[i] = __ffma2_rn(w, at(t + i + j), y[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) y[i] = make_float2(fast_silu(y[i].x), fast_silu(y[i].y));
}

template <int DK, bool DELTA>
__global__ void __launch_bounds__(DELTA ? 512 : 256) gated_chunk_prepare_kernel(const ChunkArgs ca) {
    constexpr int NT = DELTA ? 512 : 256, NW = NT / 32, P = DK + 4;
    const GatedLinearArgs& a = ca.a;
    extern __shared__ __align__(16) unsigned char gsm[];
    const PrepareLayout pl = prepare_layout(DK, DELTA ? 1 : 0, a.taps, a.rank);
    float* const Q = reinterpret_cast<float*>(gsm);               // [64][P]
    float* const K = reinterpret_cast<float*>(gsm + pl.off_k);    // [64][P]
    float* const G = reinterpret_cast<float*>(gsm + pl.off_g);    // [64][P] log2 decays, then their running sums
    float* const L = reinterpret_cast<float*>(gsm + pl.off_l);    // DELTA: [64][kAP]
    uint16_t* const X = reinterpret_cast<uint16_t*>(gsm + pl.off_x);  // DELTA: (I + L)^-1, [2][64][kAP] heads, remainders
    const int back = a.taps > 0 ? a.taps - 1 : 0;
    uint16_t* const raw_q = reinterpret_cast<uint16_t*>(gsm + pl.off_g);
    uint16_t* const raw_k = raw_q + (kGC + back) * DK;
    uint16_t* const raw_v = reinterpret_cast<uint16_t*>(gsm + pl.off_v);
    uint16_t* const sa = reinterpret_cast<uint16_t*>(gsm);        // [64][PR] decay factor
    uint16_t* const su = sa + kGC * pl.PR;                        // [DK][PR] decay map of this head
    __shared__ float beta[kGC], total[NT];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int c = blockIdx.x, h = blockIdx.y, t0 = c * kGC, n = min(kGC, a.T - t0);
    const int per = a.heads / a.kv_heads, hq = h / per, nq = a.kv_heads * a.dk, channels = 2 * nq + a.heads * a.dv;
    const int chq = hq * a.dk, chv = 2 * nq + h * a.dv;
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const bool fast = ((a.ld | a.q_off | a.k_off | a.v_off | a.dk | a.dv) & 7) == 0 && (reinterpret_cast<uintptr_t>(a.in) & 15u) == 0;
    const ChunkLayout lay = chunk_layout(DK, DELTA ? 1 : 0);
    float* const out = ca.planes + ((size_t)c * a.heads + h) * lay.floats;
    uint16_t* const planes = reinterpret_cast<uint16_t*>(out);
    uint16_t* const Ah = reinterpret_cast<uint16_t*>(out + (DELTA ? 6 : 4) * lay.plane);
    uint16_t* const Al = Ah + 2 * lay.a_plane;
    const int rank8 = round_to(a.rank, 8), runs = pl.PR / 8 - 1;
    if (pl.staged_decay)  // weights never change: ahead of the dependency wait
        for (int i = tid; i < DK * runs; i += NT) {
            const int d = i / runs, r = (i - d * runs) * 8;
            const bool live = d < a.dk && r < rank8;
            cp_async16_zfill_to((uint32_t)__cvta_generic_to_shared(su + d * pl.PR + r), live ? a.up + (size_t)(h * a.dk + d) * a.ldu + r : a.up, live ? 16u : 0u);
        }
    const float rate = decay_rate(a, h);
    constexpr int PAIRS = DK / 2, ROWS = kGC * PAIRS / NT;  // a thread convolves two channels of ROWS tokens
    const int pd = (tid % PAIRS) * 2, pt = tid / PAIRS * ROWS;
    const bool p_live = pd < a.dk, p_odd = pd + 1 >= a.dk;
    const PairTaps wq = load_taps(a, chq + pd, p_live, p_odd), wk = load_taps(a, nq + chq + pd, p_live, p_odd);
    PairTaps wv = load_taps(a, chv + pd, DELTA && pd < a.dv, pd + 1 >= a.dv);
    // log decays: a warp holds 16 x MB tokens of 8 x NB channels
    constexpr int NB = DK == 64 && NW == 16 ? 1 : DK / 64, MB = DK / NB * 4 / 8 / NW;
    const int cb = warp % (DK / 8 / NB) * NB, mb = warp / (DK / 8 / NB) * MB;
    float bias[NB][2];
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int d = (cb + b) * 8 + 2 * tq + e;
            bias[b][e] = a.bias != nullptr && d < a.dk ? bf16_bits_to_f32(a.bias[h * a.dk + d]) : 0.0f;
        }
    pdl_wait();
    if (pl.staged_decay)
        for (int i = tid; i < kGC * runs; i += NT) {
            const int t = i / runs, r = (i - t * runs) * 8;
            const bool live = t < n && r < rank8;
            cp_async16_zfill_to((uint32_t)__cvta_generic_to_shared(sa + t * pl.PR + r), live ? in + (size_t)(t0 + t) * a.ld + a.a_off + r : in, live ? 16u : 0u);
        }
    stage_rows<DK, NT>(a, raw_q, t0, n, a.q_off + chq, chq, a.dk, channels, fast);
    stage_rows<DK, NT>(a, raw_k, t0, n, a.k_off + chq, nq + chq, a.dk, channels, fast);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (DELTA) stage_rows<DK, NT>(a, raw_v, t0, n, a.v_off + h * a.dv, chv, a.dv, channels, fast);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tid < kGC) beta[tid] = !DELTA ? 1.0f : tid < n ? act_sigmoid(bf16_bits_to_f32(in[(size_t)(t0 + tid) * a.ld + a.b_off + h])) : 0.0f;
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    // ---- log decays from z = W_up a
    float z[NB][MB][4];
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int m = 0; m < MB; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) z[b][m][e] = 0.0f;
    for (int k0 = 0; k0 < rank8; k0 += 16) {
        const int ka = k0 + 2 * tq, kb = ka + 8;
        uint32_t w[NB][2];
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int d = (cb + b) * 8 + g;
            if (pl.staged_decay) {
                w[b][0] = *reinterpret_cast<const uint32_t*>(su + d * pl.PR + ka);
                w[b][1] = *reinterpret_cast<const uint32_t*>(su + d * pl.PR + kb);
            } else {
                const uint16_t* up = a.up + (size_t)(h * a.dk + d) * a.ldu;
                w[b][0] = d < a.dk && ka < rank8 ? *reinterpret_cast<const uint32_t*>(up + ka) : 0u;
                w[b][1] = d < a.dk && kb < rank8 ? *reinterpret_cast<const uint32_t*>(up + kb) : 0u;
            }
        }
#pragma unroll
        for (int m = 0; m < MB; ++m) {
            const int ra = (mb + m) * 16 + g, rb = ra + 8;
            uint32_t x[4];
            if (pl.staged_decay) {
                x[0] = *reinterpret_cast<const uint32_t*>(sa + ra * pl.PR + ka);
                x[1] = *reinterpret_cast<const uint32_t*>(sa + rb * pl.PR + ka);
                x[2] = *reinterpret_cast<const uint32_t*>(sa + ra * pl.PR + kb);
                x[3] = *reinterpret_cast<const uint32_t*>(sa + rb * pl.PR + kb);
            } else {
                const uint16_t* pa = in + (size_t)(t0 + ra) * a.ld + a.a_off;
                const uint16_t* pb = in + (size_t)(t0 + rb) * a.ld + a.a_off;
                x[0] = ra < n && ka < rank8 ? *reinterpret_cast<const uint32_t*>(pa + ka) : 0u;
                x[1] = rb < n && ka < rank8 ? *reinterpret_cast<const uint32_t*>(pb + ka) : 0u;
                x[2] = ra < n && kb < rank8 ? *reinterpret_cast<const uint32_t*>(pa + kb) : 0u;
                x[3] = rb < n && kb < rank8 ? *reinterpret_cast<const uint32_t*>(pb + kb) : 0u;
            }
#pragma unroll
            for (int b = 0; b < NB; ++b) mma_bf16(z[b][m], x, w[b][0], w[b][1]);
        }
    }
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int m = 0; m < MB; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) {  // tokens behind the last change nothing: decay 1
                const int t = (mb + m) * 16 + g + (e >> 1) * 8, d = (cb + b) * 8 + 2 * tq + (e & 1);
                z[b][m][e] = t < n && d < a.dk ? fast_log2_decay(a, z[b][m][e] + bias[b][e & 1], rate) : 0.0f;
            }
    __syncthreads();  // the decay factor and map have been read
    // ---- q and k
    {
        const float fq = a.unit_eps > 0.0f ? 1.0f : a.q_scale;
        float2 q[ROWS], k[ROWS];
#pragma unroll
        for (int i = 0; i < ROWS; ++i) q[i] = k[i] = make_float2(0.0f, 0.0f);
        if (p_live) {
            staged_rows<DK, ROWS>(a, raw_q, pt, pd, wq, chq + pd, p_odd, q);
            staged_rows<DK, ROWS>(a, raw_k, pt, pd, wk, nq + chq + pd, p_odd, k);
        }
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const bool on = p_live && pt + i < n;
            *reinterpret_cast<float2*>(Q + (pt + i) * P + pd) = make_float2(on ? q[i].x * fq : 0.0f, on && !p_odd ? q[i].y * fq : 0.0f);
            *reinterpret_cast<float2*>(K + (pt + i) * P + pd) = make_float2(on ? k[i].x : 0.0f, on && !p_odd ? k[i].y : 0.0f);
        }
    }
    __syncthreads();  // the projected rows have been read
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int m = 0; m < MB; ++m)
#pragma unroll
            for (int e = 0; e < 4; e += 2)
                *reinterpret_cast<float2*>(G + ((mb + m) * 16 + g + (e >> 1) * 8) * P + (cb + b) * 8 + 2 * tq) = make_float2(z[b][m][e], z[b][m][e + 1]);
    // ---- unit vectors; running sums of the log decays
    if (a.unit_eps > 0.0f) {
        constexpr int RN = 2 * kGC / NW, V = DK / 32;  // rows per warp, four at a time; entries per lane
#pragma unroll
        for (int r0 = 0; r0 < RN; r0 += 4) {
            float v[4][V], sum[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int r = warp * RN + r0 + x;
                const float* p = (r < kGC ? Q : K - kGC * P) + r * P + lane * V;
                sum[x] = 0.0f;
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    v[x][i] = p[i];
                    sum[x] += v[x][i] * v[x][i];
                }
            }
#pragma unroll
            for (int off = 16; off > 0; off >>= 1)
#pragma unroll
                for (int x = 0; x < 4; ++x) sum[x] += __shfl_xor_sync(0xffffffffu, sum[x], off);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int r = warp * RN + r0 + x;
                float* p = (r < kGC ? Q : K - kGC * P) + r * P + lane * V;
                const float f = (r < kGC ? a.q_scale : 1.0f) * rsqrtf(sum[x] + a.unit_eps);
#pragma unroll
                for (int i = 0; i < V; ++i) p[i] = v[x][i] * f;
            }
        }
    }
    __syncthreads();
    {
        constexpr int SEG = NT / DK, LEN = kGC / SEG;
        const int d = tid % DK, seg = tid / DK;
        float run[LEN];
#pragma unroll
        for (int i = 0; i < LEN; ++i) run[i] = G[(seg * LEN + i) * P + d];
#pragma unroll
        for (int i = 1; i < LEN; ++i) run[i] += run[i - 1];
        total[seg * DK + d] = run[LEN - 1];
        __syncthreads();
        float before = 0.0f;
        for (int s = 0; s < seg; ++s) before += total[s * DK + d];
#pragma unroll
        for (int i = 0; i < LEN; ++i) G[(seg * LEN + i) * P + d] = run[i] + before;
    }
    __syncthreads();
    // ---- A (to its planes) and L: ten 16 x 16 blocks; steep ones on the diagonal in tiles of 2 x 2 tokens, two lanes each
    unsigned steep = 0;  // bit b: block b on the diagonal
#pragma unroll
    for (int b = 0; b < 4; ++b) {
        bool far = false;
#pragma unroll
        for (int d = 0; d < DK; d += 32) far |= G[b * 16 * P + d + lane] - G[(b * 16 + 15) * P + d + lane] > 90.0f;
        steep |= __any_sync(0xffffffffu, far) ? 1u << b : 0u;
    }
    for (int u = warp; u < (steep != 0u ? 19 : 10); u += NW) {
        if (u >= 10) {
            const int p = (u - 10) * 32 + lane, half = p & 1, B = (p >> 1) / 36;
            if ((__ballot_sync(0xffffffffu, (steep >> B & 1u) != 0u)) == 0u) continue;
            const bool mine = (steep >> B & 1u) != 0u;
            int ti = 0, tj = (p >> 1) - B * 36;
            while (tj > ti) tj -= ++ti;
            const int i = B * 16 + ti * 2, j = B * 16 + tj * 2;
            const float2 minus = make_float2(-1.0f, -1.0f);
            float2 sq[2][2] = {}, sl[2][2] = {};
#pragma unroll 2
            for (int d = half * 4; d < DK; d += 8) {
                float4 gi[2], gj[2], qi[2], ki[2], kj[2];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    gi[x] = *reinterpret_cast<const float4*>(G + (i + x) * P + d);
                    gj[x] = *reinterpret_cast<const float4*>(G + (j + x) * P + d);
                    qi[x] = *reinterpret_cast<const float4*>(Q + (i + x) * P + d);
                    kj[x] = *reinterpret_cast<const float4*>(K + (j + x) * P + d);
                    if (DELTA) ki[x] = *reinterpret_cast<const float4*>(K + (i + x) * P + d);
                }
#pragma unroll
                for (int x = 0; x < 2; ++x)
#pragma unroll
                    for (int y = 0; y < 2; ++y) {
                        float2 e0 = __ffma2_rn(make_float2(gj[y].x, gj[y].y), minus, make_float2(gi[x].x, gi[x].y));
                        float2 e1 = __ffma2_rn(make_float2(gj[y].z, gj[y].w), minus, make_float2(gi[x].z, gi[x].w));
                        e0 = __fmul2_rn(make_float2(kj[y].x, kj[y].y), make_float2(ex2_approx(e0.x), ex2_approx(e0.y)));
                        e1 = __fmul2_rn(make_float2(kj[y].z, kj[y].w), make_float2(ex2_approx(e1.x), ex2_approx(e1.y)));
                        sq[x][y] = __ffma2_rn(make_float2(qi[x].x, qi[x].y), e0, sq[x][y]);
                        sq[x][y] = __ffma2_rn(make_float2(qi[x].z, qi[x].w), e1, sq[x][y]);
                        if (DELTA) {
                            sl[x][y] = __ffma2_rn(make_float2(ki[x].x, ki[x].y), e0, sl[x][y]);
                            sl[x][y] = __ffma2_rn(make_float2(ki[x].z, ki[x].w), e1, sl[x][y]);
                        }
                    }
            }
            float vq[2][2], vl[2][2];
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    vq[x][y] = sq[x][y].x + sq[x][y].y;
                    vq[x][y] += __shfl_xor_sync(0xffffffffu, vq[x][y], 1);
                    if (DELTA) {
                        vl[x][y] = sl[x][y].x + sl[x][y].y;
                        vl[x][y] += __shfl_xor_sync(0xffffffffu, vl[x][y], 1);
                    }
                }
            if (!mine) continue;
            // this lane's row i + half, columns j and j + 1; tokens behind it are not seen (their sums may be anything)
            const int r = i + half;
            uint32_t hi, lo;
            split_bf16x2(half ? vq[1][0] : vq[0][0], j + 1 <= r ? (half ? vq[1][1] : vq[0][1]) : 0.0f, hi, lo);
            *reinterpret_cast<uint32_t*>(Ah + r * kGC + j) = hi;
            *reinterpret_cast<uint32_t*>(Al + r * kGC + j) = lo;
            if (DELTA) *reinterpret_cast<float2*>(L + r * kAP + j) =
                make_float2(j < r ? beta[r] * (half ? vl[1][0] : vl[0][0]) : 0.0f, j + 1 < r ? beta[r] * (half ? vl[1][1] : vl[0][1]) : 0.0f);
            if (tj < ti) {  // the mirrored tile above the diagonal
                *reinterpret_cast<uint32_t*>(Ah + (j + half) * kGC + i) = 0u;
                *reinterpret_cast<uint32_t*>(Al + (j + half) * kGC + i) = 0u;
            }
            continue;
        }
        const int I = u < 1 ? 0 : u < 3 ? 1 : u < 6 ? 2 : 3, J = u - I * (I + 1) / 2, ref = J < I ? I * 16 - 1 : I * 16;
        if (J == I && (steep >> I & 1u) != 0u) continue;
        const int ia = I * 16 + g, ib = ia + 8;
        float ca_[2][4] = {}, cl_[2][4] = {};
#pragma unroll 4
        for (int k0 = 0; k0 < DK; k0 += 16) {
            uint32_t qh[4], ql[4], kh[4], kl[4];
            float2 gr[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {  // channels d, d + 1 of both rows
                const int d = k0 + x * 8 + 2 * tq;
                gr[x] = *reinterpret_cast<const float2*>(G + ref * P + d);
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    const int i = y == 0 ? ia : ib;
                    const float2 gi = *reinterpret_cast<const float2*>(G + i * P + d);
                    const float2 e = make_float2(ex2_approx(gi.x - gr[x].x), ex2_approx(gi.y - gr[x].y));
                    const float2 q = __fmul2_rn(*reinterpret_cast<const float2*>(Q + i * P + d), e);
                    split_bf16x2(q.x, q.y, qh[x * 2 + y], ql[x * 2 + y]);
                    if (DELTA) {
                        const float2 k = __fmul2_rn(*reinterpret_cast<const float2*>(K + i * P + d), e);
                        split_bf16x2(k.x, k.y, kh[x * 2 + y], kl[x * 2 + y]);
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
                    const float2 gj = *reinterpret_cast<const float2*>(G + j * P + d);
                    const float2 k = __fmul2_rn(*reinterpret_cast<const float2*>(K + j * P + d), make_float2(ex2_approx(gr[x].x - gj.x), ex2_approx(gr[x].y - gj.y)));
                    split_bf16x2(k.x, k.y, bh[x], bl[x]);
                }
                mma_split(ca_[nb], qh, ql, bh[0], bh[1], bl[0], bl[1]);
                if (DELTA) mma_split(cl_[nb], kh, kl, bh[0], bh[1], bl[0], bl[1]);
            }
        }
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int i = (e >> 1) ? ib : ia, j = J * 16 + nb * 8 + 2 * tq;
                uint32_t hi, lo;
                split_bf16x2(j <= i ? ca_[nb][e] : 0.0f, j + 1 <= i ? ca_[nb][e + 1] : 0.0f, hi, lo);
                *reinterpret_cast<uint32_t*>(Ah + i * kGC + j) = hi;
                *reinterpret_cast<uint32_t*>(Al + i * kGC + j) = lo;
                if (DELTA) *reinterpret_cast<float2*>(L + i * kAP + j) = make_float2(j < i ? beta[i] * cl_[nb][e] : 0.0f, j + 1 < i ? beta[i] * cl_[nb][e + 1] : 0.0f);
            }
    }
    __syncthreads();
    // ---- planes of q and k; meanwhile the first four warps invert I + L
    constexpr int IW = DELTA ? 128 : 0;  // threads that invert
    if (!DELTA || warp >= 4) {
        for (int i = tid - IW; i < kGC * DK / 2; i += NT - IW) {
            const int t = i / (DK / 2), d = (i % (DK / 2)) * 2;
            const float2 gt = *reinterpret_cast<const float2*>(G + t * P + d), gn = *reinterpret_cast<const float2*>(G + (kGC - 1) * P + d);
            const float2 q = *reinterpret_cast<const float2*>(Q + t * P + d), k = *reinterpret_cast<const float2*>(K + t * P + d);
            uint32_t hi, lo;
            uint32_t* p = reinterpret_cast<uint32_t*>(planes) + i;
            split_bf16x2(q.x * ex2_approx(gt.x), q.y * ex2_approx(gt.y), hi, lo);
            p[0] = hi;
            p[lay.plane] = lo;
            split_bf16x2(k.x * ex2_approx(gn.x - gt.x), k.y * ex2_approx(gn.y - gt.y), hi, lo);
            p[2 * lay.plane] = hi;
            p[3 * lay.plane] = lo;
        }
        float* dn = out + (DELTA ? 6 : 4) * lay.plane + 2 * lay.a_plane;
        for (int d = tid - IW; d < DK; d += NT - IW) dn[d] = ex2_approx(G[(kGC - 1) * P + d]);
    } else if (DELTA) {
        if (warp < 2) {  // the four blocks on the diagonal by forward substitution, a column per thread
            const int r0 = (tid >> 4) * 16, col = tid & 15;
            float x[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float s0 = i == col ? 1.0f : 0.0f, s1 = 0.0f;
#pragma unroll
                for (int m = 0; m < i; ++m) {
                    const float l = L[(r0 + i) * kAP + r0 + m];
                    if (m & 1) s1 = fmaf(-l, x[m], s1);
                    else s0 = fmaf(-l, x[m], s0);
                }
                x[i] = s0 + s1;
            }
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                const uint16_t hi = f32_to_bf16_bits(x[i]);
                X[(r0 + i) * kAP + r0 + col] = hi;
                X[(kGC + r0 + i) * kAP + r0 + col] = f32_to_bf16_bits(x[i] - bf16_bits_to_f32(hi));
            }
        }
        for (int dist = 1; dist < 4; ++dist) {  // X_IJ = -X_II sum_{J <= M < I} L_IM X_MJ, blocks `dist` below the diagonal
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (warp >= 4 - dist) continue;
            const int J = warp, I = J + dist;
            float pt_[2][4] = {};  // the sum, transposed: [column of X_MJ][row of L_IM]
            for (int M = J; M < I; ++M) {
                uint32_t xh[4], xl[4];
                const int ao = (M * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * kAP + J * 16 + ((lane >> 3) & 1) * 8;
                ldmatrix_x4_trans(xh, X + ao);
                ldmatrix_x4_trans(xl, X + kGC * kAP + ao);
#pragma unroll
                for (int nb = 0; nb < 2; ++nb) {
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const float2 l = *reinterpret_cast<const float2*>(L + (I * 16 + nb * 8 + g) * kAP + M * 16 + x * 8 + 2 * tq);
                        split_bf16x2(l.x, l.y, bh[x], bl[x]);
                    }
                    mma_split(pt_[nb], xh, xl, bh[0], bh[1], bl[0], bl[1]);
                }
            }
            uint32_t dh[4], dl[4];
            const int ao = (I * 16 + (lane & 15)) * kAP + I * 16 + (lane >> 4) * 8;
            ldmatrix_x4(dh, X + ao);
            ldmatrix_x4(dl, X + kGC * kAP + ao);
#pragma unroll
            for (int nb = 0; nb < 2; ++nb) {
                float r[4] = {};
                uint32_t bh[2], bl[2];
                split_bf16x2(-pt_[0][2 * nb], -pt_[0][2 * nb + 1], bh[0], bl[0]);
                split_bf16x2(-pt_[1][2 * nb], -pt_[1][2 * nb + 1], bh[1], bl[1]);
                mma_split(r, dh, dl, bh[0], bh[1], bl[0], bl[1]);
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    uint32_t hi, lo;
                    split_bf16x2(r[e], r[e + 1], hi, lo);
                    const int o = (I * 16 + g + (e >> 1) * 8) * kAP + J * 16 + nb * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(X + o) = hi;
                    *reinterpret_cast<uint32_t*>(X + kGC * kAP + o) = lo;
                }
            }
        }
    }
    if (!DELTA) return;
    // ---- W = X (beta k 2^G), U0 = X (beta v): right-hand sides as head / remainder planes [2][64][PB] in the places of q, k and the
    // decays, DK value columns at a time; a warp takes 16 columns
    constexpr int PB = DK + 8;
    uint16_t* const Rk = reinterpret_cast<uint16_t*>(gsm);
    uint16_t* const Rv = Rk + 2 * kGC * PB;
    auto put = [&](uint16_t* R, int t, float x, float y) {
        uint32_t hi, lo;
        split_bf16x2(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(R + t * PB + pd) = hi;
        *reinterpret_cast<uint32_t*>(R + (kGC + t) * PB + pd) = lo;
    };
    {
        __syncthreads();
        float2 k[ROWS];
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            const int t = pt + i;
            const float2 kk = *reinterpret_cast<const float2*>(K + t * P + pd), gg = *reinterpret_cast<const float2*>(G + t * P + pd);
            k[i] = make_float2(beta[t] * kk.x * ex2_approx(gg.x), beta[t] * kk.y * ex2_approx(gg.y));
        }
        __syncthreads();  // k and the decays have been read
#pragma unroll
        for (int i = 0; i < ROWS; ++i) put(Rk, pt + i, k[i].x, k[i].y);
    }
    for (int v0 = 0; v0 < ca.dvp; v0 += DK) {
        if (v0 > 0) {
            __syncthreads();
            stage_rows<DK, NT>(a, raw_v, t0, n, a.v_off + h * a.dv + v0, chv + v0, a.dv - v0, channels, fast);
            asm volatile("cp.async.commit_group;" ::: "memory");
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        {
            const int col = v0 + pd;
            const bool live = col < a.dv, odd = col + 1 >= a.dv;
            if (v0 > 0) wv = load_taps(a, chv + col, live, odd);
            float2 v[ROWS];
            if (live) staged_rows<DK, ROWS>(a, raw_v, pt, pd, wv, chv + col, odd, v);
#pragma unroll
            for (int i = 0; i < ROWS; ++i) {
                const bool on = live && pt + i < n;
                put(Rv, pt + i, on ? beta[pt + i] * v[i].x : 0.0f, on && !odd ? beta[pt + i] * v[i].y : 0.0f);
            }
        }
        __syncthreads();
        constexpr int CG = DK / 16;  // column groups of one right-hand side
        for (int cg = warp + (v0 > 0 ? CG : 0); cg < 2 * CG; cg += NW) {
            const bool is_v = cg >= CG;
            const uint16_t* R = is_v ? Rv : Rk;
            const int c0 = (is_v ? cg - CG : cg) * 16;
            if (is_v && v0 + c0 >= ca.dvp) break;
            uint32_t bh[4][4], bl[4][4];
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                const int bo = (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PB + c0 + (lane >> 4) * 8;
                ldmatrix_x4_trans(bh[ks], R + bo);
                ldmatrix_x4_trans(bl[ks], R + kGC * PB + bo);
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                float acc[2][4] = {};
#pragma unroll
                for (int ks = 0; ks <= m; ++ks) {  // X is lower triangular
                    uint32_t xh[4], xl[4];
                    const int ao = (m * 16 + (lane & 15)) * kAP + ks * 16 + (lane >> 4) * 8;
                    ldmatrix_x4(xh, X + ao);
                    ldmatrix_x4(xl, X + kGC * kAP + ao);
                    mma_split(acc[0], xh, xl, bh[ks][0], bh[ks][1], bl[ks][0], bl[ks][1]);
                    mma_split(acc[1], xh, xl, bh[ks][2], bh[ks][3], bl[ks][2], bl[ks][3]);
                }
#pragma unroll
                for (int b = 0; b < 2; ++b)
#pragma unroll
                    for (int e = 0; e < 4; e += 2) {
                        const int t = m * 16 + g + (e >> 1) * 8, d = c0 + b * 8 + 2 * tq;
                        if (!is_v) {
                            uint32_t hi, lo;
                            split_bf16x2(acc[b][e], acc[b][e + 1], hi, lo);
                            uint32_t* p = reinterpret_cast<uint32_t*>(out + 4 * lay.plane) + (t * DK + d) / 2;
                            p[0] = hi;
                            p[lay.plane] = lo;
                        } else if (v0 + d < ca.dvp) {
                            float* p = ca.u0 + (((size_t)c * a.heads + h) * kGC + t) * ca.dvp + v0 + d;
                            *reinterpret_cast<float2*>(p) = make_float2(acc[b][e], acc[b][e + 1]);
                        }
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
    auto copy = [&](uint16_t* tile, const uint16_t* src, auto columns) {  // head and remainder planes [2][64][columns]
        constexpr int COLS = decltype(columns)::value, RUNS = COLS / 8;
        const uint32_t dst = (uint32_t)__cvta_generic_to_shared(tile) + (uint32_t)((tid / RUNS) * (COLS + 8) + (tid % RUNS) * 8) * 2;
#pragma unroll
        for (int i = 0; i < 2 * kGC * RUNS / kGThreads; ++i)
            cp_async16_to(dst + (uint32_t)(i * (kGThreads / RUNS) * (COLS + 8)) * 2, src + (size_t)(i * kGThreads + tid) * 8);
    };
    using Keys = std::integral_constant<int, DK>;
    using Tokens = std::integral_constant<int, kGC>;
    auto source = [&](int c) { return ca.planes + ((size_t)c * a.heads + h) * lay.floats; };
    auto load_first = [&](int c) {  // q 2^G, W
        if (c < ca.chunks) {
            const float* p = source(c);
            copy(Qt, reinterpret_cast<const uint16_t*>(p), Keys{});
            if (DELTA) copy(Wt, reinterpret_cast<const uint16_t*>(p + 4 * lay.plane), Keys{});
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto load_second = [&](int c) {  // k 2^(G_n - G), A, 2^G_n
        if (c < ca.chunks) {
            const float* p = source(c);
            copy(Kt, reinterpret_cast<const uint16_t*>(p + 2 * lay.plane), Keys{});
            const float* ap = p + (DELTA ? 6 : 4) * lay.plane;
            copy(At, reinterpret_cast<const uint16_t*>(ap), Tokens{});
            if (tid < DK / 4) cp_async16_to((uint32_t)__cvta_generic_to_shared(Dn + tid * 4), ap + 2 * lay.a_plane + tid * 4);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_first(0);
    load_second(0);
    const int wr = (warp & 3) * 16;  // rows of this warp in the products with 64 rows
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const bool pairs = ((a.ld | a.v_off | a.dv) & 1) == 0;
    float2 u[4][2];      // DELTA: U0 of the next chunk, first four warps
    uint32_t uv[4][2];   // else v, as pairs of bf16
    auto load_u = [&](int c) {
        if (warp >= 4 || c >= ca.chunks) return;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                const int t = wr + g + y * 8, col = v0 + i * 8 + 2 * tq;
                if (DELTA) {
                    u[i][y] = *reinterpret_cast<const float2*>(ca.u0 + (((size_t)c * a.heads + h) * kGC + t) * ca.dvp + col);
                } else {
                    const bool row = c * kGC + t < a.T;
                    const uint16_t* v = in + (size_t)(c * kGC + t) * a.ld + a.v_off + (size_t)h * a.dv + col;
                    if (pairs) uv[i][y] = row && col < a.dv ? *reinterpret_cast<const uint32_t*>(v) : 0u;
                    else uv[i][y] = (row && col < a.dv ? (uint32_t)v[0] : 0u) | (row && col + 1 < a.dv ? (uint32_t)v[1] << 16 : 0u);
                }
            }
    };
    load_u(0);
    for (int c = 0; c < ca.chunks; ++c) {
        const int t0 = c * kGC, n = min(kGC, a.T - t0);
        // ---- the state as head / remainder planes
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
                    uint32_t hi = uv[i][y], lo = 0u;
                    if (DELTA) split_bf16x2(u[i][y].x - o[i][2 * y], u[i][y].y - o[i][2 * y + 1], hi, lo);
                    const int at_ = (wr + g + y * 8) * PU + i * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(Us + at_) = hi;
                    if (DELTA) *reinterpret_cast<uint32_t*>(Us + kGC * PU + at_) = lo;
                }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        load_first(c + 1);
        load_u(c + 1);
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
    const size_t s1 = (size_t)prepare_layout(DK, DELTA ? 1 : 0, ca.a.taps, ca.a.rank).total;
    constexpr size_t s2 = ((size_t)(DELTA ? 6 : 4) * kGC * (DK + 8) + 2 * kGC * (kGC + 8) + 2 * (size_t)DK * 40 + 2 * kGC * 40) * 2 + (size_t)DK * 4;
    cudaError_t e = allow_all_dynamic_smem(gated_chunk_prepare_kernel<DK, DELTA>);
    if (e == cudaSuccess) e = allow_all_dynamic_smem(gated_chunk_scan_kernel<DK, DELTA>);
    if (e == cudaSuccess) e = launch(gated_chunk_prepare_kernel<DK, DELTA>, dim3(ca.chunks, ca.a.heads), dim3(DELTA ? 512 : 256), s1, stream, true, ca);
    if (e == cudaSuccess) e = launch(gated_chunk_scan_kernel<DK, DELTA>, dim3(ca.a.heads, ca.dvp / 32), dim3(kGThreads), s2, stream, true, ca);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gated linear attention (chunked): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace

int gated_linear_steps(cudaStream_t stream, const GatedLinearArgs& a) {
    if (a.dk > 512) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: key size %d above 512", a.dk);
    if (a.taps > kMaxConvTaps) return fail(KMLL_ERR_UNSUPPORTED, "gated linear attention: %d taps", a.taps);
    if ((a.ldu & 7) != 0 || (a.gate_rank > 0 && (a.ldg & 7) != 0)) return fail(KMLL_ERR_SHAPE, "gated linear attention: pitches %d, %d are no multiples of 8", a.ldu, a.ldg);
    return a.in_f32 ? run_steps<true>(stream, a) : run_steps<false>(stream, a);
}

bool gated_linear_chunked_ok(const GatedLinearArgs& a) {
    return !a.in_f32 && a.dk <= 128 && a.T >= 4 && a.taps <= kMaxConvTaps && ((a.ld | a.a_off | a.ldu) & 7) == 0 && (reinterpret_cast<uintptr_t>(a.in) & 15u) == 0;
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
