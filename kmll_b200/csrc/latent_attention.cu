// Latent attention: keys and values of every head are linear maps of one normed latent c (rank values) per position, plus one
// rotated key part shared by all heads, so the cache row of a position is (c, rotated part).  Causal, with an optional sliding
// window (a position sees itself and the window - 1 positions before it).
//
//   plain form    any size, f32 arithmetic, one block per (token, head): decoders that compute in f32, sizes the others lack
//   decode form   one token over the bf16 cache with W_uk folded into the query and W_uv applied to the weighted latent, so
//                 the cache is read once for all heads (scores and weights in f32, products on bf16 MMAs, the f32 operands
//                 split into a bf16 head and remainder)
//   prompt form   keys and values written out per head by a projection, then tiled attention with online softmax
#include "internal.cuh"
#include "mma_bf16.cuh"

namespace kmll {

namespace {

template <bool F32>
__device__ inline float val(const void* p, size_t i) {
    return F32 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
// entry i of a vector of `rot` entries that is rotated as a whole
template <bool F32>
__device__ inline float rotated(const void* p, size_t base, int i, int half, const float2* cs) {
    const int j = i < half ? i : i - half;
    const float u = val<F32>(p, base + j), v = val<F32>(p, base + j + half);
    return i < half ? u * cs[j].x - v * cs[j].y : v * cs[j].x + u * cs[j].y;
}

// cache row of a position from the projected latent (row `src` of a.in)
template <bool IN32, bool C32>
__device__ inline void write_row(const LatentArgs& a, size_t src, int pos, float* scratch) {
    float s = 0.0f;
    for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
        const float v = val<IN32>(a.in, src + i);
        s += v * v;
    }
    const float inv = 1.0f / sqrtf(block_sum(s, scratch) / (float)a.rank + a.eps);
    const int half = a.rot >> 1;
    const size_t row = (size_t)pos * a.pitch;
    for (int i = threadIdx.x; i < a.rank + a.rot; i += blockDim.x) {
        const int r = i - a.rank;
        const float v = i < a.rank ? val<IN32>(a.in, src + i) * inv * bf16_bits_to_f32(a.norm_w[i])
                                   : rotated<IN32>(a.in, src + a.rank, r, half, a.table + (size_t)pos * half);
        const size_t at = row + (i < a.rank ? i : a.kr_off + r);
        if (C32) static_cast<float*>(a.cache)[at] = v;
        else static_cast<uint16_t*>(a.cache)[at] = f32_to_bf16_bits(v);
    }
}

template <bool IN32, bool C32>
__global__ void __launch_bounds__(128) latent_write_kernel(const LatentArgs a) {
    __shared__ float scratch[40];
    pdl_wait();
    const int pos = (a.at != nullptr ? a.at->position : a.pos0) + blockIdx.x;
    if (pos >= a.max_seq) return;
    write_row<IN32, C32>(a, (size_t)blockIdx.x * a.ld + a.dkv_off, pos, scratch);
}

// ---- plain form ---------------------------------------------------------------------------------------------------------------
constexpr int kPlainWarps = 4;
template <bool IN32, bool C32>
__global__ void __launch_bounds__(kPlainWarps * 32) latent_plain_kernel(const LatentArgs a) {
    extern __shared__ float psm[];
    float* const qa = psm;                     // [rank] query folded through W_uk
    float* const qr = qa + a.rank;             // [rot]
    float* const acc = qr + a.rot;             // [warps][rank]
    __shared__ float stat[2 * kPlainWarps];
    pdl_wait();
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pos = (a.at != nullptr ? a.at->position : a.pos0) + t, half = a.rot >> 1;
    const size_t q0 = (size_t)t * a.ld + a.q_off + (size_t)h * (a.dim + a.rot);
    for (int r = tid; r < a.rank; r += blockDim.x) {
        float s = 0.0f;
        for (int d = 0; d < a.dim; ++d) s = fmaf(val<IN32>(a.in, q0 + d), bf16_bits_to_f32(a.uk[(size_t)(h * a.dim + d) * a.ldu + r]), s);
        qa[r] = s;
    }
    for (int i = tid; i < a.rot; i += blockDim.x) qr[i] = rotated<IN32>(a.in, q0 + a.dim, i, half, a.table + (size_t)pos * half);
    for (int i = tid; i < kPlainWarps * a.rank; i += blockDim.x) acc[i] = 0.0f;
    __syncthreads();
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    float m = -INFINITY, l = 0.0f;
    float* const mine = acc + warp * a.rank;
    for (int j = lo + warp; j <= pos; j += kPlainWarps) {
        const size_t row = (size_t)j * a.pitch;
        float s = 0.0f;
        for (int i = lane; i < a.rank; i += 32) s = fmaf(qa[i], val<C32>(a.cache, row + i), s);
        for (int i = lane; i < a.rot; i += 32) s = fmaf(qr[i], val<C32>(a.cache, row + a.kr_off + i), s);
        s = warp_sum(s) * a.scale;
        const float mn = fmaxf(m, s), corr = expf(m - mn), w = expf(s - mn);
        m = mn;
        l = l * corr + w;
        for (int i = lane; i < a.rank; i += 32) mine[i] = mine[i] * corr + w * val<C32>(a.cache, row + i);
    }
    if (lane == 0) { stat[warp] = m; stat[kPlainWarps + warp] = l; }
    __syncthreads();
    float mx = -INFINITY, total = 0.0f, f[kPlainWarps];
    for (int w = 0; w < kPlainWarps; ++w) mx = fmaxf(mx, stat[w]);
    for (int w = 0; w < kPlainWarps; ++w) {
        f[w] = stat[w] == -INFINITY ? 0.0f : expf(stat[w] - mx);
        total += f[w] * stat[kPlainWarps + w];
    }
    for (int r = tid; r < a.rank; r += blockDim.x) {
        float s = 0.0f;
        for (int w = 0; w < kPlainWarps; ++w) s += f[w] * acc[w * a.rank + r];
        qa[r] = s / total;
    }
    __syncthreads();
    for (int v = warp; v < a.vdim; v += kPlainWarps) {
        const uint16_t* u = a.uv + (size_t)(h * a.vdim + v) * a.ldu;
        float s = 0.0f;
        for (int r = lane; r < a.rank; r += 32) s = fmaf(bf16_bits_to_f32(u[r]), qa[r], s);
        s = warp_sum(s);
        if (lane == 0) a.out[(size_t)t * a.ldo + (size_t)h * a.vdim + v] = s;
    }
}

// ---- decode form ----------------------------------------------------------------------------------------------------------------
// Widths: a cache row as staged in shared memory has kp = columns of (c, rotated part) rounded up to 32 for the score MMAs and
// rp = rank rounded up to 256 for the value MMAs (16 warps of 16-column pairs); the tile is as wide as the larger.
constexpr int kDT = 128;      // positions per tile
constexpr int kDHeads = 16;   // heads per block = MMA rows
constexpr int kDMaxSplit = 32;
constexpr int kDWarps = 16;
struct LatentDecodePlan {
    int kp, rp, width, nsplit, hgroups;
    size_t q_floats, part_floats;
};
__host__ __device__ inline int round_up(int v, int m) { return (v + m - 1) / m * m; }
LatentDecodePlan decode_plan(int heads, int rank, int rot, int span) {
    LatentDecodePlan p;
    const int kr = round_up(rank, 8);
    p.kp = round_up(kr + rot, 32);
    p.rp = round_up(rank, 256);
    p.width = p.kp > p.rp ? p.kp : p.rp;
    p.hgroups = (heads + kDHeads - 1) / kDHeads;
    p.nsplit = (span + 15) / 16;  // a split of fewer than 16 positions would not fill a step of the value MMAs
    const int cap = p.hgroups >= 148 ? 1 : 148 / p.hgroups;
    if (p.nsplit > cap) p.nsplit = cap;
    if (p.nsplit > kDMaxSplit) p.nsplit = kDMaxSplit;
    if (p.nsplit < 1) p.nsplit = 1;
    p.q_floats = (size_t)p.hgroups * kDHeads * p.kp;
    p.part_floats = (size_t)p.nsplit * heads * (rank + 2);
    return p;
}
struct DecodeRange { int lo, pos, chunk, active; };
__device__ inline DecodeRange decode_range(int pos, int window, int nsplit) {
    DecodeRange r;
    r.pos = pos;
    r.lo = window > 0 ? max(0, pos - window + 1) : 0;
    const int count = pos - r.lo + 1;
    r.chunk = max((count + nsplit - 1) / nsplit, 16);
    r.active = (count + r.chunk - 1) / r.chunk;
    return r;
}

// q folded through W_uk (times the score factor) and rotated, per head as [kp] bf16 heads and, `lo` elements further on, [kp]
// remainders; the block behind the last head writes the cache row
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LatentArgs a, uint16_t* __restrict__ q, size_t lo, int kp) {
    extern __shared__ float asm_[];  // query [dim], then reduction [16][128]
    __shared__ float scratch[40];
    float* const sq = asm_;
    float* const red = asm_ + round_up(a.dim, 4);
    const int h = blockIdx.x, tid = threadIdx.x, grp = tid >> 4, c = tid & 15, r = blockIdx.y * 128 + c * 8;
    constexpr int PRE = 8;
    uint4 w[PRE];
    const bool live = h < a.heads && r < a.ldu;
#pragma unroll
    for (int i = 0; i < PRE; ++i) {  // weights never change: fetched ahead of the dependency wait
        const int d = grp + i * 16;
        w[i] = (live && d < a.dim) ? ld_stream_u4(a.uk + (size_t)(h * a.dim + d) * a.ldu + r) : make_uint4(0u, 0u, 0u, 0u);
    }
    const int pos = a.at->position, half = a.rot >> 1;  // (written more than one launch ago)
    pdl_wait();
    if (h == a.heads) {
        if (blockIdx.y == 0 && pos < a.max_seq) write_row<true, false>(a, (size_t)a.dkv_off, pos, scratch);
        return;
    }
    const float* in = static_cast<const float*>(a.in) + a.q_off + (size_t)h * (a.dim + a.rot);
    for (int d = tid; d < a.dim; d += 256) sq[d] = in[d];
    __syncthreads();
    float acc[8] = {};
    auto add = [&](const uint4& t, float x) {
        const uint32_t ww[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            acc[2 * e] = fmaf(__uint_as_float(ww[e] << 16), x, acc[2 * e]);
            acc[2 * e + 1] = fmaf(__uint_as_float(ww[e] & 0xffff0000u), x, acc[2 * e + 1]);
        }
    };
#pragma unroll
    for (int i = 0; i < PRE; ++i)
        if (grp + i * 16 < a.dim) add(w[i], sq[grp + i * 16]);
    for (int d = grp + PRE * 16; d < a.dim; d += 16)
        if (live) add(ld_stream_u4(a.uk + (size_t)(h * a.dim + d) * a.ldu + r), sq[d]);
#pragma unroll
    for (int e = 0; e < 8; ++e) red[grp * 128 + c * 8 + e] = acc[e];
    __syncthreads();
    uint16_t* const qrow = q + (size_t)h * kp;
    auto put = [&](int col, float v) {
        const uint16_t hi = f32_to_bf16_bits(v);
        qrow[col] = hi;
        qrow[lo + col] = f32_to_bf16_bits(v - bf16_bits_to_f32(hi));
    };
    if (tid < 128) {
        const int col = blockIdx.y * 128 + tid;
        float s = 0.0f;
#pragma unroll
        for (int g = 0; g < 16; ++g) s += red[g * 128 + tid];
        if (col < a.rank) put(col, s * a.scale);
    }
    if (blockIdx.y == 0) {
        for (int i = tid; i < kp - a.rank; i += 256) {
            const int col = a.rank + i, j = col - a.kr_off;
            float v = 0.0f;
            if (j >= 0 && j < a.rot) v = rotated<true>(in, (size_t)a.dim, j, half, a.table + (size_t)pos * half) * a.scale;
            put(col, v);
        }
    }
}

__global__ void __launch_bounds__(kDWarps * 32) latent_decode_kernel(const LatentArgs a, const uint16_t* __restrict__ q, size_t lo, float* __restrict__ part,
                                                            const LatentDecodePlan pl) {
    extern __shared__ __align__(16) uint16_t dsm[];
    const int W = pl.width + 8;                 // tile row, elements
    uint16_t* const tile = dsm;                 // [kDT][W]
    uint16_t* const qh = tile + kDT * W;        // [16][W]
    uint16_t* const ql = qh + kDHeads * W;
    uint16_t* const ph = ql + kDHeads * W;      // [16][kDT + 8]
    uint16_t* const plo = ph + kDHeads * (kDT + 8);
    float* const sc = reinterpret_cast<float*>(plo + kDHeads * (kDT + 8));  // [16][kDT]
    float* const corr = sc + kDHeads * kDT;     // [16]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * kDHeads;
    // the position was written more than one launch ago, and so was every cache row but the newest
    const DecodeRange R = decode_range(a.at->position, a.window, pl.nsplit);
    const int begin = R.lo + split * R.chunk, end = min(begin + R.chunk, R.pos + 1);
    const uint16_t* cache = static_cast<const uint16_t*>(a.cache);
    const int runs = a.pitch / 8, wruns = W / 8;
    const bool active = split < R.active;
    auto load_tile = [&](int t0, int from, int to) {  // rows of positions [from, to) of the tile at t0; a warp per row
        const int rows = min(kDT, (end - t0 + 15) & ~15);  // (what the value MMAs read; rows behind the last position are zeros)
        for (int r = warp; r < rows; r += kDWarps) {
            const int p = t0 + r;
            if (p < from || p >= to) continue;
            const uint16_t* src = cache + (size_t)(p < end ? p : t0) * a.pitch;
            const uint32_t dst = (uint32_t)__cvta_generic_to_shared(tile + (size_t)r * W);
            const int live = p < end ? runs : 0;
            for (int c = lane; c < wruns; c += 32) cp_async16_zfill_to(dst + c * 16, c < live ? src + c * 8 : cache, c < live ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (active) load_tile(begin, begin, R.pos);  // all but the newest row
    pdl_wait();
    if (!active) return;
    for (int r = warp; r < 2 * kDHeads; r += kDWarps) {  // query heads and remainders
        const int h = r & (kDHeads - 1);
        const bool live = h0 + h < a.heads;
        const uint16_t* src = q + (r < kDHeads ? 0 : lo) + (size_t)(live ? h0 + h : 0) * pl.kp;
        const uint32_t dst = (uint32_t)__cvta_generic_to_shared(qh + (size_t)r * W);
        for (int c = lane; c < pl.kp / 8; c += 32) cp_async16_zfill_to(dst + c * 16, src + c * 8, live ? 16u : 0u);
    }
    load_tile(begin, max(begin, R.pos), begin + kDT);
    constexpr int MAXNB = 4;
    const int nb = pl.rp / (kDWarps * 8);  // 8-column blocks per warp (even)
    float o[MAXNB][4];
#pragma unroll
    for (int i = 0; i < MAXNB; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
    float m_run = -INFINITY, l_run = 0.0f;  // of head `warp`
    for (int t0 = begin; t0 < end; t0 += kDT) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const int live = min(kDT, end - t0);  // positions of this tile
        for (int pb = warp * 8; pb < live; pb += kDWarps * 8) {  // scores: eight positions per warp and round
            float s4[4][4] = {};  // four chains of MMAs
#pragma unroll 2
            for (int k0 = 0; k0 < pl.kp; k0 += 32) {
                uint32_t b[4], ah[4], al[4];
                ldmatrix_x4(b, tile + (size_t)(pb + (lane & 7)) * W + k0 + (lane >> 3) * 8);
#pragma unroll
                for (int kk = 0; kk < 2; ++kk) {
                    const size_t ao = (size_t)(lane & 15) * W + k0 + kk * 16 + (lane >> 4) * 8;
                    ldmatrix_x4(ah, qh + ao);
                    ldmatrix_x4(al, ql + ao);
                    mma_bf16(s4[2 * kk], ah, b[2 * kk], b[2 * kk + 1]);
                    mma_bf16(s4[2 * kk + 1], al, b[2 * kk], b[2 * kk + 1]);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e)
                sc[(g + (e >> 1) * 8) * kDT + pb + 2 * tq + (e & 1)] = (s4[0][e] + s4[1][e]) + (s4[2][e] + s4[3][e]);
        }
        __syncthreads();
        {   // softmax: warp w, head w
            float v[kDT / 32], mx = m_run, sum = 0.0f;
#pragma unroll
            for (int i = 0; i < kDT / 32; ++i) {
                v[i] = lane + 32 * i < live ? sc[warp * kDT + lane + 32 * i] : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
            mx = warp_max(mx);  // (position t0 is always live, so it is finite)
            const float cf = expf(m_run - mx);
#pragma unroll
            for (int i = 0; i < kDT / 32; ++i) {
                const float w = expf(v[i] - mx);
                sum += w;
                const uint16_t hi = f32_to_bf16_bits(w);
                ph[warp * (kDT + 8) + lane + 32 * i] = hi;
                plo[warp * (kDT + 8) + lane + 32 * i] = f32_to_bf16_bits(w - bf16_bits_to_f32(hi));
            }
            m_run = mx;
            l_run = l_run * cf + warp_sum(sum);
            if (lane == 0) corr[warp] = cf;
        }
        __syncthreads();
        {   // weighted latents: warp w, columns w * rp / 16 ..
            const float ca = corr[g], cb = corr[g + 8];
#pragma unroll
            for (int i = 0; i < MAXNB; ++i) { o[i][0] *= ca; o[i][1] *= ca; o[i][2] *= cb; o[i][3] *= cb; }
#pragma unroll
            for (int j = 0; j < kDT / 16; ++j) {
                if (j * 16 >= live) break;
                uint32_t ah[4], al[4], b[4];
                const int ao = (lane & 15) * (kDT + 8) + j * 16 + (lane >> 4) * 8;
                ldmatrix_x4(ah, ph + ao);
                ldmatrix_x4(al, plo + ao);
#pragma unroll
                for (int i = 0; i < MAXNB / 2; ++i) {
                    if (2 * i >= nb) break;
                    ldmatrix_x4_trans(b, tile + (size_t)(j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * W + warp * nb * 8 + i * 16 + (lane >> 4) * 8);
                    mma_bf16(o[2 * i], ah, b[0], b[1]);
                    mma_bf16(o[2 * i + 1], ah, b[2], b[3]);
                    mma_bf16(o[2 * i], al, b[0], b[1]);
                    mma_bf16(o[2 * i + 1], al, b[2], b[3]);
                }
            }
        }
        __syncthreads();
        if (t0 + kDT < end) load_tile(t0 + kDT, t0 + kDT, t0 + 2 * kDT);
    }
    // partial (weighted latent, maximum, sum) of this split
    float* const base = part + (size_t)split * a.heads * (a.rank + 2);
#pragma unroll
    for (int i = 0; i < MAXNB; ++i) {
        if (i >= nb) break;
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int h = h0 + g + (e >> 1) * 8, c = warp * nb * 8 + i * 8 + 2 * tq;
            if (h < a.heads && c < a.rank) {
                float* p = base + (size_t)h * (a.rank + 2) + c;
                if ((a.rank & 1) == 0) {
                    *reinterpret_cast<float2*>(p) = make_float2(o[i][e], o[i][e + 1]);
                } else {
                    p[0] = o[i][e];
                    if (c + 1 < a.rank) p[1] = o[i][e + 1];
                }
            }
        }
    }
    if (lane == 0 && h0 + warp < a.heads) {
        base[(size_t)(h0 + warp) * (a.rank + 2) + a.rank] = m_run;
        base[(size_t)(h0 + warp) * (a.rank + 2) + a.rank + 1] = l_run;
    }
}

// splits of a head merged, then W_uv: block (head, 64 values)
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatentArgs a, const float* __restrict__ part, int nsplit) {
    extern __shared__ float msm[];  // weighted latent [rank rounded up to 8] | split factors [kDMaxSplit]
    const int rp = round_up(a.rank, 8);
    float* const lat = msm;
    float* const f = msm + rp;
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    uint4 u[8][2];  // W_uv rows of this warp's eight values (rank <= 512), ahead of the dependency wait
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int v = blockIdx.y * 64 + warp + i * 8, r = lane * 8 + j * 256;
            u[i][j] = (v < a.vdim && r < rp) ? ld_stream_u4(a.uv + (size_t)(h * a.vdim + v) * a.ldu + r) : make_uint4(0u, 0u, 0u, 0u);
        }
    const DecodeRange R = decode_range(a.at->position, a.window, nsplit);  // (the position was written more than one launch ago)
    pdl_wait();
    const size_t hs = a.rank + 2, ss = (size_t)a.heads * hs;
    const float* p = part + (size_t)h * hs;
    // the splits' weighted latents of columns 2 tid, 2 tid + 1 (or tid, tid + 256 for an odd rank)
    float x[2][kDMaxSplit];
    const bool even = (a.rank & 1) == 0;
    const int c0 = even ? 2 * tid : tid, c1 = even ? 2 * tid + 1 : tid + 256;
#pragma unroll
    for (int s = 0; s < kDMaxSplit; ++s) {
        x[0][s] = x[1][s] = 0.0f;
        if (s < R.active) {
            if (even) {
                if (c0 < a.rank) {
                    const float2 t = *reinterpret_cast<const float2*>(p + s * ss + c0);
                    x[0][s] = t.x;
                    x[1][s] = t.y;
                }
            } else {
                if (c0 < a.rank) x[0][s] = p[s * ss + c0];
                if (c1 < a.rank) x[1][s] = p[s * ss + c1];
            }
        }
    }
    if (warp == 0) {
        const bool live = lane < R.active;
        const float m = live ? p[lane * ss + a.rank] : -INFINITY, l = live ? p[lane * ss + a.rank + 1] : 0.0f;
        const float mx = warp_max(m), w = live ? expf(m - mx) : 0.0f, total = warp_sum(w * l);
        f[lane] = w / total;
    }
    __syncthreads();
    {
        float v0 = 0.0f, v1 = 0.0f;
#pragma unroll
        for (int s = 0; s < kDMaxSplit; ++s) {
            v0 = fmaf(f[s], x[0][s], v0);
            v1 = fmaf(f[s], x[1][s], v1);
        }
        if (c0 < rp) lat[c0] = v0;
        if (c1 < rp) lat[c1] = v1;
    }
    __syncthreads();
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        acc[i] = 0.0f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int r = lane * 8 + j * 256;
            if (r < rp) {
                const uint32_t w[4] = {u[i][j].x, u[i][j].y, u[i][j].z, u[i][j].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[i] = fmaf(__uint_as_float(w[e] << 16), lat[r + 2 * e], acc[i]);
                    acc[i] = fmaf(__uint_as_float(w[e] & 0xffff0000u), lat[r + 2 * e + 1], acc[i]);
                }
            }
        }
    }
#pragma unroll
    for (int n = 4, off = 16; n >= 1; n >>= 1, off >>= 1) {  // eight sums over 32 lanes: lanes keep one half of them in each step
        const bool up = (lane & off) != 0;
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (i < n) {
                const float keep = up ? acc[i + n] : acc[i], give = up ? acc[i] : acc[i + n];
                acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
            }
    }
    acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 2);
    acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
    const int v = blockIdx.y * 64 + warp + (lane >> 2) * 8;
    if ((lane & 3) == 0 && v < a.vdim) a.out[(size_t)h * a.vdim + v] = acc[0];
}

// ---- prompt form ------------------------------------------------------------------------------------------------------------------
// One block: one head x 64 query rows (four warps of 16).  Key tiles of 64 positions, two in flight: the unrotated key part and
// the value from `expanded`, the rotated part from the cache.  q, k and v are bf16; scores and softmax f32; the weights are
// split into a bf16 head and remainder.
template <int DQ, int DV>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const LatentArgs a) {
    constexpr int PQ = DQ + 8, PV = DV + 8, BK = 64;
    constexpr float kLog2e = 1.4426950408889634f;
    extern __shared__ __align__(16) uint16_t fsm[];
    uint16_t* const qs = fsm;                      // [64][PQ]
    uint16_t* const ks = qs + 64 * PQ;             // [2][64][PQ]
    uint16_t* const vs = ks + 2 * BK * PQ;         // [2][64][PV]
    pdl_wait();
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int r0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 64;
    const int pos0 = a.pos0, half = a.rot >> 1, ro = round_up(a.dim, 8);  // the rotated part starts at an aligned column
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const uint16_t* ex = static_cast<const uint16_t*>(a.expanded);
    const uint16_t* cache = static_cast<const uint16_t*>(a.cache);
    const int kcol = h * a.dim, vcol = a.heads * a.dim + h * a.vdim;
    const bool fast = ((a.dim | a.rot | a.vdim | a.lde | a.pitch) & 7) == 0;
    const int last = pos0 + min(r0 + 64, a.T) - 1;  // newest position any row of this block sees
    // columns that no load writes stay zero
    for (int i = tid; i < (64 * PQ + 2 * BK * PQ + 2 * BK * PV) / 8; i += 128) reinterpret_cast<uint4*>(fsm)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int qw = a.dim + a.rot;
    if (fast && ((a.ld | a.q_off) & 7) == 0) {  // one run of eight entries at a time
        const int ru = a.dim >> 3;
        for (int r = warp; r < 64 && r0 + r < a.T; r += 4) {
            const uint16_t* row = in + (size_t)(r0 + r) * a.ld + a.q_off + (size_t)h * qw;
            for (int c = lane; c < ru; c += 32) *reinterpret_cast<uint4*>(qs + r * PQ + c * 8) = *reinterpret_cast<const uint4*>(row + c * 8);
        }
    } else {
        for (int i = tid; i < 64 * a.dim; i += 128) {
            const int r = i / a.dim, c = i - r * a.dim;
            if (r0 + r < a.T) qs[r * PQ + c] = in[(size_t)(r0 + r) * a.ld + a.q_off + (size_t)h * qw + c];
        }
    }
    for (int r = warp; r < 64 && r0 + r < a.T; r += 4) {
        const uint16_t* row = in + (size_t)(r0 + r) * a.ld + a.q_off + (size_t)h * qw + a.dim;
        const float2* cs = a.table + (size_t)(pos0 + r0 + r) * half;
        for (int j = lane; j < half; j += 32) {
            const float u = bf16_bits_to_f32(row[j]), v = bf16_bits_to_f32(row[j + half]);
            const float2 f = cs[j];
            qs[r * PQ + ro + j] = f32_to_bf16_bits(u * f.x - v * f.y);
            qs[r * PQ + ro + j + half] = f32_to_bf16_bits(v * f.x + u * f.y);
        }
    }
    auto load_tile = [&](int t0, int buf) {
        uint16_t* const kt = ks + buf * BK * PQ;
        uint16_t* const vt = vs + buf * BK * PV;
        if (fast) {
            const int ru = a.dim >> 3, rr = ru + (a.rot >> 3), rv = rr + (a.vdim >> 3);
            const int dr = 128 / rv, dc = 128 - dr * rv;
            for (int r = tid / rv, c = tid - r * rv; r < BK; r += dr, c += dc) {
                if (c >= rv) {
                    c -= rv;
                    if (++r >= BK) break;
                }
                const int p = t0 + r;
                const bool live = p <= last && p >= a.first;
                const uint16_t* src;
                uint16_t* dst;
                if (c < ru) { src = ex + (size_t)(p - a.first) * a.lde + kcol + c * 8; dst = kt + r * PQ + c * 8; }
                else if (c < rr) { src = cache + (size_t)p * a.pitch + a.kr_off + (c - ru) * 8; dst = kt + r * PQ + ro + (c - ru) * 8; }
                else { src = ex + (size_t)(p - a.first) * a.lde + vcol + (c - rr) * 8; dst = vt + r * PV + (c - rr) * 8; }
                cp_async16_zfill_to((uint32_t)__cvta_generic_to_shared(dst), live ? src : cache, live ? 16u : 0u);
            }
        } else {
            const int w = a.dim + a.rot + a.vdim;
            for (int i = tid; i < BK * w; i += 128) {
                const int r = i / w, c = i - r * w, p = t0 + r;
                const bool live = p <= last && p >= a.first;
                if (c < a.dim) kt[r * PQ + c] = live ? ex[(size_t)(p - a.first) * a.lde + kcol + c] : (uint16_t)0;
                else if (c < a.dim + a.rot) kt[r * PQ + ro + c - a.dim] = live ? cache[(size_t)p * a.pitch + a.kr_off + c - a.dim] : (uint16_t)0;
                else vt[r * PV + c - a.dim - a.rot] = live ? ex[(size_t)(p - a.first) * a.lde + vcol + c - a.dim - a.rot] : (uint16_t)0;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int row_a = r0 + warp * 16 + g, row_b = row_a + 8, pa = pos0 + row_a, pb = pos0 + row_b;
    const int lo_a = a.window > 0 ? pa - a.window + 1 : 0, lo_b = a.window > 0 ? pb - a.window + 1 : 0;
    const int warp_last = pos0 + r0 + warp * 16 + 15, warp_lo = a.window > 0 ? pos0 + r0 + warp * 16 - a.window + 1 : 0;
    const int first = a.window > 0 ? max(0, pos0 + r0 - a.window + 1) : 0;
    const float scale2 = a.scale * kLog2e;
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    load_tile(first, 0);
    int buf = 0;
#pragma unroll 1
    for (int t0 = first; t0 <= last; t0 += BK, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // tile t0 is here; the other buffer has been consumed
        if (t0 + BK <= last) load_tile(t0 + BK, buf ^ 1);
        if (t0 > warp_last || t0 + BK - 1 < warp_lo) continue;
        const uint16_t* const kt = ks + buf * BK * PQ;
        const uint16_t* const vt = vs + buf * BK * PV;
        float sacc[BK / 8][4];
#pragma unroll
        for (int i = 0; i < BK / 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) sacc[i][e] = 0.0f;
#pragma unroll
        for (int k = 0; k < DQ / 16; ++k) {
            uint32_t q[4], b[4];
            ldmatrix_x4(q, qs + (warp * 16 + (lane & 15)) * PQ + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int n2 = 0; n2 < BK / 16; ++n2) {
                ldmatrix_x4(b, kt + (n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * PQ + k * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(sacc[2 * n2], q, b[0], b[1]);
                mma_bf16(sacc[2 * n2 + 1], q, b[2], b[3]);
            }
        }
        float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
        for (int i = 0; i < BK / 8; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = t0 + i * 8 + 2 * tq + e;
                sacc[i][e] = (key <= pa && key >= lo_a) ? sacc[i][e] * scale2 : -INFINITY;
                sacc[i][2 + e] = (key <= pb && key >= lo_b) ? sacc[i][2 + e] * scale2 : -INFINITY;
                mx_a = fmaxf(mx_a, sacc[i][e]);
                mx_b = fmaxf(mx_b, sacc[i][2 + e]);
            }
#pragma unroll
        for (int off = 1; off <= 2; off <<= 1) {
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, off));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, off));
        }
        const float mn_a = fmaxf(m_run[0], mx_a), mn_b = fmaxf(m_run[1], mx_b);
        const float ma = mn_a == -INFINITY ? 0.0f : mn_a, mb = mn_b == -INFINITY ? 0.0f : mn_b;
        const float corr_a = ex2_approx(m_run[0] - ma), corr_b = ex2_approx(m_run[1] - mb);
        float ps_a = 0.0f, ps_b = 0.0f;
#pragma unroll
        for (int i = 0; i < BK / 8; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                sacc[i][e] = ex2_approx(sacc[i][e] - ma);
                sacc[i][2 + e] = ex2_approx(sacc[i][2 + e] - mb);
                ps_a += sacc[i][e];
                ps_b += sacc[i][2 + e];
            }
#pragma unroll
        for (int off = 1; off <= 2; off <<= 1) {
            ps_a += __shfl_xor_sync(0xffffffffu, ps_a, off);
            ps_b += __shfl_xor_sync(0xffffffffu, ps_b, off);
        }
        l_run[0] = l_run[0] * corr_a + ps_a;
        l_run[1] = l_run[1] * corr_b + ps_b;
        m_run[0] = mn_a;
        m_run[1] = mn_b;
        if (__any_sync(0xffffffffu, corr_a != 1.0f || corr_b != 1.0f)) {
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) { o[i][0] *= corr_a; o[i][1] *= corr_a; o[i][2] *= corr_b; o[i][3] *= corr_b; }
        }
#pragma unroll
        for (int j = 0; j < BK / 16; ++j) {
            uint32_t ph[4], pl[4], b[4];
            split_bf16x2(sacc[2 * j][0], sacc[2 * j][1], ph[0], pl[0]);
            split_bf16x2(sacc[2 * j][2], sacc[2 * j][3], ph[1], pl[1]);
            split_bf16x2(sacc[2 * j + 1][0], sacc[2 * j + 1][1], ph[2], pl[2]);
            split_bf16x2(sacc[2 * j + 1][2], sacc[2 * j + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int d2 = 0; d2 < DV / 16; ++d2) {
                ldmatrix_x4_trans(b, vt + (j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * PV + d2 * 16 + (lane >> 4) * 8);
                mma_bf16(o[2 * d2], ph, b[0], b[1]);
                mma_bf16(o[2 * d2 + 1], ph, b[2], b[3]);
                mma_bf16(o[2 * d2], pl, b[0], b[1]);
                mma_bf16(o[2 * d2 + 1], pl, b[2], b[3]);
            }
        }
    }
    const float inv_a = 1.0f / l_run[0], inv_b = 1.0f / l_run[1];
    const size_t ldo = (size_t)a.ldo;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int row = (e >> 1) ? row_b : row_a, c = i * 8 + 2 * tq + (e & 1);
            if (row < a.T && c < a.vdim) a.out[(size_t)row * ldo + (size_t)h * a.vdim + c] = o[i][e] * ((e >> 1) ? inv_b : inv_a);
        }
}

template <int DQ, int DV>
int run_prefill(cudaStream_t stream, const LatentArgs& a) {
    constexpr size_t smem = ((size_t)3 * 64 * (DQ + 8) + 2 * 64 * (DV + 8)) * 2;
    cudaError_t e = allow_all_dynamic_smem(latent_prefill_kernel<DQ, DV>);
    if (e == cudaSuccess) e = launch(latent_prefill_kernel<DQ, DV>, dim3(a.heads, (a.T + 63) / 64), dim3(128), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "latent attention (prompt): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace

int latent_write_cache(cudaStream_t stream, const LatentArgs& a) {
    auto k = a.in_f32 ? (a.cache_f32 ? latent_write_kernel<true, true> : latent_write_kernel<true, false>)
                      : (a.cache_f32 ? latent_write_kernel<false, true> : latent_write_kernel<false, false>);
    cudaError_t e = launch(k, dim3(a.T), dim3(128), 0, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "latent cache write: %s", cudaGetErrorString(e));
    return KMLL_OK;
}

int latent_attention_plain(cudaStream_t stream, const LatentArgs& a) {
    const size_t smem = ((size_t)(1 + kPlainWarps) * a.rank + a.rot) * 4;
    if (smem > 200 * 1024) return fail(KMLL_ERR_UNSUPPORTED, "latent attention: latent size %d is too large", a.rank);
    auto k = a.in_f32 ? (a.cache_f32 ? latent_plain_kernel<true, true> : latent_plain_kernel<true, false>)
                      : (a.cache_f32 ? latent_plain_kernel<false, true> : latent_plain_kernel<false, false>);
    cudaError_t e = allow_all_dynamic_smem(k);
    if (e == cudaSuccess) e = launch(k, dim3(a.T, a.heads), dim3(kPlainWarps * 32), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "latent attention (plain): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

static size_t decode_smem(const LatentDecodePlan& p) {
    return ((size_t)(kDT + 2 * kDHeads) * (p.width + 8) + 2 * (size_t)kDHeads * (kDT + 8)) * 2 + ((size_t)kDHeads * kDT + kDHeads) * 4;
}
size_t latent_decode_work_floats(int heads, int rank, int rot, int span) {
    const LatentDecodePlan p = decode_plan(heads, rank, rot, span);
    return p.q_floats + p.part_floats;
}
bool latent_decode_ok(const LatentArgs& a) {
    const LatentDecodePlan p = decode_plan(a.heads, a.rank, a.rot, 1);
    return a.T == 1 && !a.cache_f32 && a.in_f32 && a.at != nullptr && a.rank <= 512 && decode_smem(p) <= 220 * 1024 && a.dim <= 4096;
}
int latent_attention_decode(cudaStream_t stream, const LatentArgs& a) {
    const int span = a.window > 0 && a.window < a.max_seq ? a.window : a.max_seq;
    const LatentDecodePlan p = decode_plan(a.heads, a.rank, a.rot, span);
    uint16_t* const q = reinterpret_cast<uint16_t*>(a.work);
    const size_t lo = p.q_floats;  // elements: the remainders fill the second half of the area
    float* const part = a.work + p.q_floats;
    const size_t s1 = (size_t)(round_up(a.dim, 4) + 16 * 128) * 4, s3 = (size_t)(round_up(a.rank, 8) + kDMaxSplit) * 4;
    cudaError_t e = launch(latent_absorb_kernel, dim3(a.heads + 1, (a.rank + 127) / 128), dim3(256), s1, stream, true, a, q, lo, p.kp);
    if (e == cudaSuccess) e = allow_all_dynamic_smem(latent_decode_kernel);
    if (e == cudaSuccess) e = launch(latent_decode_kernel, dim3(p.nsplit, p.hgroups), dim3(kDWarps * 32), decode_smem(p), stream, true, a, (const uint16_t*)q, lo, part, p);
    if (e == cudaSuccess) e = launch(latent_merge_kernel, dim3(a.heads, (a.vdim + 63) / 64), dim3(256), s3, stream, true, a, (const float*)part, p.nsplit);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "latent attention (decode): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

bool latent_prefill_ok(const LatentArgs& a) { return !a.in_f32 && !a.cache_f32 && round_up(a.dim, 8) + a.rot <= 256 && a.vdim <= 128; }
int latent_attention_prefill(cudaStream_t stream, const LatentArgs& a) {
    if (!latent_prefill_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "latent attention: no prompt form for head sizes %d + %d, %d", a.dim, a.rot, a.vdim);
    const int dq = round_up(a.dim, 8) + a.rot;
    if (a.vdim <= 64) return dq <= 64 ? run_prefill<64, 64>(stream, a) : dq <= 128 ? run_prefill<128, 64>(stream, a) : dq <= 192 ? run_prefill<192, 64>(stream, a) : run_prefill<256, 64>(stream, a);
    return dq <= 64 ? run_prefill<64, 128>(stream, a) : dq <= 128 ? run_prefill<128, 128>(stream, a) : dq <= 192 ? run_prefill<192, 128>(stream, a) : run_prefill<256, 128>(stream, a);
}

}  // namespace kmll
