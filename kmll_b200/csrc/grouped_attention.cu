// Grouped softmax attention without rotation: query head h reads key / value head h / (heads / kv_heads); a position sees itself
// and the earlier positions of its window, of its chunk, or of the whole sequence.  The cache row of a position holds the keys
// of every key / value head, then the values, each head padded to a multiple of 8 entries (the padding is zero).
//
//   plain form    any size, f32 arithmetic, one block per (token, head): decoders that compute in f32, sizes the others lack
//   decode form   one token over the bf16 cache: up to 16 query heads of a group are the rows of the MMAs, so the cache is read
//                 once per group; positions split over the blocks of a cluster, which merge their parts through shared memory
//   prompt form   tiled attention with online softmax over the cache rows
// Scores and weights are f32; the weights (and in a decode step the queries) meet the tensor cores split into a bf16 head and
// remainder.
#include "internal.cuh"
#include "mma_bf16.cuh"

namespace kmll {

namespace {

template <bool F32>
__device__ inline float val(const void* p, size_t i) {
    return F32 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
__host__ __device__ inline int round_to(int v, int m) { return (v + m - 1) / m * m; }
// first position that position `pos` sees
__device__ inline int first_seen(int pos, int window, int chunk) {
    int lo = 0;
    if (window > 0) lo = max(lo, pos - window + 1);
    if (chunk > 0) lo = max(lo, pos - pos % chunk);
    return lo;
}

template <bool IN32, bool C32>
__global__ void __launch_bounds__(128) grouped_write_kernel(const GroupedArgs a) {
    pdl_wait();
    const int pos = (a.at != nullptr ? a.at->position : a.pos0) + blockIdx.x;
    if (pos >= a.max_seq) return;
    const size_t in = (size_t)blockIdx.x * a.ld, row = (size_t)pos * a.pitch;
    const int nk = a.kv_heads * a.dim, n = nk + a.kv_heads * a.vdim;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const bool is_k = i < nk;
        const int j = is_k ? i : i - nk, len = is_k ? a.dim : a.vdim, g = j / len;
        const float v = val<IN32>(a.in, in + (is_k ? a.k_off : a.v_off) + j);
        const size_t at = row + (is_k ? g * a.dimp : a.kv_heads * a.dimp + g * a.vdimp) + (j - g * len);
        if (C32) static_cast<float*>(a.cache)[at] = v;
        else static_cast<uint16_t*>(a.cache)[at] = f32_to_bf16_bits(v);
    }
}

// ---- plain form -----------------------------------------------------------------------------------------------------------------
constexpr int kPlainWarps = 4;
template <bool IN32, bool C32>
__global__ void __launch_bounds__(kPlainWarps * 32) grouped_plain_kernel(const GroupedArgs a) {
    extern __shared__ float psm[];
    float* const q = psm;                 // [dim]
    float* const acc = q + a.dim;         // [warps][vdim]
    __shared__ float stat[2 * kPlainWarps];
    pdl_wait();
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = h / (a.heads / a.kv_heads);
    const int pos = (a.at != nullptr ? a.at->position : a.pos0) + t;
    for (int i = tid; i < a.dim; i += blockDim.x) q[i] = val<IN32>(a.in, (size_t)t * a.ld + a.q_off + (size_t)h * a.dim + i);
    for (int i = tid; i < kPlainWarps * a.vdim; i += blockDim.x) acc[i] = 0.0f;
    __syncthreads();
    float m = -INFINITY, l = 0.0f;
    float* const mine = acc + warp * a.vdim;
    for (int j = first_seen(pos, a.window, a.chunk) + warp; j <= pos; j += kPlainWarps) {
        const size_t k = (size_t)j * a.pitch + (size_t)g * a.dimp, v = (size_t)j * a.pitch + (size_t)a.kv_heads * a.dimp + (size_t)g * a.vdimp;
        float s = 0.0f;
        for (int i = lane; i < a.dim; i += 32) s = fmaf(q[i], val<C32>(a.cache, k + i), s);
        s = warp_sum(s) * a.scale;
        const float mn = fmaxf(m, s), corr = expf(m - mn), w = expf(s - mn);
        m = mn;
        l = l * corr + w;
        for (int i = lane; i < a.vdim; i += 32) mine[i] = mine[i] * corr + w * val<C32>(a.cache, v + i);
    }
    if (lane == 0) { stat[warp] = m; stat[kPlainWarps + warp] = l; }
    __syncthreads();
    float mx = -INFINITY, total = 0.0f, f[kPlainWarps];
    for (int w = 0; w < kPlainWarps; ++w) mx = fmaxf(mx, stat[w]);
    for (int w = 0; w < kPlainWarps; ++w) {
        f[w] = stat[w] == -INFINITY ? 0.0f : expf(stat[w] - mx);
        total += f[w] * stat[kPlainWarps + w];
    }
    for (int i = tid; i < a.vdim; i += blockDim.x) {
        float s = 0.0f;
        for (int w = 0; w < kPlainWarps; ++w) s += f[w] * acc[w * a.vdim + i];
        a.out[(size_t)t * a.ldo + (size_t)h * a.vdim + i] = s / total;
    }
}

// ---- decode form ------------------------------------------------------------------------------------------------------------------
constexpr int kDT = 160;     // positions per tile
constexpr int kDRows = 16;   // query heads per block = MMA rows
constexpr int kDWarps = 8;
constexpr int kDMaxSplit = 16;
constexpr int kDMinPart = 32;  // positions per split at least
struct GroupedPlan { int tiles_per_group, tiles, kw, vw; };
__host__ __device__ inline GroupedPlan decode_plan(int heads, int kv_heads, int dim, int vdim) {
    GroupedPlan p;
    p.tiles_per_group = (heads / kv_heads + kDRows - 1) / kDRows;
    p.tiles = kv_heads * p.tiles_per_group;
    p.kw = round_to(dim, 32);
    p.vw = round_to(vdim, 16);
    return p;
}
size_t decode_smem(const GroupedPlan& p) {
    return ((size_t)(kDT + 2 * kDRows) * (p.kw + 8) + (size_t)kDT * (p.vw + 8) + 2 * (size_t)kDRows * (kDT + 8)) * 2 +
           ((size_t)kDRows * kDT + kDRows + (size_t)kDRows * kDMaxSplit) * 4;
}

__device__ inline uint32_t cluster_rank() {
    uint32_t r;
    asm("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ inline uint32_t cluster_size() {
    uint32_t r;
    asm("mov.u32 %0, %%cluster_nctaid.x;" : "=r"(r));
    return r;
}
__device__ inline void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// the float at `p` (this block's shared memory) in block `rank` of the cluster
__device__ inline float cluster_load(const float* p, uint32_t rank) {
    uint32_t at;
    float v;
    asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(at) : "memory");
    return v;
}

// One cluster per (key / value head, 16 query heads); its blocks share the positions.
__global__ void __launch_bounds__(kDWarps * 32) grouped_decode_kernel(const GroupedArgs a, const GroupedPlan pl) {
    extern __shared__ __align__(16) uint16_t dsm[];
    const int KP = pl.kw + 8, VP = pl.vw + 8;
    uint16_t* const kt = dsm;                    // [kDT][KP]
    uint16_t* const vt = kt + kDT * KP;          // [kDT][VP]
    uint16_t* const qh = vt + kDT * VP;          // [16][KP]
    uint16_t* const ql = qh + kDRows * KP;
    uint16_t* const ph = ql + kDRows * KP;       // [16][kDT + 8]
    uint16_t* const plo = ph + kDRows * (kDT + 8);
    float* const sc = reinterpret_cast<float*>(plo + kDRows * (kDT + 8));  // [16][kDT]
    float* const corr = sc + kDRows * kDT;       // [16]
    float* const f = corr + kDRows;              // [16][kDMaxSplit]
    __shared__ float stat[2 * kDRows];           // maximum and sum of this block's part, per row
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int split = (int)cluster_rank(), nsplit = (int)cluster_size(), grp = blockIdx.y / pl.tiles_per_group, sub = blockIdx.y % pl.tiles_per_group;
    const int per = a.heads / a.kv_heads, h0 = grp * per + sub * kDRows, nh = min(kDRows, per - sub * kDRows);
    // the position was written more than one launch ago, and so was every cache row but the newest
    const int pos = a.at->position, lo = first_seen(pos, a.window, a.chunk), count = pos - lo + 1;
    const int part_len = max((count + nsplit - 1) / nsplit, kDMinPart), active = (count + part_len - 1) / part_len;
    const int begin = lo + split * part_len, end = split < active ? min(begin + part_len, pos + 1) : begin;
    uint16_t* const cache = static_cast<uint16_t*>(a.cache);
    const size_t k0 = (size_t)grp * a.dimp, v0 = (size_t)a.kv_heads * a.dimp + (size_t)grp * a.vdimp;
    auto load_tile = [&](int t0) {  // rows behind the last position are zeros; the newest one comes from the projection
        const int rows = min(kDT, round_to(end - t0, 16)), rk = pl.kw / 8, runs = rk + pl.vw / 8;
        for (int r = warp; r < rows; r += kDWarps) {
            const int p = t0 + r;
            if (p == pos) continue;
            const uint16_t* src = cache + (size_t)min(p, pos) * a.pitch;
            for (int c = lane; c < runs; c += 32) {
                const bool is_k = c < rk;
                const int col = (is_k ? c : c - rk) * 8;
                const bool live = p < end && col < (is_k ? a.dimp : a.vdimp);
                const uint32_t dst = (uint32_t)__cvta_generic_to_shared(is_k ? kt + r * KP + col : vt + r * VP + col);
                cp_async16_zfill_to(dst, live ? src + (is_k ? k0 : v0) + col : cache, live ? 16u : 0u);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (begin < end) load_tile(begin);
    pdl_wait();
    const float* in = static_cast<const float*>(a.in);
    auto put_newest = [&](int t0) {
        if (pos < t0 || pos >= min(t0 + kDT, end)) return;
        const int r = pos - t0;
        for (int i = tid; i < pl.kw + pl.vw; i += kDWarps * 32) {
            const bool is_k = i < pl.kw;
            const int c = is_k ? i : i - pl.kw;
            const bool live = c < (is_k ? a.dim : a.vdim);
            const uint16_t v = live ? f32_to_bf16_bits(in[is_k ? a.k_off + grp * a.dim + c : a.v_off + grp * a.vdim + c]) : (uint16_t)0;
            if (is_k) kt[r * KP + c] = v;
            else vt[r * VP + c] = v;
            if (live && sub == 0 && pos < a.max_seq) cache[(size_t)pos * a.pitch + (is_k ? k0 : v0) + c] = v;
        }
    };
    for (int i = tid; i < kDRows * pl.kw; i += kDWarps * 32) {  // queries (times the score factor), head and remainder
        const int r = i / pl.kw, c = i - r * pl.kw;
        const float v = r < nh && c < a.dim ? in[a.q_off + (size_t)(h0 + r) * a.dim + c] * a.scale : 0.0f;
        const uint16_t hi = f32_to_bf16_bits(v);
        qh[r * KP + c] = hi;
        ql[r * KP + c] = f32_to_bf16_bits(v - bf16_bits_to_f32(hi));
    }
    constexpr int NG = 2;  // groups of 16 value columns per warp (vdim <= 256)
    float o[NG][2][4];
#pragma unroll
    for (int i = 0; i < NG; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][j][e] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};  // of rows `warp` and `warp + 8`
    for (int t0 = begin; t0 < end; t0 += kDT) {
        if (t0 > begin) load_tile(t0);
        put_newest(t0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const int live = min(kDT, end - t0);
        for (int pb = warp * 8; pb < live; pb += kDWarps * 8) {  // scores: eight positions per warp and round
            float s4[4][4] = {};
#pragma unroll 2
            for (int k = 0; k < pl.kw; k += 32) {
                uint32_t b[4], ah[4], al[4];
                ldmatrix_x4(b, kt + (size_t)(pb + (lane & 7)) * KP + k + (lane >> 3) * 8);
#pragma unroll
                for (int kk = 0; kk < 2; ++kk) {
                    const size_t ao = (size_t)(lane & 15) * KP + k + kk * 16 + (lane >> 4) * 8;
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
#pragma unroll
        for (int i = 0; i < 2; ++i) {  // softmax: warp w, rows w and w + 8
            const int r = warp + i * 8;
            float v[kDT / 32], mx = m_run[i], sum = 0.0f;
#pragma unroll
            for (int j = 0; j < kDT / 32; ++j) {
                v[j] = lane + 32 * j < live ? sc[r * kDT + lane + 32 * j] : -INFINITY;
                mx = fmaxf(mx, v[j]);
            }
            mx = warp_max(mx);  // (position t0 is always live, so it is finite)
            const float cf = expf(m_run[i] - mx);
#pragma unroll
            for (int j = 0; j < kDT / 32; ++j) {
                const float w = expf(v[j] - mx);
                sum += w;
                const uint16_t hi = f32_to_bf16_bits(w);
                ph[r * (kDT + 8) + lane + 32 * j] = hi;
                plo[r * (kDT + 8) + lane + 32 * j] = f32_to_bf16_bits(w - bf16_bits_to_f32(hi));
            }
            m_run[i] = mx;
            l_run[i] = l_run[i] * cf + warp_sum(sum);
            if (lane == 0) corr[r] = cf;
        }
        __syncthreads();
        const float ca = corr[g], cb = corr[g + 8];
#pragma unroll
        for (int i = 0; i < NG; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) { o[i][j][0] *= ca; o[i][j][1] *= ca; o[i][j][2] *= cb; o[i][j][3] *= cb; }
#pragma unroll
        for (int j = 0; j < kDT / 16; ++j) {
            if (j * 16 >= live) break;
            uint32_t ah[4], al[4], b[4];
            const int ao = (lane & 15) * (kDT + 8) + j * 16 + (lane >> 4) * 8;
            ldmatrix_x4(ah, ph + ao);
            ldmatrix_x4(al, plo + ao);
#pragma unroll
            for (int i = 0; i < NG; ++i) {
                const int c = (warp + i * kDWarps) * 16;
                if (c >= pl.vw) break;
                ldmatrix_x4_trans(b, vt + (size_t)(j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * VP + c + (lane >> 4) * 8);
                mma_bf16(o[i][0], ah, b[0], b[1]);
                mma_bf16(o[i][1], ah, b[2], b[3]);
                mma_bf16(o[i][0], al, b[0], b[1]);
                mma_bf16(o[i][1], al, b[2], b[3]);
            }
        }
        __syncthreads();
    }
    // ---- the blocks' parts: (weighted values, maximum, sum) in shared memory, merged slice by slice
    float* const part = reinterpret_cast<float*>(dsm);  // [16][vw], in the place of the key tile
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            stat[warp + i * 8] = m_run[i];
            stat[kDRows + warp + i * 8] = l_run[i];
        }
    }
#pragma unroll
    for (int i = 0; i < NG; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int c = (warp + i * kDWarps) * 16 + j * 8 + 2 * tq;
                if (c < pl.vw) *reinterpret_cast<float2*>(part + (g + (e >> 1) * 8) * pl.vw + c) = make_float2(o[i][j][e], o[i][j][e + 1]);
            }
    cluster_sync();
    for (int r = warp; r < nh; r += kDWarps) {
        const bool on = lane < active;
        const float m = on ? cluster_load(stat + r, lane) : -INFINITY, l = on ? cluster_load(stat + kDRows + r, lane) : 0.0f;
        const float mx = warp_max(m), w = on ? expf(m - mx) : 0.0f, sum = warp_sum(w * l);
        if (lane < kDMaxSplit) f[r * kDMaxSplit + lane] = w / sum;
    }
    __syncthreads();
    const int outs = nh * a.vdim, slice = (outs + nsplit - 1) / nsplit;
    for (int i = split * slice + tid; i < min((split + 1) * slice, outs); i += kDWarps * 32) {
        const int r = i / a.vdim, c = i - r * a.vdim;
        float x[kDMaxSplit], v = 0.0f;
#pragma unroll
        for (int s = 0; s < kDMaxSplit; ++s) x[s] = s < active ? cluster_load(part + r * pl.vw + c, s) : 0.0f;
#pragma unroll
        for (int s = 0; s < kDMaxSplit; ++s) v = fmaf(s < active ? f[r * kDMaxSplit + s] : 0.0f, x[s], v);
        a.out[(size_t)(h0 + r) * a.vdim + c] = v;
    }
    cluster_sync();  // (no block leaves while another reads its part)
}

// ---- prompt form --------------------------------------------------------------------------------------------------------------------
// One block: one head x 64 query rows (four warps of 16), key tiles of 64 positions, two in flight.
template <int DQ, int DV>
__global__ void __launch_bounds__(128) grouped_prefill_kernel(const GroupedArgs a) {
    constexpr int PQ = DQ + 8, PV = DV + 8, BK = 64;
    constexpr float kLog2e = 1.4426950408889634f;
    extern __shared__ __align__(16) uint16_t fsm[];
    uint16_t* const qs = fsm;                      // [64][PQ]
    uint16_t* const ks = qs + 64 * PQ;             // [2][64][PQ]
    uint16_t* const vs = ks + 2 * BK * PQ;         // [2][64][PV]
    pdl_wait();
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int r0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 64, pos0 = a.pos0, grp = h / (a.heads / a.kv_heads);
    const uint16_t* in = static_cast<const uint16_t*>(a.in);
    const uint16_t* cache = static_cast<const uint16_t*>(a.cache);
    const size_t k0 = (size_t)grp * a.dimp, v0 = (size_t)a.kv_heads * a.dimp + (size_t)grp * a.vdimp;
    const int last = pos0 + min(r0 + 64, a.T) - 1;  // newest position any row of this block sees
    if (((a.dim | a.ld | a.q_off) & 7) == 0) {
        for (int i = tid; i < 64 * (DQ / 8); i += 128) {
            const int r = i / (DQ / 8), c = (i % (DQ / 8)) * 8;
            *reinterpret_cast<uint4*>(qs + r * PQ + c) = r0 + r < a.T && c < a.dim
                ? *reinterpret_cast<const uint4*>(in + (size_t)(r0 + r) * a.ld + a.q_off + (size_t)h * a.dim + c) : make_uint4(0u, 0u, 0u, 0u);
        }
    } else {
        for (int i = tid; i < 64 * DQ; i += 128) {
            const int r = i / DQ, c = i % DQ;
            qs[r * PQ + c] = r0 + r < a.T && c < a.dim ? in[(size_t)(r0 + r) * a.ld + a.q_off + (size_t)h * a.dim + c] : (uint16_t)0;
        }
    }
    auto load_tile = [&](int t0, int buf) {
        constexpr int RK = DQ / 8, RUNS = RK + DV / 8;
        for (int i = tid; i < BK * RUNS; i += 128) {
            const int r = i / RUNS, c = i % RUNS, p = t0 + r;
            const bool is_k = c < RK;
            const int col = (is_k ? c : c - RK) * 8;
            const bool live = p <= last && col < (is_k ? a.dimp : a.vdimp);
            const uint16_t* src = live ? cache + (size_t)p * a.pitch + (is_k ? k0 : v0) + col : cache;
            uint16_t* dst = is_k ? ks + (buf * BK + r) * PQ + col : vs + (buf * BK + r) * PV + col;
            cp_async16_zfill_to((uint32_t)__cvta_generic_to_shared(dst), src, live ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int row_a = r0 + warp * 16 + g, row_b = row_a + 8, pa = pos0 + row_a, pb = pos0 + row_b;
    const int lo_a = first_seen(pa, a.window, a.chunk), lo_b = first_seen(pb, a.window, a.chunk);
    const int warp_last = min(pos0 + r0 + warp * 16 + 15, last), warp_lo = first_seen(pos0 + r0 + warp * 16, a.window, a.chunk);
    const int first = first_seen(pos0 + r0, a.window, a.chunk);
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
    const bool v2 = ((a.ldo | a.vdim) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 7u) == 0;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int row = (e >> 1) ? row_b : row_a, c = i * 8 + 2 * tq;
            const float inv = (e >> 1) ? inv_b : inv_a;
            if (row >= a.T || c >= a.vdim) continue;
            float* p = a.out + (size_t)row * a.ldo + (size_t)h * a.vdim + c;
            if (v2) {
                *reinterpret_cast<float2*>(p) = make_float2(o[i][e] * inv, o[i][e + 1] * inv);
            } else {
                p[0] = o[i][e] * inv;
                if (c + 1 < a.vdim) p[1] = o[i][e + 1] * inv;
            }
        }
}

template <int DQ, int DV>
int run_prefill(cudaStream_t stream, const GroupedArgs& a) {
    constexpr size_t smem = ((size_t)3 * 64 * (DQ + 8) + 2 * 64 * (DV + 8)) * 2;
    cudaError_t e = allow_all_dynamic_smem(grouped_prefill_kernel<DQ, DV>);
    if (e == cudaSuccess) e = launch(grouped_prefill_kernel<DQ, DV>, dim3(a.heads, (a.T + 63) / 64), dim3(128), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped attention (prompt): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace

int grouped_write_cache(cudaStream_t stream, const GroupedArgs& a) {
    auto k = a.in_f32 ? (a.cache_f32 ? grouped_write_kernel<true, true> : grouped_write_kernel<true, false>)
                      : (a.cache_f32 ? grouped_write_kernel<false, true> : grouped_write_kernel<false, false>);
    cudaError_t e = launch(k, dim3(a.T), dim3(128), 0, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped cache write: %s", cudaGetErrorString(e));
    return KMLL_OK;
}

int grouped_attention_plain(cudaStream_t stream, const GroupedArgs& a) {
    const size_t smem = ((size_t)a.dim + (size_t)kPlainWarps * a.vdim) * 4;
    if (smem > 200 * 1024) return fail(KMLL_ERR_UNSUPPORTED, "grouped attention: head sizes %d, %d are too large", a.dim, a.vdim);
    auto k = a.in_f32 ? (a.cache_f32 ? grouped_plain_kernel<true, true> : grouped_plain_kernel<true, false>)
                      : (a.cache_f32 ? grouped_plain_kernel<false, true> : grouped_plain_kernel<false, false>);
    cudaError_t e = allow_all_dynamic_smem(k);
    if (e == cudaSuccess) e = launch(k, dim3(a.T, a.heads), dim3(kPlainWarps * 32), smem, stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped attention (plain): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

bool grouped_decode_ok(const GroupedArgs& a) {
    const GroupedPlan p = decode_plan(a.heads, a.kv_heads, a.dim, a.vdim);
    return a.T == 1 && !a.cache_f32 && a.in_f32 && a.at != nullptr && a.vdim <= 16 * 2 * kDWarps && p.tiles <= 65535 && decode_smem(p) <= 220 * 1024;
}
// Blocks per cluster: 16 where all clusters are resident at once with it, else the portable 8.
static int decode_cluster(const GroupedPlan& p, size_t smem, int* out) {
    *out = 8;
    if (p.tiles * 16 > 148) return KMLL_OK;
    cudaError_t e = cudaFuncSetAttribute(grouped_decode_kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped attention (decode): %s", cudaGetErrorString(e));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(16, p.tiles);
    cfg.blockDim = dim3(kDWarps * 32);
    cfg.dynamicSmemBytes = smem;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 16;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    int clusters = 0;
    if (cudaOccupancyMaxActiveClusters(&clusters, grouped_decode_kernel, &cfg) != cudaSuccess) {
        cudaGetLastError();  // (a device that has no such clusters)
        clusters = 0;
    }
    if (clusters >= p.tiles) *out = 16;
    return KMLL_OK;
}
int grouped_attention_decode(cudaStream_t stream, const GroupedArgs& a) {
    if (!grouped_decode_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "grouped attention: no decode form for %d / %d heads of %d, %d", a.heads, a.kv_heads, a.dim, a.vdim);
    const GroupedPlan p = decode_plan(a.heads, a.kv_heads, a.dim, a.vdim);
    const size_t smem = decode_smem(p);
    cudaError_t e = allow_all_dynamic_smem(grouped_decode_kernel);
    int cluster = 8;
    if (e == cudaSuccess) KMLL_TRY_RC(decode_cluster(p, smem, &cluster));
    if (e == cudaSuccess) e = launch_cluster(grouped_decode_kernel, dim3(cluster, p.tiles), cluster, dim3(kDWarps * 32), smem, stream, true, a, p);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped attention (decode): %s", cudaGetErrorString(e));
    return KMLL_OK;
}

bool grouped_prefill_ok(const GroupedArgs& a) { return !a.in_f32 && !a.cache_f32 && a.dim <= 256 && a.vdim <= 128; }
int grouped_attention_prefill(cudaStream_t stream, const GroupedArgs& a) {
    if (!grouped_prefill_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "grouped attention: no prompt form for head sizes %d, %d", a.dim, a.vdim);
    if (a.vdim <= 64) return a.dim <= 64 ? run_prefill<64, 64>(stream, a) : a.dim <= 128 ? run_prefill<128, 64>(stream, a) : run_prefill<256, 64>(stream, a);
    return a.dim <= 64 ? run_prefill<64, 128>(stream, a) : a.dim <= 128 ? run_prefill<128, 128>(stream, a) : run_prefill<256, 128>(stream, a);
}

}  // namespace kmll
