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

// bf16 rows whose heads are multiples of 8 entries: 16 bytes per thread
__global__ void __launch_bounds__(256) grouped_copy_kernel(const GroupedArgs a) {
    pdl_wait();
    const int nk = a.kv_heads * a.dim / 8, runs = nk + a.kv_heads * a.vdim / 8;
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    const int t = (int)(i / runs), j = (int)(i - (long long)t * runs);
    if (t >= a.T || a.pos0 + t >= a.max_seq) return;
    const uint16_t* src = static_cast<const uint16_t*>(a.in) + (size_t)t * a.ld + (j < nk ? a.k_off + j * 8 : a.v_off + (j - nk) * 8);
    *reinterpret_cast<uint4*>(static_cast<uint16_t*>(a.cache) + (size_t)(a.pos0 + t) * a.pitch + j * 8) = *reinterpret_cast<const uint4*>(src);
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
// One cluster of eight blocks per (key / value head, 16 query heads).  The positions are cut into steps of 16, dealt out to the
// warps of all blocks; a warp keeps its own running softmax and weighted values, so nothing but the query is shared until the
// warps, and then the blocks, merge their parts.
constexpr int kDRows = 16;     // query heads per block = MMA rows
constexpr int kDStep = 16;     // positions per step of a warp
constexpr int kDCluster = 8;
inline int decode_tiles(const GroupedArgs& a) { return a.kv_heads * ((a.heads / a.kv_heads + kDRows - 1) / kDRows); }
__host__ __device__ constexpr int decode_warps(int KW, int VW) { return KW + VW > 256 ? 8 : 16; }
__host__ __device__ constexpr size_t decode_smem(int KW, int VW) {
    const int NW = decode_warps(KW, VW), steps = NW * kDStep * (KW + VW + 16) * 2, parts = NW * kDRows * VW * 4;
    return (size_t)2 * kDRows * (KW + 8) * 2 + (steps > parts ? steps : parts) + (size_t)kDRows * VW * 4;
}

__device__ inline uint32_t cluster_rank() {
    uint32_t r;
    asm("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
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

template <int KW, int VW>
__global__ void __launch_bounds__(decode_warps(KW, VW) * 32) grouped_decode_kernel(const GroupedArgs a) {
    constexpr int NW = decode_warps(KW, VW), KP = KW + 8, VP = VW + 8;
    extern __shared__ __align__(16) uint16_t dsm[];
    uint16_t* const qh = dsm;                    // [16][KP]
    uint16_t* const ql = qh + kDRows * KP;
    uint16_t* const steps = ql + kDRows * KP;    // per warp: keys [16][KP], values [16][VP]; later the warps' parts [NW][16][VW] f32
    float* const res = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(dsm) + decode_smem(KW, VW)) - kDRows * VW;  // [16][VW]
    __shared__ float warp_max_[NW][kDRows], warp_sum_[NW][kDRows], stat[2 * kDRows], f[kDRows * kDCluster];
    __shared__ uint16_t newest[KW + VW];  // key and value of the newest position
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
    const int per = a.heads / a.kv_heads, tiles = (per + kDRows - 1) / kDRows;
    const int split = (int)cluster_rank(), grp = blockIdx.y / tiles, sub = blockIdx.y % tiles;
    const int h0 = grp * per + sub * kDRows, nh = min(kDRows, per - sub * kDRows);
    // the position was written more than one launch ago, and so was every cache row but the newest
    const int pos = a.at->position, lo = first_seen(pos, a.window, a.chunk), n_steps = (pos - lo + kDStep) / kDStep;
    uint16_t* const cache = static_cast<uint16_t*>(a.cache);
    const size_t k0 = (size_t)grp * a.dimp, v0 = (size_t)a.kv_heads * a.dimp + (size_t)grp * a.vdimp;
    uint16_t* const kt = steps + warp * kDStep * (KP + VP);
    uint16_t* const vt = kt + kDStep * KP;
    auto load_step = [&](int st) {  // rows behind the last position are zeros; the newest one comes from the projection
        constexpr int RK = KW / 8, RUNS = RK + VW / 8;
        const int p0 = lo + st * kDStep;
#pragma unroll
        for (int i0 = 0; i0 < kDStep * RUNS; i0 += 32) {
            const int i = i0 + lane, r = i / RUNS, c = i % RUNS, p = p0 + r;
            const bool is_k = c < RK;
            const int col = (is_k ? c : c - RK) * 8;
            if (p == pos) continue;
            const bool live = p < pos && col < (is_k ? a.dimp : a.vdimp);
            const uint32_t dst = (uint32_t)__cvta_generic_to_shared(is_k ? kt + r * KP + col : vt + r * VP + col);
            cp_async16_zfill_to(dst, live ? cache + (size_t)p * a.pitch + (is_k ? k0 : v0) + col : cache, live ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    int st = split + warp * kDCluster;
    if (st < n_steps) load_step(st);
    pdl_wait();
    const float* in = static_cast<const float*>(a.in);
    for (int i = tid; i < kDRows * KW; i += NW * 32) {  // queries (times the score factor), head and remainder
        const int r = i / KW, c = i % KW;
        const float v = r < nh && c < a.dim ? in[a.q_off + (size_t)(h0 + r) * a.dim + c] * a.scale : 0.0f;
        const uint16_t hi = f32_to_bf16_bits(v);
        qh[r * KP + c] = hi;
        ql[r * KP + c] = f32_to_bf16_bits(v - bf16_bits_to_f32(hi));
    }
    if ((n_steps - 1) % kDCluster == split)  // (the block that reads the newest position)
        for (int i = tid; i < KW + VW; i += NW * 32) {
            const bool is_k = i < KW;
            const int c = is_k ? i : i - KW;
            const bool live = c < (is_k ? a.dim : a.vdim);
            const uint16_t v = live ? f32_to_bf16_bits(in[is_k ? a.k_off + grp * a.dim + c : a.v_off + grp * a.vdim + c]) : (uint16_t)0;
            newest[i] = v;
            if (live && sub == 0 && pos < a.max_seq) cache[(size_t)pos * a.pitch + (is_k ? k0 : v0) + c] = v;
        }
    __syncthreads();
    float o[VW / 8][4];
#pragma unroll
    for (int i = 0; i < VW / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};  // of rows g and g + 8
    for (; st < n_steps; st += kDCluster * NW) {
        const int p0 = lo + st * kDStep;
        if (pos < p0 + kDStep)  // the newest position is the last of the last step
            for (int i = lane; i < KW + VW; i += 32) (i < KW ? kt + (pos - p0) * KP : vt + (pos - p0) * VP - KW)[i] = newest[i];
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncwarp();
        float s[2][4] = {}, s2[2][4] = {};  // scores: heads, remainders of the query
#pragma unroll
        for (int k = 0; k < KW / 16; ++k) {
            uint32_t b[4], ah[4], al[4];
            ldmatrix_x4(b, kt + ((lane >> 4) * 8 + (lane & 7)) * KP + k * 16 + ((lane >> 3) & 1) * 8);
            ldmatrix_x4(ah, qh + (lane & 15) * KP + k * 16 + (lane >> 4) * 8);
            ldmatrix_x4(al, ql + (lane & 15) * KP + k * 16 + (lane >> 4) * 8);
            mma_bf16(s[0], ah, b[0], b[1]);
            mma_bf16(s[1], ah, b[2], b[3]);
            mma_bf16(s2[0], al, b[0], b[1]);
            mma_bf16(s2[1], al, b[2], b[3]);
        }
        float mx[2] = {m_run[0], m_run[1]};
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[i][e] = p0 + i * 8 + 2 * tq + (e & 1) <= pos ? s[i][e] + s2[i][e] : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
            }
#pragma unroll
        for (int y = 0; y < 2; ++y) {
            mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 1));
            mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 2));  // (the step's first position is always seen, so it is finite)
        }
        const float ca = expf(m_run[0] - mx[0]), cb = expf(m_run[1] - mx[1]);
        float sum[2] = {0.0f, 0.0f};
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[i][e] = expf(s[i][e] - mx[e >> 1]);
                sum[e >> 1] += s[i][e];
            }
#pragma unroll
        for (int y = 0; y < 2; ++y) {
            sum[y] += __shfl_xor_sync(0xffffffffu, sum[y], 1);
            sum[y] += __shfl_xor_sync(0xffffffffu, sum[y], 2);
            m_run[y] = mx[y];
        }
        l_run[0] = l_run[0] * ca + sum[0];
        l_run[1] = l_run[1] * cb + sum[1];
        uint32_t ph[4], pl[4];
        split_bf16x2(s[0][0], s[0][1], ph[0], pl[0]);
        split_bf16x2(s[0][2], s[0][3], ph[1], pl[1]);
        split_bf16x2(s[1][0], s[1][1], ph[2], pl[2]);
        split_bf16x2(s[1][2], s[1][3], ph[3], pl[3]);
#pragma unroll
        for (int d2 = 0; d2 < VW / 16; ++d2) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, vt + (((lane >> 3) & 1) * 8 + (lane & 7)) * VP + d2 * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                float (&c)[4] = o[2 * d2 + i];
                c[0] *= ca; c[1] *= ca; c[2] *= cb; c[3] *= cb;
                mma_bf16(c, ph, b[2 * i], b[2 * i + 1]);
                mma_bf16(c, pl, b[2 * i], b[2 * i + 1]);
            }
        }
        __syncwarp();
        if (st + kDCluster * NW < n_steps) load_step(st + kDCluster * NW);
    }
    // ---- the warps' parts -> this block's (weighted values, maximum, sum)
    if (tq == 0) {
        warp_max_[warp][g] = m_run[0];
        warp_max_[warp][g + 8] = m_run[1];
        warp_sum_[warp][g] = l_run[0];
        warp_sum_[warp][g + 8] = l_run[1];
    }
    __syncthreads();  // every step has been read
    float* const parts = reinterpret_cast<float*>(steps);
#pragma unroll
    for (int i = 0; i < VW / 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int r = g + (e >> 1) * 8;
            if (r < nh) *reinterpret_cast<float2*>(parts + (warp * kDRows + r) * VW + i * 8 + 2 * tq) = make_float2(o[i][e], o[i][e + 1]);
        }
    if (warp < kDRows && lane < NW)
        for (int r = warp; r < nh; r += NW) {  // lane w: warp w's factor of row r
            const float m = warp_max_[lane][r];
            float mx = m;
#pragma unroll
            for (int off = NW / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync((1u << (NW - 1)) * 2u - 1u, mx, off));
            const float w = m == -INFINITY ? 0.0f : expf(m - mx);
            float l = w * warp_sum_[lane][r];
#pragma unroll
            for (int off = NW / 2; off > 0; off >>= 1) l += __shfl_xor_sync((1u << (NW - 1)) * 2u - 1u, l, off);
            warp_sum_[lane][r] = w;  // (read above by this lane only)
            if (lane == 0) { stat[r] = mx; stat[kDRows + r] = l; }
        }
    __syncthreads();
    for (int i = tid; i < nh * VW; i += NW * 32) {
        const int r = i / VW, c = i % VW;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < NW; ++w) v = fmaf(warp_sum_[w][r], parts[(w * kDRows + r) * VW + c], v);
        res[i] = v;
    }
    cluster_sync();
    // ---- the blocks' parts, a slice of the outputs each
    for (int i = tid; i < nh * kDCluster; i += NW * 32) f[i] = cluster_load(stat + i / kDCluster, i % kDCluster);
    const int outs = nh * a.vdim, slice = (outs + kDCluster - 1) / kDCluster;
    __syncthreads();
    for (int i = split * slice + tid; i < min((split + 1) * slice, outs); i += NW * 32) {
        const int r = i / a.vdim, c = i - r * a.vdim;
        float x[kDCluster], l[kDCluster], mx = -INFINITY, v = 0.0f, total = 0.0f;
#pragma unroll
        for (int s = 0; s < kDCluster; ++s) {
            x[s] = cluster_load(res + r * VW + c, s);
            l[s] = cluster_load(stat + kDRows + r, s);
            mx = fmaxf(mx, f[r * kDCluster + s]);
        }
#pragma unroll
        for (int s = 0; s < kDCluster; ++s) {
            const float m = f[r * kDCluster + s], w = m == -INFINITY ? 0.0f : expf(m - mx);
            v = fmaf(w, x[s], v);
            total = fmaf(w, l[s], total);
        }
        a.out[(size_t)(h0 + r) * a.vdim + c] = v / total;
    }
    cluster_sync();  // (no block leaves while another reads its part)
}

template <int KW, int VW>
int run_decode(cudaStream_t stream, const GroupedArgs& a) {
    cudaError_t e = allow_all_dynamic_smem(grouped_decode_kernel<KW, VW>);
    if (e == cudaSuccess)
        e = launch_cluster(grouped_decode_kernel<KW, VW>, dim3(kDCluster, decode_tiles(a)), kDCluster, dim3(decode_warps(KW, VW) * 32), decode_smem(KW, VW), stream, true, a);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped attention (decode): %s", cudaGetErrorString(e));
    return KMLL_OK;
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
    if (!a.in_f32 && !a.cache_f32 && a.at == nullptr && ((a.dim | a.vdim | a.ld | a.k_off | a.v_off) & 7) == 0 && (reinterpret_cast<uintptr_t>(a.in) & 15u) == 0) {
        const long long items = (long long)a.T * a.kv_heads * (a.dim + a.vdim) / 8;
        cudaError_t e = launch(grouped_copy_kernel, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, stream, true, a);
        if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "grouped cache write: %s", cudaGetErrorString(e));
        return KMLL_OK;
    }
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
    return a.T == 1 && !a.cache_f32 && a.in_f32 && a.at != nullptr && a.dim <= 256 && a.vdim <= 256 && decode_tiles(a) <= 65535;
}
int grouped_attention_decode(cudaStream_t stream, const GroupedArgs& a) {
    if (!grouped_decode_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "grouped attention: no decode form for %d / %d heads of %d, %d", a.heads, a.kv_heads, a.dim, a.vdim);
    if (a.dim <= 64) return a.vdim <= 64 ? run_decode<64, 64>(stream, a) : a.vdim <= 128 ? run_decode<64, 128>(stream, a) : run_decode<64, 256>(stream, a);
    if (a.dim <= 128) return a.vdim <= 64 ? run_decode<128, 64>(stream, a) : a.vdim <= 128 ? run_decode<128, 128>(stream, a) : run_decode<128, 256>(stream, a);
    return a.vdim <= 64 ? run_decode<256, 64>(stream, a) : a.vdim <= 128 ? run_decode<256, 128>(stream, a) : run_decode<256, 256>(stream, a);
}

bool grouped_prefill_ok(const GroupedArgs& a) { return !a.in_f32 && !a.cache_f32 && a.dim <= 256 && a.vdim <= 128; }
int grouped_attention_prefill(cudaStream_t stream, const GroupedArgs& a) {
    if (!grouped_prefill_ok(a)) return fail(KMLL_ERR_UNSUPPORTED, "grouped attention: no prompt form for head sizes %d, %d", a.dim, a.vdim);
    if (a.vdim <= 64) return a.dim <= 64 ? run_prefill<64, 64>(stream, a) : a.dim <= 128 ? run_prefill<128, 64>(stream, a) : run_prefill<256, 64>(stream, a);
    return a.dim <= 64 ? run_prefill<64, 128>(stream, a) : a.dim <= 128 ? run_prefill<128, 128>(stream, a) : run_prefill<256, 128>(stream, a);
}

}  // namespace kmll
