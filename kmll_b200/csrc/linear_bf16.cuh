// Linear layers over bf16 weights (KMLL_FORMAT_BF16: rows as a checkpoint stores them, at a pitch of a multiple of 8
// elements), included by linear.cu.  Used by the layered decoders.
//
//   bf16_matvec_kernel   one row of x (decode): f32 activations, f32 accumulation, with the step before the projection
//                        (norm, PolyNorm, gate of a mixer's output) as a prologue and residual / SiLU / arg-max as epilogues
//   linear_gemm_bf16_kernel  many rows of x (prefill) in bf16 on tcgen05: TMA, tensor memory, persistent
//   gemm_f32_kernel      many rows of x with f32 activations on the CUDA cores (every product and sum in f32)
#pragma once

#include <cuda.h>

#include <algorithm>

#include "activations.cuh"

namespace kmll {

// ---- one row of x -------------------------------------------------------------------------------------------------------
// Block b owns a contiguous, evenly cut range of output rows; its 16 warps split K into pieces of 256 columns (512 bytes of a
// weight row: one 16-byte copy per lane).  The copies go through a lane-private shared-memory ring (a lane reads back exactly
// what its own copies wrote, so cp.async.wait_group is the only synchronisation), and the first kVDepth of them are issued
// before the dependency wait because weights never change.  A warp keeps 16 rows of partial sums in registers, folds them
// across its lanes with 16 shuffles, and leaves them in shared memory; one block barrier before the epilogue is all the
// synchronisation of the main loop.
constexpr int kVWarps = 16;
constexpr int kVThreads = kVWarps * 32;
constexpr int kVRows = 16;     // rows whose sums a warp holds in registers
constexpr int kVDepth = 8;     // 16-byte copies in flight per lane (64 KB per block, two blocks per SM)
constexpr int kVPiece = 256;   // columns per warp and step

// index of column k in the staged vector: two planes, so that the 16-byte reads of a warp are free of bank conflicts
__device__ inline int vec_slot(int k, int half) { return ((k >> 2) & 1) * half + ((k >> 3) << 2) + (k & 3); }

// three block sums at once; every thread gets them (scratch: 16 * 3 + 3 floats)
__device__ inline void block_sum3(float (&v)[3], float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
    for (int i = 0; i < 3; ++i) v[i] = warp_sum(v[i]);
    __syncthreads();
    if (lane == 0)
#pragma unroll
        for (int i = 0; i < 3; ++i) scratch[i * 32 + warp] = v[i];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        float t = lane < nw ? scratch[i * 32 + lane] : 0.0f;
        v[i] = warp_sum(t);
    }
}

struct MatvecArgs {
    Bf16Matvec a;
    int half, kpieces, rows_cap, n_heads;  // n_heads: of all segments
    int off_x, off_part, off_head;  // byte offsets in shared memory (the ring is at 0)
};

__global__ void __launch_bounds__(kVThreads, 2) bf16_matvec_kernel(const MatvecArgs p) {
    extern __shared__ __align__(16) unsigned char vsmem[];
    __shared__ float scratch[96];
    __shared__ unsigned int s_last;
    const Bf16Matvec& a = p.a;
    float* const xs = reinterpret_cast<float*>(vsmem + p.off_x);
    float* const part = reinterpret_cast<float*>(vsmem + p.off_part);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int unit = a.pair_act != 0 ? 2 : 1, units = a.rows / unit;
    const int r0 = unit * (int)((long long)blockIdx.x * units / gridDim.x), r1 = unit * (int)((long long)(blockIdx.x + 1) * units / gridDim.x);
    const int nrows = r1 - r0, ngroups = (nrows + kVRows - 1) / kVRows;
    const int mine = p.kpieces > warp ? (p.kpieces - warp + kVWarps - 1) / kVWarps : 0;  // pieces of this warp
    const uint32_t ring = smem_u32(vsmem) + (uint32_t)tid * 16u;

    // requests: piece `ci` of row `r` of group `g`; rows or columns that do not exist are zero-filled without a read
    auto request = [&](int g, int ci, int r) {
        const int k = (warp + ci * kVWarps) * kVPiece + lane * 8, row = g * kVRows + r;
        const bool live = g < ngroups && row < nrows && k < a.ldw;
        const uint16_t* src = live ? a.w + (size_t)(r0 + row) * a.ldw + k : a.w;
        asm volatile("cp.async.cg.shared.global.L2::128B [%0], [%1], 16, %2;" ::"r"(ring + (uint32_t)(r % kVDepth) * (kVThreads * 16)), "l"(src),
                     "r"(live ? 16u : 0u)
                     : "memory");
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (mine > 0)
#pragma unroll
        for (int r = 0; r < kVDepth; ++r) request(0, 0, r);

    pdl_wait();
    // ---- x -> shared memory through the prologue; columns K .. are zeros
    const int kpad = p.kpieces * kVPiece;
    if (a.pro == PRO_NORM && a.norm.kind == KMLL_NORM_LAYER) {
        float s = 0.0f;
        int n = 0;
        for (int k = tid; k < kpad; k += kVThreads) {
            const float v = k < a.K ? a.x[k] : 0.0f;
            if (k < a.K) { s += v; ++n; }
            xs[vec_slot(k, p.half)] = v;
        }
        Moments m{(float)n, n > 0 ? s / (float)n : 0.0f, 0.0f};
        for (int k = tid; k < a.K; k += kVThreads) {
            const float v = xs[vec_slot(k, p.half)] - m.mean;
            m.dev += v * v;
        }
        m = block_moments(m, scratch);
        const float inv = inv_rms(m.dev, a.K, a.norm.eps);
        for (int k = tid; k < a.K; k += kVThreads)
            xs[vec_slot(k, p.half)] = (xs[vec_slot(k, p.half)] - m.mean) * inv * (a.norm.offset + bf16_bits_to_f32(a.norm.w[k])) + bf16_bits_to_f32(a.norm.b[k]);
    } else if (a.pro == PRO_NORM) {
        float s = 0.0f;
        for (int k = tid; k < kpad; k += kVThreads) {
            const float v = k < a.K ? a.x[k] : 0.0f;
            s += v * v;
            xs[vec_slot(k, p.half)] = v;
        }
        const float inv = inv_rms(block_sum(s, scratch), a.K, a.norm.eps);
        for (int k = tid; k < a.K; k += kVThreads) xs[vec_slot(k, p.half)] *= inv * (a.norm.offset + bf16_bits_to_f32(a.norm.w[k]));
    } else if (a.pro == PRO_POLYNORM) {
        float s[3] = {0.0f, 0.0f, 0.0f};
        for (int k = tid; k < kpad; k += kVThreads) {
            const float v = k < a.K ? a.x[k] : 0.0f, v2 = v * v;
            s[0] += v2;
            s[1] += v2 * v2;
            s[2] += v2 * v2 * v2;
            xs[vec_slot(k, p.half)] = v;
        }
        block_sum3(s, scratch);
        const float c1 = bf16_bits_to_f32(a.coef[0]) * inv_rms(s[0], a.K, a.eps), c2 = bf16_bits_to_f32(a.coef[1]) * inv_rms(s[1], a.K, a.eps),
                    c3 = bf16_bits_to_f32(a.coef[2]) * inv_rms(s[2], a.K, a.eps), c0 = bf16_bits_to_f32(a.coef[3]);
        for (int k = tid; k < a.K; k += kVThreads) {
            const float v = xs[vec_slot(k, p.half)];
            xs[vec_slot(k, p.half)] = ((c3 * v + c2) * v + c1) * v + c0;
        }
    } else if (a.pro == PRO_GATED) {
        float s[kMaxSegments] = {};
        for (int k = tid; k < kpad; k += kVThreads) {
            const float v = k < a.K ? a.x[k] : 0.0f;
#pragma unroll
            for (int j = 0; j < kMaxSegments; ++j)
                if (j < a.n_seg && k >= a.seg[j].begin && k < a.seg[j].begin + a.seg[j].cols) s[j] += v * v;
            xs[vec_slot(k, p.half)] = v;
        }
        float* const hinv = reinterpret_cast<float*>(vsmem + p.off_head);  // one entry per head of the segments that norm by head
        int heads0 = 0;
        float joint[kMaxSegments] = {};
        __syncthreads();
#pragma unroll
        for (int j = 0; j < kMaxSegments; ++j) {
            if (j >= a.n_seg) break;
            const GateSegment& g = a.seg[j];
            if (g.norm == KMLL_OUT_NORM_JOINT) {
                joint[j] = inv_rms(block_sum(s[j], scratch), g.cols, g.eps);
            } else if (g.norm != KMLL_OUT_NORM_NONE) {
                const int nh = g.cols / g.head_len;
                for (int h = warp; h < nh; h += kVWarps) {
                    float t = 0.0f;
                    for (int i = lane; i < g.head_len; i += 32) {
                        const float v = xs[vec_slot(g.begin + h * g.head_len + i, p.half)];
                        t += v * v;
                    }
                    t = warp_sum(t);
                    if (lane == 0) hinv[heads0 + h] = inv_rms(t, g.head_len, g.eps);
                }
                heads0 += nh;
            }
        }
        __syncthreads();
        heads0 = 0;
        int covered = 0;
#pragma unroll
        for (int j = 0; j < kMaxSegments; ++j) {
            if (j >= a.n_seg) break;
            const GateSegment& g = a.seg[j];
            for (int k = covered + tid; k < g.begin; k += kVThreads) xs[vec_slot(k, p.half)] = 0.0f;
            covered = g.begin + g.cols;
            const float* const gate = static_cast<const float*>(g.gate);
            for (int i = tid; i < g.cols; i += kVThreads) {
                float f = g.scale;
                if (g.norm == KMLL_OUT_NORM_JOINT) {
                    f *= joint[j] * bf16_bits_to_f32(g.norm_w[i]);
                } else if (g.norm != KMLL_OUT_NORM_NONE) {
                    const int h = i / g.head_len;
                    f *= hinv[heads0 + h];
                    if (g.norm == KMLL_OUT_NORM_HEAD_WEIGHTED) f *= bf16_bits_to_f32(g.norm_w[i - h * g.head_len]);
                }
                if (gate != nullptr) f *= apply_act(gate[g.gate_len == 1 ? i : i / g.gate_len], g.act);
                xs[vec_slot(g.begin + i, p.half)] *= f;
            }
            if (g.norm == KMLL_OUT_NORM_PER_HEAD || g.norm == KMLL_OUT_NORM_HEAD_WEIGHTED) heads0 += g.cols / g.head_len;
        }
        for (int k = covered + tid; k < a.K; k += kVThreads) xs[vec_slot(k, p.half)] = 0.0f;
    } else {
        for (int k = tid; k < kpad; k += kVThreads) xs[vec_slot(k, p.half)] = k < a.K ? a.x[k] : 0.0f;
    }
    __syncthreads();

    // ---- main loop
    if (mine > 0) {
        int ng = 0, nc = 0;  // group / piece of the request that follows the ring
        for (int g = 0; g < ngroups; ++g) {
            float acc[kVRows];
#pragma unroll
            for (int r = 0; r < kVRows; ++r) acc[r] = 0.0f;
            for (int ci = 0; ci < mine; ++ci) {
                const int k8 = ((warp + ci * kVWarps) * kVPiece >> 3) + lane;
                const float4 xa = *reinterpret_cast<const float4*>(xs + k8 * 4), xb = *reinterpret_cast<const float4*>(xs + p.half + k8 * 4);
                ng = g;
                nc = ci + 1;
                if (nc == mine) { nc = 0; ng = g + 1; }
#pragma unroll
                for (int r = 0; r < kVRows; ++r) {
                    asm volatile("cp.async.wait_group %0;" ::"n"(kVDepth - 1) : "memory");
                    const uint4 w = *reinterpret_cast<const uint4*>(vsmem + (size_t)(r % kVDepth) * (kVThreads * 16) + (size_t)tid * 16);
                    if (r + kVDepth < kVRows) request(g, ci, r + kVDepth);
                    else request(ng, nc, r + kVDepth - kVRows);
                    float2 s = make_float2(acc[r], 0.0f);
                    s = __ffma2_rn(make_float2(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xffff0000u)), make_float2(xa.x, xa.y), s);
                    s = __ffma2_rn(make_float2(__uint_as_float(w.y << 16), __uint_as_float(w.y & 0xffff0000u)), make_float2(xa.z, xa.w), s);
                    s = __ffma2_rn(make_float2(__uint_as_float(w.z << 16), __uint_as_float(w.z & 0xffff0000u)), make_float2(xb.x, xb.y), s);
                    s = __ffma2_rn(make_float2(__uint_as_float(w.w << 16), __uint_as_float(w.w & 0xffff0000u)), make_float2(xb.z, xb.w), s);
                    acc[r] = s.x + s.y;
                }
            }
            // fold 16 sums over 32 lanes: lanes keep one half of the rows in each step
#pragma unroll
            for (int n = kVRows / 2, off = 16; n >= 1; n >>= 1, off >>= 1) {
                const bool up = (lane & off) != 0;
#pragma unroll
                for (int i = 0; i < kVRows / 2; ++i)
                    if (i < n) {
                        const float keep = up ? acc[i + n] : acc[i], give = up ? acc[i] : acc[i + n];
                        acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
                    }
            }
            const float total = acc[0] + __shfl_xor_sync(0xffffffffu, acc[0], 1);
            if ((lane & 1) == 0) part[warp * p.rows_cap + g * kVRows + (lane >> 1)] = total;
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();

    // ---- epilogue: the warps' sums in warp order
    const int nw = p.kpieces < kVWarps ? p.kpieces : kVWarps;
    float best = -INFINITY;
    uint32_t best_row = 0xffffffffu;
    if (a.pair_act != 0) {
        for (int r = 2 * tid; r < nrows; r += 2 * kVThreads) {
            float gate = 0.0f, v = 0.0f;
            for (int w = 0; w < nw; ++w) {
                const float2 t = *reinterpret_cast<const float2*>(part + w * p.rows_cap + r);
                gate += t.x;
                v += t.y;
            }
            a.y[(r0 + r) >> 1] = apply_act(gate, a.pair_act) * v;
        }
        return;
    }
    for (int r = tid; r < nrows; r += kVThreads) {
        float v = 0.0f;
        for (int w = 0; w < nw; ++w) v += part[w * p.rows_cap + r];
        const int row = r0 + r;
        if (row < a.silu_rows) v = act_silu(v);
        v *= a.out_scale;
        if (a.residual != nullptr) v += a.residual[row];
        a.y[row] = v;
        if (top1_better(v, (uint32_t)row, best, best_row)) { best = v; best_row = (uint32_t)row; }
    }
    if (a.packed == nullptr) return;
    // arg-max: per-block result, merged by the block that arrives last, which also ends the decode step
    auto fold = [&](float& v, uint32_t& t) {
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, off);
            const uint32_t ot = __shfl_xor_sync(0xffffffffu, t, off);
            if (top1_better(ov, ot, v, t)) { v = ov; t = ot; }
        }
    };
    uint32_t* const stok = reinterpret_cast<uint32_t*>(scratch + 32);
    auto block_best = [&]() {
        fold(best, best_row);
        __syncthreads();
        if (lane == 0) { scratch[warp] = best; stok[warp] = best_row; }
        __syncthreads();
        if (warp == 0) {
            best = lane < kVWarps ? scratch[lane] : -INFINITY;
            best_row = lane < kVWarps ? stok[lane] : 0xffffffffu;
            fold(best, best_row);
        }
    };
    block_best();
    if (tid == 0) {
        a.part_logit[blockIdx.x] = best;
        a.part_tok[blockIdx.x] = best_row;
        __threadfence();
        s_last = atomicAdd(a.counter, 1u) == gridDim.x - 1 ? 1u : 0u;
    }
    __syncthreads();
    if (s_last == 0u) return;
    __threadfence();
    best = -INFINITY;
    best_row = 0xffffffffu;
    for (int b = tid; b < (int)gridDim.x; b += kVThreads) {
        const float v = __ldcg(a.part_logit + b);
        const uint32_t t = __ldcg(a.part_tok + b);
        if (top1_better(v, t, best, best_row)) { best = v; best_row = t; }
    }
    block_best();
    if (tid == 0) {
        *a.counter = 0u;
        if (best_row >= (uint32_t)a.rows) best_row = 0u;  // (all logits NaN)
        a.packed[0] = pack_top1(best, best_row);
        if (a.state != nullptr) {
            a.state->next_top = pack_top1(best, best_row);
            a.state->position += 1;
            a.state->step += 1;
        }
    }
}

int bf16_matvec(cudaStream_t stream, const Bf16Matvec& a) {
    if (a.rows <= 0 || a.K <= 0 || a.ldw < a.K || (a.ldw & 7) != 0) return fail(KMLL_ERR_SHAPE, "bf16_matvec: rows %d, K %d, pitch %d", a.rows, a.K, a.ldw);
    MatvecArgs p;
    memset(&p, 0, sizeof(p));
    p.a = a;
    p.kpieces = (a.K + kVPiece - 1) / kVPiece;
    p.half = p.kpieces * kVPiece / 2;
    if (a.pair_act != 0 && ((a.rows & 1) != 0 || a.packed != nullptr || a.residual != nullptr)) return fail(KMLL_ERR_SHAPE, "bf16_matvec: %d rows are not pairs", a.rows);
    p.n_heads = 0;
    for (int j = 0; a.pro == PRO_GATED && j < a.n_seg; ++j)
        if (a.seg[j].norm == KMLL_OUT_NORM_PER_HEAD || a.seg[j].norm == KMLL_OUT_NORM_HEAD_WEIGHTED) p.n_heads += a.seg[j].cols / a.seg[j].head_len;
    const size_t ring = (size_t)kVDepth * kVThreads * 16, xbytes = (size_t)p.kpieces * kVPiece * 4, hbytes = ((size_t)p.n_heads * 4 + 15) & ~(size_t)15;
    p.off_x = (int)ring;
    p.off_head = (int)(ring + xbytes);
    p.off_part = (int)(ring + xbytes + hbytes);
    // one block per SM, fewer for small matrices (at least 4 rows each), more when the partial sums would not fit
    int grid = a.rows / 4 < 148 ? (a.rows + 3) / 4 : 148;
    size_t smem = 0;
    for (;; grid += 148) {
        const int unit = a.pair_act != 0 ? 2 : 1;
        p.rows_cap = (unit * ((a.rows / unit + grid - 1) / grid) + kVRows - 1) / kVRows * kVRows;
        smem = ring + xbytes + hbytes + (size_t)kVWarps * p.rows_cap * 4;
        if (smem <= 220 * 1024) break;
        if (p.rows_cap <= kVRows) return fail(KMLL_ERR_UNSUPPORTED, "bf16_matvec: in_dim %d does not fit in shared memory", a.K);
    }
    if (a.packed != nullptr && grid > kMatvecMaxBlocks) return fail(KMLL_ERR_UNSUPPORTED, "bf16_matvec: %d output rows are too many for the arg-max", a.rows);
    cudaError_t e = allow_all_dynamic_smem(bf16_matvec_kernel);
    if (e == cudaSuccess) e = launch(bf16_matvec_kernel, dim3(grid), dim3(kVThreads), smem, stream, true, p);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "bf16_matvec: %s", cudaGetErrorString(e));
    return KMLL_OK;
}

// ---- many rows of x, bf16, tcgen05 -----------------------------------------------------------------------------------------
// y[t, r] = sum_k W[r, k] x[t, k].  128 weight rows are the M side of the MMA (tensor-memory lanes), up to 256 rows of x the
// N side, so a warp's stores of one row of x are 32 consecutive outputs.  Both operands come by TMA (128-byte swizzle, columns
// beyond K zero-filled); persistent blocks walk the tiles, two accumulators in tensor memory let the epilogue of a tile
// overlap the MMAs of the next.  Tensor maps cover this GPU's memory only, no multicast; every wait is bounded and a time-out
// raises the device status word.  Few tiles with a long K are cut into K pieces, one block each; the block that arrives last adds
// the partial tiles in the order of the pieces.
constexpr int kHRows = 128, kHMaxN = 256, kHKT = 64;
constexpr int kHEpiWarps = 8;
constexpr int kHThreads = (2 + kHEpiWarps) * 32;  // warp 0: TMA, warp 1: MMA, warps 2..9: epilogue

struct GemmBf16Params {
    int rows, K, T, n_block, stages, row_tiles, x_tiles, tiles, ksplit;
    void* out;
    int out_bf16, ldo, silu_rows, pair_act;
    float out_scale;
    const float* residual;
    float* partial;          // ksplit > 1 (one item per block): [tiles][ksplit][n_block][128]
    unsigned int* counters;  // [tiles], zero between launches
};

__host__ __device__ constexpr uint32_t gemm_idesc_bf16(int m, int n) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

__global__ void __launch_bounds__(kHThreads, 1) linear_gemm_bf16_kernel(const GemmBf16Params p, const __grid_constant__ CUtensorMap map_w,
                                                                       const __grid_constant__ CUtensorMap map_x) {
    extern __shared__ unsigned char hsmem_raw[];
    unsigned char* hsmem = hsmem_raw + ((1024u - (smem_u32(hsmem_raw) & 1023u)) & 1023u);
    const int stages = p.stages;
    const int a_bytes = kHRows * 128, b_bytes = p.n_block * 128, stage_bytes = a_bytes + b_bytes;  // multiples of 1024
    uint64_t* full = reinterpret_cast<uint64_t*>(hsmem + (size_t)stages * stage_bytes);
    uint64_t* empty = full + stages;
    uint64_t* acc_full = empty + stages;  // [2]
    uint64_t* acc_free = acc_full + 2;    // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_free + 2);
    __shared__ unsigned int s_last;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int KT = (p.K + kHKT - 1) / kHKT, kt_per = (KT + p.ksplit - 1) / p.ksplit, items = p.tiles * p.ksplit;

    if (tid == 0) {
        for (int s = 0; s < stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&acc_full[b], 1); mbar_init(&acc_free[b], kHEpiWarps); }
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t smem_base = smem_u32(hsmem);
    const uint32_t idesc = gemm_idesc_bf16(kHRows, p.n_block);

    pdl_wait();
    bool ok = true;
    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            for (int item = blockIdx.x; ok && item < items; item += gridDim.x) {
                const int tile = item / p.ksplit, kt0 = (item % p.ksplit) * kt_per, kt1 = min(kt0 + kt_per, KT);
                const int row0 = (tile / p.x_tiles) * kHRows, t0 = (tile % p.x_tiles) * p.n_block;
#pragma unroll 1
                for (int kt = kt0; kt < kt1; ++kt, ++it) {
                    const int s = it % stages, use = it / stages;
                    if (use > 0 && !mbar_wait<false>(&empty[s], (uint32_t)(use - 1) & 1u)) { ok = false; break; }
                    const uint32_t st = smem_base + (uint32_t)s * stage_bytes;
                    mbar_arrive_expect_tx(&full[s], (uint32_t)stage_bytes);
                    tma_load_2d(st, &map_w, kt * kHKT, row0, &full[s]);
                    tma_load_2d(st + a_bytes, &map_x, kt * kHKT, t0, &full[s]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int it = 0, n = 0;
            for (int item = blockIdx.x; ok && item < items; item += gridDim.x, ++n) {
                const int buf = n & 1, kt0 = (item % p.ksplit) * kt_per, kt1 = min(kt0 + kt_per, KT);
                if (n >= 2 && !mbar_wait<false>(&acc_free[buf], (uint32_t)((n >> 1) - 1) & 1u)) { ok = false; break; }
                tcgen05_fence_after();
                const uint32_t acc = tmem_base + (uint32_t)buf * 256u;
#pragma unroll 1
                for (int kt = kt0; kt < kt1; ++kt, ++it) {
                    const int s = it % stages, use = it / stages;
                    if (!mbar_wait<false>(&full[s], (uint32_t)use & 1u)) { ok = false; break; }
                    tcgen05_fence_after();
                    const uint32_t st = smem_base + (uint32_t)s * stage_bytes;
#pragma unroll
                    for (int ks = 0; ks < kHKT / 16; ++ks)
                        gemm_mma_f16(acc, gemm_smem_desc(st + ks * 32), gemm_smem_desc(st + a_bytes + ks * 32), idesc, (kt > kt0 || ks > 0) ? 1u : 0u);
                    umma_commit(&empty[s]);
                }
                if (ok) umma_commit(&acc_full[buf]);
            }
        }
    } else {
        const int q = warp & 3, half = (warp - 2) >> 2;  // lane quarter this warp may read; which half of the columns
        const int rl = q * 32 + lane;
        auto finish = [&](int t, int row, float v, bool act) {
            const size_t o = (size_t)t * p.ldo + row;
            if (act) v = act_silu(v);
            v *= p.out_scale;
            if (p.residual != nullptr) v += p.residual[o];
            if (p.out_bf16) static_cast<uint16_t*>(p.out)[o] = f32_to_bf16_bits(v);
            else static_cast<float*>(p.out)[o] = v;
        };
        int n = 0;
        for (int item = blockIdx.x; item < items; item += gridDim.x, ++n) {
            const int buf = n & 1, tile = item / p.ksplit;
            float* const part = p.ksplit > 1 ? p.partial + (size_t)item * p.n_block * kHRows : nullptr;
            const int row0 = (tile / p.x_tiles) * kHRows, t0 = (tile % p.x_tiles) * p.n_block;
            if (!mbar_wait<true>(&acc_full[buf], (uint32_t)(n >> 1) & 1u)) ok = false;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tcgen05_fence_after();
            const int row = row0 + rl, ncols = p.n_block / 2;
            const bool live = row < p.rows, act = row < p.silu_rows;
#pragma unroll 1
            for (int c0 = half * ncols; c0 < (half + 1) * ncols; c0 += 8) {
                if (t0 + c0 >= p.T) break;
                uint32_t d[8];
                const uint32_t taddr = tmem_base + (uint32_t)buf * 256u + ((uint32_t)(q * 32) << 16) + (uint32_t)c0;
                asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                             : "=r"(d[0]), "=r"(d[1]), "=r"(d[2]), "=r"(d[3]), "=r"(d[4]), "=r"(d[5]), "=r"(d[6]), "=r"(d[7])
                             : "r"(taddr)
                             : "memory");
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    if (part != nullptr) {
                        part[(size_t)(c0 + j) * kHRows + rl] = __uint_as_float(d[j]);
                    } else if (p.pair_act != 0) {  // even lanes hold the gate, odd lanes its value
                        const float v = __shfl_xor_sync(0xffffffffu, __uint_as_float(d[j]), 1);
                        if (live && (lane & 1) == 0 && t0 + c0 + j < p.T) finish(t0 + c0 + j, row >> 1, apply_act(__uint_as_float(d[j]), p.pair_act) * v, false);
                    } else if (live && t0 + c0 + j < p.T) finish(t0 + c0 + j, row, __uint_as_float(d[j]), act);
                }
            }
            tcgen05_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_free[buf]);
            if (part != nullptr) {  // (this block's only item)
                __threadfence();
                asm volatile("bar.sync 1, %0;" ::"n"(kHEpiWarps * 32) : "memory");
                if (tid == 64) s_last = atomicAdd(&p.counters[tile], 1u) == (unsigned)p.ksplit - 1u ? 1u : 0u;
                asm volatile("bar.sync 1, %0;" ::"n"(kHEpiWarps * 32) : "memory");
                if (s_last != 0u) {
                    __threadfence();
                    const float* base = p.partial + (size_t)tile * p.ksplit * p.n_block * kHRows;
                    const int cols = min(p.n_block, p.T - t0);
                    const size_t piece = (size_t)p.n_block * kHRows;
                    for (int i = tid - 64; i < cols * (kHRows / 4); i += kHEpiWarps * 32) {
                        const int r = (i & (kHRows / 4 - 1)) * 4, c = i / (kHRows / 4);
                        const float* src = base + (size_t)c * kHRows + r;
                        float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
                        for (int z0 = 0; z0 < p.ksplit; z0 += 8) {  // eight pieces in flight
                            float4 x[8];
#pragma unroll
                            for (int z = 0; z < 8; ++z)
                                x[z] = z0 + z < p.ksplit ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)(z0 + z) * piece)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                            for (int z = 0; z < 8; ++z) { v[0] += x[z].x; v[1] += x[z].y; v[2] += x[z].z; v[3] += x[z].w; }
                        }
                        if (p.pair_act != 0) {
#pragma unroll
                            for (int e = 0; e < 4; e += 2)
                                if (row0 + r + e < p.rows) finish(t0 + c, (row0 + r + e) >> 1, apply_act(v[e], p.pair_act) * v[e + 1], false);
                        } else {
#pragma unroll
                            for (int e = 0; e < 4; ++e)
                                if (row0 + r + e < p.rows) finish(t0 + c, row0 + r + e, v[e], row0 + r + e < p.silu_rows);
                        }
                    }
                    if (tid == 64) p.counters[tile] = 0u;
                }
            }
        }
    }
    __syncwarp();
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
    if (!ok) atomicCAS(&g_device_status, 0, 1);
}

// ---- many rows of x, f32 on the CUDA cores -----------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) gemm_f32_kernel(const Bf16Gemm g) {
    constexpr int BT = 64, BR = 64, BK = 16;
    __shared__ float xt[BK][BT + 4], wt[BK][BR + 4];
    pdl_wait();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int r0 = blockIdx.x * BR, t0 = blockIdx.y * BT;
    const float* x = static_cast<const float*>(g.x);
    float acc[4][4] = {};
    for (int k0 = 0; k0 < g.K; k0 += BK) {
        for (int i = tid; i < BT * BK; i += 256) {
            const int k = i & (BK - 1), m = i >> 4;
            xt[k][m] = (t0 + m < g.T && k0 + k < g.K) ? x[(size_t)(t0 + m) * g.ldx + k0 + k] : 0.0f;
            wt[k][m] = (r0 + m < g.rows && k0 + k < g.K) ? bf16_bits_to_f32(g.w[(size_t)(r0 + m) * g.ldw + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xt[k][ty * 4 + i]; b[i] = wt[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
    float* const out = static_cast<float*>(g.out);
    if (g.pair_act != 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int t = t0 + ty * 4 + i, row = r0 + tx * 4 + j;
                if (t < g.T && row < g.rows) out[(size_t)t * g.ldo + (row >> 1)] = apply_act(acc[i][j], g.pair_act) * acc[i][j + 1];
            }
        return;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, row = r0 + tx * 4 + j;
            if (t < g.T && row < g.rows) {
                float v = acc[i][j];
                if (row < g.silu_rows) v = act_silu(v);
                v *= g.out_scale;
                const size_t o = (size_t)t * g.ldo + row;
                if (g.residual != nullptr) v += g.residual[o];
                out[o] = v;
            }
        }
}

int bf16_gemm(cudaStream_t stream, const Bf16Gemm& g) {
    if (g.T <= 0 || g.rows <= 0 || g.K <= 0 || g.ldw < g.K || g.ldx < g.K) return fail(KMLL_ERR_SHAPE, "bf16_gemm: T %d, rows %d, K %d", g.T, g.rows, g.K);
    if (g.pair_act != 0 && ((g.rows & 1) != 0 || g.residual != nullptr)) return fail(KMLL_ERR_SHAPE, "bf16_gemm: %d rows are not pairs", g.rows);
    if (g.x_f32) {
        if (g.out_bf16) return fail(KMLL_ERR_UNSUPPORTED, "bf16_gemm: f32 activations give f32 results");
        cudaError_t e = launch(gemm_f32_kernel, dim3((g.rows + 63) / 64, (g.T + 63) / 64), dim3(256), 0, stream, true, g);
        if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "gemm_f32: %s", cudaGetErrorString(e));
        return KMLL_OK;
    }
    if ((g.ldw & 7) != 0 || (g.ldx & 7) != 0 || (reinterpret_cast<uintptr_t>(g.w) & 15u) != 0 || (reinterpret_cast<uintptr_t>(g.x) & 15u) != 0)
        return fail(KMLL_ERR_SHAPE, "bf16_gemm: operands need 16-byte aligned rows");
    GemmBf16Params p;
    memset(&p, 0, sizeof(p));
    p.rows = g.rows; p.K = g.K; p.T = g.T;
    p.out = g.out; p.out_bf16 = g.out_bf16; p.ldo = g.ldo; p.residual = g.residual; p.silu_rows = g.silu_rows;
    p.pair_act = g.pair_act; p.out_scale = g.out_scale;
    p.row_tiles = (g.rows + kHRows - 1) / kHRows;
    // rows of x per tile: the size whose rounds over 148 SMs cost least (measured with K = 4096: 24 us at 64 rows, 32 at 256)
    const int nmax = g.T >= kHMaxN ? kHMaxN : (g.T + 15) / 16 * 16;
    int best = nmax;
    long long best_cost = -1;
    for (int nb = nmax; nb >= 64 || nb == nmax; nb -= 16) {
        const long long tiles = (long long)p.row_tiles * ((g.T + nb - 1) / nb), cost = (tiles + 147) / 148 * (600 + nb);
        if (best_cost < 0 || cost < best_cost) { best = nb; best_cost = cost; }
    }
    p.n_block = best;
    p.x_tiles = (g.T + best - 1) / best;  // walked fastest: the blocks at work share their weight rows, and x stays in L2
    const long long tiles = (long long)p.row_tiles * p.x_tiles;
    if (tiles > 0x3fffffff) return fail(KMLL_ERR_UNSUPPORTED, "bf16_gemm: too many tiles");
    p.tiles = (int)tiles;
    p.ksplit = 1;
    if (g.partial != nullptr && g.T <= kGemmSplitRows && p.tiles <= 74) {  // at least eight k-tiles per piece
        const int KT = (g.K + kHKT - 1) / kHKT;
        const int want = std::min({148 / p.tiles, KT / 8, 16});
        if (want > 1) {
            const int per = (KT + want - 1) / want;
            p.ksplit = (KT + per - 1) / per;  // (no empty piece)
            p.partial = g.partial;
            p.counters = g.counters;
        }
    }
    const size_t stage = (size_t)kHRows * 128 + (size_t)p.n_block * 128;
    p.stages = (int)((220 * 1024) / stage);
    if (p.stages > 8) p.stages = 8;
    const size_t smem = p.stages * stage + (2 * p.stages + 4) * 8 + 16 + 1024;
    CUtensorMap map_w, map_x;
    KMLL_TRY_RC(make_map_2d(&map_w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, g.w, (uint64_t)g.K, (uint64_t)g.rows, (uint64_t)g.ldw * 2, kHKT, kHRows,
                            CU_TENSOR_MAP_SWIZZLE_128B));
    KMLL_TRY_RC(make_map_2d(&map_x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, g.x, (uint64_t)g.K, (uint64_t)g.T, (uint64_t)g.ldx * 2, kHKT, (uint32_t)p.n_block,
                            CU_TENSOR_MAP_SWIZZLE_128B));
    cudaError_t e = allow_all_dynamic_smem(linear_gemm_bf16_kernel);
    if (e == cudaSuccess)
        e = launch(linear_gemm_bf16_kernel, dim3(p.tiles * p.ksplit < 148 ? p.tiles * p.ksplit : 148), dim3(kHThreads), smem, stream, true, p, map_w, map_x);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "linear_gemm_bf16: %s", cudaGetErrorString(e));
    return KMLL_OK;
}

}  // namespace kmll
