// Row operators of the layered decoders' prompt path: what stands between two projections, one block per row, f32 arithmetic,
// result in the type the next projection reads.  (A decode step runs the same steps as prologues of bf16_matvec_kernel.)
#include "activations.cuh"

namespace kmll {

namespace {

constexpr int kRowThreads = 256;

template <bool F32>
__device__ inline float load1(const void* p, size_t i) {
    return F32 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
template <bool F32>
__device__ inline void store1(void* p, size_t i, float v) {
    if (F32) static_cast<float*>(p)[i] = v;
    else static_cast<uint16_t*>(p)[i] = f32_to_bf16_bits(v);
}
// V consecutive elements; V = 4 needs 16-byte (f32) / 8-byte (bf16) aligned addresses
template <bool F32, int V>
__device__ inline void loadv(const void* p, size_t i, float (&v)[V]) {
    if (V == 4) {
        if (F32) {
            const float4 t = *reinterpret_cast<const float4*>(static_cast<const float*>(p) + i);
            v[0] = t.x; v[1 % V] = t.y; v[2 % V] = t.z; v[3 % V] = t.w;
        } else {
            const uint2 t = *reinterpret_cast<const uint2*>(static_cast<const uint16_t*>(p) + i);
            v[0] = __uint_as_float(t.x << 16); v[1 % V] = __uint_as_float(t.x & 0xffff0000u);
            v[2 % V] = __uint_as_float(t.y << 16); v[3 % V] = __uint_as_float(t.y & 0xffff0000u);
        }
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = load1<F32>(p, i + e);
    }
}
template <bool F32, int V>
__device__ inline void storev(void* p, size_t i, const float (&v)[V]) {
    if (V == 4) {
        if (F32) {
            *reinterpret_cast<float4*>(static_cast<float*>(p) + i) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
        } else {
            uint2 t;
            t.x = (uint32_t)f32_to_bf16_bits(v[0]) | ((uint32_t)f32_to_bf16_bits(v[1 % V]) << 16);
            t.y = (uint32_t)f32_to_bf16_bits(v[2 % V]) | ((uint32_t)f32_to_bf16_bits(v[3 % V]) << 16);
            *reinterpret_cast<uint2*>(static_cast<uint16_t*>(p) + i) = t;
        }
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) store1<F32>(p, i + e, v[e]);
    }
}

// One block per row; entry i of a row is always held by the same thread.
__global__ void __launch_bounds__(1024) embed_rows_kernel(const EmbedArgs a) {
    __shared__ float scratch[96];
    pdl_wait();
    const int t = blockIdx.x;
    int pos = a.pos0 + t;
    uint32_t token;
    if (a.state != nullptr) {
        const uint64_t packed = a.state->next_top;
        token = (uint32_t)(packed & 0xffffffffull);
        if (token >= (uint32_t)a.vocab) token = (uint32_t)a.vocab - 1;
        pos = a.state->position;
        if (threadIdx.x == 0) {
            const int step = a.state->step;
            a.token_log[pos] = token;
            if (step < a.history_cap) a.history[step] = packed;
            a.state->seq_len = pos + 1;
        }
    } else {
        token = a.tokens[t];
        if (token >= (uint32_t)a.vocab) token = (uint32_t)a.vocab - 1;
    }
    const uint16_t* e = a.table + (size_t)token * a.ld;
    const uint16_t* p = a.pos_table != nullptr ? a.pos_table + (size_t)pos * a.dim : nullptr;
    float* x = a.x + (size_t)t * a.dim;
    auto value = [&](int i) {
        float v = bf16_bits_to_f32(e[i]) * a.scale;
        if (p != nullptr) v += bf16_bits_to_f32(p[i]);
        return v;
    };
    if (a.norm.w == nullptr) {
        for (int i = threadIdx.x; i < a.dim; i += blockDim.x) x[i] = value(i);
        return;
    }
    float s = 0.0f, q = 0.0f;
    int n = 0;
    for (int i = threadIdx.x; i < a.dim; i += blockDim.x) {
        const float v = value(i);
        s += v;
        q += v * v;
        ++n;
    }
    float mean = 0.0f, inv;
    if (a.norm.kind == KMLL_NORM_LAYER) {
        Moments m{(float)n, n > 0 ? s / (float)n : 0.0f, 0.0f};
        for (int i = threadIdx.x; i < a.dim; i += blockDim.x) {
            const float v = value(i) - m.mean;
            m.dev += v * v;
        }
        m = block_moments(m, scratch);
        mean = m.mean;
        inv = inv_rms(m.dev, a.dim, a.norm.eps);
    } else {
        inv = inv_rms(block_sum(q, scratch), a.dim, a.norm.eps);
    }
    for (int i = threadIdx.x; i < a.dim; i += blockDim.x) {
        float v = (value(i) - mean) * inv * (a.norm.offset + bf16_bits_to_f32(a.norm.w[i]));
        if (a.norm.kind == KMLL_NORM_LAYER) v += bf16_bits_to_f32(a.norm.b[i]);
        x[i] = v;
    }
}

template <bool LAYER, bool OUT32, int V>
__global__ void __launch_bounds__(kRowThreads) norm_rows_kernel(const float* __restrict__ x, int dim, const int* __restrict__ row, const NormArgs norm, void* out,
                                                                int ldo) {
    __shared__ float scratch[96];
    pdl_wait();
    const int t = blockIdx.x;
    const float* xr = x + (size_t)(row != nullptr ? row[t] : t) * dim;
    float s = 0.0f, mean = 0.0f, inv, v[V], g[V], b[V];
    int n = 0;
    for (int i = threadIdx.x * V; i < dim; i += kRowThreads * V) {
        loadv<true, V>(xr, i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) s += LAYER ? v[e] : v[e] * v[e];
        n += V;
    }
    if (LAYER) {
        Moments m{(float)n, n > 0 ? s / (float)n : 0.0f, 0.0f};
        for (int i = threadIdx.x * V; i < dim; i += kRowThreads * V) {
            loadv<true, V>(xr, i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) m.dev += (v[e] - m.mean) * (v[e] - m.mean);
        }
        m = block_moments(m, scratch);
        mean = m.mean;
        inv = inv_rms(m.dev, dim, norm.eps);
    } else {
        inv = inv_rms(block_sum(s, scratch), dim, norm.eps);
    }
    for (int i = threadIdx.x * V; i < dim; i += kRowThreads * V) {
        loadv<true, V>(xr, i, v);
        loadv<false, V>(norm.w, i, g);
        if (LAYER) loadv<false, V>(norm.b, i, b);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            v[e] = (v[e] - mean) * inv * (norm.offset + g[e]);
            if (LAYER) v[e] += b[e];
        }
        storev<OUT32, V>(out, (size_t)t * ldo + i, v);
    }
}

template <bool F32, int V>
__global__ void __launch_bounds__(kRowThreads) polynorm_rows_kernel(const void* __restrict__ z, int ldz, int n, const uint16_t* __restrict__ coef,
                                                                    float eps, void* out, int ldo) {
    __shared__ float scratch[40];
    pdl_wait();
    const size_t zr = (size_t)blockIdx.x * ldz, orow = (size_t)blockIdx.x * ldo;
    float s1 = 0.0f, s2 = 0.0f, s3 = 0.0f, v[V];
    for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
        loadv<F32, V>(z, zr + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float q = v[e] * v[e];
            s1 += q;
            s2 += q * q;
            s3 += q * q * q;
        }
    }
    s1 = block_sum(s1, scratch);
    s2 = block_sum(s2, scratch);
    s3 = block_sum(s3, scratch);
    const float c1 = bf16_bits_to_f32(coef[0]) * inv_rms(s1, n, eps), c2 = bf16_bits_to_f32(coef[1]) * inv_rms(s2, n, eps),
                c3 = bf16_bits_to_f32(coef[2]) * inv_rms(s3, n, eps), c0 = bf16_bits_to_f32(coef[3]);
    for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
        loadv<F32, V>(z, zr + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = ((c3 * v[e] + c2) * v[e] + c1) * v[e] + c0;
        storev<F32, V>(out, orow + i, v);
    }
}

// one segment of a mixer's output: normed, times act(gate), times its scale; zeros behind it up to column `end`
template <bool GATE32, bool OUT32, int V>
__global__ void __launch_bounds__(kRowThreads) gated_rows_kernel(const float* __restrict__ o, int ldi, const GateSegment seg, int ldg, int end, void* out, int ldo) {
    __shared__ float scratch[40];
    pdl_wait();
    const float* orow = o + (size_t)blockIdx.x * ldi + seg.begin;
    const size_t gr = (size_t)blockIdx.x * ldg, outr = (size_t)blockIdx.x * ldo + seg.begin;
    const int n = seg.cols, len = seg.head_len;
    float v[V], g[V], w[V];
    for (int i = n + threadIdx.x; i < end - seg.begin; i += kRowThreads) store1<OUT32>(out, outr + i, 0.0f);
    auto gates = [&](int i) {  // of entries i .. i + V - 1 (one head, when heads share a gate)
        if (seg.gate == nullptr) {
#pragma unroll
            for (int e = 0; e < V; ++e) g[e] = seg.scale;
        } else if (seg.gate_len == 1) {
            loadv<GATE32, V>(seg.gate, gr + i, g);
#pragma unroll
            for (int e = 0; e < V; ++e) g[e] = seg.scale * apply_act(g[e], seg.act);
        } else {
            const float f = seg.scale * apply_act(load1<GATE32>(seg.gate, gr + i / seg.gate_len), seg.act);
#pragma unroll
            for (int e = 0; e < V; ++e) g[e] = f;
        }
    };
    if (seg.norm == KMLL_OUT_NORM_JOINT || seg.norm == KMLL_OUT_NORM_NONE) {
        float inv = 1.0f;
        if (seg.norm == KMLL_OUT_NORM_JOINT) {
            float s = 0.0f;
            for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
                loadv<true, V>(orow, i, v);
#pragma unroll
                for (int e = 0; e < V; ++e) s += v[e] * v[e];
            }
            inv = inv_rms(block_sum(s, scratch), n, seg.eps);
        }
        for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
            loadv<true, V>(orow, i, v);
            gates(i);
            if (seg.norm == KMLL_OUT_NORM_JOINT) {
                loadv<false, V>(seg.norm_w, i, w);
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] *= inv * w[e];
            }
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] *= g[e];
            storev<OUT32, V>(out, outr + i, v);
        }
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int h0 = warp * len; h0 < n; h0 += (kRowThreads / 32) * len) {  // a warp per head
        float s = 0.0f;
        for (int i = lane * V; i < len; i += 32 * V) {
            loadv<true, V>(orow, h0 + i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) s += v[e] * v[e];
        }
        const float inv = inv_rms(warp_sum(s), len, seg.eps);
        for (int i = lane * V; i < len; i += 32 * V) {
            loadv<true, V>(orow, h0 + i, v);
            gates(h0 + i);
            if (seg.norm == KMLL_OUT_NORM_HEAD_WEIGHTED) {
                loadv<false, V>(seg.norm_w, i, w);
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] *= w[e];
            }
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] *= inv * g[e];
            storev<OUT32, V>(out, outr + h0 + i, v);
        }
    }
}

__global__ void rotation_table_kernel(const double* __restrict__ freqs, int half, int positions, double magnitude, float2* __restrict__ table) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)positions * half) return;
    double s, c;
    sincos((double)(i / half) * freqs[i % half], &s, &c);
    table[i] = make_float2((float)(c * magnitude), (float)(s * magnitude));
}

bool by4(std::initializer_list<int> v) {
    for (int x : v)
        if (x & 3) return false;
    return true;
}
bool aligned(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (uintptr_t)(bytes - 1)) == 0; }

}  // namespace

#define KMLL_ROWS_CHECK(expr, what)                                                              \
    do {                                                                                         \
        cudaError_t e__ = (expr);                                                                \
        if (e__ != cudaSuccess) return fail(KMLL_ERR_CUDA, what ": %s", cudaGetErrorString(e__)); \
        return KMLL_OK;                                                                          \
    } while (0)

int embed_rows(cudaStream_t stream, const EmbedArgs& a) {
    const int threads = a.dim >= 1024 ? 1024 : (a.dim + 31) / 32 * 32;
    KMLL_ROWS_CHECK(launch(embed_rows_kernel, dim3(a.T), dim3(threads), 0, stream, true, a), "embed_rows");
}

int norm_rows(cudaStream_t stream, const float* x, int dim, const int* row, int T, const NormArgs& norm, int out_f32, void* out, int ldo) {
    const bool v4 = by4({dim, ldo}) && aligned(x, 16) && aligned(norm.w, 8) && aligned(out, 16) && (norm.b == nullptr || aligned(norm.b, 8));
    void (*k)(const float*, int, const int*, const NormArgs, void*, int) = nullptr;
    if (norm.kind == KMLL_NORM_LAYER)
        k = out_f32 ? (v4 ? norm_rows_kernel<true, true, 4> : norm_rows_kernel<true, true, 1>) : (v4 ? norm_rows_kernel<true, false, 4> : norm_rows_kernel<true, false, 1>);
    else
        k = out_f32 ? (v4 ? norm_rows_kernel<false, true, 4> : norm_rows_kernel<false, true, 1>) : (v4 ? norm_rows_kernel<false, false, 4> : norm_rows_kernel<false, false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, x, dim, row, norm, out, ldo), "norm_rows");
}

int polynorm_rows(cudaStream_t stream, const void* z, int f32, int ldz, int n, int T, const uint16_t* coef, float eps, void* out, int ldo) {
    const bool v4 = by4({n, ldz, ldo}) && aligned(z, 16) && aligned(out, 16);
    auto k = f32 ? (v4 ? polynorm_rows_kernel<true, 4> : polynorm_rows_kernel<true, 1>) : (v4 ? polynorm_rows_kernel<false, 4> : polynorm_rows_kernel<false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, z, ldz, n, coef, eps, out, ldo), "polynorm_rows");
}

int gated_rows(cudaStream_t stream, const float* o, int ldi, int T, const GateSegment& seg, int gate_f32, int ldg, int end, int out_f32, void* out, int ldo) {
    const bool v4 = by4({seg.begin, seg.cols, ldi, ldo}) && (seg.norm == KMLL_OUT_NORM_JOINT || (seg.norm == KMLL_OUT_NORM_NONE && seg.gate_len == 1) || by4({seg.head_len})) &&
                    (seg.gate == nullptr || (seg.gate_len == 1 ? by4({ldg}) && aligned(seg.gate, 16) : by4({seg.gate_len}))) && aligned(o, 16) && aligned(out, 16) &&
                    (seg.norm_w == nullptr || aligned(seg.norm_w, 8));
    void (*k)(const float*, int, const GateSegment, int, int, void*, int) = nullptr;
    if (gate_f32)
        k = out_f32 ? (v4 ? gated_rows_kernel<true, true, 4> : gated_rows_kernel<true, true, 1>) : (v4 ? gated_rows_kernel<true, false, 4> : gated_rows_kernel<true, false, 1>);
    else
        k = out_f32 ? (v4 ? gated_rows_kernel<false, true, 4> : gated_rows_kernel<false, true, 1>) : (v4 ? gated_rows_kernel<false, false, 4> : gated_rows_kernel<false, false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, o, ldi, seg, ldg, end, out, ldo), "gated_rows");
}

int rotation_table(cudaStream_t stream, const double* freqs, int half, int positions, double magnitude, float2* table) {
    const long long n = (long long)half * positions;
    KMLL_ROWS_CHECK(launch(rotation_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, false, freqs, half, positions, magnitude, table),
                    "rotation_table");
}

}  // namespace kmll
