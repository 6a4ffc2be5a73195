// Row operators of the layered decoders' prompt path: what stands between two projections, one block per row, f32 arithmetic,
// result in the type the next projection reads.  (A decode step runs the same steps as prologues of bf16_matvec_kernel.)
#include "internal.cuh"

namespace kmll {

namespace {

constexpr int kRowThreads = 256;

__device__ inline float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ inline float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ inline float gate_f(float z, int act) { return act == KMLL_ACT_SILU ? silu_f(z) : act == KMLL_ACT_SIGMOID ? sigmoid_f(z) : z; }
__device__ inline float inv_rms_f(float sum_sq, int n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }

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

__global__ void embed_rows_kernel(const uint16_t* __restrict__ table, const uint16_t* __restrict__ pos_table, int vocab, int dim,
                                  const uint32_t* __restrict__ tokens, int pos0, float* __restrict__ x) {
    pdl_wait();
    const int t = blockIdx.x;
    uint32_t token = tokens[t];
    if (token >= (uint32_t)vocab) token = (uint32_t)vocab - 1;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float v = bf16_bits_to_f32(table[(size_t)token * dim + i]);
        if (pos_table != nullptr) v += bf16_bits_to_f32(pos_table[(size_t)(pos0 + t) * dim + i]);
        x[(size_t)t * dim + i] = v;
    }
}

template <bool OUT32, int V>
__global__ void __launch_bounds__(kRowThreads) norm_rows_kernel(const float* __restrict__ x, int dim, const int* __restrict__ row,
                                                                const uint16_t* __restrict__ w, float offset, float eps, void* out, int ldo) {
    __shared__ float scratch[40];
    pdl_wait();
    const int t = blockIdx.x;
    const float* xr = x + (size_t)(row != nullptr ? row[t] : t) * dim;
    float s = 0.0f, v[V], g[V];
    for (int i = threadIdx.x * V; i < dim; i += kRowThreads * V) {
        loadv<true, V>(xr, i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) s += v[e] * v[e];
    }
    const float inv = inv_rms_f(block_sum(s, scratch), dim, eps);
    for (int i = threadIdx.x * V; i < dim; i += kRowThreads * V) {
        loadv<true, V>(xr, i, v);
        loadv<false, V>(w, i, g);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] *= inv * (offset + g[e]);
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
    const float c1 = bf16_bits_to_f32(coef[0]) * inv_rms_f(s1, n, eps), c2 = bf16_bits_to_f32(coef[1]) * inv_rms_f(s2, n, eps),
                c3 = bf16_bits_to_f32(coef[2]) * inv_rms_f(s3, n, eps), c0 = bf16_bits_to_f32(coef[3]);
    for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
        loadv<F32, V>(z, zr + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = ((c3 * v[e] + c2) * v[e] + c1) * v[e] + c0;
        storev<F32, V>(out, orow + i, v);
    }
}

// o normed (per head without weight, or over the whole row with norm_w), times gate_act(gate)
template <bool F32, int V>
__global__ void __launch_bounds__(kRowThreads) gated_rows_kernel(const float* __restrict__ o, int ldi, int n, const uint16_t* __restrict__ norm_w,
                                                                 int head_len, float eps, const void* __restrict__ gate, int ldg, int gate_act,
                                                                 void* out, int ldo) {
    __shared__ float scratch[40];
    pdl_wait();
    const float* orow = o + (size_t)blockIdx.x * ldi;
    const size_t gr = (size_t)blockIdx.x * ldg, outr = (size_t)blockIdx.x * ldo;
    float v[V], g[V], w[V];
    if (norm_w != nullptr) {
        float s = 0.0f;
        for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
            loadv<true, V>(orow, i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) s += v[e] * v[e];
        }
        const float inv = inv_rms_f(block_sum(s, scratch), n, eps);
        for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
            loadv<true, V>(orow, i, v);
            loadv<F32, V>(gate, gr + i, g);
            loadv<false, V>(norm_w, i, w);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] *= inv * w[e] * gate_f(g[e], gate_act);
            storev<F32, V>(out, outr + i, v);
        }
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int h0 = warp * head_len; h0 < n; h0 += (kRowThreads / 32) * head_len) {  // a warp per head
        float s = 0.0f;
        for (int i = lane * V; i < head_len; i += 32 * V) {
            loadv<true, V>(orow, h0 + i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) s += v[e] * v[e];
        }
        const float inv = inv_rms_f(warp_sum(s), head_len, eps);
        for (int i = lane * V; i < head_len; i += 32 * V) {
            loadv<true, V>(orow, h0 + i, v);
            loadv<F32, V>(gate, gr + h0 + i, g);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] *= inv * gate_f(g[e], gate_act);
            storev<F32, V>(out, outr + h0 + i, v);
        }
    }
}

template <bool OUT32, int V>
__global__ void __launch_bounds__(kRowThreads) convert_rows_kernel(const float* __restrict__ x, int ldi, int n, void* out, int ldo) {
    pdl_wait();
    float v[V];
    for (int i = threadIdx.x * V; i < n; i += kRowThreads * V) {
        loadv<true, V>(x, (size_t)blockIdx.x * ldi + i, v);
        storev<OUT32, V>(out, (size_t)blockIdx.x * ldo + i, v);
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

int embed_rows(cudaStream_t stream, const uint16_t* table, const uint16_t* pos_table, int vocab, int dim, const uint32_t* tokens, int pos0, int T, float* x) {
    KMLL_ROWS_CHECK(launch(embed_rows_kernel, dim3(T), dim3(256), 0, stream, true, table, pos_table, vocab, dim, tokens, pos0, x), "embed_rows");
}

int norm_rows(cudaStream_t stream, const float* x, int dim, const int* row, int T, const uint16_t* w, float offset, float eps, int out_f32, void* out, int ldo) {
    const bool v4 = by4({dim, ldo}) && aligned(x, 16) && aligned(w, 8) && aligned(out, 16);
    auto k = out_f32 ? (v4 ? norm_rows_kernel<true, 4> : norm_rows_kernel<true, 1>) : (v4 ? norm_rows_kernel<false, 4> : norm_rows_kernel<false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, x, dim, row, w, offset, eps, out, ldo), "norm_rows");
}

int polynorm_rows(cudaStream_t stream, const void* z, int f32, int ldz, int n, int T, const uint16_t* coef, float eps, void* out, int ldo) {
    const bool v4 = by4({n, ldz, ldo}) && aligned(z, 16) && aligned(out, 16);
    auto k = f32 ? (v4 ? polynorm_rows_kernel<true, 4> : polynorm_rows_kernel<true, 1>) : (v4 ? polynorm_rows_kernel<false, 4> : polynorm_rows_kernel<false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, z, ldz, n, coef, eps, out, ldo), "polynorm_rows");
}

int gated_rows(cudaStream_t stream, const float* o, int ldi, int n, int T, const uint16_t* norm_w, int head_len, float eps, const void* gate, int f32,
               int ldg, int gate_act, void* out, int ldo) {
    const bool v4 = by4({n, ldi, ldg, ldo, head_len}) && aligned(o, 16) && aligned(gate, 16) && aligned(out, 16) && (norm_w == nullptr || aligned(norm_w, 8));
    auto k = f32 ? (v4 ? gated_rows_kernel<true, 4> : gated_rows_kernel<true, 1>) : (v4 ? gated_rows_kernel<false, 4> : gated_rows_kernel<false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, o, ldi, n, norm_w, head_len, eps, gate, ldg, gate_act, out, ldo), "gated_rows");
}

int convert_rows(cudaStream_t stream, const float* x, int ldi, int n, int T, int out_f32, void* out, int ldo) {
    const bool v4 = by4({n, ldi, ldo}) && aligned(x, 16) && aligned(out, 16);
    auto k = out_f32 ? (v4 ? convert_rows_kernel<true, 4> : convert_rows_kernel<true, 1>) : (v4 ? convert_rows_kernel<false, 4> : convert_rows_kernel<false, 1>);
    KMLL_ROWS_CHECK(launch(k, dim3(T), dim3(kRowThreads), 0, stream, true, x, ldi, n, out, ldo), "convert_rows");
}

int rotation_table(cudaStream_t stream, const double* freqs, int half, int positions, double magnitude, float2* table) {
    const long long n = (long long)half * positions;
    KMLL_ROWS_CHECK(launch(rotation_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, false, freqs, half, positions, magnitude, table),
                    "rotation_table");
}

}  // namespace kmll
