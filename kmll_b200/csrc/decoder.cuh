// The decoder object behind kmll_decoder_t: shared by runtime.cu (kmll's uniform quantized decoder, the decode loop, the
// session-level entry points) and layered.cu (decoders over a list of layer descriptions).
#pragma once

#include <nccl.h>

#include <vector>

#include "../../include/kmll_b200_runtime.h"
#include "internal.cuh"

namespace kmll {

#define KMLL_TRY(expr)                 \
    do {                               \
        int rc__ = (expr);             \
        if (rc__ != KMLL_OK) return rc__; \
    } while (0)

#define KMLL_CUDA(expr)                                                                        \
    do {                                                                                       \
        cudaError_t e__ = (expr);                                                              \
        if (e__ != cudaSuccess) return fail(KMLL_ERR_CUDA, "%s: %s", #expr, cudaGetErrorString(e__)); \
    } while (0)

struct Layered;  // layered.cu

struct QWeight {
    void* w = nullptr;       // int8 values or packed nibbles
    void* scales = nullptr;  // float[rows] or half[rows, cols/128]
    int rows = 0, cols = 0;  // local (sharded) shape
    uint8_t* prep = nullptr;  // W4-G128: the same values in the prepared layout the batch-1 kernels stream
};

struct Layer {
    uint16_t* attention_norm = nullptr;
    uint16_t* q_norm = nullptr;  // optional per-head RMSNorm weights [head_dim] of the query / key rows (null: the model has none)
    uint16_t* k_norm = nullptr;
    uint16_t* ffn_norm = nullptr;
    QWeight wq, wk, wv, wo, w1, w3, w2;
    uint8_t* w13_prep = nullptr;  // W4-G128: gate (w1) and up (w3) interleaved in the prepared layout
    float* key_cache = nullptr;
    float* value_cache = nullptr;
};

enum ShardKind { SHARD_NONE, SHARD_ROWS, SHARD_COLS };

struct Decoder {
    kmll_decoder_config cfg;
    int device = 0;
    int n_heads_l = 0, n_kv_l = 0, hidden_l = 0, vocab_l = 0;  // per-rank sizes
    std::vector<Layer> layers;
    uint16_t* final_norm = nullptr;
    uint16_t* embedding = nullptr;
    QWeight output;
    float* freqs = nullptr;
    // per-token scratch (crates/inference/src/model.rs:9339-9498 allocates the same set once)
    float *hidden_a = nullptr, *hidden_b = nullptr, *hidden_mid = nullptr;
    float *normed = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *q_rot = nullptr, *k_rot = nullptr;
    float *attn = nullptr, *delta = nullptr, *gate = nullptr, *up = nullptr, *act = nullptr;
    float* attn_ws = nullptr;
    uint32_t* part_tok = nullptr;
    float* part_logit = nullptr;
    uint64_t* packed = nullptr;      // this rank's arg-max
    uint64_t* packed_all = nullptr;  // [tp_size]
    uint64_t* packed_final = nullptr;
    DecodeState* state = nullptr;
    uint64_t* history = nullptr;
    int history_cap = 0;
    uint64_t* pinned = nullptr;  // host, pinned
    int host_position = 0;
    bool have_next = false;
    bool warmed = false;
    cudaGraphExec_t graph = nullptr;
    unsigned long long graph_trace_generation = 0;  // trace_generation() when `graph` was captured
    cudaStream_t capture_stream = nullptr;  // the caller's stream may be the legacy default stream, which cannot capture
    ncclComm_t comm = nullptr;
    // peer-memory exchange (tensor parallel decode step); null = NCCL collectives
    TpExchange* xc = nullptr;          // device copy of the tables
    TpExchange xc_host;                // the same tables on the host (the chained kernel takes them by value)
    void* xc_local = nullptr;          // this rank's exchange buffer (shared with the peers through CUDA IPC)
    unsigned int* xc_epoch = nullptr;  // inside xc_local
    void* xc_peer_base[kMaxTp] = {};   // peers' buffers as mapped here (null for the own rank)
    std::vector<void*> allocs;
    size_t weight_bytes = 0, kv_bytes = 0, resident_bytes = 0;  // resident = every device allocation of this decoder
    int launches_per_step = 0;
    bool weights_set = false;
    // chained decode step (W4-G128, fused): prepared weights, exchange words also on a single GPU
    bool chain = false;            // the decode step runs linear_chain_kernel
    bool chain_split = true;       // ... one launch per projection (default) instead of one launch per layer (KMLL_CHAIN=layer)
    bool chain_words = false;      // one GPU, one launch per projection: still hand the vectors over as exchange words (KMLL_CHAIN=words)
    bool prepared_valid = false;   // the prepared buffers match the canonical tensors
    unsigned int* top1_counter = nullptr;
    Layered* lay = nullptr;  // a decoder over a list of layer descriptions (layered.cu); null = kmll's uniform layers
};

template <typename T>
inline int dalloc(Decoder* d, T** out, size_t count) {
    void* p = nullptr;
    cudaError_t e = cudaMalloc(&p, count * sizeof(T) + 16);
    if (e != cudaSuccess) return fail(KMLL_ERR_CUDA, "cudaMalloc(%zu bytes): %s", count * sizeof(T), cudaGetErrorString(e));
    d->allocs.push_back(p);
    d->resident_bytes += count * sizeof(T);
    *out = static_cast<T*>(p);
    return KMLL_OK;
}

// ---- layered decoders (layered.cu), called by the entry points of runtime.cu ------------------------------------------
// One decode step: consumes state->next_top, leaves the logits in the decoder and the arg-max in state->next_top.
int layered_enqueue_step(Decoder* d, cudaStream_t s, int* launches);
// The next `n` tokens of the sequence (host or device memory) from position d->host_position; logits rows of the positions
// in `want` (offsets into these tokens, ascending) go to the device buffer logits_out [n_want, vocab].  With `top` the
// logits and the arg-max of the last token are produced as after a decode step.
int layered_forward(Decoder* d, cudaStream_t s, const uint32_t* tokens_host, const uint32_t* tokens_device, int n, const int* want, int n_want,
                    float* logits_out, bool top);
int layered_reset(Decoder* d, cudaStream_t s);             // zero states: the next token is at position 0
int layered_save_state(Decoder* d, cudaStream_t s);        // remember the recurrent states at d->host_position
int layered_rewind(Decoder* d, cudaStream_t s, int position);  // states of an earlier position (replays from the nearest remembered one)
int layered_hold_state(Decoder* d, cudaStream_t s, bool restore);  // around a warm-up step: copy the states away / back
const float* layered_logits(const Decoder* d);
bool layered_tapped(const Decoder* d);
int layered_set_tensor(Decoder* d, int layer, int tensor, const void* values);
int layered_get_tensor(Decoder* d, int layer, int tensor, void* values);
int layered_init_random(Decoder* d, uint64_t seed, float std, int tie_embeddings);
void layered_destroy(Decoder* d);

}  // namespace kmll
