/*
 * kmll_b200_runtime.h — C ABI of the decode runtime built on the operators of kmll_b200.h.
 *
 * The runtime is the counterpart of kmll's quantized-weights runtime
 * (MinistralAllLinearInt8Runtime / RuntimeCore, crates/inference/src/model.rs:5151-5166,
 * :6327-6384): resident quantized weights, per-layer f32 KV caches [max_seq, n_kv, head_dim]
 * (crates/inference/src/model.rs:9308-9324), scratch allocated once, `prefill` then greedy
 * generation (generate_greedy_until_i8_top1_from_next, crates/inference/src/model.rs:6021-6106).
 * Differences: the per-token work is captured once in a CUDA graph and replayed; the next token
 * stays on the device between steps (kmll reads it back every token,
 * crates/inference/src/model.rs:10655); tensor parallelism over several GPUs is supported.
 *
 * All functions return 0 or a KMLL_ERR_* code (kmll_b200.h); kmll_last_error() has the message.
 * A decoder belongs to the CUDA device that was current when it was created and must be used
 * from one thread at a time.
 */
#ifndef KMLL_B200_RUNTIME_H
#define KMLL_B200_RUNTIME_H

#include <stddef.h>
#include <stdint.h>

#include "kmll_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef void* kmll_decoder_t;

enum { KMLL_FORMAT_RS_I8 = 0, KMLL_FORMAT_W4G128 = 1, KMLL_FORMAT_BF16 = 2 /* layered decoders: bf16 rows as a checkpoint stores them */ };

/* Tensor ids for kmll_decoder_*_tensor.  Linear weights are [out_features, in_features]
 * (crates/inference/src/model.rs:8711-8760); names follow kmll's layer fields. */
enum {
    KMLL_T_ATTENTION_NORM = 0, /* bf16 [dim] */
    KMLL_T_WQ = 1,             /* [n_heads*head_dim, dim] */
    KMLL_T_WK = 2,             /* [n_kv_heads*head_dim, dim] */
    KMLL_T_WV = 3,
    KMLL_T_WO = 4,             /* [dim, n_heads*head_dim] */
    KMLL_T_FFN_NORM = 5,       /* bf16 [dim] */
    KMLL_T_W1 = 6,             /* gate [hidden_dim, dim] */
    KMLL_T_W3 = 7,             /* up   [hidden_dim, dim] */
    KMLL_T_W2 = 8,             /* down [dim, hidden_dim] */
    KMLL_T_FINAL_NORM = 9,     /* bf16 [dim]            (layer = -1) */
    KMLL_T_EMBEDDING = 10,     /* bf16 [vocab, dim]     (layer = -1) */
    KMLL_T_OUTPUT = 11,        /* lm_head [vocab, dim]  (layer = -1) */
    KMLL_T_Q_NORM = 12,        /* optional, bf16 [head_dim]: per-head RMSNorm of the query rows before RoPE (model.rs:10165-10194); */
    KMLL_T_K_NORM = 13,        /* same for the key rows.  Set them before the first decode step; a model without them sets neither. */
    /* layered decoders (kmll_layered_create).  ATTENTION_NORM / FFN_NORM are the norms ahead of the mixer and of the feed-forward,
     * WQ / WK / WV / WO the mixer's projections, W3 / W2 the feed-forward's up and down projections. */
    KMLL_T_POSITION = 14,      /* learned position vectors [position_rows, dim]   (layer = -1) */
    KMLL_T_GATE = 15,          /* linear attention: output gate [heads*vdim, dim] */
    KMLL_T_MIX_NORM = 16,      /* linear attention: weight [heads*vdim] of the norm over all heads */
    KMLL_T_DKV = 17,           /* latent attention: [kv_rank + rot_dim, dim] */
    KMLL_T_DKV_NORM = 18,      /* latent attention: [kv_rank] */
    KMLL_T_UK = 19,            /* latent attention: latent -> keys [heads*dim, kv_rank] */
    KMLL_T_UV = 20,            /* latent attention: latent -> values [heads*vdim, kv_rank] */
    KMLL_T_ACT = 21,           /* PolyNorm coefficients a, b, c, e [4] */
    KMLL_T_ATTENTION_NORM_BIAS = 22, /* [dim], layer norms */
    KMLL_T_FFN_NORM_BIAS = 23,
    KMLL_T_FINAL_NORM_BIAS = 24,     /* (layer = -1) */
    KMLL_T_EMBED_NORM = 25,          /* norm of the embedding [dim] (layer = -1) */
    KMLL_T_EMBED_NORM_BIAS = 26,     /* (layer = -1) */
    KMLL_T_DECAY_DOWN = 27,    /* gated linear attention: [decay_rank, dim] */
    KMLL_T_DECAY_UP = 28,      /* [heads*dim_k, decay_rank] */
    KMLL_T_DECAY_BIAS = 29,    /* [heads*dim_k] */
    KMLL_T_DECAY_LOG = 30,     /* [heads], KMLL_DECAY_SOFTPLUS */
    KMLL_T_BETA = 31,          /* delta rule: write strength [heads, dim] */
    KMLL_T_Q_CONV = 32,        /* short convolutions [channels, conv], the current token's tap last */
    KMLL_T_K_CONV = 33,
    KMLL_T_V_CONV = 34,
    KMLL_T_GATE_DOWN = 35,     /* low-rank output gate: [gate_rank, dim] */
    KMLL_T_GATE_UP = 36,       /* [heads*vdim, gate_rank] */
    KMLL_T_BESIDE = 64         /* added to a mixer's tensor id: that tensor of the layer's second mixer */
};

/* TextConfig of kmll (crates/inference/src/model.rs:271-366) reduced to what the decoder path uses. */
typedef struct {
    int n_layers;
    int dim;
    int n_heads;
    int n_kv_heads;
    int head_dim;
    int hidden_dim;
    int vocab_size;
    int rotary_dim; /* <= head_dim, even */
    float rope_theta;
    float norm_eps;
    int max_seq_len;
    int format;   /* KMLL_FORMAT_* */
    int fused;    /* 1: fused kernels (RMSNorm+QKV, gate*up, +residual, lm_head arg-max); 0: one
                     launch per kmll operator, in kmll's order (crates/inference/src/model.rs:10102-10300) */
    int tp_rank;  /* tensor parallel rank / size; 0 / 1 for a single GPU */
    int tp_size;
    int kv_bf16;  /* 1: the KV cache holds bf16 (rounded to nearest-even when a row is written) instead of kmll's f32 rows
                     (crates/inference/src/model.rs:10160-10186 writes f32): half the cache bytes and half the attention
                     traffic, results no longer bit-equal to kmll's. */
    int sliding_window;  /* > 0: every position attends only the last `sliding_window` positions (itself included), the
                            mask of Mistral-style checkpoints; 0: full causal attention, which is all kmll implements
                            (crates/inference/src/kernels/inference.rs:1420-1686).  The cache still keeps every row. */
} kmll_decoder_config;

/* sizeof(kmll_decoder_config) as this library was compiled: a binding checks its own mirror of the struct against it
   (fields are only ever appended) */
size_t kmll_decoder_config_bytes(void);
int kmll_decoder_create(const kmll_decoder_config* config, kmll_decoder_t* out);
int kmll_decoder_destroy(kmll_decoder_t dec);

/* Random-init weights, generated and quantized on the device: linear weights ~ N(0, std) (rounded to
 * bf16 first for RS-I8, as kmll quantizes bf16 checkpoints), embeddings ~ N(0, std) bf16, norm
 * weights 1.  With tie_embeddings != 0 the output matrix is the quantized embedding table.  Under
 * tensor parallelism every rank generates the full tensor with the same seed and keeps its shard,
 * so shards are slices of the single-GPU tensors. */
int kmll_decoder_init_random(kmll_decoder_t dec, uint64_t seed, float std, int tie_embeddings);

/* Upload one tensor from host memory: bf16 bits for norms/embedding; for linear weights the
 * already quantized parts (RS-I8: int8 values + float scales; W4-G128: packed bytes + binary16
 * group scales).  Full (unsharded) tensors; the decoder keeps its tensor-parallel shard. */
int kmll_decoder_set_tensor(kmll_decoder_t dec, int layer, int tensor, const void* values,
                            const void* scales);
/* Download this rank's shard of a tensor to host memory (sizes as uploaded; tp_size == 1 gives the
 * full tensor).  Either pointer may be null. */
int kmll_decoder_get_tensor(kmll_decoder_t dec, int layer, int tensor, void* values, void* scales);

/* Tensor parallelism over NCCL.  Rank 0 obtains an id, the caller distributes the 128 bytes to all
 * ranks (any transport), then every rank calls kmll_decoder_tp_init with the same id. */
int kmll_tp_unique_id(unsigned char id_out[128]);
int kmll_decoder_tp_init(kmll_decoder_t dec, const unsigned char id[128]);

/* prefill (crates/inference/src/model.rs:5945-5968): runs the prompt through the batched path,
 * fills the KV caches and leaves the arg-max of the last position ready.  Resets the sequence. */
int kmll_decoder_prefill(kmll_decoder_t dec, kmll_stream_t stream, const uint32_t* tokens_host,
                         int n_tokens);
/* Same result through the per-token decode path (prefill_token_loop_reference,
 * crates/inference/src/model.rs:6393-6395). */
int kmll_decoder_prefill_token_loop(kmll_decoder_t dec, kmll_stream_t stream,
                                    const uint32_t* tokens_host, int n_tokens);

/* Greedy generation: n_steps tokens, each step = forward of the pending token + lm_head arg-max.
 * The whole step is one CUDA graph; tokens never leave the device during the loop.  On return
 * tokens_out[i] / logits_out[i] hold token and logit of step i (GreedyGenerationStep,
 * crates/inference/src/model.rs:6072-6077).  Synchronises the stream at the end. */
int kmll_decoder_generate_greedy(kmll_decoder_t dec, kmll_stream_t stream, int n_steps,
                                 uint32_t* tokens_out, float* logits_out);
/* The same steps without waiting and without reading anything back (timing loops). */
int kmll_decoder_enqueue_steps(kmll_decoder_t dec, kmll_stream_t stream, int n_steps);
/* The device keeps the packed (logit, token) of every step since the last prefill / rewind / generate_greedy:
 * packed_out[i] = entry first + i (the token step first + i consumed).  Lets a timing loop built on
 * kmll_decoder_enqueue_steps check afterwards what it generated.  Synchronises the stream. */
int kmll_decoder_history(kmll_decoder_t dec, kmll_stream_t stream, int first, int count, uint64_t* packed_out);
/* One step the way kmll's host loop does it: the token comes from host memory, the packed
 * (logit, token) result is copied back and the stream is synchronised
 * (crates/inference/src/model.rs:10655).  *packed_out = (f32 bits << 32) | next token. */
int kmll_decoder_step_host(kmll_decoder_t dec, kmll_stream_t stream, uint32_t token,
                           uint64_t* packed_out);

/* Pending next token (arg-max of the last logits) as packed (f32 bits << 32) | token; synchronises. */
int kmll_decoder_next_top(kmll_decoder_t dec, kmll_stream_t stream, uint64_t* packed_out);
/* Truncate the sequence to `position` tokens (<= current position); the pending token is kept.  Used to
 * replay the same positions again (timing legs, speculative roll-back). */
int kmll_decoder_rewind(kmll_decoder_t dec, kmll_stream_t stream, int position);
/* Replace the pending token (packed (f32 bits << 32) | token) that the next step will consume; with kmll_decoder_rewind
 * this replays a recorded continuation from an earlier position. */
int kmll_decoder_set_pending(kmll_decoder_t dec, kmll_stream_t stream, uint64_t packed);
/* Number of tokens in the sequence (= next position). */
int kmll_decoder_position(kmll_decoder_t dec);
/* Final hidden state of the last forward [dim] to host (parity checks); synchronises. */
int kmll_decoder_last_hidden(kmll_decoder_t dec, kmll_stream_t stream, float* hidden_out);
/* Replace the RoPE frequency table (rotary_dim / 2 host values), e.g. with YaRN-scaled frequencies
 * (yarn_rope_frequencies, crates/inference/src/model.rs:9257-9306).  Synchronises the device. */
int kmll_decoder_set_rope_freqs(kmll_decoder_t dec, const float* freqs_host, int count);
/* Next-token logits [vocab_size] of the sequence as it stands (final RMSNorm + lm_head over the last hidden state) into a
 * DEVICE buffer of the caller; enqueues only.  Replaces what next_logits_to_host / next_top_logits start from
 * (crates/inference/src/model.rs:5319-5352).  One GPU only (a tensor-parallel rank holds a slice of the vocabulary). */
int kmll_decoder_next_logits(kmll_decoder_t dec, kmll_stream_t stream, float* logits_device);
/* Kernel launches per decode step; bytes of weights / KV cache resident on this rank; bytes of every device allocation of
 * the decoder (weights + KV cache + scratch: RuntimeMemoryStats, crates/inference/src/model.rs:803-808,5368-5391). */
int kmll_decoder_launches_per_step(kmll_decoder_t dec);
size_t kmll_decoder_weight_bytes(kmll_decoder_t dec);
size_t kmll_decoder_kv_bytes(kmll_decoder_t dec);
size_t kmll_decoder_resident_bytes(kmll_decoder_t dec);

/* ---- layered decoders ----------------------------------------------------------------------------------------------
 * A decoder over a list of layer descriptions with bf16 weights: pre-norm layers (x += mixer(norm(x)), x += feed_forward(
 * norm(x))) in any order and with sizes of their own.  The mixers are latent attention, grouped softmax attention, linear
 * attention with a fixed decay per head, and linear attention with a decay per key channel and token (optionally with the delta
 * rule); a layer may hold two of them side by side.  The handle is an ordinary kmll_decoder_t: prefill, generate_greedy,
 * enqueue_steps, history, step_host, next_top, set_pending, rewind, position, last_hidden, next_logits, set_tensor / get_tensor /
 * init_random, the byte counts and destroy work on it (rewind replays tokens from the nearest remembered state, since a recurrent
 * state cannot be cut back).  No counterpart in kmll.  Not for layered decoders: tensor parallelism, the lockstep batch,
 * archives, prefill_token_loop. */
enum { KMLL_MIXER_NONE = 0, KMLL_MIXER_LATENT_ATTENTION = 1, KMLL_MIXER_LINEAR_ATTENTION = 2, KMLL_MIXER_ATTENTION = 3, KMLL_MIXER_GATED_LINEAR = 4 };
enum { KMLL_ACT_NONE = 0, KMLL_ACT_SILU = 1, KMLL_ACT_SIGMOID = 2, KMLL_ACT_GELU_TANH = 3 };
enum {
    KMLL_MLP_NONE = 0,
    KMLL_MLP_POLYNORM = 1, /* W_down polynorm(W_up h) */
    KMLL_MLP_GATED = 2     /* W_down (mlp_act(W_gate h) * (W_up h)) */
};
enum { KMLL_NORM_RMS = 0, KMLL_NORM_LAYER = 1 /* mean taken off, weight and bias */ };
/* norm of a mixer's output ahead of its gate */
enum {
    KMLL_OUT_NORM_PER_HEAD = 0,      /* each head over its own root mean square, no weight */
    KMLL_OUT_NORM_JOINT = 1,         /* all heads together, weight [heads*vdim] */
    KMLL_OUT_NORM_HEAD_WEIGHTED = 2, /* each head over its own root mean square, weight [vdim] shared by the heads */
    KMLL_OUT_NORM_NONE = 3
};
/* decay of a key channel from z = W_up (W_down h) + bias */
enum { KMLL_DECAY_LOGISTIC = 1 /* sigmoid(z)^(1 / decay_tau) */, KMLL_DECAY_SOFTPLUS = 2 /* exp(-exp(A_head) softplus(z)) */ };

typedef struct {
    int mixer;       /* KMLL_MIXER_* */
    int heads;
    int dim;         /* per head: query / key size (latent attention: the part that is not rotated) */
    int vdim;        /* per head: value size */
    /* latent attention: one latent of kv_rank values (RMS-normed) and one rotated key part of rot_dim values per position;
     * scores (q . W_uk c + q_rot . k_rot) * score_scale, values W_uv c */
    int kv_rank;
    int rot_dim;     /* even; 0 = no rotated part */
    int window;      /* attention, > 0: a position sees itself and the window - 1 positions before it; 0: every earlier position */
    float score_scale;
    /* linear attention: S <- decay S + k v^T, o = S^T q; q, k, v through qkv_act, the first rot_dim entries of q and k rotated,
     * k times key_scale; o normed (out_norm), times gate_act(W_g h) */
    int qkv_act;     /* KMLL_ACT_NONE / KMLL_ACT_SILU */
    int gate_act;    /* KMLL_ACT_SILU / KMLL_ACT_SIGMOID */
    int out_norm;    /* KMLL_OUT_NORM_* */
    float key_scale;
    /* grouped attention: query head h uses key / value head h / (heads / kv_heads); no rotation */
    int kv_heads;    /* divides heads; also for gated linear attention: heads of q and k */
    int chunk;       /* > 0: a position sees the positions of its own chunk only (chunks counted from position 0) */
    int head_gate;   /* 1: head i's output times gate_act(W_g h)_i, W_g [heads, dim] */
    float out_scale; /* factor on the mixer's output (1 for none) */
    /* gated linear attention: S <- diag(alpha) S + k u^T, o = S^T q, one decay alpha per key channel and token */
    float q_scale;
    int decay;       /* KMLL_DECAY_* */
    float decay_tau;
    int decay_rank;
    int delta;       /* 0: u = v; 1: u = beta (v - (diag(alpha) S)^T k), beta = sigmoid(W_beta h) per head */
    int conv;        /* taps of the causal convolution on q, k and v, followed by SiLU; 0: none */
    float unit_eps;  /* > 0: q and k over sqrt(sum of squares + unit_eps) */
    int gate_rank;   /* 0: gate W_g h, W_g [heads*vdim, dim]; > 0: W_gate_up (W_gate_down h) */
} kmll_mixer_spec;

typedef struct {
    kmll_mixer_spec mixers[2]; /* the second: KMLL_MIXER_NONE, or a mixer beside the first that reads the same normed input; their
                                  outputs, each times its out_scale, are added */
    int mlp;         /* KMLL_MLP_* */
    int mlp_act;     /* KMLL_MLP_GATED: KMLL_ACT_SILU / KMLL_ACT_GELU_TANH */
    int ff;          /* feed-forward width */
} kmll_layer_spec;

typedef struct {
    int n_layers;
    int dim;
    int vocab_size;
    int max_seq_len;
    int position_rows; /* > 0: a learned position vector is added to the embedding (max_seq_len <= position_rows); 0: none */
    float norm_eps;
    float norm_offset; /* layer and final norms multiply by (norm_offset + w): 1 for weights stored around zero, else 0 */
    int compute_f32;   /* 0: bf16 activations into the tensor-core projections of a prompt, bf16 caches; 1: f32 throughout */
    int norm;          /* KMLL_NORM_*: layer, final and embedding norms */
    float embed_scale; /* factor on the embedding (ahead of the position vector) */
    int embed_norm;    /* 1: the embedding is normed */
    float logit_scale;
    int tie_output;    /* 1: the logits read the embedding table (no KMLL_T_OUTPUT) */
} kmll_layered_config;

size_t kmll_layer_spec_bytes(void);
size_t kmll_layered_config_bytes(void);
int kmll_layered_create(const kmll_layered_config* config, const kmll_layer_spec* layers, kmll_decoder_t* out);
/* Rotation of a layer with rot_dim > 0: rot_dim / 2 frequencies and the factor on cos and sin.  Entry i is paired with entry
 * i + rot_dim / 2; the table is built on the device in f64 and rounded once. */
int kmll_layered_set_rotation(kmll_decoder_t dec, int layer, const double* freqs_host, int count, double magnitude);
/* Decay of every head of a linear-attention layer. */
int kmll_layered_set_decay(kmll_decoder_t dec, int layer, const double* decay_host, int count);
/* The next n tokens of the sequence, continuing at kmll_decoder_position (a portion of a prompt, or one decoded token).
 * want[n_want]: ascending offsets into `tokens` whose logits go to the device buffer logits_device [n_want, vocab_size].
 * Leaves the arg-max of the last token pending.  Enqueues, then synchronises. */
int kmll_decoder_extend(kmll_decoder_t dec, kmll_stream_t stream, const uint32_t* tokens_host, int n, const int* want, int n_want, float* logits_device);
/* Forget the sequence: the next kmll_decoder_extend starts at position 0. */
int kmll_decoder_reset(kmll_decoder_t dec, kmll_stream_t stream);
/* The residual stream behind every layer for the last extend call is kept when a buffer [n_layers, n, dim] is attached (null
 * detaches); parity checks. */
int kmll_layered_tap(kmll_decoder_t dec, float* residual_device);

/* Operators of the layered decoders that take a mixer description (more of them in kmll_b200.h).
 *
 * y = W norm(x) * out_scale, one row of x in f32; norm: KMLL_NORM_*, norm_weight null: none.  pair_act != 0: rows 2 i and 2 i + 1
 * of w are a gate and its value, y[i] = pair_act(gate) * value (rows / 2 results). */
int kmll_normed_linear_bf16(kmll_stream_t stream, const float* x, const uint16_t* w, int pitch, int rows, int cols, int norm, const uint16_t* norm_weight,
                            const uint16_t* norm_bias, float eps, int pair_act, float out_scale, float* y);
/* The same pairs for a batch of rows: out [batch, rows / 2] in the type of x (workspace as for kmll_linear_batched_bf16). */
int kmll_pair_linear_batched_bf16(kmll_stream_t stream, const void* x, int x_f32, int ldx, int batch, const uint16_t* w, int pitch, int rows, int cols,
                                  int pair_act, void* workspace, void* out);
/* rows [batch, dim] f32 normed into bf16 */
int kmll_norm_rows_bf16(kmll_stream_t stream, const float* x, int batch, int dim, int norm, const uint16_t* weight, const uint16_t* bias, float eps, uint16_t* out);
/* y = W z (+ residual) for one row, where z is the outputs of one or two mixers side by side in x [cols] (the second from the next
 * multiple of 8 on): each normed, gated and scaled as its description says.  gates: f32, one pointer per mixer (null: none), heads
 * or heads*vdim values. */
int kmll_mixer_output_linear_bf16(kmll_stream_t stream, const kmll_mixer_spec* mixers, int n_mixers, const float* x, const uint16_t* const* norm_weights,
                                  const float* const* gates, float eps, const uint16_t* w, int pitch, int rows, int cols, const float* residual, float* y);
/* Grouped attention over a cache [max_seq, pitch] (f32 or bf16): keys of every key / value head, each padded to a multiple of 8
 * entries (zeros), then the values likewise.  in [tokens, ld]: q, k, v at their column offsets.  The tokens' cache rows are
 * written, then every position they see is attended.  One token at *position_device: the decode form (f32 input, bf16 cache);
 * bf16 input and cache: the prompt form; else plain f32 arithmetic. */
int kmll_grouped_attention(kmll_stream_t stream, const kmll_mixer_spec* mixer, const void* in, int in_f32, int ld, int q_off, int k_off, int v_off, int tokens,
                           int position, const int* position_device, void* cache, int cache_f32, int pitch, int max_seq, float* out, int ldo);
/* Gated linear attention.  in [tokens, ld]: q, k, v, the decay factor (decay_rank), the logits of beta (heads) and the gate factor
 * (gate_rank) at offsets[0 .. 5]; the maps' columns are padded with zeros to their pitch (a multiple of 8).  conv [q | k | v channels][taps]; ring [taps][channels] f32 holds the inputs of earlier
 * positions.  state [heads, dim, vdim] f32 and ring are updated.  scratch == null: token after token in f32, the low-rank gate goes
 * to gate [tokens, heads*vdim]; else (bf16 input, dim up to 128, 4 or more tokens) chunks of 64 tokens on the tensor cores,
 * _scratch_floats() floats, no gate. */
typedef struct {
    const uint16_t *decay_up; /* [heads*dim, decay_pitch] */
    int decay_pitch;
    const uint16_t *decay_bias, *decay_log, *conv;
    const uint16_t *gate_up;  /* [heads*vdim, gate_pitch] */
    int gate_pitch;
} kmll_gated_linear_weights;
size_t kmll_gated_linear_scratch_floats(const kmll_mixer_spec* mixer, int tokens);
int kmll_gated_linear_attention(kmll_stream_t stream, const kmll_mixer_spec* mixer, const kmll_gated_linear_weights* weights, const void* in, int in_f32, int ld,
                                const int* offsets, int tokens, int position, const int* position_device, float* state, float* ring, float* scratch, float* gate,
                                float* out, int ldo);

/* ---- on-disk archive of the quantized linear weights ---------------------------------------------------------
 * The directory layout of kmll's quantization export, so an archive written by either side loads on the other:
 *   manifest.json with "quantization": "row-symmetric-int8-with-f32-row-scales" (crates/inference/src/model.rs:9047-9053),
 *   NNNN_<name>.i8 (raw int8, row-major) and NNNN_<name>.scales.f32 (little-endian f32) per tensor, where <name> has
 *   every non-alphanumeric character replaced by '_' (crates/inference/src/rowwise_scaled.rs:141-157) and NNNN is the
 *   tensor index: 0 = output.weight, 1 + layer * 7 + offset for wq, wk, wv, wo, w1, w3, w2
 *   (crates/inference/src/model.rs:9082-9140, :9185-9187).
 * W4-G128 archives (no counterpart in kmll) use the manifest value "group128-symmetric-int4-with-f16-group-scales" and
 * the suffixes .w4 (packed nibbles) / .gscales.f16.  Host functions; `values` / `scales` are HOST pointers.
 * Norm weights and embeddings are not part of kmll's archive (they stay in the checkpoint). */
int kmll_archive_tensor_index(int layer, int offset); /* layer < 0: 0 (output.weight); exported_int8_layer_tensor_index */
int kmll_archive_file_paths(const char* dir, int index, const char* name, int format, char* values_path, char* scales_path,
                            size_t capacity);
int kmll_archive_write_tensor(const char* dir, int index, const char* name, int format, int rows, int cols,
                              const void* values, const void* scales);
/* RowwiseScaledI8Matrix::read_exported (rowwise_scaled.rs:94-106): fails unless both files have exactly the bytes of
 * a rows x cols tensor. */
int kmll_archive_read_tensor(const char* dir, int index, const char* name, int format, int rows, int cols, void* values,
                             void* scales);
int kmll_archive_write_manifest(const char* dir, const kmll_decoder_config* config, const char* weights_path);
/* validate_all_linear_int8_export_archive (crates/inference/src/model.rs:8984-9035): directory, manifest key, byte
 * length of every expected file; with expected_weights_path also the manifest's weights_path. */
int kmll_archive_validate(const char* dir, const kmll_decoder_config* config, const char* expected_weights_path);
/* Write every linear tensor of a single-GPU decoder + the manifest / validate an archive and upload it (new_from_export,
 * crates/inference/src/model.rs:6327-6384); `config` is the configuration the decoder was created with. */
int kmll_decoder_export_archive(kmll_decoder_t dec, const kmll_decoder_config* config, const char* dir, const char* weights_path);
int kmll_decoder_load_archive(kmll_decoder_t dec, const kmll_decoder_config* config, const char* dir,
                              const char* expected_weights_path);

/* ---- lockstep batch of sequences (new; kmll decodes one sequence at a time) -------------------------
 * Up to 16 independent sequences at the same position are decoded together so that every weight is read
 * once per step for all of them.  The batch shares the decoder's weights and owns its KV caches
 * ([batch] x the decoder's cache size).  Each sequence is prefilled with the ordinary decoder and then
 * adopted into a slot (its KV rows and pending token are copied); all sequences must be at the same
 * position.  Single GPU, rotary_dim == head_dim.  The per-sequence results equal those of the
 * single-sequence decoder up to the rounding of the batched linear kernel. */
typedef void* kmll_batch_t;
int kmll_batch_create(kmll_decoder_t dec, int batch, kmll_batch_t* out);
int kmll_batch_destroy(kmll_batch_t batch);
int kmll_batch_adopt(kmll_batch_t batch, kmll_stream_t stream, int slot);
/* n_steps greedy tokens for every sequence: tokens_out / logits_out are [batch][n_steps]. */
int kmll_batch_generate_greedy(kmll_batch_t batch, kmll_stream_t stream, int n_steps, uint32_t* tokens_out,
                               float* logits_out);
int kmll_batch_enqueue_steps(kmll_batch_t batch, kmll_stream_t stream, int n_steps);
int kmll_batch_position(kmll_batch_t batch);
int kmll_batch_launches_per_step(kmll_batch_t batch);

#ifdef __cplusplus
}
#endif
#endif /* KMLL_B200_RUNTIME_H */
