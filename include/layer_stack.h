/*
 * layer_stack — C ABI of the decoder-only layer-stack models with dense bfloat16 weights (libstack_b200.so).
 *
 * A model is a list of layers; a layer is a mixer (one of TBL_MIXER_*) and, optionally, a gated feed-forward, each
 * with its pre-norm (TBL_NORM_*).  The residual is either one stream, with a learned average over the embedding output
 * and the results of all layers so far after a layer, or several streams that every sublayer reads and writes through
 * small matrices (hyper-connections).
 * The conventions are those of ternary_b200.h: plain pointers and sizes, an int status, no allocation, no
 * synchronisation, everything enqueued on the caller's stream, buffers borrowed; status codes, device status word
 * and launch counter are declared there too (each library has its own copy of the latter two).
 *
 * Precision.  TBL_BF16: matrix-product operands (weights, normed rows, cached latents, queries) are bfloat16 with
 * fp32 accumulation.  TBL_F32: activations and caches are fp32 and every product is a plain fp32 FMA.  In both, the
 * residual stream, norms, rotations, attention scores and weights, decays, step sizes, gates of the recurrence and
 * recurrent states are fp32.
 *
 * These models have no counterpart in the reference runtime.
 */
#ifndef LAYER_STACK_H
#define LAYER_STACK_H

#include "ternary_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

#define TBL_F32 0
#define TBL_BF16 1

#define TBL_MIXER_GENERAL_DELTA 0
#define TBL_MIXER_LATENT_ATTENTION 1
#define TBL_MIXER_ATTENTION 2

#define TBL_NORM_RMS 0               /* x / sqrt(mean x^2 + eps) * weight                       */
#define TBL_NORM_DYNAMIC_TANH 1      /* tanh(alpha x) * weight + bias                           */

#define TBL_ACT_SILU 0
#define TBL_ACT_GELU_TANH 1          /* 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))         */

#define TBL_MAX_STACK_LAYERS 256
#define TBL_MAX_DELTA_DIM 256        /* key/value size of a delta-rule head                      */
#define TBL_MAX_LATENT 1024          /* latent size + rotated part of a latent-attention layer   */
#define TBL_MAX_ATTENTION_DIM 512    /* query/key size of one map, and value size, of an attention head */
#define TBL_MAX_STREAMS 8            /* residual streams of a model with hyper-connections       */
#define TBL_PAIR_BLOCK 32            /* gate / up rows of a feed-forward alternate in blocks of this many rows */

/* y = W x + b; weight bf16 [outputs, inputs] row-major, 16-byte aligned; bias fp32 [outputs] or NULL. */
typedef struct tbl_dense_view {
    const void* weight;
    const float* bias;
    int inputs, outputs;
} tbl_dense_view;

/* Generalized delta rule, per head (unit key u = k / sqrt(sum k^2 + key_eps)):
 *   S <- diag(w) S - (a * u)(u^T S) + k v^T,   o = S^T r,
 *   w = exp(-decay_rate * sigmoid(W_w2 tanh(W_w1 h) + w0)),  a = sigmoid(W_a h + b_a);
 * o is divided by its root mean square per head, times norm, times sigmoid(W_g h), then W_o.
 * decay_up is W_w2 with w0 as its bias.  `in` stacks the rows of W_r | W_k | W_v | W_g | W_a (heads*dim each) | W_w1 (rank); its bias carries b_a. */
typedef struct tbl_delta_mixer {
    tbl_dense_view in, decay_up, out;
    const float* norm;               /* [heads*dim]                              */
    int heads, dim, rank;
    float decay_rate, key_eps;
} tbl_delta_mixer;

/* Latent attention: per head `dim` unrotated and `rot_dim` rotated query/key dimensions, values of `vdim`; keys
 * and values are W_uk c and W_uv c of a cached latent c (kv_rank) and one rotated key part shared by the heads.
 * `in` stacks W_dq (q_rank) | W_dkv (kv_rank + rot_dim) | W_g (heads*vdim).  rope tables fp32
 * [rope_positions, rot_dim/2]: entry i rotates dimension i with i + rot_dim/2. */
typedef struct tbl_latent_mixer {
    tbl_dense_view in, uq, uk, uv, out;
    const void* uk_t;                /* bf16 [heads][kv_rank][dim]: W_uk once more, transposed per head; NULL: the
                                        attention over the latent cache stays off the tensor cores */
    const float *q_norm, *kv_norm;   /* [q_rank], [kv_rank]                      */
    const float *rope_cos, *rope_sin;
    int heads, dim, rot_dim, vdim, q_rank, kv_rank, rope_positions;
    float scale;
} tbl_latent_mixer;

/* Softmax attention over cached keys and values: `heads` query heads share `kv_heads` key/value heads (query head h uses
 * h / (heads / kv_heads)), causal, no rotation.  `in` stacks W_q (heads*maps*dim rows, head by head) | W_k
 * (kv_heads*maps*dim) | W_v (kv_heads*vdim) | W_g (heads*vdim, only when gated); its bias carries theirs.
 *   score = temperature[position of the query] * scale * (q . k)
 * maps = 1: a head's output is the softmax average of the values.  maps = 2 (differential attention): every head has two
 * query/key maps over the same values, o = a1 - lambda a2, divided by its root mean square over the head (eps of the
 * model's norms) and multiplied by out_scale.  gated: times sigmoid(W_g h).  Then `out`.
 * kv_from >= 0: the layer has no W_k and W_v (their rows are left out of `in`) and reads the cache of that earlier
 * layer, which has projections of its own and the same kv_heads, maps, dim and vdim; -1: its own cache. */
typedef struct tbl_attention_mixer {
    tbl_dense_view in, out;
    const float* temperature;        /* [temperature_positions]; NULL: 1         */
    int temperature_positions, heads, kv_heads, dim, vdim, maps, gated, kv_from;
    float scale, lambda, out_scale;
} tbl_attention_mixer;

/* Hyper-connection of one sublayer with `streams` residual streams x_s (fp32 arrays):
 *   input = sum_s in[s] x_s,   x_t <- sum_s mix[s*streams + t] x_s + out[t] * sublayer(norm(input)). */
typedef struct tbl_hyper {
    const float *in, *mix, *out;
} tbl_hyper;

/* What Dynamic Tanh has beside its weight. */
typedef struct tbl_tanh_norm {
    const float* bias;               /* [width]                                  */
    float alpha;
} tbl_tanh_norm;

/* Feed-forward W_down(act(W_gate h + b) * (W_up h + b)) + b.  gate_up stacks blocks of TBL_PAIR_BLOCK gate rows
 * and the TBL_PAIR_BLOCK up rows that go with them (zero rows fill the last block). */
typedef struct tbl_stack_layer {
    int mixer;                       /* TBL_MIXER_*                              */
    const float* norm1;              /* [width]                                  */
    tbl_delta_mixer delta;
    tbl_latent_mixer latent;
    int ff;                          /* 0: no feed-forward                       */
    const float* norm2;
    tbl_dense_view gate_up, down;
    const float* depth_weights;      /* [layer index + 2]: the average after this layer; NULL: none */
    tbl_attention_mixer attention;
    tbl_tanh_norm tanh1, tanh2;      /* models with TBL_NORM_DYNAMIC_TANH        */
    tbl_hyper hyper1, hyper2;        /* models with streams: of the mixer, of the feed-forward */
    int activation;                  /* TBL_ACT_* of the feed-forward            */
} tbl_stack_layer;

typedef struct tbl_stack_model {
    int width, vocab, n_layers;
    const void* embedding;           /* bf16 [vocab, width]                      */
    float embedding_scale, norm_eps;
    const tbl_stack_layer* layers;
    const float* final_norm;
    tbl_dense_view head;             /* width -> vocab                           */
    int norm_kind;                   /* TBL_NORM_*                               */
    tbl_tanh_norm final_tanh;
    int streams;                     /* 0: one residual stream; otherwise hyper-connections, all streams equal to the
                                        embedding output at first and summed up at the end (no depth average) */
} tbl_stack_model;

/* Device state of `slots` sequences with room for `capacity` tokens each: positions, delta-rule states (fp32,
 * [head][value][key]), latent caches [token][kv_rank + rot_dim], and attention caches [kv head][token][keys of every map |
 * values], each part padded to a multiple of 16 (layers that read another's cache have none).  reset clears one slot (its position and
 * recurrent states), or the whole state when slot < 0: the latter once before the first use, so that cached rows
 * nobody has written hold finite numbers (they are read under a zero weight). */
size_t tbl_stack_state_bytes(const tbl_stack_model* model, int precision, int slots, int capacity);
int tbl_stack_state_reset(const tbl_stack_model* model, int precision, int slots, int capacity, int slot,
                          void* state_dev, size_t state_bytes, void* stream);
/* Scratch for a step of n_seq sequences x n_tok tokens whose longest sequence then holds `context` tokens. */
size_t tbl_stack_workspace_bytes(const tbl_stack_model* model, int precision, int n_seq, int n_tok, int context);

/* Enqueues one step: n_seq sequences bring n_tok tokens each (decode: n_tok = 1; a portion of a prompt: n_seq = 1,
 * or several prompts in lockstep).  slots_dev int32 [n_seq] names their state slots (distinct; the caller's
 * responsibility), tokens_dev int32 [n_seq*n_tok] their tokens, row = sequence*n_tok + token.  Positions live on
 * the device and advance by n_tok.  `context` bounds the tokens any of the sequences holds after the step (<=
 * capacity); a captured step may be replayed while it does.  want_rows_dev int32 [n_want] lists the rows whose
 * logits go to logits_dev fp32 [n_want, vocab] (n_want 0: no logits).  hidden_trace_dev (may be NULL): fp32
 * [n_layers, rows, width], the residual stream after every layer.  state_dev and workspace_dev 256-byte aligned.
 * A sequence past its capacity, or past the rotary table, sets TBL_DEV_CACHE_FULL and its rows are undefined. */
int tbl_stack_step(const tbl_stack_model* model, int precision, int slots, int capacity, void* state_dev,
                   const int32_t* slots_dev, int n_seq, int n_tok, int context, const int32_t* tokens_dev,
                   const int32_t* want_rows_dev, int n_want, float* logits_dev, float* hidden_trace_dev,
                   void* workspace_dev, size_t workspace_bytes, void* stream);

/* ---- the step's operators, one entry point each ----------------------------------------------------------------
 * Activations `x` have the precision's type (bf16 or fp32), strides in elements. */

/* out[m, :] = W x[m, :] + b [+ residual[m, :]], fp32 out (ld = outputs of the view).  route: 0 the kernel the step
 * would take, 1 the SIMT kernel, 2 the GEMV, 3 the tcgen05 GEMM (bf16 only), 4 the row-streaming kernel (bf16 only);
 * TBL_ERR_SHAPE when the route does not take the shape. */
int tbl_dense_forward(const tbl_dense_view* view, int precision, int route, const void* x_dev, int ldx, int rows,
                      const float* residual_dev, float* out_dev, void* stream);
/* out[m, :ff] (precision's type, ld = ff) = silu(gate) * up for a gate_up view of 2*round_up(ff, 32) rows. */
int tbl_gated_dense_forward(const tbl_dense_view* gate_up, int precision, int route, const void* x_dev, int ldx,
                            int rows, int ff, void* out_dev, void* stream);
/* The same with an activation TBL_ACT_* in place of silu. */
int tbl_gated_dense_act_forward(const tbl_dense_view* gate_up, int precision, int route, int activation, const void* x_dev,
                                int ldx, int rows, int ff, void* out_dev, void* stream);
/* The delta rule on stacked projections proj fp32 [n_seq*n_tok, in.outputs] (biases already added): out (precision's
 * type) [rows, heads*dim] is the normed, gated readout; states_dev [slots][heads][dim][dim] is updated.
 * workspace_dev: tbl_delta_workspace_bytes.  route: 0 as the step, 1 the scan kernel, 2 the single-token kernel. */
size_t tbl_delta_workspace_bytes(const tbl_delta_mixer* mixer, int precision, int rows);
int tbl_delta_forward(const tbl_delta_mixer* mixer, int precision, int route, float eps, const float* proj_dev,
                      float* states_dev, const int32_t* slots_dev, int n_seq, int n_tok, void* out_dev,
                      void* workspace_dev, size_t workspace_bytes, void* stream);
/* Latent attention on stacked projections proj fp32 [rows, in.outputs]: norms, rotation, cache append at
 * positions_dev[slot] .., attention, output gate -> out (precision's type) [rows, heads*vdim].  positions_dev is not
 * advanced.  route: 0 as the step, 1 over the latent cache (SIMT), 2 over the latent cache (tensor cores), 3 over
 * expanded keys and values (tensor cores); 2 and 3 take bf16 only. */
size_t tbl_latent_workspace_bytes(const tbl_latent_mixer* mixer, int precision, int n_seq, int n_tok, int context);
int tbl_latent_forward(const tbl_latent_mixer* mixer, int precision, int route, float eps, const float* proj_dev,
                       void* cache_dev, int capacity, const int32_t* slots_dev, const int32_t* positions_dev,
                       int n_seq, int n_tok, int context, void* out_dev, void* workspace_dev, size_t workspace_bytes,
                       void* stream);
/* Attention on stacked projections proj fp32 [rows, in.outputs]: cache append at positions_dev[slot] .. (not when kv_from
 * >= 0), attention, head norm, output gate -> out (precision's type) [rows, heads*vdim].  cache_dev [slots][kv_heads]
 * [capacity][tbl_attention_cache_width], zeroed before the first use.  positions_dev is not advanced.  route: 0 as the
 * step, 1 SIMT, 2 the cache-streaming kernel (warp-level MMAs), 3 the flash kernel (tcgen05); 2 and 3 take bf16 only. */
int tbl_attention_cache_width(const tbl_attention_mixer* mixer);
size_t tbl_attention_workspace_bytes(const tbl_attention_mixer* mixer, int precision, int n_seq, int n_tok, int context);
int tbl_attention_forward(const tbl_attention_mixer* mixer, int precision, int route, float eps, const float* proj_dev,
                          void* cache_dev, int slots, int capacity, const int32_t* slots_dev, const int32_t* positions_dev,
                          int n_seq, int n_tok, int context, void* out_dev, void* workspace_dev, size_t workspace_bytes,
                          void* stream);
/* One boundary between sublayers with hyper-connections.  streams_dev fp32 [streams] arrays [rows, width] at `stride`
 * floats.  With y_dev (fp32 [rows, width], the last sublayer's result): x_t <- sum_s mix[s, t] x_s + out[t] y, stored in
 * place when `store`; in_weights (NULL: ones) then give u = sum_t in[t] x_t, and h (precision's type) = norm(u), a
 * TBL_NORM_*; sum_dev (may be NULL) receives the plain sum of the streams.  row_index (may be NULL) selects source rows;
 * nothing is stored then. */
int tbl_stream_norm(float* streams_dev, size_t stride, int streams, const float* y_dev, const float* mix_dev,
                    const float* out_weights_dev, int store, const float* in_weights_dev, int precision, const int32_t* row_index_dev,
                    int rows, int width, int norm_kind, float eps, float alpha, const float* norm_dev, const float* norm_bias_dev,
                    float* sum_dev, void* h_dev, void* stream);
/* x[r, :] = sum_j weights[j] * history[j][r, :] (history: `count` fp32 arrays [rows, width] at `history_stride`
 * floats; weights NULL: the last array alone), written to x_dev (may be NULL), and h = x / rms(x) * norm in the
 * precision's type (norm NULL: no h).  row_index (may be NULL) selects source rows. */
int tbl_depth_norm(const float* history_dev, size_t history_stride, int count, const float* weights_dev, int precision,
                   const int32_t* row_index_dev, int rows, int width, float eps, const float* norm_dev, float* x_dev,
                   void* h_dev, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* LAYER_STACK_H */
