/* Adding parts to the engine from outside: the model spec (JSON) and the C interface a new kind of
 * norm, position encoding, mixer, feed-forward, block arrangement, embedding or head has to offer.
 *
 * The reference chooses between such variants with flags and optional per-layer tensors on one struct
 * (is_swa[], kv_donor[], act_gelu, rope_neox, embd_scale, final_softcap: fastgguf.c:4064-4100, :4191-4229).
 * Here a layer names the KIND of each of its parts, kinds are looked up in one registry per role, and a
 * kind the library does not have is registered with fg_register_part - no file of the library changes.
 *
 * The model spec
 *   {"hidden_size": E, "vocab_size": V, "max_positions": N,
 *    "embedding":  PART, "final_norm": PART, "head": PART,
 *    "layers":   [{"block": "prenorm", "mixer": PART, "feed_forward": PART, "mixer_norm": PART,
 *                  "feed_forward_norm": PART}, ...],            "feed_forward": null: a layer without one (then
 *                                                               no feed_forward_norm either); optional
 *                                                               "mixer_post_norm", "feed_forward_post_norm": PART;
 *                                                               block "parallel" has no feed_forward_norm, or one
 *                                                               (then each sublayer reads a norm of its own);
 *                                                               block "postnorm" has neither, only post norms;
 *                                                               optional "token_input": PART, role token_input:
 *                                                               x <- x + f(x, the rows' tokens) behind the sublayers
 *    "schedule": [{"layer": 0, "cache_from": null}, ...],      the order in which layers run: an entry may
 *                                                               name a layer twice (a cache of its own each
 *                                                               time) or read an EARLIER entry's cache;
 *                                                               "reenter": true runs the spec's "reentry" part on
 *                                                               the stream in front of the entry ("pass": the number of the
 *                                                               pass of a looped span that begins there, default 0)
 *    "reentry": PART (optional),                                x <- f(x, the embedding's output), role stream_map
 *    "stop_token_ids": [...], "ignored_tensors": ["regex", ...]}
 *   PART = {"kind": "rmsnorm", "params": {...}, "tensors": {"local name": "checkpoint name"}}
 *   A parameter whose value is itself {"kind": ..., "params": ...} is a nested part (the position encoding
 *   of an attention mixer); nested parts with equal kind and parameters are built once and shared.
 *
 * Built-in kinds
 *   norm          "rmsnorm"        {size, eps, offset: 0.0, gain: 1.0}     y = x / rms(x) * gain * (offset + w)
 *   position      "rope"           {head_dim, theta, scaling: null | {rope_type: "linear", factor} | {rope_type: "llama3", ...} | {rope_type: "yarn", factor,
 *                                   original_max_position_embeddings, beta_fast, beta_slow},
 *                                   rotary_dim: head_dim, layout: "halves" | "adjacent"}
 *   mixer         "gqa_attention"  {hidden_size, n_heads, n_kv_heads, head_dim, position: PART | null,
 *                                   scale: null = 1/sqrt(head_dim), window: null, keep_first: 0,
 *                                   v_head_dim: head_dim}        tensors q/k/v/o_proj.weight
 *                 "retention"      {hidden_size, n_heads, head_dim, v_head_dim, decay: [per head], position: PART | null,
 *                                   k_scale: null = 1/sqrt(head_dim), eps, qkv_activation: null | "silu", norm: "head" |
 *                                   "whole", gate_activation: "silu" | "sigmoid"}   linear attention with a fixed decay per
 *                                   head, state [heads, head_dim, v_head_dim] float32 per sequence; a unit norm per head, or one
 *                                   over all heads with a weight (then the gate may be a sigmoid); tensors
 *                                   q/k/v/g/o_proj.weight, norm.weight (norm "whole")
 *                 "gated_linear_attention"  {hidden_size, n_heads, head_dim, v_head_dim, tau, q_scale, eps, decay_rank: from the
 *                                   checkpoint}   a decay per key channel and token, sigmoid(low-rank(h) + b)^(1/tau); state as
 *                                   retention's; tensors q/k/v/g/o_proj.weight, decay_down/up.weight, decay_up.bias, norm.weight
 *                 "sink_attention" {hidden_size, n_heads, n_kv_heads, head_dim, v_head_dim, scale, window: 0, softcap: 0,
 *                                   chunk: 0, conv_taps: 0, bias: false, o_bias: false, sink: false, unit_sink: false,
 *                                   qk_norm: null | "whole" | "head", gate: null | "head" | "full", values: null | "keys",
 *                                   differential: null | d, eps, position: PART | null}
 *                                   grouped-query attention with biases, a short convolution over time (its last inputs are
 *                                   per-sequence state), norms over the whole of q and of k ("whole": weights [heads * head_dim])
 *                                   or per head ("head": one weight [head_dim] for all heads), rotation in the position part's
 *                                   layout (adjacent pairs, or halves of the rotated part), capped scores, a sink, a sigmoid
 *                                   gate per head from the mixer's input ("head": g_proj.weight [heads, hidden]) or per number
 *                                   ("full": [heads * v_head_dim, hidden]); chunk c instead of a window: a row sees the keys of
 *                                   its run of c positions counted from the sequence's first; unit_sink: a sink of score 0; values "keys": the values are the
 *                                   keys as projected; differential: two maps a head over the same values, subtracted with weight
 *                                   exp(lq1 . lk1) - exp(lq2 . lk2) + d, normalised per head, times 1 - d; tensors
 *                                   q/k/v/o_proj.weight, q/k/v_proj.bias, o_proj.bias, q/k/v_conv.weight, q/k_norm.weight,
 *                                   sinks, g_proj.weight, lambda_q1/k1/q2/k2
 *                 "latent_attention" {hidden_size, n_heads, head_dim, rot_dim, v_head_dim, kv_rank, q_rank, scale, eps,
 *                                   sink: false, gate: false, shared_kv: false, position: PART}   keys and values from one latent
 *                                   a token plus a shared rotated key part (only those are cached); shared_kv: no latent of its
 *                                   own, the schedule entry reads an earlier entry's cache; tensors q_down/q_up/kv_down/k_up/
 *                                   v_up/o_proj/g_proj.weight, q_down_norm/kv_down_norm.weight, sinks
 *                 "state_space"    {hidden_size, n_heads, v_head_dim, state_size, n_groups: 1, conv_taps: 1, norm_groups: 1, eps}
 *                                   in_proj = [z | x | B | C | dt], convolution + SiLU over x, B, C, S_t = exp(-exp(A_log) dt)
 *                                   S_(t-1) + dt B x^T, y = S^T C + D x, y silu(z) normalised in norm_groups parts; state
 *                                   (convolution inputs and S) float32 per sequence; tensors in_proj/o_proj.weight, conv.weight,
 *                                   conv.bias, dt_bias, A_log, D, norm.weight
 *                 "gated_delta"    {hidden_size, n_heads, n_kv_heads, head_dim, v_head_dim, conv_taps: 1, eps, unit_eps: 1e-6,
 *                                   q_scale: null = 1/sqrt(head_dim)}   convolved q, k, v, unit q and k, S <- g S; u = beta (v -
 *                                   S^T k); S <- S + k u^T; o = S^T q, a norm per head and a SiLU gate; tensors q/k/v/b/a/g/
 *                                   o_proj.weight, q/k/v_conv.weight, A_log, dt_bias, norm.weight
 *                 "rglru"          {hidden_size, width, n_blocks: 1, conv_taps: 1, gain: 8.0}   a recurrent block around the real-gated
 *                                   linear recurrent unit: y = gelu_tanh(W_y h + b), u = convolution(W_x h + b) + b, r and i sigmoids
 *                                   of block-diagonal maps of u, log a = -gain r softplus(lam), S = a S + sqrt(1 - a^2) i u, output
 *                                   W_o (S y); state (a ring of convolution inputs, and S) float32 per sequence; tensors y/x/
 *                                   o_proj.weight, y/x_proj.bias, conv.weight, conv.bias, r/i_gate.weight [n_blocks, s, s],
 *                                   r/i_gate.bias [n_blocks, s], lam
 *                 "mixer_pair"     {hidden_size, left: {kind, params}, right: {kind, params}, left_scale: 1, right_scale: 1,
 *                                   normalize: false, eps}   two mixers on the same rows, y = left_scale f(left) + right_scale
 *                                   f(right), f an RMS norm over the width with a weight where normalize is true; tensors
 *                                   left.<the left mixer's>, right.<the right mixer's>, left_norm.weight, right_norm.weight
 *   feed_forward  "swiglu"         {hidden_size, d_ff, activation: "silu" | "gelu_tanh" | "relu"}   down(act(gate x) * (up x))
 *                 "mlp"            {hidden_size, d_ff, activation: "relu2"}   down(act(up x))
 *                 "moe"            {hidden_size, d_ff, n_experts, top_k, limit, alpha: 1.702, router: "sigmoid_input"}
 *                                   tensors router.weight, experts.<e>.gate/up/down_proj.weight
 *                                  {hidden_size, d_ff, n_experts, top_k, router: "softmax_grouped", n_identity: 0, n_groups: 1,
 *                                   keep_groups: n_groups, route_scale: 1.0, shared_d_ff: 0}   softmax scores over n_experts +
 *                                   n_identity outputs; the choice on score + router.bias among the keep_groups best of n_groups
 *                                   groups of neighbours; weights = chosen scores / their sum * route_scale on the experts'
 *                                   outputs; the last n_identity outputs return the input; experts silu(gate) * up; a shared
 *                                   expert on every row; tensors router.weight, router.bias, experts.<e>.*, shared.gate/up/
 *                                   down_proj.weight
 *                                  {hidden_size, d_ff, n_experts, top_k, router: "softmax_chosen", activation: "gated" | "relu2"}   the
 *                                   largest logits + router.bias; weights = softmax over the chosen ones, on the experts' outputs;
 *                                   relu2: experts down(max(up x, 0)^2) without gate_proj; tensors router.weight, router.bias, experts.<e>.*
 *   block         "prenorm"        x += mixer(norm1(x)); x += feed_forward(norm2(x))
 *                 "sandwich"       x += post1(mixer(norm1(x))); x += post2(feed_forward(norm2(x)))
 *                 "postnorm"       x += post1(mixer(x)); x += post2(feed_forward(x)): the sublayers read the stream itself
 *                 "parallel"       x += mixer(norm1(x)) + feed_forward(norm1(x)), or, with a feed_forward_norm,
 *                                  x += mixer(norm1(x)) + feed_forward(norm2(x)), both norms of the same x
 *   token_input   "gated_token_embedding"  {hidden_size, vocab_size, dim, table_dim, column, eps}   e = table[token, column ..
 *                                   column + dim), y = W_proj (gelu_tanh(W_gate x) * e), x <- x + y / rms(y) * w; tensors table
 *                                   [vocab, table_dim] (layers may share it), gate [dim, E], proj [E, dim], norm [E]
 *   stream_map    "concat_linear"  {hidden_size}   x <- W [x; embedding output], W [E, 2 E]; tensor weight
 *                 "add_row"        {hidden_size, rows}   x <- x + table[pass], table [rows, E]; tensor table
 *   embedding     "embedding"      {vocab_size, hidden_size, scale: 1.0}
 *   head          "lm_head"        {vocab_size, hidden_size, softcap: null}   logits <- cap tanh(logits / cap)
 *
 * What a part may rely on in fg_batch_view: every device array, and the host integers n_seq, n_rows,
 * n_want, max_new, max_len, single_token, want_all, table_width.  The three host_* arrays are NULL when the
 * step is being recorded into a CUDA graph (the decode step of the generation loop): a part that needs
 * per-sequence bounds then reads cu_rows / seq_start / slots on the device.  Under graph replay rows of
 * finished or padded sequences name the slot `n_slots` (a spare row that every state array has) and page 0
 * of every cache group, so whatever a part writes for them lands where nothing reads.
 * A part launches its work on call->stream and takes scratch memory from call->alloc (valid until the step
 * ends; the same addresses at every replay of a recorded step).  It must not allocate, free or synchronise.
 */
#pragma once
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define FG_ROLE_NORM 0
#define FG_ROLE_POSITION 1
#define FG_ROLE_MIXER 2
#define FG_ROLE_FEED_FORWARD 3
#define FG_ROLE_BLOCK 4
#define FG_ROLE_EMBEDDING 5
#define FG_ROLE_HEAD 6
#define FG_ROLE_STREAM_MAP 7   /* built-in kinds only: a map of the residual stream that also reads the embedding's output */
#define FG_ROLE_TOKEN_INPUT 8  /* built-in kinds only: what a layer adds to the stream from its tokens, behind its sublayers */

typedef struct fg_tensor_decl {
    char name[96];           /* the part's local tensor name */
    int ndim;
    int64_t shape[4];
    int is_int;              /* 0: a float tensor (follows the engine's dtype policy); 1: an int32 table */
    int init;                /* random weights: 0 = N(0, std), 1 = 1 + N(0, std) */
    float std;
} fg_tensor_decl;

typedef struct fg_dev_tensor {
    void *data;              /* device memory */
    int dtype;               /* FG_F32 0, FG_BF16 1, FG_I32 3 */
    int ndim;
    int64_t shape[4];
    int64_t ld;              /* elements between rows of a 2-d tensor */
} fg_dev_tensor;

typedef struct fg_batch_view {
    int n_seq, n_rows, n_want, max_new, max_len, single_token, want_all;
    const int *tokens;       /* [n_rows] token ids */
    const int *positions;    /* [n_rows] position of each row in its sequence */
    const int *row_seq;      /* [n_rows] index of the row's sequence within the step */
    const int *cu_rows;      /* [n_seq + 1] first row of each sequence */
    const int *seq_start;    /* [n_seq] length of each sequence before the step */
    const int *slots;        /* [n_seq] cache / state slot of each sequence */
    const int *want_rows;    /* [n_want] rows whose logits are wanted, or NULL */
    int n_groups;
    const int *const *block_tables;   /* per cache group: [n_seq, table_width] page ids (device) */
    int table_width;
    const int *host_cu_rows, *host_seq_start, *host_slots;   /* host copies; NULL while a graph records */
    void *stream;
} fg_batch_view;

typedef struct fg_layer_io {
    int group;               /* cache group of this entry (index into block_tables), -1 = none */
    void *k_pool, *v_pool;   /* [n_pages, n_kv_heads, page_size, head_dim] in the engine's dtype, or NULL */
    int n_pages, page_size, n_kv_heads, head_dim, cache_dtype;
    int write_cache;         /* 0: the pools belong to an earlier entry; read only */
    void *state;             /* [n_slots + 1, state_bytes] fixed-size state of this entry, or NULL */
    int64_t state_bytes;
    int n_slots;
    int v_head_dim;          /* v_pool is [n_pages, n_kv_heads, page_size, v_head_dim]; equal to head_dim unless asked otherwise */
} fg_layer_io;

struct fg_part_call;
typedef struct fg_block_ops {       /* what a block arrangement may ask the engine to run (ctx = call) */
    /* which: 0 = the mixer's norm, 1 = the feed-forward's norm; returns normalised rows [M, E] */
    int (*norm)(const struct fg_part_call *call, int which, fg_dev_tensor *xn_out);
    int (*mixer)(const struct fg_part_call *call, const fg_dev_tensor *xn);          /* adds into call->residual */
    int (*feed_forward)(const struct fg_part_call *call, const fg_dev_tensor *xn);   /* adds into call->residual */
} fg_block_ops;

typedef struct fg_part_call {
    int role;
    const fg_batch_view *batch;
    const fg_layer_io *io;          /* mixer and block: the entry's cache pools and state */
    fg_dev_tensor x;                /* norm: the residual stream in, f32 [M, E]; embedding: f32 [M, E] to fill */
    fg_dev_tensor xn;               /* mixer, feed_forward, head: normalised rows in the activation dtype */
    fg_dev_tensor out;              /* norm: [R, E] in the activation dtype; head: f32 [R, V] */
    fg_dev_tensor residual;         /* mixer, feed_forward, block: f32 [M, E]; ADD the part's output into it */
    const int *rows;                /* norm: device indices of the R rows to normalise, or NULL for all */
    int n_rows;
    void *(*alloc)(void *alloc_ctx, size_t bytes);   /* 256-byte aligned device scratch for this step */
    void *alloc_ctx;
    const fg_block_ops *block_ops;  /* block only */
    void *engine_ctx;               /* block only: opaque */
    void *stream;
} fg_part_call;

typedef struct fg_part_vtable {
    /* A new instance from the part's parameters (JSON text).  dtype: the engine's activation dtype.
     * NULL with a message in err refuses the parameters. */
    void *(*create)(const char *params_json, int dtype, void *user, char *err, size_t err_cap);
    void (*destroy)(void *self);
    int (*n_tensors)(void *self);
    int (*tensor_decl)(void *self, int i, fg_tensor_decl *out);
    /* Tensor i on the device (engine dtype policy applied); it lives as long as the engine. */
    int (*load)(void *self, int i, const fg_dev_tensor *t);
    /* mixer: 1 and the three numbers if it keeps keys and values per position (window 0 = all of them); values
     * have the keys' head size */
    int (*cache_request)(void *self, int *n_kv_heads, int *head_dim, int *window);
    /* mixer: bytes of fixed-size state per sequence (zeroed when a sequence takes its slot); 0 = none */
    int64_t (*state_bytes)(void *self);
    /* position: fill cos/sin [max_positions, head_dim / 2] (host, float32) for pairs (j, j + head_dim / 2), and
     * perm [head_dim]: perm[i] = the row of a head (as stored) that becomes row i, so that the stored pairs
     * land on (j, j + head_dim / 2); the identity for the halves layout. */
    int (*position_tables)(void *self, int max_positions, int head_dim, float *cos_out, float *sin_out, int *perm);
    /* every other role: run on call->stream; 0 or an FG_E_* status */
    int (*forward)(void *self, const fg_part_call *call);
    void *user;
} fg_part_vtable;

/* Unused entries may be NULL.  The table is copied; `kind` must not clash with a built-in kind. */
int fg_register_part(int role, const char *kind, const fg_part_vtable *vt);

#ifdef __cplusplus
}
#endif
