/*
 * teeny_hybrid -- C ABI of the hybrid decoder runner (libteeny_b200.so): decoders whose layers mix recurrent token
 * mixers, sliding-window, full and latent attention, in any order, over an f32 residual stream.
 *
 * A layer is   x <- x + sum of branches(norm1(x))   and, when it has a feed-forward,   x <- x + ff(norm2(x));   with
 * POST_NORM it is   x <- x + residual_mult norm1_post(sum of branches(norm1(x)))   and likewise for the feed-forward.
 * All branches of a layer read one fused input projection W_in norm1(x) and write one row that the fused output
 * projection W_out takes back to the width, so parallel branches cost no extra matrix products.
 *
 * A sequence's state has a constant size (per branch: a ring or a full-length cache of keys and values, a cache of latents,
 * a matrix state per head, or a vector state) and lives in a slot; a step runs any number of entries, each the next tokens
 * of one slot.
 *
 * The reference has no such models; execution follows the same scheme as its model executor and as teeny_qwen3.h.
 * All pointers are device pointers owned by the caller unless stated; nothing here allocates device memory.
 * Status codes are those of teeny_b200.h.
 */
#ifndef TEENY_HYBRID_H_
#define TEENY_HYBRID_H_

#include "teeny_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* Branch kinds.  pad8(n) = n rounded up to a multiple of 8; h = norm1(x).
 *   ATTENTION  grouped-query attention over the last `window` tokens (0: all of them).  Input rows: q [heads * dim], k
 *              [kv_heads * dim], unless KEYS_ARE_VALUES v [kv_heads * vdim], and with OUT_GATE g [heads * vdim].  QK_NORM:
 *              per-head RMS norms of q and k before the rotation.  Rotate-half positions on the first rot_dims dimensions (cos
 *              and sin times rot_scale), score = (q . k) * score_scale, with softcap > 0 softcap * tanh(score / softcap).
 *              SINK: exp(SINK of the head) joins the softmax denominator.  OUT_GATE: the output is multiplied by sigmoid(g).
 *              With window 0 and values of their own: VALUE_MIX, v <- (1 - lambda) v + lambda v_first, where v_first are the
 *              values of the model's first branch with VALUE_MIX (which keeps its own) and lambda is VALUE_MIX's weight.
 *   LATENT     attention whose keys and values are made from a latent: c_q = rms_norm(D_q h) * Q_NORM, q = UQ c_q; c =
 *              rms_norm(D_c h) * K_NORM; one rotated key part D_r h for all heads; the other key dimensions and the values are
 *              per-head products with c.  Scores and rotation as above.  Input rows: D_q [q_rank], D_c [rank], D_r
 *              [rot_dims].  dim (unrotated dimensions of a head), vdim and rot_dims are multiples of 8; a head of q is
 *              [rot_dims rotated (rotate-half layout), dim unrotated].
 *   DELTA      generalized delta rule, S <- diag(w) S - (a u)(u^T S) + k v^T, o = S^T r, w = exp(-decay_coef *
 *              sigmoid(W_low tanh(W_1 h) + DECAY_BIAS)), a = sigmoid(A h + RATE_BIAS), u = k / sqrt(sum k^2 + unit_eps); each
 *              head's o is RMS-normed, times O_NORM, times sigmoid(G h).
 *              Input rows: r, k, v, a, g [heads * dim each], W_1 [rank].
 *   DECAY      S <- decay_head S + k v^T, o = S^T q with silu on q, k, v; o is RMS-normed over all heads together, times
 *              O_NORM, times sigmoid(G h).  Input rows: q, k [heads * dim], v, g [heads * vdim].
 *   MIN_GRU    S <- (1 - z) S + z g(u), z = sigmoid(Z h + Z_BIAS), u = X h + X_BIAS, output S * silu(G h).
 *              Input rows: z, x, g [dim each].
 * Every part of the input rows starts at a multiple of 8 (zero rows in between), in the order given; branches follow one
 * another.  A branch's output (heads * vdim, or dim for MIN_GRU; attention with KEYS_ARE_VALUES: heads * dim) is
 * multiplied by out_scale and also starts at a multiple of 8. */
enum { TEENY_HYBRID_ATTENTION = 0, TEENY_HYBRID_DELTA, TEENY_HYBRID_DECAY, TEENY_HYBRID_MIN_GRU, TEENY_HYBRID_LATENT };
enum {
  TEENY_HYBRID_QK_NORM = 1, TEENY_HYBRID_KEYS_ARE_VALUES = 2, TEENY_HYBRID_SINK = 4, TEENY_HYBRID_OUT_GATE = 8,
  TEENY_HYBRID_VALUE_MIX = 16
};
/* Layer flags: a bias on the fused input projection; norms behind the sublayers. */
enum { TEENY_HYBRID_IN_BIAS = 1, TEENY_HYBRID_POST_NORM = 2 };
/* Feed-forward activations of the gated dense kind: act(gate) * up. */
enum { TEENY_HYBRID_ACT_SILU = 1, TEENY_HYBRID_ACT_GELU_TANH = 2 };

typedef struct {
  int num_layers, num_branches, width, vocab;
  float eps;          /* of every norm of the model */
  float embed_scale;
  float residual_mult; /* factor of what a POST_NORM layer adds to the residual */
  int f32;            /* 0: weights, activations and caches bf16; 1: everything f32 (true f32 products) */
  int max_batch;      /* state slots, and most entries of a step */
  int max_len;        /* most positions of a sequence */
  int max_tokens;     /* most tokens of a step */
  int max_rows;       /* most rows of logits of a step */
  int max_new_tokens; /* capacity of the generated-token history */
} teeny_hybrid_config;

typedef struct {
  int first_branch, num_branches;
  int ff, act;        /* ff = 0: no feed-forward */
  int flags;
} teeny_hybrid_layer;

typedef struct {
  int kind, heads, kv_heads, dim, vdim, rank, q_rank, window, rot_dims, flags;
  float score_scale, out_scale, decay_coef, unit_eps, softcap, rot_scale;
} teeny_hybrid_branch;

typedef struct teeny_hybrid teeny_hybrid;

/* Weights.  Matrices are row-major in the model's element type with rows pad8(columns) elements apart; vectors are f32.
 * Per layer (branch ignored): NORM1, NORM2 [width]; IN [input rows, width]; OUT [width, output columns]; GATE_UP [2 * pad64(ff),
 * width], gate and up rows interleaved in blocks of 64 (zero rows beyond ff); DOWN [width, pad64(ff)].
 * IN_BIAS [input rows] in the model's element type; NORM1_POST, NORM2_POST [width].
 * Per branch of the layer: Q_NORM, K_NORM [dim] (LATENT: [pad8(q_rank)], [pad8(rank)], zero beyond the rank); O_NORM; LOW [heads * dim, rank] (a matrix); DECAY_BIAS, RATE_BIAS [heads *
 * dim]; Z_BIAS, X_BIAS [dim]; DECAY [heads]; INV_FREQ [rot_dims / 2]; SINK [heads]; VALUE_MIX [1].  LATENT, with KR =
 * pad8(rank), DL = KR + rot_dims (a cache row is [c, rotated key part]) and D = rot_dims + dim: UQ [heads * D, q_rank];
 * EXPAND [heads * (D + vdim), DL], which makes a cache row's per-head keys [rotated part, unrotated part], then its values;
 * ABSORB [heads, KR, dim], the key projection transposed; VALUE_UP [heads, vdim, KR].
 * Model: EMBED [vocab, width] (rows width apart), FINAL_NORM, LM_HEAD [vocab, width]. */
enum {
  TEENY_HYBRID_W_NORM1 = 0, TEENY_HYBRID_W_NORM2, TEENY_HYBRID_W_IN, TEENY_HYBRID_W_OUT, TEENY_HYBRID_W_GATE_UP,
  TEENY_HYBRID_W_DOWN, TEENY_HYBRID_W_IN_BIAS, TEENY_HYBRID_W_NORM1_POST, TEENY_HYBRID_W_NORM2_POST,
  TEENY_HYBRID_W_Q_NORM = 50, TEENY_HYBRID_W_K_NORM, TEENY_HYBRID_W_O_NORM, TEENY_HYBRID_W_LOW, TEENY_HYBRID_W_DECAY_BIAS,
  TEENY_HYBRID_W_RATE_BIAS, TEENY_HYBRID_W_Z_BIAS, TEENY_HYBRID_W_X_BIAS, TEENY_HYBRID_W_DECAY, TEENY_HYBRID_W_INV_FREQ,
  TEENY_HYBRID_W_SINK, TEENY_HYBRID_W_VALUE_MIX, TEENY_HYBRID_W_UQ, TEENY_HYBRID_W_EXPAND, TEENY_HYBRID_W_ABSORB,
  TEENY_HYBRID_W_VALUE_UP,
  TEENY_HYBRID_W_EMBED = 100, TEENY_HYBRID_W_FINAL_NORM, TEENY_HYBRID_W_LM_HEAD
};
enum {
  TEENY_HYBRID_BUF_LOGITS = 0, /* element type [rows, pad8(vocab)]: logits of the last step's rows */
  TEENY_HYBRID_BUF_NEXT_IDS,   /* int32 [batch]: token chosen by the last step (input of the next) */
  TEENY_HYBRID_BUF_HISTORY,    /* int32 [max_new_tokens, batch] */
  TEENY_HYBRID_BUF_STATE,      /* int32 [3]: position, live length, tokens generated (of the first sequence) */
  TEENY_HYBRID_BUF_RESIDUAL,   /* f32 [tokens, width]: the residual stream before the last sublayer's output was added ... */
  TEENY_HYBRID_BUF_LAST_DELTA  /* ... and that output (before its POST_NORM), element type [tokens, pad8(width)] */
};

/* Bytes of workspace (activations, states, caches, generation state); 0 if the configuration is not supported.  The
 * arrays are host memory: num_layers layers, num_branches branches. */
size_t teeny_hybrid_workspace_bytes(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches);
/* Bytes of state one slot holds over all branches (the part of the workspace that grows with max_batch alone). */
size_t teeny_hybrid_slot_bytes(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches);
int teeny_hybrid_create(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches,
                        void* workspace, size_t workspace_bytes, teeny_stream_t stream, teeny_hybrid** out);
void teeny_hybrid_destroy(teeny_hybrid* model);
int teeny_hybrid_set_weight(teeny_hybrid* model, int layer, int branch, int which, const void* device_ptr);
/* One step: entry e brings the next lens[e] tokens of slot slots[e], the first at position positions[e]; position 0 starts a
 * new sequence in the slot.  slots, positions, lens (n entries each) and rows (n_rows) are host arrays; ids: device
 * int32, the entries' tokens one after the other.  rows: which of the step's tokens get logits (row numbers in ids).  A
 * slot must not appear twice in a step. */
int teeny_hybrid_step(teeny_hybrid* model, const int* ids, const int* slots, const int* positions, const int* lens, int n,
                      const int* rows, int n_rows, teeny_stream_t stream);
/* Generation over the sequences of the last step: begin picks every entry's first token from the logits of its last
 * token (the step must have asked for exactly one row per entry, in order) and records it; each decode then appends one
 * token per sequence.  decode launches the kernels; capture_decode records one step as a CUDA graph, decode_replay
 * launches it. */
int teeny_hybrid_begin(teeny_hybrid* model, teeny_stream_t stream);
int teeny_hybrid_decode(teeny_hybrid* model, teeny_stream_t stream);
int teeny_hybrid_set_sampling(teeny_hybrid* model, float temperature, int top_k, float top_p, unsigned long long seed);
int teeny_hybrid_capture_decode(teeny_hybrid* model, teeny_stream_t stream);
int teeny_hybrid_decode_replay(teeny_hybrid* model, teeny_stream_t stream);
void* teeny_hybrid_buffer(teeny_hybrid* model, int which);

/* The runner's kernels on their own.  seqs: device int32 [n_seqs][4] = {slot, position of the first token, first row, tokens}
 * per entry; max_len: the longest entry.  f32: element type of the void pointers (0 bf16, 1 f32).  Row strides and column
 * offsets are in elements.
 *
 * Matrix-state recurrences over [slots, heads, dk, dv] f32 states; o [rows, ldo] f32, head h at column h * dv.  mode 0:
 * generalized delta rule (proj columns off_q, off_k, off_v, off_a; wz the decay's low-rank product; w_bias, a_bias [heads * dk]);
 * mode 1: scalar decay per head with silu on q, k, v. */
int teeny_state_scan(int mode, int f32, const void* proj, long long ld, int off_q, int off_k, int off_v, int off_a, const void* wz,
                     long long ld_wz, const float* w_bias, const float* a_bias, const float* decay, float decay_coef,
                     float unit_eps, float* state, float* o, long long ldo, int heads, int dk, int dv, const int* seqs,
                     int n_seqs, int max_len, teeny_stream_t stream);
/* out = o / rms(groups of group_size columns) * weight * sigmoid(gate) * scale */
int teeny_gated_rms_norm(int f32, const float* o, long long ldo, const void* gate, long long ldg, const float* weight, void* out,
                         long long ldout, int rows, int cols, int group_size, float eps, float scale, teeny_stream_t stream);
/* Element-wise gated recurrence with the z, x and gate columns of proj; state [slots, width] f32. */
int teeny_min_gru(int f32, const void* proj, long long ld, int off_z, int off_x, int off_g, const float* z_bias, const float* x_bias,
                  float* state, void* out, long long ldout, int width, float scale, const int* seqs, int n_seqs, int max_len,
                  teeny_stream_t stream);
/* Per-head RMS norm (q_weight / k_weight [dim] f32, or null for none) and rotate-half positions on the first rot_dims
 * dimensions: q [rows, ldq] in place, k_raw -> k_out; angles position * inv_freq[i] in f32. */
int teeny_head_norm_rope(int f32, void* q, long long ldq, const void* k_raw, long long ldkr, void* k_out, long long ldk,
                         const float* q_weight, const float* k_weight, const float* inv_freq, int heads, int kv_heads, int dim,
                         int rot_dims, float eps, const int* seqs, int n_seqs, int max_len, teeny_stream_t stream);
/* Sliding-window attention of every entry's tokens over the ring caches [slots, kv_heads, ring, dim] (keys older than the
 * entry) and the entry's own k_new / v_new rows, which are then appended to the rings.  uniform_fresh: the entries are whole
 * prompts of one length from position 0, rows in order (a faster kernel for head size 128). */
int teeny_window_attention(int f32, const void* q, long long ldq, const void* k_new, long long ldk, const void* v_new, long long ldv,
                           void* k_ring, void* v_ring, int slots, int ring, int window, void* out, long long ldo, int heads,
                           int kv_heads, int dim, int vdim, float score_scale, float out_scale, int uniform_fresh,
                           const int* seqs, int n_seqs, int max_len, teeny_stream_t stream);
/* x [rows, n] f32 += delta (or null); y = rms_norm(x) * weight.  post (or null): rms_norm(delta) * post * mult is added instead. */
int teeny_residual_rms_norm(int f32, float* x, const void* delta, long long ldd, void* y, long long ldy, const float* weight, int rows,
                            int n, float eps, const float* post, float mult, teeny_stream_t stream);
/* Positions and cache append of full attention: rotate-half positions on q [rows, heads, dim] (in place) and on k, which goes to
 * the cache [slots, kv_heads, max_len, dim]; v goes to its cache [.., vdim].  mix_mode 1: v is also copied to v_first [rows,
 * kv_heads * vdim]; 2: v <- (1 - *mix) v + *mix v_first. */
int teeny_rope_cache(int f32, void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* k_cache,
                     void* v_cache, int max_cached, const float* inv_freq, float rot_scale, int heads, int kv_heads, int dim, int vdim,
                     int rot_dims, int mix_mode, void* v_first, const float* mix, const int* seqs, int n_seqs, int max_len,
                     teeny_stream_t stream);
/* Causal attention of every entry's tokens over caches that hold the entries' own keys and values already.  softcap 0: none;
 * sink [heads] or null; gate [rows, ldg] (heads vdim apart) or null.  scratch: teeny_attn_decode_scratch_bytes(entries, heads,
 * 128, max_cached) bytes and `counters` entries * kv_heads words, zero before the first call (both may be null: a slower kernel
 * for single tokens).  host_seqs: the step table in host memory, or null. */
int teeny_cached_attention(int f32, const void* q, long long ldq, void* k_cache, void* v_cache, int slots, int max_cached, void* out,
                           long long ldo, int heads, int kv_heads, int dim, int vdim, float score_scale, float softcap,
                           const float* sink, const void* gate, long long ldg, void* scratch, size_t scratch_bytes,
                           unsigned* counters, const int* seqs, const int* host_seqs, int n_seqs, int max_len, teeny_stream_t stream);
/* Latent attention's front: proj columns off_q [q_rank], off_c [rank], off_r [rot_dims] -> cq [rows, ldcq] = rms_norm * q_weight,
 * the cache row [slots, max_cached, pad8(rank) + rot_dims] and, unless null, the same row in latents [rows, ..]. */
int teeny_latent_prepare(int f32, const void* proj, long long ld, int off_q, int off_c, int off_r, int q_rank, int rank, int rot_dims,
                         const float* q_weight, const float* c_weight, const float* inv_freq, float eps, float rot_scale, void* cq,
                         long long ldcq, void* latents, void* cache, int max_cached, const int* seqs, int n_seqs, int max_len,
                         teeny_stream_t stream);
/* y[t, h * y_head + n] = sum_k x[t, h * x_head + k] w[h, n, k]; with rot_dims > 0 the head's elements x[t, h * x_head + rot_off ..]
 * are rotated (rotate-half) and follow the n columns. */
int teeny_head_linear(int f32, const void* x, long long ldx, long long x_head, const void* w, void* y, long long ldy, long long y_head,
                      int heads, int n, int k, int rows, int rot_dims, int rot_off, const float* inv_freq, float rot_scale, const int* seqs,
                      int n_seqs, teeny_stream_t stream);
/* Causal attention of `heads` query heads over one cached row per token (its first vdim elements are the value): q [rows, ldq]
 * with heads dim apart, cache [slots, max_cached, dim], out with heads vdim apart.  scratch: teeny_latent_attention_scratch_bytes
 * (or null: a long cache is then not shared between CTAs). */
size_t teeny_latent_attention_scratch_bytes(int vdim);
int teeny_latent_attention(int f32, const void* q, long long ldq, int rows, const void* cache, int slots, int max_cached, void* out,
                           long long ldo, int heads, int dim, int vdim, float score_scale, void* scratch, size_t scratch_bytes,
                           const int* seqs, int n_seqs, int max_len, teeny_stream_t stream);

#ifdef __cplusplus
}
#endif
#endif /* TEENY_HYBRID_H_ */
