/* C ABI of the row-wise and mixer kernels of layered (hybrid) decoders: per-layer mixers over a latent KV cache or a
 * recurrent state, gated 32-bit residual streams, norms without statistics, row-normalised activations. Mirrored by
 * ctypes.Structures in crosspool_b200/native/__init__.py; XP_ABI_VERSION covers these structs too.
 *
 * `f32` selects the element type of activations, caches and weights: 0 bf16, 1 fp32. */
#ifndef XPOOL_MIXER_API_H_
#define XPOOL_MIXER_API_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* resid[r] = ids ? table[ids[r]] : resid[r] + (sum of parts)[r] * sigmoid(gate[r]);  out[i] = norm(resid[r]),
 * with r = sel ? sel[i] : i. With sel the residual is read only. */
typedef struct XpResidNormArgs {
  float* resid;          /* [*, hidden] */
  const void* parts[8];  /* activations [*, ld_part] */
  const void* gate;      /* optional logits [*, ld_gate]; null: no gate */
  const int* ids;        /* optional: start the residual from the embedding table */
  const void* table;     /* [vocab, hidden] */
  const int* sel;        /* optional row selection */
  const float* weight;   /* [hidden] */
  const float* bias;     /* optional [hidden] */
  const float* alpha;    /* dynamic tanh: one device float */
  void* out;             /* [rows, ld_out]; null: residual update only */
  int rows, hidden, nparts, ld_part, ld_gate, ld_out, vocab;
  int kind;              /* 0 rms, 1 layernorm, 2 dynamic tanh */
  float eps;
  int f32;
} XpResidNormArgs;

/* out = coef0 N(z) + coef1 N(z^2) + coef2 N(z^3) + coef3 over each row, N dividing by the root mean square. */
typedef struct XpPolyNormArgs {
  const void* z;
  const float* coef;     /* 4 device floats */
  void* out;
  int rows, cols, ld_z, ld_out;
  float eps;
  int f32;
} XpPolyNormArgs;

/* out = rmsnorm(o) * weight * sigmoid(gate), o in fp32. */
typedef struct XpGatedRmsArgs {
  const float* o;
  const float* weight;
  const void* gate;      /* logits [rows, ld_gate] */
  void* out;
  int rows, cols, ld_o, ld_gate, ld_out;
  float eps;
  int f32;
} XpGatedRmsArgs;

/* Norms behind a sublayer: y = branches[0], or with branch weights the mean over the branches of rmsnorm(b_i) * branch_w[i];
 * v = resid[r] + rmsnorm(y) * weight (or v = table[ids[r]]), stored to resid[r];
 * out[i] = out_weight ? rmsnorm(v) * out_weight : v,  with r = sel ? sel[i] : i. With sel the residual is read only. */
typedef struct XpPostNormArgs {
  float* resid;            /* [*, hidden] */
  const void* branches[2]; /* activations [*, ld_branch[i]] */
  const float* branch_w[2];/* [hidden], or null: a single branch is taken as it is */
  const int* ids;          /* optional: start the residual from the embedding table */
  const void* table;       /* [vocab, hidden] */
  const int* sel;          /* optional row selection */
  const float* weight;     /* [hidden] */
  const float* out_weight; /* optional [hidden] */
  void* out;               /* [rows, ld_out]; null: residual update only */
  int rows, hidden, nbranches;
  int ld_branch[2];
  int ld_out, vocab;
  float eps;
  float embed_scale;       /* ids: the table's rows are multiplied by this; 0 = 1 */
  int f32;
} XpPostNormArgs;

/* out = rmsnorm(o) * weight * silu(gate), o in fp32, the norm over each head of `dim` columns. */
typedef struct XpHeadGateArgs {
  const float* o;        /* [rows, heads * dim] */
  const float* weight;   /* [dim], or [heads * dim] with per_head_weight */
  const void* gate;      /* logits [rows, ld_gate] */
  void* out;             /* [rows, ld_out] */
  int rows, heads, dim, ld_o, ld_gate, ld_out;
  float eps;
  int f32;
  int per_head_weight;
  int sigmoid_gate;      /* sigmoid instead of silu */
} XpHeadGateArgs;

/* out = act(min(g, limit)) (clamp(u, +-limit) + up_add), act(g) = g sigmoid(alpha g (1 + cubic g^2)), g and u the halves of
 * z's rows, in fp32. */
typedef struct XpGluArgs {
  const float* z;        /* [rows, ld_z]: g (cols), u (cols) */
  float* out;            /* [rows, ld_out] */
  int rows, cols, ld_z, ld_out;
  float limit, up_add, alpha, cubic;
} XpGluArgs;

/* Elementwise, in fp32; out may be z. kind 0: out = act(z) * e, act as above; 1: out = z * sigmoid(e); 2: out = max(z, 0)^2. */
typedef struct XpGateMulArgs {
  const float* z;        /* [rows, ld_z] */
  const float* e;        /* [rows, ld_e], kinds 0 and 1 */
  float* out;            /* [rows, ld_out] */
  int rows, cols, ld_z, ld_e, ld_out;
  float alpha, cubic;
  int kind;
} XpGateMulArgs;

/* Between the projection and grouped-query attention, per token row: RMS norm of query and key heads, rotation of their first
 * 2 rot_pairs channels (the order of the two does not matter for a norm without a weight; one with a weight comes first),
 * queries laid out [rows, kv_heads, group_pad, dq], keys and values written to the cache row of the token, everything
 * zero-padded. Values may be the projected keys (v_off = k_off). With pool > 0 the first pool_rows rows (row r of table row r)
 * also store the means of the blocks that they complete (XpBlockMeanArgs). */
typedef struct XpGroupedPrepArgs {
  const void* proj;      /* [rows, ld_proj]: q (heads x dim), k (kv_heads x dim), v (kv_heads x vdim) at the offsets */
  const float* q_norm;   /* [dim], or null: no weight */
  const float* k_norm;
  const int* slots;      /* [rows] cache row, -1: none */
  void* k_cache;         /* [tokens, kv_heads, dq] */
  void* v_cache;         /* [tokens, kv_heads, dv] */
  void* q_out;
  int rows, heads, kv_heads, group_pad, dim, vdim, dq, dv, ld_proj, q_off, k_off, v_off;
  float eps;
  int f32;
  int norm;              /* queries and keys are divided by their root mean square */
  int rot_pairs;         /* 0: no rotation */
  int rot_positions;
  int interleaved;       /* pairs (2 i, 2 i + 1) instead of (i, i + rot_pairs) */
  const float* rot;      /* [rot_positions, rot_pairs, 2]: cos, sin */
  const int* positions;  /* [rows], rotation and pooling */
  const int* block_table;/* pooling */
  void* k_pool;          /* [pages, pool_page, kv_heads, dq] */
  void* v_pool;
  int pool, pool_page, pool_rows, page_size, max_blocks;
} XpGroupedPrepArgs;

/* Means over blocks of `pool` cached tokens: every row whose position completes block b stores the mean of the block's keys and
 * values in row b % pool_page of page block_table[b / pool_page] of k_pool and v_pool. */
typedef struct XpBlockMeanArgs {
  const void* k_cache;   /* [pages, page_size, kv_heads, dq] */
  const void* v_cache;
  void* k_pool;
  void* v_pool;
  const int* row_seq;    /* [rows] table row, or null: row r uses table row r */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] < 0: padding row */
  const int* block_table;
  int rows, kv_heads, dq, dv, page_size, max_blocks, pool, pool_page;
  int f32;
} XpBlockMeanArgs;

/* Between the projection and grouped-query attention: causal convolution over time of every query, key and value channel
 * (conv_w null: none), rotary positions on the first 2 rot_pairs channels of queries and keys (pairs (i, i + rot_pairs)),
 * queries laid out [rows, kv_heads, group_pad, dq], keys and values written to the cache row of the token, zero-padded.
 * own_kv = 0: queries only. The convolution's inputs are kept per slot as a ring, position p in entry p % taps. */
typedef struct XpConvRopeArgs {
  const void* proj;      /* [rows, ld_proj]: q (heads x dim), k (kv_heads x dim), v (kv_heads x vdim) at the offsets */
  const float* conv_w;   /* [taps, channels], channels = q, k, v; the last tap belongs to the token itself */
  void* ring;            /* [slots, taps, channels] activations */
  const float* rot;      /* [rot_positions, rot_pairs, 2]: cos, sin */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] cache row, -1: none */
  const int* state_slots;/* [seqs] */
  const int* q_starts;   /* [seqs] prefill: first row */
  const int* q_lens;     /* [seqs] prefill: rows */
  void* k_cache;         /* [tokens, kv_heads, dq] */
  void* v_cache;         /* [tokens, kv_heads, dv] */
  void* q_out;
  int rows, seqs, max_q, heads, kv_heads, group_pad, dim, vdim, dq, dv, own_kv, ld_proj, q_off, k_off, v_off, taps, rot_pairs, rot_positions;
  int row_floats;        /* set by the library */
  int f32;
} XpConvRopeArgs;

/* Attention of single rows against the paged cache of grouped keys and values, plain form for any sizes. Row r attends to
 * positions[r] + 1 tokens of block-table row row_seq[r]; softcap > 0: scores become softcap tanh(score / softcap); window >
 * 0: only to the last `window` of them and to the first `keep_first`. */
typedef struct XpGroupedAttnArgs {
  const void* q;         /* [rows, kv_heads, group_pad, dq] */
  const void* k_cache;   /* [pages, page_size, kv_heads, dq] */
  const void* v_cache;   /* [pages, page_size, kv_heads, dv] */
  void* out;             /* [rows, ld_out]: heads x vdim */
  const void* gate;      /* optional output gate logits [rows, ld_gate]: one per head, or per output element (gate_elems) */
  const int* row_seq;    /* [rows], or null: row r uses table row r */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] < 0: padding row (zeros are stored) */
  const int* block_table;
  int rows, heads, kv_heads, group_pad, dim, vdim, dq, dv, ld_gate, ld_out, page_size, max_blocks;
  float scale, softcap;
  int f32;
  int window, keep_first, gate_elems;
  const float* sink;         /* [heads], or null: exp(sink) joins the softmax's sum */
  const float* sigmoid_bias; /* [heads]: weights are sigmoid(score + bias), not normalised (null: softmax) */
  const void* k_pool;        /* pool > 0: keys and values of the blocks behind the window, seen beside it */
  const void* v_pool;
  int pool, pool_page;
} XpGroupedAttnArgs;

/* Linear attention with a decay per key channel: S = diag(alpha) S + k v^T, o = S^T q qscale, log alpha = -softplus(-z) / tau.
 * Decode computes z itself (z = a2 a1 + a2_bias) and stores rmsnorm(o) * norm * silu(gate); prefill reads z and stores o. */
typedef struct XpGatedLinearArgs {
  const void* proj;      /* [rows, ld_proj]: q, k (heads x dim), v, gate (heads x vdim), a1 (rank) at the offsets */
  const float* z;        /* prefill: [rows, heads * dim] */
  const void* a2;        /* decode: [heads * dim, ld_a2] */
  const float* a2_bias;  /* decode: [heads * dim] */
  const float* norm;     /* decode: [vdim] */
  float* state;          /* [slots, heads, dim, vdim] */
  void* out;             /* decode: activations [rows, ld_out]; prefill: fp32 [rows, ld_out] */
  const int* positions;
  const int* slots;      /* [rows] KV slot of the row, < 0: padding row */
  const int* state_slots;
  const int* q_starts;
  const int* q_lens;
  float* ws;             /* chunked prefill, segs > 1: [seqs, heads, segs, dim * vdim + dim] */
  void* records;         /* chunked prefill: xp_gated_linear_record_bytes(); z is overwritten */
  int rows, seqs, max_q, heads, dim, vdim, ld_proj, ld_out, q_off, k_off, v_off, g_off, a_off, rank, ld_a2;
  int segs, seg_tokens, force_sequential;
  float inv_tau, qscale, eps;
  int f32;
} XpGatedLinearArgs;

/* Gated delta rule: S = g S; u = beta (v - S^T k); S = S + k u^T; o = S^T q. The convolution's inputs are kept per slot as a
 * ring, position p in entry p % taps. Decode does everything from the projection to rmsnorm(o) * norm * silu(gate); prefill
 * convolves into qkv (activations behind silu, unnormalised), writes the factors that make queries and keys unit vectors
 * (queries times qscale), beta and log g, and runs the recurrence on those. */
typedef struct XpDeltaArgs {
  const void* proj;      /* [rows, ld_proj] at the offsets: q, k (kv_heads x dim), v (heads x vdim), gate, b, a (heads) */
  const float* conv_w;   /* [channels, taps], channels = q, k, v */
  void* conv_state;      /* [slots, taps, channels] activations */
  const float* neg_a;    /* [heads] -exp(A_log) */
  const float* dt_bias;  /* [heads] */
  const float* norm;     /* decode: [vdim] */
  float* state;          /* [slots, heads, dim, vdim] */
  void* out;             /* decode: activations [rows, ld_out]; prefill: fp32 [rows, ld_out] */
  void* qkv;             /* prefill: [rows, channels] */
  float* qk_scale;       /* prefill: [rows, 2, kv_heads] */
  float* beta_g;         /* prefill: [rows, 2, heads]: beta, log g */
  void* ws;              /* chunked prefill: xp_delta_ws_bytes() */
  const int* positions;
  const int* slots;
  const int* state_slots;
  const int* q_starts;
  const int* q_lens;
  int rows, seqs, max_q, heads, kv_heads, dim, vdim, taps, ld_proj, ld_out, q_off, k_off, v_off, g_off, b_off, a_off;
  int force_sequential;
  float qscale, eps;
  int f32;
} XpDeltaArgs;

/* Matrix memory with exponential gates: i = cap tanh(z_i / cap), f = log sigmoid(cap tanh(z_f / cap)); m' = max(f + m, i);
 * S' = e^(f + m - m') S + e^(i - m') k v^T, n' likewise with k alone; o = S'^T q / (max(|n' . q|, e^-m') + 1e-6), q scaled by
 * qscale. A head's state is [dim x vdim | n (dim) | m] in head_state floats. Decode stores rmsnorm(o) * norm * sigmoid(gate);
 * prefill stores o. */
typedef struct XpMemoryArgs {
  const void* proj;      /* [rows, ld_proj]: q, k (heads x dim), v, gate (heads x vdim) at the offsets */
  const float* gates;    /* [rows, ld_gates]: z_i and z_f (heads) at their offsets, biases added */
  const float* norm;     /* decode: [heads * vdim] */
  float* state;          /* [slots, heads, head_state] */
  void* out;             /* decode: activations [rows, ld_out]; prefill: fp32 [rows, ld_out] */
  float* planes;         /* prefill: [3, heads, rows] */
  float* before;         /* prefill: [seqs, heads, dim + 1] */
  float* ws;             /* chunked prefill, segs > 1: [seqs, heads, segs, head_state] */
  const int* positions;
  const int* slots;      /* [rows] KV slot of the row, < 0: padding row */
  const int* state_slots;
  const int* q_starts;
  const int* q_lens;
  int rows, seqs, max_q, heads, dim, vdim, head_state, ld_proj, ld_gates, ld_out, q_off, k_off, v_off, g_off, i_off, f_off;
  int segs, seg_tokens, force_sequential;
  float qscale, cap, eps;
  int f32;
} XpMemoryArgs;

/* Latent attention, per token row: normalise the latent, rotate the shared key part, write both to the cache row of the
 * token; rotate the rotary part of every query head and lay the queries out for the absorbed form
 * (q_plain head-major, q_abs columns [kv_rank, +rot)) and/or the expanded form (q_exp). Queries may come from a buffer of
 * their own (q), as a map of the q_rank projected columns at ql_off that still lacks the division by their root mean square. */
typedef struct XpLatentPrepArgs {
  const void* proj;      /* [rows, ld_proj]: q at q_off (heads x (dim + rot)), latent + key at kv_off (kv_rank + rot) */
  const float* norm_w;   /* [kv_rank] */
  const double* freq;    /* [rot_dims / 2] rotary frequencies */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] cache row, -1: none */
  void* cache;           /* [tokens, ld_cache] */
  void* q_plain;         /* [heads, qp_rows, dim_p], or null */
  void* q_abs;           /* [heads, qp_rows, ld_abs], or null */
  void* q_exp;           /* [rows, heads, dq_pad] zero-padded, or null */
  int rows, heads, dim, rot, rot_dims, kv_rank, ld_proj, q_off, kv_off, ld_cache, qp_rows, dim_p, ld_abs, dq_pad;
  int abs_rows;          /* rows < abs_rows are laid out for the absorbed form, the others for the expanded one */
  float eps;
  int f32;
  const void* q;         /* optional [rows, ld_q]: heads x (dim + rot), instead of the columns at q_off */
  int ld_q, q_rank, ql_off;
  int interleaved;       /* pairs (2 i, 2 i + 1) instead of (i, i + rot_dims / 2) */
} XpLatentPrepArgs;

/* Attention of single rows against the latent cache (keys: the first kv_rank + rot columns of a cache row shared by
 * every head; values: its first kv_rank columns). Row r attends to positions[r] + 1 tokens of table row row_seq[r]. */
typedef struct XpLatentAttnArgs {
  const void* q;         /* [heads, q_rows, ld_q] (kv_rank + rot columns) */
  const void* cache;     /* [pages, page_size, ld_cache] */
  void* out;             /* [heads, q_rows, ld_out] (kv_rank columns) */
  const void* gate;      /* optional per-head output gate logits [rows, ld_gate] */
  const int* row_seq;    /* [rows] block-table row, or null: row r uses table row r */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] < 0: padding row (zeros are stored) */
  const int* block_table;
  float* ws;             /* split partials */
  uint32_t* status;      /* optional: set to 8 when a bounded wait ran out */
  int rows, heads, kv_rank, rot, q_rows, ld_q, ld_cache, ld_out, ld_gate, page_size, max_blocks;
  int num_splits, chunk_tokens;
  float scale;
  int f32;
  int force_simt;        /* plain kernel */
  int window;            /* > 0: rows see the last `window` of their tokens; slices count over those */
} XpLatentAttnArgs;

/* Copies the cached latents of each sequence to a dense workspace: sequence i's ctx + q tokens start at row starts[i]. With a
 * window the copy begins at the 64-token boundary at or before the first token that the first query sees. */
typedef struct XpLatentGatherArgs {
  const void* cache;
  void* out;             /* [*, ld_cache] */
  const int* block_table;
  const int* ctx_lens;
  const int* q_lens;
  const int* starts;     /* [n_seqs] first workspace row */
  int n_seqs, max_len, page_size, max_blocks, ld_cache, elem_bytes, window;
} XpLatentGatherArgs;

/* Decayed linear attention S = decay S + k v^T, o = S^T q; the state of sequence slot s is
 * state[s][heads][dim][vdim] in fp32. A sequence whose first row sits at position 0 starts from a zero state. */
typedef struct XpLinearAttnArgs {
  const void* proj;      /* [rows, ld_proj]: q, k (heads x dim) and v (heads x vdim) at the three offsets */
  float* state;
  const float* decay;    /* [heads] */
  const float* decay_pow;/* [heads, 65]: decay^0 .. decay^64 */
  float* out;            /* [rows, heads * vdim] fp32 */
  const int* positions;  /* [rows] */
  const int* slots;      /* [rows] KV slot of the row, < 0: padding row */
  const int* state_slots;/* [seqs] */
  const int* q_starts;   /* [seqs] prefill: first row */
  const int* q_lens;     /* [seqs] prefill: rows */
  float* ws;             /* [seqs, heads, segs, dim, vdim] states between segments, segs > 1 */
  int rows, seqs, heads, dim, vdim, ld_proj, q_off, k_off, v_off;
  int force_sequential;
  int segs, seg_tokens;  /* chunked prefill: segments of a portion that run at the same time (multiples of 64 tokens) */
  int f32;
} XpLinearAttnArgs;

int xp_resid_norm(const XpResidNormArgs* a, void* stream);
int xp_polynorm(const XpPolyNormArgs* a, void* stream);
int xp_gated_rms(const XpGatedRmsArgs* a, void* stream);
int xp_post_norm(const XpPostNormArgs* a, void* stream);
int xp_head_gate(const XpHeadGateArgs* a, void* stream);
int xp_glu_f32(const XpGluArgs* a, void* stream);
int xp_gate_mul_f32(const XpGateMulArgs* a, void* stream);
int xp_grouped_prep(const XpGroupedPrepArgs* a, void* stream);
int xp_block_mean(const XpBlockMeanArgs* a, void* stream);
int xp_conv_rope_decode(const XpConvRopeArgs* a, void* stream);
int xp_conv_rope_prefill(const XpConvRopeArgs* a, void* stream);
int xp_grouped_attn(const XpGroupedAttnArgs* a, void* stream);
int xp_memory_decode(const XpMemoryArgs* a, void* stream);
int xp_memory_prefill(const XpMemoryArgs* a, void* stream);
int xp_gated_linear_decode(const XpGatedLinearArgs* a, void* stream);
int xp_gated_linear_prefill(const XpGatedLinearArgs* a, void* stream);
int xp_delta_decode(const XpDeltaArgs* a, void* stream);
int xp_delta_prep(const XpDeltaArgs* a, void* stream);
int xp_delta_prefill(const XpDeltaArgs* a, void* stream);
int xp_delta_chunked(const XpDeltaArgs* a, void* stream);           /* 1: sizes not covered */
int xp_gated_linear_chunked(const XpGatedLinearArgs* a, void* stream);
size_t xp_delta_ws_bytes(int rows, int seqs, int heads);
size_t xp_gated_linear_record_bytes(int rows, int seqs, int heads);
int xp_latent_prep(const XpLatentPrepArgs* a, void* stream);
int xp_latent_attn(const XpLatentAttnArgs* a, void* stream);
int xp_latent_gather(const XpLatentGatherArgs* a, void* stream);
int xp_linear_attn_decode(const XpLinearAttnArgs* a, void* stream);
int xp_linear_attn_prefill(const XpLinearAttnArgs* a, void* stream);
/* out[b][r][n] = sum_k x[b][r][k] w[b][n][k] (* out_scale) (+ bias), silu below column silu_cols, in true fp32 (no
 * reduced-precision product). */
int xp_gemm_f32(const float* x, const float* w, const float* bias, float* out, int rows, int n, int k, int ldx, int ldw, int ldo,
                int batch, int64_t sx, int64_t sw, int64_t so, float out_scale, int silu_cols, void* stream);
/* Grouped form over a device table of int4 {group, first feature (multiples of 128), first row, row end}, tiles of at most 64
 * rows: group g uses w rows [g * w_rows_per_group, + n). max_tiles bounds *n_tiles. */
int xp_gemm_f32_grouped(const float* x, const float* w, float* out, const void* tiles, const int* n_tiles, int max_tiles, int n, int k,
                        int ldx, int ldw, int ldo, int w_rows_per_group, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* XPOOL_MIXER_API_H_ */
