/*
 * dense_b200.h — C ABI of libdense_b200.so: decoder layers with dense bf16 (or fp32) weights on NVIDIA B200 (sm_100a).
 * Projections with fused row preparation and epilogues, latent attention (keys and values in one low-rank row per token),
 * grouped-query attention with one or two softmax maps per head, and a selective state-space recurrence.
 *
 * Every pointer inside the argument blocks is a DEVICE pointer.  Entry points are asynchronous on `stream`, never
 * synchronise, allocate or free, and return 0 or a negative GPTQ_ERR_* code (gptq_b200.h).
 *
 * dtype: 0 = bf16 weights and activations with fp32 accumulation, 1 = fp32 throughout (no reduced-precision products).
 * Weights are [N, K] with K contiguous.  Feature sizes (K, head parts, latent rank) are multiples of 16: the caller pads
 * weights and rows with zeros; sizes that enter a mean are passed as true sizes beside the padded ones.
 */
#ifndef DENSE_B200_H
#define DENSE_B200_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define DENSE_CONTROL_BYTES 16384      /* control buffer of an engine: zeroed once; its last word is the status word */

/* epilogues of dense_matmul */
#define DENSE_EPI_F32     0            /* out fp32 [M, ldo] = scale * result */
#define DENSE_EPI_T       1            /* out in the activation dtype */
#define DENSE_EPI_GATED   2            /* weight rows in groups of 16: 8 gate rows, 8 up rows; out[8 g + j] = act(gate_j) * up_j */
#define DENSE_EPI_QKV     3            /* rotary queries | raw fp32 latent rows | sigmoid gates */
#define DENSE_EPI_LOGITS  4            /* F32, and with `best` set the greedy choice per row (decode rows only) */
#define DENSE_EPI_TABLE   5            /* out in the activation dtype = act(result) * tab[token, tab_col + n] */

#define DENSE_EPI_MIXED   6            /* the first n_q columns in the activation dtype to out, n_kv further ones in fp32 to kv_out [M, n_kv] */

/* activations of GATED and TABLE */
#define DENSE_ACT_SILU 0
#define DENSE_ACT_GELU 1               /* the tanh form */

/* norms of a row (mean, variance and mean square over `width` of the `ld` columns) */
#define DENSE_NORM_NONE  0
#define DENSE_NORM_LAYER 1             /* (v - mean) / sqrt(var + eps) */
#define DENSE_NORM_RMS   2             /* v / sqrt(mean(v^2) + eps) */
#define DENSE_MAX_NORM_GROUPS 256

/* Row preparation.  x = table[token] (+ pos_table[pos]), or x_in; with y set, x += y_norm(y) * gain + shift (gain absent: 1,
 * shift absent: 0).  x_out (optional, never the same as x_in) receives x.  The prepared row is fin_norm(x) * fin_w + fin_b (each
 * optional); an RMS norm may work on fin_groups equal parts of the row, each by its own mean square (then y must be absent). */
typedef struct {
	const void *x_in;                  /* fp32, or (x_t) in the activation dtype */
	int x_t;
	float *x_out;
	const float *y;
	const float *gain, *shift;
	const float *fin_w, *fin_b;
	const void *table;
	const int64_t *token;
	int64_t vocab;
	const void *pos_table;             /* [max_pos, ld] */
	const int32_t *pos;                /* [M] */
	int max_pos;
	int y_norm, fin_norm, fin_groups;
	int width, ld;
	float eps;
	int *status;
} dense_rows_t;

typedef struct {
	int mode;
	void *out;
	int64_t ldo;
	float scale;
	/* QKV: n_q query columns, heads of head_dim; in each head the pairs (2i, 2i+1) of [rot_at, rot_at + rot_dims) are rotated by
	 * the table row of pos[m]; n_kv raw columns; n_gate gate columns */
	int n_q, head_dim, rot_at, rot_dims, n_kv, n_gate;
	const float *cos_t, *sin_t;        /* [max_pos, rot_dims / 2] */
	const int32_t *pos;                /* [M] */
	int max_pos;
	void *q_out;
	int q_f32;
	float *kv_out;
	float *gate_out;
	int *status;
	/* LOGITS */
	unsigned long long *best;          /* [M], zero before and after every launch */
	unsigned *ticket;
	int64_t *tok;                      /* receives the arg-max (lowest index on ties) */
	int32_t *pos_inout;                /* incremented */
	/* GATED, TABLE */
	int act;
	const void *tab;                   /* [tab_rows, tab_ld] in the activation dtype */
	int64_t tab_ld, tab_rows;
	int tab_col;
	const int64_t *tab_token;          /* [M] */
} dense_epilogue_t;

/* Latent attention, absorbed form.  A cache row is [latent (kv_rank) | rotated key part (rot_dim)]. */
typedef struct {
	int M, rows_per_seq;               /* query rows, rows_per_seq consecutive rows per sequence */
	int heads, dim, rot_dim, vdim, kv_rank, kv_width, rot_dims, max_seq, splits;
	float scale, eps;
	const int32_t *pos;                /* [M] */
	const float *q;                    /* [M, heads * (dim + rot_dim)] fp32, rotated */
	const void *w_uk, *w_uv;           /* [heads * dim, kv_rank], [heads * vdim, kv_rank] */
	const float *kv_raw;               /* [M, kv_rank + rot_dim], or NULL: another layer has written the cache rows */
	const float *kv_norm;              /* [kv_rank] */
	const float *cos_t, *sin_t;
	void *cache;                       /* [sequences, max_seq, kv_rank + rot_dim] */
	void *qa_hi, *qa_lo;               /* bf16 [M, heads, kv_rank + rot_dim] */
	float *qa_f32;                     /* dtype 1 */
	float *part_ml;                    /* [M, heads, splits, 2] */
	float *part_acc;                   /* [M, heads, splits, kv_rank] */
	const float *gate;                 /* [M, gate_ld], or NULL */
	int gate_ld;
	void *out;                         /* [M, out_ld] */
	int64_t out_ld;
	int *status;
} dense_latent_t;

/* Latent attention of a prompt portion of one sequence, expanded form, bf16. */
typedef struct {
	int t, start, S;                   /* t query rows at positions start ..; S = start + t keys */
	int heads, dim, rot_dim, vdim, kv_rank;
	float scale;
	const void *q;                     /* bf16 [t, heads * (dim + rot_dim)], rotated */
	const void *k;                     /* bf16 [S, heads * dim] */
	const void *vt;                    /* bf16 [heads * vdim, ldv]: values transposed, ldv a multiple of 8 */
	int64_t ldv;
	const void *cache;                 /* bf16 [S, kv_rank + rot_dim] */
	const float *gate;
	int gate_ld;
	void *out;                         /* bf16 [t, out_ld] */
	int64_t out_ld;
	int *status;
} dense_latent_prefill_t;

/* Grouped-query attention with `maps` (1 or 2) softmax maps per head over shared values.  Query head h reads key / value head
 * h / (heads / kv_heads).  Per map: score = cap * tanh(q . k * scale / cap) (cap 0: q . k * scale), causal softmax, a_map = sum p v.
 * Result per head: o = a_1, or a_1 - lambda * a_2; with out_norm o / sqrt(mean(o^2) + eps); times out_mul.
 * A raw row is [queries: heads * maps * dim | keys: kv_heads * maps * dim | values: kv_heads * vdim]; queries and keys are
 * RMS-normed per head and map when q_norm / k_norm are given. */
typedef struct {
	int M, rows_per_seq;               /* query rows, rows_per_seq consecutive rows per sequence */
	int heads, kv_heads, maps, dim, vdim;      /* dim and vdim padded to multiples of 16 */
	int dim_true, vdim_true;           /* what the norms average over */
	int max_seq, splits;
	float scale, cap, eps, lambda, out_mul;
	float bound;                       /* |q . k * scale / cap| is known to be at most this (0: nothing known); used by the prompt kernel */
	int out_norm;
	const int32_t *pos;                /* [M] */
	const void *raw;                   /* [M, raw_ld] fp32, or (raw_t) in the activation dtype */
	int raw_t;
	int64_t raw_ld;
	const float *q_norm, *k_norm;      /* [dim] or NULL */
	void *k_cache;                     /* [sequences, max_seq, kv_heads * maps * dim] */
	void *v_cache;                     /* [sequences, max_seq, kv_heads * vdim] */
	void *q_hi, *q_lo;                 /* bf16 [M, heads * maps * dim]: normed queries times scale (/ cap), high part and remainder */
	float *q_f32;                      /* dtype 1 */
	float *part_ml;                    /* [M, heads * maps, splits, 2] */
	float *part_acc;                   /* [M, heads * maps, splits, vdim] */
	void *out;                         /* [M, out_ld] */
	int64_t out_ld;
	int *status;
} dense_gqa_t;

/* Selective state-space recurrence with a short causal convolution in front (Mamba-2).  A raw row is
 * [z: inner | x: inner, B: groups * state, C: groups * state], inner = heads * vdim, sections at z_at and conv_at; dt is separate.
 *   u = silu(conv(x, B, C) + conv_b);  dt = softplus(dt + dt_bias);  S = exp(a * dt) S + dt x B^T;  y = S C + d * x;  out = y * silu(z)
 * The last `taps` convolution inputs of a sequence are kept in a ring (slot = position mod taps).  At position 0 the state and
 * the inputs before it are taken as zero, whatever the buffers hold. */
#define DENSE_SSM_CHUNK 128
typedef struct {
	int M, rows_per_seq;
	int heads, vdim, state, groups, taps;
	int z_at, conv_at, conv_ld;        /* conv_ld: padded number of convolution channels */
	int64_t raw_ld, dt_ld;
	const void *raw;                   /* [M, raw_ld] */
	const float *dt;                   /* [M, dt_ld] */
	const int32_t *pos;                /* [M] */
	const float *conv_w, *conv_b;      /* [taps, conv_ld] (last tap: the current token), [conv_ld] */
	const float *dt_bias, *a, *d;      /* [heads] */
	float *ring;                       /* [sequences, taps, conv_ld] */
	float *s;                          /* [sequences, heads, vdim, state] */
	void *u;                           /* scratch of portions: [M, conv_ld], the type of raw */
	float *chunk_s;                    /* scratch of dense_ssm_chunked: [sequences, chunks, heads, vdim, state] */
	float *chunk_decay;                /* [sequences, chunks, heads] */
	void *out;                         /* [M, out_ld], the type of raw */
	int64_t out_ld;
	int *status;
} dense_ssm_t;

int dense_version(void);
int dense_last_cuda_error(void);

/* y = epilogue(rows x W^T).  With `rows` the kernel prepares its input rows itself (few rows only, see dense_decode_rows_ok),
 * else x is [M, ldx].  w is [N, ldw].  Chooses the decode kernel, the tensor-core kernel or the fp32 kernel by shape. */
int dense_matmul(const void *x, int64_t ldx, const void *w, int64_t ldw, int M, int K, int N, int dtype, const dense_rows_t *rows, const dense_epilogue_t *epi,
				 float *scratch, int *status, void *stream);
/* fp32 values of scratch with which dense_matmul splits the K range of a narrow output (two kernels); 0: it would not.  scratch may be
 * NULL. */
int64_t dense_matmul_scratch(int M, int K, int N, int dtype);
int dense_decode_rows_ok(int M, int K, int dtype);      /* the decode kernel (and row preparation inside it) covers M rows of K */
int dense_prepare_rows(const dense_rows_t *rows, int M, void *h, int64_t ldh, int dtype, void *stream);

int dense_latent_splits(int M, int heads, int max_seq, int dtype);
int dense_latent_append(const dense_latent_t *args, int dtype, void *stream);       /* cache rows only */
int dense_latent_absorb(const dense_latent_t *args, int dtype, void *stream);       /* absorbed queries and, with kv_raw, cache rows */
int dense_latent_attend(const dense_latent_t *args, int dtype, void *stream);
int dense_latent_value(const dense_latent_t *args, int dtype, void *stream);
int dense_latent_prefill_ok(int dim, int rot_dim, int vdim);
int dense_latent_prefill(const dense_latent_prefill_t *args, void *stream);

int dense_gqa_splits(int M, int heads, int kv_heads, int maps, int max_seq, int dtype);
int dense_gqa_append(const dense_gqa_t *args, int dtype, void *stream);      /* normed queries, cache rows */
int dense_gqa_attend(const dense_gqa_t *args, int dtype, void *stream);      /* partial results per key range */
int dense_gqa_merge(const dense_gqa_t *args, int dtype, void *stream);       /* key ranges and maps into the output */
/* A prompt portion of one sequence at positions start .. start + M - 1 on the tensor cores, bf16: keys and values from the
 * cache, queries from q_hi.  dense_gqa_prefill_maps: 2: both maps at once, writes out; 1: writes partials (splits = 1) for
 * dense_gqa_merge; 0: sizes that do not fit. */
int dense_gqa_prefill_maps(int maps, int dim, int vdim);
int dense_gqa_prefill(const dense_gqa_t *args, int start, void *stream);

int dense_ssm_step(const dense_ssm_t *args, void *stream);                   /* rows_per_seq = 1, raw fp32 */
int dense_ssm_conv(const dense_ssm_t *args, int dtype, void *stream);        /* portions: u */
int dense_ssm_scan(const dense_ssm_t *args, void *stream);                   /* portions, raw and u fp32: out, state, ring, token by token */
/* The same for bf16 raw and u in chunks.  One tensor-core kernel per sequence when vdim and state are multiples of 16 and state is at
 * most 128, else three kernels, which need chunk_s and chunk_decay (dense_ssm_chunked_scratch = 1). */
int dense_ssm_chunked(const dense_ssm_t *args, void *stream);
int dense_ssm_chunked_scratch(const dense_ssm_t *args);

#ifdef __cplusplus
}
#endif
#endif
