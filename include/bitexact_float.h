/* C ABI of libbitexact_float.so: sm_100a kernels of the float models (hybrids of recurrent and attention layers served
 * from bf16 weights, or in 32-bit throughout). Same conventions as bitexact_b200.h: device pointers unless said
 * otherwise, BX_* status codes, `stream` is a cudaStream_t, calls are asynchronous and allocate nothing.
 *
 * Element type T of a call: dtype BXF_BF16 (bfloat16) or BXF_F32 (float, no reduced-precision product anywhere).
 * "row" = one token of the step. Rows of one sequence are consecutive and in position order.
 * Leading dimensions (ld*) and group strides (gs*) count elements. In bf16, operands of the products start on 16-byte
 * boundaries and have leading dimensions and group strides that are multiples of 8; the extents themselves are free.
 */
#ifndef BITEXACT_FLOAT_H
#define BITEXACT_FLOAT_H

#include "bitexact_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

#define BXF_BF16 0
#define BXF_F32 1

#define BXF_MAX_TOP 32          /* experts per token */
#define BXF_MAX_EXPERTS 1024
#define BXF_MAX_STREAMS 8       /* residual streams */
#define BXF_MAX_TAPS 16         /* of a causal convolution */
#define BXF_MAX_STATE 512       /* key channels of a matrix-valued recurrent state */

/* Row flags (bxf_row_flags): first / last row of its sequence in this step, first token of the sequence, padding. */
#define BXF_ROW_FIRST 1
#define BXF_ROW_LAST 2
#define BXF_ROW_START 4
#define BXF_ROW_PAD 8

/* What a product does with its accumulators. */
#define BXF_EPI_STORE 0         /* out[m, n] = act(acc + main_bias[n]); rows n >= n_main go to side[m, n - n_main] = acc + bias (float) */
#define BXF_EPI_ADD 1           /* out (float) [m, n] += acc */
#define BXF_EPI_ROPE 2          /* n < n_main: out[m, n] = acc; the others are rotated pairs, see rot_* */
#define BXF_EPI_GATE 3          /* out[m, n] = acc * gate[m, group] */
#define BXF_EPI_GLU 4           /* rows 2 i and 2 i + 1 are a pair: out (T) [m, i] = act(acc[2 i]) * acc[2 i + 1]; N even */

#define BXF_OUT_T 0
#define BXF_OUT_F32 1
#define BXF_OUT_I64 2           /* round(v * 2^24), the fixed-point logits of the integer sampler */

#define BXF_ACT_NONE 0
#define BXF_ACT_RELU2 1         /* max(z, 0)^2 */
#define BXF_ACT_XIELU 2         /* z > 0: act_p z^2 + z / 2; else act_q (e^z - 1 - z) + z / 2 */
#define BXF_ACT_GELU 3          /* tanh form */
#define BXF_ACT_SOFTCAP 4       /* act_q tanh(act_p z) */
#define BXF_ACT_SCALE 5         /* act_p z */

typedef struct {
  int kind, out_type, act, n_main;
  float act_p, act_q;
  void* out;                    /* T, float or int64 */
  int64_t ldo, gso;
  float* side;                  /* BXF_EPI_STORE, n >= n_main */
  int64_t lds;
  const float* bias;            /* [N - n_main] or NULL */
  const float* gate;            /* BXF_EPI_GATE: float [M, groups], row stride ldg */
  int64_t ldg;
  const float* cs;              /* BXF_EPI_ROPE: (cos, sin) pairs float [M, rot_dim / 2, 2] */
  void* rot_out;                /* T: row m, head h, entry j -> rot_out[m * ldr + h * hsr + j] */
  int64_t ldr, hsr;
  int rot_dim;
  int pad_;
  const float* main_bias;       /* BXF_EPI_STORE: [n_main] or NULL */
} bxf_epilogue;

/* The recurrence of a minGRU layer after its three products (update, candidate, output gate). */
typedef struct {
  const float *bias_z, *bias_x; /* [width] */
  float* state;                 /* [slots, width] */
  const int* flags;             /* [M] row flags */
  const int64_t* seq;           /* [M] state slot of each row */
  void* out;                    /* T [M, ldo]: state * silu(gate) */
  int64_t ldo;
} bxf_gru;

/* Residual streams x float [M, streams, D] (hyper-connections). In this order: ids != NULL: every stream = embed[ids]; else,
 * with y (a sublayer's output, float [M, D]), x_t = sum_s mix[s, t] x_s + out[t] y. Then u = sum_s in[s] x_s (in NULL: the plain
 * sum) goes to h (T [M, ldh]) as u / sqrt(mean(u^2) + eps) * w and, with sum, to sum float [M, D]. Without h the streams
 * themselves are left as they were. */
typedef struct {
  float* x;
  const int64_t* ids;
  const void* embed;            /* T [vocab, D] */
  int64_t vocab;
  const float *y, *out, *mix;   /* mix [streams, streams] = [from, to] */
  const float* in;
  const float* w;               /* [D] */
  void* h;
  int64_t ldh;
  float* sum;
  float eps;
  int streams, D, pad_;
} bxf_streams_step;

/* After the projection of a grouped-query attention layer, y T [M, ldy] = [q: heads dim | k: kv_heads dim | v: kv_heads vdim]:
 * q and k each divided by the root mean square of all their rows (times q_norm / k_norm; NULL: no norm), the first rot_dims
 * entries of every head turned by cs (entry i with i + rot_dims / 2), q to T [kv_heads, M, heads / kv_heads, ldq], k and v to
 * the cache row of the token's slot: T [pages, kv_heads, page, ldc] with the value from entry voff on. */
typedef struct {
  const void* y;
  int64_t ldy;
  int heads, kv_heads, dim, vdim, rot_dims, page;
  const float *q_norm, *k_norm; /* [heads dim], [kv_heads dim] */
  const float* cs;              /* bxf_angles */
  const int64_t* slot;          /* [M]; negative: row 0 */
  void* q;
  int64_t ldq;
  void* cache;
  int64_t ldc, voff;
  float eps;
  int pad_;
} bxf_gqa_rows;

/* A causal convolution per channel over the rows of a sequence, followed by silu: c[m, ch] = silu(b[ch] + sum_j w[j, ch]
 * u[m - taps + 1 + j, ch]); rows before the step come from the sequence's state (its last taps - 1 inputs, oldest first),
 * rows before the sequence are zero. */
typedef struct {
  const void* u;                /* T [M, ldu] */
  int64_t ldu;
  const float *w, *b;           /* [taps, channels], [channels] */
  void* state;                  /* T [slots, taps - 1, channels] */
  const int* flags;             /* [M] row flags */
  const int64_t *seq, *pos;     /* [M] */
  int channels, taps;
} bxf_conv;

#define BXF_DECAY_CHANNEL 0     /* one decay per key channel */
#define BXF_DECAY_HEAD 1        /* one decay per head */

/* Linear recurrence with a matrix state per head: S_t = diag(a_t) S_(t-1) + k_t v_t^T (K x V), o_t = S_t^T q_t.
 * q, k, v are columns of y (T [M, ldy]) from q0, k0, v0 on: q and k by group (K entries each; head h uses group
 * h / (heads / groups)), v by head.
 *   BXF_DECAY_CHANNEL (groups = heads): side float [M, lds] holds `rank` entries; z = a2 side + a2_b (a2 float [rank, heads K]),
 *     a = sigmoid(z)^inv_tau; q is multiplied by q_scale.
 *   BXF_DECAY_HEAD: side float [M, lds] holds the step sizes before softplus; dt = softplus(side), a = exp(-exp(A_log) dt),
 *     k is multiplied by dt, and skip[h] v_t is added to o_t.
 * state float [slots, heads, K, V] is advanced by the rows of every sequence; out T [M, ldo] = o (heads concatenated). */
typedef struct {
  int kind, heads, groups, K, V, rank, q0, k0, v0;
  int batch;                    /* bxf_recurrence, bf16: 1 = sequences of one row (decoding) are the usual case */
  const void* y;
  int64_t ldy;
  const float* side;
  int64_t lds;
  const float *a2, *a2_b;
  float inv_tau, q_scale;
  float* decays;                /* bxf_recurrence, BXF_DECAY_CHANNEL: scratch float [M, heads K] */
  const float *A_log, *skip;
  float* state;
  const int* flags;
  const int64_t* seq;
  void* out;
  int64_t ldo;
} bxf_recurrence_rows;

/* Gate and norm of a recurrent layer's output o (T [M, ldo], n entries in `parts` equal parts), z T [M, ldz]:
 * gate_first: out = rms(o silu(z)) w, else out = rms(o) w silu(z); every part by its own root mean square, w float [wn] used
 * periodically. With conv.w the convolution's state is advanced over the rows of the step. */
typedef struct {
  const void *o, *z;
  int64_t ldo, ldz;
  const float* w;
  void* out;
  int64_t ldout;
  int n, parts, wn, gate_first;
  float eps;
  int pad_;
  bxf_conv conv;
} bxf_gate_rows;

int bxf_version(void);
long long bxf_launch_count(void);
int bxf_device_status(void);            /* as bx_device_status, for the kernels of this library */
int bxf_clear_device_status(void);
int bxf_set_device_status(int value);

/* acc[g][m, n] = sum_k x[g][m, k] w[g][n, k] in 32-bit accumulation, then the epilogue (HOST pointer, copied).
 *   w T [groups, N, ldw] (group stride gsw), x T [groups, M, ldx] (group stride gsx)
 *   counts NULL: every group has the M rows. Else int32 [groups]: the rows of x are ordered by group, group e has
 *   counts[e] of the M rows (experts; gsx unused, and out's rows are the rows of x).
 *   tile 0 = automatic; bf16: 16, 32, 64 = token rows of a weight-major tile, 128, 256 = weight rows of a token-major
 *   tile (128 tokens). Results do not depend on it beyond rounding. */
int bxf_linear(int dtype, const void* w, int64_t ldw, int64_t gsw, const void* x, int64_t ldx, int64_t gsx, int groups,
               int M, int N, int K, const int* counts, const bxf_epilogue* epi, int tile, void* stream);

/* minGRU: acc_z, acc_x, acc_g = three products of the normed row; z = sigmoid(acc_z + bias_z), u = acc_x + bias_x,
 * candidate = u + 1/2 (u >= 0) or sigmoid(u), S = (1 - z) S + z candidate along the rows of a sequence, from `state` (zero
 * on BXF_ROW_START) and back into it; out = S silu(acc_g).
 *   bxf_gru_linear  products and recurrence in one kernel, for at most bxf_gru_rows(dtype) rows (decoding, short portions):
 *                   w T [3, width, ldw] (planes z, x, g), x T [M, ldx]
 *   bxf_gru_scan    the recurrence alone, any M: y float [M, 3 width] = [acc_z | acc_x | acc_g] (overwritten); fold: scratch
 *                   float [bxf_gru_chunks(M), width, 2] */
int bxf_gru_rows(int dtype);
int bxf_gru_chunks(int M);
int bxf_gru_linear(int dtype, const void* w, int64_t ldw, const void* x, int64_t ldx, int M, int width, int K,
                   const bxf_gru* gru, void* stream);
int bxf_gru_scan(int dtype, float* y, float* fold, int M, int width, const bxf_gru* gru, void* stream);

/* flags int32 [M] from seq / slot / pos int64 [M] (slot < 0: padding row). */
int bxf_row_flags(const int64_t* seq, const int64_t* slot, const int64_t* pos, int* flags, int M, void* stream);

/* x float [M, D]: ids != NULL: x = embed[ids] (embed T [V, D], vocab V); else, with top > 0,
 * x += sum_k weight[m, k] y[place[m, k]] (y float [*, D]: the experts' outputs). Then, with h, the layer norm
 * (w, b float [D]) of x as T [M, ldh]. zero / nzero: int32 words cleared on the way (expert counters). */
int bxf_norm(int dtype, float* x, const int64_t* ids, const void* embed, int64_t V, const float* y, const int* place,
             const float* weight, int top, const float* w, const float* b, float eps, void* h, int64_t ldh, int* zero,
             int nzero, int M, int D, void* stream);

/* Routing: logits float [M, ldl] over `experts` -> chosen int32 [M, top], weight float [M, top] (softmax over the
 * chosen), rank int32 [M, top] (place within the expert); counts int32 [experts] must be zero and receives the sizes. */
int bxf_route(const float* logits, int64_t ldl, int experts, int top, int* chosen, float* weight, int* rank, int* counts,
              int M, void* stream);
/* Rows of h T [M, ldh] gathered in expert order into hp T [M * top, ldh]; place int32 [M, top] = the row of each pair. */
int bxf_gather(int dtype, const void* h, int64_t ldh, int D, const int* chosen, const int* rank, const int* counts,
               int experts, int top, void* hp, int* place, int M, void* stream);

/* After the first projection of a latent attention layer, y float [M, ldy] = [query latent (q_rank) | key latent
 * (kv_rank) | rotated key part (rot_dim) | head gates (heads)]:
 *   cq T [M, ldcq] = RMS norm of the query latent (weight wq), gate float [M, heads] = sigmoid of the gates,
 *   cs float [M, rot_dim / 2, 2] = (cos, sin) of pos * freq, and the cache row of the token's slot (T [*, ldc]):
 *   [RMS norm of the key latent (weight wkv) | rotated key part]. slot int64 [M] (negative: row 0). */
int bxf_latent_prepare(int dtype, const float* y, int64_t ldy, int q_rank, int kv_rank, int rot_dim, int heads,
                       const float* wq, const float* wkv, float eps, const float* freq, const int64_t* pos,
                       const int64_t* slot, void* cq, int64_t ldcq, void* cache, int64_t ldc, float* cs, float* gate,
                       int M, void* stream);

/* Attention over the latent cache (keys and values are the cache rows themselves; the value part is the first kv_rank
 * entries), one sliding window, a sink per head in the denominator.
 *   q T [M, heads, ldq] (first kv_rank + rot_dim entries used), cache T [nb, bs, ldc], bt int32 / int64 [*, nblk],
 *   seq int64 [M] table row of each query row, pos int64 [M]; window 0: none; sink float [heads] or NULL
 *   tiles int32 [ntiles, 3] (table row, first query row, rows) or NULL (every row by itself)
 *   out T [M, heads, ldo]; scratch of bxf_latent_attention_scratch bytes (may be NULL: no split over keys)
 *   variant 0 automatic, 1 one CTA per (row, head), 2 tensor cores. */
size_t bxf_latent_attention_scratch(int M, int heads, int kv_rank);
int bxf_latent_attention_tile(int heads);     /* query rows of a tile of the tensor-core kernel (at least 1) */
int bxf_latent_attention(int dtype, const void* q, int64_t ldq, int M, int heads, int kv_rank, int rot_dim,
                         const void* cache, int64_t ldc, int bs, int nb, const void* bt, int bt_is64, int64_t bt_stride,
                         int nblk, const int64_t* seq, const int64_t* pos, const int* tiles, int ntiles, int window,
                         const float* sink, float scale, void* out, int64_t ldo, void* scratch, size_t scratch_bytes,
                         int variant, void* stream);

/* cs float [M, half, 2] = (cos, sin) of pos * freq[i] (freq double [half], angles reduced in double). */
int bxf_angles(const double* freq, int half, const int64_t* pos, float* cs, int M, void* stream);
int bxf_gqa_prepare(int dtype, const bxf_gqa_rows* rows, int M, void* stream);

/* Grouped-query attention over a paged cache of [key | value] rows (T [nb, kv_heads, bs, ldc], value from entry voff on, a
 * multiple of 8 in bf16), otherwise like bxf_latent_attention. q T [kv_heads, M, heads / kv_heads, ldq]; out T [M, ldo] =
 * heads concatenated; tiles as above with bxf_latent_attention_tile(heads / kv_heads) rows. */
size_t bxf_gqa_attention_scratch(int M, int heads, int kv_heads, int vdim);
int bxf_gqa_attention(int dtype, const void* q, int64_t ldq, int M, int heads, int kv_heads, int dim, int vdim,
                      const void* cache, int64_t ldc, int64_t voff, int bs, int nb, const void* bt, int bt_is64,
                      int64_t bt_stride, int nblk, const int64_t* seq, const int64_t* pos, const int* tiles, int ntiles,
                      int window, const float* sink, float scale, void* out, int64_t ldo, void* scratch,
                      size_t scratch_bytes, int variant, void* stream);

int bxf_streams(int dtype, const bxf_streams_step* step, int M, void* stream);
int bxf_causal_conv(int dtype, const bxf_conv* conv, void* out, int64_t ldo, int M, void* stream);
int bxf_recurrence(int dtype, const bxf_recurrence_rows* rows, int M, void* stream);
/* The same over prompts, in chunks of up to 64 rows on the tensor cores. bxf_recurrence_chunk_rows: rows of a chunk, 0 when the
 * sizes or the element type do not fit (bxf_recurrence takes those). q0, k0, v0, ldy multiples of 8. */
typedef struct {
  const int* runs;              /* int32 [nruns, 3] = (first row, rows, first chunk) of every sequence of the step */
  const int* chunks;            /* int32 [nchunks, 2] = (first row, rows): every run cut at multiples of the chunk rows, in order */
  const int* segments;          /* int32 [nsegments, 3] = (first row, rows, first chunk): every run cut at multiples of chunks;
                                   they are computed side by side. nsegments 0: one CTA walks a whole run */
  const int* spans;             /* int32 [nruns, 3] = (first row, first segment, segments) */
  int nruns, nchunks, nsegments, pad_;
} bxf_chunk_table;
int bxf_recurrence_chunk_rows(int dtype, int K, int V);
size_t bxf_recurrence_chunk_scratch(int kind, int M, int chunks, int segments, int heads, int K, int V);
int bxf_recurrence_chunks(int dtype, const bxf_recurrence_rows* rows, const bxf_chunk_table* table, void* scratch,
                          size_t scratch_bytes, int M, void* stream);
int bxf_gated_norm(int dtype, const bxf_gate_rows* rows, int M, void* stream);

#ifdef __cplusplus
}
#endif
#endif
