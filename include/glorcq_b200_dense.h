/*
 * glorcq_b200, unquantized models -- C ABI of the sm_100a kernels behind the decoders whose weights stay in bfloat16
 * (or float32): matrix products with their activation folded in, the stabilised matrix-memory recurrence, latent
 * attention, softmax routing with a correction term, and the norms between them.
 *
 * Same conventions as glorcq_b200.h: device pointers, everything enqueued on the given stream, nothing allocated or
 * synchronised, argument errors decided on the host.  `dtype` names the storage of weights, activations and caches;
 * norms, routing, attention weights and recurrent state are float in both.
 */
#ifndef GLORCQ_B200_DENSE_H
#define GLORCQ_B200_DENSE_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define GLQ_DT_BF16 0
#define GLQ_DT_F32 1

#define GLQ_ACT_NONE 0
#define GLQ_ACT_RELU2 1    /* max(z, 0)^2 */
#define GLQ_ACT_GELU_ERF 2 /* z * Phi(z)  */
#define GLQ_ACT_GELU_TANH 3
/* gated: rows of W in blocks of 16, 8 of the gate and the same 8 of the other half; silu(gate) * other, N / 2 columns */
#define GLQ_ACT_SILU_GLU 4

#define GLQ_GATE_SIGMOID 0
#define GLQ_GATE_SILU 1

const char* glq_dense_status_string(int status);
int glq_dense_last_cuda_error(void);
/* error word of the bounded waits: (code, ., ., block << 32 | thread), zero when no wait ran out */
int glq_dense_debug_error(unsigned long long* out4, int clear);

/* y = alpha * act(x . W^T) for every problem of a list.  W holds the problems' (N, K) matrices one after the other.
 * Plain product: slot_index NULL, one problem of `rows` rows.  Grouped: problem s < *n_slots uses matrix slot_index[s]
 * and entries slot_offset[s] .. + slot_count[s]; entry e reads x row entry_row[e] (NULL: row e) and writes output row e.
 * Columns [0, split) go to y (of `dtype`), columns [split, N) to y32 (float); split = 0 sends all to y32.
 * A gated activation needs N % 16 == 0 and split = N, and writes N / 2 columns of y.
 * mul (not with a gated activation): the activated product is multiplied by mul[mul_row[row] (NULL: row)][column] before
 * it is stored.  residual (split = 0, plain, no mul): y32 += product, and y, unless NULL, receives the sum in `dtype`. */
typedef struct glq_dense_mm {
    int32_t dtype, act, N, K;
    int32_t rows;          /* entries in all (grouped: an upper bound) */
    int32_t n_matrices;
    int32_t max_slots;     /* grouped: upper bound of *n_slots */
    int32_t max_slot_rows; /* grouped: upper bound of slot_count */
    int32_t split;
    float alpha;
    const int32_t* slot_index;
    const int32_t* n_slots;
    const int32_t* slot_count;
    const int32_t* slot_offset;
    const int32_t* entry_row;
    const void* x;
    int64_t ldx;
    const void* W;
    int64_t ldw;           /* row stride of W, 0: K */
    void* y;
    int64_t ldy;
    float* y32;
    int64_t ldy32;
    void* gather;          /* (rows, K) scratch for entry_row on the tensor-core path, or NULL when entry_row is */
    /* up to 8 rows, bf16, instead of x: row = rms_norm over each of hn_heads equal parts of hn_o (rows, K) float, times
     * hn_w (K), times sigmoid(hn_g (rows, K) bf16, row stride hn_ldg) */
    const float* hn_o;
    const void* hn_g;
    int64_t hn_ldg;
    const float* hn_w;
    int32_t hn_heads;
    float hn_eps;
    const void* mul;       /* of dtype, row stride ldmul, mul_rows rows */
    int64_t ldmul;
    const int64_t* mul_row;
    int32_t mul_rows, residual;
} glq_dense_mm_t;
int glq_dense_matmul(const glq_dense_mm_t* a, void* stream);
/* 0: generic kernel, 1: streaming kernel (few rows), 2: tcgen05 kernel */
int glq_dense_matmul_path(const glq_dense_mm_t* a);

/* Residual stream x (rows, C) float, kept by the caller:
 *   embed:      x = table[ids], h = dtype(x), or with hw: h = dtype(rms(x) * hw)
 *   add_norm:   x += layer_norm(y) * w, h = dtype(x); with final_w: h = dtype(layer_norm(x) * final_w)
 *   rms_add:    x += alpha * (rms(y) * w + rms(y2) * w2), h = dtype(rms(x) * hw); rms(v) = v / sqrt(mean(v^2) + eps).
 *               Without w (and w2) y and y2 are added as they are, without hw h = dtype(x); y2, y (nothing is added) and
 *               h may be NULL.  ldy, ldy2: row strides.                                                            */
int glq_dense_embed(int dtype, const int64_t* ids, const void* table, int rows, int C, int vocab, const float* hw, float eps, float* x,
                    void* h, void* stream);
int glq_dense_rms_add(int dtype, const float* y, int64_t ldy, const float* w, const float* y2, int64_t ldy2, const float* w2, float alpha,
                      const float* hw, float eps, int rows, int C, float* x, void* h, void* stream);
int glq_dense_add_norm(int dtype, const float* y, const float* w, const float* final_w, float eps, int rows, int C,
                       float* x, void* h, void* stream);

/* Matrix memory (per head: S (D, V), n (D), running log maximum m), one position after the other:
 *   i = cap tanh((gi + bi) / cap), f = logsigmoid(cap tanh((gf + bf) / cap)), m' = max(f + m, i)
 *   S = e^(f + m - m') S + e^(i - m') k v^T (n alike), o = S^T q / (max(|n.q|, e^-m') + 1e-6), q scaled by D^-1/2
 *   out = rms_norm_per_head(o) * norm_w * sigmoid(g)
 * qkvg (B*T, ldp): q (H*D) | k (H*D) | v (H*V) | g (H*V) of `dtype`; gates (B*T, ldg) float: i (H) | f (H).
 * State: S (B, H, slices, D, 32), n (B, H, slices, D), m (B, H, slices) float, slices = glq_mlstm_slices(V).             */
typedef struct glq_mlstm {
    int32_t dtype, B, T, H, D, V;
    int32_t state_idle;    /* step: 1 when the launch right before this one on the stream does not touch this state */
    float gate_cap, eps;
    const void* qkvg;
    int64_t ldp;
    const float* gates;
    int64_t ldg;
    const float* bias_i;
    const float* bias_f;
    const float* norm_w;
    float* S;
    float* n;
    float* m;
    float* o;              /* (B*T, H*V) float: the recurrence's output before norm and gate */
    void* out;             /* (B*T, H*V) of dtype; step: NULL leaves norm and gate to the caller (glq_dense_matmul, hn_o) */
    void* workspace;       /* chunk */
    size_t workspace_bytes;
} glq_mlstm_t;
int glq_mlstm_slices(int V);
size_t glq_mlstm_workspace_bytes(const glq_mlstm_t* a);
int glq_mlstm_step(const glq_mlstm_t* a, void* stream);    /* recurrent form, any T */
int glq_mlstm_chunk(const glq_mlstm_t* a, void* stream);   /* chunkwise form on the tensor cores, bf16 */

/* Linear attention with decay (per head: S (D, V)), one position after the other:
 *   q, k: the first rot_dims elements turned by the position (pairs (i, i + rot_dims/2), or with rot_pairs (2i, 2i + 1)),
 *   times q_scale, k_scale;  S = diag(alpha) S + k v^T,  o = S^T q,
 *   out = rms_norm_per_head(o) * norm_w * gate(g)     (norm_w: head h at norm_w + h * norm_stride, or NULL)
 * alpha: decay[h], or per key channel sigmoid(z)^(1/tau) with z = a2 . a + a2b (a2 (H*D, rank) of `dtype`, a2b (H*D) float,
 * a (B*T, lda) float).  q, k (B*T, H*D), v, g (B*T, H*V) of `dtype`, all with row stride ldp; cos/sin (max_len, rot_dims/2).
 * State: S (B, H, slices, D, 32) float, slices = glq_decay_slices(V).                                                   */
typedef struct glq_decay {
    int32_t dtype, B, T, H, D, V, rank, rot_dims, rot_pairs, max_len;
    int32_t norm_stride, gate;
    int32_t state_idle;    /* step: 1 when the launch right before this one on the stream does not touch this state */
    float q_scale, k_scale, eps, tau;
    const void* q;
    const void* k;
    const void* v;
    const void* g;
    int64_t ldp;
    const float* decay;
    const float* a;
    int64_t lda;
    const void* a2;
    const float* a2b;
    const int64_t* start;  /* device: position of the first new token */
    const float* cos_t;
    const float* sin_t;
    const float* norm_w;
    float* S;
    float* o;              /* (B*T, H*V) float scratch: the recurrence's output before norm and gate */
    void* out;             /* (B*T, H*V) of dtype */
    void* workspace;       /* chunk */
    size_t workspace_bytes;
} glq_decay_t;
int glq_decay_slices(int V);
size_t glq_decay_workspace_bytes(const glq_decay_t* a);
int glq_decay_step(const glq_decay_t* a, void* stream);             /* recurrent form, any T */
int glq_decay_chunk_supported(const glq_decay_t* a);
int glq_decay_chunk(const glq_decay_t* a, void* stream);            /* chunkwise form on the tensor cores, bf16 */

/* Grouped-query attention: query head h reads key head h / (H/G).  q, k: the first rot_dims elements of every head turned
 * by the position (as above), then with qk_norm divided by sqrt(mean(.^2) + eps); scores (q . k) * scale, causal softmax.
 * q (B*T, H*D; turned in place where the form asks for it), k (B*T, G*D), v (B*T, G*V; may be k itself: the keys as
 * projected are then the values), all of `dtype` with row stride ldp.  kc (B, max_len, G, D), vc (B, max_len, G, V): the
 * rows start .. start + T - 1 are written.                                                                          */
typedef struct glq_gqa {
    int32_t dtype, B, T, H, G, D, V, rot_dims, rot_pairs, qk_norm, max_len;
    int32_t S;             /* start + T on the host; needed by form 2 only */
    int32_t state_idle;    /* form 1: 1 when the launch right before this one on the stream does not touch this cache */
    float scale, eps;
    const int64_t* start;  /* device: position of the first new token */
    void* q;
    const void* k;
    const void* v;
    int64_t ldp;
    const float* cos_t;    /* (max_len, rot_dims / 2) */
    const float* sin_t;
    void* kc;
    void* vc;
    void* out;             /* (B*T, H*V) of dtype */
    void* workspace;       /* form 1 */
    size_t workspace_bytes;
} glq_gqa_t;
/* 0: generic, 1: decode form (up to 8 positions), 2: tcgen05 form */
int glq_gqa_form(const glq_gqa_t* a);
size_t glq_gqa_decode_workspace_bytes(const glq_gqa_t* a);
int glq_gqa(const glq_gqa_t* a, void* stream);

/* Latent attention.  Cache row of a position: latent (K) | rotated key part (R), `dtype`, row stride ldc.
 * prep (before prefill): latents of the new positions are RMS-normed (weight norm_w), the shared key part and every
 *   head's rotated query part (in place in q) are turned, and the cache rows start .. start + T - 1 are written.
 *   q (B*T, ldq): head by head D | R.  ckr (B*T, ldk) float: K | R.  cos/sin (max_len, rot_dims / 2) float.
 * absorbed (decode, short portions, any T in float32; turns q and writes the cache rows itself): scores against the cached latents themselves with
 *   q' = uk^T q, then the value projection uv of the weighted latent, times sigmoid of the head's gate.
 *   ukt (H, K, D), uv (H, V, K) of dtype, gate (B*T, ldk) float at column offset given by the pointer.
 * prefill (bf16): keys and values already projected, kv (B*S, ldkv): H*D keys | H*V values for positions 0..S-1,
 *   S = start + T; the rotated part comes from the cache.                                                        */
typedef struct glq_latent {
    int32_t dtype, B, T, H, D, R, V, K;
    int32_t rot_dims, max_len;
    float scale, eps;
    const int64_t* start;  /* device: position of the first new token */
    void* q;
    int64_t ldq;
    const float* ckr;
    int64_t ldk;
    const float* gate;
    const float* norm_w;
    const float* cos_t;
    const float* sin_t;
    void* cache;           /* (B, max_len, ldc) */
    int64_t ldc;
    const void* ukt;
    const void* uv;
    void* out;             /* (B*T, H*V) of dtype */
    const void* kv;
    int64_t ldkv;
    const void* vt;        /* prefill on tcgen05: values transposed, (B, H*V, ldvt); kv then holds keys only */
    int64_t ldvt;
    int32_t S;             /* prefill: positions in kv */
    int32_t max_splits;    /* absorbed: upper bound of the position splits */
    void* workspace;
    size_t workspace_bytes;
} glq_latent_t;
int glq_latent_prep(const glq_latent_t* a, void* stream);
size_t glq_latent_absorbed_workspace_bytes(const glq_latent_t* a);
int glq_latent_absorbed(const glq_latent_t* a, void* stream);
/* 0: not covered, 1: mma form (kv = keys | values), 2: tcgen05 form (kv = keys, vt = values transposed) */
int glq_latent_prefill_form(const glq_latent_t* a);
int glq_latent_prefill(const glq_latent_t* a, void* stream);

/* Routing: s = softmax(logits) over E experts and `identity` pass-through experts, the `top` largest of
 * s + correction are chosen (ties: lowest index), weighted by s.  sel (n, top), wts (n, top).
 * Then the entry lists of the experts below E, slots of at most `chunk` rows (0: one slot per expert):
 * lists needs glq_route_list_ints(...) ints, laid out as the offsets in glq_route_lists describe.                */
typedef struct glq_route {
    int32_t n, E, identity, top, chunk, reserved;
    const float* logits;
    int64_t ldl;
    const float* correction;
    int32_t* sel;
    float* wts;
    float* entry_scale;
    int32_t* tok_entries;  /* (n, top): entry of (token, slot), -1 for pass-through */
    int32_t* entry_row;    /* 2 * n * top */
    int32_t* active;       /* each list: 3 * max_slots ints */
    int32_t* slot_count;
    int32_t* slot_offset;
    int32_t* n_active;     /* 2 ints */
    int32_t max_slots, reserved2;
    int32_t* block_counts; /* ceil(n * top / 512) * E ints */
} glq_route_t;
int glq_route_max_slots(int n, int E, int top, int chunk);
int glq_route(const glq_route_t* a, void* stream);
/* x += layer_norm(sum_j wts_j * (entry_out[tok_entries_j] or x)) * w, h as in add_norm */
int glq_dense_combine_norm(int dtype, const void* entry_out, int64_t lde, const int32_t* tok_entries, const float* wts, int top,
                           const float* w, const float* final_w, float eps, int rows, int C, float* x, void* h, void* stream);

/* logits = scale * x . W^T for up to 8 rows with the arg-max of every row folded in (bf16 weights, float logits) */
size_t glq_dense_head_workspace_bytes(void);
int glq_dense_head(const void* x, int64_t ldx, const void* W, int B, int V, int H, float scale, float* logits, int64_t ldl,
                   int64_t* argmax_out, void* workspace, size_t workspace_bytes, int32_t* counter, void* stream);

#ifdef __cplusplus
}
#endif
#endif
