/* socket_b200_blocks — C ABI of the decoder building blocks beside the sparse-attention step:
 * residual stream and norms, gated units, softmax attention with chunk and window masks, distance bias,
 * capped scores and sinks (prefill and split-KV decode), rotary keys that share their cache rows with
 * the values, attention on low-rank latents, a selective state-space mixer and a matrix-memory mixer.
 *
 * Same conventions as socket_b200.h: device pointers, sizes and a stream; kernels are enqueued and the
 * call returns; nothing allocates device memory; 0 or a negative sk_status; conditions that only the
 * device can see are OR-ed into an optional device status word (SK_DEV_*) and the access is skipped.
 *
 * `dtype` is the element type of activations and weights: SK_BF16 or SK_F32.  Residual streams, norms,
 * scores, softmax, angles and recurrent state are fp32 in both.
 *
 * A portion of a sequence is S consecutive tokens of each of B sequences, the first at position
 * `start`, or at *pos when `pos` (device int64) is given: the form a captured decode step uses.
 */
#ifndef SOCKET_B200_BLOCKS_H_
#define SOCKET_B200_BLOCKS_H_

#include "socket_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

SK_API int skb_abi_version(void);
SK_API const char* skb_status_string(int status);
SK_API const char* skb_last_error(void);

/* x[row] = table[tokens[row]] * scale in fp32; x_copy (or NULL) gets the same rows.  A token outside
 * [0, vocab) sets SK_DEV_INDEX_OUT_OF_RANGE and reads as zero. */
SK_API int skb_embed_rows(const int64_t* tokens, const void* table, int dtype, int64_t rows, int64_t vocab, int width,
                          float scale, float* x, float* x_copy, int32_t* status, void* stream);

/* One step of the fp32 residual stream x [rows, width], with the next sublayer's input:
 *   in_mode  SKB_IN_NONE     x stays
 *            SKB_IN_ADD_NORM x += y / rms(y) * w_in
 *            SKB_IN_REPLACE  x = y + w_in            (w_in [width], added to every row)
 *            SKB_IN_ADD      x += y
 *   out_mode SKB_OUT_NONE    nothing
 *            SKB_OUT_NORM    out [rows, width]   = x / rms(x) * w_out
 *            SKB_OUT_CONCAT  out [rows, 2 width] = [x ; x0]
 *            SKB_OUT_LAYER_NORM  out [rows, width] = (x - mean(x)) / rms(x - mean(x)) * w_out
 * rms(v) = sqrt(mean(v^2) + eps).  y rows are y_ld elements apart, of y_dtype (dtype or SK_F32). */
enum { SKB_IN_NONE = 0, SKB_IN_ADD_NORM = 1, SKB_IN_REPLACE = 2, SKB_IN_ADD = 3 };
enum { SKB_OUT_NONE = 0, SKB_OUT_NORM = 1, SKB_OUT_CONCAT = 2, SKB_OUT_LAYER_NORM = 3 };
typedef struct sk_residual_params {
    float* x;
    const void* y;
    const void* w_in;
    const float* x0;
    const void* w_out;
    void* out;
    int64_t rows, y_ld;
    int width, in_mode, out_mode, dtype, y_dtype;
    float eps;
} sk_residual_params;
SK_API int skb_residual_norm(const sk_residual_params* p, void* stream);

/* Gated unit of a feed-forward; gate and up rows are `ld` elements apart, out rows out_ld:
 *   SKB_GLU_CLAMPED  out = g * sigmoid(slope * g) * (u + 1), g = min(gate, limit), u = clamp(up, -limit, limit)
 *   SKB_GLU_SILU     out = gate * sigmoid(gate) * up */
enum { SKB_GLU_CLAMPED = 0, SKB_GLU_SILU = 1 };
SK_API int skb_glu(const void* gate, const void* up, int dtype, int64_t rows, int ff, int64_t ld, int kind, float limit,
                   float slope, void* out, int64_t out_ld, void* stream);

/* Keys and values of a portion into rings of `ring` rows: position p goes to row p % ring of
 * k_cache [B, ring, k_row] / v_cache [B, ring, v_row].  SKB_RING_CHUNK writes only the positions of the
 * last block of `ring` positions (the others cannot be visible to a later token of a chunked mask),
 * SKB_RING_WINDOW the last `ring` positions.  v and v_cache may be NULL (rows that hold both).
 * With `pos`, S must be 1. */
enum { SKB_RING_CHUNK = 0, SKB_RING_WINDOW = 1 };
SK_API int skb_ring_append(const void* k, const void* v, int dtype, int B, int S, int64_t k_bs, int64_t k_ss,
                           int64_t v_bs, int64_t v_ss, int k_row, int v_row, int ring, int keep, const int64_t* pos,
                           int64_t start, void* k_cache, void* v_cache, void* stream);

/* Queries and cache rows of attention whose values are its unrotated keys.  q_in rows [H, dim] and k_in
 * rows [G, dim] (in_ld elements apart) of B x S tokens; the first rot_dims elements of a head are turned
 * by the position's angles (element j with element j + rot_dims / 2).  A cache row holds, per head,
 *   [key as projected (dim) | turned elements (rot_dims)]
 * so that the value is row[0 .. dim) and the key is row[rot_dims .. rot_dims + dim), in the element order
 * [unturned | turned]; q_out [B, S, H, dim] has the same order.  angles [n_pos, rot_dims / 2, 2] fp32.
 *   rows_out [B, rows_cap, G, dim + rot_dims]; token s goes to row prev + s, and rows 0 .. prev - 1 get
 *   positions start - prev .. start - 1 out of `ring` [B, ring_rows, ...] (position p in row p % ring_rows);
 *   with `pos` (S = 1) the token goes to row pos % rows_cap: rows_out is the ring itself and prev = 0. */
typedef struct sk_rotary_rows_params {
    const void *q_in, *k_in, *ring;
    void *q_out, *rows_out;
    const float* angles;
    const int64_t* pos;
    int32_t* status;
    int64_t in_ld, start, n_pos, rows_cap, ring_rows;
    int dtype, B, S, H, G, dim, rot_dims, prev;
} sk_rotary_rows_params;
SK_API int skb_rotary_rows(const sk_rotary_rows_params* p, void* stream);

/* Softmax attention of a portion:
 *   score(i, j) = cap(<q_i, k_j> * scale) + bias[h, min(i - j, bias_len - 1)],  j <= i; when chunk > 0 also
 *   j / chunk == i / chunk (integer division), and when window > 0 also i - j < window;
 *   cap(s) = softcap * tanh(s / softcap) when softcap > 0, else s;
 *   out_i = sum_j exp(score) v_j / (sum_j exp(score) + exp(sink[h]))
 * Query head h reads key/value head h / (H / G).  Strides in elements: _bs batch, _ss / _ts token or
 * key row, _hs head; the last dimension is contiguous.  Key row r holds position kv_start + r, or,
 * with ring != 0 (one token per call), position floor(i / chunk) * chunk + r, or, without a chunk, the
 * latest position up to i that is r modulo kv_rows (kv_rows <= window).  kv_rows rows exist.
 * Keys and values may be overlapping slices of the same rows: the decode kernel then reads a row once.
 * `path`: SKB_ATTN_AUTO picks the kernel, the others pin one (SK_ERR_UNSUPPORTED outside its shapes).
 * `workspace` (skb_attn_workspace_bytes; need not be cleared) serves the split decode kernel. */
enum { SKB_ATTN_AUTO = 0, SKB_ATTN_ROWS = 1, SKB_ATTN_PREFILL_TC = 2, SKB_ATTN_DECODE = 3 };
typedef struct sk_attn_params {
    const void *q, *k, *v;
    void* out;
    const float *bias, *sink;      /* [H, bias_len] or NULL; [H] or NULL */
    const int64_t* pos;
    int32_t* status;
    void* workspace;
    size_t workspace_bytes;
    int64_t q_bs, q_ss, q_hs, k_bs, k_ts, k_hs, v_bs, v_ts, v_hs, o_bs, o_ss, o_hs;
    int64_t start, kv_start, kv_rows, bias_len;
    int dtype, B, S, H, G, dqk, dv, chunk, window, ring, path;
    float scale, softcap;
} sk_attn_params;
SK_API size_t skb_attn_workspace_bytes(const sk_attn_params* p);
SK_API int skb_attn(const sk_attn_params* p, void* stream);
/* which kernel SKB_ATTN_AUTO takes for these parameters (an SKB_ATTN_* value) */
SK_API int skb_attn_path(const sk_attn_params* p);

/* Latent attention, cache side: dkv rows [rank | rot] become cache rows [latent | rotated part] of
 * cache [B, cap, cache_ld]: the first `rank` elements RMS-normed with norm_w, the last `rot` turned by
 * the position's angles (pairs (2i, 2i+1) of the first rot_dims).  The rotated parts of the queries,
 * q rows [H, dim + rot], are turned in place.  angles [cap, rot_dims / 2, 2] = (cos, sin) fp32. */
typedef struct sk_latent_params {
    const void* dkv;
    void* q;
    const void* norm_w;
    const float* angles;
    void* cache;
    const int64_t* pos;
    int32_t* status;
    int64_t dkv_ld, q_ld, cap, cache_ld, start;
    int dtype, B, S, H, dim, rot, rot_dims, rank;
    float eps;
} sk_latent_params;
SK_API int skb_latent_append(const sk_latent_params* p, void* stream);
/* Queries for attention on the latent rows themselves: out[row, h] = [W_uk[h]^T q_unrotated (rank) |
 * q_rotated (rot) | 0 ...], out rows [H, out_ld]; uk [H * dim, rank]. */
SK_API int skb_latent_absorb(const void* q, int64_t q_ld, int dtype, const void* uk, int64_t rows, int H, int dim,
                             int rot, int rank, int out_ld, void* out, void* stream);
/* out[row, h * vdim + e] = <uv[h * vdim + e], o[row, h]>; o [rows, H, rank], uv [H * vdim, rank]. */
SK_API int skb_latent_up(const void* o, int dtype, const void* uv, int64_t rows, int H, int vdim, int rank, void* out,
                         void* stream);

/* State-space mixer.  Input projection rows (in_ld elements apart): xbc_in points at the [x (H P) | B
 * (G N) | C (G N)] columns, dt_in at the H step columns.  skb_ssm_conv: depthwise causal convolution
 * (conv_w [channels, taps], last tap = current token) + silu into xbc rows (xbc_ld apart), carried
 * inputs conv_state [B, taps - 1, channels].  skb_ssm_scan: the recurrence on those rows,
 * state [B, H, N, P] fp32, y [B, S, H P] (with the skip D x).  Position 0 starts from zero state.
 * `path`: SKB_SSM_STEPS walks token by token, SKB_SSM_CHUNKS uses matrix products per block of tokens. */
enum { SKB_SSM_AUTO = 0, SKB_SSM_STEPS = 1, SKB_SSM_CHUNKS = 2, SKB_SSM_TENSOR = 3 };
typedef struct sk_ssm_params {
    const void *xbc_in, *dt_in, *conv_w, *conv_b;
    void *conv_state, *xbc, *y;
    const float *dt_bias, *A_log, *D;
    float* state;
    const int64_t* pos;
    void* workspace;
    size_t workspace_bytes;
    int64_t in_ld, xbc_ld, start;
    int dtype, B, S, H, P, N, G, taps, path;
} sk_ssm_params;
SK_API int skb_ssm_conv(const sk_ssm_params* p, void* stream);
SK_API size_t skb_ssm_workspace_bytes(const sk_ssm_params* p);
SK_API int skb_ssm_scan(const sk_ssm_params* p, void* stream);
SK_API int skb_ssm_path(const sk_ssm_params* p);

/* Matrix-memory mixer.  Rows of B x S tokens, in_ld elements apart: q, k [H, N], v, z [H, P]; gates fp32
 * rows [input (H) | forget (H)], gates_ld apart, before their biases.  Per head, with
 *   i = cap tanh((input + i_bias) / cap),  f = logsigmoid(cap tanh((forget + f_bias) / cap)),
 *   m' = max(f + m, i),  (S, n)' = exp(f + m - m') (S, n) + exp(i - m') (k v^T, k),
 *   o = q_scale S'^T q / (max(|q_scale n' . q|, exp(-m')) + 1e-6),
 *   out = o / rms(o) * norm_w * sigmoid(z)              out rows [H P], out_ld apart
 * State: S [B, H, N, P], n [B, H, N], m [B, H], all fp32; position 0 starts from zero state and m = 0.
 * num [B S, H P] (of dtype), den [B S, H] and m_next [B, H] (fp32) are scratch.
 * `path`: SKB_SSM_STEPS walks token by token, SKB_SSM_CHUNKS uses warp-level matrix products per block of 64
 * tokens, SKB_SSM_TENSOR tensor-memory ones per chunk of 128, all chunks of a portion side by side. */
typedef struct sk_mlstm_params {
    const void *q, *k, *v, *z, *norm_w;
    const float *gates, *i_bias, *f_bias;
    float *S_state, *n_state, *m_state;
    void* num;
    float *den, *m_next;
    void* out;
    const int64_t* pos;
    int32_t* status;
    void* workspace;
    size_t workspace_bytes;
    int64_t in_ld, gates_ld, out_ld, start;
    int dtype, B, S, H, N, P, path;
    float cap, q_scale, eps;
} sk_mlstm_params;
SK_API size_t skb_mlstm_workspace_bytes(const sk_mlstm_params* p);
SK_API int skb_mlstm(const sk_mlstm_params* p, void* stream);
SK_API int skb_mlstm_path(const sk_mlstm_params* p);

/* t = y * silu(z); out = t / rms(t over each of `parts` equal slices) * w; y, out [rows, inner]. */
SK_API int skb_gated_group_norm(const void* y, const void* z, int64_t z_ld, const void* w, int dtype, int64_t rows,
                                int inner, int parts, float eps, void* out, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* SOCKET_B200_BLOCKS_H_ */
