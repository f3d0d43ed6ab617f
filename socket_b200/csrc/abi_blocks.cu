// extern "C" entry points of libsocket_b200_blocks.so: argument checks and kernel choice.
#include "abi_check.cuh"
#include "blocks.cuh"

using namespace sk;

namespace {

inline bool block_dtype(int d) { return d == SK_F32 || d == SK_BF16; }

int check_attn(const sk_attn_params* p) {
    SK_REQUIRE(p != nullptr, "skb_attn: null parameter block");
    SK_REQUIRE(p->q && p->k && p->v && p->out, "skb_attn: null pointer");
    SK_REQUIRE(block_dtype(p->dtype), "skb_attn: bad dtype");
    SK_REQUIRE(p->B > 0 && p->S > 0 && p->H > 0 && p->G > 0 && p->dqk > 0 && p->dv > 0, "skb_attn: sizes must be positive");
    SK_REQUIRE(p->H % p->G == 0, "skb_attn: %d query heads are not a multiple of %d key/value heads", p->H, p->G);
    SK_REQUIRE(p->kv_rows > 0 && p->start >= 0 && p->kv_start >= 0 && p->chunk >= 0 && p->window >= 0, "skb_attn: bad positions");
    SK_REQUIRE(p->softcap >= 0.f, "skb_attn: a score cap is positive (0: none)");
    SK_REQUIRE(p->bias == nullptr || p->bias_len > 0, "skb_attn: empty bias table");
    SK_REQUIRE(!p->ring || ((p->chunk > 0 || (p->window > 0 && p->kv_rows <= p->window)) && p->S == 1),
               "skb_attn: a ring serves one token under a chunk mask, or one of a window that is no smaller than the ring");
    SK_REQUIRE(p->pos != nullptr || p->ring || p->start + p->S - 1 - p->kv_start < p->kv_rows,
               "skb_attn: keys of positions up to %lld are needed, %lld rows from %lld exist",
               (long long)(p->start + p->S - 1), (long long)p->kv_rows, (long long)p->kv_start);
    return SK_OK;
}

int attn_path(const sk_attn_params& p) {
    if (p.path != SKB_ATTN_AUTO) return p.path;
    if (p.S <= (p.G == 1 ? 32 : 1) && attn_decode_mma_applicable(p)) return SKB_ATTN_DECODE;
    if (attn_prefill_tc_applicable(p)) return SKB_ATTN_PREFILL_TC;
    return SKB_ATTN_ROWS;
}

int check_ssm(const sk_ssm_params* p) {
    SK_REQUIRE(p != nullptr, "skb_ssm: null parameter block");
    SK_REQUIRE(p->xbc_in && p->dt_in && p->conv_w && p->conv_b && p->xbc && p->y && p->dt_bias && p->A_log && p->D && p->state,
               "skb_ssm: null pointer");
    SK_REQUIRE(p->taps >= 1 && (p->taps == 1 || p->conv_state), "skb_ssm: no buffer for the carried inputs");
    SK_REQUIRE(block_dtype(p->dtype), "skb_ssm: bad dtype");
    SK_REQUIRE(p->B > 0 && p->S > 0 && p->H > 0 && p->P > 0 && p->N > 0 && p->G > 0 && p->start >= 0,
               "skb_ssm: sizes must be positive");
    SK_REQUIRE(p->path >= SKB_SSM_AUTO && p->path <= SKB_SSM_CHUNKS, "skb_ssm: unknown path %d", p->path);
    SK_REQUIRE(p->H % p->G == 0, "skb_ssm: %d heads are not a multiple of %d groups", p->H, p->G);
    SK_REQUIRE(p->xbc_ld >= p->H * p->P + 2 * p->G * p->N, "skb_ssm: row stride smaller than row");
    return SK_OK;
}

int ssm_path(const sk_ssm_params& p) {
    if (p.path != SKB_SSM_AUTO) return p.path;
    return p.S >= 16 && ssm_chunks_applicable(p) ? SKB_SSM_CHUNKS : SKB_SSM_STEPS;
}

int check_mlstm(const sk_mlstm_params* p) {
    SK_REQUIRE(p != nullptr, "skb_mlstm: null parameter block");
    SK_REQUIRE(p->q && p->k && p->v && p->z && p->norm_w && p->gates && p->i_bias && p->f_bias && p->S_state && p->n_state &&
                   p->m_state && p->num && p->den && p->m_next && p->out, "skb_mlstm: null pointer");
    SK_REQUIRE(block_dtype(p->dtype), "skb_mlstm: bad dtype");
    SK_REQUIRE(p->B > 0 && p->S > 0 && p->H > 0 && p->N > 0 && p->P > 0 && p->start >= 0 && p->cap > 0.f,
               "skb_mlstm: sizes and the gates' cap must be positive");
    SK_REQUIRE(p->gates_ld >= 2 * p->H && p->out_ld >= (int64_t)p->H * p->P && p->in_ld >= (int64_t)p->H * (p->N > p->P ? p->N : p->P),
               "skb_mlstm: row stride smaller than row");
    return SK_OK;
}

int mlstm_path(const sk_mlstm_params& p) {
    if (p.path != SKB_SSM_AUTO) return p.path;
    if (p.S >= 256 && mlstm_tc_applicable(p)) return SKB_SSM_TENSOR;
    return p.S >= 16 && mlstm_chunks_applicable(p) ? SKB_SSM_CHUNKS : SKB_SSM_STEPS;
}

size_t mlstm_workspace(const sk_mlstm_params& p) {
    const int path = mlstm_path(p);
    return path == SKB_SSM_TENSOR ? mlstm_tc_workspace(p) : path == SKB_SSM_CHUNKS ? mlstm_chunks_workspace(p) : 0;
}

}  // namespace

extern "C" {

int skb_abi_version(void) { return SK_ABI_VERSION; }
const char* skb_status_string(int status) { return status_string(status); }
const char* skb_last_error(void) { return last_error(); }

int skb_embed_rows(const int64_t* tokens, const void* table, int dtype, int64_t rows, int64_t vocab, int width, float scale,
                   float* x, float* x_copy, int32_t* status, void* stream) {
    SK_REQUIRE(tokens && table && x, "skb_embed_rows: null pointer");
    SK_REQUIRE(block_dtype(dtype) && rows > 0 && vocab > 0 && width > 0, "skb_embed_rows: bad sizes or dtype");
    return launch_embed_rows(tokens, table, dtype, rows, vocab, width, scale, x, x_copy, status, (cudaStream_t)stream);
}

int skb_residual_norm(const sk_residual_params* p, void* stream) {
    SK_REQUIRE(p && p->x && p->rows > 0 && p->width > 0, "skb_residual_norm: null pointer or empty stream");
    SK_REQUIRE(block_dtype(p->dtype) && (p->y_dtype == p->dtype || p->y_dtype == SK_F32), "skb_residual_norm: bad dtype");
    SK_REQUIRE(p->in_mode >= 0 && p->in_mode <= 3 && p->out_mode >= 0 && p->out_mode <= 3, "skb_residual_norm: bad mode");
    SK_REQUIRE(p->in_mode == SKB_IN_NONE || (p->y && (p->w_in || p->in_mode == SKB_IN_ADD) && p->y_ld >= p->width),
               "skb_residual_norm: input missing");
    SK_REQUIRE(p->out_mode == SKB_OUT_NONE || p->out, "skb_residual_norm: output missing");
    SK_REQUIRE((p->out_mode != SKB_OUT_NORM && p->out_mode != SKB_OUT_LAYER_NORM) || p->w_out,
               "skb_residual_norm: norm weight missing");
    SK_REQUIRE(p->out_mode != SKB_OUT_CONCAT || p->x0, "skb_residual_norm: second stream missing");
    return launch_residual_norm(*p, (cudaStream_t)stream);
}

int skb_glu(const void* gate, const void* up, int dtype, int64_t rows, int ff, int64_t ld, int kind, float limit, float slope,
            void* out, int64_t out_ld, void* stream) {
    SK_REQUIRE(gate && up && out && block_dtype(dtype) && rows > 0 && ff > 0 && ld >= ff && out_ld >= ff,
               "skb_glu: null pointer, bad sizes or dtype");
    SK_REQUIRE(kind == SKB_GLU_CLAMPED || kind == SKB_GLU_SILU, "skb_glu: unknown unit %d", kind);
    return launch_glu(gate, up, dtype, rows, ff, ld, kind, limit, slope, out, out_ld, (cudaStream_t)stream);
}

int skb_ring_append(const void* k, const void* v, int dtype, int B, int S, int64_t k_bs, int64_t k_ss, int64_t v_bs,
                    int64_t v_ss, int k_row, int v_row, int ring, int keep, const int64_t* pos, int64_t start, void* k_cache,
                    void* v_cache, void* stream) {
    SK_REQUIRE(k && k_cache && (v == nullptr) == (v_cache == nullptr) && block_dtype(dtype), "skb_ring_append: null pointer or bad dtype");
    SK_REQUIRE(B > 0 && S > 0 && k_row > 0 && (v == nullptr || v_row > 0) && ring > 0 && start >= 0,
               "skb_ring_append: sizes must be positive");
    SK_REQUIRE(keep == SKB_RING_CHUNK || keep == SKB_RING_WINDOW, "skb_ring_append: unknown rule %d", keep);
    SK_REQUIRE(pos == nullptr || S == 1, "skb_ring_append: a device position serves one token");
    return launch_ring_append(k, v, dtype, B, S, k_bs, k_ss, v_bs, v_ss, k_row, v_row, ring, keep, pos, start, k_cache, v_cache,
                              (cudaStream_t)stream);
}

int skb_rotary_rows(const sk_rotary_rows_params* p, void* stream) {
    SK_REQUIRE(p && p->q_in && p->k_in && p->q_out && p->rows_out && p->angles, "skb_rotary_rows: null pointer");
    SK_REQUIRE(block_dtype(p->dtype) && p->B > 0 && p->S > 0 && p->H > 0 && p->G > 0 && p->dim > 0 && p->start >= 0,
               "skb_rotary_rows: sizes must be positive");
    SK_REQUIRE(p->rot_dims >= 0 && p->rot_dims % 2 == 0 && p->rot_dims <= p->dim, "skb_rotary_rows: %d rotated of %d dimensions",
               p->rot_dims, p->dim);
    SK_REQUIRE(p->prev >= 0 && (p->prev == 0 || (p->ring && p->prev <= p->ring_rows && p->prev <= p->start && p->pos == nullptr)),
               "skb_rotary_rows: %d earlier rows cannot be had", p->prev);
    SK_REQUIRE(p->pos ? p->S == 1 && p->rows_cap > 0 : p->rows_cap >= p->prev + p->S, "skb_rotary_rows: rows do not fit");
    return launch_rotary_rows(*p, (cudaStream_t)stream);
}

size_t skb_attn_workspace_bytes(const sk_attn_params* p) {
    return p != nullptr && attn_path(*p) == SKB_ATTN_DECODE ? attn_decode_mma_workspace(*p) : 0;
}

int skb_attn_path(const sk_attn_params* p) { return p != nullptr ? attn_path(*p) : SKB_ATTN_ROWS; }

int skb_attn(const sk_attn_params* p, void* stream) {
    if (int rc = check_attn(p)) return rc;
    const cudaStream_t st = (cudaStream_t)stream;
    switch (attn_path(*p)) {
        case SKB_ATTN_DECODE:
            if (!attn_decode_mma_applicable(*p)) return fail(SK_ERR_UNSUPPORTED, "skb_attn: shape outside the decode kernel");
            if (p->workspace == nullptr || p->workspace_bytes < attn_decode_mma_workspace(*p))
                return fail(SK_ERR_WORKSPACE, "skb_attn: workspace of %zu bytes needed, %zu given",
                            attn_decode_mma_workspace(*p), p->workspace_bytes);
            return launch_attn_decode_mma(*p, st);
        case SKB_ATTN_PREFILL_TC:
            if (!attn_prefill_tc_applicable(*p)) return fail(SK_ERR_UNSUPPORTED, "skb_attn: shape outside the prefill kernel");
            return launch_attn_prefill_tc(*p, st);
        default:
            return launch_attn_rows(*p, st);
    }
}

int skb_latent_append(const sk_latent_params* p, void* stream) {
    SK_REQUIRE(p && p->dkv && p->q && p->norm_w && p->angles && p->cache, "skb_latent_append: null pointer");
    SK_REQUIRE(block_dtype(p->dtype) && p->B > 0 && p->S > 0 && p->H > 0 && p->dim >= 0 && p->rot > 0 && p->rank > 0,
               "skb_latent_append: sizes must be positive");
    SK_REQUIRE(p->rot_dims >= 0 && p->rot_dims % 2 == 0 && p->rot_dims <= p->rot, "skb_latent_append: %d rotated of %d dimensions",
               p->rot_dims, p->rot);
    SK_REQUIRE(p->cache_ld >= p->rank + p->rot && p->cap > 0, "skb_latent_append: row stride smaller than row");
    return launch_latent_append(*p, (cudaStream_t)stream);
}

int skb_latent_absorb(const void* q, int64_t q_ld, int dtype, const void* uk, int64_t rows, int H, int dim, int rot, int rank,
                      int out_ld, void* out, void* stream) {
    SK_REQUIRE(q && uk && out && block_dtype(dtype), "skb_latent_absorb: null pointer or bad dtype");
    SK_REQUIRE(rows > 0 && H > 0 && dim > 0 && rot > 0 && rank > 0 && out_ld >= rank + rot, "skb_latent_absorb: bad sizes");
    return launch_latent_absorb(q, q_ld, dtype, uk, rows, H, dim, rot, rank, out_ld, out, (cudaStream_t)stream);
}

int skb_latent_up(const void* o, int dtype, const void* uv, int64_t rows, int H, int vdim, int rank, void* out, void* stream) {
    SK_REQUIRE(o && uv && out && block_dtype(dtype), "skb_latent_up: null pointer or bad dtype");
    SK_REQUIRE(rows > 0 && H > 0 && vdim > 0 && rank > 0, "skb_latent_up: sizes must be positive");
    return launch_latent_up(o, dtype, uv, rows, H, vdim, rank, out, (cudaStream_t)stream);
}

int skb_ssm_conv(const sk_ssm_params* p, void* stream) {
    if (int rc = check_ssm(p)) return rc;
    return launch_ssm_conv(*p, (cudaStream_t)stream);
}

size_t skb_ssm_workspace_bytes(const sk_ssm_params* p) {
    return p != nullptr && ssm_path(*p) == SKB_SSM_CHUNKS ? ssm_chunks_workspace(*p) : 0;
}

int skb_ssm_path(const sk_ssm_params* p) { return p != nullptr ? ssm_path(*p) : SKB_SSM_STEPS; }

int skb_ssm_scan(const sk_ssm_params* p, void* stream) {
    if (int rc = check_ssm(p)) return rc;
    if (ssm_path(*p) == SKB_SSM_CHUNKS) {
        if (!ssm_chunks_applicable(*p)) return fail(SK_ERR_UNSUPPORTED, "skb_ssm_scan: shape outside the block kernel");
        if (ssm_chunks_workspace(*p) > 0 && (p->workspace == nullptr || p->workspace_bytes < ssm_chunks_workspace(*p)))
            return fail(SK_ERR_WORKSPACE, "skb_ssm_scan: workspace of %zu bytes needed, %zu given", ssm_chunks_workspace(*p),
                        p->workspace_bytes);
        return launch_ssm_chunks(*p, (cudaStream_t)stream);
    }
    return launch_ssm_steps(*p, (cudaStream_t)stream);
}

size_t skb_mlstm_workspace_bytes(const sk_mlstm_params* p) {
    return p != nullptr ? mlstm_workspace(*p) : 0;
}

int skb_mlstm_path(const sk_mlstm_params* p) { return p != nullptr ? mlstm_path(*p) : SKB_SSM_STEPS; }

int skb_mlstm(const sk_mlstm_params* p, void* stream) {
    if (int rc = check_mlstm(p)) return rc;
    const cudaStream_t st = (cudaStream_t)stream;
    const int path = mlstm_path(*p);
    if (path == SKB_SSM_CHUNKS ? !mlstm_chunks_applicable(*p) : path == SKB_SSM_TENSOR && !mlstm_tc_applicable(*p))
        return fail(SK_ERR_UNSUPPORTED, "skb_mlstm: shape outside the block kernels");
    if (mlstm_workspace(*p) > 0 && (p->workspace == nullptr || p->workspace_bytes < mlstm_workspace(*p)))
        return fail(SK_ERR_WORKSPACE, "skb_mlstm: workspace of %zu bytes needed, %zu given", mlstm_workspace(*p), p->workspace_bytes);
    const int rc = path == SKB_SSM_TENSOR ? launch_mlstm_tc(*p, st) : path == SKB_SSM_CHUNKS ? launch_mlstm_chunks(*p, st)
                                                                                            : launch_mlstm_steps(*p, st);
    return rc != SK_OK ? rc : launch_mlstm_finish(*p, st);
}

int skb_gated_group_norm(const void* y, const void* z, int64_t z_ld, const void* w, int dtype, int64_t rows, int inner,
                         int parts, float eps, void* out, void* stream) {
    SK_REQUIRE(y && z && w && out && block_dtype(dtype), "skb_gated_group_norm: null pointer or bad dtype");
    SK_REQUIRE(rows > 0 && inner > 0 && parts > 0 && inner % parts == 0 && z_ld >= inner,
               "skb_gated_group_norm: %d elements do not split into %d parts", inner, parts);
    return launch_gated_group_norm(y, z, z_ld, w, dtype, rows, inner, parts, eps, out, (cudaStream_t)stream);
}

}  // extern "C"
