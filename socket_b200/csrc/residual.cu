// Everything between two matrix products that touches the fp32 residual stream: the scaled embedding,
// the residual update with a norm on the sublayer's output fused with the norm of the next sublayer's
// input, and the gated units of the feed-forwards.
#include "blocks.cuh"

namespace sk {
namespace {

template <typename T, int V>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const int64_t* __restrict__ tokens, const T* __restrict__ table, int64_t vocab, int width, float scale,
                  float* __restrict__ x, float* __restrict__ x_copy, int32_t* status) {
    const int64_t row = blockIdx.x;
    const int i = (blockIdx.y * 256 + threadIdx.x) * V;
    const int64_t tok = tokens[row];
    const bool ok = tok >= 0 && tok < vocab;              // outside the table: flagged, the row reads zero
    if (!ok && i == 0 && status != nullptr) atomicOr(status, SK_DEV_INDEX_OUT_OF_RANGE);
    if (i >= width) return;
    float v[V];
    if (ok) load_vec<T, V>(table + tok * width + i, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = ok ? v[e] * scale : 0.f;
    store_vec<float, V>(x + row * width + i, v);
    if (x_copy != nullptr) store_vec<float, V>(x_copy + row * width + i, v);
}

// One CTA per row; the row lives in registers (NV vectors of V elements per thread).
//   in_mode  0: x stays; 1: x += rms(y) * w_in; 2: x = y + w_in; 3: x += y
//   out_mode 0: nothing; 1: out = rms(x) * w_out; 2: out = [x ; x0]; 3: out = layer norm of x * w_out
template <typename T, typename TY, int V, int NV>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(sk_residual_params p) {
    __shared__ float red[3][32];
    const int64_t row = blockIdx.x;
    const int W = p.width, nt = blockDim.x, t = threadIdx.x;
    float* xr = p.x + row * W;
    const T* w_in = (const T*)p.w_in;
    const T* w_out = (const T*)p.w_out;
    float xv[NV][V];
    if (p.in_mode != 0) {
        const TY* yr = (const TY*)p.y + row * p.y_ld;
        float yv[NV][V], ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * nt + t) * V;
            if (i < W) {
                load_vec<TY, V>(yr + i, yv[n]);
                if (p.in_mode != 2) load_vec<float, V>(xr + i, xv[n]);
#pragma unroll
                for (int e = 0; e < V; ++e) ss = fmaf(yv[n][e], yv[n][e], ss);
            }
        }
        float inv = 1.f;
        if (p.in_mode == 1) inv = 1.f / sqrtf(block_sum(ss, red[0]) / (float)W + p.eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * nt + t) * V;
            if (i < W) {
                float w[V];
                if (p.in_mode != 3) load_vec<T, V>(w_in + i, w);
#pragma unroll
                for (int e = 0; e < V; ++e)
                    xv[n][e] = p.in_mode == 1 ? xv[n][e] + yv[n][e] * inv * w[e]
                                              : (p.in_mode == 2 ? yv[n][e] + w[e] : xv[n][e] + yv[n][e]);
                store_vec<float, V>(xr + i, xv[n]);
            }
        }
    } else {
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * nt + t) * V;
            if (i < W) load_vec<float, V>(xr + i, xv[n]);
        }
    }
    if (p.out_mode == 1 || p.out_mode == 3) {
        float mean = 0.f;
        if (p.out_mode == 3) {                            // centred in registers; the stream itself is written already
            float sum = 0.f;
#pragma unroll
            for (int n = 0; n < NV; ++n)
                if ((n * nt + t) * V < W)
#pragma unroll
                    for (int e = 0; e < V; ++e) sum += xv[n][e];
            mean = block_sum(sum, red[2]) / (float)W;
        }
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n)
            if ((n * nt + t) * V < W)
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    xv[n][e] -= mean;
                    ss = fmaf(xv[n][e], xv[n][e], ss);
                }
        const float inv = 1.f / sqrtf(block_sum(ss, red[1]) / (float)W + p.eps);
        T* o = (T*)p.out + row * W;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * nt + t) * V;
            if (i < W) {
                float w[V], r[V];
                load_vec<T, V>(w_out + i, w);
#pragma unroll
                for (int e = 0; e < V; ++e) r[e] = xv[n][e] * inv * w[e];
                store_vec<T, V>(o + i, r);
            }
        }
    } else if (p.out_mode == 2) {
        T* o = (T*)p.out + row * 2 * W;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = (n * nt + t) * V;
            if (i < W) {
                float r[V];
                load_vec<float, V>(p.x0 + row * W + i, r);
                store_vec<T, V>(o + i, xv[n]);
                store_vec<T, V>(o + W + i, r);
            }
        }
    }
}

// KIND SKB_GLU_CLAMPED: y = g * sigmoid(slope * g) * (u + 1), g and u clamped; SKB_GLU_SILU: y = g * sigmoid(g) * u
template <typename T, int V, int KIND>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ gate, const T* __restrict__ up, int64_t rows, int ff, int64_t ld, float limit, float slope,
           T* __restrict__ out, int64_t out_ld) {
    const int i = (blockIdx.x * 256 + threadIdx.x) * V;
    if (i >= ff) return;
    for (int64_t row = blockIdx.y; row < rows; row += gridDim.y) {
        float g[V], u[V], r[V];
        load_vec<T, V>(gate + row * ld + i, g);
        load_vec<T, V>(up + row * ld + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            if (KIND == SKB_GLU_CLAMPED) {
                const float a = fminf(g[e], limit), b = fminf(fmaxf(u[e], -limit), limit);
                r[e] = a * sigmoid_scaled<T>(a, slope) * (b + 1.f);
            } else {
                r[e] = silu<T>(g[e]) * u[e];
            }
        }
        store_vec<T, V>(out + row * out_ld + i, r);
    }
}

// The newest tokens of a portion, from token s0 on, into a ring of `ring` rows (row of position p: p % ring).
// s0 leaves out what no later token sees, so that no two tokens of a portion meet in one row.
template <typename T>
__global__ void __launch_bounds__(256)
ring_append_kernel(const T* __restrict__ k, const T* __restrict__ v, int64_t k_bs, int64_t k_ss, int64_t v_bs,
                   int64_t v_ss, int k_row, int v_row, int ring, const int64_t* __restrict__ pos, int64_t start, int s0,
                   T* __restrict__ k_cache, T* __restrict__ v_cache) {
    const int s = s0 + blockIdx.x, b = blockIdx.y;
    const int64_t slot = (first_position(pos, start) + s) % ring;
    const T* ks = k + b * k_bs + s * k_ss;
    T* kd = k_cache + ((int64_t)b * ring + slot) * k_row;
    for (int i = threadIdx.x; i < k_row; i += blockDim.x) kd[i] = ks[i];
    if (v != nullptr) {
        const T* vs = v + b * v_bs + s * v_ss;
        T* vd = v_cache + ((int64_t)b * ring + slot) * v_row;
        for (int i = threadIdx.x; i < v_row; i += blockDim.x) vd[i] = vs[i];
    }
}

template <typename T, typename TY, int V>
int residual_dispatch(const sk_residual_params& p, cudaStream_t st) {
    const int vecs = (p.width + V - 1) / V;
    // few rows: one vector per thread (latency); many rows: smaller blocks, more of them per SM
    int nt = p.rows < 296 ? 1024 : 256;
    while (nt > 32 && nt / 2 >= vecs) nt /= 2;
    while (nt < 1024 && (vecs + nt - 1) / nt > 8) nt *= 2;
    const int nv = (vecs + nt - 1) / nt;
    dim3 grid((unsigned)p.rows);
    if (nv <= 1) residual_norm_kernel<T, TY, V, 1><<<grid, nt, 0, st>>>(p);
    else if (nv <= 2) residual_norm_kernel<T, TY, V, 2><<<grid, nt, 0, st>>>(p);
    else if (nv <= 4) residual_norm_kernel<T, TY, V, 4><<<grid, nt, 0, st>>>(p);
    else if (nv <= 8) residual_norm_kernel<T, TY, V, 8><<<grid, nt, 0, st>>>(p);
    else return fail(SK_ERR_UNSUPPORTED, "sk_residual_norm: width %d is too large", p.width);
    return check_launch("residual_norm_kernel");
}

}  // namespace

int launch_embed_rows(const int64_t* tokens, const void* table, int dtype, int64_t rows, int64_t vocab, int width,
                      float scale, float* x, float* x_copy, int32_t* status, cudaStream_t st) {
    const int V = width % 4 == 0 ? 4 : 1;
    dim3 grid((unsigned)rows, (unsigned)((width + 256 * V - 1) / (256 * V)));
#define SK_EMBED(T, V) embed_rows_kernel<T, V><<<grid, 256, 0, st>>>(tokens, (const T*)table, vocab, width, scale, x, x_copy, status)
    if (dtype == SK_BF16) { if (V == 4) SK_EMBED(__nv_bfloat16, 4); else SK_EMBED(__nv_bfloat16, 1); }
    else { if (V == 4) SK_EMBED(float, 4); else SK_EMBED(float, 1); }
#undef SK_EMBED
    return check_launch("embed_rows_kernel");
}

int launch_residual_norm(const sk_residual_params& p, cudaStream_t st) {
    const bool v4 = p.width % 4 == 0 && p.y_ld % 4 == 0;
    if (p.dtype == SK_F32) return v4 ? residual_dispatch<float, float, 4>(p, st) : residual_dispatch<float, float, 1>(p, st);
    using bf = __nv_bfloat16;
    if (p.y_dtype == SK_F32) return v4 ? residual_dispatch<bf, float, 4>(p, st) : residual_dispatch<bf, float, 1>(p, st);
    return v4 ? residual_dispatch<bf, bf, 4>(p, st) : residual_dispatch<bf, bf, 1>(p, st);
}

int launch_glu(const void* gate, const void* up, int dtype, int64_t rows, int ff, int64_t ld, int kind, float limit, float slope,
               void* out, int64_t out_ld, cudaStream_t st) {
    const size_t es = dtype == SK_BF16 ? 2 : 4;
    auto vec = [&](int v) {
        return ff % v == 0 && ld % v == 0 && out_ld % v == 0 &&
               ((uintptr_t)gate | (uintptr_t)up | (uintptr_t)out) % (v * es) == 0;
    };
    const bool v4 = vec(4), v8 = dtype == SK_BF16 && vec(8);
    const int V = v8 ? 8 : (v4 ? 4 : 1);
    dim3 grid((unsigned)((ff + 256 * V - 1) / (256 * V)), (unsigned)(rows < 32768 ? rows : 32768));
#define SK_GLU(T, V)                                                                                                       \
    do {                                                                                                                   \
        auto kern = kind == SKB_GLU_CLAMPED ? glu_kernel<T, V, SKB_GLU_CLAMPED> : glu_kernel<T, V, SKB_GLU_SILU>;          \
        kern<<<grid, 256, 0, st>>>((const T*)gate, (const T*)up, rows, ff, ld, limit, slope, (T*)out, out_ld);             \
    } while (0)
    if (dtype == SK_BF16) { if (v8) SK_GLU(__nv_bfloat16, 8); else if (v4) SK_GLU(__nv_bfloat16, 4); else SK_GLU(__nv_bfloat16, 1); }
    else { if (v4) SK_GLU(float, 4); else SK_GLU(float, 1); }
#undef SK_GLU
    return check_launch("glu_kernel");
}

int launch_ring_append(const void* k, const void* v, int dtype, int B, int S, int64_t k_bs, int64_t k_ss, int64_t v_bs,
                       int64_t v_ss, int k_row, int v_row, int ring, int keep, const int64_t* pos, int64_t start, void* k_cache,
                       void* v_cache, cudaStream_t st) {
    // first position to write: of the last block of `ring` positions, or of the last `ring` positions
    const int64_t first = keep == SKB_RING_CHUNK ? (start + S - 1) / ring * ring : start + S - ring;
    const int s0 = pos == nullptr && first > start ? (int)(first - start) : 0;   // a device position: one token
    dim3 grid((unsigned)(S - s0), (unsigned)B);
    if (dtype == SK_BF16)
        ring_append_kernel<<<grid, 256, 0, st>>>((const __nv_bfloat16*)k, (const __nv_bfloat16*)v, k_bs, k_ss, v_bs, v_ss,
                                                 k_row, v_row, ring, pos, start, s0, (__nv_bfloat16*)k_cache,
                                                 (__nv_bfloat16*)v_cache);
    else
        ring_append_kernel<<<grid, 256, 0, st>>>((const float*)k, (const float*)v, k_bs, k_ss, v_bs, v_ss, k_row, v_row,
                                                 ring, pos, start, s0, (float*)k_cache, (float*)v_cache);
    return check_launch("ring_append_kernel");
}

}  // namespace sk
