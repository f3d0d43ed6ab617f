// Exact softmax attention for any head sizes, element types and visibility rule the parameter block can
// express: one CTA per (token, query head), 128 keys at a time, fp32 arithmetic throughout.  This is the
// fp32 path of the attention blocks and the fallback for shapes the tensor-core kernels do not cover.
#include "blocks.cuh"

namespace sk {
namespace {

constexpr int AR_THREADS = 128;
constexpr int AR_MAX_EV = 8;               // value sizes up to 1024

template <typename T, int EV>
__global__ void __launch_bounds__(AR_THREADS)
attn_rows_kernel(sk_attn_params p) {
    extern __shared__ float q_s[];         // [dqk]
    __shared__ float w_s[AR_THREADS], red[2][AR_THREADS / 32];
    const int s = blockIdx.x, h = blockIdx.y, b = blockIdx.z, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    const int g = h / (p.H / p.G);
    const int64_t i = first_position(p.pos, p.start) + s;
    const int64_t chunk_lo = p.chunk > 0 ? i / p.chunk * p.chunk : 0;
    const bool wrap = p.ring && p.chunk == 0;                    // row r: the latest position that is r modulo kv_rows
    const int64_t base = wrap ? 0 : (p.ring ? chunk_lo : p.kv_start);    // position of key row 0
    const int64_t lo = p.window > 0 && !wrap && i - p.window + 1 > chunk_lo ? i - p.window + 1 : chunk_lo;
    const int64_t row_lo = lo > base ? lo - base : 0;            // visible rows [row_lo, row_hi]
    const int64_t row_hi = wrap && i >= p.kv_rows ? p.kv_rows - 1 : i - base;
    T* out = (T*)p.out + b * p.o_bs + s * p.o_ss + h * p.o_hs;
    if (row_hi < 0 || row_hi >= p.kv_rows) {                     // outside the cache: flagged, the row reads zero
        if (t == 0 && p.status != nullptr) atomicOr(p.status, SK_DEV_POS_OUT_OF_RANGE);
        for (int e = t; e < p.dv; e += AR_THREADS) out[e] = from_f32<T>(0.f);
        return;
    }
    const T* q = (const T*)p.q + b * p.q_bs + s * p.q_ss + h * p.q_hs;
    const T* kb = (const T*)p.k + b * p.k_bs + g * p.k_hs;
    const T* vb = (const T*)p.v + b * p.v_bs + g * p.v_hs;
    for (int d = t; d < p.dqk; d += AR_THREADS) q_s[d] = to_f32(q[d]);
    __syncthreads();
    float m = -INFINITY, l = 0.f, acc[EV];
#pragma unroll
    for (int e = 0; e < EV; ++e) acc[e] = 0.f;
    for (int64_t r0 = row_lo; r0 <= row_hi; r0 += AR_THREADS) {
        const int64_t r = r0 + t;
        float sc = -INFINITY;
        if (r <= row_hi) {
            const T* k = kb + r * p.k_ts;
            float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
            int d = 0;
            for (; d + 4 <= p.dqk; d += 4) {
                d0 = fmaf(q_s[d], to_f32(k[d]), d0);
                d1 = fmaf(q_s[d + 1], to_f32(k[d + 1]), d1);
                d2 = fmaf(q_s[d + 2], to_f32(k[d + 2]), d2);
                d3 = fmaf(q_s[d + 3], to_f32(k[d + 3]), d3);
            }
            for (; d < p.dqk; ++d) d0 = fmaf(q_s[d], to_f32(k[d]), d0);
            sc = ((d0 + d1) + (d2 + d3)) * p.scale;
            if (p.softcap > 0.f) sc = soft_cap_f32(sc, p.softcap);
            if (p.bias != nullptr) {
                int64_t n = i - (base + r);
                if (wrap) n %= p.kv_rows;
                sc += p.bias[(int64_t)h * p.bias_len + (n < p.bias_len ? n : p.bias_len - 1)];
            }
        }
        float mt = sc;
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(FULL, mt, o));
        if (lane == 0) red[0][warp] = mt;
        __syncthreads();
        mt = fmaxf(fmaxf(red[0][0], red[0][1]), fmaxf(red[0][2], red[0][3]));
        const float mn = fmaxf(m, mt);                           // finite: every tile holds a visible key
        const float w = r <= row_hi ? expf(sc - mn) : 0.f;
        w_s[t] = w;
        const float ws = warp_sum(w);
        if (lane == 0) red[1][warp] = ws;
        __syncthreads();
        const float f = expf(m - mn);
        l = l * f + ((red[1][0] + red[1][1]) + (red[1][2] + red[1][3]));
        m = mn;
        const int n_here = (int)(row_hi - r0 + 1 < AR_THREADS ? row_hi - r0 + 1 : AR_THREADS);
#pragma unroll
        for (int e = 0; e < EV; ++e) {
            const int c = e * AR_THREADS + t;
            if (c < p.dv) {
                float a = acc[e] * f;
                const T* v = vb + r0 * p.v_ts + c;
                for (int j = 0; j < n_here; ++j) a = fmaf(w_s[j], to_f32(v[j * p.v_ts]), a);
                acc[e] = a;
            }
        }
        __syncthreads();
    }
    float f = 1.f;
    if (p.sink != nullptr) {
        const float sk = p.sink[h], mn = fmaxf(m, sk);
        f = expf(m - mn);
        l = l * f + expf(sk - mn);
    }
#pragma unroll
    for (int e = 0; e < EV; ++e) {
        const int c = e * AR_THREADS + t;
        if (c < p.dv) out[c] = from_f32<T>(acc[e] * f / l);
    }
}

template <typename T> int dispatch(const sk_attn_params& p, cudaStream_t st) {
    dim3 grid((unsigned)p.S, (unsigned)p.H, (unsigned)p.B);
    const size_t smem = (size_t)p.dqk * sizeof(float);
    const int ev = (p.dv + AR_THREADS - 1) / AR_THREADS;
    if (ev > AR_MAX_EV || smem > 40 * 1024)
        return fail(SK_ERR_UNSUPPORTED, "sk_attn: head sizes (%d, %d) are too large", p.dqk, p.dv);
    if (ev <= 1) attn_rows_kernel<T, 1><<<grid, AR_THREADS, smem, st>>>(p);
    else if (ev <= 4) attn_rows_kernel<T, 4><<<grid, AR_THREADS, smem, st>>>(p);
    else attn_rows_kernel<T, 8><<<grid, AR_THREADS, smem, st>>>(p);
    return check_launch("attn_rows_kernel");
}

}  // namespace

int launch_attn_rows(const sk_attn_params& p, cudaStream_t st) {
    return p.dtype == SK_BF16 ? dispatch<__nv_bfloat16>(p, st) : dispatch<float>(p, st);
}

}  // namespace sk
