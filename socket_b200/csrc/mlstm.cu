// Matrix-memory mixer, token by token: exponential input gate, sigmoid forget gate, both stabilised by a
// running maximum m, in fp32:
//   m_t = max(f + m_{t-1}, i),  (S, n)_t = exp(f + m_{t-1} - m_t) (S, n)_{t-1} + exp(i - m_t) (k v^T, k)
//   o = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)
// and the norm per head with the sigmoid gate behind it.  The normaliser n is kept as one more value
// column whose value is always 1, so it costs what a column costs and nothing of it is computed twice.
// A portion that starts at position 0 starts from zero state whatever the buffers hold.
//
// The recurrence kernels leave the numerators (num), the denominators (den) and the last m (m_next); the
// finishing kernel divides, norms, gates, and moves m_next into the state, after every reader of the old m.
#include "blocks.cuh"

namespace sk {
namespace {

constexpr int MS_COLS = 16, MS_GROUPS = 16;

// A CTA owns 16 of the P + 1 columns of one head; thread (column, group) keeps N / 16 state elements in registers.
template <typename T, int NPT>
__global__ void __launch_bounds__(MS_COLS * MS_GROUPS)
mlstm_steps_kernel(sk_mlstm_params p) {
    __shared__ float red[2][8][MS_COLS];
    const int t = threadIdx.x, c = t & (MS_COLS - 1), grp = t >> 4, warp = t >> 5, lane = t & 31;
    const int col = blockIdx.x * MS_COLS + c, h = blockIdx.y, b = blockIdx.z;
    const bool live = col <= p.P, norm = col == p.P;          // the column behind the last value is the normaliser
    const bool fresh = first_position(p.pos, p.start) == 0;
    const int64_t head = (int64_t)b * p.H + h;
    const float ib = p.i_bias[h], fb = p.f_bias[h];
    float* st = norm ? p.n_state + head * p.N : p.S_state + head * p.N * p.P + col;
    const int64_t ld = norm ? 1 : p.P;
    float s[NPT], m = fresh ? 0.f : p.m_state[head];
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
        const int n = grp + k * MS_GROUPS;
        s[k] = (!fresh && live && n < p.N) ? st[n * ld] : 0.f;
    }
    for (int tok = 0; tok < p.S; ++tok) {
        const int64_t row = (int64_t)b * p.S + tok;
        const float gi = soft_cap_f32(p.gates[row * p.gates_ld + h] + ib, p.cap);
        const float gf = log_sigmoid_f32(soft_cap_f32(p.gates[row * p.gates_ld + p.H + h] + fb, p.cap));
        const float mn = fmaxf(gf + m, gi), keep = expf(gf + m - mn), add = expf(gi - mn);
        m = mn;
        const float v = !live ? 0.f : (norm ? 1.f : to_f32(((const T*)p.v)[row * p.in_ld + (int64_t)h * p.P + col]));
        const float va = v * add;
        const T* q = (const T*)p.q + row * p.in_ld + (int64_t)h * p.N;
        const T* kk = (const T*)p.k + row * p.in_ld + (int64_t)h * p.N;
        float y = 0.f;
#pragma unroll
        for (int k = 0; k < NPT; ++k) {
            const int n = grp + k * MS_GROUPS;
            if (n < p.N) {
                s[k] = fmaf(s[k], keep, to_f32(kk[n]) * va);
                y = fmaf(s[k], to_f32(q[n]), y);
            }
        }
        y += __shfl_xor_sync(FULL, y, 16);
        float (*rd)[MS_COLS] = red[tok & 1];
        if (lane < 16) rd[warp][c] = y;
        __syncthreads();
        if (t < MS_COLS && live) {
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += rd[w][c];
            o *= p.q_scale;
            if (norm) p.den[row * p.H + h] = fmaxf(fabsf(o), expf(-m)) + 1e-6f;
            else ((T*)p.num)[row * p.H * p.P + (int64_t)h * p.P + col] = from_f32<T>(o);
        }
    }
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
        const int n = grp + k * MS_GROUPS;
        if (live && n < p.N) st[n * ld] = s[k];
    }
    if (norm && grp == 0) p.m_next[head] = m;
}

// One CTA per (token, head): o = num / den, its RMS norm, the gate; the last token's CTA commits m.
template <typename T, int V, int NV>
__global__ void __launch_bounds__(1024)
mlstm_finish_kernel(sk_mlstm_params p) {
    __shared__ float red[32];
    const int64_t row = blockIdx.x;
    const int h = blockIdx.y, nt = blockDim.x, t = threadIdx.x;
    const float inv_den = 1.f / p.den[row * p.H + h];
    const T* num = (const T*)p.num + (row * p.H + h) * p.P;
    float v[NV][V], ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * nt + t) * V;
        if (i < p.P) {
            load_vec<T, V>(num + i, v[n]);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                v[n][e] *= inv_den;
                ss = fmaf(v[n][e], v[n][e], ss);
            }
        }
    }
    if (t == 0 && row % p.S == p.S - 1) {
        const int64_t head = row / p.S * p.H + h;
        p.m_state[head] = p.m_next[head];
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.P + p.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * nt + t) * V;
        if (i < p.P) {
            float w[V], z[V];
            load_vec<T, V>((const T*)p.norm_w + h * p.P + i, w);
            load_vec<T, V>((const T*)p.z + row * p.in_ld + (int64_t)h * p.P + i, z);
#pragma unroll
            for (int e = 0; e < V; ++e) v[n][e] *= inv * w[e] * sigmoid_scaled<T>(z[e], 1.f);
            store_vec<T, V>((T*)p.out + row * p.out_ld + (int64_t)h * p.P + i, v[n]);
        }
    }
}

template <typename T, int V> int finish_dispatch(const sk_mlstm_params& p, cudaStream_t st) {
    const int vecs = (p.P + V - 1) / V;
    int nt = 256;
    while (nt > 32 && nt / 2 >= vecs) nt /= 2;
    while (nt < 1024 && (vecs + nt - 1) / nt > 8) nt *= 2;
    const int nv = (vecs + nt - 1) / nt;
    dim3 grid((unsigned)((int64_t)p.B * p.S), (unsigned)p.H);
    if (nv <= 1) mlstm_finish_kernel<T, V, 1><<<grid, nt, 0, st>>>(p);
    else if (nv <= 2) mlstm_finish_kernel<T, V, 2><<<grid, nt, 0, st>>>(p);
    else if (nv <= 8) mlstm_finish_kernel<T, V, 8><<<grid, nt, 0, st>>>(p);
    else return fail(SK_ERR_UNSUPPORTED, "skb_mlstm: value size %d is too large", p.P);
    return check_launch("mlstm_finish_kernel");
}

template <typename T> int steps_dispatch(const sk_mlstm_params& p, cudaStream_t st) {
    dim3 grid((unsigned)((p.P + MS_COLS) / MS_COLS), (unsigned)p.H, (unsigned)p.B);      // P + 1 columns
    const int npt = (p.N + MS_GROUPS - 1) / MS_GROUPS;
    if (npt <= 2) mlstm_steps_kernel<T, 2><<<grid, 256, 0, st>>>(p);
    else if (npt <= 4) mlstm_steps_kernel<T, 4><<<grid, 256, 0, st>>>(p);
    else if (npt <= 8) mlstm_steps_kernel<T, 8><<<grid, 256, 0, st>>>(p);
    else if (npt <= 16) mlstm_steps_kernel<T, 16><<<grid, 256, 0, st>>>(p);
    else if (npt <= 32) mlstm_steps_kernel<T, 32><<<grid, 256, 0, st>>>(p);
    else if (npt <= 64) mlstm_steps_kernel<T, 64><<<grid, 256, 0, st>>>(p);
    else return fail(SK_ERR_UNSUPPORTED, "skb_mlstm: key size %d is too large", p.N);
    return check_launch("mlstm_steps_kernel");
}

}  // namespace

int launch_mlstm_steps(const sk_mlstm_params& p, cudaStream_t st) {
    return p.dtype == SK_BF16 ? steps_dispatch<__nv_bfloat16>(p, st) : steps_dispatch<float>(p, st);
}

int launch_mlstm_finish(const sk_mlstm_params& p, cudaStream_t st) {
    const size_t es = p.dtype == SK_BF16 ? 2 : 4;
    auto vec = [&](int v) {
        return p.P % v == 0 && p.in_ld % v == 0 && p.out_ld % v == 0 &&
               ((uintptr_t)p.z | (uintptr_t)p.out | (uintptr_t)p.num | (uintptr_t)p.norm_w) % (v * es) == 0;
    };
    if (p.dtype == SK_BF16)
        return vec(8) ? finish_dispatch<__nv_bfloat16, 8>(p, st) : vec(4) ? finish_dispatch<__nv_bfloat16, 4>(p, st)
                                                                          : finish_dispatch<__nv_bfloat16, 1>(p, st);
    return vec(4) ? finish_dispatch<float, 4>(p, st) : finish_dispatch<float, 1>(p, st);
}

}  // namespace sk
