// Selective state-space mixer, token by token: the short causal convolution with its carried inputs,
// the recurrence S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T, y_t = S_t^T C_t + D x_t in fp32, and
// the gated group norm of its output.  A portion that starts at position 0 starts from zero state
// whatever the state buffers hold, so a slot needs no clearing between sequences.
#include "blocks.cuh"

namespace sk {
namespace {

// ---------------------------------------------------------------- convolution
// in  = the [x | B | C] columns of the input projection, rows `ld` apart
// One thread: V channels of CONV_TOK consecutive tokens.
constexpr int CONV_TOK = 16;

template <typename T, int V>
__device__ __forceinline__ void conv_tap_input(const sk_ssm_params& p, int b, int s, int ch, bool fresh, int channels, float (&r)[V]) {
    if (s >= 0) {
        load_vec<T, V>((const T*)p.xbc_in + ((int64_t)b * p.S + s) * p.in_ld + ch, r);
    } else {
        const int slot = p.taps - 1 + s;                          // carried inputs, oldest first
#pragma unroll
        for (int e = 0; e < V; ++e)
            r[e] = fresh || slot < 0 ? 0.f : to_f32(((const T*)p.conv_state)[((int64_t)b * (p.taps - 1) + slot) * channels + ch + e]);
    }
}

template <typename T, int V, int TAPS>      // TAPS: 0 = any number
__global__ void __launch_bounds__(128)
ssm_conv_kernel(sk_ssm_params p) {
    const int channels = p.H * p.P + 2 * p.G * p.N;
    const int ch = (blockIdx.x * 128 + threadIdx.x) * V, b = blockIdx.z, s0 = blockIdx.y * CONV_TOK;
    if (ch >= channels) return;
    const bool fresh = first_position(p.pos, p.start) == 0;
    const T* w = (const T*)p.conv_w;
    float bias[V];
#pragma unroll
    for (int e = 0; e < V; ++e) bias[e] = to_f32(((const T*)p.conv_b)[ch + e]);
    const int s1 = s0 + CONV_TOK < p.S ? s0 + CONV_TOK : p.S;
    if (TAPS > 0) {                                               // the window slides through registers
        constexpr int K = TAPS > 0 ? TAPS : 1;
        float wt[K][V], win[K][V];
#pragma unroll
        for (int j = 0; j < K; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) wt[j][e] = to_f32(w[(int64_t)(ch + e) * K + j]);
#pragma unroll
        for (int j = 1; j < K; ++j) conv_tap_input<T, V>(p, b, s0 - K + j, ch, fresh, channels, win[j]);
        constexpr int U = 4;                                      // tokens requested together
        for (int s = s0; s < s1; s += U) {
            float in[U][V];
#pragma unroll
            for (int u = 0; u < U; ++u) conv_tap_input<T, V>(p, b, s + u < s1 ? s + u : s1 - 1, ch, fresh, channels, in[u]);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                float acc[V];
#pragma unroll
                for (int e = 0; e < V; ++e) {
#pragma unroll
                    for (int j = 0; j + 1 < K; ++j) win[j][e] = win[j + 1][e];
                    win[K - 1][e] = in[u][e];
                    acc[e] = bias[e];
#pragma unroll
                    for (int j = 0; j < K; ++j) acc[e] = fmaf(wt[j][e], win[j][e], acc[e]);
                    acc[e] = silu<T>(acc[e]);
                }
                if (s + u < s1) store_vec<T, V>((T*)p.xbc + ((int64_t)b * p.S + s + u) * p.xbc_ld + ch, acc);
            }
        }
    } else
    for (int s = s0; s < s1; ++s) {
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = bias[e];
        for (int j = 0; j < p.taps; ++j) {
            float in[V];
            conv_tap_input<T, V>(p, b, s - (p.taps - 1) + j, ch, fresh, channels, in);
#pragma unroll
            for (int e = 0; e < V; ++e) acc[e] = fmaf(to_f32(w[(int64_t)(ch + e) * p.taps + j]), in[e], acc[e]);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = silu<T>(acc[e]);
        store_vec<T, V>((T*)p.xbc + ((int64_t)b * p.S + s) * p.xbc_ld + ch, acc);
    }
    // one token: this thread is the only reader of its channels' carried inputs, so it moves them on itself
    if (p.S == 1) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            T* cs = (T*)p.conv_state + (int64_t)b * (p.taps - 1) * channels + ch + e;
            for (int j = 0; j + 1 < p.taps - 1; ++j) cs[(int64_t)j * channels] = fresh ? from_f32<T>(0.f) : cs[(int64_t)(j + 1) * channels];
            if (p.taps > 1) cs[(int64_t)(p.taps - 2) * channels] = ((const T*)p.xbc_in)[(int64_t)b * p.in_ld + ch + e];
        }
    }
}

// Carried inputs after a portion of several tokens (runs after the convolution has read the old ones).
template <typename T>
__global__ void __launch_bounds__(128)
ssm_conv_state_kernel(sk_ssm_params p) {
    const int channels = p.H * p.P + 2 * p.G * p.N;
    const int ch = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
    if (ch >= channels) return;
    const bool fresh = first_position(p.pos, p.start) == 0;
    T* cs = (T*)p.conv_state + (int64_t)b * (p.taps - 1) * channels + ch;
    for (int j = 0; j < p.taps - 1; ++j) {                        // ascending: slot S + j is read before it is written
        const int s = p.S - (p.taps - 1) + j;
        T v;
        if (s >= 0) v = ((const T*)p.xbc_in)[((int64_t)b * p.S + s) * p.in_ld + ch];
        else v = fresh ? from_f32<T>(0.f) : cs[(int64_t)(p.S + j) * channels];
        cs[(int64_t)j * channels] = v;
    }
}

// ---------------------------------------------------------------- recurrence
// A CTA owns 16 value columns of one head; thread (column, group) keeps N / 16 state elements in registers.
constexpr int ST_COLS = 16, ST_GROUPS = 16;

template <typename T, int NPT>
__global__ void __launch_bounds__(ST_COLS * ST_GROUPS)
ssm_steps_kernel(sk_ssm_params p) {
    __shared__ float red[2][8][ST_COLS];
    const int t = threadIdx.x, c = t & (ST_COLS - 1), grp = t >> 4, warp = t >> 5, lane = t & 31;
    const int col = blockIdx.x * ST_COLS + c, h = blockIdx.y, b = blockIdx.z;
    const bool live = col < p.P;
    const int g = h / (p.H / p.G), I = p.H * p.P;
    const bool fresh = first_position(p.pos, p.start) == 0;
    const float a_rate = -expf(p.A_log[h]), dt_bias = p.dt_bias[h], skip = p.D[h];
    float* st = p.state + ((int64_t)(b * p.H + h) * p.N) * p.P + col;
    float s[NPT];
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
        const int n = grp + k * ST_GROUPS;
        s[k] = (!fresh && live && n < p.N) ? st[(int64_t)n * p.P] : 0.f;
    }
    for (int tok = 0; tok < p.S; ++tok) {
        const int64_t row = (int64_t)b * p.S + tok;
        const T* r = (const T*)p.xbc + row * p.xbc_ld;
        const float dt = softplus_f32(to_f32(((const T*)p.dt_in)[row * p.in_ld + h]) + dt_bias);
        const float decay = expf(a_rate * dt);
        const float x = live ? to_f32(r[h * p.P + col]) : 0.f;
        const float xd = x * dt;
        const T* Bp = r + I + g * p.N;
        const T* Cp = Bp + p.G * p.N;
        float y = 0.f;
#pragma unroll
        for (int k = 0; k < NPT; ++k) {
            const int n = grp + k * ST_GROUPS;
            if (n < p.N) {
                s[k] = fmaf(s[k], decay, to_f32(Bp[n]) * xd);
                y = fmaf(s[k], to_f32(Cp[n]), y);
            }
        }
        y += __shfl_xor_sync(FULL, y, 16);
        float (*rd)[ST_COLS] = red[tok & 1];
        if (lane < 16) rd[warp][c] = y;
        __syncthreads();
        if (t < ST_COLS && live) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) v += rd[w][c];
            ((T*)p.y)[row * I + h * p.P + col] = from_f32<T>(fmaf(skip, x, v));
        }
    }
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
        const int n = grp + k * ST_GROUPS;
        if (live && n < p.N) st[(int64_t)n * p.P] = s[k];
    }
}

// ---------------------------------------------------------------- gate, then RMS norm of each part
template <typename T, int V, int NV>
__global__ void __launch_bounds__(1024)
gated_group_norm_kernel(const T* __restrict__ y, const T* __restrict__ z, int64_t z_ld, const T* __restrict__ w, int inner,
                        int part, float eps, T* __restrict__ out) {
    __shared__ float red[32];
    const int64_t row = blockIdx.x;
    const int c0 = blockIdx.y * part, nt = blockDim.x, t = threadIdx.x;
    float v[NV][V], ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * nt + t) * V;
        if (i < part) {
            float zz[V];
            load_vec<T, V>(y + row * inner + c0 + i, v[n]);
            load_vec<T, V>(z + row * z_ld + c0 + i, zz);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                v[n][e] *= silu<T>(zz[e]);
                ss = fmaf(v[n][e], v[n][e], ss);
            }
        }
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)part + eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * nt + t) * V;
        if (i < part) {
            float ww[V];
            load_vec<T, V>(w + c0 + i, ww);
#pragma unroll
            for (int e = 0; e < V; ++e) v[n][e] *= inv * ww[e];
            store_vec<T, V>(out + row * inner + c0 + i, v[n]);
        }
    }
}

template <typename T, int V>
int norm_dispatch(const void* y, const void* z, int64_t z_ld, const void* w, int64_t rows, int inner, int parts, float eps,
                  void* out, cudaStream_t st) {
    const int part = inner / parts, vecs = (part + V - 1) / V;
    int nt = rows * parts < 296 ? 1024 : 256;
    while (nt > 32 && nt / 2 >= vecs) nt /= 2;
    while (nt < 1024 && (vecs + nt - 1) / nt > 8) nt *= 2;
    const int nv = (vecs + nt - 1) / nt;
    dim3 grid((unsigned)rows, (unsigned)parts);
#define SK_GN(NV) gated_group_norm_kernel<T, V, NV><<<grid, nt, 0, st>>>((const T*)y, (const T*)z, z_ld, (const T*)w, inner, part, eps, (T*)out)
    if (nv <= 1) SK_GN(1);
    else if (nv <= 2) SK_GN(2);
    else if (nv <= 4) SK_GN(4);
    else if (nv <= 8) SK_GN(8);
    else return fail(SK_ERR_UNSUPPORTED, "sk_gated_group_norm: part of %d elements is too large", part);
#undef SK_GN
    return check_launch("gated_group_norm_kernel");
}

template <typename T> int steps_dispatch(const sk_ssm_params& p, cudaStream_t st) {
    dim3 grid((unsigned)((p.P + ST_COLS - 1) / ST_COLS), (unsigned)p.H, (unsigned)p.B);
    const int npt = (p.N + ST_GROUPS - 1) / ST_GROUPS;
    if (npt <= 2) ssm_steps_kernel<T, 2><<<grid, 256, 0, st>>>(p);
    else if (npt <= 4) ssm_steps_kernel<T, 4><<<grid, 256, 0, st>>>(p);
    else if (npt <= 8) ssm_steps_kernel<T, 8><<<grid, 256, 0, st>>>(p);
    else if (npt <= 16) ssm_steps_kernel<T, 16><<<grid, 256, 0, st>>>(p);
    else return fail(SK_ERR_UNSUPPORTED, "sk_ssm: state size %d is too large", p.N);
    return check_launch("ssm_steps_kernel");
}

template <typename T> int conv_dispatch(const sk_ssm_params& p, cudaStream_t st) {
    const int channels = p.H * p.P + 2 * p.G * p.N;
    // the first column of [x | B | C] sits behind the gate's H * P columns
    auto vec = [&](int v) {
        return channels % v == 0 && p.in_ld % v == 0 && p.xbc_ld % v == 0 && (uintptr_t)p.xbc_in % (v * sizeof(T)) == 0;
    };
    const int V = p.S == 1 ? 1 : sizeof(T) == 2 && vec(8) && p.taps == 4 ? 8 : (vec(4) ? 4 : 1);
    dim3 grid((unsigned)((channels + 128 * V - 1) / (128 * V)), (unsigned)((p.S + CONV_TOK - 1) / CONV_TOK), (unsigned)p.B);
    if (V == 8) {
        if constexpr (sizeof(T) == 2) ssm_conv_kernel<T, 8, 4><<<grid, 128, 0, st>>>(p);
    } else if (V == 4 && p.taps == 4) ssm_conv_kernel<T, 4, 4><<<grid, 128, 0, st>>>(p);
    else if (V == 4) ssm_conv_kernel<T, 4, 0><<<grid, 128, 0, st>>>(p);
    else ssm_conv_kernel<T, 1, 0><<<grid, 128, 0, st>>>(p);
    if (int rc = check_launch("ssm_conv_kernel")) return rc;
    if (p.S > 1 && p.taps > 1) {
        ssm_conv_state_kernel<T><<<dim3((unsigned)((channels + 127) / 128), (unsigned)p.B), 128, 0, st>>>(p);
        return check_launch("ssm_conv_state_kernel");
    }
    return SK_OK;
}

}  // namespace

int launch_ssm_conv(const sk_ssm_params& p, cudaStream_t st) {
    return p.dtype == SK_BF16 ? conv_dispatch<__nv_bfloat16>(p, st) : conv_dispatch<float>(p, st);
}

int launch_ssm_steps(const sk_ssm_params& p, cudaStream_t st) {
    return p.dtype == SK_BF16 ? steps_dispatch<__nv_bfloat16>(p, st) : steps_dispatch<float>(p, st);
}

int launch_gated_group_norm(const void* y, const void* z, int64_t z_ld, const void* w, int dtype, int64_t rows,
                            int inner, int parts, float eps, void* out, cudaStream_t st) {
    const int part = inner / parts;
    const bool v4 = part % 4 == 0 && z_ld % 4 == 0;
    if (dtype == SK_BF16 && part % 8 == 0 && z_ld % 8 == 0 && (uintptr_t)z % 16 == 0)
        return norm_dispatch<__nv_bfloat16, 8>(y, z, z_ld, w, rows, inner, parts, eps, out, st);
    if (dtype == SK_BF16)
        return v4 ? norm_dispatch<__nv_bfloat16, 4>(y, z, z_ld, w, rows, inner, parts, eps, out, st)
                  : norm_dispatch<__nv_bfloat16, 1>(y, z, z_ld, w, rows, inner, parts, eps, out, st);
    return v4 ? norm_dispatch<float, 4>(y, z, z_ld, w, rows, inner, parts, eps, out, st)
              : norm_dispatch<float, 1>(y, z, z_ld, w, rows, inner, parts, eps, out, st);
}

}  // namespace sk
