// Latent attention around the softmax: a token's down-projection becomes a cache row
// [normed latent | rotated key part], the queries' rotated parts are turned in place, and - for
// attention directly on the latent rows - the key up-projection is moved to the query side
// (q -> W_uk^T q per head) and the value up-projection behind the weighted sum.
#include "blocks.cuh"

namespace sk {
namespace {

__device__ __forceinline__ void rotate_pair(float& u, float& v, const float* cs) {
    const float a = u * cs[0] - v * cs[1], b = v * cs[0] + u * cs[1];
    u = a;
    v = b;
}

// One CTA per token.  q rows [H, dim + rot] at q + row * q_ld (rotated in place), dkv rows [rank + rot].
template <typename T>
__global__ void __launch_bounds__(256)
latent_append_kernel(sk_latent_params p) {
    __shared__ float red[32];
    const int s = blockIdx.x, b = blockIdx.y, t = threadIdx.x;
    const int64_t i = first_position(p.pos, p.start) + s;
    const int64_t row = (int64_t)b * p.S + s;
    if (i < 0 || i >= p.cap) {
        if (t == 0 && p.status != nullptr) atomicOr(p.status, SK_DEV_POS_OUT_OF_RANGE);
        return;
    }
    const T* d = (const T*)p.dkv + row * p.dkv_ld;
    T* c = (T*)p.cache + ((int64_t)b * p.cap + i) * p.cache_ld;
    const T* w = (const T*)p.norm_w;
    const float* cs = p.angles + i * p.rot_dims;                 // [rot_dims / 2][cos, sin]
    float ss = 0.f;
    for (int j = t; j < p.rank; j += blockDim.x) {
        const float x = to_f32(d[j]);
        ss = fmaf(x, x, ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
    for (int j = t; j < p.rank; j += blockDim.x) c[j] = from_f32<T>(to_f32(d[j]) * inv * to_f32(w[j]));
    for (int j = t; j < p.rot / 2; j += blockDim.x) {
        float u = to_f32(d[p.rank + 2 * j]), v = to_f32(d[p.rank + 2 * j + 1]);
        if (2 * j < p.rot_dims) rotate_pair(u, v, cs + 2 * j);
        c[p.rank + 2 * j] = from_f32<T>(u);
        c[p.rank + 2 * j + 1] = from_f32<T>(v);
    }
    if ((p.rot & 1) && t == 0) c[p.rank + p.rot - 1] = d[p.rank + p.rot - 1];
    for (int j = p.rank + p.rot + t; j < p.cache_ld; j += blockDim.x) c[j] = from_f32<T>(0.f);    // row padding
    T* q = (T*)p.q + row * p.q_ld;
    const int half = p.rot_dims / 2;
    for (int j = t; j < p.H * half; j += blockDim.x) {
        const int h = j / half, k = j - h * half;
        T* e = q + (int64_t)h * (p.dim + p.rot) + p.dim + 2 * k;
        float u = to_f32(e[0]), v = to_f32(e[1]);
        rotate_pair(u, v, cs + 2 * k);
        e[0] = from_f32<T>(u);
        e[1] = from_f32<T>(v);
    }
}

// out[row, h, :] = [ W_uk[h]^T q_unrotated (rank) | q_rotated (rot) | zeros up to out_ld ].  A CTA owns 64 columns of one head; its eight
// warps split the head's `dim` rows of W_uk (coalesced along the columns) and meet in shared memory.
constexpr int AB_ROWS = 8;
template <typename T>
__global__ void __launch_bounds__(256)
latent_absorb_kernel(const T* __restrict__ q, int64_t q_ld, const T* __restrict__ uk, int64_t rows, int H, int dim, int rot,
                     int rank, int out_ld, T* __restrict__ out) {
    extern __shared__ float sm[];                                // q [AB_ROWS][dim], partials [8][AB_ROWS][64]
    float* part = sm + AB_ROWS * dim;
    const int h = blockIdx.x, c0 = blockIdx.y * 64, t = threadIdx.x, warp = t >> 5, lane = t & 31;
    const int64_t r0 = (int64_t)blockIdx.z * AB_ROWS;
    const int n = (int)(rows - r0 < AB_ROWS ? rows - r0 : AB_ROWS);
    for (int j = t; j < n * dim; j += 256) {
        const int r = j / dim, d = j - r * dim;
        sm[r * dim + d] = to_f32(q[(r0 + r) * q_ld + (int64_t)h * (dim + rot) + d]);
    }
    __syncthreads();
    float acc[AB_ROWS][2];
#pragma unroll
    for (int r = 0; r < AB_ROWS; ++r) acc[r][0] = acc[r][1] = 0.f;
    const int ca = c0 + 2 * lane, cb = ca + 1;
    const bool pair = (rank % 2 == 0) && cb < rank;
    for (int d = warp; d < dim; d += 8) {
        const T* w = uk + ((int64_t)h * dim + d) * rank;
        float wa = 0.f, wb = 0.f;
        if (pair && sizeof(T) == 2) {
            const uint32_t u = *reinterpret_cast<const uint32_t*>(w + ca);
            T e[2];
            *reinterpret_cast<uint32_t*>(e) = u;
            wa = to_f32(e[0]);
            wb = to_f32(e[1]);
        } else {
            if (ca < rank) wa = to_f32(w[ca]);
            if (cb < rank) wb = to_f32(w[cb]);
        }
#pragma unroll
        for (int r = 0; r < AB_ROWS; ++r) {
            if (r < n) {
                const float x = sm[r * dim + d];
                acc[r][0] = fmaf(x, wa, acc[r][0]);
                acc[r][1] = fmaf(x, wb, acc[r][1]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < AB_ROWS; ++r) {
        part[(warp * AB_ROWS + r) * 64 + 2 * lane] = acc[r][0];
        part[(warp * AB_ROWS + r) * 64 + 2 * lane + 1] = acc[r][1];
    }
    __syncthreads();
    for (int j = t; j < n * 64; j += 256) {
        const int r = j >> 6, c = c0 + (j & 63);
        if (c < out_ld) {
            float v = 0.f;
            if (c < rank) {
#pragma unroll
                for (int k = 0; k < 8; ++k) v += part[(k * AB_ROWS + r) * 64 + (j & 63)];
            } else if (c < rank + rot) {
                v = to_f32(q[(r0 + r) * q_ld + (int64_t)h * (dim + rot) + dim + (c - rank)]);
            }
            out[((r0 + r) * H + h) * (int64_t)out_ld + c] = from_f32<T>(v);
        }
    }
}

// The same for bf16 and a rank that is a multiple of 8: a CTA owns 128 columns of one head, 16 threads along them
// (8 columns each) and 16 along the head's rows of W_uk, so that a thread's loads are few, wide and in flight together.
template <int ROWS>
__global__ void __launch_bounds__(256)
latent_absorb_vec_kernel(const __nv_bfloat16* __restrict__ q, int64_t q_ld, const __nv_bfloat16* __restrict__ uk, int64_t rows,
                         int H, int dim, int rot, int rank, int out_ld, __nv_bfloat16* __restrict__ out) {
    extern __shared__ float sm[];                                // q [ROWS][dim], partials [16][ROWS][128]
    float* part = sm + ROWS * dim;
    const int h = blockIdx.x, c0 = blockIdx.y * 128, t = threadIdx.x, cl = t & 15, dg = t >> 4;
    const int64_t r0 = (int64_t)blockIdx.z * ROWS;
    const int n = (int)(rows - r0 < ROWS ? rows - r0 : ROWS), c = c0 + cl * 8;
    float acc[ROWS][8];
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = 0.f;
    const bool live = c < rank;
    const __nv_bfloat16* w = uk + (int64_t)h * dim * rank + c;
    constexpr int U = 8;                                         // rows of W_uk in flight per thread
    uint4 wv[U];
    auto load = [&](int d0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int d = d0 + dg + 16 * u;
            wv[u] = live && d < dim ? __ldg(reinterpret_cast<const uint4*>(w + (int64_t)d * rank)) : make_uint4(0, 0, 0, 0);
        }
    };
    load(0);
    for (int r = 0; r < n; ++r)
        for (int d = t; d < dim; d += 256) sm[r * dim + d] = to_f32(q[(r0 + r) * q_ld + (int64_t)h * (dim + rot) + d]);
    for (int r = n; r < ROWS; ++r)
        for (int d = t; d < dim; d += 256) sm[r * dim + d] = 0.f;
    __syncthreads();
    for (int d0 = 0; d0 < dim; d0 += 16 * U) {
        if (d0 > 0) load(d0);
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int d = d0 + dg + 16 * u;
            if (d < dim) {
                const uint32_t x[4] = {wv[u].x, wv[u].y, wv[u].z, wv[u].w};
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    const float qv = sm[r * dim + d];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        acc[r][2 * e] = fmaf(qv, __uint_as_float(x[e] << 16), acc[r][2 * e]);
                        acc[r][2 * e + 1] = fmaf(qv, __uint_as_float(x[e] & 0xffff0000u), acc[r][2 * e + 1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) part[(dg * ROWS + r) * 128 + cl * 8 + e] = acc[r][e];
    __syncthreads();
    for (int j = t; j < n * 128; j += 256) {
        const int r = j >> 7, cc = c0 + (j & 127);
        if (cc < out_ld) {
            float v = 0.f;
            if (cc < rank) {
#pragma unroll
                for (int k = 0; k < 16; ++k) v += part[(k * ROWS + r) * 128 + (j & 127)];
            } else if (cc < rank + rot) {
                v = to_f32(q[(r0 + r) * q_ld + (int64_t)h * (dim + rot) + dim + (cc - rank)]);
            }
            out[((r0 + r) * H + h) * (int64_t)out_ld + cc] = __float2bfloat16_rn(v);
        }
    }
}

// out[row, h * vdim + e] for bf16 and a rank that is a multiple of 8: one warp per output element and row group
template <int ROWS>
__global__ void __launch_bounds__(128)
latent_up_vec_kernel(const __nv_bfloat16* __restrict__ o, const __nv_bfloat16* __restrict__ uv, int64_t rows, int H, int vdim,
                     int rank, __nv_bfloat16* __restrict__ out) {
    const int lane = threadIdx.x & 31;
    const int e = blockIdx.x * 4 + (threadIdx.x >> 5);
    const int64_t r0 = (int64_t)blockIdx.y * ROWS;
    if (e >= H * vdim) return;
    const int h = e / vdim, n = (int)(rows - r0 < ROWS ? rows - r0 : ROWS);
    const __nv_bfloat16* w = uv + (int64_t)e * rank;
    float acc[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
#pragma unroll 2
    for (int j = 8 * lane; j < rank; j += 256) {
        const uint4 wq = __ldg(reinterpret_cast<const uint4*>(w + j));
        const uint32_t x[4] = {wq.x, wq.y, wq.z, wq.w};
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            if (r < n) {
                const uint4 oq = *reinterpret_cast<const uint4*>(o + ((r0 + r) * H + h) * (int64_t)rank + j);
                const uint32_t y[4] = {oq.x, oq.y, oq.z, oq.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    acc[r] = fmaf(__uint_as_float(x[k] << 16), __uint_as_float(y[k] << 16), acc[r]);
                    acc[r] = fmaf(__uint_as_float(x[k] & 0xffff0000u), __uint_as_float(y[k] & 0xffff0000u), acc[r]);
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (r < n) {
            const float v = warp_sum(acc[r]);
            if (lane == 0) out[(r0 + r) * (int64_t)H * vdim + e] = __float2bfloat16_rn(v);
        }
}

// out[row, h * vdim + e] = <W_uv[h * vdim + e, :], o[row, h, :]>: one warp per output element and row group
template <typename T>
__global__ void __launch_bounds__(256)
latent_up_kernel(const T* __restrict__ o, const T* __restrict__ uv, int64_t rows, int H, int vdim, int rank, T* __restrict__ out) {
    const int lane = threadIdx.x & 31;
    const int e = blockIdx.x * 8 + (threadIdx.x >> 5);           // flat (head, value dimension)
    const int64_t r0 = (int64_t)blockIdx.y * AB_ROWS;
    if (e >= H * vdim) return;
    const int h = e / vdim, n = (int)(rows - r0 < AB_ROWS ? rows - r0 : AB_ROWS);
    const T* w = uv + (int64_t)e * rank;
    float acc[AB_ROWS];
#pragma unroll
    for (int r = 0; r < AB_ROWS; ++r) acc[r] = 0.f;
    if (rank % 4 == 0) {
        for (int j = 4 * lane; j < rank; j += 128) {
            float wv[4];
            load_vec<T, 4>(w + j, wv);
#pragma unroll
            for (int r = 0; r < AB_ROWS; ++r)
                if (r < n) {
                    float x[4];
                    load_vec<T, 4>(o + ((r0 + r) * H + h) * (int64_t)rank + j, x);
#pragma unroll
                    for (int k = 0; k < 4; ++k) acc[r] = fmaf(wv[k], x[k], acc[r]);
                }
        }
    } else {
        for (int j = lane; j < rank; j += 32) {
            const float wv = to_f32(w[j]);
#pragma unroll
            for (int r = 0; r < AB_ROWS; ++r)
                if (r < n) acc[r] = fmaf(wv, to_f32(o[((r0 + r) * H + h) * (int64_t)rank + j]), acc[r]);
        }
    }
#pragma unroll
    for (int r = 0; r < AB_ROWS; ++r)
        if (r < n) {
            const float v = warp_sum(acc[r]);
            if (lane == 0) out[(r0 + r) * (int64_t)H * vdim + e] = from_f32<T>(v);
        }
}

}  // namespace

int launch_latent_append(const sk_latent_params& p, cudaStream_t st) {
    dim3 grid((unsigned)p.S, (unsigned)p.B);
    if (p.dtype == SK_BF16) latent_append_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(p);
    else latent_append_kernel<float><<<grid, 256, 0, st>>>(p);
    return check_launch("latent_append_kernel");
}

int launch_latent_absorb(const void* q, int64_t q_ld, int dtype, const void* uk, int64_t rows, int H, int dim, int rot,
                         int rank, int out_ld, void* out, cudaStream_t st) {
    if (dtype == SK_BF16 && rank % 8 == 0 && (uintptr_t)uk % 16 == 0 && dim <= 512) {
        const __nv_bfloat16 *qb = (const __nv_bfloat16*)q, *ub = (const __nv_bfloat16*)uk;
        const int R = rows == 1 ? 1 : 4;
        dim3 grid((unsigned)H, (unsigned)((out_ld + 127) / 128), (unsigned)((rows + R - 1) / R));
        const size_t smem = (size_t)(R * dim + 16 * R * 128) * sizeof(float);
        if (R == 1) latent_absorb_vec_kernel<1><<<grid, 256, smem, st>>>(qb, q_ld, ub, rows, H, dim, rot, rank, out_ld, (__nv_bfloat16*)out);
        else latent_absorb_vec_kernel<4><<<grid, 256, smem, st>>>(qb, q_ld, ub, rows, H, dim, rot, rank, out_ld, (__nv_bfloat16*)out);
        return check_launch("latent_absorb_vec_kernel");
    }
    dim3 grid((unsigned)H, (unsigned)((out_ld + 63) / 64), (unsigned)((rows + AB_ROWS - 1) / AB_ROWS));
    const size_t smem = (size_t)(AB_ROWS * dim + 8 * AB_ROWS * 64) * sizeof(float);
    if (smem > 48 * 1024) return fail(SK_ERR_UNSUPPORTED, "sk_latent_absorb: head size %d is too large", dim);
    if (dtype == SK_BF16)
        latent_absorb_kernel<<<grid, 256, smem, st>>>((const __nv_bfloat16*)q, q_ld, (const __nv_bfloat16*)uk, rows, H, dim,
                                                      rot, rank, out_ld, (__nv_bfloat16*)out);
    else
        latent_absorb_kernel<<<grid, 256, smem, st>>>((const float*)q, q_ld, (const float*)uk, rows, H, dim, rot, rank,
                                                      out_ld, (float*)out);
    return check_launch("latent_absorb_kernel");
}

int launch_latent_up(const void* o, int dtype, const void* uv, int64_t rows, int H, int vdim, int rank, void* out,
                     cudaStream_t st) {
    if (dtype == SK_BF16 && rank % 8 == 0 && (uintptr_t)uv % 16 == 0 && (uintptr_t)o % 16 == 0) {
        const __nv_bfloat16 *ob = (const __nv_bfloat16*)o, *ub = (const __nv_bfloat16*)uv;
        const int R = rows == 1 ? 1 : 4;
        dim3 grid((unsigned)((H * vdim + 3) / 4), (unsigned)((rows + R - 1) / R));
        if (R == 1) latent_up_vec_kernel<1><<<grid, 128, 0, st>>>(ob, ub, rows, H, vdim, rank, (__nv_bfloat16*)out);
        else latent_up_vec_kernel<4><<<grid, 128, 0, st>>>(ob, ub, rows, H, vdim, rank, (__nv_bfloat16*)out);
        return check_launch("latent_up_vec_kernel");
    }
    dim3 grid((unsigned)((H * vdim + 7) / 8), (unsigned)((rows + AB_ROWS - 1) / AB_ROWS));
    if (dtype == SK_BF16)
        latent_up_kernel<<<grid, 256, 0, st>>>((const __nv_bfloat16*)o, (const __nv_bfloat16*)uv, rows, H, vdim, rank,
                                               (__nv_bfloat16*)out);
    else
        latent_up_kernel<<<grid, 256, 0, st>>>((const float*)o, (const float*)uv, rows, H, vdim, rank, (float*)out);
    return check_launch("latent_up_kernel");
}

}  // namespace sk
