// Decoder building blocks (libsocket_b200_blocks.so): launcher declarations and the few helpers the
// block kernels share.  Residual streams, norms, scores, softmax and recurrent state are fp32
// throughout; activations and matrix operands have the element type of the model (bf16 or fp32).
#pragma once
#include "../../include/socket_b200_blocks.h"
#include "common.cuh"

namespace sk {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) v += __shfl_xor_sync(FULL, v, o);
    return v;
}

// Sum over the block; `red` holds one float per warp (32), every thread gets the result.  Two uses in
// a row need different `red` arrays or a barrier in between.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (int)((blockDim.x + 31) >> 5);
    if (nw == 1) return v;
    if (lane == 0) red[warp] = v;
    __syncthreads();
    return warp_sum(lane < nw ? red[lane] : 0.f);
}

// V consecutive elements at p <-> fp32 registers; p aligned to V elements
template <typename T, int V> __device__ __forceinline__ void load_vec(const T* p, float (&r)[V]) {
    if constexpr (V == 4 && sizeof(T) == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        r[0] = a.x; r[1] = a.y; r[2] = a.z; r[3] = a.w;
    } else if constexpr (V == 4 && sizeof(T) == 2) {
        const uint2 a = *reinterpret_cast<const uint2*>(p);
        T e[4];
        *reinterpret_cast<uint2*>(e) = a;
#pragma unroll
        for (int i = 0; i < 4; ++i) r[i] = to_f32(e[i]);
    } else if constexpr (V == 8 && sizeof(T) == 2) {
        const uint4 a = *reinterpret_cast<const uint4*>(p);
        T e[8];
        *reinterpret_cast<uint4*>(e) = a;
#pragma unroll
        for (int i = 0; i < 8; ++i) r[i] = to_f32(e[i]);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) r[i] = to_f32(p[i]);
    }
}
template <typename T, int V> __device__ __forceinline__ void store_vec(T* p, const float (&r)[V]) {
    if constexpr (V == 4 && sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]);
    } else if constexpr (V == 4 && sizeof(T) == 2) {
        T e[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) e[i] = from_f32<T>(r[i]);
        *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(e);
    } else if constexpr (V == 8 && sizeof(T) == 2) {
        T e[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) e[i] = from_f32<T>(r[i]);
        *reinterpret_cast<uint4*>(p) = *reinterpret_cast<uint4*>(e);
    } else {
#pragma unroll
        for (int i = 0; i < V; ++i) p[i] = from_f32<T>(r[i]);
    }
}

__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// activations: full fp32 accuracy for fp32 models; for bf16 ones the hardware exponential and division,
// whose error is far below the rounding of the result
template <typename T> __device__ __forceinline__ float sigmoid_scaled(float x, float slope) {
    if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-slope * x));
    else return 1.f / (1.f + expf(-slope * x));
}
template <typename T> __device__ __forceinline__ float silu(float x) { return x * sigmoid_scaled<T>(x, 1.f); }
// cap * tanh(x / cap) in full fp32 accuracy
__device__ __forceinline__ float soft_cap_f32(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
// tanh(x) with an absolute error of about 1e-7, from one hardware exponential and one division
__device__ __forceinline__ float tanh_exp2(float x) {
    return 1.f - __fdividef(2.f, 1.f + exp2_fast(x * 2.8853900817779268f));        // 2 log2(e)
}
// tanh(x) / x for |x| <= 1/2 as a polynomial in x^2: interpolation at Chebyshev nodes, error 1.3e-8
constexpr float TANH_POLY_RANGE = 0.5f;
constexpr double TANH_POLY[5] = {0.999999987, -0.333330719, 0.13324829, -0.0529892412, 0.017141319};
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// position of the first token of a portion: on the device (decode) or given by the host
__device__ __forceinline__ int64_t first_position(const int64_t* pos, int64_t start) { return pos != nullptr ? pos[0] : start; }

// ---------------------------------------------------------------- launchers
int launch_embed_rows(const int64_t* tokens, const void* table, int dtype, int64_t rows, int64_t vocab, int width,
                      float scale, float* x, float* x_copy, int32_t* status, cudaStream_t st);
int launch_residual_norm(const sk_residual_params& p, cudaStream_t st);
int launch_glu(const void* gate, const void* up, int dtype, int64_t rows, int ff, int64_t ld, int kind, float limit, float slope,
               void* out, int64_t out_ld, cudaStream_t st);
int launch_ring_append(const void* k, const void* v, int dtype, int B, int S, int64_t k_bs, int64_t k_ss, int64_t v_bs,
                       int64_t v_ss, int k_row, int v_row, int ring, int keep, const int64_t* pos, int64_t start, void* k_cache,
                       void* v_cache, cudaStream_t st);
int launch_rotary_rows(const sk_rotary_rows_params& p, cudaStream_t st);
int launch_attn_rows(const sk_attn_params& p, cudaStream_t st);
bool attn_prefill_tc_applicable(const sk_attn_params& p);
int launch_attn_prefill_tc(const sk_attn_params& p, cudaStream_t st);
bool attn_decode_mma_applicable(const sk_attn_params& p);
size_t attn_decode_mma_workspace(const sk_attn_params& p);
int launch_attn_decode_mma(const sk_attn_params& p, cudaStream_t st);
int launch_latent_append(const sk_latent_params& p, cudaStream_t st);
int launch_latent_absorb(const void* q, int64_t q_ld, int dtype, const void* uk, int64_t rows, int H, int dim, int rot,
                         int rank, int out_ld, void* out, cudaStream_t st);
int launch_latent_up(const void* o, int dtype, const void* uv, int64_t rows, int H, int vdim, int rank, void* out,
                     cudaStream_t st);
int launch_ssm_conv(const sk_ssm_params& p, cudaStream_t st);
int launch_ssm_steps(const sk_ssm_params& p, cudaStream_t st);
bool ssm_chunks_applicable(const sk_ssm_params& p);
size_t ssm_chunks_workspace(const sk_ssm_params& p);
int launch_ssm_chunks(const sk_ssm_params& p, cudaStream_t st);
int launch_gated_group_norm(const void* y, const void* z, int64_t z_ld, const void* w, int dtype, int64_t rows,
                            int inner, int parts, float eps, void* out, cudaStream_t st);
bool mlstm_chunks_applicable(const sk_mlstm_params& p);
size_t mlstm_chunks_workspace(const sk_mlstm_params& p);
int launch_mlstm_chunks(const sk_mlstm_params& p, cudaStream_t st);
bool mlstm_tc_applicable(const sk_mlstm_params& p);
size_t mlstm_tc_workspace(const sk_mlstm_params& p);
int launch_mlstm_tc(const sk_mlstm_params& p, cudaStream_t st);
int launch_mlstm_steps(const sk_mlstm_params& p, cudaStream_t st);
int launch_mlstm_finish(const sk_mlstm_params& p, cudaStream_t st);

}  // namespace sk
