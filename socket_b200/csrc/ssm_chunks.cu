// Selective state-space recurrence over a prompt portion as matrix products per block of 64 tokens (bf16
// inputs).  With cum_t the running sum of the log decays inside a block,
//   y_t = exp(cum_t) C_t^T S_in + sum_{s <= t} (C_t . B_s) exp(cum_t - cum_s) dt_s x_s + D x_t
//   S_out = exp(cum_end) S_in + sum_s B_s (exp(cum_end - cum_s) dt_s x_s)^T
// A first kernel computes the step sizes and running decays (base-2 logarithms) of all blocks.  Then a CTA owns
// 32 value columns of one head and walks the blocks in order, two CTAs per SM; the state stays in fp32
// accumulator registers.  B, C and x are bf16 as the convolution leaves them, products accumulate in fp32,
// and every factor that carries a decay, a step size or the state enters a product as two bf16 numbers
// (value and remainder, 16 significant bits together), so that nothing of the recurrence is rounded to
// 8 bits.
#include "blocks.cuh"
#include "warp_mma.cuh"

namespace sk {
namespace {

constexpr int SC_TOK = 64, SC_P = 32, SC_THR = 256;
constexpr int SC_PS = SC_P + 8;              // shared-memory row of 32 columns
constexpr float SC_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 r = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&r);
}

// dt[b][h][t] = softplus(step column + bias), cum[b][h][t] = running sum of -exp(A_log) dt log2(e) inside t's block;
// tokens past the portion's end get dt = 0 and leave the sum as it is.  A CTA: 64 tokens of 32 heads.
__global__ void __launch_bounds__(256)
ssm_decay_kernel(sk_ssm_params p, int blocks, float* __restrict__ dt, float* __restrict__ cum) {
    __shared__ float tile[32][SC_TOK + 1];
    const int blk = blockIdx.x, h0 = blockIdx.y * 32, b = blockIdx.z, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    const int h = h0 + lane;
    const float bias = h < p.H ? p.dt_bias[h] : 0.f;
    for (int s = warp; s < SC_TOK; s += 8) {
        const int tok = blk * SC_TOK + s;
        float d = 0.f;
        if (h < p.H && tok < p.S)
            d = softplus_f32(to_f32(((const __nv_bfloat16*)p.dt_in)[((int64_t)b * p.S + tok) * p.in_ld + h]) + bias);
        tile[lane][s] = d;
    }
    __syncthreads();
    for (int k = warp; k < 32 && h0 + k < p.H; k += 8) {
        const float rate = -expf(p.A_log[h0 + k]) * SC_LOG2E;
        const float d0 = tile[k][2 * lane], d1 = tile[k][2 * lane + 1];
        float sum = rate * d0 + rate * d1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(FULL, sum, o);
            if (lane >= o) sum += x;
        }
        const int64_t at = (((int64_t)b * p.H + h0 + k) * blocks + blk) * SC_TOK + 2 * lane;
        *reinterpret_cast<float2*>(dt + at) = make_float2(d0, d1);
        *reinterpret_cast<float2*>(cum + at) = make_float2(sum - rate * d1, sum);
    }
}

// NM: 16-row tiles of the state per warp (8 warps x 16 NM >= N)
template <int NM>
__global__ void __launch_bounds__(SC_THR, NM == 1 ? 2 : 1)
ssm_chunks_kernel(sk_ssm_params p, int ns, int blocks, const float* __restrict__ dt_g, const float* __restrict__ cum_g) {
    extern __shared__ __align__(16) char sc_raw[];
    __shared__ __align__(16) float cum_sh[2][SC_TOK], dt_sh[2][SC_TOK];
    __shared__ float w_sh[SC_TOK];
    using bf = __nv_bfloat16;
    const int n16 = (p.N + 15) / 16 * 16;
    bf* b_s = reinterpret_cast<bf*>(sc_raw);                  // [2][64][ns]
    bf* c_s = b_s + 2 * SC_TOK * ns;                          // [2][64][ns]
    bf* x_s = c_s + 2 * SC_TOK * ns;                          // [2][64][40]
    bf* st_s = x_s + 2 * SC_TOK * SC_PS;                      // [hi, lo][n16][40]
    float4* ex_s = reinterpret_cast<float4*>(st_s + 2 * n16 * SC_PS);   // [warp][2][lane]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, fr = lane >> 2, fc = (lane & 3) * 2;
    const int p0 = blockIdx.x * SC_P, h = blockIdx.y, b = blockIdx.z;
    const int g = h / (p.H / p.G), I = p.H * p.P, pc = p.P - p0 < SC_P ? p.P - p0 : SC_P;
    const bool fresh = first_position(p.pos, p.start) == 0;
    const float skip = p.D[h];
    const bf* rows = (const bf*)p.xbc + (int64_t)b * p.S * p.xbc_ld;
    const int nc = p.N / 8, xc = pc / 8;
    const float* dt_h = dt_g + ((int64_t)b * p.H + h) * blocks * SC_TOK;
    const float* cum_h = cum_g + ((int64_t)b * p.H + h) * blocks * SC_TOK;

    auto fetch = [&](int blk, int stage) {
        const int t0 = blk * SC_TOK;
        for (int r = warp; r < SC_TOK; r += SC_THR / 32) {    // a warp per token, lanes along its row
            const bool live = t0 + r < p.S;
            const bf* row = rows + (int64_t)(live ? t0 + r : p.S - 1) * p.xbc_ld;
            const bf* bsrc = row + I + g * p.N;
            const bf* csrc = bsrc + p.G * p.N;
            const uint32_t bd = saddr(b_s + (stage * SC_TOK + r) * ns), cd = saddr(c_s + (stage * SC_TOK + r) * ns);
            for (int c = lane; c < 2 * nc; c += 32) {
                if (c < nc) cp16(bd + c * 16, bsrc + c * 8, live);
                else cp16(cd + (c - nc) * 16, csrc + (c - nc) * 8, live);
            }
        }
        for (int r = tid >> 2; r < SC_TOK; r += SC_THR / 4) { // four lanes per token: up to 32 columns of x
            const bool live = t0 + r < p.S;
            if ((tid & 3) < xc)
                cp16(saddr(x_s + (stage * SC_TOK + r) * SC_PS + (tid & 3) * 8),
                     rows + (int64_t)(live ? t0 + r : p.S - 1) * p.xbc_ld + h * p.P + p0 + (tid & 3) * 8, live);
        }
        if (tid < SC_TOK / 4) cp16(saddr(&dt_sh[stage][tid * 4]), dt_h + t0 + tid * 4, true);
        else if (tid < SC_TOK / 2) cp16(saddr(&cum_sh[stage][(tid - SC_TOK / 4) * 4]), cum_h + t0 + (tid - SC_TOK / 4) * 4, true);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    // columns that round N up to 16 and a narrow last slice up to 32 stay zero
    for (int e = tid; e < 4 * SC_TOK * (ns - p.N); e += SC_THR) {
        const int w = ns - p.N, r = e / w;
        b_s[(int64_t)r * ns + p.N + (e - r * w)] = __float2bfloat16_rn(0.f);   // b_s and c_s are one array of 256 rows
    }
    for (int e = tid; e < 2 * SC_TOK * (SC_PS - pc); e += SC_THR) {
        const int w = SC_PS - pc, r = e / w;
        x_s[r * SC_PS + pc + (e - r * w)] = __float2bfloat16_rn(0.f);
    }

    // state rows of this warp: tiles warp, warp + 8 of 16 rows each
    float st[NM][4][4];
    float* gst = p.state + ((int64_t)(b * p.H + h) * p.N) * p.P + p0;
#pragma unroll
    for (int u = 0; u < NM; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = (warp + 8 * u) * 16 + fr + 8 * (e >> 1), c = v * 8 + fc + (e & 1);
                st[u][v][e] = (!fresh && n < p.N && c < pc) ? gst[(int64_t)n * p.P + c] : 0.f;
            }
    auto publish_state = [&]() {                              // the state as two bf16 parts, for C . S
#pragma unroll
        for (int u = 0; u < NM; ++u) {
            const int n = (warp + 8 * u) * 16 + fr;
            if ((warp + 8 * u) * 16 < n16) {
#pragma unroll
                for (int v = 0; v < 4; ++v)
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        uint32_t hi, lo;
                        split_bf16(st[u][v][2 * k], st[u][v][2 * k + 1], hi, lo);
                        bf* dst = st_s + (n + 8 * k) * SC_PS + v * 8 + fc;
                        *reinterpret_cast<uint32_t*>(dst) = hi;
                        *reinterpret_cast<uint32_t*>(dst + n16 * SC_PS) = lo;
                    }
            }
        }
    };
    publish_state();
    const int mt = warp & 3, half = warp >> 2;                // 16-token tile; half of the keys / of the value columns
    const bool own_keys = half == 0 || mt >= 2;               // keys 32.. are later than tokens 0..31
    const bool partner_keys = half == 1 || mt >= 2;

    for (int blk = 0; blk < blocks; ++blk) {
        const int stage = blk & 1, t0 = blk * SC_TOK;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                      // the block's rows and the state are there, the other stage is free
        if (blk + 1 < blocks) fetch(blk + 1, stage ^ 1);
        const bf* bt = b_s + stage * SC_TOK * ns;
        const bf* ct = c_s + stage * SC_TOK * ns;
        const bf* xt = x_s + stage * SC_TOK * SC_PS;
        const float* cum = cum_sh[stage];
        const float* dt = dt_sh[stage];
        const float total = cum[SC_TOK - 1];
        if (tid < SC_TOK) w_sh[tid] = dt[tid] * exp2f(total - cum[tid]);
        // ---- C . B of 16 tokens x 32 keys, C . S of 16 tokens x 16 value columns
        float gacc[4][4], y[2][4];
#pragma unroll
        for (int v = 0; v < 4; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) gacc[v][e] = 0.f;
#pragma unroll
        for (int v = 0; v < 2; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[v][e] = 0.f;
        const uint32_t ca = saddr(ct + (mt * 16 + (lane & 15)) * ns + (lane >> 4) * 8);
        const uint32_t ba = saddr(bt + (half * 32 + (lane & 7) + (lane >> 4) * 8) * ns + ((lane >> 3) & 1) * 8);
        const uint32_t sa = saddr(st_s + (lane & 15) * SC_PS + half * 16 + (lane >> 4) * 8);
#pragma unroll 2
        for (int k = 0; k < n16 / 16; ++k) {
            uint32_t a[4], bb[4];
            ldsm4(ca + k * 32, a);
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                ldsm4t(sa + (part * n16 + k * 16) * SC_PS * 2, bb);
                mma16816(y[0], a, bb[0], bb[1]);
                mma16816(y[1], a, bb[2], bb[3]);
            }
            if (own_keys) {
#pragma unroll
                for (int v = 0; v < 4; v += 2) {
                    ldsm4(ba + v * 8 * ns * 2 + k * 32, bb);
                    mma16816(gacc[v], a, bb[0], bb[1]);
                    mma16816(gacc[v + 1], a, bb[2], bb[3]);
                }
            }
        }
        const int tr[2] = {mt * 16 + fr, mt * 16 + fr + 8};
        const float ct_r[2] = {cum[tr[0]], cum[tr[1]]};
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float f = exp2f(ct_r[k]);
#pragma unroll
            for (int v = 0; v < 2; ++v) {
                y[v][2 * k] *= f;
                y[v][2 * k + 1] *= f;
            }
        }
        // ---- (weighted C . B) . x over this warp's keys, all 32 columns; the partner's columns change hands
        if (own_keys) {
            float z[4][4];
#pragma unroll
            for (int v = 0; v < 4; ++v)
#pragma unroll
                for (int e = 0; e < 4; ++e) z[v][e] = 0.f;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int s0 = half * 32 + k * 16;
                if (s0 > mt * 16) continue;                   // all keys later than the tokens
                uint32_t a[2][4];
#pragma unroll
                for (int v = 0; v < 2; ++v) {
                    const int s = s0 + v * 8 + fc;
                    const float c0 = cum[s], c1 = cum[s + 1], d0 = dt[s], d1 = dt[s + 1];
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const float w0 = s <= tr[r] ? gacc[2 * k + v][2 * r] * (exp2f(ct_r[r] - c0) * d0) : 0.f;
                        const float w1 = s + 1 <= tr[r] ? gacc[2 * k + v][2 * r + 1] * (exp2f(ct_r[r] - c1) * d1) : 0.f;
                        split_bf16(w0, w1, a[0][2 * v + r], a[1][2 * v + r]);
                    }
                }
#pragma unroll
                for (int c = 0; c < 4; c += 2) {
                    uint32_t bb[4];
                    ldsm4t(saddr(xt + (s0 + (lane & 15)) * SC_PS + c * 8 + (lane >> 4) * 8), bb);
#pragma unroll
                    for (int part = 0; part < 2; ++part) {
                        mma16816(z[c], a[part], bb[0], bb[1]);
                        mma16816(z[c + 1], a[part], bb[2], bb[3]);
                    }
                }
            }
#pragma unroll
            for (int v = 0; v < 2; ++v) {
                float own[4], other[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    own[e] = half == 0 ? z[v][e] : z[2 + v][e];
                    other[e] = half == 0 ? z[2 + v][e] : z[v][e];
                    y[v][e] += own[e];
                }
                ex_s[(warp * 2 + v) * 32 + lane] = make_float4(other[0], other[1], other[2], other[3]);
            }
        }
        __syncthreads();
        if (partner_keys) {
#pragma unroll
            for (int v = 0; v < 2; ++v) {
                const float4 o = ex_s[((warp ^ 4) * 2 + v) * 32 + lane];
                y[v][0] += o.x;
                y[v][1] += o.y;
                y[v][2] += o.z;
                y[v][3] += o.w;
            }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            if (t0 + tr[k] < p.S) {
#pragma unroll
                for (int v = 0; v < 2; ++v) {
                    const int c = half * 16 + v * 8 + fc;
                    if (c < pc) {
                        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xt + tr[k] * SC_PS + c);
                        *reinterpret_cast<__nv_bfloat162*>((bf*)p.y + ((int64_t)b * p.S + t0 + tr[k]) * I + h * p.P + p0 + c) =
                            __floats2bfloat162_rn(fmaf(skip, __low2float(x), y[v][2 * k]),
                                                  fmaf(skip, __high2float(x), y[v][2 * k + 1]));
                    }
                }
            }
        }
        // ---- state: (weighted B)^T . x on top of the decayed state
        const float f = exp2f(total);
#pragma unroll
        for (int u = 0; u < NM; ++u) {
            const int n0 = (warp + 8 * u) * 16;
            if (n0 < n16) {
#pragma unroll
                for (int v = 0; v < 4; ++v)
#pragma unroll
                    for (int e = 0; e < 4; ++e) st[u][v][e] *= f;
#pragma unroll
                for (int k = 0; k < SC_TOK / 16; ++k) {
                    uint32_t raw[4], a[2][4];                 // B^T: rows n, columns tokens, stored token by token
                    ldsm4t(saddr(bt + (k * 16 + (lane & 7) + (lane >> 4) * 8) * ns + n0 + ((lane >> 3) & 1) * 8), raw);
                    const float2 w0 = *reinterpret_cast<const float2*>(w_sh + k * 16 + fc);
                    const float2 w1 = *reinterpret_cast<const float2*>(w_sh + k * 16 + 8 + fc);
#pragma unroll
                    for (int r = 0; r < 4; ++r) {
                        const float2 w = r < 2 ? w0 : w1;
                        split_bf16(__uint_as_float(raw[r] << 16) * w.x, __uint_as_float(raw[r] & 0xffff0000u) * w.y, a[0][r], a[1][r]);
                    }
#pragma unroll
                    for (int v = 0; v < 4; v += 2) {
                        uint32_t bb[4];
                        ldsm4t(saddr(xt + (k * 16 + (lane & 15)) * SC_PS + v * 8 + (lane >> 4) * 8), bb);
#pragma unroll
                        for (int part = 0; part < 2; ++part) {
                            mma16816(st[u][v], a[part], bb[0], bb[1]);
                            mma16816(st[u][v + 1], a[part], bb[2], bb[3]);
                        }
                    }
                }
            }
        }
        publish_state();                                      // C . S of this block was read before the last barrier
    }
#pragma unroll
    for (int u = 0; u < NM; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = (warp + 8 * u) * 16 + fr + 8 * (e >> 1), c = v * 8 + fc + (e & 1);
                if (n < p.N && c < pc) gst[(int64_t)n * p.P + c] = st[u][v][e];
            }
}

size_t chunks_smem(int N, int* ns) {
    const int n16 = (N + 15) / 16 * 16;
    *ns = n16 + 8;
    return ((size_t)4 * SC_TOK * *ns + 2 * SC_TOK * SC_PS + (size_t)2 * n16 * SC_PS) * 2 + (size_t)(SC_THR / 32) * 2 * 32 * 16;
}

int chunk_blocks(const sk_ssm_params& p) { return (p.S + SC_TOK - 1) / SC_TOK; }

}  // namespace

bool ssm_chunks_applicable(const sk_ssm_params& p) {
    return p.dtype == SK_BF16 && p.pos == nullptr && p.N % 8 == 0 && p.N <= 256 && p.P % 8 == 0 && p.xbc_ld % 8 == 0 &&
           (uintptr_t)p.xbc % 16 == 0;
}

size_t ssm_chunks_workspace(const sk_ssm_params& p) {         // step sizes and running decays
    return (size_t)2 * p.B * p.H * chunk_blocks(p) * SC_TOK * sizeof(float);
}

int launch_ssm_chunks(const sk_ssm_params& p, cudaStream_t st) {
    int ns;
    const size_t smem = chunks_smem(p.N, &ns);
    const int blocks = chunk_blocks(p);
    float* dt = (float*)p.workspace;
    float* cum = dt + (size_t)p.B * p.H * blocks * SC_TOK;
    ssm_decay_kernel<<<dim3((unsigned)blocks, (unsigned)((p.H + 31) / 32), (unsigned)p.B), 256, 0, st>>>(p, blocks, dt, cum);
    if (int rc = check_launch("ssm_decay_kernel")) return rc;
    auto kern = p.N <= 128 ? ssm_chunks_kernel<1> : ssm_chunks_kernel<2>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "ssm_chunks_kernel smem attribute: %s", cudaGetErrorString(e));
    kern<<<dim3((unsigned)((p.P + SC_P - 1) / SC_P), (unsigned)p.H, (unsigned)p.B), SC_THR, smem, st>>>(p, ns, blocks, dt, cum);
    return check_launch("ssm_chunks_kernel");
}

}  // namespace sk
