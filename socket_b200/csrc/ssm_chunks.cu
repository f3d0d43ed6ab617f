// Selective state-space recurrence over a prompt portion as matrix products per block of 64 tokens (bf16
// inputs).  With cum_t the running sum of the log decays inside a block,
//   y_t = exp(cum_t) C_t^T S_in + sum_{s <= t} (C_t . B_s) exp(cum_t - cum_s) dt_s x_s + D x_t
//   S_out = exp(cum_end) S_in + sum_s B_s (exp(cum_end - cum_s) dt_s x_s)^T
// A CTA owns 32 value columns of one head and walks the blocks in order; the state stays in fp32
// accumulator registers.  B, C and x are bf16 as the convolution leaves them, products accumulate in fp32, and every factor
// that carries a decay, a step size or the state enters a product as two bf16 numbers (value and
// remainder, 16 significant bits together), so that nothing of the recurrence is rounded to 8 bits.
#include "blocks.cuh"
#include "warp_mma.cuh"

namespace sk {
namespace {

constexpr int SC_TOK = 64, SC_P = 32, SC_THR = 256;
constexpr int SC_PS = SC_P + 8;              // shared-memory row of 32 columns
constexpr int SC_MS = SC_TOK + 8;            // shared-memory row of 64 tokens

__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 r = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&r);
}

// NM: 16-row tiles of the state per warp (8 warps x 16 NM >= N)
template <int NM>
__global__ void __launch_bounds__(SC_THR)
ssm_chunks_kernel(sk_ssm_params p, int ns) {  // ns: shared-memory row of B and C, elements
    extern __shared__ __align__(16) char sc_raw[];
    __shared__ float cum_s[SC_TOK], dt_s[SC_TOK];
    using bf = __nv_bfloat16;
    const int n16 = (p.N + 15) / 16 * 16;
    bf* b_s = reinterpret_cast<bf*>(sc_raw);                  // [2][64][ns]
    bf* c_s = b_s + 2 * SC_TOK * ns;                          // [2][64][ns]
    bf* x_s = c_s + 2 * SC_TOK * ns;                          // [2][64][40]
    bf* st_s = x_s + 2 * SC_TOK * SC_PS;                      // [hi, lo][n16][40]
    bf* m_s = st_s + 2 * n16 * SC_PS;                         // [hi, lo][64][72]
    bf* w_s = m_s + 2 * SC_TOK * SC_MS;                       // [hi, lo][64][40]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, fr = lane >> 2, fc = (lane & 3) * 2;
    const int p0 = blockIdx.x * SC_P, h = blockIdx.y, b = blockIdx.z;
    const int g = h / (p.H / p.G), I = p.H * p.P, pc = p.P - p0 < SC_P ? p.P - p0 : SC_P;
    const bool fresh = first_position(p.pos, p.start) == 0;
    const float a_rate = -expf(p.A_log[h]), dt_bias = p.dt_bias[h], skip = p.D[h];
    const bf* rows = (const bf*)p.xbc + (int64_t)b * p.S * p.xbc_ld;
    const int nc = p.N / 8, xc = pc / 8, blocks = (p.S + SC_TOK - 1) / SC_TOK;

    auto fetch = [&](int blk, int stage) {
        const int t0 = blk * SC_TOK;
        for (int e = tid; e < SC_TOK * nc * 2; e += SC_THR) {
            const int which = e / (SC_TOK * nc), k = e - which * SC_TOK * nc, r = k / nc, c = k - r * nc;
            const bool live = t0 + r < p.S;
            const bf* src = rows + (int64_t)(live ? t0 + r : p.S - 1) * p.xbc_ld + I + (which * p.G + g) * p.N + c * 8;
            cp16(saddr((which ? c_s : b_s) + (stage * SC_TOK + r) * ns + c * 8), src, live);
        }
        for (int e = tid; e < SC_TOK * xc; e += SC_THR) {
            const int r = e / xc, c = e - r * xc;
            const bool live = t0 + r < p.S;
            cp16(saddr(x_s + (stage * SC_TOK + r) * SC_PS + c * 8),
                 rows + (int64_t)(live ? t0 + r : p.S - 1) * p.xbc_ld + h * p.P + p0 + c * 8, live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // columns that round N up to 16 and a narrow last slice up to 32 stay zero
    for (int e = tid; e < 4 * SC_TOK * (ns - p.N); e += SC_THR) {
        const int w = ns - p.N, r = e / w;
        b_s[(int64_t)r * ns + p.N + (e - r * w)] = __float2bfloat16_rn(0.f);   // b_s and c_s are one array of 256 rows
    }
    for (int e = tid; e < 2 * SC_TOK * (SC_PS - pc); e += SC_THR) {
        const int w = SC_PS - pc, r = e / w;
        x_s[r * SC_PS + pc + (e - r * w)] = __float2bfloat16_rn(0.f);
    }
    fetch(0, 0);

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
    const int mt = warp & 3, half = warp >> 2;                // 16-token tile, half of the keys / value columns

    for (int blk = 0; blk < blocks; ++blk) {
        const int stage = blk & 1, t0 = blk * SC_TOK;
        __syncthreads();
        if (blk + 1 < blocks) {
            fetch(blk + 1, stage ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        // ---- step sizes and running log decays (warp 0, two tokens per lane); the state as two bf16 parts
        if (warp == 0) {
            float d[2], a[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int t = t0 + 2 * lane + k;
                d[k] = t < p.S ? softplus_f32(to_f32(((const bf*)p.dt_in)[((int64_t)b * p.S + t) * p.in_ld + h]) + dt_bias) : 0.f;
                a[k] = a_rate * d[k];
            }
            float sum = a[0] + a[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(FULL, sum, o);
                if (lane >= o) sum += x;
            }
            dt_s[2 * lane] = d[0];
            dt_s[2 * lane + 1] = d[1];
            cum_s[2 * lane] = sum - a[1];
            cum_s[2 * lane + 1] = sum;
        }
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
        __syncthreads();
        const bf* bt = b_s + stage * SC_TOK * ns;
        const bf* ct = c_s + stage * SC_TOK * ns;
        const bf* xt = x_s + stage * SC_TOK * SC_PS;
        const float total = cum_s[SC_TOK - 1];
        // ---- inputs weighted for the state update
        for (int e = tid; e < SC_TOK * SC_P / 2; e += SC_THR) {
            const int r = e / (SC_P / 2), c = 2 * (e - r * (SC_P / 2));
            const float w = dt_s[r] * expf(total - cum_s[r]);
            const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xt + r * SC_PS + c);
            uint32_t hi, lo;
            split_bf16(__low2float(x) * w, __high2float(x) * w, hi, lo);
            *reinterpret_cast<uint32_t*>(w_s + r * SC_PS + c) = hi;
            *reinterpret_cast<uint32_t*>(w_s + (SC_TOK + r) * SC_PS + c) = lo;
        }
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
        const bool keys_seen = half == 0 || mt >= 2;          // keys 32.. are later than tokens 0..31
        const uint32_t ca = saddr(ct + (mt * 16 + (lane & 15)) * ns + (lane >> 4) * 8);
        const uint32_t ba = saddr(bt + (half * 32 + (lane & 7) + (lane >> 4) * 8) * ns + ((lane >> 3) & 1) * 8);
        const uint32_t sa = saddr(st_s + (lane & 15) * SC_PS + half * 16 + (lane >> 4) * 8);
        for (int k = 0; k < n16 / 16; ++k) {
            uint32_t a[4], bb[4];
            ldsm4(ca + k * 32, a);
            if (keys_seen) {
#pragma unroll
                for (int v = 0; v < 4; v += 2) {
                    ldsm4(ba + v * 8 * ns * 2 + k * 32, bb);
                    mma16816(gacc[v], a, bb[0], bb[1]);
                    mma16816(gacc[v + 1], a, bb[2], bb[3]);
                }
            }
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                ldsm4t(sa + (part * n16 + k * 16) * SC_PS * 2, bb);
                mma16816(y[0], a, bb[0], bb[1]);
                mma16816(y[1], a, bb[2], bb[3]);
            }
        }
        const int tr[2] = {mt * 16 + fr, mt * 16 + fr + 8};
        const float ct_r[2] = {cum_s[tr[0]], cum_s[tr[1]]};
        if (keys_seen) {
#pragma unroll
            for (int v = 0; v < 4; ++v) {
                const int s = half * 32 + v * 8 + fc;
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    float w[2];
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        w[e] = s + e <= tr[k] ? gacc[v][2 * k + e] * (expf(ct_r[k] - cum_s[s + e]) * dt_s[s + e]) : 0.f;
                    uint32_t hi, lo;
                    split_bf16(w[0], w[1], hi, lo);
                    *reinterpret_cast<uint32_t*>(m_s + tr[k] * SC_MS + s) = hi;
                    *reinterpret_cast<uint32_t*>(m_s + (SC_TOK + tr[k]) * SC_MS + s) = lo;
                }
            }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float f = expf(ct_r[k]);
#pragma unroll
            for (int v = 0; v < 2; ++v) {
                y[v][2 * k] *= f;
                y[v][2 * k + 1] *= f;
            }
        }
        __syncthreads();
        // ---- weights . x, then the outputs
        for (int k = 0; k <= mt; ++k) {
            uint32_t bb[4];
            ldsm4t(saddr(xt + (k * 16 + (lane & 15)) * SC_PS + half * 16 + (lane >> 4) * 8), bb);
#pragma unroll
            for (int part = 0; part < 2; ++part) {
                uint32_t a[4];
                ldsm4(saddr(m_s + (part * SC_TOK + mt * 16 + (lane & 15)) * SC_MS + k * 16 + (lane >> 4) * 8), a);
                mma16816(y[0], a, bb[0], bb[1]);
                mma16816(y[1], a, bb[2], bb[3]);
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
        // ---- state: B^T . weighted inputs on top of the decayed state
        const float f = expf(total);
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
                    uint32_t a[4];                            // B^T: rows n, columns tokens, stored token by token
                    ldsm4t(saddr(bt + (k * 16 + (lane & 7) + (lane >> 4) * 8) * ns + n0 + ((lane >> 3) & 1) * 8), a);
#pragma unroll
                    for (int part = 0; part < 2; ++part)
#pragma unroll
                        for (int v = 0; v < 4; v += 2) {
                            uint32_t bb[4];
                            ldsm4t(saddr(w_s + (part * SC_TOK + k * 16 + (lane & 15)) * SC_PS + v * 8 + (lane >> 4) * 8), bb);
                            mma16816(st[u][v], a, bb[0], bb[1]);
                            mma16816(st[u][v + 1], a, bb[2], bb[3]);
                        }
                }
            }
        }
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
    return ((size_t)4 * SC_TOK * *ns + 2 * SC_TOK * SC_PS + (size_t)2 * n16 * SC_PS + 2 * SC_TOK * SC_MS + 2 * SC_TOK * SC_PS) * 2;
}

}  // namespace

bool ssm_chunks_applicable(const sk_ssm_params& p) {
    return p.dtype == SK_BF16 && p.pos == nullptr && p.N % 8 == 0 && p.N <= 256 && p.P % 8 == 0 && p.xbc_ld % 8 == 0 &&
           (uintptr_t)p.xbc % 16 == 0;
}

size_t ssm_chunks_workspace(const sk_ssm_params&) { return 0; }

int launch_ssm_chunks(const sk_ssm_params& p, cudaStream_t st) {
    int ns;
    const size_t smem = chunks_smem(p.N, &ns);
    auto kern = p.N <= 128 ? ssm_chunks_kernel<1> : ssm_chunks_kernel<2>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "ssm_chunks_kernel smem attribute: %s", cudaGetErrorString(e));
    kern<<<dim3((unsigned)((p.P + SC_P - 1) / SC_P), (unsigned)p.H, (unsigned)p.B), SC_THR, smem, st>>>(p, ns);
    return check_launch("ssm_chunks_kernel");
}

}  // namespace sk
