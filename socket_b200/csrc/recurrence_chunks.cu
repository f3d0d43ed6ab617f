// Linear recurrences with a scalar decay per head and token, over a prompt portion, as matrix products per block of
// 64 tokens (bf16 inputs): the state-space mixer and the matrix memory.  In both, with weights W that depend on the
// head's gates only,
//   y_t   = W_in(t) q_t^T S_in + sum_{s <= t} (q_t . k_s) W(t, s) v_s        S_out = W_in(end) S_in + sum_s W(end, s) k_s v_s^T
// State space (k = B, q = C, v = x; cum_t the running sum of the log decays inside a block):
//   W(t, s) = exp(cum_t - cum_s) dt_s,  W_in(t) = exp(cum_t),  and D x_t is added to y_t.
// Matrix memory (f, i the log gates, b_t the running sum of f, a_s = i_s - b_s, A_t = max_{s <= t} a_s, M_t = max(m_in, A_t),
// so that the stabiliser is m_t = b_t + M_t):
//   W(t, s) = exp(a_s - M_t),  W_in(t) = exp(m_in - M_t);  m_in of the next block is b_end + M_end.
// Its normaliser is one more value column whose value is 1; that column's results become the denominators.
// A first kernel computes the per-token quantities (base-2 logarithms) of all blocks.  Then a CTA owns
// 32 value columns of one head and walks the blocks in order, two CTAs per SM; the state stays in fp32
// accumulator registers.  q, k and v are bf16 as they come, products accumulate in fp32,
// and every factor that carries a decay, a gate, a step size or the state enters a product as two bf16 numbers
// (value and remainder, 16 significant bits together), so that nothing of the recurrence is rounded to
// 8 bits.
#include "blocks.cuh"
#include "warp_mma.cuh"

namespace sk {
namespace {

constexpr int SC_TOK = 64, SC_P = 32, SC_THR = 256;
constexpr int SC_PS = SC_P + 8;              // shared-memory row of 32 columns
constexpr float SC_LOG2E = 1.4426950408889634f;

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

// a[b][h][t] = i - b_t, top[b][h][t] = running maximum of a, sum[b][h][t] = b_t inside t's block, all in log2 units;
// tokens past the portion's end add nothing (a = -inf) and leave the sum as it is.  A CTA: 64 tokens of 32 heads.
__global__ void __launch_bounds__(256)
mlstm_gates_kernel(sk_mlstm_params p, int blocks, float* __restrict__ a, float* __restrict__ top, float* __restrict__ sum) {
    __shared__ float in_s[32][SC_TOK + 1], fo_s[32][SC_TOK + 1];
    const int blk = blockIdx.x, h0 = blockIdx.y * 32, b = blockIdx.z, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    const int h = h0 + lane;
    const float ib = h < p.H ? p.i_bias[h] : 0.f, fb = h < p.H ? p.f_bias[h] : 0.f;
    for (int s = warp; s < SC_TOK; s += 8) {
        const int tok = blk * SC_TOK + s;
        float gi = -INFINITY, gf = 0.f;
        if (h < p.H && tok < p.S) {
            const float* g = p.gates + ((int64_t)b * p.S + tok) * p.gates_ld;
            gi = soft_cap_f32(g[h] + ib, p.cap) * SC_LOG2E;
            gf = log_sigmoid_f32(soft_cap_f32(g[p.H + h] + fb, p.cap)) * SC_LOG2E;
        }
        in_s[lane][s] = gi;
        fo_s[lane][s] = gf;
    }
    __syncthreads();
    for (int k = warp; k < 32 && h0 + k < p.H; k += 8) {
        const float f1 = fo_s[k][2 * lane + 1];
        float acc = fo_s[k][2 * lane] + f1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(FULL, acc, o);
            if (lane >= o) acc += x;
        }
        const float b0 = acc - f1, a0 = in_s[k][2 * lane] - b0, a1 = in_s[k][2 * lane + 1] - acc;
        float mx = fmaxf(a0, a1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(FULL, mx, o);
            if (lane >= o) mx = fmaxf(mx, x);
        }
        const float before = __shfl_up_sync(FULL, mx, 1);
        const int64_t at = (((int64_t)b * p.H + h0 + k) * blocks + blk) * SC_TOK + 2 * lane;
        *reinterpret_cast<float2*>(a + at) = make_float2(a0, a1);
        *reinterpret_cast<float2*>(top + at) = make_float2(lane > 0 ? fmaxf(before, a0) : a0, mx);
        *reinterpret_cast<float2*>(sum + at) = make_float2(b0, acc);
    }
}

struct RecurrenceParams {
    const __nv_bfloat16 *q, *k, *v;          // token 0: q and k [H / rep, N], v [H, P]
    __nv_bfloat16* y;                        // [B S, H P]
    float *state, *n_state, *den, *m_next;   // n_state, den, m_state, m_next: matrix memory only
    const float *m_state, *skip;
    const float *e0, *e1, *e2;               // [B, H, blocks, 64]: running decay, step size | a, its running maximum, b
    const int64_t* pos;
    int64_t ld, start;                       // elements between tokens in q, k and v
    int S, H, P, N, rep, ns, blocks;
    float q_scale;
};

// NM: 16-row tiles of the state per warp (8 warps x 16 NM >= N).  MEMORY: the matrix memory, else the state space
template <int NM, bool MEMORY>
__global__ void __launch_bounds__(SC_THR, NM == 1 ? 2 : 1)
recurrence_chunks_kernel(const __grid_constant__ RecurrenceParams p) {
    extern __shared__ __align__(16) char sc_raw[];
    constexpr int NE = MEMORY ? 3 : 2;
    __shared__ __align__(16) float e_sh[NE][2][SC_TOK];
    __shared__ float w_sh[SC_TOK];
    const int ns = p.ns, blocks = p.blocks;
    using bf = __nv_bfloat16;
    const int n16 = (p.N + 15) / 16 * 16;
    bf* b_s = reinterpret_cast<bf*>(sc_raw);                  // [2][64][ns]
    bf* c_s = b_s + 2 * SC_TOK * ns;                          // [2][64][ns]
    bf* x_s = c_s + 2 * SC_TOK * ns;                          // [2][64][40]
    bf* st_s = x_s + 2 * SC_TOK * SC_PS;                      // [hi, lo][n16][40]
    float4* ex_s = reinterpret_cast<float4*>(st_s + 2 * n16 * SC_PS);   // [warp][2][lane]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, fr = lane >> 2, fc = (lane & 3) * 2;
    const int p0 = blockIdx.x * SC_P, h = blockIdx.y, b = blockIdx.z;
    const int g = h / p.rep, I = p.H * p.P;
    const int pc = p.P - p0 < SC_P ? p.P - p0 : SC_P;         // value columns of this CTA; the normaliser, if it has it, is column pc
    const bool fresh = first_position(p.pos, p.start) == 0;
    const int64_t head = (int64_t)b * p.H + h;
    const float skip = MEMORY ? 0.f : p.skip[h];
    float m_in = MEMORY && !fresh ? p.m_state[head] * SC_LOG2E : 0.f;
    const bf* q_rows = p.q + (int64_t)b * p.S * p.ld + (int64_t)g * p.N;
    const bf* k_rows = p.k + (int64_t)b * p.S * p.ld + (int64_t)g * p.N;
    const bf* v_rows = p.v + (int64_t)b * p.S * p.ld + (int64_t)h * p.P + p0;
    const int nc = p.N / 8, xc = pc / 8;
    const int64_t e_at = head * blocks * SC_TOK;
    const float* e_h[3] = {p.e0 + e_at, p.e1 + e_at, MEMORY ? p.e2 + e_at : nullptr};

    auto fetch = [&](int blk, int stage) {
        const int t0 = blk * SC_TOK;
        for (int r = warp; r < SC_TOK; r += SC_THR / 32) {    // a warp per token, lanes along its row
            const bool live = t0 + r < p.S;
            const int64_t off = (int64_t)(live ? t0 + r : p.S - 1) * p.ld;
            const bf* bsrc = k_rows + off;
            const bf* csrc = q_rows + off;
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
                     v_rows + (int64_t)(live ? t0 + r : p.S - 1) * p.ld + (tid & 3) * 8, live);
        }
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int piece = tid - e * (SC_TOK / 4);
            if (piece >= 0 && piece < SC_TOK / 4) cp16(saddr(&e_sh[e][stage][piece * 4]), e_h[e] + t0 + piece * 4, true);
        }
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
        x_s[r * SC_PS + pc + (e - r * w)] = __float2bfloat16_rn(MEMORY && e == r * w && pc < SC_P ? 1.f : 0.f);
    }

    // state rows of this warp: tiles warp, warp + 8 of 16 rows each
    float st[NM][4][4];
    float* gst = p.state + head * p.N * p.P + p0;
    auto state_at = [&](int n, int c) -> float* {             // element (n, c) of this CTA's columns, or none
        if (n < p.N && c < pc) return gst + (int64_t)n * p.P + c;
        return MEMORY && n < p.N && c == pc && pc < SC_P ? p.n_state + head * p.N + n : nullptr;
    };
#pragma unroll
    for (int u = 0; u < NM; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float* at = state_at((warp + 8 * u) * 16 + fr + 8 * (e >> 1), v * 8 + fc + (e & 1));
                st[u][v][e] = !fresh && at != nullptr ? *at : 0.f;
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
        const float* e0 = e_sh[0][stage];
        const float* e1 = e_sh[1][stage];
        // exponent of a token's row factor, without the state's; of the last token: the state's own
        auto row_exp = [&](int t) { return MEMORY ? -fmaxf(m_in, e1[t]) : e0[t]; };
        auto weight = [&](float row, float c, float d) { return MEMORY ? exp2f(c + row) : exp2f(row - c) * d; };
        const float total = row_exp(SC_TOK - 1);
        if (tid < SC_TOK) w_sh[tid] = weight(total, e0[tid], e1[tid]);
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
        const float row_r[2] = {row_exp(tr[0]), row_exp(tr[1])};
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float f = exp2f(MEMORY ? row_r[k] + m_in : row_r[k]);
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
                    const float c0 = e0[s], c1 = e0[s + 1], d0 = MEMORY ? 1.f : e1[s], d1 = MEMORY ? 1.f : e1[s + 1];
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const float w0 = s <= tr[r] ? gacc[2 * k + v][2 * r] * weight(row_r[r], c0, d0) : 0.f;
                        const float w1 = s + 1 <= tr[r] ? gacc[2 * k + v][2 * r + 1] * weight(row_r[r], c1, d1) : 0.f;
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
                        *reinterpret_cast<__nv_bfloat162*>(p.y + ((int64_t)b * p.S + t0 + tr[k]) * I + h * p.P + p0 + c) =
                            MEMORY ? __floats2bfloat162_rn(y[v][2 * k] * p.q_scale, y[v][2 * k + 1] * p.q_scale)
                                   : __floats2bfloat162_rn(fmaf(skip, __low2float(x), y[v][2 * k]),
                                                           fmaf(skip, __high2float(x), y[v][2 * k + 1]));
                    } else if (MEMORY && c == pc) {           // n . q; m_t = b_t + M_t
                        const float m = e_sh[NE - 1][stage][tr[k]] - row_r[k];
                        p.den[((int64_t)b * p.S + t0 + tr[k]) * p.H + h] =
                            fmaxf(fabsf(y[v][2 * k] * p.q_scale), exp2f(-m)) + 1e-6f;
                    }
                }
            }
        }
        // ---- state: (weighted B)^T . x on top of the decayed state
        const float f = exp2f(MEMORY ? total + m_in : total);
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
        publish_state();                                      // q . S of this block was read before the last barrier
        if (MEMORY) m_in = e_sh[NE - 1][stage][SC_TOK - 1] - total;
    }
#pragma unroll
    for (int u = 0; u < NM; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float* at = state_at((warp + 8 * u) * 16 + fr + 8 * (e >> 1), v * 8 + fc + (e & 1));
                if (at != nullptr) *at = st[u][v][e];
            }
    if (MEMORY && pc < SC_P && tid == 0) p.m_next[head] = m_in * (1.f / SC_LOG2E);
}

size_t chunks_smem(int N, int* ns) {
    const int n16 = (N + 15) / 16 * 16;
    *ns = n16 + 8;
    return ((size_t)4 * SC_TOK * *ns + 2 * SC_TOK * SC_PS + (size_t)2 * n16 * SC_PS) * 2 + (size_t)(SC_THR / 32) * 2 * 32 * 16;
}

int chunk_blocks(int S) { return (S + SC_TOK - 1) / SC_TOK; }

template <bool MEMORY> int launch_blocks(RecurrenceParams& r, int B, cudaStream_t st) {
    const size_t smem = chunks_smem(r.N, &r.ns);
    auto kern = r.N <= 128 ? recurrence_chunks_kernel<1, MEMORY> : recurrence_chunks_kernel<2, MEMORY>;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "recurrence_chunks_kernel smem attribute: %s", cudaGetErrorString(e));
    const int cols = r.P + (MEMORY ? 1 : 0);
    kern<<<dim3((unsigned)((cols + SC_P - 1) / SC_P), (unsigned)r.H, (unsigned)B), SC_THR, smem, st>>>(r);
    return check_launch("recurrence_chunks_kernel");
}

}  // namespace

// ---------------------------------------------------------------- state space
bool ssm_chunks_applicable(const sk_ssm_params& p) {
    return p.dtype == SK_BF16 && p.pos == nullptr && p.N % 8 == 0 && p.N <= 256 && p.P % 8 == 0 && p.xbc_ld % 8 == 0 &&
           (uintptr_t)p.xbc % 16 == 0;
}

size_t ssm_chunks_workspace(const sk_ssm_params& p) {         // step sizes and running decays
    return (size_t)2 * p.B * p.H * chunk_blocks(p.S) * SC_TOK * sizeof(float);
}

int launch_ssm_chunks(const sk_ssm_params& p, cudaStream_t st) {
    const int blocks = chunk_blocks(p.S), I = p.H * p.P;
    float* dt = (float*)p.workspace;
    float* cum = dt + (size_t)p.B * p.H * blocks * SC_TOK;
    ssm_decay_kernel<<<dim3((unsigned)blocks, (unsigned)((p.H + 31) / 32), (unsigned)p.B), 256, 0, st>>>(p, blocks, dt, cum);
    if (int rc = check_launch("ssm_decay_kernel")) return rc;
    RecurrenceParams r{};
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.xbc;     // row: [x (H P) | B (G N) | C (G N)]
    r.v = x;
    r.k = x + I;
    r.q = r.k + p.G * p.N;
    r.ld = p.xbc_ld;
    r.y = (__nv_bfloat16*)p.y;
    r.state = p.state;
    r.skip = p.D;
    r.e0 = cum;
    r.e1 = dt;
    r.pos = p.pos;
    r.start = p.start;
    r.S = p.S;
    r.H = p.H;
    r.P = p.P;
    r.N = p.N;
    r.rep = p.H / p.G;
    r.blocks = blocks;
    return launch_blocks<false>(r, p.B, st);
}

// ---------------------------------------------------------------- matrix memory
bool mlstm_chunks_applicable(const sk_mlstm_params& p) {
    return p.dtype == SK_BF16 && p.pos == nullptr && p.N % 8 == 0 && p.N <= 256 && p.P % 8 == 0 && p.in_ld % 8 == 0 &&
           ((uintptr_t)p.q | (uintptr_t)p.k | (uintptr_t)p.v) % 16 == 0;
}

size_t mlstm_chunks_workspace(const sk_mlstm_params& p) {     // a, its running maximum, b
    return (size_t)3 * p.B * p.H * chunk_blocks(p.S) * SC_TOK * sizeof(float);
}

int launch_mlstm_chunks(const sk_mlstm_params& p, cudaStream_t st) {
    const int blocks = chunk_blocks(p.S);
    const size_t n = (size_t)p.B * p.H * blocks * SC_TOK;
    float *a = (float*)p.workspace, *top = a + n, *sum = top + n;
    mlstm_gates_kernel<<<dim3((unsigned)blocks, (unsigned)((p.H + 31) / 32), (unsigned)p.B), 256, 0, st>>>(p, blocks, a, top, sum);
    if (int rc = check_launch("mlstm_gates_kernel")) return rc;
    RecurrenceParams r{};
    r.q = (const __nv_bfloat16*)p.q;
    r.k = (const __nv_bfloat16*)p.k;
    r.v = (const __nv_bfloat16*)p.v;
    r.ld = p.in_ld;
    r.y = (__nv_bfloat16*)p.num;
    r.state = p.S_state;
    r.n_state = p.n_state;
    r.den = p.den;
    r.m_state = p.m_state;
    r.m_next = p.m_next;
    r.e0 = a;
    r.e1 = top;
    r.e2 = sum;
    r.pos = p.pos;
    r.start = p.start;
    r.S = p.S;
    r.H = p.H;
    r.P = p.P;
    r.N = p.N;
    r.rep = 1;
    r.blocks = blocks;
    r.q_scale = p.q_scale;
    return launch_blocks<true>(r, p.B, st);
}

}  // namespace sk
