// Matrix memory over a prompt portion on the 5th-generation tensor cores (bf16), in chunks of 128 tokens.  With the
// per-token quantities of a chunk (f, i the log gates in log2 units, b_t the running sum of f, a_s = i_s - b_s,
// A_t = max_{s <= t} a_s) and the stabiliser m_in the chunk starts with, M_t = max(m_in, A_t):
//   num_t = 2^(m_in - M_t) q_t^T S_in + sum_{s <= t} 2^(a_s - M_t) (q_t . k_s) v_s         (n likewise, with v = 1)
//   S_out = 2^(m_in - M_end) S_in + sum_s 2^(a_s - M_end) k_s v_s^T,    m_out = b_end + M_end
// 1. gates: a, A, b of every chunk;  2. sums: sum_s 2^(a_s - A_end) k_s;  3. carry: m_in and n_in of every chunk, in order.
// 4. states: a CTA owns 128 x 64 elements of one head's S in tensor memory and walks the chunks in order; K comes by
//    TMA, the weighted values are made by four warps, and the state a chunk starts with goes to memory by TMA.
// 5. outputs: every (chunk, head, 128 value columns) by itself: scores Q K^T, weights back into tensor memory,
//    Q S_in beside them, weights times V, and the two parts joined in fp32.
// Whatever carries a gate or the state enters a product as two bf16 numbers, value and remainder (16 significant
// bits); sums are fp32 and the state never leaves fp32 on its way through the chunks.
// Every wait is bounded; one that runs out makes all roles leave, and is reported in the status word.
#include "blocks.cuh"
#include "tcgen05.cuh"
#include "tensor_map.cuh"
#include "warp_mma.cuh"

namespace sk {
namespace {

constexpr int MT_TOK = 128;                                   // tokens of a chunk
constexpr uint32_t MT_PANEL = MT_TOK * 128;                   // 128 rows x 64 bf16
constexpr float MT_LOG2E = 1.4426950408889634f;

struct MtShape {
    const __nv_bfloat16 *k, *v;
    __nv_bfloat16* num;
    float *S_state, *n_state, *m_next, *den;
    const float *m_state, *gates, *i_bias, *f_bias;
    float *a, *top, *sum;             // [B, H, chunks, 128]
    float *u, *n_in;                  // [B, H, chunks, N]
    float* m_in;                      // [B, H, chunks], log2 units
    int32_t* status;
    int64_t in_ld, gates_ld, start;
    int B, S, H, N, P, chunks;
    float cap, q_scale;
};

// ---------------------------------------------------------------- per-token quantities
// A CTA: 128 tokens of 16 heads; a lane owns four consecutive tokens of a head.
constexpr int MT_GATE_HEADS = 16;
__global__ void __launch_bounds__(256)
mlstm_tc_gates_kernel(const __grid_constant__ MtShape p) {
    __shared__ float in_s[MT_GATE_HEADS][MT_TOK + 4], fo_s[MT_GATE_HEADS][MT_TOK + 4];
    const int c = blockIdx.x, h0 = blockIdx.y * MT_GATE_HEADS, b = blockIdx.z, t = threadIdx.x, lane = t & 31, warp = t >> 5;
    for (int e = t; e < MT_TOK * MT_GATE_HEADS; e += 256) {
        const int s = e / MT_GATE_HEADS, k = e % MT_GATE_HEADS, h = h0 + k, tok = c * MT_TOK + s;
        float gi = -INFINITY, gf = 0.f;                       // past the portion's end: nothing enters, nothing fades
        if (h < p.H && tok < p.S) {
            const float* g = p.gates + ((int64_t)b * p.S + tok) * p.gates_ld;
            gi = soft_cap_f32(g[h] + p.i_bias[h], p.cap) * MT_LOG2E;
            gf = log_sigmoid_f32(soft_cap_f32(g[p.H + h] + p.f_bias[h], p.cap)) * MT_LOG2E;
        }
        in_s[k][s] = gi;
        fo_s[k][s] = gf;
    }
    __syncthreads();
    for (int k = warp; k < MT_GATE_HEADS && h0 + k < p.H; k += 8) {
        float f[4], a[4], top[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) f[e] = fo_s[k][4 * lane + e];
        float acc = (f[0] + f[1]) + (f[2] + f[3]);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(FULL, acc, o);
            if (lane >= o) acc += x;
        }
        float run = __shfl_up_sync(FULL, acc, 1), mx = -INFINITY;
        if (lane == 0) run = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            run += f[e];
            f[e] = run;
            a[e] = in_s[k][4 * lane + e] - run;
            mx = fmaxf(mx, a[e]);
            top[e] = mx;
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(FULL, mx, o);
            if (lane >= o) mx = fmaxf(mx, x);
        }
        const float before = __shfl_up_sync(FULL, mx, 1);
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (lane > 0) top[e] = fmaxf(top[e], before);
        const int64_t at = (((int64_t)b * p.H + h0 + k) * p.chunks + c) * MT_TOK + 4 * lane;
        store_vec<float, 4>(p.a + at, a);
        store_vec<float, 4>(p.top + at, top);
        store_vec<float, 4>(p.sum + at, f);
    }
}

// u[n] = sum_s 2^(a_s - A_end) k_s[n] of a chunk; 8 columns per thread, the tokens dealt to 256 / (N / 8) groups
__global__ void __launch_bounds__(256)
mlstm_tc_sums_kernel(const __grid_constant__ MtShape p) {
    __shared__ float w[MT_TOK];
    __shared__ float part[256][9];
    const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, t = threadIdx.x;
    const int64_t hc = ((int64_t)b * p.H + h) * p.chunks + c;
    if (t < MT_TOK) w[t] = exp2f(p.a[hc * MT_TOK + t] - p.top[hc * MT_TOK + MT_TOK - 1]);
    __syncthreads();
    const int cols = p.N / 8, groups = 256 / cols, g = t / cols, col = t - g * cols;
    const int n_tok = p.S - c * MT_TOK < MT_TOK ? p.S - c * MT_TOK : MT_TOK;
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (g < groups) {
        const __nv_bfloat16* k = p.k + ((int64_t)b * p.S + c * MT_TOK) * p.in_ld + (int64_t)h * p.N + col * 8;
#pragma unroll 4
        for (int s = g; s < n_tok; s += groups) {
            float x[8];
            load_vec<__nv_bfloat16, 8>(k + s * p.in_ld, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[e] = fmaf(w[s], x[e], acc[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) part[t][e] = acc[e];
    __syncthreads();
    for (int n = t; n < p.N; n += 256) {
        float v = 0.f;
        for (int q = 0; q < groups; ++q) v += part[q * cols + (n >> 3)][n & 7];
        p.u[hc * p.N + n] = v;
    }
}

// m_in and n_in of every chunk, and what the portion leaves; a CTA per head, a thread per key column
__global__ void __launch_bounds__(256)
mlstm_tc_carry_kernel(const __grid_constant__ MtShape p) {
    const int h = blockIdx.x, b = blockIdx.y, t = threadIdx.x;
    const int64_t head = (int64_t)b * p.H + h;
    const bool fresh = p.start == 0, live = t < p.N;
    float m = fresh ? 0.f : p.m_state[head] * MT_LOG2E, n = fresh || !live ? 0.f : p.n_state[head * p.N + t];
    constexpr int U = 8;
    for (int c0 = 0; c0 < p.chunks; c0 += U) {
        float u[U], top[U], sum[U];
#pragma unroll
        for (int e = 0; e < U; ++e) {                         // all loads of a round in flight together
            const int64_t hc = head * p.chunks + (c0 + e < p.chunks ? c0 + e : p.chunks - 1);
            u[e] = live ? p.u[hc * p.N + t] : 0.f;
            top[e] = p.top[hc * MT_TOK + MT_TOK - 1];
            sum[e] = p.sum[hc * MT_TOK + MT_TOK - 1];
        }
#pragma unroll
        for (int e = 0; e < U; ++e) {
            if (c0 + e < p.chunks) {
                const int64_t hc = head * p.chunks + c0 + e;
                if (t == 0) p.m_in[hc] = m;
                if (live) p.n_in[hc * p.N + t] = n;
                const float mm = fmaxf(m, top[e]);
                n = exp2f(m - mm) * n + exp2f(top[e] - mm) * u[e];
                m = sum[e] + mm;
            }
        }
    }
    if (live) p.n_state[head * p.N + t] = n;
    if (t == 0) p.m_next[head] = m * (1.f / MT_LOG2E);
}

// ---------------------------------------------------------------- states
constexpr int ST_P = 64;                                      // value columns of a CTA; 128 key columns
constexpr int ST_THREADS = 288;                               // warps 0-3: tensor memory; 4-7: weighted values; 8: TMA and MMA
constexpr int ST_KSTAGES = 4;                                 // chunks of K in flight
constexpr uint32_t ST_SMEM = (ST_KSTAGES + 2 + 1) * 2 * MT_PANEL + 1024;   // K; two stages of weighted V; the outgoing state

struct StShared {
    uint64_t k_full[ST_KSTAGES], v_full[2], v_empty[2], s_ready, mma_done, drained;
    uint32_t tmem_base;
    int failed;
};

__device__ __forceinline__ void split8(const float (&x)[8], uint4& hi, uint4& lo) {
    split_bf16(x[0], x[1], hi.x, lo.x);
    split_bf16(x[2], x[3], hi.y, lo.y);
    split_bf16(x[4], x[5], hi.z, lo.z);
    split_bf16(x[6], x[7], hi.w, lo.w);
}

// barrier 1 of 128 threads, and whether `ok` held for all of them
__device__ __forceinline__ bool all_of_128(bool ok) {
    uint32_t r;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.u32 p, %1, 0;\n\t"
        "bar.red.and.pred q, 1, 128, p;\n\t"
        "selp.u32 %0, 1, 0, q;\n\t}"
        : "=r"(r)
        : "r"(ok ? 1u : 0u)
        : "memory");
    return r != 0;
}

__global__ void __launch_bounds__(ST_THREADS, 1)
mlstm_tc_states_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_s,
                       const __grid_constant__ MtShape p) {
    extern __shared__ char st_raw[];
    __shared__ StShared sh;
    char* k_s = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(st_raw) + 1023) & ~(uintptr_t)1023);   // [stage][panel]
    char* v_s = k_s + ST_KSTAGES * 2 * MT_PANEL;              // [stage][value, remainder]
    char* o_s = v_s + 2 * 2 * MT_PANEL;                       // [value, remainder]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int p0 = blockIdx.x * ST_P, n0 = blockIdx.y * 128, b = blockIdx.z / p.H, h = blockIdx.z - b * p.H;
    const int64_t head = (int64_t)b * p.H + h;
    volatile int* failed = &sh.failed;
    if (tid == 0) {
        for (int s = 0; s < ST_KSTAGES; ++s) mbar_init_count(&sh.k_full[s], 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init_count(&sh.v_full[s], 4);
            mbar_init_count(&sh.v_empty[s], 1);
        }
        mbar_init_count(&sh.s_ready, 4);
        mbar_init_count(&sh.mma_done, 1);
        mbar_init_count(&sh.drained, 1);
        sh.failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 8) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(&sh.tmem_base)), "r"(64u)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sh.tmem_base;
    const float* top_end = p.top + head * p.chunks * MT_TOK + MT_TOK - 1;      // A_end of chunk c: [c * 128]
    const float* m_in = p.m_in + head * p.chunks;

    if (warp < 4) {
        // ---- the state between two chunks: thread = key column
        const int r = warp * 32 + lane, n = n0 + r;
        const uint32_t row = tmem + ((uint32_t)(warp * 32) << 16);
        float* gst = p.S_state + (head * p.N + n) * p.P + p0;
        const int cols = n >= p.N ? 0 : (p.P - p0 < ST_P ? p.P - p0 : ST_P);
        float mi = m_in[0], tp = top_end[0];
        bool ok = true;
        for (int c = 0; c <= p.chunks; ++c) {
            float s[2][32];
            if (c > 0) ok = *failed == 0 && mbar_wait_bounded(&sh.mma_done, (uint32_t)((c - 1) & 1));
            // the copy before has left the buffer; and the four warps agree on whether to go on
            if (tid == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
            ok = all_of_128(ok);
            if (!ok) break;
            if (c == 0) {
#pragma unroll
                for (int j = 0; j < 64; ++j) s[j >> 5][j & 31] = p.start > 0 && j < cols ? gst[j] : 0.f;
            } else {
                tc_fence_after();
                tmem_ld32(row, reinterpret_cast<uint32_t(&)[32]>(s[0]));
                tmem_ld32(row + 32, reinterpret_cast<uint32_t(&)[32]>(s[1]));
            }
            if (c == p.chunks) {                              // what the portion leaves
#pragma unroll
                for (int j = 0; j < 64; j += 8)
                    if (j < cols) {                           // P is a multiple of 8
                        *reinterpret_cast<float4*>(gst + j) = make_float4(s[j >> 5][j & 31], s[j >> 5][(j & 31) + 1], s[j >> 5][(j & 31) + 2], s[j >> 5][(j & 31) + 3]);
                        *reinterpret_cast<float4*>(gst + j + 4) = make_float4(s[j >> 5][(j & 31) + 4], s[j >> 5][(j & 31) + 5], s[j >> 5][(j & 31) + 6], s[j >> 5][(j & 31) + 7]);
                    }
                break;
            }
            const float f = exp2f(mi - fmaxf(mi, tp));
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t w[32];
#pragma unroll
                for (int j = 0; j < 32; ++j) w[j] = __float_as_uint(s[half][j] * f);
                tmem_st32(row + half * 32, w);
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sh.s_ready);
            if (c + 1 < p.chunks) {
                mi = m_in[c + 1];
                tp = top_end[(int64_t)(c + 1) * MT_TOK];
            }
            // the state the chunk starts with, to memory
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                float x[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = s[j >> 2][(j & 3) * 8 + e];
                uint4 hi, lo;
                split8(x, hi, lo);
                char* dst = o_s + r * 128 + ((j ^ (r & 7)) << 4);
                *reinterpret_cast<uint4*>(dst) = hi;
                *reinterpret_cast<uint4*>(dst + MT_PANEL) = lo;
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (tid == 0) {
                const int hc = (int)(head * p.chunks + c);
#pragma unroll
                for (int part = 0; part < 2; ++part)
                    asm volatile("cp.async.bulk.tensor.4d.global.shared::cta.bulk_group [%0, {%1, %2, %3, %4}], [%5];" ::"l"(&map_s),
                                 "r"(p0), "r"(part), "r"(n0), "r"(hc), "r"(smem_addr(o_s + part * MT_PANEL))
                                 : "memory");
                asm volatile("cp.async.bulk.commit_group;" ::: "memory");
            }
        }
        if (!ok) *failed = 1;
        if (tid == 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
        tc_fence_before();
    } else if (warp < 8) {
        // ---- weighted values: eight lanes along a token's 64 columns, 16 tokens at a time
        const int vw = warp - 4, piece = lane & 7;
        const bool live_col = p0 + piece * 8 < p.P;
        const __nv_bfloat16* v = p.v + (int64_t)b * p.S * p.in_ld + (int64_t)h * p.P + p0 + piece * 8;
        const float* a = p.a + head * p.chunks * MT_TOK;
        // a chunk's values are requested two chunks ahead
        uint4 raw[2][8];
        float e[2][8], mi[2], tp[2];
        auto load = [&](int c, uint4 (&r)[8], float (&x)[8], float& m, float& t) {
#pragma unroll
            for (int it = 0; it < 8; ++it) {
                const int s = it * 16 + vw * 4 + (lane >> 3), tok = c * MT_TOK + s;
                r[it] = live_col && tok < p.S ? __ldg(reinterpret_cast<const uint4*>(v + (int64_t)tok * p.in_ld)) : make_uint4(0, 0, 0, 0);
                x[it] = a[(int64_t)c * MT_TOK + s];
            }
            m = m_in[c];
            t = top_end[(int64_t)c * MT_TOK];
        };
        load(0, raw[0], e[0], mi[0], tp[0]);
        if (p.chunks > 1) load(1, raw[1], e[1], mi[1], tp[1]);
        bool ok = true;
        for (int c2 = 0; ok && c2 < p.chunks; c2 += 2)
#pragma unroll
        for (int stage = 0; stage < 2; ++stage) {
            const int c = c2 + stage;
            if (c >= p.chunks) break;
            if (c >= 2 && (__any_sync(FULL, *failed != 0) ||
                           !__all_sync(FULL, mbar_wait_bounded(&sh.v_empty[stage], (uint32_t)(((c >> 1) - 1) & 1))))) {
                *failed = 1;
                ok = false;
                break;
            }
            const float mm = fmaxf(mi[stage], tp[stage]);
            char* dst = v_s + stage * 2 * MT_PANEL;
#pragma unroll
            for (int it = 0; it < 8; ++it) {
                const int s = it * 16 + vw * 4 + (lane >> 3);
                const float w = exp2_fast(e[stage][it] - mm);
                const uint32_t q[4] = {raw[stage][it].x, raw[stage][it].y, raw[stage][it].z, raw[stage][it].w};
                float x[8];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    x[2 * j] = __uint_as_float(q[j] << 16) * w;
                    x[2 * j + 1] = __uint_as_float(q[j] & 0xffff0000u) * w;
                }
                uint4 hi, lo;
                split8(x, hi, lo);
                char* d = dst + s * 128 + ((piece ^ (s & 7)) << 4);
                *reinterpret_cast<uint4*>(d) = hi;
                *reinterpret_cast<uint4*>(d + MT_PANEL) = lo;
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&sh.v_full[stage]);
            if (c + 2 < p.chunks) load(c + 2, raw[stage], e[stage], mi[stage], tp[stage]);
        }
    } else if (lane == 0) {
        // ---- K by TMA, MMAs: S += K^T (weighted V)
        auto fetch = [&](int c) {
            const int s = c % ST_KSTAGES;
            char* dst = k_s + s * 2 * MT_PANEL;
            mbar_expect(&sh.k_full[s], 2 * MT_PANEL);
            for (int q = 0; q < 2; ++q) tma_load_4d(dst + q * MT_PANEL, &map_k, n0 + q * 64, h, c * MT_TOK, b, &sh.k_full[s]);
        };
        const uint32_t idesc = umma_idesc_bf16(ST_P, true) | UMMA_A_MN;
        const uint32_t ka = smem_addr(k_s), va = smem_addr(v_s);
        int sent = 0;
        for (; sent < p.chunks && sent < ST_KSTAGES; ++sent) fetch(sent);
        bool ok = true;
        int c = 0;
        for (; c < p.chunks && !*failed; ++c) {
            const int stage = c & 1;
            ok = mbar_wait_bounded(&sh.s_ready, (uint32_t)(c & 1));           // which follows the MMAs of chunk c - 1
            if (!ok) break;
            if (c >= 1 && sent < p.chunks) fetch(sent++);                     // into the stage chunk c - 1 has left
            ok = mbar_wait_bounded(&sh.k_full[c % ST_KSTAGES], (uint32_t)((c / ST_KSTAGES) & 1)) &&
                 mbar_wait_bounded(&sh.v_full[stage], (uint32_t)((c >> 1) & 1));
            if (!ok) break;
            tc_fence_after();
            for (int part = 0; part < 2; ++part)
                for (int k = 0; k < MT_TOK / 16; ++k)
                    umma_ss(tmem, umma_desc_sw128_mn(ka + (c % ST_KSTAGES) * 2 * MT_PANEL + k * 2048, MT_PANEL),
                            umma_desc_sw128_mn(va + (stage * 2 + part) * MT_PANEL + k * 2048, MT_PANEL), idesc, 1);
            umma_commit(&sh.mma_done);
            umma_commit(&sh.v_empty[stage]);
        }
        if (!ok) *failed = 1;
        if (c < p.chunks)                                     // left early: no copy stays in flight
            for (int q = c; q < sent; ++q) mbar_wait_bounded(&sh.k_full[q % ST_KSTAGES], (uint32_t)((q / ST_KSTAGES) & 1));
        umma_commit(&sh.drained);
        mbar_wait_bounded(&sh.drained, 0);
    }
    __syncthreads();
    if (tid == 0 && sh.failed && p.status != nullptr) atomicOr(p.status, SK_DEV_WAIT_TIMEOUT);
    if (warp == 8)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(64u) : "memory");
}

// ---------------------------------------------------------------- outputs
constexpr int OT_P = 128;                                     // value columns of a CTA
constexpr int OT_THREADS = 192;                               // warps 0-3: token rows; 4: TMA; 5: MMA
constexpr int OT_STAGES = 4;
constexpr uint32_t OT_STAGE = 2 * MT_PANEL;                   // two K panels, 64 rows of the state, or V
constexpr uint32_t OT_S_PANEL = 64 * 128;                     // 64 key columns x 64 value columns of the state

struct OtShared {
    uint64_t q_full, full[OT_STAGES], empty[OT_STAGES], s_full, p_full, done, drained;
    uint32_t tmem_base;
    int failed;
    float a[MT_TOK], n[256];
};

__global__ void __launch_bounds__(OT_THREADS, 1)
mlstm_tc_out_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                    const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_s,
                    const __grid_constant__ MtShape p) {
    extern __shared__ char ot_raw[];
    __shared__ __align__(16) OtShared sh;
    const int np = (p.N + 63) / 64;
    char* q_s = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(ot_raw) + 1023) & ~(uintptr_t)1023);   // [panel]
    char* ring = q_s + np * MT_PANEL;                         // [stage]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int p0 = blockIdx.x * OT_P, c = blockIdx.y, b = blockIdx.z / p.H, h = blockIdx.z - b * p.H;
    const int64_t head = (int64_t)b * p.H + h, hc = head * p.chunks + c;
    const int k_items = (np + 1) / 2, items = k_items + np + 1;
    volatile int* failed = &sh.failed;
    if (tid == 0) {
        mbar_init_count(&sh.q_full, 1);
        for (int s = 0; s < OT_STAGES; ++s) {
            mbar_init_count(&sh.full[s], 1);
            mbar_init_count(&sh.empty[s], 1);
        }
        mbar_init_count(&sh.s_full, 1);
        mbar_init_count(&sh.p_full, 4);
        mbar_init_count(&sh.done, 1);
        mbar_init_count(&sh.drained, 1);
        sh.failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(&sh.tmem_base)), "r"(512u)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    if (tid < MT_TOK) sh.a[tid] = p.a[hc * MT_TOK + tid];
    for (int n = tid; n < 256; n += OT_THREADS) sh.n[n] = n < p.N ? p.n_in[hc * p.N + n] : 0.f;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sh.tmem_base;                       // columns: Q S | weights V | scores | weights, 128 each
    const uint32_t t_qs = tmem, t_wv = tmem + 128, t_sc = tmem + 256, t_w = tmem + 384;

    if (warp == 4) {
        if (lane == 0) {
            mbar_expect(&sh.q_full, np * MT_PANEL);
            for (int q = 0; q < np; ++q) tma_load_4d(q_s + q * MT_PANEL, &map_q, q * 64, h, c * MT_TOK, b, &sh.q_full);
            int i = 0;
            for (; i < items && !*failed; ++i) {
                const int s = i % OT_STAGES;
                char* dst = ring + s * OT_STAGE;
                if (i >= OT_STAGES && !mbar_wait_bounded(&sh.empty[s], (uint32_t)((i / OT_STAGES - 1) & 1))) {
                    *failed = 1;
                    break;
                }
                if (i < k_items) {
                    const int n = np - 2 * i < 2 ? 1 : 2;
                    mbar_expect(&sh.full[s], n * MT_PANEL);
                    for (int q = 0; q < n; ++q) tma_load_4d(dst + q * MT_PANEL, &map_k, (2 * i + q) * 64, h, c * MT_TOK, b, &sh.full[s]);
                } else if (i < items - 1) {
                    mbar_expect(&sh.full[s], 4 * OT_S_PANEL);
                    for (int q = 0; q < 4; ++q)
                        tma_load_4d(dst + q * OT_S_PANEL, &map_s, p0 + (q & 1) * 64, q >> 1, (i - k_items) * 64, (int)hc, &sh.full[s]);
                } else {
                    mbar_expect(&sh.full[s], 2 * MT_PANEL);
                    for (int q = 0; q < 2; ++q) tma_load_4d(dst + q * MT_PANEL, &map_v, p0 + q * 64, h, c * MT_TOK, b, &sh.full[s]);
                }
            }
            if (*failed) {                                    // leave no copy in flight
                mbar_wait_bounded(&sh.q_full, 0);
                for (int q = i > OT_STAGES ? i - OT_STAGES : 0; q < i; ++q)
                    mbar_wait_bounded(&sh.full[q % OT_STAGES], (uint32_t)((q / OT_STAGES) & 1));
            }
        }
    } else if (warp == 5) {
        if (lane == 0) {
            const uint32_t id_k = umma_idesc_bf16(MT_TOK, false), id_mn = umma_idesc_bf16(OT_P, true);
            const uint32_t qa = smem_addr(q_s), ra = smem_addr(ring);
            const int k16 = (p.N + 15) / 16;
            bool ok = mbar_wait_bounded(&sh.q_full, 0);
            int i = 0;
            for (; ok && i < items && !*failed; ++i) {
                const int s = i % OT_STAGES;
                if (i == items - 1) ok = mbar_wait_bounded(&sh.p_full, 0);
                ok = ok && mbar_wait_bounded(&sh.full[s], (uint32_t)((i / OT_STAGES) & 1));
                if (!ok) break;
                tc_fence_after();
                const uint32_t sa = ra + s * OT_STAGE;
                if (i < k_items) {                            // scores
                    for (int k = i * 8; k < k16 && k < i * 8 + 8; ++k) {
                        const uint32_t off = (uint32_t)(k >> 2) * MT_PANEL + (k & 3) * 32;
                        umma_ss(t_sc, umma_desc_sw128(qa + off), umma_desc_sw128(sa + off - i * 2 * MT_PANEL), id_k, k > 0);
                    }
                    if (i == k_items - 1) umma_commit(&sh.s_full);
                } else if (i < items - 1) {                   // Q S_in, value and remainder
                    const int j = i - k_items;
                    for (int part = 0; part < 2; ++part)
                        for (int k = j * 4; k < k16 && k < j * 4 + 4; ++k)
                            umma_ss(t_qs, umma_desc_sw128(qa + (uint32_t)j * MT_PANEL + (k & 3) * 32),
                                    umma_desc_sw128_mn(sa + part * 2 * OT_S_PANEL + (k & 3) * 2048, OT_S_PANEL), id_mn, k > 0 || part > 0);
                } else {                                      // weights V, value and remainder
                    for (int part = 0; part < 2; ++part)
                        for (int k = 0; k < MT_TOK / 16; ++k)
                            umma_ts(t_wv, t_w + part * 64 + k * 8, umma_desc_sw128_mn(sa + k * 2048, MT_PANEL), id_mn, k > 0 || part > 0);
                    umma_commit(&sh.done);
                }
                umma_commit(&sh.empty[s]);
            }
            if (!ok) *failed = 1;
            umma_commit(&sh.drained);                         // leave no MMA and no barrier arrival in flight
            mbar_wait_bounded(&sh.drained, 0);
        }
    } else {
        // ---- thread = token
        const int t = warp * 32 + lane;
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        const float m_in = p.m_in[hc], mt = fmaxf(m_in, p.top[hc * MT_TOK + t]), bt = p.sum[hc * MT_TOK + t];
        const float carry = exp2f(m_in - mt);
        bool ok = true;
        float qn = 0.f;
        if (blockIdx.x == 0) {                                // q . n_in, from the swizzled rows of Q
            ok = __all_sync(FULL, mbar_wait_bounded(&sh.q_full, 0));
            if (ok) {
                float s4[4] = {0.f, 0.f, 0.f, 0.f};
                for (int j = 0; j < np * 8; ++j) {
                    const uint4 raw = *reinterpret_cast<const uint4*>(q_s + (j >> 3) * MT_PANEL + t * 128 + (((j & 7) ^ (t & 7)) << 4));
                    const uint32_t x[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        s4[e] = fmaf(__uint_as_float(x[e] << 16), sh.n[j * 8 + 2 * e], s4[e]);
                        s4[e] = fmaf(__uint_as_float(x[e] & 0xffff0000u), sh.n[j * 8 + 2 * e + 1], s4[e]);
                    }
                }
                qn = (s4[0] + s4[1]) + (s4[2] + s4[3]);
            }
        }
        ok = ok && __all_sync(FULL, mbar_wait_bounded(&sh.s_full, 0));
        float row_sum = 0.f;
        if (ok) {
            tc_fence_after();
#pragma unroll
            for (int c0 = 0; c0 < MT_TOK; c0 += 32) {
                float s[32];
                uint32_t hi[16], lo[16];
                tmem_ld32(t_sc + lane_base + c0, reinterpret_cast<uint32_t(&)[32]>(s));
#pragma unroll
                for (int e = 0; e < 32; e += 4) {
                    const float4 a = *reinterpret_cast<const float4*>(&sh.a[c0 + e]);
                    const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float w = c0 + e + j <= t ? exp2_fast(av[j] - mt) : 0.f;
                        s[e + j] *= w;
                        row_sum += s[e + j];
                    }
                }
#pragma unroll
                for (int e = 0; e < 16; ++e) split_bf16(s[2 * e], s[2 * e + 1], hi[e], lo[e]);
                tmem_st16(t_w + lane_base + c0 / 2, hi);
                tmem_st16(t_w + lane_base + 64 + c0 / 2, lo);
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sh.p_full);
            const int tok = c * MT_TOK + t;
            if (blockIdx.x == 0 && tok < p.S)
                p.den[((int64_t)b * p.S + tok) * p.H + h] =
                    fmaxf(fabsf(fmaf(carry, qn, row_sum) * p.q_scale), exp2f(-(bt + mt))) + 1e-6f;
            ok = __all_sync(FULL, mbar_wait_bounded(&sh.done, 0));
            if (ok) {
                tc_fence_after();
                __nv_bfloat16* o = p.num + (((int64_t)b * p.S + tok) * p.H + h) * p.P + p0;
                const int cols = tok < p.S ? p.P - p0 : 0;
                const float fq = carry * p.q_scale;
#pragma unroll
                for (int c0 = 0; c0 < OT_P; c0 += 32) {
                    float x[32], y[32];
                    tmem_ld32(t_qs + lane_base + c0, reinterpret_cast<uint32_t(&)[32]>(x));
                    tmem_ld32(t_wv + lane_base + c0, reinterpret_cast<uint32_t(&)[32]>(y));
#pragma unroll
                    for (int e = 0; e < 32; e += 8) {
                        if (c0 + e < cols) {
                            float r[8];
#pragma unroll
                            for (int j = 0; j < 8; ++j) r[j] = fmaf(fq, x[e + j], y[e + j] * p.q_scale);
                            store_vec<__nv_bfloat16, 8>(o + c0 + e, r);
                        }
                    }
                }
            }
        }
        if (!ok) *failed = 1;
        tc_fence_before();
    }
    __syncthreads();
    if (tid == 0 && sh.failed && p.status != nullptr) atomicOr(p.status, SK_DEV_WAIT_TIMEOUT);
    if (warp == 5)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
}

int mt_chunks(const sk_mlstm_params& p) { return (p.S + MT_TOK - 1) / MT_TOK; }

// floats: a, top, sum | u, n_in | m_in; then the states of all chunks as two bf16 each
size_t mt_floats(const sk_mlstm_params& p) {
    const size_t hc = (size_t)p.B * p.H * mt_chunks(p);
    return (hc * (3 * MT_TOK + 2 * p.N + 1) + 31) / 32 * 32;
}

}  // namespace

size_t mlstm_tc_workspace(const sk_mlstm_params& p) {
    return mt_floats(p) * sizeof(float) + (size_t)p.B * p.H * mt_chunks(p) * p.N * p.P * 4;
}

bool mlstm_tc_applicable(const sk_mlstm_params& p) {
    return p.dtype == SK_BF16 && p.pos == nullptr && p.N % 8 == 0 && p.N <= 256 && p.P % 8 == 0 &&
           (int64_t)p.B * p.H <= 65535 && mt_chunks(p) <= 65535 &&
           head_map_ok(p.q, p.N, p.N, p.in_ld, (int64_t)p.S * p.in_ld) && head_map_ok(p.k, p.N, p.N, p.in_ld, (int64_t)p.S * p.in_ld) &&
           head_map_ok(p.v, p.P, p.P, p.in_ld, (int64_t)p.S * p.in_ld) && (uintptr_t)p.num % 16 == 0 && (uintptr_t)p.S_state % 16 == 0 &&
           mlstm_tc_workspace(p) <= (size_t)8 << 30;
}

int launch_mlstm_tc(const sk_mlstm_params& p, cudaStream_t st) {
    MtShape m{};
    const int chunks = mt_chunks(p);
    const size_t hc = (size_t)p.B * p.H * chunks;
    m.k = (const __nv_bfloat16*)p.k;
    m.v = (const __nv_bfloat16*)p.v;
    m.num = (__nv_bfloat16*)p.num;
    m.S_state = p.S_state;
    m.n_state = p.n_state;
    m.m_state = p.m_state;
    m.m_next = p.m_next;
    m.den = p.den;
    m.gates = p.gates;
    m.i_bias = p.i_bias;
    m.f_bias = p.f_bias;
    m.a = (float*)p.workspace;
    m.top = m.a + hc * MT_TOK;
    m.sum = m.top + hc * MT_TOK;
    m.u = m.sum + hc * MT_TOK;
    m.n_in = m.u + hc * p.N;
    m.m_in = m.n_in + hc * p.N;
    void* states = (float*)p.workspace + mt_floats(p);        // [B H chunks][value, remainder][N][P]
    m.status = p.status;
    m.in_ld = p.in_ld;
    m.gates_ld = p.gates_ld;
    m.start = p.start;
    m.B = p.B;
    m.S = p.S;
    m.H = p.H;
    m.N = p.N;
    m.P = p.P;
    m.chunks = chunks;
    m.cap = p.cap;
    m.q_scale = p.q_scale;
    const int64_t bs = (int64_t)p.S * p.in_ld, np = (int64_t)p.N * p.P;
    CUtensorMap mq, mk, mv, ms_out, ms_in;
    if (int rc = make_head_map(&mq, p.q, p.N, p.H, p.S, p.B, p.N, p.in_ld, bs, MT_TOK)) return rc;
    if (int rc = make_head_map(&mk, p.k, p.N, p.H, p.S, p.B, p.N, p.in_ld, bs, MT_TOK)) return rc;
    if (int rc = make_head_map(&mv, p.v, p.P, p.H, p.S, p.B, p.P, p.in_ld, bs, MT_TOK)) return rc;
    if (int rc = make_head_map(&ms_out, states, p.P, 2, p.N, (int)hc, np, p.P, 2 * np, MT_TOK)) return rc;
    if (int rc = make_head_map(&ms_in, states, p.P, 2, p.N, (int)hc, np, p.P, 2 * np, 64)) return rc;

    mlstm_tc_gates_kernel<<<dim3((unsigned)chunks, (unsigned)((p.H + MT_GATE_HEADS - 1) / MT_GATE_HEADS), (unsigned)p.B), 256, 0, st>>>(m);
    if (int rc = check_launch("mlstm_tc_gates_kernel")) return rc;
    mlstm_tc_sums_kernel<<<dim3((unsigned)chunks, (unsigned)p.H, (unsigned)p.B), 256, 0, st>>>(m);
    if (int rc = check_launch("mlstm_tc_sums_kernel")) return rc;
    mlstm_tc_carry_kernel<<<dim3((unsigned)p.H, (unsigned)p.B), 256, 0, st>>>(m);
    if (int rc = check_launch("mlstm_tc_carry_kernel")) return rc;
    cudaError_t e = cudaFuncSetAttribute(mlstm_tc_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ST_SMEM);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "mlstm_tc_states_kernel smem attribute: %s", cudaGetErrorString(e));
    mlstm_tc_states_kernel<<<dim3((unsigned)((p.P + ST_P - 1) / ST_P), (unsigned)((p.N + 127) / 128), (unsigned)(p.B * p.H)), ST_THREADS,
                             ST_SMEM, st>>>(mk, ms_out, m);
    if (int rc = check_launch("mlstm_tc_states_kernel")) return rc;
    const uint32_t smem = (uint32_t)((p.N + 63) / 64) * MT_PANEL + OT_STAGES * OT_STAGE + 1024;
    e = cudaFuncSetAttribute(mlstm_tc_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "mlstm_tc_out_kernel smem attribute: %s", cudaGetErrorString(e));
    mlstm_tc_out_kernel<<<dim3((unsigned)((p.P + OT_P - 1) / OT_P), (unsigned)chunks, (unsigned)(p.B * p.H)), OT_THREADS, smem, st>>>(
        mq, mk, mv, ms_in, m);
    return check_launch("mlstm_tc_out_kernel");
}

}  // namespace sk
