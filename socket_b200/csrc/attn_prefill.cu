// Softmax attention of a prompt portion on the 5th-generation tensor cores (bf16).
//
// A CTA owns 256 consecutive queries of one head as two tiles of 128.  One warp feeds 128-key tiles of K
// and V by TMA (128-byte swizzle), one thread issues the MMAs: S = Q K^T into tensor memory (fp32,
// shared-memory operands), O += P V with P read from tensor memory.  Each query tile has four softmax warps, one
// thread per query row: they read the row's 128 scores, scale / bias / mask them, keep the running maximum and sum,
// and write the weights back over the scores as bf16.  While one tile is in its softmax the tensor
// core works on the other.  The accumulator is rescaled only when a row's maximum has grown by more than
// 2^8 since the last time (the final division by the sum makes the choice of reference invisible).  Scores under
// a cap are bounded, so weights are taken relative to zero: no maximum, no rescaling.
//
// Visibility is causal, optionally restricted to the query's own chunk of positions or to a sliding window; tiles
// that no row of a query tile can see are not visited.  Out-of-range rows and columns of a tile are zero-filled by TMA.
// Every wait is bounded; one that runs out makes all roles leave, and is reported in the status word.
#include "blocks.cuh"
#include "tcgen05.cuh"
#include "tensor_map.cuh"

namespace sk {
namespace {

constexpr int FP_TILE = 128;                                  // queries of a tile = keys of a tile
constexpr int FP_SOFTMAX_WARP0 = 4;                           // warps 4-7: tile 0, warps 8-11: tile 1
constexpr int FP_THREADS = 32 * (FP_SOFTMAX_WARP0 + 8);
constexpr uint32_t FP_PANEL = FP_TILE * 128;                  // 128 rows x 64 bf16
constexpr int FP_BIAS_SPAN = 160;                             // distances a warp's 32 rows x 128 keys can have
constexpr uint32_t FP_BIAS_BYTES = 8 * FP_BIAS_SPAN * sizeof(float);
constexpr uint32_t FP_SMEM_MAX = 232448 - 1024 - 512;         // opt-in limit minus alignment slack and static data
constexpr float FP_RESCALE = 8.f;                             // log2 units
constexpr float FP_LOG2E = 1.4426950408889634f;

struct FpShared {
    uint64_t q_full;
    uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
    uint64_t s_full[2], p_full[2], o_full[2];
    uint64_t drained;
    uint32_t tmem_base;
    int failed;
};

struct FpShape {            // what the kernel needs beside the tensor maps
    void* out;
    const float *bias, *sink;
    int32_t* status;
    int64_t o_bs, o_ss, o_hs, start, kv_start, bias_len;
    int S, H, G, dqk, dv, chunk, window, nk, nv;      // nk, nv: stages of the K and V rings
    float scale_log2, cap_in, cap_out;        // softcap: s <- cap_out tanh(s cap_in), log2 units
    float cap_poly[5], cap_small;             // the same for s^2 <= cap_small: s times a polynomial in s^2
};
// Softcap: none, any, or one so low that exp of a capped score and sums of it stay far inside the fp32 range
enum { FP_CAP_NONE = 0, FP_CAP = 1, FP_CAP_BOUND = 2 };
constexpr float FP_CAP_BOUND_LOG2 = 80.f;

// first key row (in key-row coordinates, may be negative) that query row i sees
__device__ __forceinline__ int64_t fp_first_row(const FpShape& p, int64_t i) {
    int64_t lo = -p.kv_start;
    if (p.chunk > 0) lo = (i + p.kv_start) / p.chunk * p.chunk - p.kv_start;
    if (p.window > 0 && i - p.window + 1 > lo) lo = i - p.window + 1;
    return lo;
}

// s <- cap_out tanh(s cap_in) for 32 scores from c0 on; the caller's loops are unrolled
template <int N> __device__ __forceinline__ void fp_cap32(const FpShape& p, float (&s)[N], int c0) {
    uint64_t t[16];
    float top[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const uint64_t x = pack2(s[c0 + 2 * i], s[c0 + 2 * i + 1]);
        t[i] = mul2(x, x);
        float a, b;
        unpack2(t[i], a, b);
        top[i & 1] = max3(top[i & 1], a, b);
    }
    if (__any_sync(FULL, !(fmaxf(top[0], top[1]) <= p.cap_small))) {
#pragma unroll
        for (int c = 0; c < 32; ++c) s[c0 + c] = p.cap_out * tanh_exp2(s[c0 + c] * p.cap_in);
    } else {
        const uint64_t k0 = pack2(p.cap_poly[0], p.cap_poly[0]), k1 = pack2(p.cap_poly[1], p.cap_poly[1]),
                       k2 = pack2(p.cap_poly[2], p.cap_poly[2]), k3 = pack2(p.cap_poly[3], p.cap_poly[3]),
                       k4 = pack2(p.cap_poly[4], p.cap_poly[4]);
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            uint64_t r = fma2(t[i], k4, k3);
            r = fma2(t[i], r, k2);
            r = fma2(t[i], r, k1);
            r = fma2(t[i], r, k0);
            r = mul2(r, pack2(s[c0 + 2 * i], s[c0 + 2 * i + 1]));
            unpack2(r, s[c0 + 2 * i], s[c0 + 2 * i + 1]);
        }
    }
}

template <bool BIAS, int CAP>
__global__ void __launch_bounds__(FP_THREADS, 1)
attn_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                    const __grid_constant__ CUtensorMap map_v, const FpShape p) {
    extern __shared__ char fp_raw[];
    __shared__ FpShared sh;
    char* tiles = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(fp_raw) + 1023) & ~(uintptr_t)1023);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G);
    const int np = (p.dqk + 63) / 64, nvp = (p.dv + 63) / 64;
    char* q_s = tiles;                                        // [tile][panel]
    char* k_s = q_s + 2 * np * FP_PANEL;                      // [stage][panel]
    char* v_s = k_s + p.nk * np * FP_PANEL;
    float* bias_s = reinterpret_cast<float*>(v_s + p.nv * nvp * FP_PANEL);

    // query tiles, and the range [beg, end) of key tiles each of them visits; key rows count from kv_start
    const int q0 = (int)(gridDim.x - 1 - blockIdx.x) * 2 * FP_TILE;       // long rows first
    int64_t i0[2];
    int beg[2], end[2];
    int64_t base = 0;
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        const int first = q0 + t * FP_TILE;
        i0[t] = p.start + first - p.kv_start;
        int64_t lo = fp_first_row(p, i0[t]);
        if (lo < 0) lo = 0;
        if (t == 0) base = lo;
        const int rows = p.S - first < FP_TILE ? p.S - first : FP_TILE;
        beg[t] = (int)((lo - base) / FP_TILE);
        end[t] = rows > 0 ? (int)((i0[t] + rows - 1 - base) / FP_TILE) + 1 : 0;
        if (rows <= 0) beg[t] = 0;
    }
    const int n = end[1] > end[0] ? end[1] : end[0];

    if (tid == 0) {
        mbar_init_count(&sh.q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init_count(&sh.k_full[s], 1);
            mbar_init_count(&sh.k_empty[s], 1);
            mbar_init_count(&sh.v_full[s], 1);
            mbar_init_count(&sh.v_empty[s], 1);
            mbar_init_count(&sh.s_full[s], 1);
            mbar_init_count(&sh.p_full[s], 4);
            mbar_init_count(&sh.o_full[s], 1);
        }
        mbar_init_count(&sh.drained, 1);
        sh.failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(&sh.tmem_base)),
                     "r"(512u)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sh.tmem_base;                       // columns: S0 | S1 | O0 | O1, 128 each
    volatile int* failed = &sh.failed;

    if (warp == 0) {
        // ---- TMA producer
        if (lane == 0) {
            const uint32_t k_bytes = np * FP_PANEL, v_bytes = nvp * FP_PANEL;
            mbar_expect(&sh.q_full, 2 * k_bytes);
            for (int t = 0; t < 2; ++t)
                for (int c = 0; c < np; ++c)
                    tma_load_4d(q_s + (t * np + c) * FP_PANEL, &map_q, c * 64, h, q0 + t * FP_TILE, b, &sh.q_full);
            int j = 0;
            bool k_sent = false;
            for (; j < n && !*failed; ++j) {
                const int ks = j % p.nk, vs = j % p.nv, row = (int)base + j * FP_TILE;
                if (j >= p.nk && !mbar_wait_bounded(&sh.k_empty[ks], (uint32_t)((j / p.nk - 1) & 1))) { *failed = 1; break; }
                mbar_expect(&sh.k_full[ks], k_bytes);
                for (int c = 0; c < np; ++c)
                    tma_load_4d(k_s + (ks * np + c) * FP_PANEL, &map_k, c * 64, g, row, b, &sh.k_full[ks]);
                k_sent = true;
                if (j >= p.nv && !mbar_wait_bounded(&sh.v_empty[vs], (uint32_t)((j / p.nv - 1) & 1))) { *failed = 1; break; }
                mbar_expect(&sh.v_full[vs], v_bytes);
                for (int c = 0; c < nvp; ++c)
                    tma_load_4d(v_s + (vs * nvp + c) * FP_PANEL, &map_v, c * 64, g, row, b, &sh.v_full[vs]);
                k_sent = false;
            }
            if (*failed) {                                    // leave no copy in flight
                mbar_wait_bounded(&sh.q_full, 0);
                const int nk_sent = j + (k_sent ? 1 : 0);
                for (int i = nk_sent > p.nk ? nk_sent - p.nk : 0; i < nk_sent; ++i)
                    mbar_wait_bounded(&sh.k_full[i % p.nk], (uint32_t)((i / p.nk) & 1));
                for (int i = j > p.nv ? j - p.nv : 0; i < j; ++i)
                    mbar_wait_bounded(&sh.v_full[i % p.nv], (uint32_t)((i / p.nv) & 1));
            }
        }
    } else if (warp == 1) {
        // ---- MMA issuer
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc_bf16(FP_TILE, false), idesc_o = umma_idesc_bf16((p.dv + 15) / 16 * 16, true);
            const int k_steps = (p.dqk + 15) / 16;
            const uint32_t q_addr = smem_addr(q_s), k_addr = smem_addr(k_s), v_addr = smem_addr(v_s);
            auto scores = [&](int t, int j) {                 // S_t = Q_t K_j^T
                const uint32_t qa = q_addr + t * np * FP_PANEL, ka = k_addr + (j % p.nk) * np * FP_PANEL;
                for (int k = 0; k < k_steps; ++k) {
                    const uint32_t off = (uint32_t)(k >> 2) * FP_PANEL + (k & 3) * 32;
                    umma_ss(tmem + t * FP_TILE, umma_desc_sw128(qa + off), umma_desc_sw128(ka + off), idesc_s, k > 0);
                }
                umma_commit(&sh.s_full[t]);
            };
            bool ok = mbar_wait_bounded(&sh.q_full, 0) && mbar_wait_bounded(&sh.k_full[0], 0);
            if (ok) {
                tc_fence_after();
                for (int t = 0; t < 2; ++t)
                    if (beg[t] == 0 && end[t] > 0) scores(t, 0);
                umma_commit(&sh.k_empty[0]);
            }
            for (int j = 0; ok && j < n && !*failed; ++j) {
                const bool more = j + 1 < n;
                if (more) ok = mbar_wait_bounded(&sh.k_full[(j + 1) % p.nk], (uint32_t)(((j + 1) / p.nk) & 1));
                ok = ok && mbar_wait_bounded(&sh.v_full[j % p.nv], (uint32_t)((j / p.nv) & 1));
                for (int t = 0; ok && t < 2; ++t) {
                    if (j >= beg[t] && j < end[t]) {
                        ok = mbar_wait_bounded(&sh.p_full[t], (uint32_t)((j - beg[t]) & 1));
                        if (!ok) break;
                        tc_fence_after();
                        const uint32_t va = v_addr + (j % p.nv) * nvp * FP_PANEL;
                        for (int k = 0; k < FP_TILE / 16; ++k)
                            umma_ts(tmem + 2 * FP_TILE + t * FP_TILE, tmem + t * FP_TILE + k * 8,
                                    umma_desc_sw128_mn(va + k * 2048, FP_PANEL), idesc_o, j > beg[t] || k > 0);
                        if (j + 1 == end[t]) umma_commit(&sh.o_full[t]);
                    }
                    // the scores of the next key tile replace weights that the MMAs above still read: same
                    // issuing thread, so they execute in order
                    if (more && j + 1 >= beg[t] && j + 1 < end[t]) scores(t, j + 1);
                }
                if (!ok) break;
                umma_commit(&sh.v_empty[j % p.nv]);
                if (more) umma_commit(&sh.k_empty[(j + 1) % p.nk]);
            }
            if (!ok) *failed = 1;
            umma_commit(&sh.drained);                         // leave no MMA and no barrier arrival in flight
            mbar_wait_bounded(&sh.drained, 0);
        }
    } else if (warp >= FP_SOFTMAX_WARP0) {
        // ---- softmax: thread = query row
        const int t = (warp - FP_SOFTMAX_WARP0) >> 2, quad = warp & 3, a = quad * 32 + lane;
        const uint32_t lane_base = (uint32_t)(quad * 32) << 16;
        const uint32_t s_addr = tmem + lane_base + t * FP_TILE, o_addr = tmem + lane_base + 2 * FP_TILE + t * FP_TILE;
        const int64_t i = i0[t] + a;                          // query row in key-row coordinates
        const float cc = BIAS || CAP != FP_CAP_NONE ? 1.f : p.scale_log2;    // log2 units per unit of s below
        const int64_t lo_row = fp_first_row(p, i), lo_last = fp_first_row(p, i0[t] + FP_TILE - 1);
        float* bt = bias_s + (warp - FP_SOFTMAX_WARP0) * FP_BIAS_SPAN;
        const float* bias_h = BIAS ? p.bias + (int64_t)h * p.bias_len : nullptr;
        float m = CAP == FP_CAP_BOUND ? 0.f : -INFINITY, l = 0.f;
        bool ok = true;
        for (int j = beg[t]; j < end[t]; ++j) {
            const int it = j - beg[t];
            const int64_t r0 = base + (int64_t)j * FP_TILE;
            if (BIAS) {                                       // this warp's distances: row - key = first + 0 .. 158
                const int64_t first = i0[t] + quad * 32 - r0 - (FP_TILE - 1);
                __syncwarp();
                for (int e = lane; e < FP_BIAS_SPAN; e += 32) {
                    int64_t d = first + e;
                    d = d < 0 ? 0 : (d < p.bias_len ? d : p.bias_len - 1);
                    bt[e] = __ldg(bias_h + d) * FP_LOG2E;
                }
                __syncwarp();
            }
            if (__any_sync(FULL, *failed != 0) || !__all_sync(FULL, mbar_wait_bounded(&sh.s_full[t], (uint32_t)(it & 1)))) {
                ok = false;
                break;
            }
            tc_fence_after();
            const bool partial = r0 + FP_TILE - 1 > i0[t] || r0 < lo_last;    // some row does not see the whole tile
            const int hi_c = (int)(i - r0 < FP_TILE ? i - r0 : FP_TILE), lo_c = (int)(lo_row - r0 > 0 ? lo_row - r0 : 0);
            if constexpr (CAP == FP_CAP_BOUND) {
                // nothing depends on the whole row: 32 scores at a time become 16 columns of weights, which overwrite
                // only scores that have been read
                uint64_t ls[2] = {0, 0};                      // two pairs of sums
#pragma unroll
                for (int c0 = 0; c0 < FP_TILE; c0 += 32) {
                    float s[32];
                    tmem_ld32(s_addr + c0, reinterpret_cast<uint32_t(&)[32]>(s));
                    fp_cap32(p, s, 0);
                    if (partial) {
#pragma unroll
                        for (int c = 0; c < 32; ++c)
                            if (c0 + c > hi_c || c0 + c < lo_c) s[c] = -INFINITY;
                    }
                    uint32_t w[16];
#pragma unroll
                    for (int c = 0; c < 16; ++c) {
                        const float x = exp2_fast(s[2 * c]), y = exp2_fast(s[2 * c + 1]);
                        ls[c & 1] = add2(ls[c & 1], pack2(x, y));
                        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
                        w[c] = *reinterpret_cast<const uint32_t*>(&v);
                    }
                    tmem_st16(s_addr + c0 / 2, w);
                }
                float l0, l1;
                unpack2(add2(ls[0], ls[1]), l0, l1);
                l += l0 + l1;
            } else {
                float s[FP_TILE];
                tmem_ld128(s_addr, reinterpret_cast<uint32_t(&)[FP_TILE]>(s));
                if (CAP != FP_CAP_NONE) {                         // small scores: a polynomial, off the exponential's unit
#pragma unroll
                    for (int c = 0; c < FP_TILE; c += 32) fp_cap32(p, s, c);
                }
                if (BIAS) {
#pragma unroll
                    for (int c = 0; c < FP_TILE; ++c) s[c] = fmaf(s[c], CAP != FP_CAP_NONE ? 1.f : p.scale_log2, bt[lane + FP_TILE - 1 - c]);
                }
                if (partial) {
#pragma unroll
                    for (int c = 0; c < FP_TILE; ++c)
                        if (c > hi_c || c < lo_c) s[c] = -INFINITY;
                }
                float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int c = 0; c < FP_TILE; c += 2) mx[(c >> 1) & 3] = max3(mx[(c >> 1) & 3], s[c], s[c + 1]);
                const float mn = fmaxf(m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));
                if (it == 0) {
                    m = mn;
                } else if (__any_sync(FULL, (mn - m) * cc > FP_RESCALE)) {
                    // the scores of this tile were issued after the previous tile's P V, so O is complete
                    const float f = mn == -INFINITY ? 1.f : exp2_fast((m - mn) * cc);
                    l *= f;
                    m = mn;
                    for (int c = 0; c < p.dv; c += 32) {
                        uint32_t r[32];
                        tmem_ld32(o_addr + c, r);
#pragma unroll
                        for (int e = 0; e < 32; ++e) r[e] = __float_as_uint(__uint_as_float(r[e]) * f);
                        tmem_st32(o_addr + c, r);
                    }
                }
                const float mc = m == -INFINITY ? 0.f : m * cc;
                const uint64_t scale2 = pack2(cc, cc), shift2 = pack2(-mc, -mc);
                uint64_t ls[2] = {0, 0};
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t w[32];
#pragma unroll
                    for (int c = 0; c < 32; ++c) {
                        float x = s[half * 64 + 2 * c], y = s[half * 64 + 2 * c + 1];
                        unpack2(fma2(pack2(x, y), scale2, shift2), x, y);
                        x = exp2_fast(x);
                        y = exp2_fast(y);
                        ls[c & 1] = add2(ls[c & 1], pack2(x, y));
                        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
                        w[c] = *reinterpret_cast<const uint32_t*>(&v);
                    }
                    tmem_st32(s_addr + half * 32, w);
                }
                float l0, l1;
                unpack2(add2(ls[0], ls[1]), l0, l1);
                l += l0 + l1;
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sh.p_full[t]);
        }
        if (ok && end[t] > 0) {
            ok = __all_sync(FULL, mbar_wait_bounded(&sh.o_full[t], 0));
            if (ok) {
                tc_fence_after();
                const float mc = m == -INFINITY ? 0.f : m * cc;
                if (p.sink != nullptr) l += exp2f(p.sink[h] * FP_LOG2E - mc);
                const float inv = 1.f / l;
                const int row = q0 + t * FP_TILE + a;
                __nv_bfloat16* o = (__nv_bfloat16*)p.out + (int64_t)b * p.o_bs + (int64_t)row * p.o_ss + h * p.o_hs;
                for (int c = 0; c < p.dv; c += 32) {
                    uint32_t r[32];
                    tmem_ld32(o_addr + c, r);
                    if (row < p.S) {
#pragma unroll
                        for (int e = 0; e < 32; e += 8) {
                            if (c + e < p.dv) {
                                uint32_t w[4];
#pragma unroll
                                for (int k = 0; k < 4; ++k) {
                                    const __nv_bfloat162 v = __floats2bfloat162_rn(__uint_as_float(r[e + 2 * k]) * inv,
                                                                                   __uint_as_float(r[e + 2 * k + 1]) * inv);
                                    w[k] = *reinterpret_cast<const uint32_t*>(&v);
                                }
                                *reinterpret_cast<uint4*>(o + c + e) = make_uint4(w[0], w[1], w[2], w[3]);
                            }
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
    if (warp == 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
}

// Stages of the two rings and the dynamic shared memory they take; 0 bytes when the shape does not fit
uint32_t plan_smem(int dqk, int dv, bool bias, int* nk, int* nv) {
    const uint32_t np = (dqk + 63) / 64, nvp = (dv + 63) / 64, extra = bias ? FP_BIAS_BYTES : 0;
    const int plans[3][2] = {{2, 2}, {2, 1}, {1, 1}};
    for (auto& pl : plans) {
        const uint32_t bytes = ((2 + pl[0]) * np + pl[1] * nvp) * FP_PANEL + extra;
        if (bytes <= FP_SMEM_MAX) {
            *nk = pl[0];
            *nv = pl[1];
            return bytes + 1024;
        }
    }
    return 0;
}

}  // namespace

bool attn_prefill_tc_applicable(const sk_attn_params& p) {
    int nk, nv;
    return p.dtype == SK_BF16 && p.pos == nullptr && !p.ring && p.dv <= 128 && p.dqk <= 256 && p.scale > 0.f &&
           p.start >= p.kv_start && p.kv_rows < (int64_t)1 << 30 && head_map_ok(p.q, p.dqk, p.q_hs, p.q_ss, p.q_bs) &&
           head_map_ok(p.k, p.dqk, p.k_hs, p.k_ts, p.k_bs) && head_map_ok(p.v, p.dv, p.v_hs, p.v_ts, p.v_bs) &&
           head_map_ok(p.out, p.dv, p.o_hs, p.o_ss, p.o_bs) && plan_smem(p.dqk, p.dv, p.bias != nullptr, &nk, &nv) > 0;
}

int launch_attn_prefill_tc(const sk_attn_params& p, cudaStream_t st) {
    FpShape f;
    f.out = p.out;
    f.bias = p.bias;
    f.sink = p.sink;
    f.status = p.status;
    f.o_bs = p.o_bs;
    f.o_ss = p.o_ss;
    f.o_hs = p.o_hs;
    f.start = p.start;
    f.kv_start = p.kv_start;
    f.bias_len = p.bias_len;
    f.S = p.S;
    f.H = p.H;
    f.G = p.G;
    f.dqk = p.dqk;
    f.dv = p.dv;
    f.chunk = p.chunk;
    f.window = p.window;
    f.scale_log2 = p.scale * FP_LOG2E;
    f.cap_in = p.softcap > 0.f ? p.scale / p.softcap : 0.f;
    f.cap_out = p.softcap * FP_LOG2E;
    double c = p.scale * 1.4426950408889634, c2 = (double)f.cap_in * f.cap_in;
    for (int k = 0; k < 5; ++k, c *= c2) f.cap_poly[k] = (float)(TANH_POLY[k] * c);
    f.cap_small = f.cap_in > 0.f ? (TANH_POLY_RANGE / f.cap_in) * (TANH_POLY_RANGE / f.cap_in) : 0.f;
    const uint32_t smem = plan_smem(p.dqk, p.dv, p.bias != nullptr, &f.nk, &f.nv);
    CUtensorMap mq, mk, mv;
    if (int rc = make_head_map(&mq, p.q, p.dqk, p.H, p.S, p.B, p.q_hs, p.q_ss, p.q_bs, FP_TILE)) return rc;
    if (int rc = make_head_map(&mk, p.k, p.dqk, p.G, p.kv_rows, p.B, p.k_hs, p.k_ts, p.k_bs, FP_TILE)) return rc;
    if (int rc = make_head_map(&mv, p.v, p.dv, p.G, p.kv_rows, p.B, p.v_hs, p.v_ts, p.v_bs, FP_TILE)) return rc;
    auto kern = p.bias != nullptr ? attn_prefill_kernel<true, FP_CAP_NONE> : attn_prefill_kernel<false, FP_CAP_NONE>;
    if (p.softcap > 0.f)
        kern = p.bias != nullptr ? attn_prefill_kernel<true, FP_CAP>
                                 : (f.cap_out <= FP_CAP_BOUND_LOG2 ? attn_prefill_kernel<false, FP_CAP_BOUND> : attn_prefill_kernel<false, FP_CAP>);
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "attn_prefill_kernel smem attribute: %s", cudaGetErrorString(e));
    dim3 grid((unsigned)((p.S + 2 * FP_TILE - 1) / (2 * FP_TILE)), (unsigned)p.H, (unsigned)p.B);
    kern<<<grid, FP_THREADS, smem, st>>>(mq, mk, mv, f);
    return check_launch("attn_prefill_kernel");
}

}  // namespace sk
