// Softmax attention of one or a few query tokens against a long cache (bf16), split over the keys.
//
// All query rows that share a key/value head (rep heads x S tokens) are worked on together, up to 16 or 32 rows
// per CTA, so a key is read once for all of them; with one key/value head for every query head - attention on
// latent rows - this is what makes the step read each cache row once.  A CTA walks its share of 64-key tiles
// (TMA, 128-byte swizzle, double buffer), computes the scores with m16n8k16 MMAs (rows are too few for the 128-row tensor
// core tiles), keeps the running maximum per row and accumulates P V with each warp owning a slice of the value columns.
// When keys and values are slices of the same rows in memory (values a prefix of latent rows; rotary keys that share
// all but their turned elements with the values), one tile of the whole rows serves both.  A second kernel
// merges the partial results of the splits.  The live length is read on the device; the grid is fixed.
#include "blocks.cuh"
#include "tcgen05.cuh"
#include "tensor_map.cuh"
#include "warp_mma.cuh"

#include <type_traits>

namespace sk {
namespace {

constexpr int DM_WARPS = 8, DM_KEYS = 64;      // warps per 16-row tile, keys per tile
constexpr uint32_t DM_PANEL = DM_KEYS * 128;             // 64 keys x 64 columns
constexpr float DM_LOG2E = 1.4426950408889634f;
constexpr int DM_MAX_SPLITS = 160;

struct DmPlan {
    int mt;                 // 16-row tiles per CTA
    int nvt;                // 8-column value tiles per warp
    int groups;             // row groups per (batch, key/value head)
    int splits;
    bool shared_v;
    int k_off;              // first key column of a shared tile, whose column 0 is the first value column
    int q_stride;           // elements per shared-memory row of the queries
    int np, nvp;            // 64-column panels of a key and of a value tile (0: the key tile serves)
    size_t smem;
    size_t part_floats;     // per split: 16 mt rows x (dv + 2)
};

bool dm_plan(const sk_attn_params& p, DmPlan* d) {
    if (p.dtype != SK_BF16 || p.dqk % 8 || p.dv % 8 || p.dv > 512 || p.dqk > 640 || p.kv_rows >= (int64_t)1 << 30) return false;
    const int rows = p.S * (p.H / p.G);
    d->mt = rows <= 16 ? 1 : 2;
    d->nvt = p.dv <= 128 ? 2 : (p.dv <= 256 ? 4 : 8);
    d->groups = (rows + 16 * d->mt - 1) / (16 * d->mt);
    const int64_t delta = ((intptr_t)p.k - (intptr_t)p.v) / 2;
    d->shared_v = p.v_ts == p.k_ts && p.v_bs == p.k_bs && (p.G == 1 || p.v_hs == p.k_hs) && delta >= 0 && delta % 8 == 0 &&
                  delta + p.dqk <= 640 && p.dv <= delta + p.dqk && delta + p.dqk <= p.k_ts && (p.G == 1 || delta + p.dqk <= p.k_hs);
    d->k_off = d->shared_v ? (int)delta : 0;
    d->q_stride = (p.dqk + 15) / 16 * 16 + 8;
    d->np = (d->k_off + (p.dqk + 15) / 16 * 16 + 63) / 64;
    d->nvp = d->shared_v ? 0 : (p.dv + 63) / 64;
    d->smem = 1024 + (size_t)2 * (d->np + d->nvp) * DM_PANEL + (size_t)16 * d->mt * (DM_KEYS + 8) * 2 +
              (d->mt == 1 ? (size_t)16 * d->q_stride * 2 : (size_t)4 * 32 * (DM_KEYS + 8) * 4);   // queries / partial scores
    if (d->smem > 220 * 1024) return false;
    const int per_sm = d->smem > 110 * 1024 ? 1 : (d->smem > 72 * 1024 || d->mt == 2 ? 2 : 3);
    const int64_t ctas = (int64_t)d->groups * p.G * p.B, tiles = (p.kv_rows + DM_KEYS - 1) / DM_KEYS;
    int64_t sp = ((int64_t)sm_count() * per_sm) / ctas;
    if (sp > tiles) sp = tiles;
    if (sp > DM_MAX_SPLITS) sp = DM_MAX_SPLITS;
    d->splits = sp < 1 ? 1 : (int)sp;
    d->part_floats = (size_t)16 * d->mt * (p.dv + 2);
    return true;
}

// Visible key rows of one call in key-row coordinates, and how they are dealt to the splits
struct DmRange {
    int64_t i_first, base;      // position of token 0, position of key row 0
    int lo, hi;                 // rows any query of the call sees: [lo, hi]
    int tiles, per_split;
    int wrap;                   // rows of a ring that holds the latest positions (0: rows are in order)
    bool outside;               // a token lies beyond the cache
};
__device__ __forceinline__ DmRange dm_range(const sk_attn_params& p, int splits) {
    DmRange r;
    r.i_first = first_position(p.pos, p.start);
    const int64_t chunk_lo = p.chunk > 0 ? r.i_first / p.chunk * p.chunk : 0;
    r.wrap = p.ring && p.chunk == 0 ? (int)p.kv_rows : 0;
    r.base = r.wrap ? 0 : (p.ring ? chunk_lo : p.kv_start);
    int64_t lo = chunk_lo;
    if (p.window > 0 && !r.wrap && r.i_first - p.window + 1 > lo) lo = r.i_first - p.window + 1;
    r.lo = (int)(lo > r.base ? lo - r.base : 0);
    int64_t hi = r.i_first + p.S - 1 - r.base;
    r.outside = hi >= p.kv_rows && !r.wrap;                      // flagged by the first CTA
    if (hi >= p.kv_rows) hi = p.kv_rows - 1;
    r.hi = (int)hi;
    r.tiles = r.hi >= r.lo ? (r.hi - r.lo) / DM_KEYS + 1 : 0;
    r.per_split = (r.tiles + splits - 1) / splits;
    return r;
}

// What one query row (token s of the call) sees: key rows [lo, hi], at the distance origin - row (+ wrap if negative)
struct DmRow {
    int lo, hi;
    int64_t origin;
};
__device__ __forceinline__ DmRow dm_row(const sk_attn_params& p, const DmRange& rg, int s, bool live) {
    const int64_t i = rg.i_first + s;
    DmRow r;
    r.origin = rg.wrap ? i % rg.wrap : i - rg.base;
    int64_t lo = p.chunk > 0 ? i / p.chunk * p.chunk - rg.base : 0;
    if (p.window > 0 && !rg.wrap) lo = max(lo, i - p.window + 1 - rg.base);
    r.lo = (int)max((int64_t)0, lo);
    r.hi = !live ? -1 : rg.wrap ? rg.hi : (int)min(r.origin, (int64_t)rg.hi);      // an absent row sees nothing
    return r;
}
// scaled score in log2 units, without bias: in, out = scale / softcap, softcap under a cap, else out = scale
template <bool CAP> __device__ __forceinline__ float dm_score(float dot, float in, float out) {
    return CAP ? out * tanh_exp2(dot * in) : dot * out;
}

// Up to 16 query rows: a warp computes the scores of 8 keys of a tile.  NVT: 8-column value tiles per warp
template <int NVT, bool CAP>
__global__ void __launch_bounds__(DM_WARPS * 32)
attn_decode_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const __grid_constant__ sk_attn_params p,
                   int splits, int groups, int np, int nvp, int k_off, int q_stride, size_t part_floats) {
    extern __shared__ char dm_raw[];
    constexpr int ROWS = 16, WARPS = DM_WARPS, KG = 8;
    __shared__ __align__(16) float wmax[2][ROWS][KG];
    __shared__ float row_sum[ROWS][KG];
    __shared__ uint64_t full[2];
    using bf = __nv_bfloat16;
    char* ks = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(dm_raw) + 1023) & ~(uintptr_t)1023);   // [2][panel][64][128 B]
    char* vs = nvp > 0 ? ks + 2 * np * DM_PANEL : ks;
    const int v_panels = nvp > 0 ? nvp : np;                    // stage stride of the value tiles
    bf* qs = reinterpret_cast<bf*>(ks + 2 * (np + nvp) * DM_PANEL);   // [ROWS][q_stride]
    constexpr int PS = DM_KEYS + 8;
    bf* ps = qs + ROWS * q_stride;                              // [ROWS][64 + 8]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, g = blockIdx.y / groups, grp = blockIdx.y % groups, b = blockIdx.z;
    const int rep = p.H / p.G, n_rows = p.S * rep, r_first = grp * ROWS;
    pdl_launch_dependents();
    const DmRange rg = dm_range(p, splits);
    if (split == 0 && grp == 0 && tid == 0 && p.status != nullptr && rg.outside)
        atomicOr(p.status, SK_DEV_POS_OUT_OF_RANGE);
    const int t_beg = split * rg.per_split;
    const int t_end = t_beg + rg.per_split < rg.tiles ? t_beg + rg.per_split : rg.tiles;
    if (t_beg >= t_end) return;                                 // the merge knows which splits exist

    // one thread: the 64-column panels of a tile; rows past the end of the tensor read as zero, rows past the live
    // end are masked
    auto fetch = [&](int tile, int stage) {
        const int row = rg.lo + tile * DM_KEYS;
        mbar_expect(&full[stage], (uint32_t)(np + nvp) * DM_PANEL);
        for (int c = 0; c < np; ++c) tma_load_4d(ks + (stage * np + c) * DM_PANEL, &map_k, c * 64, g, row, b, &full[stage]);
        for (int c = 0; c < nvp; ++c) tma_load_4d(vs + (stage * nvp + c) * DM_PANEL, &map_v, c * 64, g, row, b, &full[stage]);
    };
    if (tid == 0) {
        mbar_init_count(&full[0], 1);
        mbar_init_count(&full[1], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fetch(t_beg, 0);
    }
    const int k16 = (p.dqk + 15) / 16, kc = p.dqk / 8;
    // queries, and the zero columns that round a row up to 16
    for (int r = warp; r < ROWS; r += WARPS) {
        const int row = r_first + r, s = row / rep, hh = row - s * rep;
        const bf* src = (const bf*)p.q + (int64_t)b * p.q_bs + (int64_t)s * p.q_ss + (int64_t)(g * rep + hh) * p.q_hs;
        for (int c = lane; c < k16 * 2; c += 32) {
            const uint4 v = row < n_rows && c < kc ? *reinterpret_cast<const uint4*>(src + c * 8) : make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(qs + r * q_stride + c * 8) = v;
        }
    }

    // rows of this thread
    const int kg = warp;                                        // key group
    const int fr = lane >> 2, fc = (lane & 3) * 2;              // fragment row and first column
    DmRow see[2];
    const float* brow[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int row = r_first + fr + 8 * k, s = row / rep;
        see[k] = dm_row(p, rg, s, row < n_rows);
        brow[k] = p.bias != nullptr && row < n_rows ? p.bias + (int64_t)(g * rep + row - s * rep) * p.bias_len : nullptr;
    }
    const float cap_in = CAP ? p.scale / p.softcap : 0.f, sl = (CAP ? p.softcap : p.scale) * DM_LOG2E;
    float m_own[2] = {-INFINITY, -INFINITY}, l_own[2] = {0.f, 0.f};
    float acc[NVT][4];
#pragma unroll
    for (int v = 0; v < NVT; ++v)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[v][e] = 0.f;
    const int col0 = warp * NVT * 8;
    bool in_time = true;

    for (int t = t_beg; t < t_end; ++t) {
        const int it = t - t_beg, stage = it & 1;
        __syncthreads();                                        // the other stage is free
        if (tid == 0 && t + 1 < t_end) fetch(t + 1, stage ^ 1);
        if (in_time) in_time = mbar_wait_bounded(&full[stage], (uint32_t)((it >> 1) & 1));
        // ---- scores of 16 rows x 8 keys, two independent sums along the head dimension
        float sc[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[u][e] = 0.f;
        // a lane reads row (lane & 7) of its 8-key group; 16-byte piece c of a row sits at piece c ^ (row & 7)
        const uint32_t qa = saddr(qs + ((lane & 15)) * q_stride + (lane >> 4) * 8);
        const uint32_t ka = saddr(ks + stage * np * DM_PANEL + (kg * 8 + (lane & 7)) * 128);
        const int sw = lane & 7, kp = k_off / 8;                // the keys begin at 16-byte piece kp of a row
        auto dot = [&](auto shifted) {                          // keys that begin a row: panels and pieces by kk alone
            auto piece = [&](int kk, int i) {
                const int c = kk * 2 + i + (shifted.value ? kp : 0);
                return shifted.value ? ka + (c >> 3) * DM_PANEL + (((c & 7) ^ sw) << 4)
                                     : ka + (kk >> 2) * DM_PANEL + ((((kk & 3) * 2 + i) ^ sw) << 4);
            };
            int kk = 0;
#pragma unroll 4
            for (; kk + 2 <= k16; kk += 2) {                    // 32 head dimensions at a time
                uint32_t a0[4], a1[4], bb[4];
                ldsm4(piece(kk, lane >> 3), bb);
                ldsm4(qa + kk * 32, a0);
                ldsm4(qa + kk * 32 + 32, a1);
                mma16816(sc[0], a0, bb[0], bb[1]);
                mma16816(sc[1], a1, bb[2], bb[3]);
            }
            if (kk < k16) {
                uint32_t a0[4], b0, b1;
                ldsm2(piece(kk, (lane >> 3) & 1), b0, b1);
                ldsm4(qa + kk * 32, a0);
                mma16816(sc[0], a0, b0, b1);
            }
        };
        if (kp == 0) dot(std::false_type{});
        else dot(std::true_type{});
        const int r0 = rg.lo + t * DM_KEYS + kg * 8;            // key row of column 0 of this warp
        float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = e >> 1, r = r0 + fc + (e & 1);
            float v = dm_score<CAP>(sc[0][e] + sc[1][e], cap_in, sl);
            if (r >= see[k].lo && r <= see[k].hi) {
                if (brow[k] != nullptr) {
                    int64_t d = see[k].origin - r;
                    if (d < 0) d += rg.wrap;
                    v = fmaf(__ldg(brow[k] + (d < p.bias_len ? d : p.bias_len - 1)), DM_LOG2E, v);
                }
            } else {
                v = -INFINITY;
            }
            sc[0][e] = v;
            mt[k] = fmaxf(mt[k], v);
        }
        float (*wm)[KG] = wmax[it & 1];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            mt[k] = fmaxf(mt[k], __shfl_xor_sync(FULL, mt[k], 1));
            mt[k] = fmaxf(mt[k], __shfl_xor_sync(FULL, mt[k], 2));
            if ((lane & 3) == 0) wm[fr + 8 * k][kg] = mt[k];
        }
        __syncthreads();
        // ---- new maxima: accumulators follow them, scores become weights
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float4* w4 = reinterpret_cast<const float4*>(wm[fr + 8 * k]);
            const float4 x = w4[0], y = w4[1];
            const float mn = fmaxf(fmaxf(fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w)), fmaxf(fmaxf(y.x, y.y), fmaxf(y.z, y.w))), m_own[k]);
            if (mn != m_own[k]) {
                const float f = exp2_fast(m_own[k] - mn);       // mn is finite here
#pragma unroll
                for (int v = 0; v < NVT; ++v) {
                    acc[v][2 * k] *= f;
                    acc[v][2 * k + 1] *= f;
                }
                l_own[k] *= f;
                m_own[k] = mn;
            }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float mc = m_own[k] == -INFINITY ? 0.f : m_own[k];
            const float x = exp2_fast(sc[0][2 * k] - mc), y = exp2_fast(sc[0][2 * k + 1] - mc);
            l_own[k] += x + y;
            *reinterpret_cast<__nv_bfloat162*>(ps + (fr + 8 * k) * PS + kg * 8 + fc) = __floats2bfloat162_rn(x, y);
        }
        __syncthreads();
        // ---- P V: every warp its own value columns
        if (col0 < p.dv) {
            const uint32_t va = saddr(vs + stage * v_panels * DM_PANEL + (lane & 15) * 128);
#pragma unroll
            for (int k = 0; k < DM_KEYS / 16; ++k) {
                uint32_t a[4];
                ldsm4(saddr(ps + (lane & 15) * PS + k * 16 + (lane >> 4) * 8), a);
#pragma unroll
                for (int v = 0; v < NVT; v += 2) {
                    if (col0 + v * 8 < p.dv) {
                        uint32_t bb[4];
                        const int c = (col0 >> 3) + v + (lane >> 4);
                        ldsm4t(va + (c >> 3) * DM_PANEL + k * 2048 + (((c & 7) ^ sw) << 4), bb);
                        mma16816(acc[v], a, bb[0], bb[1]);
                        mma16816(acc[v + 1], a, bb[2], bb[3]);
                    }
                }
            }
        }
    }
    if (!in_time) {                                             // a copy did not land: reported, and none left in flight
        if (p.status != nullptr) atomicOr(p.status, SK_DEV_WAIT_TIMEOUT);
        mbar_wait_bounded(&full[(t_end - 1 - t_beg) & 1], (uint32_t)(((t_end - 1 - t_beg) >> 1) & 1));
        if (t_end - t_beg > 1) mbar_wait_bounded(&full[(t_end - t_beg) & 1], (uint32_t)(((t_end - 2 - t_beg) >> 1) & 1));
    }
    // ---- partial result: rows x (dv sums | maximum | sum of weights)
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        l_own[k] += __shfl_xor_sync(FULL, l_own[k], 1);
        l_own[k] += __shfl_xor_sync(FULL, l_own[k], 2);
        if ((lane & 3) == 0) row_sum[fr + 8 * k][kg] = l_own[k];
    }
    __syncthreads();
    float* part = (float*)p.workspace + ((((int64_t)b * p.G + g) * groups + grp) * splits + split) * part_floats;
    if (tid < ROWS) {
        float l = 0.f;
#pragma unroll
        for (int w = 0; w < KG; ++w) l += row_sum[tid][w];
        part[(int64_t)ROWS * p.dv + ROWS + tid] = l;
    }
    if (warp == 0 && (lane & 3) == 0)
#pragma unroll
        for (int k = 0; k < 2; ++k) part[(int64_t)ROWS * p.dv + fr + 8 * k] = m_own[k];
#pragma unroll
    for (int v = 0; v < NVT; ++v) {
        const int c = col0 + v * 8 + fc;
        if (c < p.dv) {
#pragma unroll
            for (int k = 0; k < 2; ++k)
                *reinterpret_cast<float2*>(part + (int64_t)(fr + 8 * k) * p.dv + c) = make_float2(acc[v][2 * k], acc[v][2 * k + 1]);
        }
    }
}

// The form for more than 16 query rows (latent attention with many heads): 32 rows per CTA, 8 warps.  Four warps
// split the head dimension and two the keys of a tile, so that every warp keeps its share of the queries in
// registers and no key is read from shared memory twice; the partial scores meet in shared memory, where eight
// lanes own a row: they sum, mask, keep its maximum and sum of weights, and write the weights for P V.
// KS: 16-column steps of the head dimension per warp, NVT: 8-column value tiles per warp
template <int KS, int NVT, bool CAP>
__global__ void __launch_bounds__(DM_WARPS * 32)
attn_decode_wide_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                        const __grid_constant__ sk_attn_params p, int splits, int groups, int np, int nvp, int k_off, size_t part_floats) {
    extern __shared__ char dm_raw[];
    constexpr int ROWS = 32, PS = DM_KEYS + 8, RS = DM_KEYS + 8;
    __shared__ float f_s[ROWS];
    __shared__ uint64_t full[2];
    using bf = __nv_bfloat16;
    char* ks = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(dm_raw) + 1023) & ~(uintptr_t)1023);   // [2][panel][64][128 B]
    char* vs = nvp > 0 ? ks + 2 * np * DM_PANEL : ks;
    const int v_panels = nvp > 0 ? nvp : np;
    float* red = reinterpret_cast<float*>(ks + 2 * (np + nvp) * DM_PANEL);   // [4][ROWS][RS]
    bf* ps = reinterpret_cast<bf*>(red + 4 * ROWS * RS);                     // [ROWS][PS]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, g = blockIdx.y / groups, grp = blockIdx.y % groups, b = blockIdx.z;
    const int rep = p.H / p.G, n_rows = p.S * rep, r_first = grp * ROWS;
    pdl_launch_dependents();
    const DmRange rg = dm_range(p, splits);
    if (split == 0 && grp == 0 && tid == 0 && p.status != nullptr && rg.outside)
        atomicOr(p.status, SK_DEV_POS_OUT_OF_RANGE);
    const int t_beg = split * rg.per_split;
    const int t_end = t_beg + rg.per_split < rg.tiles ? t_beg + rg.per_split : rg.tiles;
    if (t_beg >= t_end) return;
    auto fetch = [&](int tile, int stage) {                     // one thread, as in the narrow form
        const int row = rg.lo + tile * DM_KEYS;
        mbar_expect(&full[stage], (uint32_t)(np + nvp) * DM_PANEL);
        for (int c = 0; c < np; ++c) tma_load_4d(ks + (stage * np + c) * DM_PANEL, &map_k, c * 64, g, row, b, &full[stage]);
        for (int c = 0; c < nvp; ++c) tma_load_4d(vs + (stage * nvp + c) * DM_PANEL, &map_v, c * 64, g, row, b, &full[stage]);
    };
    if (tid == 0) {
        mbar_init_count(&full[0], 1);
        mbar_init_count(&full[1], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fetch(t_beg, 0);
    }
    // ---- this warp's slice of the queries, as MMA fragments
    const int fr = lane >> 2, fc = (lane & 3) * 2;
    const int k16 = (p.dqk + 15) / 16, per = (k16 + 3) / 4, kq = warp & 3, kg = warp >> 2;
    const int k_lo = kq * per, k_n = k_lo + per < k16 ? per : k16 - k_lo;    // <= KS steps, none for a short head
    uint32_t qf[2][KS][4];
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int row = r_first + mt * 16 + fr + 8 * e, s = row / rep, hh = row - s * rep;
            const bf* src = (const bf*)p.q + (int64_t)b * p.q_bs + (int64_t)s * p.q_ss + (int64_t)(g * rep + hh) * p.q_hs;
#pragma unroll
            for (int k = 0; k < KS; ++k)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int c = (k_lo + k) * 16 + half * 8 + fc;
                    qf[mt][k][half * 2 + e] = row < n_rows && k < k_n && c < p.dqk ? *reinterpret_cast<const uint32_t*>(src + c) : 0u;
                }
        }
    // ---- the row this lane helps to own, and the positions it may see
    const int own = warp * 4 + (lane >> 3), own_row = r_first + own, own_s = own_row / rep;
    const bool live_row = own_row < n_rows;
    const DmRow see = dm_row(p, rg, own_s, live_row);
    const float* brow = p.bias != nullptr && live_row ? p.bias + (int64_t)(g * rep + own_row - own_s * rep) * p.bias_len : nullptr;
    const float cap_in = CAP ? p.scale / p.softcap : 0.f, sl = (CAP ? p.softcap : p.scale) * DM_LOG2E;
    float m = -INFINITY, l = 0.f;
    float acc[2][NVT][4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int v = 0; v < NVT; ++v)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[t][v][e] = 0.f;
    const int col0 = warp * NVT * 8, sw = lane & 7, kp = k_off / 8;
    bool in_time = true;

    for (int t = t_beg; t < t_end; ++t) {
        const int it = t - t_beg, stage = it & 1;
        __syncthreads();                                        // the other stage is free
        if (tid == 0 && t + 1 < t_end) fetch(t + 1, stage ^ 1);
        if (in_time) in_time = mbar_wait_bounded(&full[stage], (uint32_t)((it >> 1) & 1));
        // ---- 32 rows x 32 keys over this warp's slice of the head dimension
        {
            float sc[2][4][4];
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int n = 0; n < 4; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) sc[mt][n][e] = 0.f;
            const uint32_t ka = saddr(ks + stage * np * DM_PANEL + (kg * 32 + (lane & 7) + (lane >> 4) * 8) * 128);
#pragma unroll
            for (int k = 0; k < KS; ++k) {
                if (k < k_n) {
                    const int kk = k_lo + k;
                    const int c = kk * 2 + ((lane >> 3) & 1) + kp;
                    const uint32_t at = ka + (c >> 3) * DM_PANEL + (((c & 7) ^ sw) << 4);
                    uint32_t b0[4], b1[4];
                    ldsm4(at, b0);
                    ldsm4(at + 16 * 128, b1);
#pragma unroll
                    for (int mt = 0; mt < 2; ++mt) {
                        mma16816(sc[mt][0], qf[mt][k], b0[0], b0[1]);
                        mma16816(sc[mt][1], qf[mt][k], b0[2], b0[3]);
                        mma16816(sc[mt][2], qf[mt][k], b1[0], b1[1]);
                        mma16816(sc[mt][3], qf[mt][k], b1[2], b1[3]);
                    }
                }
            }
            float* rd = red + kq * ROWS * RS + kg * 32 + fc;
#pragma unroll
            for (int mt = 0; mt < 2; ++mt)
#pragma unroll
                for (int n = 0; n < 4; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        *reinterpret_cast<float2*>(rd + (mt * 16 + fr + 8 * e) * RS + n * 8) =
                            make_float2(sc[mt][n][2 * e], sc[mt][n][2 * e + 1]);
        }
        __syncthreads();
        // ---- the owned row: keys 4 (lane % 8) .. + 3 and 32 more
        {
            float v[8];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float* src = red + own * RS + u * 32 + (lane & 7) * 4;
                float4 x = *reinterpret_cast<const float4*>(src);
#pragma unroll
                for (int q = 1; q < 4; ++q) {
                    const float4 y = *reinterpret_cast<const float4*>(src + q * ROWS * RS);
                    x.x += y.x;
                    x.y += y.y;
                    x.z += y.z;
                    x.w += y.w;
                }
                v[4 * u] = x.x;
                v[4 * u + 1] = x.y;
                v[4 * u + 2] = x.z;
                v[4 * u + 3] = x.w;
            }
            float mn = m;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const int r = rg.lo + t * DM_KEYS + (e >> 2) * 32 + (lane & 7) * 4 + (e & 3);
                float x = dm_score<CAP>(v[e], cap_in, sl);
                if (r >= see.lo && r <= see.hi) {
                    if (brow != nullptr) {
                        int64_t d = see.origin - r;
                        if (d < 0) d += rg.wrap;
                        x = fmaf(__ldg(brow + (d < p.bias_len ? d : p.bias_len - 1)), DM_LOG2E, x);
                    }
                } else {
                    x = -INFINITY;
                }
                v[e] = x;
                mn = fmaxf(mn, x);
            }
#pragma unroll
            for (int o = 4; o >= 1; o >>= 1) mn = fmaxf(mn, __shfl_xor_sync(FULL, mn, o));
            const float mc = mn == -INFINITY ? 0.f : mn;
            const float f = mn == m ? 1.f : exp2_fast(m - mc);
            m = mn;
            l *= f;
            if ((lane & 7) == 0) f_s[own] = f;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                float w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    w[e] = exp2_fast(v[4 * u + e] - mc);
                    l += w[e];
                }
                store_vec<bf, 4>(ps + own * PS + u * 32 + (lane & 7) * 4, w);
            }
        }
        __syncthreads();
        // ---- P V: every warp all rows, its own value columns
        if (col0 < p.dv) {
            float f[2][2];
            bool any = false;
#pragma unroll
            for (int tt = 0; tt < 2; ++tt)
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    f[tt][k] = f_s[tt * 16 + fr + 8 * k];
                    any |= f[tt][k] != 1.f;
                }
            if (__any_sync(FULL, any)) {
#pragma unroll
                for (int tt = 0; tt < 2; ++tt)
#pragma unroll
                    for (int v = 0; v < NVT; ++v)
#pragma unroll
                        for (int e = 0; e < 4; ++e) acc[tt][v][e] *= f[tt][e >> 1];
            }
            const uint32_t va = saddr(vs + stage * v_panels * DM_PANEL + (lane & 15) * 128);
#pragma unroll
            for (int k = 0; k < DM_KEYS / 16; ++k) {
                uint32_t a[2][4];
#pragma unroll
                for (int tt = 0; tt < 2; ++tt) ldsm4(saddr(ps + (tt * 16 + (lane & 15)) * PS + k * 16 + (lane >> 4) * 8), a[tt]);
#pragma unroll
                for (int v = 0; v < NVT; v += 2) {
                    if (col0 + v * 8 < p.dv) {
                        uint32_t bb[4];
                        const int c = (col0 >> 3) + v + (lane >> 4);
                        ldsm4t(va + (c >> 3) * DM_PANEL + k * 2048 + (((c & 7) ^ sw) << 4), bb);
#pragma unroll
                        for (int tt = 0; tt < 2; ++tt) {
                            mma16816(acc[tt][v], a[tt], bb[0], bb[1]);
                            mma16816(acc[tt][v + 1], a[tt], bb[2], bb[3]);
                        }
                    }
                }
            }
        }
    }
    if (!in_time) {
        if (p.status != nullptr) atomicOr(p.status, SK_DEV_WAIT_TIMEOUT);
        mbar_wait_bounded(&full[(t_end - 1 - t_beg) & 1], (uint32_t)(((t_end - 1 - t_beg) >> 1) & 1));
        if (t_end - t_beg > 1) mbar_wait_bounded(&full[(t_end - t_beg) & 1], (uint32_t)(((t_end - 2 - t_beg) >> 1) & 1));
    }
    float* part = (float*)p.workspace + ((((int64_t)b * p.G + g) * groups + grp) * splits + split) * part_floats;
#pragma unroll
    for (int o = 4; o >= 1; o >>= 1) l += __shfl_xor_sync(FULL, l, o);
    if ((lane & 7) == 0) {
        part[(int64_t)ROWS * p.dv + own] = m;
        part[(int64_t)ROWS * p.dv + ROWS + own] = l;
    }
#pragma unroll
    for (int tt = 0; tt < 2; ++tt)
#pragma unroll
        for (int v = 0; v < NVT; ++v) {
            const int c = col0 + v * 8 + fc;
            if (c < p.dv) {
#pragma unroll
                for (int k = 0; k < 2; ++k)
                    *reinterpret_cast<float2*>(part + (int64_t)(tt * 16 + fr + 8 * k) * p.dv + c) =
                        make_float2(acc[tt][v][2 * k], acc[tt][v][2 * k + 1]);
            }
        }
}

// One CTA per query row and 128 value columns: merge the splits that exist, add the sink, divide.  A warp takes
// every sixteenth split, a lane four columns.
constexpr int DG_WARPS = 16, DG_COLS = 128;
__global__ void __launch_bounds__(DG_WARPS * 32)
attn_decode_merge_kernel(sk_attn_params p, int splits, int groups, int rows_per_group, size_t part_floats, int col_blocks) {
    __shared__ float w_s[DM_MAX_SPLITS];
    __shared__ float red[2][DG_WARPS];
    __shared__ float4 acc_s[DG_WARPS][32];
    const int rep = p.H / p.G, row = blockIdx.x / col_blocks, g = blockIdx.y, b = blockIdx.z, t = threadIdx.x;
    const int warp = t >> 5, lane = t & 31, c = (blockIdx.x - row * col_blocks) * DG_COLS + 4 * lane;
    const int s = row / rep, h = g * rep + row - s * rep, grp = row / rows_per_group, r = row - grp * rows_per_group;
    const float sink = p.sink != nullptr ? p.sink[h] * DM_LOG2E : -INFINITY;
    const DmRange rg = dm_range(p, splits);
    const int n = rg.tiles > 0 ? (rg.tiles + rg.per_split - 1) / rg.per_split : 0;      // <= DM_MAX_SPLITS
    const float* part = (const float*)p.workspace + (((int64_t)b * p.G + g) * groups + grp) * splits * part_floats;
    const float* stat = part + (int64_t)rows_per_group * p.dv + r;
    pdl_wait();
    float mk = -INFINITY, lk = 0.f;
    if (t < n) {
        mk = __ldcg(stat + t * part_floats);
        lk = __ldcg(stat + t * part_floats + rows_per_group);
    }
    constexpr int U = DM_MAX_SPLITS / DG_WARPS;                 // splits of a warp, all requested at once
    float4 v[U];
#pragma unroll
    for (int k = 0; k < U; ++k) {
        const int sp = warp + k * DG_WARPS;
        v[k] = sp < n && c < p.dv ? __ldcg(reinterpret_cast<const float4*>(part + sp * part_floats + (int64_t)r * p.dv + c))
                                  : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float m = fmaxf(mk, sink);
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) m = fmaxf(m, __shfl_xor_sync(FULL, m, o));
    if (lane == 0) red[0][warp] = m;
    __syncthreads();
    m = sink;
#pragma unroll
    for (int w = 0; w < DG_WARPS; ++w) m = fmaxf(m, red[0][w]);
    const float mc = m == -INFINITY ? 0.f : m;
    const float wk = exp2f(mk - mc);
    if (t < DM_MAX_SPLITS) w_s[t] = t < n ? wk : 0.f;
    const float lw = warp_sum(t < n ? wk * lk : 0.f);
    if (lane == 0) red[1][warp] = lw;
    __syncthreads();
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < U; ++k) {
        const float w = w_s[warp + k * DG_WARPS];
        a.x = fmaf(w, v[k].x, a.x);
        a.y = fmaf(w, v[k].y, a.y);
        a.z = fmaf(w, v[k].z, a.z);
        a.w = fmaf(w, v[k].w, a.w);
    }
    acc_s[warp][lane] = a;
    __syncthreads();
    if (warp == 0 && c < p.dv) {
        float l = exp2f(sink - mc), o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int w = 0; w < DG_WARPS; ++w) {
            const float4 x = acc_s[w][lane];
            l += red[1][w];
            o[0] += x.x;
            o[1] += x.y;
            o[2] += x.z;
            o[3] += x.w;
        }
        const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] *= inv;
        store_vec<__nv_bfloat16, 4>((__nv_bfloat16*)p.out + (int64_t)b * p.o_bs + (int64_t)s * p.o_ss + (int64_t)h * p.o_hs + c, o);
    }
}

template <bool CAP>
int launch_splits(const sk_attn_params& p, const DmPlan& d, const CUtensorMap& mk, const CUtensorMap& mv, dim3 grid, cudaStream_t st) {
#define SK_DM(kernel, ...)                                                                                               \
    do {                                                                                                                 \
        auto kern = kernel;                                                                                              \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)d.smem);      \
        if (e != cudaSuccess) return fail(SK_ERR_CUDA, "attn_decode kernel smem attribute: %s", cudaGetErrorString(e));  \
        kern<<<grid, DM_WARPS * 32, d.smem, st>>>(mk, mv, p, d.splits, d.groups, d.np, d.nvp, d.k_off, __VA_ARGS__);     \
    } while (0)
#define SK_DM_WIDE(KS)                                                                                    \
    do {                                                                                                  \
        if (d.nvt == 2) SK_DM((attn_decode_wide_kernel<KS, 2, CAP>), d.part_floats);                           \
        else if (d.nvt == 4) SK_DM((attn_decode_wide_kernel<KS, 4, CAP>), d.part_floats);                      \
        else SK_DM((attn_decode_wide_kernel<KS, 8, CAP>), d.part_floats);                                      \
    } while (0)
    if (d.mt == 1) {
        if (d.nvt == 2) SK_DM((attn_decode_kernel<2, CAP>), d.q_stride, d.part_floats);
        else if (d.nvt == 4) SK_DM((attn_decode_kernel<4, CAP>), d.q_stride, d.part_floats);
        else SK_DM((attn_decode_kernel<8, CAP>), d.q_stride, d.part_floats);
    } else if (p.dqk <= 256) {
        SK_DM_WIDE(4);
    } else {
        SK_DM_WIDE(10);
    }
#undef SK_DM_WIDE
#undef SK_DM
    return check_launch("attn_decode_kernel");
}

}  // namespace

bool attn_decode_mma_applicable(const sk_attn_params& p) {
    DmPlan d;
    return dm_plan(p, &d) && head_map_ok(p.q, p.dqk, p.q_hs, p.q_ss, p.q_bs) && head_map_ok(p.k, p.dqk, p.k_hs, p.k_ts, p.k_bs) &&
           head_map_ok(p.v, p.dv, p.v_hs, p.v_ts, p.v_bs) && head_map_ok(p.out, p.dv, p.o_hs, p.o_ss, p.o_bs);
}

size_t attn_decode_mma_workspace(const sk_attn_params& p) {
    DmPlan d;
    if (!dm_plan(p, &d)) return 0;
    return (size_t)p.B * p.G * d.groups * d.splits * d.part_floats * sizeof(float);
}

int launch_attn_decode_mma(const sk_attn_params& p, cudaStream_t st) {
    DmPlan d;
    if (!dm_plan(p, &d)) return fail(SK_ERR_UNSUPPORTED, "skb_attn: shape outside the decode kernel");
    CUtensorMap mk, mv;
    if (int rc = make_head_map(&mk, d.shared_v ? p.v : p.k, d.k_off + p.dqk, p.G, p.kv_rows, p.B, p.k_hs, p.k_ts, p.k_bs, DM_KEYS)) return rc;
    if (int rc = make_head_map(&mv, p.v, p.dv, p.G, p.kv_rows, p.B, p.v_hs, p.v_ts, p.v_bs, DM_KEYS)) return rc;
    dim3 grid((unsigned)d.splits, (unsigned)(p.G * d.groups), (unsigned)p.B);
    const int rc_split = p.softcap > 0.f ? launch_splits<true>(p, d, mk, mv, grid, st) : launch_splits<false>(p, d, mk, mv, grid, st);
    if (rc_split != SK_OK) return rc_split;
    const int col_blocks = (p.dv + DG_COLS - 1) / DG_COLS;
    const cudaError_t e = launch_after(attn_decode_merge_kernel, dim3((unsigned)(p.S * (p.H / p.G) * col_blocks), (unsigned)p.G, (unsigned)p.B),
                                       dim3(DG_WARPS * 32), 0, st, p, d.splits, d.groups, 16 * d.mt, d.part_floats, col_blocks);
    if (e != cudaSuccess) return fail(SK_ERR_CUDA, "attn_decode_merge_kernel: %s", cudaGetErrorString(e));
    return SK_OK;
}

}  // namespace sk
