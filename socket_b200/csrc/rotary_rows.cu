// Queries and cache rows of attention whose values are its unrotated keys.  A cache row holds a key as
// projected, followed by its turned elements: the value is the row's first `dim` elements, the key the
// `dim` elements behind the first rot_dims, and the two share everything that is not turned.  Queries get
// the keys' element order, [unturned | turned].
#include "blocks.cuh"

namespace sk {
namespace {

constexpr int RR_THREADS = 256;

// One CTA per row: the first `prev` rows of a sequence come out of the ring, the others are its new tokens.
template <typename T, int V>
__global__ void __launch_bounds__(RR_THREADS)
rotary_rows_kernel(const sk_rotary_rows_params p) {
    const int row = blockIdx.x, b = blockIdx.y, t = threadIdx.x;
    const int rot = p.rot_dims, half = rot / 2, rest = p.dim - rot, hrow = p.dim + rot;
    const int64_t first = first_position(p.pos, p.start);
    T* rows = (T*)p.rows_out + (int64_t)b * p.rows_cap * p.G * hrow;
    if (row < p.prev) {
        const int64_t slot = (first - p.prev + row) % p.ring_rows;
        const T* src = (const T*)p.ring + ((int64_t)b * p.ring_rows + slot) * p.G * hrow;
        for (int i = t * V; i < p.G * hrow; i += RR_THREADS * V) {
            float r[V];
            load_vec<T, V>(src + i, r);
            store_vec<T, V>(rows + (int64_t)row * p.G * hrow + i, r);
        }
        return;
    }
    const int s = row - p.prev;
    const int64_t i = first + s;
    if (i < 0 || i >= p.n_pos) {                             // beyond the angles and the cache: flagged, not written
        if (t == 0 && p.status != nullptr) atomicOr(p.status, SK_DEV_POS_OUT_OF_RANGE);
        return;
    }
    T* dst_row = rows + (p.pos != nullptr ? i % p.rows_cap : row) * p.G * hrow;
    const int64_t in = ((int64_t)b * p.S + s) * p.in_ld;
    const float* cs = p.angles + i * rot;                    // [half][cos, sin]
    const int n_rest = rest / V, per = n_rest + half / V;    // vectors of a head: unturned ones, then pairs
    for (int item = t; item < (p.H + p.G) * per; item += RR_THREADS) {
        const int head = item / per, j = item - head * per;
        const bool key = head >= p.H;
        const T* src = key ? (const T*)p.k_in + in + (int64_t)(head - p.H) * p.dim : (const T*)p.q_in + in + (int64_t)head * p.dim;
        // turned elements follow the unturned ones; a key's row starts with its turned ones as projected
        T* dst = key ? dst_row + (int64_t)(head - p.H) * hrow + rot
                     : (T*)p.q_out + (((int64_t)b * p.S + s) * p.H + head) * p.dim;
        if (j < n_rest) {
            float r[V];
            load_vec<T, V>(src + rot + j * V, r);
            store_vec<T, V>(dst + j * V, r);
        } else {
            const int k = (j - n_rest) * V;
            float u[V], v[V], x[V], y[V];
            load_vec<T, V>(src + k, u);
            load_vec<T, V>(src + half + k, v);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                const float c = cs[2 * (k + e)], sn = cs[2 * (k + e) + 1];
                x[e] = u[e] * c - v[e] * sn;
                y[e] = v[e] * c + u[e] * sn;
            }
            store_vec<T, V>(dst + rest + k, x);
            store_vec<T, V>(dst + rest + half + k, y);
            if (key) {
                store_vec<T, V>(dst - rot + k, u);
                store_vec<T, V>(dst - rot + half + k, v);
            }
        }
    }
}

}  // namespace

int launch_rotary_rows(const sk_rotary_rows_params& p, cudaStream_t st) {
    const size_t es = p.dtype == SK_BF16 ? 2 : 4;
    auto vec = [&](int v) {
        return p.dim % v == 0 && (p.rot_dims / 2) % v == 0 && p.in_ld % v == 0 &&
               ((uintptr_t)p.q_in | (uintptr_t)p.k_in | (uintptr_t)p.ring | (uintptr_t)p.q_out | (uintptr_t)p.rows_out) % (v * es) == 0;
    };
    dim3 grid((unsigned)(p.prev + p.S), (unsigned)p.B);
#define SK_RR(T, V) rotary_rows_kernel<T, V><<<grid, RR_THREADS, 0, st>>>(p)
    if (p.dtype == SK_BF16) {
        if (vec(8)) SK_RR(__nv_bfloat16, 8);
        else if (vec(4)) SK_RR(__nv_bfloat16, 4);
        else SK_RR(__nv_bfloat16, 1);
    } else {
        if (vec(4)) SK_RR(float, 4);
        else SK_RR(float, 1);
    }
#undef SK_RR
    return check_launch("rotary_rows_kernel");
}

}  // namespace sk
