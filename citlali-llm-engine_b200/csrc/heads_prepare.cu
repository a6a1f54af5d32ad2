// From a row's projections q | k | v to what attention reads, in one pass:
//
//   * a bias a channel (optional);
//   * an RMS norm over all of q at once and over all of k at once, ahead of the split into heads, each with a weight of its
//     own size (optional);
//   * the rotation of the first rot_dims elements of every q and k head by position * inv_freq[i], element i with element
//     i + rot_dims / 2 (halves) or 2i with 2i + 1 (pairs), cosine and sine times `amplitude`;
//   * the rotation of every v head over its whole length by position * v_freq[m] (optional), halves or pairs;
//   * q to a buffer, k and v to the row's place in the paged cache.
// With v_freq the row's cosines and sines go to turns [rows, vd / 2] (cos, sin), from which the attention kernels turn their
// output back.  Everything is float32 until the one rounding at the store.
//
// With maps > 1 a head of d elements is `maps` equal parts that score on their own (the maps of differential attention): each
// part is rotated by itself, and a query head becomes `maps` heads of d whose other parts are zeros, so that one key of d
// elements serves them all.
//
// One block a row, its size given by the projections' width alone (so are the orders of the sums).
#include "api.h"
#include "common.cuh"

namespace citlali {
namespace {

template <typename T, int N>
__device__ __forceinline__ void put(T* p, const float (&v)[N]) {
    if constexpr (N == 4 && sizeof(T) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    } else if constexpr (N == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        stf(p, 0, v[0]);
    }
}
template <int N>
__device__ __forceinline__ void get(const float* __restrict__ p, float (&v)[N]) {
    if constexpr (N == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
        v[0] = p[0];
    }
}

struct HeadsArgs {
    const float* proj;
    size_t proj_stride;
    const float *bias, *q_gain, *k_gain, *inv_freq, *v_freq;
    const int32_t *row_slot, *row_pos, *page_table;
    float2* turns;
    int rot_dims, rot_pairs, v_pairs, table_stride, page_size, nq, nkv, d, vd, maps;
    float amplitude, eps;
};

// N elements of a row at a time: 4 where sizes and addresses allow, else 1.
template <typename T, typename TQ, int N>
__global__ void __launch_bounds__(512)
heads_prepare_kernel(HeadsArgs a, T* __restrict__ k_pool, T* __restrict__ v_pool, TQ* __restrict__ q_out) {
    extern __shared__ float2 trig[];                          // [rot_dims / 2] of q and k, then [vd / 2] of v
    __shared__ float2 scratch[32];
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x, pos = a.row_pos[row], slot = a.row_slot[row];
    const int half = a.rot_dims / 2, vhalf = a.v_freq ? a.vd / 2 : 0;
    for (int i = threadIdx.x; i < half + vhalf; i += blockDim.x) {
        const bool is_v = i >= half;
        float sn, cs;
        sincosf((float)pos * (is_v ? a.v_freq[i - half] : a.inv_freq[i]), &sn, &cs);
        if (is_v) a.turns[(size_t)row * vhalf + i - half] = make_float2(cs, sn);
        trig[i] = is_v ? make_float2(cs, sn) : make_float2(cs * a.amplitude, sn * a.amplitude);
    }
    const float* x = a.proj + (size_t)row * a.proj_stride;
    const int Cq = a.nq * a.d, Ck = a.nkv * a.d, Cv = a.nkv * a.vd, dm = a.d / a.maps;
    float q_inv = 1.0f, k_inv = 1.0f;
    if (a.q_gain) {
        float sq = 0.0f, sk = 0.0f;
#pragma unroll 4
        for (int c = threadIdx.x * N; c < Cq + Ck; c += blockDim.x * N) {
            float v[N], b[N];
            get<N>(x + c, v);
            if (a.bias) {
                get<N>(a.bias + c, b);
#pragma unroll
                for (int e = 0; e < N; ++e) v[e] += b[e];
            }
            float s = 0.0f;
#pragma unroll
            for (int e = 0; e < N; ++e) s = fmaf(v[e], v[e], s);
            if (c < Cq) sq += s; else sk += s;
        }
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) scratch[warp] = make_float2(sq, sk);
        __syncthreads();
        const float2 part = lane < (blockDim.x >> 5) ? scratch[lane] : make_float2(0.0f, 0.0f);
        q_inv = 1.0f / sqrtf(warp_sum(part.x) / (float)Cq + a.eps);
        k_inv = 1.0f / sqrtf(warp_sum(part.y) / (float)Ck + a.eps);
    }
    __syncthreads();                                          // the table of cosines and sines is complete
    const int page = a.page_table[(size_t)slot * a.table_stride + pos / a.page_size];
    const size_t cache_row = (size_t)page * a.nkv * a.page_size + pos % a.page_size;       // + head * page_size
    auto value = [&](int c, float (&v)[N]) {                  // N channels from c on, biased and normed
        get<N>(x + c, v);
        if (a.bias) {
            float b[N];
            get<N>(a.bias + c, b);
#pragma unroll
            for (int e = 0; e < N; ++e) v[e] += b[e];
        }
        if (a.q_gain && c < Cq + Ck) {
            float g[N];
            get<N>(c < Cq ? a.q_gain + c : a.k_gain + c - Cq, g);
            const float inv = c < Cq ? q_inv : k_inv;
#pragma unroll
            for (int e = 0; e < N; ++e) v[e] = v[e] * inv * g[e];
        }
    };
    for (int c = threadIdx.x * N; c < Cq + Ck + Cv; c += blockDim.x * N) {
        const bool is_q = c < Cq, is_v = c >= Cq + Ck;
        const int at = is_q ? c : (is_v ? c - Cq - Ck : c - Cq);
        const int n = is_v ? a.vd : a.d;
        const int head = at / n, in_head = at % n, i = is_v || a.maps == 1 ? in_head : in_head % dm;
        const int h = is_v ? vhalf : half;                    // pairs of the rotation
        const bool pairs = is_v ? a.v_pairs != 0 : a.rot_pairs != 0;
        const float2* t = is_v ? trig + half : trig;
        float v[N];
        value(c, v);
        if (i < 2 * h) {
            if (pairs) {
                if constexpr (N == 4) {
#pragma unroll
                    for (int e = 0; e < 4; e += 2) {
                        const float2 cs = t[(i + e) >> 1];
                        const float u = v[e], w = v[e + 1];
                        v[e] = u * cs.x - w * cs.y;
                        v[e + 1] = w * cs.x + u * cs.y;
                    }
                } else {
                    float o[N];
                    value((i & 1) ? c - 1 : c + 1, o);
                    const float2 cs = t[i >> 1];
                    v[0] = (i & 1) ? v[0] * cs.x + o[0] * cs.y : v[0] * cs.x - o[0] * cs.y;
                }
            } else {
                float o[N];
                const bool low = i < h;
                value(low ? c + h : c - h, o);
#pragma unroll
                for (int e = 0; e < N; ++e) {
                    const float2 cs = t[(low ? i : i - h) + e];
                    v[e] = low ? v[e] * cs.x - o[e] * cs.y : v[e] * cs.x + o[e] * cs.y;
                }
            }
        }
        if (is_q && a.maps > 1) {
            TQ* dst = q_out + ((size_t)row * Cq + (size_t)head * a.d) * a.maps + in_head;
            const float zeros[N] = {};
            for (int s = 0; s < a.maps; ++s)
                if (s == in_head / dm) put<TQ, N>(dst + (size_t)s * a.d, v);
                else put<TQ, N>(dst + (size_t)s * a.d, zeros);
        }
        else if (is_q) put<TQ, N>(q_out + (size_t)row * Cq + c, v);
        else if (is_v) put<T, N>(v_pool + (cache_row + (size_t)head * a.page_size) * a.vd + i, v);
        else put<T, N>(k_pool + (cache_row + (size_t)head * a.page_size) * a.d + in_head, v);
    }
}

}  // namespace
}  // namespace citlali

using namespace citlali;

extern "C" int citlali_heads_prepare(const float* proj, int proj_stride, const float* bias, const float* q_gain, const float* k_gain,
                                     float eps, const float* inv_freq, int rot_dims, int rot_pairs, float amplitude,
                                     const float* v_freq, int v_pairs, float* turns, const int32_t* row_slot,
                                     const int32_t* row_pos, const int32_t* page_table, int table_stride, void* k_pool,
                                     void* v_pool, int cache_dtype, int page_size, void* q_out, int q_dtype, int rows, int nq,
                                     int nkv, int d, int vd, int maps, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || d <= 0 || vd <= 0 || page_size <= 0 || (q_gain == nullptr) != (k_gain == nullptr)) {
        set_last_error("heads_prepare: %d query heads over %d key/value heads of %d (values %d)", nq, nkv, d, vd);
        return kBadShape;
    }
    if (maps < 1 || d % maps != 0) {
        set_last_error("heads_prepare: heads of %d do not split into %d equal parts", d, maps);
        return kBadShape;
    }
    if (rot_dims < 0 || rot_dims % 2 != 0 || rot_dims > d / maps || (rot_dims > 0 && inv_freq == nullptr) ||
        (v_freq != nullptr && (vd % 2 != 0 || turns == nullptr))) {
        set_last_error("heads_prepare: %d rotated elements must be even and at most the head size %d; rotated values (%d) need an "
                       "even size and room for their cosines", rot_dims, d, vd);
        return kBadShape;
    }
    const size_t smem = (size_t)(rot_dims / 2 + (v_freq ? vd / 2 : 0)) * sizeof(float2);
    if (smem > 48 * 1024) {
        set_last_error("heads_prepare: heads of %d (values %d) are too large", d, vd);
        return kTooLarge;
    }
    HeadsArgs a{proj, (size_t)proj_stride, bias, q_gain, k_gain, inv_freq, v_freq, row_slot, row_pos, page_table, (float2*)turns,
                rot_dims, rot_pairs, v_pairs, table_stride, page_size, nq, nkv, d, vd, maps, amplitude, eps};
    // four elements at a time: no piece crosses a head, a rotation's half or its end
    const bool vec = (d / maps) % 4 == 0 && vd % 4 == 0 && proj_stride % 4 == 0 && rot_dims % 4 == 0 && (rot_pairs || rot_dims % 8 == 0) &&
                     (v_freq == nullptr || v_pairs || vd % 8 == 0) &&
                     (((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)q_gain | (uintptr_t)k_gain | (uintptr_t)k_pool |
                       (uintptr_t)v_pool | (uintptr_t)q_out) & 15u) == 0;
    const int C = (nq + nkv) * d + nkv * vd;
    int threads = ((C / (vec ? 4 : 1) + 31) / 32) * 32;
    threads = threads < 64 ? 64 : (threads > 512 ? 512 : threads);
    return CITLALI_DISPATCH_FLOAT(cache_dtype, T, [&] {
        return CITLALI_DISPATCH_FLOAT(q_dtype, TQ, [&] {
            if (vec) launch_kernel(heads_prepare_kernel<T, TQ, 4>, rows, threads, smem, stream, a, (T*)k_pool, (T*)v_pool, (TQ*)q_out);
            else launch_kernel(heads_prepare_kernel<T, TQ, 1>, rows, threads, smem, stream, a, (T*)k_pool, (T*)v_pool, (TQ*)q_out);
            return CITLALI_LAUNCH_CHECK();
        });
    });
}
