// RMS norm over equal parts of a row, alone or with a short causal convolution over time behind it.
//
//   group_rms_norm     out[i] = norm(x[index[i]]) * w: a row of `hidden` elements is `groups` equal consecutive parts, each
//                      divided by its own sqrt(mean(part^2) + eps); then the whole row times w.
//   group_norm_conv    h = norm(x) * w as above, for every row of a step, and beside it  h + conv(h)  with
//                      conv(h)_t = sum_j taps_w[:, j] h_(t - taps + 1 + j)  per channel; tokens before the step come from
//                      what the sequence kept (its last taps - 1 rows h, float32, zero at its start).  Both results are
//                      rounded once at their store; the convolution reads the unrounded h.  A sequence that brings one token
//                      keeps its new row in the same kernel; one that brings more has it done by the kernel below.
//   group_norm_keep    every sequence that brought several tokens keeps its last taps - 1 rows h.
//
// A row's sums are taken in pieces of at most kPiece elements of a part, one warp a piece, added in piece order: the order
// depends on the row's length and the number of parts alone, never on the step.
#include "api.h"
#include "common.cuh"

namespace citlali {

constexpr int kPiece = 512;            // elements of a part one warp sums
constexpr int kNormThreads = 256;
constexpr int kWideThreads = 1024;     // at most, for kernels whose blocks have one row (or a sequence's kept rows) to themselves
constexpr int kMaxTaps = 16;


__host__ __device__ __forceinline__ int pieces_of(int part) { return (part + kPiece - 1) / kPiece; }

template <typename TE>
__device__ __forceinline__ void put4(TE* p, const float4& v) {
    if constexpr (sizeof(TE) == 2) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    } else {
        *reinterpret_cast<float4*>(p) = v;
    }
}
template <typename TG>
__device__ __forceinline__ float4 get4(const TG* p) {
    if constexpr (sizeof(TG) == 2) {
        const uint2 w = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
        return make_float4(lo.x, lo.y, hi.x, hi.y);
    } else {
        return *reinterpret_cast<const float4*>(p);
    }
}

// a b c, every product rounded (never part of a fused multiply-add: a row h is the same wherever it is formed)
__device__ __forceinline__ float rounded3(float a, float b, float c) { return __fmul_rn(__fmul_rn(a, b), c); }

// inv[r * groups + g] = 1 / sqrt(mean of squares of part g of source row r + eps) for `n` rows; `row_of(r)` names the row (below
// zero: none, inv stays unset).  `sums` holds n * groups * pieces floats.  Ends with a barrier.
template <bool VEC, typename RowOf>
__device__ __forceinline__ void inverse_roots(const float* __restrict__ x, int hidden, int groups, float eps, int n, float* sums,
                                              float* inv, RowOf row_of) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int part = hidden / groups, pieces = pieces_of(part), per_row = groups * pieces;
    if constexpr (VEC) {
        constexpr int U = 2, Q = kPiece / 128;                 // pieces in flight a warp, 16-byte words of one a lane holds
        for (int t0 = warp; t0 < n * per_row; t0 += warps * U) {
            float4 v[U][Q];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int task = t0 + u * warps;
                const int r = task / per_row, g = (task % per_row) / pieces, i0 = task % pieces * kPiece;
                const int row = task < n * per_row ? row_of(r) : -1;
                const float* src = x + (size_t)max(row, 0) * hidden + (size_t)g * part;
#pragma unroll
                for (int k = 0; k < Q; ++k) {
                    const int i = i0 + (k * 32 + lane) * 4;
                    v[u][k] = row >= 0 && i < min(part, i0 + kPiece) ? *reinterpret_cast<const float4*>(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                float ss = 0.0f;
#pragma unroll
                for (int k = 0; k < Q; ++k) {
                    ss = fmaf(v[u][k].x, v[u][k].x, ss); ss = fmaf(v[u][k].y, v[u][k].y, ss);
                    ss = fmaf(v[u][k].z, v[u][k].z, ss); ss = fmaf(v[u][k].w, v[u][k].w, ss);
                }
                ss = warp_sum(ss);
                if (lane == 0 && t0 + u * warps < n * per_row) sums[t0 + u * warps] = ss;
            }
        }
    } else {
        for (int task = warp; task < n * per_row; task += warps) {
            const int r = task / per_row, g = (task % per_row) / pieces, i0 = task % pieces * kPiece;
            const int row = row_of(r), i1 = min(part, i0 + kPiece);
            if (row < 0) continue;
            const float* src = x + (size_t)row * hidden + (size_t)g * part;
            float ss = 0.0f;
            for (int i = i0 + lane; i < i1; i += 32) ss = fmaf(src[i], src[i], ss);
            ss = warp_sum(ss);
            if (lane == 0) sums[task] = ss;
        }
    }
    __syncthreads();
    for (int t = threadIdx.x; t < n * groups; t += blockDim.x) {
        if (row_of(t / groups) < 0) continue;
        float ss = 0.0f;
        for (int p = 0; p < pieces; ++p) ss += sums[(size_t)t * pieces + p];
        inv[t] = 1.0f / sqrtf(ss / (float)part + eps);
    }
    __syncthreads();
}

template <typename TG, typename TO, bool VEC>
__global__ void __launch_bounds__(kNormThreads)
group_rms_norm_kernel(const float* __restrict__ x, const TG* __restrict__ gain, const int32_t* __restrict__ row_index,
                      TO* __restrict__ out, int hidden, int groups, float eps) {
    extern __shared__ float sm[];                              // [groups * pieces] sums, [groups] inverse roots
    dependents_may_launch();
    wait_for_predecessor();
    const int part = hidden / groups;
    float* inv = sm + groups * pieces_of(part);
    const int row = row_index ? row_index[blockIdx.x] : (int)blockIdx.x;
    inverse_roots<VEC>(x, hidden, groups, eps, 1, sm, inv, [&](int) { return row; });
    const float* src = x + (size_t)row * hidden;
    TO* dst = out + (size_t)blockIdx.x * hidden;
    if constexpr (VEC) {
        for (int c = threadIdx.x * 4; c < hidden; c += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + c), g = get4(gain + c);
            const float k = inv[c / part];
            put4(dst + c, make_float4(v.x * k * g.x, v.y * k * g.y, v.z * k * g.z, v.w * k * g.w));
        }
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) stf(dst, c, src[c] * inv[c / part] * ldf(gain, c));
    }
}

// A block takes R consecutive rows of the step and the taps - 1 rows ahead of them.
template <typename TG, typename TO, int TAPS, int R>
__global__ void __launch_bounds__(R == 1 ? kWideThreads : kNormThreads)
group_norm_conv_vec_kernel(const float* __restrict__ x, const TG* __restrict__ gain, const float* __restrict__ taps_w,
                           float* __restrict__ state, size_t state_stride, const int32_t* __restrict__ row_slot,
                           TO* __restrict__ h_out, TO* __restrict__ c_out, int rows, int hidden, int groups, float eps) {
    extern __shared__ float sm[];
    dependents_may_launch();
    wait_for_predecessor();
    constexpr int BACK = TAPS - 1;
    const int part = hidden / groups, per = groups * pieces_of(part);
    float* inv = sm + (size_t)(R + BACK) * per;                // local row r stands for row r0 - before + r
    const int r0 = blockIdx.x * R, nr = min(R, rows - r0);
    int before = 0;                                            // rows ahead of r0 that belong to its sequence
    while (before < BACK && r0 - before - 1 >= 0 && row_slot[r0 - before - 1] == row_slot[r0]) ++before;
    inverse_roots<true>(x, hidden, groups, eps, before + nr, sm, inv, [&](int r) { return r0 - before + r; });
    for (int c = threadIdx.x * 4; c < hidden; c += blockDim.x * 4) {
        const float4 g = get4(gain + c);
        const int grp = c / part;
        float4 w[TAPS];                                        // w[j]: tap j of the four channels
        {
            float t[4 * TAPS];
#pragma unroll
            for (int i = 0; i < TAPS; ++i) {
                const float4 v = *reinterpret_cast<const float4*>(taps_w + (size_t)c * TAPS + 4 * i);
                t[4 * i] = v.x; t[4 * i + 1] = v.y; t[4 * i + 2] = v.z; t[4 * i + 3] = v.w;
            }
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = make_float4(t[j], t[TAPS + j], t[2 * TAPS + j], t[3 * TAPS + j]);
        }
        float4 own[R];                                         // the block's rows, fetched before any of them is used
#pragma unroll
        for (int k = 0; k < R; ++k)
            own[k] = k < nr ? *reinterpret_cast<const float4*>(x + (size_t)(r0 + k) * hidden + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        auto scaled = [&](const float4& v, int local) {
            const float k = inv[local * groups + grp];
            return make_float4(rounded3(v.x, k, g.x), rounded3(v.y, k, g.y), rounded3(v.z, k, g.z), rounded3(v.w, k, g.w));
        };
        float4 hist[BACK];                                     // the rows ahead, oldest first
        const int slot = row_slot[r0];
#pragma unroll
        for (int i = 0; i < BACK; ++i) {
            const int back = BACK - i;
            if (back <= before) hist[i] = scaled(*reinterpret_cast<const float4*>(x + (size_t)(r0 - back) * hidden + c), before - back);
            else hist[i] = *reinterpret_cast<const float4*>(state + (size_t)slot * state_stride + (size_t)(i + before) * hidden + c);
        }
#pragma unroll
        for (int k = 0; k < R; ++k) {
            if (k >= nr) break;
            const int r = r0 + k;
            const int s = row_slot[r];
            const bool starts = r == 0 || row_slot[r - 1] != s;
            const bool ends = r + 1 == rows || row_slot[r + 1] != s;
            float* kept = state + (size_t)s * state_stride + c;
            if (starts && k != 0) {
#pragma unroll
                for (int i = 0; i < BACK; ++i) hist[i] = *reinterpret_cast<const float4*>(kept + (size_t)i * hidden);
            }
            const float4 h = scaled(own[k], before + k);
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < BACK; ++i) {
                a.x = fmaf(w[i].x, hist[i].x, a.x); a.y = fmaf(w[i].y, hist[i].y, a.y);
                a.z = fmaf(w[i].z, hist[i].z, a.z); a.w = fmaf(w[i].w, hist[i].w, a.w);
            }
            a.x = fmaf(w[BACK].x, h.x, a.x); a.y = fmaf(w[BACK].y, h.y, a.y);
            a.z = fmaf(w[BACK].z, h.z, a.z); a.w = fmaf(w[BACK].w, h.w, a.w);
            put4(h_out + (size_t)r * hidden + c, h);
            put4(c_out + (size_t)r * hidden + c, make_float4(h.x + a.x, h.y + a.y, h.z + a.z, h.w + a.w));
#pragma unroll
            for (int i = 0; i + 1 < BACK; ++i) hist[i] = hist[i + 1];
            hist[BACK - 1] = h;
            if (starts && ends) {                              // a single new token: what is kept moves on by one row
#pragma unroll
                for (int i = 0; i < BACK; ++i) *reinterpret_cast<float4*>(kept + (size_t)i * hidden) = hist[i];
            }
        }
    }
}

// Any number of taps and any row length: a block a row.
template <typename TG, typename TO>
__global__ void __launch_bounds__(kNormThreads)
group_norm_conv_kernel(const float* __restrict__ x, const TG* __restrict__ gain, const float* __restrict__ taps_w, int taps,
                       float* __restrict__ state, size_t state_stride, const int32_t* __restrict__ row_slot,
                       TO* __restrict__ h_out, TO* __restrict__ c_out, int rows, int hidden, int groups, float eps) {
    extern __shared__ float sm[];
    dependents_may_launch();
    wait_for_predecessor();
    const int back_rows = taps - 1;
    const int part = hidden / groups, per = groups * pieces_of(part);
    float* inv = sm + (size_t)taps * per;
    const int row = blockIdx.x, slot = row_slot[row];
    int before = 0;
    while (before < back_rows && row - before - 1 >= 0 && row_slot[row - before - 1] == slot) ++before;
    const bool alone = (row == 0 || row_slot[row - 1] != slot) && (row + 1 == rows || row_slot[row + 1] != slot);
    inverse_roots<false>(x, hidden, groups, eps, taps, sm, inv, [&](int r) { return r >= back_rows - before ? row - back_rows + r : -1; });
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const int grp = c / part;
        const float g = ldf(gain, c);
        float* kept = state ? state + (size_t)slot * state_stride + c : nullptr;
        float a = 0.0f, h = 0.0f;
        for (int j = 0; j < taps; ++j) {
            const int back = back_rows - j;
            float v;
            if (back <= before) v = rounded3(x[(size_t)(row - back) * hidden + c], inv[j * groups + grp], g);
            else v = kept[(size_t)(j + before) * hidden];
            a = fmaf(taps_w[(size_t)c * taps + j], v, a);
            h = v;                                             // the last one is the row itself
        }
        stf(h_out, (size_t)row * hidden + c, h);
        stf(c_out, (size_t)row * hidden + c, h + a);
        if (alone && back_rows > 0) {
            for (int i = 0; i + 1 < back_rows; ++i) kept[(size_t)i * hidden] = kept[(size_t)(i + 1) * hidden];
            kept[(size_t)(back_rows - 1) * hidden] = h;
        }
    }
}

// Sequences of several new tokens: the last taps - 1 rows h (older ones move up where the step brought fewer).
template <typename TG, bool VEC>
__global__ void __launch_bounds__(kWideThreads)
group_norm_keep_kernel(const float* __restrict__ x, const TG* __restrict__ gain, int taps, float* __restrict__ state,
                       size_t state_stride, const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot, int hidden,
                       int groups, float eps) {
    extern __shared__ float sm[];
    dependents_may_launch();
    wait_for_predecessor();
    const int keep = taps - 1;
    const int part = hidden / groups, per = groups * pieces_of(part);
    float* inv = sm + (size_t)keep * per;
    const int end = seq_start[blockIdx.x + 1], n = end - seq_start[blockIdx.x];
    if (n < 2) return;                                         // the kernel ahead did it
    const int fresh = min(n, keep), old = keep - fresh;
    inverse_roots<VEC>(x, hidden, groups, eps, fresh, sm, inv, [&](int r) { return end - fresh + r; });
    float* base = state + (size_t)seq_slot[blockIdx.x] * state_stride;
    if constexpr (VEC) {
        for (int c = threadIdx.x * 4; c < hidden; c += blockDim.x * 4) {
            const float4 g = get4(gain + c);
            for (int i = 0; i < old; ++i)
                *reinterpret_cast<float4*>(base + (size_t)i * hidden + c) = *reinterpret_cast<const float4*>(base + (size_t)(i + fresh) * hidden + c);
#pragma unroll 4
            for (int i = 0; i < fresh; ++i) {
                const float4 v = *reinterpret_cast<const float4*>(x + (size_t)(end - fresh + i) * hidden + c);
                const float k = inv[i * groups + c / part];
                *reinterpret_cast<float4*>(base + (size_t)(old + i) * hidden + c) =
                    make_float4(rounded3(v.x, k, g.x), rounded3(v.y, k, g.y), rounded3(v.z, k, g.z), rounded3(v.w, k, g.w));
            }
        }
        return;
    }
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float g = ldf(gain, c);
        for (int i = 0; i < old; ++i) base[(size_t)i * hidden + c] = base[(size_t)(i + fresh) * hidden + c];
        for (int i = 0; i < fresh; ++i)
            base[(size_t)(old + i) * hidden + c] = 
                rounded3(x[(size_t)(end - fresh + i) * hidden + c], inv[i * groups + c / part], g);
    }
}

static bool group_shape_ok(const char* what, int hidden, int groups, int rows_at_once) {
    if (hidden <= 0 || groups <= 0 || hidden % groups != 0) {
        set_last_error("%s: a row of %d does not split into %d equal parts", what, hidden, groups);
        return false;
    }
    if ((size_t)rows_at_once * groups * (pieces_of(hidden / groups) + 1) * sizeof(float) > 48 * 1024) {
        set_last_error("%s: %d parts of a row of %d, %d rows at once, need more than 48 KB of sums", what, groups, hidden, rows_at_once);
        return false;
    }
    return true;
}
static size_t group_smem(int hidden, int groups, int rows) {
    return (size_t)rows * groups * (pieces_of(hidden / groups) + 1) * sizeof(float);
}
static int wide_threads(int hidden) {
    const int t = (hidden / 4 + 31) / 32 * 32;
    return t < 64 ? 64 : (t > kWideThreads ? kWideThreads : t);
}
static bool group_vec_ok(int hidden, int groups, const void* a, const void* b, const void* c, const void* d) {
    return (hidden / groups) % 4 == 0 && (((uintptr_t)a | (uintptr_t)b | (uintptr_t)c | (uintptr_t)d) & 15u) == 0;
}

}  // namespace citlali

using namespace citlali;

extern "C" int citlali_group_rms_norm(const float* x, const void* gain, int gain_dtype, const int32_t* row_index, void* out,
                                      int out_dtype, int rows, int hidden, int groups, float eps, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (!group_shape_ok("group_rms_norm", hidden, groups, 1)) return kBadShape;
    const bool vec = group_vec_ok(hidden, groups, x, gain, out, nullptr);
    const size_t smem = group_smem(hidden, groups, 1);
    return CITLALI_DISPATCH_FLOAT(gain_dtype, TG, [&] {
        return CITLALI_DISPATCH_FLOAT(out_dtype, TO, [&] {
            if (vec) launch_kernel(group_rms_norm_kernel<TG, TO, true>, rows, kNormThreads, smem, stream, x, (const TG*)gain, row_index, (TO*)out, hidden, groups, eps);
            else launch_kernel(group_rms_norm_kernel<TG, TO, false>, rows, kNormThreads, smem, stream, x, (const TG*)gain, row_index, (TO*)out, hidden, groups, eps);
            return CITLALI_LAUNCH_CHECK();
        });
    });
}

extern "C" int citlali_group_norm_conv(const float* x, const void* gain, int gain_dtype, const float* taps_w, int taps, float* state,
                                       size_t state_stride, const int32_t* row_slot, const int32_t* seq_start,
                                       const int32_t* seq_slot, int sequences, void* h_out, void* c_out, int out_dtype, int rows,
                                       int hidden, int groups, float eps, int single_tokens, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (taps < 1 || taps > kMaxTaps || (taps > 1 && (state == nullptr || state_stride < (size_t)(taps - 1) * hidden))) {
        set_last_error("group_norm_conv: %d taps (1 to %d; more than one need a region for the rows a sequence keeps)", taps, kMaxTaps);
        return kBadShape;
    }
    // rows a block takes: several where the step has many (the rows ahead are normed once more by every block)
    const bool many = rows > 4 * device_sm_count();
    if (!group_shape_ok("group_norm_conv", hidden, groups, 8 + taps)) return kBadShape;
    const bool vec = taps >= 2 && taps <= 4 && group_vec_ok(hidden, groups, x, gain, h_out, c_out) && ((uintptr_t)taps_w & 15u) == 0 &&
                     ((uintptr_t)state & 15u) == 0 && state_stride % 4 == 0;
    const int code = CITLALI_DISPATCH_FLOAT(gain_dtype, TG, [&] {
        return CITLALI_DISPATCH_FLOAT(out_dtype, TO, [&] {
            if (vec) {
                auto go = [&](auto kernel, int R) {
                    launch_kernel(kernel, (rows + R - 1) / R, R == 1 ? wide_threads(hidden) : kNormThreads, group_smem(hidden, groups, R + taps - 1), stream, x, (const TG*)gain,
                                  taps_w, state, state_stride, row_slot, (TO*)h_out, (TO*)c_out, rows, hidden, groups, eps);
                };
                if (taps == 2) many ? go(group_norm_conv_vec_kernel<TG, TO, 2, 8>, 8) : go(group_norm_conv_vec_kernel<TG, TO, 2, 1>, 1);
                else if (taps == 3) many ? go(group_norm_conv_vec_kernel<TG, TO, 3, 8>, 8) : go(group_norm_conv_vec_kernel<TG, TO, 3, 1>, 1);
                else many ? go(group_norm_conv_vec_kernel<TG, TO, 4, 8>, 8) : go(group_norm_conv_vec_kernel<TG, TO, 4, 1>, 1);
            } else {
                launch_kernel(group_norm_conv_kernel<TG, TO>, rows, kNormThreads, group_smem(hidden, groups, taps), stream, x, (const TG*)gain,
                              taps_w, taps, state, state_stride, row_slot, (TO*)h_out, (TO*)c_out, rows, hidden, groups, eps);
            }
            return CITLALI_LAUNCH_CHECK();
        });
    });
    if (code != 0 || taps == 1 || single_tokens) return code;
    const size_t smem = group_smem(hidden, groups, taps - 1);
    return CITLALI_DISPATCH_FLOAT(gain_dtype, TG, [&] {
        if (vec) launch_kernel(group_norm_keep_kernel<TG, true>, sequences, wide_threads(hidden), smem, stream, x, (const TG*)gain, taps, state, state_stride, seq_start, seq_slot, hidden, groups, eps);
        else launch_kernel(group_norm_keep_kernel<TG, false>, sequences, kNormThreads, smem, stream, x, (const TG*)gain, taps, state, state_stride, seq_start, seq_slot, hidden, groups, eps);
        return CITLALI_LAUNCH_CHECK();
    });
}
