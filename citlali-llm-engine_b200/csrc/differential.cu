// The output stage of differential attention: per row and head, of two maps' results a1, a2 over the same values,
//   o = a1 - lambda a2;   o / sqrt(mean(o^2) + eps) * factor * sigmoid(gate of the head), rounded once.
// One warp a (row, head); the results stay in registers between the sum of squares and the store.
#include "api.h"
#include "common.cuh"

namespace citlali {
namespace {

constexpr int kPerLane = 8;                                   // head sizes up to 256

// VEC: two times four neighbouring elements a lane (sizes that are multiples of four, 16-byte rows).
template <typename TO, bool VEC>
__global__ void __launch_bounds__(256)
differential_output_kernel(const float* __restrict__ a, float lambda, float factor, float eps, const float* __restrict__ gate,
                           size_t gate_stride, TO* __restrict__ out, int H, int V) {
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (h >= H) return;
    const float* a1 = a + ((size_t)row * 2 * H + 2 * h) * V;
    const float* a2 = a1 + V;
    float o[kPerLane];
    float ss = 0.0f;
    auto element = [&](int j) { return VEC ? (j >> 2) * 128 + 4 * lane + (j & 3) : j * 32 + lane; };
#pragma unroll
    for (int j = 0; j < kPerLane; j += 4) {
        if constexpr (VEC) {
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f), y = x;
            if (element(j) < V) {
                x = *reinterpret_cast<const float4*>(a1 + element(j));
                y = *reinterpret_cast<const float4*>(a2 + element(j));
            }
            o[j] = fmaf(-lambda, y.x, x.x); o[j + 1] = fmaf(-lambda, y.y, x.y);
            o[j + 2] = fmaf(-lambda, y.z, x.z); o[j + 3] = fmaf(-lambda, y.w, x.w);
        } else {
#pragma unroll
            for (int e = j; e < j + 4; ++e) o[e] = element(e) < V ? fmaf(-lambda, a2[element(e)], a1[element(e)]) : 0.0f;
        }
#pragma unroll
        for (int e = j; e < j + 4; ++e) ss = fmaf(o[e], o[e], ss);
    }
    ss = warp_sum(ss);
    float f = factor / sqrtf(ss / (float)V + eps);
    if (gate) f *= 1.0f / (1.0f + expf(-gate[(size_t)row * gate_stride + h]));
    TO* dst = out + ((size_t)row * H + h) * V;
#pragma unroll
    for (int j = 0; j < kPerLane; j += 4) {
        if constexpr (VEC) {
            if (element(j) >= V) continue;
            if constexpr (sizeof(TO) == 2) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(o[j] * f, o[j + 1] * f), hi = __floats2bfloat162_rn(o[j + 2] * f, o[j + 3] * f);
                *reinterpret_cast<uint2*>(dst + element(j)) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                *reinterpret_cast<float4*>(dst + element(j)) = make_float4(o[j] * f, o[j + 1] * f, o[j + 2] * f, o[j + 3] * f);
            }
        } else {
#pragma unroll
            for (int e = j; e < j + 4; ++e)
                if (element(e) < V) stf(dst, element(e), o[e] * f);
        }
    }
}

}  // namespace
}  // namespace citlali

using namespace citlali;

extern "C" int citlali_differential_output(const float* a, float lambda, float factor, float eps, const float* gate,
                                           size_t gate_stride, void* out, int out_dtype, int rows, int H, int V,
                                           cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (H <= 0 || V <= 0 || V > 32 * kPerLane || (H + 7) / 8 > 65535) {
        set_last_error("differential_output: %d heads of %d (at most %d)", H, V, 32 * kPerLane);
        return kBadShape;
    }
    const bool vec = V % 4 == 0 && (((uintptr_t)a | (uintptr_t)out) & 15u) == 0;
    const dim3 grid(rows, (H + 7) / 8);
    const int threads = H < 8 ? 32 * H : 256;
    return CITLALI_DISPATCH_FLOAT(out_dtype, TO, [&] {
        if (vec) launch_kernel(differential_output_kernel<TO, true>, grid, threads, 0, stream, a, lambda, factor, eps, gate, gate_stride, (TO*)out, H, V);
        else launch_kernel(differential_output_kernel<TO, false>, grid, threads, 0, stream, a, lambda, factor, eps, gate, gate_stride, (TO*)out, H, V);
        return CITLALI_LAUNCH_CHECK();
    });
}
