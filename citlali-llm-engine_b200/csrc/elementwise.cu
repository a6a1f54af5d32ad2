// Row-wise kernels: embedding gather, RMSNorm, the SiLU gate.  One implementation serves
// the 32-bit path and the bfloat16 path; only storage types differ.
#include "api.h"
#include "common.cuh"

#include <cstdarg>
#include <cstdio>

namespace citlali {

static thread_local char g_last_error[512] = "";
static bool g_dependent_launch = true;

bool dependent_launch_enabled() { return g_dependent_launch; }

void set_last_error(const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_last_error, sizeof(g_last_error), fmt, ap);
    va_end(ap);
}

// x = E[token] * scale; the reference copies the row with no scaling (embed_kernel, kernels.cu:27-35),
// which is scale = 1 (a product with 1.0f changes no bit).
// A token outside the vocabulary is not read: the row is zeroed and the flag is raised.
template <typename TW>
__global__ void embed_rows_kernel(const TW* __restrict__ table, const int32_t* __restrict__ tokens,
                                  float* __restrict__ out, int hidden, int vocab, float scale, int32_t* error_flag,
                                  int copies, size_t copy_stride) {
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x;
    const int tok = tokens[row];
    const bool ok = tok >= 0 && tok < vocab;
    if (!ok && threadIdx.x == 0 && error_flag) atomicExch(error_flag, 1);
    const TW* src = table + (size_t)(ok ? tok : 0) * hidden;
    float* dst = out + (size_t)row * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = ok ? ldf(src, i) * scale : 0.0f;
        for (int c = 0; c < copies; ++c) dst[c * copy_stride + i] = v;         // every residual stream starts as this row
    }
}

__device__ __forceinline__ void load4_as_float(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void load4_as_float(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(w.x << 16); v[1] = __uint_as_float(w.x & 0xffff0000u);
    v[2] = __uint_as_float(w.y << 16); v[3] = __uint_as_float(w.y & 0xffff0000u);
}

// x = E[token] * scale + P[row] * pair_scale with row = (previous token * mul_prev + token * mul_cur) mod buckets, and row
// `buckets` for a sequence's first token.  The token before a sequence's first row of the step is what the sequence kept
// (state[slot], read only past position 0); the block of that row leaves the sequence's last token of the step there.
template <typename TW>
__global__ void __launch_bounds__(1024)
embed_rows_paired_kernel(const TW* __restrict__ table, const TW* __restrict__ pairs,
                                         const int32_t* __restrict__ tokens, const int32_t* __restrict__ row_slot,
                                         const int32_t* __restrict__ row_pos, const int32_t* __restrict__ seq_start, int sequences,
                                         int32_t* __restrict__ state, float* __restrict__ out, int hidden, int vocab, int buckets,
                                         long long mul_prev, long long mul_cur, float scale, float pair_scale, int32_t* error_flag) {
    __shared__ int pair_row;
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x;
    const int tok = tokens[row];
    const bool ok = tok >= 0 && tok < vocab;
    if (threadIdx.x == 0) {
        if (!ok && error_flag) atomicExch(error_flag, 1);
        const int slot = row_slot[row];
        const bool starts = row == 0 || row_slot[row - 1] != slot;
        int at = buckets;
        if (row_pos[row] > 0) {
            const long long prev = starts ? state[slot] : tokens[row - 1];
            at = (int)((((prev * mul_prev + (long long)tok * mul_cur) % buckets) + buckets) % buckets);
        }
        pair_row = at;
        if (starts) {                                         // the sequence whose rows begin here
            int lo = 0, hi = sequences;
            while (hi - lo > 1) {
                const int mid = (lo + hi) / 2;
                if (seq_start[mid] <= row) lo = mid; else hi = mid;
            }
            state[slot] = tokens[seq_start[lo + 1] - 1];
        }
    }
    __syncthreads();
    const TW* src = table + (size_t)(ok ? tok : 0) * hidden;
    const TW* pair = pairs + (size_t)pair_row * hidden;
    float* dst = out + (size_t)row * hidden;
    if (hidden % 4 == 0) {                                    // rows start on 8-byte (bfloat16) or 16-byte boundaries
        for (int i = threadIdx.x * 4; i < hidden; i += blockDim.x * 4) {
            float a[4], b[4];
            load4_as_float(src + i, a);
            load4_as_float(pair + i, b);
            float4 v = make_float4(fmaf(b[0], pair_scale, a[0] * scale), fmaf(b[1], pair_scale, a[1] * scale),
                                   fmaf(b[2], pair_scale, a[2] * scale), fmaf(b[3], pair_scale, a[3] * scale));
            if (!ok) v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            *reinterpret_cast<float4*>(dst + i) = v;
        }
        return;
    }
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = ok ? fmaf(ldf(pair, i), pair_scale, ldf(src, i) * scale) : 0.0f;
}

// What a layer norm that lives in the products around it needs of rows it has not seen come out of a product: the rows
// as bfloat16 and the sums of their squares over each 32 consecutive features (see citlali_gemm_tc_normed).  One block a
// row, one warp a group of 32 features at a time.
__global__ void norm_inputs_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ rows_out,
                                   float* __restrict__ sumsq, int hidden) {
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int groups = hidden >> 5;
    for (int g = warp; g < groups; g += warps) {
        const float v = x[(size_t)row * hidden + g * 32 + lane];
        rows_out[(size_t)row * hidden + g * 32 + lane] = __float2bfloat16_rn(v);
        const float sq = warp_sum(v * v);
        if (lane == 0) sumsq[(size_t)row * groups + g] = sq;
    }
}

// x *= scale over n floats (a logit scale; the reference has none).
__global__ void scale_kernel(float* __restrict__ x, size_t n, float scale) {
    dependents_may_launch();
    wait_for_predecessor();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) x[i] *= scale;
}

// x = cap tanh(x / cap) over n floats (a soft cap on the logits), in 32-bit.
__global__ void soft_cap_kernel(float* __restrict__ x, size_t n, float cap, float inv_cap) {
    dependents_may_launch();
    wait_for_predecessor();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv_cap);
}

// out[r] = [a[r] | b[r]] (two float32 matrices of `width` columns side by side), rounded once to out's type.  VEC: four
// neighbouring columns a thread (width a multiple of four, 16-byte aligned rows).
template <typename TO, bool VEC>
__global__ void concat_rows_kernel(const float* __restrict__ a, const float* __restrict__ b, TO* __restrict__ out, size_t rows,
                                   int width) {
    dependents_may_launch();
    wait_for_predecessor();
    constexpr int PER = VEC ? 4 : 1;
    const size_t n = rows * 2 * (size_t)width / PER;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t e = i * PER, r = e / (2 * (size_t)width);
        const int c = (int)(e % (2 * (size_t)width));
        const float* src = c < width ? a + r * width + c : b + r * width + c - width;
        if constexpr (VEC) {
            const float4 v = *reinterpret_cast<const float4*>(src);
            if constexpr (sizeof(TO) == 2) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
                *reinterpret_cast<uint2*>(out + e) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                *reinterpret_cast<float4*>(out + e) = v;
            }
        } else {
            stf(out, e, src[0]);
        }
    }
}

// inv = rsqrt(sum x^2 / n + eps); y = x * inv * gain (reference: rms_norm_kernel,
// kernels.cu:73-92, which runs one block per vector; here one block per row).
template <typename TG, typename TO>
__global__ void rms_norm_kernel(const float* __restrict__ x, const TG* __restrict__ gain,
                                const int32_t* __restrict__ row_index, TO* __restrict__ out,
                                int hidden, float eps) {
    __shared__ float scratch[32];
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x;
    const float* src = x + (size_t)(row_index ? row_index[row] : row) * hidden;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = src[i];
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)hidden + eps);
    TO* dst = out + (size_t)row * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) stf(dst, i, src[i] * inv * ldf(gain, i));
}

// The same for rows of at most 8192 elements that are a multiple of 4: every thread keeps its
// part of the row in registers, so the row is read once, with 16-byte loads.
template <typename TG, typename TO>
__global__ void __launch_bounds__(256)
rms_norm_rows_kernel(const float* __restrict__ x, const TG* __restrict__ gain,
                     const int32_t* __restrict__ row_index, TO* __restrict__ out, int hidden, float eps) {
    __shared__ float scratch[32];
    dependents_may_launch();
    // the gains (weights) and the row's index (from the host) are fetched while the kernel ahead still runs
    const int row = blockIdx.x;
    const float4* src = reinterpret_cast<const float4*>(x + (size_t)(row_index ? row_index[row] : row) * hidden);
    const int quads = hidden >> 2;
    float4 g[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int q = threadIdx.x + j * 256;
        g[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (q < quads) {
            if constexpr (sizeof(TG) == 2) {
                const uint2 w = *reinterpret_cast<const uint2*>(gain + q * 4);
                const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
                const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
                g[j] = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
                g[j] = *reinterpret_cast<const float4*>(gain + q * 4);
            }
        }
    }
    wait_for_predecessor();
    float4 v[8];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int q = threadIdx.x + j * 256;
        v[j] = q < quads ? src[q] : make_float4(0.f, 0.f, 0.f, 0.f);
        ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss);
        ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)hidden + eps);
    TO* dst = out + (size_t)row * hidden;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int q = threadIdx.x + j * 256;
        if (q < quads) {
            const int i = q * 4;
            const float a = v[j].x * inv * g[j].x, b = v[j].y * inv * g[j].y;
            const float c = v[j].z * inv * g[j].z, d = v[j].w * inv * g[j].w;
            if constexpr (sizeof(TO) == 2) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
                *reinterpret_cast<uint2*>(dst + i) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
            } else {
                *reinterpret_cast<float4*>(dst + i) = make_float4(a, b, c, d);
            }
        }
    }
}

// act = g / (1 + exp(-g)) * u (reference: swiglu_kernel, kernels.cu:474-482).
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, T* __restrict__ act, int inter, int run) {
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= inter) return;
    const size_t base = (size_t)row * 2 * inter + (size_t)(i / run) * 2 * run + (i % run);
    const float g = ldf(gate_up, base);
    const float u = ldf(gate_up, base + run);
    stf(act, (size_t)row * inter + i, g / (1.0f + expf(-g)) * u);
}

}  // namespace citlali

using namespace citlali;

extern "C" const char* citlali_last_error(void) { return g_last_error; }

// 0: launch every kernel only after the one before it has finished; 1 (default): kernels may
// start early and wait on the device for their predecessor (programmatic dependent launch).
extern "C" void citlali_set_dependent_launch(int enabled) { g_dependent_launch = enabled != 0; }

extern "C" int citlali_embed_rows_copies(const void* table, int table_dtype, const int32_t* tokens, float* out,
                                         int rows, int hidden, int vocab, float scale, int32_t* error_flag, int copies,
                                         size_t copy_stride, cudaStream_t stream) {
    if (rows <= 0 || copies <= 0) return 0;
    return CITLALI_DISPATCH_FLOAT(table_dtype, TW, [&] {
        launch_kernel(embed_rows_kernel<TW>, rows, 256, 0, stream, (const TW*)table, tokens, out, hidden, vocab, scale, error_flag,
                      copies, copy_stride);
        return CITLALI_LAUNCH_CHECK();
    });
}

extern "C" int citlali_embed_rows(const void* table, int table_dtype, const int32_t* tokens, float* out,
                                  int rows, int hidden, int vocab, float scale, int32_t* error_flag, cudaStream_t stream) {
    return citlali_embed_rows_copies(table, table_dtype, tokens, out, rows, hidden, vocab, scale, error_flag, 1, 0, stream);
}

extern "C" int citlali_embed_rows_paired(const void* table, const void* pairs, int table_dtype, const int32_t* tokens,
                                         const int32_t* row_slot, const int32_t* row_pos, const int32_t* seq_start, int sequences,
                                         int32_t* state, float* out, int rows, int hidden, int vocab, int buckets,
                                         long long mul_prev, long long mul_cur, float scale, float pair_scale,
                                         int32_t* error_flag, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (buckets <= 0 || sequences <= 0 || mul_prev > (1ll << 31) || mul_cur > (1ll << 31) || mul_prev < -(1ll << 31) ||
        mul_cur < -(1ll << 31)) {
        set_last_error("embed_rows_paired: %d buckets, %d sequences, multipliers %lld and %lld (32 bits each)", buckets, sequences,
                       mul_prev, mul_cur);
        return kBadShape;
    }
    if (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) & 15u) {
        set_last_error("embed_rows_paired: the tables and the output must start on 16-byte boundaries");
        return kBadAlignment;
    }
    int threads = (hidden / 4 + 31) / 32 * 32;
    threads = threads < 64 ? 64 : (threads > 1024 ? 1024 : threads);
    return CITLALI_DISPATCH_FLOAT(table_dtype, TW, [&] {
        launch_kernel(embed_rows_paired_kernel<TW>, rows, threads, 0, stream, (const TW*)table, (const TW*)pairs, tokens, row_slot,
                      row_pos, seq_start, sequences, state, out, hidden, vocab, buckets, mul_prev, mul_cur, scale, pair_scale,
                      error_flag);
        return CITLALI_LAUNCH_CHECK();
    });
}

extern "C" int citlali_norm_inputs(const float* x, void* rows_out, float* sumsq, int rows, int hidden, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (hidden <= 0 || hidden % 32 != 0) {
        set_last_error("norm_inputs: the width %d must be a multiple of 32", hidden);
        return kBadShape;
    }
    launch_kernel(norm_inputs_kernel, rows, hidden >= 2048 ? 512 : 128, 0, stream, x, (__nv_bfloat16*)rows_out, sumsq, hidden);
    return CITLALI_LAUNCH_CHECK();
}

extern "C" int citlali_scale(float* x, size_t n, float scale, cudaStream_t stream) {
    if (n == 0) return 0;
    const size_t blocks = (n + 255) / 256;
    launch_kernel(scale_kernel, (int)(blocks < 4096 ? blocks : 4096), 256, 0, stream, x, n, scale);
    return CITLALI_LAUNCH_CHECK();
}

extern "C" int citlali_soft_cap(float* x, size_t n, float cap, cudaStream_t stream) {
    if (n == 0) return 0;
    if (!(cap > 0.0f)) {
        set_last_error("soft_cap: the cap %g must be positive", (double)cap);
        return kBadShape;
    }
    const size_t blocks = (n + 255) / 256;
    launch_kernel(soft_cap_kernel, (int)(blocks < 4096 ? blocks : 4096), 256, 0, stream, x, n, cap, 1.0f / cap);
    return CITLALI_LAUNCH_CHECK();
}

extern "C" int citlali_concat_rows(const float* a, const float* b, void* out, int out_dtype, int rows, int width,
                                   cudaStream_t stream) {
    if (rows <= 0 || width <= 0) return 0;
    const bool vec = width % 4 == 0 && (((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & 15u) == 0;
    const size_t n = (size_t)rows * 2 * width / (vec ? 4 : 1), blocks = (n + 255) / 256;
    const int grid = (int)(blocks < 8192 ? blocks : 8192);
    return CITLALI_DISPATCH_FLOAT(out_dtype, TO, [&] {
        if (vec) launch_kernel(concat_rows_kernel<TO, true>, grid, 256, 0, stream, a, b, (TO*)out, (size_t)rows, width);
        else launch_kernel(concat_rows_kernel<TO, false>, grid, 256, 0, stream, a, b, (TO*)out, (size_t)rows, width);
        return CITLALI_LAUNCH_CHECK();
    });
}

extern "C" int citlali_rms_norm(const float* x, const void* gain, int gain_dtype, const int32_t* row_index,
                                void* out, int out_dtype, int rows, int hidden, float eps, cudaStream_t stream) {
    if (rows <= 0) return 0;
    const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
    return CITLALI_DISPATCH_FLOAT(gain_dtype, TG, [&] {
        return CITLALI_DISPATCH_FLOAT(out_dtype, TO, [&] {
            if (hidden % 4 == 0 && hidden <= 8192 && (((uintptr_t)gain | (uintptr_t)x | (uintptr_t)out) & 15u) == 0)
                launch_kernel(rms_norm_rows_kernel<TG, TO>, rows, 256, 0, stream, x, (const TG*)gain, row_index, (TO*)out, hidden, eps);
            else
                launch_kernel(rms_norm_kernel<TG, TO>, rows, threads, 0, stream, x, (const TG*)gain, row_index, (TO*)out, hidden, eps);
            return CITLALI_LAUNCH_CHECK();
        });
    });
}

extern "C" int citlali_swiglu(const void* gate_up, void* act, int dtype, int rows, int inter, int run,
                              cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (run <= 0 || inter % run != 0) {
        set_last_error("swiglu: gate/up run %d does not divide the intermediate size %d", run, inter);
        return kBadShape;
    }
    if ((inter + 255) / 256 > 65535) {
        set_last_error("swiglu: intermediate size %d exceeds the grid limit", inter);
        return kTooLarge;
    }
    return CITLALI_DISPATCH_FLOAT(dtype, T, [&] {
        dim3 grid(rows, (inter + 255) / 256);
        launch_kernel(swiglu_kernel<T>, grid, 256, 0, stream, (const T*)gate_up, (T*)act, inter, run);
        return CITLALI_LAUNCH_CHECK();
    });
}
