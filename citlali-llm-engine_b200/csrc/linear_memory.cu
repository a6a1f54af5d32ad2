// Mixers whose memory of a sequence is a decayed sum of outer products, a matrix S [D, V] per head in float32:
//
//   S <- keep S + write k v^T,   o = S^T q,      and with a key sum  n <- keep n + write k,  s = n . q
//
// with keep and write numbers of the head and the token: a fixed decay a head (keep = decay[h], write = 1), or the
// exponentials of logs [row, h] = (log keep, log write) that memory_gates makes.  q, k and v are read where the projection
// left them (float32 rows `stride` apart, head after head), through SiLU if asked for, q times q_scale.
//
//   memory_gates           log gates with a running maximum m of the head: i = cap tanh(z_i / cap), f = logsigmoid(cap
//                          tanh(z_f / cap)); m_t = max(f + m_(t-1), i); log keep = f + m_(t-1) - m_t, log write = i - m_t;
//                          and exp(-m_t), what the key sum is held against.  One warp a (sequence, head), tokens in order.
//   linear_memory_scan     one warp a (sequence, head, 8 columns of S), four lanes a column, tokens in order: one order of
//                          operations for prompts, parts of prompts and single tokens.  The key sum is column V, with v = 1.
//   linear_memory_chunks   for long runs in bfloat16: a block a (sequence, head, 32 columns) walks its sequence 64 tokens at a
//                          time on the tensor cores, S in float32 accumulators throughout (see there).
//   linear_memory_output   y = o / (max(|s|, exp(-m)) + 1e-6) (without a key sum: o), divided by the root mean square of
//                          each of `groups` equal parts of the row, times a weight, times the sigmoid of a gate.
//
// A sequence's region of the state: S of every head [H, D, V] first; the key sums [H, D] at sum_off, the maxima [H] at max_off.
#include "api.h"
#include "common.cuh"
#include "mma_common.cuh"

namespace citlali {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ void copy_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

struct MemoryArgs {
    const float *q, *k, *v;              // the first head's first element in row 0
    size_t stride;                       // floats from row to row
    const float* decay;                  // [H], or null: logs [rows, H] (log keep, log write)
    const float2* logs;
    float* state;
    size_t state_stride, sum_off;
    const int32_t *seq_start, *seq_slot;
    float *out, *sums;                   // [rows, H V], and [rows, H] with a key sum (else null)
    float q_scale;
    int sequences, H, D, V, act;         // act 1: SiLU on q, k and v
};

// ---- the gates -------------------------------------------------------------------------------------------------------

__global__ void __launch_bounds__(128)
memory_gates_kernel(const float* __restrict__ zi, const float* __restrict__ zf, size_t stride, const float* __restrict__ bi,
                    const float* __restrict__ bf, float cap, float* __restrict__ state, size_t state_stride, size_t max_off,
                    const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot, int sequences, int H,
                    float2* __restrict__ logs, float* __restrict__ floors) {
    dependents_may_launch();
    wait_for_predecessor();
    const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= sequences * H) return;
    const int seq = unit / H, h = unit % H;
    const int r0 = seq_start[seq], r1 = seq_start[seq + 1];
    float* slot = state + (size_t)seq_slot[seq] * state_stride + max_off + h;
    const float b_i = bi ? bi[h] : 0.0f, b_f = bf ? bf[h] : 0.0f;
    float m = *slot;
    constexpr int AHEAD = 4;                                  // runs of 32 tokens whose inputs are on their way
    float next_i[AHEAD], next_f[AHEAD];
    auto fetch = [&](int base, int j) {
        const int row = base + lane;
        if (row < r1) { next_i[j] = zi[row * stride + h]; next_f[j] = zf[row * stride + h]; }
    };
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) fetch(r0 + 32 * j, j);
    for (int group = r0; group < r1; group += 32 * AHEAD)
#pragma unroll
    for (int g = 0; g < AHEAD; ++g) {                        // a lane a token; the maxima in order
        const int base = group + 32 * g;
        if (base >= r1) break;
        const int row = base + lane, n = min(32, r1 - base);
        float i = 0.0f, f = 0.0f;
        if (row < r1) {
            i = cap * tanhf((next_i[g] + b_i) / cap);
            const float z = cap * tanhf((next_f[g] + b_f) / cap);
            f = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
        }
        fetch(base + 32 * AHEAD, g);
        float before = 0.0f, after = 0.0f;
#pragma unroll
        for (int j = 0; j < 32; ++j) {
            const float fj = __shfl_sync(0xffffffffu, f, j), ij = __shfl_sync(0xffffffffu, i, j);
            if (j < n) {                                     // (the same for all lanes)
                const float next = fmaxf(fj + m, ij);
                if (lane == j) { before = m; after = next; }
                m = next;
            }
        }
        if (row < r1) {
            logs[(size_t)row * H + h] = make_float2(f + before - after, i - after);
            floors[(size_t)row * H + h] = expf(-after);
        }
    }
    if (lane == 0) *slot = m;
}

// ---- token by token --------------------------------------------------------------------------------------------------

// The layout of a warp's share follows the delta rule's kernel: four lanes hold a column's rows in registers, in 16-byte groups
// g with g mod 4 = the lane's part; the inputs of the next STAGES - 1 tokens are on their way into a ring in shared memory.
template <int DP, int STAGES>
__global__ void __launch_bounds__(128)
linear_memory_scan_kernel(MemoryArgs a) {
    constexpr int STRIDE = 2 * DP + 16;          // floats a token takes in the ring: k | q | v of 8 columns | two logs
    __shared__ __align__(16) float ring[4][STAGES][STRIDE];
    dependents_may_launch();
    wait_for_predecessor();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, part = lane & 3;
    const int columns = a.V + (a.sums ? 1 : 0), chunks = (columns + 7) / 8;
    const long unit = (long)blockIdx.x * 4 + warp;
    if (unit >= (long)a.sequences * a.H * chunks) return;
    const int chunk = (int)(unit % chunks), head = (int)((unit / chunks) % a.H), seq = (int)(unit / ((long)chunks * a.H));
    const int col = chunk * 8 + (lane >> 2), D = a.D, V = a.V;
    const bool live = col < columns, is_sum = live && col == V;
    const int r0 = a.seq_start[seq], r1 = a.seq_start[seq + 1];
    float* region = a.state + (size_t)a.seq_slot[seq] * a.state_stride;
    float* S_g = is_sum ? region + a.sum_off + (size_t)head * D : region + (size_t)head * D * V + col;
    const int pitch = is_sum ? 1 : V;
    constexpr int GROUPS = DP / 16;
    float S[GROUPS][4];
#pragma unroll
    for (int j = 0; j < GROUPS; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (4 * j + part) * 4 + e;
            S[j][e] = (live && i < D) ? S_g[(size_t)i * pitch] : 0.0f;
        }
    constexpr int PER = DP / 32;
    for (int i = lane; i < STAGES * STRIDE; i += 32) (&ring[warp][0][0])[i] = 0.0f;     // rows beyond D and dead columns stay zero
    __syncwarp();
    const bool my_v = lane < 8 && chunk * 8 + lane < V;
    auto issue = [&](int row) {
        if (row < r1) {
            float* dst = ring[warp][(row - r0) % STAGES];
            const float* k = a.k + (size_t)row * a.stride + (size_t)head * D;
            const float* q = a.q + (size_t)row * a.stride + (size_t)head * D;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = j * 32 + lane;
                if (i < D) {
                    copy_async4(dst + i, k + i);
                    copy_async4(dst + DP + i, q + i);
                }
            }
            if (my_v) copy_async4(dst + 2 * DP + lane, a.v + (size_t)row * a.stride + (size_t)head * V + chunk * 8 + lane);
            if (a.logs && (lane == 8 || lane == 9))
                copy_async4(dst + 2 * DP + lane, reinterpret_cast<const float*>(a.logs + (size_t)row * a.H + head) + (lane - 8));
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int s = 0; s < STAGES - 1; ++s) issue(r0 + s);
    const float fixed = a.decay ? a.decay[head] : 0.0f;
    for (int row = r0; row < r1; ++row) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        float* cur = ring[warp][(row - r0) % STAGES];
        // every lane finishes what it fetched itself
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int i = j * 32 + lane;
            if (i < D) {
                const float q = cur[DP + i];
                if (a.act) cur[i] = silu(cur[i]);
                cur[DP + i] = (a.act ? silu(q) : q) * a.q_scale;
            }
        }
        if (a.act && my_v) cur[2 * DP + lane] = silu(cur[2 * DP + lane]);
        __syncwarp();                            // this row's inputs are visible; the row before is no longer read
        issue(row + STAGES - 1);
        const float keep = a.decay ? fixed : expf(cur[2 * DP + 8]), write = a.decay ? 1.0f : expf(cur[2 * DP + 9]);
        const float u = write * (is_sum ? 1.0f : cur[2 * DP + (lane >> 2)]);
        float o0 = 0.0f, o1 = 0.0f, o2 = 0.0f, o3 = 0.0f;
#pragma unroll
        for (int j = 0; j < GROUPS; ++j) {
            const float4 k4 = *reinterpret_cast<const float4*>(cur + (4 * j + part) * 4);
            const float4 q4 = *reinterpret_cast<const float4*>(cur + DP + (4 * j + part) * 4);
            S[j][0] = fmaf(k4.x, u, keep * S[j][0]); o0 = fmaf(S[j][0], q4.x, o0);
            S[j][1] = fmaf(k4.y, u, keep * S[j][1]); o1 = fmaf(S[j][1], q4.y, o1);
            S[j][2] = fmaf(k4.z, u, keep * S[j][2]); o2 = fmaf(S[j][2], q4.z, o2);
            S[j][3] = fmaf(k4.w, u, keep * S[j][3]); o3 = fmaf(S[j][3], q4.w, o3);
        }
        float o = (o0 + o1) + (o2 + o3);
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        if (live && part == 0) {
            if (is_sum) a.sums[(size_t)row * a.H + head] = o;
            else a.out[(size_t)row * a.H * V + (size_t)head * V + col] = o;
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (live) {
#pragma unroll
        for (int j = 0; j < GROUPS; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = (4 * j + part) * 4 + e;
                if (i < D) S_g[(size_t)i * pitch] = S[j][e];
            }
    }
}

// ---- 64 tokens at a time -----------------------------------------------------------------------------------------------

// With A_t the sum of the chunk's log keeps up to token t, w_s the log write of token s, and S the state ahead of the chunk:
//   o_t = exp(A_t) S^T q_t + sum_(s <= t) exp(A_t - A_s + w_s) (q_t . k_s) v_s
//   S  <- exp(A_63) S + sum_s exp(A_63 - A_s + w_s) k_s v_s^T.
// All exponents are at most zero.  The products run as mma.sync m16n8k16: bfloat16 operands (S as the sum of two bfloat16
// numbers, so that it enters with 16 bits of mantissa), float32 sums.  S stays in float32 accumulators from chunk to chunk;
// exponents and their sums are float32.  Sixteen warps: warp (band, quarter) makes the weights of tokens 16 band .. + 15 for the
// keys 16 quarter .. + 15 (shared memory passes them on, rounded), and of those tokens' results and of the rows D/4 band .. of S
// the columns 8 quarter .. + 7; the first quarter also takes the key sum, as one more column whose v is 1.
constexpr int kChunk = 64, kCols = 32, kColPitch = 56, kWeightPitch = 72;  // columns a block; pitches of tiles in shared memory
constexpr int kChunkThreads = 512;

// VEC: sizes and strides are multiples of four and addresses of 16 bytes.
template <int DP, bool VEC>
__global__ void __launch_bounds__(kChunkThreads, 1)
linear_memory_chunks_kernel(MemoryArgs a) {
    using namespace fa;
    constexpr int PITCH = DP + 8, MT = DP / 64;
    extern __shared__ __align__(16) uint8_t smem[];
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem);              // [64][PITCH]
    __nv_bfloat16* sk = sq + kChunk * PITCH;
    __nv_bfloat16* sv = sk + kChunk * PITCH;                                 // [64][kColPitch] v
    __nv_bfloat16* sw = sv + kChunk * kColPitch;                             // the same times exp(A_63 - A_s + w_s)
    __nv_bfloat16* s_hi = sw + kChunk * kColPitch;                           // [DP][kColPitch] S, rounded
    __nv_bfloat16* s_lo = s_hi + DP * kColPitch;                             // and what the rounding left
    __nv_bfloat16* sp = s_lo + DP * kColPitch;                               // [64][kWeightPitch] the chunk's weights
    __shared__ float sum_a[kChunk], from[kChunk], share[kChunk];             // A_t, w_s - A_s, exp(A_63 - A_s + w_s); in log2 units
    dependents_may_launch();
    wait_for_predecessor();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, band = warp & 3, quarter = warp >> 2;
    const int D = a.D, V = a.V, slices = (V + kCols - 1) / kCols;
    const int slice = blockIdx.x % slices, head = (blockIdx.x / slices) % a.H, seq = blockIdx.x / (slices * a.H);
    const int col0 = slice * kCols;
    const bool with_sum = a.sums != nullptr && slice == 0;
    const int r0 = a.seq_start[seq], n = a.seq_start[seq + 1] - r0;
    float* region = a.state + (size_t)a.seq_slot[seq] * a.state_stride;
    float* S_g = region + (size_t)head * D * V;
    float* n_g = region + a.sum_off + (size_t)head * D;
    const int tiles = (quarter == 0 && with_sum) ? 2 : 1;                    // column tiles of eight this warp works on
    auto tile_col = [&](int j) { return j == 1 ? kCols : quarter * 8; };
    // element (i, e) of an accumulator: row lane/4 (+ 8 for e >= 2), column (lane % 4) * 2 + e % 2
    auto place = [&](int m, int j, int e) -> float* {
        const int d = (band * MT + m) * 16 + (lane >> 2) + (e >> 1) * 8, c = tile_col(j) + (lane & 3) * 2 + (e & 1);
        if (d >= D) return nullptr;
        if (j == 1) return c == kCols ? n_g + d : nullptr;
        return col0 + c < V ? S_g + (size_t)d * V + col0 + c : nullptr;
    };
    float S[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float* p = j < tiles ? place(m, j, e) : nullptr;
                S[m][j][e] = p ? *p : 0.0f;
            }
    const float log_keep = a.decay ? (a.decay[head] > 0.0f ? log2f(a.decay[head]) : -1e30f) : 0.0f;   // (a decay of zero: finite, 64 of them too)
    // four neighbouring elements of a row as they are (zeros past `limit`), and through the activation as two words
    auto fetch = [&](const float* row, int c, int limit) -> float4 {
        float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if constexpr (VEC) {
            if (c < limit) x = *reinterpret_cast<const float4*>(row + c);
        } else {
            if (c < limit) x.x = row[c];
            if (c + 1 < limit) x.y = row[c + 1];
            if (c + 2 < limit) x.z = row[c + 2];
            if (c + 3 < limit) x.w = row[c + 3];
        }
        return x;
    };
    auto words = [&](float4 x) -> uint2 {
        if (a.act) {
            x.x = __fdividef(x.x, 1.0f + __expf(-x.x)); x.y = __fdividef(x.y, 1.0f + __expf(-x.y));
            x.z = __fdividef(x.z, 1.0f + __expf(-x.z)); x.w = __fdividef(x.w, 1.0f + __expf(-x.w));
        }
        return make_uint2(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w));
    };
    // a thread's pieces of the chunk's rows: q and k of up to 128 elements, and v, wait in registers while the chunk before is
    // worked on; wider heads fetch half of their pieces at a time when the tiles are filled
    constexpr int PIECES = kChunk * (DP / 4) / kChunkThreads;
    static_assert(kChunk * (kCols / 4) == kChunkThreads && PIECES >= 1, "a piece of v a thread");
    constexpr bool AHEAD = DP <= 128;
    constexpr int HELD = AHEAD ? PIECES : PIECES / 2;
    float4 rq[HELD], rk[HELD], rv;
    const int v_row = tid / (kCols / 4), v_col = tid % (kCols / 4) * 4;
    const size_t chunk_step = (size_t)kChunk * a.stride;
    const float* v_next = a.v + (size_t)(r0 + v_row) * a.stride + (size_t)head * V;
    constexpr int ROWS_APART = AHEAD ? kChunkThreads / (DP / 4) : 1;          // rows from one of a thread's pieces to the next
    const int q_row = tid / (DP / 4), q_col = tid % (DP / 4) * 4;
    const float* q_next = a.q + (size_t)(r0 + q_row) * a.stride + (size_t)head * D;
    const float* k_next = a.k + (size_t)(r0 + q_row) * a.stride + (size_t)head * D;
    auto fetch_next_qk = [&](int t0) {
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
            const int limit = t0 + q_row + i * ROWS_APART < n ? D : 0;
            rq[i] = fetch(q_next + (size_t)(i * ROWS_APART) * a.stride, q_col, limit);
            rk[i] = fetch(k_next + (size_t)(i * ROWS_APART) * a.stride, q_col, limit);
        }
        q_next += chunk_step;
        k_next += chunk_step;
    };
    auto fetch_qk = [&](int t0, int first) {
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
            const int at = tid + (first + i) * kChunkThreads, t = at / (DP / 4), c = at % (DP / 4) * 4;
            const size_t row = (size_t)(r0 + t0 + t) * a.stride + (size_t)head * D;
            const int limit = t0 + t < n ? D : 0;
            rq[i] = fetch(a.q + row, c, limit);
            rk[i] = fetch(a.k + row, c, limit);
        }
    };
    auto store_qk = [&](int first) {
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
            const int at = tid + (first + i) * kChunkThreads, t = at / (DP / 4), c = at % (DP / 4) * 4;
            *reinterpret_cast<uint2*>(sq + t * PITCH + c) = words(rq[i]);
            *reinterpret_cast<uint2*>(sk + t * PITCH + c) = words(rk[i]);
        }
    };
    auto fetch_v = [&](int t0) {
        rv = fetch(v_next, col0 + v_col, t0 + v_row < n ? V : 0);
        v_next += chunk_step;
    };
    float2 next_log[2];
    auto fetch_logs = [&](int t0) {
#pragma unroll
        for (int e = 0; e < 2; ++e)
            if (!a.decay && t0 + 2 * lane + e < n) next_log[e] = a.logs[(size_t)(r0 + t0 + 2 * lane + e) * a.H + head];
    };
    if (warp == 0) fetch_logs(0);
    if constexpr (AHEAD) fetch_next_qk(0);
    fetch_v(0);
    const uint32_t q_addr = (uint32_t)__cvta_generic_to_shared(sq), k_addr = (uint32_t)__cvta_generic_to_shared(sk);
    const uint32_t v_addr = (uint32_t)__cvta_generic_to_shared(sv), w_addr = (uint32_t)__cvta_generic_to_shared(sw);
    const uint32_t hi_addr = (uint32_t)__cvta_generic_to_shared(s_hi), lo_addr = (uint32_t)__cvta_generic_to_shared(s_lo);
    const uint32_t p_addr = (uint32_t)__cvta_generic_to_shared(sp);

    for (int t0 = 0; t0 < n; t0 += kChunk) {
        const int here = min(kChunk, n - t0);
        // A_t, by two tokens a lane of the first warp
        if (warp == 0) {
            float keep[2], write[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const bool on = 2 * lane + e < here;
                keep[e] = on ? (a.decay ? log_keep : next_log[e].x * kLog2e) : 0.0f;
                write[e] = on && !a.decay ? next_log[e].y * kLog2e : 0.0f;
            }
            fetch_logs(t0 + kChunk);
            float run = keep[0] + keep[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run += up;
            }
            const float total = __shfl_sync(0xffffffffu, run, 31);
            const float a1 = run, a0 = run - keep[1];
            sum_a[2 * lane] = a0; sum_a[2 * lane + 1] = a1;
            from[2 * lane] = write[0] - a0; from[2 * lane + 1] = write[1] - a1;
            share[2 * lane] = 2 * lane < here ? exp2f(total + (write[0] - a0)) : 0.0f;
            share[2 * lane + 1] = 2 * lane + 1 < here ? exp2f(total + (write[1] - a1)) : 0.0f;
        }
        // the state ahead of the chunk as two bfloat16 tiles
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j)
                if (j < tiles) {
#pragma unroll
                    for (int e = 0; e < 4; e += 2) {
                        const int d = (band * MT + m) * 16 + (lane >> 2) + (e >> 1) * 8, c = tile_col(j) + (lane & 3) * 2;
                        const __nv_bfloat16 h0 = __float2bfloat16_rn(S[m][j][e]), h1 = __float2bfloat16_rn(S[m][j][e + 1]);
                        *reinterpret_cast<__nv_bfloat162*>(s_hi + d * kColPitch + c) = __nv_bfloat162(h0, h1);
                        *reinterpret_cast<uint32_t*>(s_lo + d * kColPitch + c) =
                            pack_bf16(S[m][j][e] - __bfloat162float(h0), S[m][j][e + 1] - __bfloat162float(h1));
                    }
                }
        // the chunk's rows
        if constexpr (AHEAD) {
            store_qk(0);
            if (t0 + kChunk < n) fetch_next_qk(t0 + kChunk);  // on its way while this chunk is worked on
        } else {
#pragma unroll 1
            for (int first = 0; first < PIECES; first += HELD) {
                fetch_qk(t0, first);
                store_qk(first);
            }
        }
        __syncthreads();                         // (q, k, the state and the shares are there)
        {
            const uint2 vw = words(rv);
            *reinterpret_cast<uint2*>(sv + v_row * kColPitch + v_col) = vw;
            const float f = share[v_row];
            const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vw.x));
            const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vw.y));
            *reinterpret_cast<uint2*>(sw + v_row * kColPitch + v_col) = make_uint2(pack_bf16(lo.x * f, lo.y * f), pack_bf16(hi.x * f, hi.y * f));
            if (t0 + kChunk < n) fetch_v(t0 + kChunk);
        }
        if (with_sum && tid < kChunk) {          // the key sum's column of ones, and seven of zeros
            *reinterpret_cast<uint4*>(sv + tid * kColPitch + kCols) = make_uint4(tid < here ? 0x3f80u : 0u, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(sw + tid * kColPitch + kCols) = make_uint4(pack_bf16(share[tid], 0.0f), 0u, 0u, 0u);
        }
        // S^T q of this warp's tokens and columns, and its sixteen by sixteen weights of the chunk's own tokens
        float o[2][4], p[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = p[j][0] = p[j][1] = p[j][2] = p[j][3] = 0.0f;
        const int arow = band * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, acol = (lane >> 4) * 8;
        const int t_a = band * 16 + (lane >> 2), t_b = t_a + 8;
        const bool rows_here = band * 16 < here, seen = quarter <= band;      // (later tokens are not seen)
        if (rows_here) {
            const uint32_t half_addr = (lane >> 4) ? lo_addr : hi_addr;       // one load brings both parts of sixteen rows of S
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t q0, q1, q2, q3, b0, b1, b2, b3;
                ldmatrix_x4(q_addr + (arow * PITCH + ks * 16 + acol) * 2, q0, q1, q2, q3);
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (j < tiles) {
                        ldmatrix_x4_trans(half_addr + ((ks * 16 + (lane & 15)) * kColPitch + tile_col(j)) * 2, b0, b1, b2, b3);
                        mma_16816(o[j], q0, q1, q2, q3, b0, b1);
                        mma_16816(o[j], q0, q1, q2, q3, b2, b3);
                    }
                if (seen) {
                    const int r = quarter * 16 + (lane & 7) + (lane >> 4) * 8, c = ((lane >> 3) & 1) * 8;
                    ldmatrix_x4(k_addr + (r * PITCH + ks * 16 + c) * 2, b0, b1, b2, b3);
                    mma_16816(p[0], q0, q1, q2, q3, b0, b1);
                    mma_16816(p[1], q0, q1, q2, q3, b2, b3);
                }
            }
            const float A_a = sum_a[t_a], A_b = sum_a[t_b], g_a = exp2f(A_a) * a.q_scale, g_b = exp2f(A_b) * a.q_scale;
#pragma unroll
            for (int j = 0; j < 2; ++j) { o[j][0] *= g_a; o[j][1] *= g_a; o[j][2] *= g_b; o[j][3] *= g_b; }
            if (seen) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int s = quarter * 16 + i * 8 + (lane & 3) * 2;
                    const float f0 = from[s], f1 = from[s + 1];
                    const float w0 = s <= t_a ? p[i][0] * (a.q_scale * exp2f(A_a + f0)) : 0.0f, w1 = s + 1 <= t_a ? p[i][1] * (a.q_scale * exp2f(A_a + f1)) : 0.0f;
                    const float w2 = s <= t_b ? p[i][2] * (a.q_scale * exp2f(A_b + f0)) : 0.0f, w3 = s + 1 <= t_b ? p[i][3] * (a.q_scale * exp2f(A_b + f1)) : 0.0f;
                    *reinterpret_cast<uint32_t*>(sp + t_a * kWeightPitch + s) = pack_bf16(w0, w1);
                    *reinterpret_cast<uint32_t*>(sp + t_b * kWeightPitch + s) = pack_bf16(w2, w3);
                }
            }
        }
        __syncthreads();                         // (weights and values are there)
        if (rows_here) {
#pragma unroll
            for (int np = 0; np < kChunk / 16; np += 2) {
                if (np > band) break;
                uint32_t b[2][4];
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (j < tiles) ldmatrix_x4_trans(v_addr + ((np * 16 + lane) * kColPitch + tile_col(j)) * 2, b[j][0], b[j][1], b[j][2], b[j][3]);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    if (np + i > band) break;
                    uint32_t p0, p1, p2, p3;
                    ldmatrix_x4(p_addr + (arow * kWeightPitch + (np + i) * 16 + acol) * 2, p0, p1, p2, p3);
#pragma unroll
                    for (int j = 0; j < 2; ++j)
                        if (j < tiles) mma_16816(o[j], p0, p1, p2, p3, b[j][2 * i], b[j][2 * i + 1]);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int t = e < 2 ? t_a : t_b, c = col0 + quarter * 8 + (lane & 3) * 2;
                if (t < here) {
                    const size_t row = r0 + t0 + t;
                    float* dst = a.out + row * a.H * V + (size_t)head * V + c;
                    if (V % 2 == 0) {
                        if (c < V) *reinterpret_cast<float2*>(dst) = make_float2(o[0][e], o[0][e + 1]);
                    } else {
                        if (c < V) dst[0] = o[0][e];
                        if (c + 1 < V) dst[1] = o[0][e + 1];
                    }
                    if (tiles == 2 && (lane & 3) == 0) a.sums[row * a.H + head] = o[1][e];
                }
            }
        }
        // the state behind the chunk
        const float g = exp2f(sum_a[kChunk - 1]);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j) { S[m][j][0] *= g; S[m][j][1] *= g; S[m][j][2] *= g; S[m][j][3] *= g; }
#pragma unroll
        for (int kt = 0; kt < kChunk / 16; kt += 2) {
            if (kt * 16 >= here) break;
            uint32_t b[2][4];
#pragma unroll
            for (int j = 0; j < 2; ++j)
                if (j < tiles) ldmatrix_x4_trans(w_addr + ((kt * 16 + lane) * kColPitch + tile_col(j)) * 2, b[j][0], b[j][1], b[j][2], b[j][3]);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    // K^T: the tile lies as [token][d], its transpose is the operand
                    const int r = (kt + i) * 16 + (lane & 7) + (lane >> 4) * 8, c = (band * MT + m) * 16 + ((lane >> 3) & 1) * 8;
                    uint32_t k0, k1, k2, k3;
                    ldmatrix_x4_trans(k_addr + (r * PITCH + c) * 2, k0, k1, k2, k3);
#pragma unroll
                    for (int j = 0; j < 2; ++j)
                        if (j < tiles) mma_16816(S[m][j], k0, k1, k2, k3, b[j][2 * i], b[j][2 * i + 1]);
                }
        }
        __syncthreads();                         // everyone is done with the tiles
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float* p = j < tiles ? place(m, j, e) : nullptr;
                if (p) *p = S[m][j][e];
            }
}

// ---- the output --------------------------------------------------------------------------------------------------------

// One warp a (row, part) for parts of up to 256 elements, else a block (threads by the part's size alone).  A thread holds up to
// KEEP runs of W neighbouring elements between the two passes (W 4: a head's and a part's size are multiples of four, 16-byte
// rows); what a longer part has beyond them is read again.
template <typename TO, bool WARP, int W>
__global__ void __launch_bounds__(WARP ? 256 : 1024)
linear_memory_output_kernel(const float* __restrict__ o, const float* __restrict__ sums, const float* __restrict__ floors,
                            const float* __restrict__ gate, size_t gate_stride, const float* __restrict__ weight,
                            TO* __restrict__ y, int H, int V, int groups, float eps) {
    __shared__ float scratch[32];
    dependents_may_launch();
    wait_for_predecessor();
    const int row = blockIdx.x, inner = H * V, n = inner / groups;
    const int grp = WARP ? blockIdx.y * 8 + (threadIdx.x >> 5) : blockIdx.y;
    if (grp >= groups) return;
    const int tid = WARP ? threadIdx.x & 31 : threadIdx.x, step = (WARP ? 32 : blockDim.x) * W;
    const float* src = o + (size_t)row * inner;
    auto value = [&](int c, float (&v)[W]) {
        if constexpr (W == 4) {
            const float4 f = *reinterpret_cast<const float4*>(src + c);
            v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
        } else {
            v[0] = src[c];
        }
        if (!sums) return;
        const size_t at = (size_t)row * H + c / V;
        const float den = fmaxf(fabsf(sums[at]), floors[at]) + 1e-6f;
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] /= den;
    };
    constexpr int KEEP = W == 4 ? 2 : 8;
    float kept[KEEP][W], more[W], ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = tid * W + j * step;
        if (i < n) {
            value(grp * n + i, kept[j]);
#pragma unroll
            for (int e = 0; e < W; ++e) ss = fmaf(kept[j][e], kept[j][e], ss);
        }
    }
    for (int i = tid * W + KEEP * step; i < n; i += step) {
        value(grp * n + i, more);
#pragma unroll
        for (int e = 0; e < W; ++e) ss = fmaf(more[e], more[e], ss);
    }
    ss = WARP ? warp_sum(ss) : block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    const float* gt = gate + (size_t)row * gate_stride;
    TO* dst = y + (size_t)row * inner;
    auto gated = [&](float v, float w, float z) { return v * inv * w / (1.0f + expf(-z)); };
    auto finish = [&](int c, const float (&v)[W]) {
        if constexpr (W == 4) {
            const float4 w = *reinterpret_cast<const float4*>(weight + c), z = *reinterpret_cast<const float4*>(gt + c);
            const float4 r = make_float4(gated(v[0], w.x, z.x), gated(v[1], w.y, z.y), gated(v[2], w.z, z.z), gated(v[3], w.w, z.w));
            if constexpr (sizeof(TO) == 2)
                *reinterpret_cast<uint2*>(dst + c) = make_uint2(fa::pack_bf16(r.x, r.y), fa::pack_bf16(r.z, r.w));
            else
                *reinterpret_cast<float4*>(dst + c) = r;
        } else {
            stf(dst, c, gated(v[0], weight[c], gt[c]));
        }
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = tid * W + j * step;
        if (i < n) finish(grp * n + i, kept[j]);
    }
    for (int i = tid * W + KEEP * step; i < n; i += step) {
        value(grp * n + i, more);
        finish(grp * n + i, more);
    }
}

template <int DP, int STAGES>
int launch_scan(const MemoryArgs& a, cudaStream_t stream) {
    const long units = (long)a.sequences * a.H * ((a.V + (a.sums ? 1 : 0) + 7) / 8);
    launch_kernel(linear_memory_scan_kernel<DP, STAGES>, (unsigned)((units + 3) / 4), 128, 0, stream, a);
    return CITLALI_LAUNCH_CHECK();
}

template <int DP, bool VEC>
int launch_chunks(const MemoryArgs& a, cudaStream_t stream) {
    constexpr int smem = (2 * kChunk * (DP + 8) + 2 * kChunk * kColPitch + 2 * DP * kColPitch + kChunk * kWeightPitch) * 2;
    auto kernel = linear_memory_chunks_kernel<DP, VEC>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const long blocks = (long)a.sequences * a.H * ((a.V + kCols - 1) / kCols);
    launch_kernel(kernel, (unsigned)blocks, kChunkThreads, smem, stream, a);
    return CITLALI_LAUNCH_CHECK();
}

template <int DP>
int pick_chunks(const MemoryArgs& a, cudaStream_t stream) {
    const bool vec = a.D % 4 == 0 && a.V % 4 == 0 && a.stride % 4 == 0 && (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) & 15u) == 0;
    return vec ? launch_chunks<DP, true>(a, stream) : launch_chunks<DP, false>(a, stream);
}

}  // namespace
}  // namespace citlali

using namespace citlali;

extern "C" int citlali_memory_gates(const float* zi, const float* zf, size_t stride, const float* bi, const float* bf, float cap,
                                    float* state, size_t state_stride, size_t max_off, const int32_t* seq_start,
                                    const int32_t* seq_slot, int sequences, int H, float* logs, float* floors,
                                    cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (H <= 0 || !(cap > 0.0f) || ((uintptr_t)logs & 7u)) {
        set_last_error("memory_gates: %d heads, a cap of %g (must be positive); the logs must be 8-byte aligned", H, cap);
        return kBadShape;
    }
    launch_kernel(memory_gates_kernel, (unsigned)(((long)sequences * H + 3) / 4), 128, 0, stream, zi, zf, stride, bi, bf, cap, state,
                  state_stride, max_off, seq_start, seq_slot, sequences, H, (float2*)logs, floors);
    return CITLALI_LAUNCH_CHECK();
}

extern "C" int citlali_linear_memory(const float* q, const float* k, const float* v, size_t stride, int act, float q_scale,
                                     const float* decay, const float* logs, float* state, size_t state_stride, size_t sum_off,
                                     const int32_t* seq_start, const int32_t* seq_slot, int sequences, int H, int D, int V,
                                     float* out, float* sums, int form, cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (H <= 0 || D <= 0 || V <= 0 || (decay == nullptr) == (logs == nullptr) || (act != 0 && act != 1) || form < 0 || form > 2) {
        set_last_error("linear_memory: %d heads of %d (values %d), form %d; either fixed decays or logs are given", H, D, V, form);
        return kBadShape;
    }
    if (D > 256) {
        set_last_error("linear_memory: a head size of %d exceeds 256", D);
        return kTooLarge;
    }
    const MemoryArgs a{q, k, v, stride, decay, (const float2*)logs, state, state_stride, sum_off, seq_start, seq_slot, out, sums,
                       q_scale, sequences, H, D, V, act};
    if (form == 2) {
        switch ((D + 63) / 64) {
            case 1: return pick_chunks<64>(a, stream);
            case 2: return pick_chunks<128>(a, stream);
            case 3: return pick_chunks<192>(a, stream);
            default: return pick_chunks<256>(a, stream);
        }
    }
#define CITLALI_SCAN(DP, ST) return form == 1 ? launch_scan<DP, 2>(a, stream) : launch_scan<DP, ST>(a, stream)
    switch ((D + 31) / 32) {
        case 1: CITLALI_SCAN(32, 8);
        case 2: CITLALI_SCAN(64, 8);
        case 3: CITLALI_SCAN(96, 8);
        case 4: CITLALI_SCAN(128, 8);
        case 5: CITLALI_SCAN(160, 4);
        case 6: CITLALI_SCAN(192, 4);
        case 7: CITLALI_SCAN(224, 4);
        default: CITLALI_SCAN(256, 4);
    }
#undef CITLALI_SCAN
}

extern "C" int citlali_linear_memory_output(const float* o, const float* sums, const float* floors, const float* gate,
                                            size_t gate_stride, const float* weight, void* y, int y_dtype, int rows, int H, int V,
                                            int groups, float eps, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (H <= 0 || V <= 0 || groups <= 0 || (H * V) % groups != 0 || groups > 65535 || (sums == nullptr) != (floors == nullptr)) {
        set_last_error("linear_memory_output: %d heads of %d in %d equal parts; key sums come with what they are held against", H, V, groups);
        return kBadShape;
    }
    const int n = H * V / groups;
    const bool vec = V % 4 == 0 && n % 4 == 0 && gate_stride % 4 == 0 &&
                     (((uintptr_t)o | (uintptr_t)gate | (uintptr_t)weight | (uintptr_t)y) & 15u) == 0;
    int threads = ((n / 4 + 31) / 32) * 32;
    threads = threads < 64 ? 64 : (threads > 1024 ? 1024 : threads);
    return CITLALI_DISPATCH_FLOAT(y_dtype, TO, [&] {
        auto go = [&](auto kernel, dim3 grid, int block) {
            launch_kernel(kernel, grid, block, 0, stream, o, sums, floors, gate, gate_stride, weight, (TO*)y, H, V, groups, eps);
        };
        if (n <= 256) {
            const dim3 grid(rows, (groups + 7) / 8);
            const int block = groups < 8 ? 32 * groups : 256;
            if (vec) go(linear_memory_output_kernel<TO, true, 4>, grid, block);
            else go(linear_memory_output_kernel<TO, true, 1>, grid, block);
        } else {
            const dim3 grid(rows, groups);
            if (vec) go(linear_memory_output_kernel<TO, false, 4>, grid, threads);
            else go(linear_memory_output_kernel<TO, false, 1>, grid, threads);
        }
        return CITLALI_LAUNCH_CHECK();
    });
}
