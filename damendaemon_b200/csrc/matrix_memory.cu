// A matrix memory per head: linear attention whose state fades by one number per head and token.
//
// Per head, token by token, with S [dk, dv] float32 per request from zero:
//     S <- (1 - fade_t) S + take_t k_t v_t^T,      o_t = S^T q_t        (q, k, v optionally through silu, q times a scale)
// Two sources of fade and take:
//   fixed    fade = 1 - decay of the head, take = 1;
//   gated    exponential gates kept in range by a running maximum M (from zero, per request and head): with the log input
//            gate i = cap tanh(z_i / cap) and the log forget gate f = log sigmoid(cap tanh(z_f / cap)),
//            M' = max(f + M, i), fade = 1 - exp(f + M - M'), take = exp(i - M'). A vector n <- (1 - fade) n + take k goes with
//            S; the read-out is o / (max(|n . q|, exp(-M')) + den_eps). n is one more column of S, whose value is 1.
// The fade travels as such, not as the decay: a decay near one would lose its distance from one to rounding. f + M - M' is
// formed as (M - M') + f: where the forget path wins, M - M' is exact and what M' lost to rounding comes back in the fade.
//
//   dd_memory_gates    fade, take and exp(-M') of a step's tokens; a block walks an entry and head, 128 tokens at a time: the
//                      transcendental functions side by side, the maximum one token after the other, so the result does not
//                      depend on how a prompt was cut
//   dd_memory_prepare  q, take k and v (and the column of ones) as float32 rows, padded to 16-byte pieces
//   dd_memory_scan     the recurrence. Column j of o depends on column j of S only: a block owns (entry, head, a run of
//                      columns); a column's rows are dealt out over neighbouring lanes and a thread holds the same few rows
//                      of several columns in registers, so an operand read from shared memory serves them all. No token's
//                      update waits for an exchange between lanes; the read-outs of four tokens are exchanged together.
//                      Tokens are staged 16 at a time by cp.async, two buffers in turn.
//   dd_memory_step     a step of single tokens in one kernel, gates included. A head's columns are dealt out over the blocks
//                      of a cluster; with a norm per head the blocks exchange their sums of squares through distributed
//                      shared memory and write the normed, weighted, gated result themselves.
//   dd_memory_finish   o (over its denominator, if it has one) over equal stretches of one or of all heads divided by the
//                      stretch's root mean square, times a weight and the sigmoid of a gate, rounded once
// The state lies column by column ([slots, H, dv (+ 1), DKP], DKP = dk rounded up to 8 times a power of two; rows past dk
// stay zero). The state's update of a single token has the scan's bits.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace {
__device__ __forceinline__ float mm_silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }
__device__ __forceinline__ float mm_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

// The log gates of one token from their projections.
__device__ __forceinline__ void mm_log_gates(float zi, float zf, float cap, float& i, float& f) {
    i = cap * tanhf(zi / cap);
    const float c = cap * tanhf(zf / cap);
    f = fminf(c, 0.f) - log1pf(expf(-fabsf(c)));
}

struct MemoryGates { float fade, take, floor; };
__device__ __forceinline__ MemoryGates mm_gates(float i, float f, float before, float now) {
    MemoryGates g;
    g.fade = -expm1f(__fadd_rn(__fsub_rn(before, now), f));
    g.take = expf(i - now);
    g.floor = expf(-now);
    return g;
}

constexpr int MG_TOKENS = 128;

__global__ void __launch_bounds__(MG_TOKENS)
memory_gates_kernel(const float* __restrict__ z, int z_stride, float cap, const int* __restrict__ entry_start,
                    const int* __restrict__ entry_slot, float* __restrict__ peak, float* __restrict__ fade,
                    float* __restrict__ take, float* __restrict__ floor_out, int H) {
    __shared__ __align__(16) float2 logs[MG_TOKENS];     // (i, f) of a token
    __shared__ float maxima[MG_TOKENS + 1];              // M before the first token, then after every one
    dd_launch_dependents();
    const int h = blockIdx.x, e = blockIdx.y, tid = threadIdx.x;
    const int start = entry_start[e], end = entry_start[e + 1];
    dd_grid_wait();
    float* mine = peak + (size_t)entry_slot[e] * H + h;
    float M = *mine;
    for (int t0 = start; t0 < end; t0 += MG_TOKENS) {
        const int n = min(MG_TOKENS, end - t0);
        float i = -INFINITY, f = 0.f;                    // (no token: the maximum stays as it is)
        if (tid < n) {
            const float* row = z + (size_t)(t0 + tid) * z_stride + h;
            mm_log_gates(row[0], row[H], cap, i, f);
        }
        logs[tid] = make_float2(i, f);
        __syncthreads();
        if (tid < 32) {
            // one warp walks the tokens, all lanes alike; eight at a time, so that their loads lie ahead of the chain
            if (tid == 0) maxima[0] = M;
            for (int j = 0; j < n; j += 8) {
                float2 l[8];
#pragma unroll
                for (int u = 0; u < 8; ++u) l[u] = logs[j + u];
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    M = fmaxf(__fadd_rn(l[u].y, M), l[u].x);
                    if (tid == u) maxima[j + u + 1] = M;
                }
            }
        }
        __syncthreads();
        if (tid < n) {
            const MemoryGates g = mm_gates(i, f, maxima[tid], maxima[tid + 1]);
            const size_t at = (size_t)(t0 + tid) * H + h;
            fade[at] = g.fade;
            take[at] = g.take;
            floor_out[at] = g.floor;
        }
    }
    if (tid == 0 && start < end) *mine = M;
}

// Four neighbouring elements from c on (those past n as zeros); WIDE: one load.
template <typename T, bool WIDE>
__device__ __forceinline__ float4 mm_load4(const T* row, int c, int n) {
    if (WIDE && c < n) {
        if (sizeof(T) == 2) {
            const uint2 u = *reinterpret_cast<const uint2*>(row + c);
            return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                               __uint_as_float(u.y & 0xffff0000u));
        }
        return *reinterpret_cast<const float4*>(row + c);
    }
    float4 x;
    x.x = c < n ? dd_to_f32(row[c]) : 0.f;
    x.y = c + 1 < n ? dd_to_f32(row[c + 1]) : 0.f;
    x.z = c + 2 < n ? dd_to_f32(row[c + 2]) : 0.f;
    x.w = c + 3 < n ? dd_to_f32(row[c + 3]) : 0.f;
    return x;
}

// A thread owns four neighbouring elements of a head's q, k or v; the blocks of grid column t share token t.
template <typename T, bool WIDE>
__global__ void __launch_bounds__(256)
memory_prepare_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int stride, float q_scale,
                      int silu, const float* __restrict__ take, float* __restrict__ q_out, float* __restrict__ k_out,
                      float* __restrict__ v_out, int H, int dk, int dv, int ones, int qk_row, int v_row) {
    dd_launch_dependents();
    dd_grid_wait();
    const int t = blockIdx.x, qk4 = qk_row / 4, v4 = v_row / 4;
    int piece = blockIdx.y * 256 + threadIdx.x;
    const int kind = piece < H * qk4 ? 0 : (piece < 2 * H * qk4 ? 1 : 2);
    piece -= kind * H * qk4;
    const int per = kind < 2 ? qk4 : v4, h = piece / per, c = (piece - h * per) * 4;
    if (h >= H) return;
    const size_t item = (size_t)t * H + h;
    float4 x;
    if (kind < 2) x = mm_load4<T, WIDE>((kind ? k : q) + (size_t)t * stride + (size_t)h * dk, c, dk);
    else x = mm_load4<T, WIDE>(v + (size_t)t * stride + (size_t)h * dv, c, dv);
    if (silu) { x.x = mm_silu(x.x); x.y = mm_silu(x.y); x.z = mm_silu(x.z); x.w = mm_silu(x.w); }
    if (kind < 2) {
        const float by = kind == 0 ? q_scale : (take ? take[item] : 1.0f);
        *reinterpret_cast<float4*>((kind ? k_out : q_out) + item * qk_row + c) = make_float4(x.x * by, x.y * by, x.z * by, x.w * by);
        return;
    }
    if (ones && dv - c >= 0 && dv - c < 4) {             // the column of ones
        if (dv == c) x.x = 1.0f;
        else if (dv == c + 1) x.y = 1.0f;
        else if (dv == c + 2) x.z = 1.0f;
        else x.w = 1.0f;
    }
    *reinterpret_cast<float4*>(v_out + item * v_row + c) = x;
}

__device__ __forceinline__ void mm_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void mm_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// One row of one column: the update every kernel here uses, rounding by rounding.
__device__ __forceinline__ float mm_update(float s, float fade, float k, float v) {
    return __fmaf_rn(k, v, __fmaf_rn(-fade, s, s));
}

// Two neighbouring rows at a time: each half is rounded as the single instruction would round it.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 mm_pack(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float mm_half_sum(f32x2 x) {
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(x));
    return __fadd_rn(lo, hi);
}
__device__ __forceinline__ f32x2 mm_fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mm_mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// N sums, of which every one of a column's LPC lanes holds a part: at every exchange (O = 1, 2, 4, .. lanes apart) a lane gives
// away half of its sums and keeps the other half while it has more than one. Returns the index of the first sum the lane is
// left with, in read[0].
template <int N, int O, int LPC>
__device__ __forceinline__ int mm_spread_sums(float* read, int sub) {
    if constexpr (O >= LPC) {
        return 0;
    } else if constexpr (N > 1) {
        const bool up = (sub & O) != 0;
#pragma unroll
        for (int i = 0; i < N / 2; ++i) {
            const float give = up ? read[i] : read[i + N / 2];
            const float keep = up ? read[i + N / 2] : read[i];
            read[i] = keep + __shfl_xor_sync(0xffffffffu, give, O);
        }
        return (up ? N / 2 : 0) + mm_spread_sums<N / 2, O * 2, LPC>(read, sub);
    } else {
        read[0] += __shfl_xor_sync(0xffffffffu, read[0], O);
        return mm_spread_sums<1, O * 2, LPC>(read, sub);
    }
}

constexpr int MM_TOKENS = 16;          // tokens staged together

struct ScanArgs {
    const float* q;              // [N, H, qk_row]
    const float* k;
    const float* v;              // [N, H, v_row]
    const float* fade;           // [N, H], or null: fixed
    const float* fixed;          // [H]
    const int* entry_start;
    const int* entry_slot;
    float* state;                // [slots, H, cols, R * LPC]
    float* out;                  // [N, H, v_row]
    int H, cols, qk_row, v_row;
};

// R rows and C columns of the state a thread (R a multiple of 4, 16-byte pieces that lie a whole sweep of the column's LPC
// lanes apart, so that neighbouring lanes read neighbouring pieces); THREADS / LPC * C columns a block.
template <int R, int C, int LPC, int THREADS>
__global__ void __launch_bounds__(THREADS)
memory_scan_kernel(const ScanArgs a) {
    constexpr int DKP = R * LPC, COLS = THREADS / LPC * C, P = R / 4;
    constexpr int BUF = MM_TOKENS * (2 * DKP + COLS) + MM_TOKENS;       // floats of one buffer: q, k, v, fade
    extern __shared__ __align__(16) float staged[];
    dd_launch_dependents();
    const int e = blockIdx.z, h = blockIdx.y, H = a.H;
    const int col0 = blockIdx.x * COLS;
    const int my_col = threadIdx.x / LPC * C, sub = threadIdx.x % LPC;
    const int start = a.entry_start[e], end = a.entry_start[e + 1];
    // rows past qk_row and columns past v_row are never copied into: they stay the zeros written here, and so do the tokens
    // past an entry's last one in its last buffer (a token of zeros leaves the state as it is)
    for (int i = threadIdx.x; i < 2 * BUF; i += THREADS) staged[i] = 0.f;
    auto stage = [&](int t0, int buf) {
        const int n = min(MM_TOKENS, end - t0);
        float* bq = staged + buf * BUF;
        float* bk = bq + MM_TOKENS * DKP;
        float* bv = bk + MM_TOKENS * DKP;
        float* bf = bv + MM_TOKENS * COLS;
        for (int i = threadIdx.x; i < n * (DKP / 4); i += THREADS) {
            const int tt = i / (DKP / 4), c = (i % (DKP / 4)) * 4;
            if (c < a.qk_row) {
                const size_t at = ((size_t)(t0 + tt) * H + h) * a.qk_row + c;
                mm_copy16(bq + tt * DKP + c, a.q + at);
                mm_copy16(bk + tt * DKP + c, a.k + at);
            }
        }
        for (int i = threadIdx.x; i < n * (COLS / 4); i += THREADS) {
            const int tt = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
            if (col0 + c < a.v_row) mm_copy16(bv + tt * COLS + c, a.v + ((size_t)(t0 + tt) * H + h) * a.v_row + col0 + c);
        }
        if (a.fade) for (int i = threadIdx.x; i < n; i += THREADS) mm_copy4(bf + i, a.fade + (size_t)(t0 + i) * H + h);
    };
    dd_grid_wait();
    const float fixed = a.fade ? 0.f : a.fixed[h];
    float* sp = a.state + ((size_t)a.entry_slot[e] * H + h) * a.cols * DKP + sub * 4;
    f32x2 s[C][R / 2];
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int col = min(col0 + my_col + c, a.cols - 1);
#pragma unroll
        for (int p = 0; p < P; ++p) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(sp + (size_t)col * DKP + p * 4 * LPC);
            s[c][2 * p] = x.x; s[c][2 * p + 1] = x.y;
        }
    }
    __syncthreads();                                    // the zeros are written before any copy lands
    if (start < end) stage(start, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    int buf = 0;
    for (int t0 = start; t0 < end; t0 += MM_TOKENS, buf ^= 1) {
        const int n = min(MM_TOKENS, end - t0);
        if (t0 + MM_TOKENS < end) {
            if (t0 + 2 * MM_TOKENS > end) {             // the last, shorter run: its buffer holds older tokens behind it
                float* b = staged + (buf ^ 1) * BUF;
                const int left = end - t0 - MM_TOKENS;
                for (int i = threadIdx.x + left * DKP; i < MM_TOKENS * DKP; i += THREADS) {
                    b[i] = 0.f;
                    b[MM_TOKENS * DKP + i] = 0.f;
                }
                for (int i = threadIdx.x + left; i < MM_TOKENS; i += THREADS) b[MM_TOKENS * (2 * DKP + COLS) + i] = 0.f;
            }
            stage(t0 + MM_TOKENS, buf ^ 1);             // (that buffer's tokens were read before the last barrier)
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float* sq = staged + buf * BUF + sub * 4;
        const float* sv = staged + buf * BUF + 2 * MM_TOKENS * DKP + my_col;
        const float* sf = staged + buf * BUF + MM_TOKENS * (2 * DKP + COLS);
        // A token's operands are requested while the token before is worked through.
        f32x2 ops[2][2][R / 2], ff[2];
        float vv[2][C];
        auto fetch = [&](int tt, int slot) {
#pragma unroll
            for (int w = 0; w < 2; ++w)
#pragma unroll
                for (int p = 0; p < P; ++p) {
                    const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(sq + (w * MM_TOKENS + tt) * DKP + p * 4 * LPC);
                    ops[slot][w][2 * p] = x.x; ops[slot][w][2 * p + 1] = x.y;
                }
#pragma unroll
            for (int c = 0; c < C; ++c) vv[slot][c] = sv[tt * COLS + c];
            // a fixed fade does not touch the tokens past the end either: the state would fade
            const float lost = -(a.fade ? sf[tt] : (tt < n ? fixed : 0.f));
            ff[slot] = mm_pack(lost, lost);
        };
        fetch(0, 0);
        // (all sixteen, tokens of zeros among them: one group's exchanges then lie under the next group's products)
#pragma unroll
        for (int tt0 = 0; tt0 < MM_TOKENS; tt0 += 4) {
            float read[4 * C];                          // index token * C + column
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int slot = j & 1;
                fetch(min(tt0 + j + 1, MM_TOKENS - 1), slot ^ 1);
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    const f32x2 value = mm_pack(vv[slot][c], vv[slot][c]);
                    f32x2 part;
#pragma unroll
                    for (int i = 0; i < R / 2; ++i) {
                        s[c][i] = mm_fma2(ops[slot][1][i], value, mm_fma2(ff[slot], s[c][i], s[c][i]));
                        part = i ? mm_fma2(s[c][i], ops[slot][0][i], part) : mm_mul2(s[c][i], ops[slot][0][i]);
                    }
                    read[j * C + c] = mm_half_sum(part);
                }
            }
            const int first = mm_spread_sums<4 * C, 1, LPC>(read, sub);
            constexpr int MINE = 4 * C / LPC > 1 ? 4 * C / LPC : 1;      // sums a lane is left with
            const bool writes = LPC <= 4 * C || sub < 4 * C;            // (more lanes than sums: the others hold copies)
#pragma unroll
            for (int i = 0; i < MINE; ++i) {
                const int tt = tt0 + (first + i) / C, c = (first + i) % C;
                const int col = col0 + my_col + c;
                if (writes && tt < n && col < a.cols) a.out[((size_t)(t0 + tt) * H + h) * a.v_row + col] = read[i];
            }
        }
        __syncthreads();                                // all have read this buffer before the copies after next fill it
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (start < end) {
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int col = col0 + my_col + c;
            if (col >= a.cols) continue;
#pragma unroll
            for (int p = 0; p < P; ++p)
                *reinterpret_cast<ulonglong2*>(sp + (size_t)col * DKP + p * 4 * LPC) = make_ulonglong2(s[c][2 * p], s[c][2 * p + 1]);
        }
    }
}

struct StepArgs {
    int stride;                  // of q, k, v and gate
    float q_scale;
    int silu;
    const float* z;              // gate projections [N, z_stride] (input gates, then forget gates), or null: fixed
    int z_stride;
    float cap;
    const float* fixed;          // [H]
    float* peak;                 // [slots, H]
    const int* entry_slot;
    float* state;                // [slots, H, dv (+ 1), DKP]
    const float* weight;         // [H * dv] (FUSED)
    float eps, den_eps;
    int out_stride;
    float* o;                    // [N, H, v_row] (not FUSED)
    float* floor_out;            // [N, H] (not FUSED, gated)
    int H, dk, dv, v_row;
};

// Single tokens: token t is entry t. A cluster owns (entry, head), its blocks share the columns out. Gated: every block works
// n out for itself (it needs n . q), an element a thread; the first block writes it and the maximum, once all have read them.
constexpr int ST_THREADS = 256, ST_AHEAD = 2;
template <typename T, int LPC, bool FUSED>
__global__ void __launch_bounds__(ST_THREADS)
memory_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ gate,
                   T* __restrict__ out, const StepArgs a) {
    constexpr int DKP = 8 * LPC, COLS = ST_THREADS / LPC;
    extern __shared__ __align__(16) float sh[];          // q, k [DKP] each, then v and o of the block's columns
    __shared__ float scratch[8], n_parts[8], parts[8];
    dd_launch_dependents();
    const int slice = blockIdx.x, slices = gridDim.x, h = blockIdx.y, e = blockIdx.z;
    cg::cluster_group cluster = cg::this_cluster();
    if (FUSED && slices > 1) cluster.barrier_arrive();   // (waited for before the first write into another block's memory)
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int my_col = tid / LPC, sub = tid % LPC;
    const bool gated = a.z != nullptr;
    const int per = (a.dv + slices - 1) / slices;
    const int c_from = min(slice * per, a.dv), mine = min(per, a.dv - c_from);
    float *sq = sh, *sk = sq + DKP, *sv = sk + DKP, *so = sv + per;
    const int slot = a.entry_slot[e];
    float* base = a.state + ((size_t)slot * a.H + h) * (a.dv + (gated ? 1 : 0)) * DKP;
    float* n_at = base + (size_t)a.dv * DKP + tid;       // (gated, tid < DKP)
    for (int c = tid; c < mine * DKP / 32; c += ST_THREADS)      // the block's columns on their way into L2 (one line a thread)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(base + (size_t)c_from * DKP + (size_t)c * 32));
    dd_grid_wait();
    const size_t row = (size_t)e * a.stride;
    float now = 0.f;
    MemoryGates g = {0.f, 1.f, 0.f};
    if (gated) {
        float i, f;
        mm_log_gates(a.z[(size_t)e * a.z_stride + h], a.z[(size_t)e * a.z_stride + a.H + h], a.cap, i, f);
        const float before = a.peak[(size_t)slot * a.H + h];
        now = fmaxf(__fadd_rn(f, before), i);
        g = mm_gates(i, f, before, now);
    } else {
        g.fade = a.fixed[h];
    }
    auto act = [&](T x) {
        const float f = dd_to_f32(x);
        return a.silu ? mm_silu(f) : f;
    };
    for (int i = tid; i < DKP; i += ST_THREADS) {
        sq[i] = i < a.dk ? act(q[row + (size_t)h * a.dk + i]) * a.q_scale : 0.f;
        sk[i] = i < a.dk ? act(k[row + (size_t)h * a.dk + i]) * g.take : 0.f;
    }
    for (int i = tid; i < mine; i += ST_THREADS) sv[i] = act(v[row + (size_t)h * a.dv + c_from + i]);
    const float n_before = gated && tid < DKP ? *n_at : 0.f;
    const size_t at = (size_t)h * a.dv + c_from;
    // the gate and weight of a thread's first element, ready when the sum of squares is
    const float gate_ahead = FUSED && tid < mine ? dd_to_f32(gate[row + at + tid]) : 0.f, weight_ahead = FUSED && tid < mine ? a.weight[at + tid] : 0.f;
    __syncthreads();
    float n_now = 0.f;
    if (gated) {
        if (tid < DKP) n_now = mm_update(n_before, g.fade, sk[tid], 1.0f);
        const float part = dd_warp_sum(tid < DKP ? n_now * sq[tid] : 0.f);
        if (lane == 0) n_parts[warp] = part;
    }
    const float4 qa = *reinterpret_cast<const float4*>(sq + sub * 8), qb = *reinterpret_cast<const float4*>(sq + sub * 8 + 4);
    const float4 ka = *reinterpret_cast<const float4*>(sk + sub * 8), kb = *reinterpret_cast<const float4*>(sk + sub * 8 + 4);
    const float qq[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
    const float kk[8] = {ka.x, ka.y, ka.z, ka.w, kb.x, kb.y, kb.z, kb.w};
    base += (size_t)c_from * DKP + sub * 8;
    for (int c0 = my_col; c0 - my_col < mine; c0 += ST_AHEAD * COLS) {
        float s[ST_AHEAD][8];
#pragma unroll
        for (int w = 0; w < ST_AHEAD; ++w) {
            const float* sp = base + (size_t)min(c0 + w * COLS, mine - 1) * DKP;
            const float4 x = *reinterpret_cast<const float4*>(sp), y = *reinterpret_cast<const float4*>(sp + 4);
            s[w][0] = x.x; s[w][1] = x.y; s[w][2] = x.z; s[w][3] = x.w; s[w][4] = y.x; s[w][5] = y.y; s[w][6] = y.z; s[w][7] = y.w;
        }
#pragma unroll
        for (int w = 0; w < ST_AHEAD; ++w) {
            const int c = c0 + w * COLS;
            const float vv = sv[min(c, mine - 1)];
            float even = 0.f, odd = 0.f;
#pragma unroll
            for (int i = 0; i < 8; i += 2) {
                s[w][i] = mm_update(s[w][i], g.fade, kk[i], vv);
                s[w][i + 1] = mm_update(s[w][i + 1], g.fade, kk[i + 1], vv);
                even = __fmaf_rn(s[w][i], qq[i], even);
                odd = __fmaf_rn(s[w][i + 1], qq[i + 1], odd);
            }
            float read = even + odd;
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) read += __shfl_xor_sync(0xffffffffu, read, o);
            if (c < mine) {
                float* sp = base + (size_t)c * DKP;
                *reinterpret_cast<float4*>(sp) = make_float4(s[w][0], s[w][1], s[w][2], s[w][3]);
                *reinterpret_cast<float4*>(sp + 4) = make_float4(s[w][4], s[w][5], s[w][6], s[w][7]);
                if (sub == 0) so[c] = read;
            }
        }
    }
    __syncthreads();
    float n_dot_q = 0.f;
    if (gated) {
#pragma unroll
        for (int w = 0; w < ST_THREADS / 32; ++w) n_dot_q += n_parts[w];
    }
    if (FUSED) {
        const float over = gated ? 1.0f / (fmaxf(fabsf(n_dot_q), g.floor) + a.den_eps) : 1.0f;
        float sum = 0.f;
        for (int i = tid; i < mine; i += ST_THREADS) {
            const float x = so[i] * over;
            so[i] = x;
            sum = fmaf(x, x, sum);
        }
        sum = dd_warp_sum(sum);
        if (lane == 0) scratch[warp] = sum;
        __syncthreads();
        sum = 0.f;
#pragma unroll
        for (int w = 0; w < ST_THREADS / 32; ++w) sum += scratch[w];
        if (slices > 1) {
            cluster.barrier_wait();                      // every block of the cluster has started
            if (tid < slices) *cluster.map_shared_rank(&parts[slice], tid) = sum;
            cluster.sync();
            sum = 0.f;
            for (int w = 0; w < slices; ++w) sum += parts[w];
        }
        const float inv = 1.0f / sqrtf(sum / (float)a.dv + a.eps);
        for (int i = tid; i < mine; i += ST_THREADS) {
            const float z = i == tid ? gate_ahead : dd_to_f32(gate[row + at + i]), w = i == tid ? weight_ahead : a.weight[at + i];
            out[(size_t)e * a.out_stride + at + i] = dd_from_f32<T>(so[i] * inv * w * mm_sigmoid(z));
        }
    } else {
        float* o = a.o + ((size_t)e * a.H + h) * a.v_row;
        for (int i = tid; i < mine; i += ST_THREADS) o[c_from + i] = so[i];
        if (gated && slice == 0 && tid == 0) {
            o[a.dv] = n_dot_q;
            a.floor_out[(size_t)e * a.H + h] = g.floor;
        }
        if (gated && slices > 1) cluster.sync();
    }
    if (gated && slice == 0) {                           // every block of the cluster has read the old n and the old maximum
        if (tid < DKP) *n_at = n_now;
        if (tid == 0) a.peak[(size_t)slot * a.H + h] = now;
    }
}

struct FinishArgs {
    const float* o;              // [N, H, v_row]; element dv of a head is n . q where floor is given
    const float* floor;          // [N, H] or null
    const float* weight;         // [H * dv]
    float eps, den_eps;
    int gate_stride, out_stride, n_tokens, H, dv, v_row;
    int heads;                   // heads that are normed together: 1 or H
};

// A team of TEAM threads owns a stretch (a token's head, or a token's heads together); V elements a load, KEEP loads a thread
// kept in registers (beyond, it reads again).
template <typename T, int TEAM, int V, int KEEP>
__global__ void __launch_bounds__(256)
memory_finish_kernel(const T* __restrict__ gate, T* __restrict__ out, const FinishArgs a) {
    __shared__ float scratch[8];
    dd_launch_dependents();
    const int sub = threadIdx.x % TEAM, per_token = a.H / a.heads;
    const long long stretch = (long long)blockIdx.x * (256 / TEAM) + threadIdx.x / TEAM;
    const bool none = stretch >= (long long)a.n_tokens * per_token;      // (a team past the end: it still takes part in its warp's sums)
    const int t = none ? 0 : (int)(stretch / per_token), h0 = none ? 0 : (int)(stretch % per_token) * a.heads;
    const int size = none ? 0 : a.heads * a.dv;
    const float* w = a.weight + (size_t)h0 * a.dv;
    float weights[KEEP][V];                              // (parameters: read before the wait for the kernel before)
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (sub + j * TEAM) * V;
#pragma unroll
        for (int i = 0; i < V; ++i) weights[j][i] = c < size ? w[c + i] : 0.f;
    }
    dd_grid_wait();
    const float* row = a.o + (size_t)t * a.H * a.v_row;
    auto over_of = [&](int h) {
        return a.floor ? 1.0f / (fmaxf(fabsf(row[(size_t)h * a.v_row + a.dv]), a.floor[(size_t)t * a.H + h]) + a.den_eps) : 1.0f;
    };
    const float alone = a.heads == 1 ? over_of(h0) : 1.0f;
    auto load = [&](int c, float* x) {
        const int h = a.heads == 1 ? h0 : h0 + c / a.dv;
        const float over = a.heads == 1 ? alone : over_of(h);
        const float* at = row + (size_t)h * a.v_row + (c - (h - h0) * a.dv);
        if (V == 4) {
            const float4 y = *reinterpret_cast<const float4*>(at);
            x[0] = y.x * over; x[1] = y.y * over; x[2] = y.z * over; x[3] = y.w * over;
        } else {
            x[0] = *at * over;
        }
    };
    const T* g = gate + (size_t)t * a.gate_stride + (size_t)h0 * a.dv;
    T* dst = out + (size_t)t * a.out_stride + (size_t)h0 * a.dv;
    auto gate_of = [&](int c, float* z) {
        __align__(16) T gv[V];
        if (V == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(gv) = *reinterpret_cast<const uint2*>(g + c);
        else if (V == 4) *reinterpret_cast<uint4*>(gv) = *reinterpret_cast<const uint4*>(g + c);
        else gv[0] = g[c];
#pragma unroll
        for (int i = 0; i < V; ++i) z[i] = dd_to_f32(gv[i]);
    };
    float kept[KEEP][V], gates[KEEP][V];
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (sub + j * TEAM) * V;
        if (c < size) {
            load(c, kept[j]);
            gate_of(c, gates[j]);                        // (ready when the sum is)
#pragma unroll
            for (int i = 0; i < V; ++i) sum = fmaf(kept[j][i], kept[j][i], sum);
        }
    }
    for (int c = (sub + KEEP * TEAM) * V; c < size; c += TEAM * V) {
        float x[V];
        load(c, x);
#pragma unroll
        for (int i = 0; i < V; ++i) sum = fmaf(x[i], x[i], sum);
    }
#pragma unroll
    for (int o = (TEAM < 32 ? TEAM : 32) / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (TEAM > 32) {
        if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = sum;
        __syncthreads();
        sum = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) sum += scratch[w];
    }
    const float inv = 1.0f / sqrtf(sum / (float)size + a.eps);
    auto store = [&](int c, const float* x, const float* z, const float* by) {
        __align__(16) T y[V];
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = dd_from_f32<T>(x[i] * inv * by[i] * mm_sigmoid(z[i]));
        if (V == 4 && sizeof(T) == 2) *reinterpret_cast<uint2*>(dst + c) = *reinterpret_cast<const uint2*>(y);
        else if (V == 4) *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(y);
        else dst[c] = y[0];
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (sub + j * TEAM) * V;
        if (c < size) store(c, kept[j], gates[j], weights[j]);
    }
    for (int c = (sub + KEEP * TEAM) * V; c < size; c += TEAM * V) {
        float x[V], z[V];
        load(c, x);
        gate_of(c, z);
        store(c, x, z, w + c);
    }
}

int memory_lanes(int dk) {
    int lpc = 1;
    while (lpc * 8 < dk) lpc *= 2;
    return lpc;
}

template <typename T, int L, bool FUSED>
int launch_memory_step(const void* q, const void* k, const void* v, const void* gate, void* out, const StepArgs& a, int n_entries,
                       int slices, cudaStream_t s) {
    const int per = (a.dv + slices - 1) / slices;
    const size_t smem = (size_t)(2 * 8 * L + 2 * per) * sizeof(float);
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3(slices, a.H, n_entries);
    config.blockDim = dim3(ST_THREADS);
    config.dynamicSmemBytes = smem;
    config.stream = s;
    cudaLaunchAttribute attribute[2];
    attribute[0].id = cudaLaunchAttributeClusterDimension;
    attribute[0].val.clusterDim.x = slices;
    attribute[0].val.clusterDim.y = attribute[0].val.clusterDim.z = 1;
    attribute[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[1].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attribute;
    config.numAttrs = dd_pdl_enabled ? 2 : 1;
    cudaLaunchKernelEx(&config, memory_step_kernel<T, L, FUSED>, (const T*)q, (const T*)k, (const T*)v, (const T*)gate, (T*)out, a);
    return dd_check_launch("dd_memory_step");
}

template <typename T, bool FUSED>
int launch_memory_step_sized(int lpc, const void* q, const void* k, const void* v, const void* gate, void* out, const StepArgs& a,
                             int n_entries, int slices, cudaStream_t s) {
    switch (lpc) {
        case 1: return launch_memory_step<T, 1, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
        case 2: return launch_memory_step<T, 2, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
        case 4: return launch_memory_step<T, 4, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
        case 8: return launch_memory_step<T, 8, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
        case 16: return launch_memory_step<T, 16, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
        default: return launch_memory_step<T, 32, FUSED>(q, k, v, gate, out, a, n_entries, slices, s);
    }
}

template <typename T, int TEAM, int V, int KEEP>
int launch_memory_finish(const void* gate, void* out, const FinishArgs& a, cudaStream_t s) {
    const long long stretches = (long long)a.n_tokens * (a.H / a.heads);
    dd_launch(memory_finish_kernel<T, TEAM, V, KEEP>, dim3(dd_ceil_div(stretches, 256 / TEAM)), dim3(256), 0, s, (const T*)gate, (T*)out, a);
    return dd_check_launch("dd_memory_finish");
}

template <typename T>
int launch_memory_finish_sized(const void* gate, void* out, const FinishArgs& a, cudaStream_t s) {
    const bool wide = a.dv % 4 == 0 && a.gate_stride % 4 == 0 && a.out_stride % 4 == 0 &&
                      !(((uintptr_t)gate | (uintptr_t)out) & (4 * sizeof(T) - 1)) && !((uintptr_t)a.o & 15);
    const int size = a.heads * a.dv;
    if (!wide) return size <= 512 ? launch_memory_finish<T, 32, 1, 16>(gate, out, a, s) : launch_memory_finish<T, 256, 1, 16>(gate, out, a, s);
    if (size <= 64) return launch_memory_finish<T, 16, 4, 1>(gate, out, a, s);
    if (size <= 128) return launch_memory_finish<T, 32, 4, 1>(gate, out, a, s);
    if (size <= 512) return launch_memory_finish<T, 32, 4, 4>(gate, out, a, s);
    if (size <= 2048) return launch_memory_finish<T, 256, 4, 2>(gate, out, a, s);
    return launch_memory_finish<T, 256, 4, 4>(gate, out, a, s);
}
}  // namespace

// z: float32 rows of z_stride with H input-gate projections followed by H forget-gate projections; peak: float32 [slots, H],
// read and written; fade, take, floor_out: float32 [N, H].
DD_API int dd_memory_gates(const float* z, int z_stride, float cap, const int* entry_start, const int* entry_slot, int n_entries,
                           float* peak, float* fade, float* take, float* floor_out, int H, void* stream) {
    if (n_entries <= 0) return 0;
    if (H <= 0 || n_entries > 65535 || !(cap > 0.f) || z_stride < 2 * H) return dd_fail("dd_memory_gates: bad sizes (%d heads)", H);
    dd_launch(memory_gates_kernel, dim3(H, n_entries), dim3(MG_TOKENS), 0, (cudaStream_t)stream, z, z_stride, cap, entry_start, entry_slot,
              peak, fade, take, floor_out, H);
    return dd_check_launch("dd_memory_gates");
}

// q, k: [N] rows of `stride` elements with H heads of dk, v likewise with heads of dv; take: float32 [N, H] or null (1).
// q_out, k_out: float32 [N, H, roundup(dk, 4)]; v_out: float32 [N, H, roundup(dv + ones, 4)] (16-byte aligned).
DD_API int dd_memory_prepare(const void* q, const void* k, const void* v, int stride, float q_scale, int silu, const float* take,
                             float* q_out, float* k_out, float* v_out, int n, int H, int dk, int dv, int ones, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || dk <= 0 || dv <= 0 || (ones != 0 && ones != 1)) return dd_fail("dd_memory_prepare: bad sizes");
    if (((uintptr_t)q_out | (uintptr_t)k_out | (uintptr_t)v_out) & 15) return dd_fail("dd_memory_prepare: outputs must be 16-byte aligned");
    cudaStream_t s = (cudaStream_t)stream;
    const int qk_row = (dk + 3) / 4 * 4, v_row = (dv + ones + 3) / 4 * 4;
    const int size = dtype == DD_F32 ? 4 : 2;
    const bool wide = dk % 4 == 0 && dv % 4 == 0 && stride % 4 == 0 && !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & (4 * size - 1));
    const dim3 grid(n, dd_ceil_div((long long)H * (2 * qk_row + v_row) / 4, 256));
#define DD_PREP(T, WIDE)                                                                                                           \
    dd_launch(memory_prepare_kernel<T, WIDE>, grid, dim3(256), 0, s, (const T*)q, (const T*)k, (const T*)v, stride, q_scale, silu, take, \
              q_out, k_out, v_out, H, dk, dv, ones, qk_row, v_row)
    if (dtype == DD_F32) { if (wide) DD_PREP(float, true); else DD_PREP(float, false); }
    else if (dtype == DD_BF16) { if (wide) DD_PREP(__nv_bfloat16, true); else DD_PREP(__nv_bfloat16, false); }
    else return dd_fail("dd_memory_prepare: unknown dtype %d", dtype);
#undef DD_PREP
    return dd_check_launch("dd_memory_prepare");
}

// Operands as dd_memory_prepare leaves them; fade: float32 [N, H], or null and fixed: float32 [H]; state: float32
// [slots, H, dv + ones, 8 * lanes], read and written; out: float32 [N, H, roundup(dv + ones, 4)].
DD_API int dd_memory_scan(const float* q, const float* k, const float* v, const float* fade, const float* fixed,
                          const int* entry_start, const int* entry_slot, int n_entries, float* state, float* out, int H, int dk,
                          int dv, int ones, void* stream) {
    if (n_entries <= 0) return 0;
    if (dk <= 0 || dk > 256 || dv <= 0 || H <= 0 || H > 65535 || n_entries > 65535 || (!fade && !fixed) || (ones != 0 && ones != 1))
        return dd_fail("dd_memory_scan: %d heads of %d by %d are not supported (keys of at most 256)", H, dk, dv);
    if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state) & 15) return dd_fail("dd_memory_scan: operands must be 16-byte aligned");
    ScanArgs a;
    a.q = q; a.k = k; a.v = v; a.fade = fade; a.fixed = fixed; a.entry_start = entry_start; a.entry_slot = entry_slot;
    a.state = state; a.out = out; a.H = H; a.cols = dv + ones; a.qk_row = (dk + 3) / 4 * 4; a.v_row = (dv + ones + 3) / 4 * 4;
    cudaStream_t s = (cudaStream_t)stream;
    // blocks of CB columns (more where a warp holds more)
#define DD_SCAN(R, C, L, CB)                                                                                            \
    do {                                                                                                                \
        constexpr int TH = L * CB / C > 32 ? L * CB / C : 32, COLS = TH / L * C;                                        \
        const size_t smem = (size_t)2 * (MM_TOKENS * (2 * R * L + COLS + 1)) * sizeof(float);                           \
        if (smem > 48 * 1024)                                                                                           \
            cudaFuncSetAttribute(memory_scan_kernel<R, C, L, TH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        dd_launch_in_order(memory_scan_kernel<R, C, L, TH>, dim3(dd_ceil_div(a.cols, COLS), H, n_entries), dim3(TH), smem, s, a);     \
    } while (0)
    switch (8 * memory_lanes(dk)) {
        case 8: DD_SCAN(4, 4, 2, 16); break;
        case 16: DD_SCAN(4, 4, 4, 16); break;
        case 32: DD_SCAN(4, 4, 8, 16); break;
        case 64: DD_SCAN(8, 2, 8, 16); break;
        case 128: DD_SCAN(8, 2, 16, 16); break;
        default: DD_SCAN(8, 4, 32, 32); break;
    }
#undef DD_SCAN
    return dd_check_launch("dd_memory_scan");
}

// A step of single tokens (token t is entry t). q, k, v, gate: [N] rows of `stride` elements. z (float32, see
// dd_memory_gates) and peak, or null and fixed: float32 [H]. weight (float32 [H * dv]) given: out receives the normed (per
// head), weighted, gated result, rows of out_stride; null: o (float32 [N, H, roundup(dv + gated, 4)]) and, gated, floor_out
// [N, H] receive what dd_memory_scan and dd_memory_gates leave. slices: blocks of a cluster that share a head's columns (1,
// 2, 4 or 8; at most dv).
DD_API int dd_memory_step(const void* q, const void* k, const void* v, const void* gate, int stride, float q_scale, int silu,
                          const float* z, int z_stride, float cap, const float* fixed, float* peak, const int* entry_slot,
                          int n_entries, float* state, const float* weight, float eps, float den_eps, void* out, int out_stride,
                          float* o, float* floor_out, int H, int dk, int dv, int slices, int dtype, void* stream) {
    if (n_entries <= 0) return 0;
    if (dk <= 0 || dk > 256 || dv <= 0 || dv > 4096 || H <= 0 || H > 65535 || n_entries > 65535)
        return dd_fail("dd_memory_step: %d heads of %d by %d are not supported (keys of at most 256, values of at most 4096)", H, dk, dv);
    if ((slices != 1 && slices != 2 && slices != 4 && slices != 8) || slices > dv) return dd_fail("dd_memory_step: %d slices", slices);
    if ((!z && !fixed) || (z && (!peak || !(cap > 0.f) || z_stride < 2 * H)) || (weight ? !out || !gate : !o || (z && !floor_out)))
        return dd_fail("dd_memory_step: operands are missing");
    if ((uintptr_t)state & 15) return dd_fail("dd_memory_step: the state must be 16-byte aligned");
    StepArgs a;
    a.stride = stride; a.q_scale = q_scale; a.silu = silu; a.z = z; a.z_stride = z_stride; a.cap = cap; a.fixed = fixed;
    a.peak = peak; a.entry_slot = entry_slot; a.state = state; a.weight = weight; a.eps = eps; a.den_eps = den_eps;
    a.out_stride = out_stride; a.o = o; a.floor_out = floor_out; a.H = H; a.dk = dk; a.dv = dv;
    a.v_row = (dv + (z ? 1 : 0) + 3) / 4 * 4;
    cudaStream_t s = (cudaStream_t)stream;
    const int lpc = memory_lanes(dk);
    if (dtype == DD_F32)
        return weight ? launch_memory_step_sized<float, true>(lpc, q, k, v, gate, out, a, n_entries, slices, s)
                      : launch_memory_step_sized<float, false>(lpc, q, k, v, gate, out, a, n_entries, slices, s);
    if (dtype == DD_BF16)
        return weight ? launch_memory_step_sized<__nv_bfloat16, true>(lpc, q, k, v, gate, out, a, n_entries, slices, s)
                      : launch_memory_step_sized<__nv_bfloat16, false>(lpc, q, k, v, gate, out, a, n_entries, slices, s);
    return dd_fail("dd_memory_step: unknown dtype %d", dtype);
}

// o: float32 [N, H, roundup(dv + gated, 4)] as dd_memory_scan leaves it; floor: float32 [N, H] (gated) or null; gate and out:
// rows in `dtype`; weight: float32 [H * dv]; together: all heads of a token are normed as one stretch.
DD_API int dd_memory_finish(const float* o, const float* floor, const void* gate, int gate_stride, const float* weight, float eps,
                            float den_eps, int together, void* out, int out_stride, int n_tokens, int H, int dv, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || dv <= 0) return dd_fail("dd_memory_finish: bad sizes");
    FinishArgs a;
    a.o = o; a.floor = floor; a.weight = weight; a.eps = eps; a.den_eps = den_eps; a.gate_stride = gate_stride;
    a.out_stride = out_stride; a.n_tokens = n_tokens; a.H = H; a.dv = dv; a.v_row = (dv + (floor ? 1 : 0) + 3) / 4 * 4;
    a.heads = together ? H : 1;
    if (dtype == DD_F32) return launch_memory_finish_sized<float>(gate, out, a, (cudaStream_t)stream);
    if (dtype == DD_BF16) return launch_memory_finish_sized<__nv_bfloat16>(gate, out, a, (cudaStream_t)stream);
    return dd_fail("dd_memory_finish: unknown dtype %d", dtype);
}
