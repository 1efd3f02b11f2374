// Time mixing with a matrix state per head and a decay per key channel that depends on the token, and the norms whose
// rows are blended with the row of the token before.
//
// dd_token_mix reads the float32 stream once and leaves up to two normed rows (two weights over the same root mean
// square) and `n_mix` blends of the first one with the row before it in its sequence,
//     mix_s[t] = n[t] + (n[t-1] - n[t]) * mu_s,     n[t] = x[t] / sqrt(mean(x[t]^2) + eps) * (offset + w),
// all float32 inside and rounded once to the engine's type. n[t-1] of a step's first token is the float32 row the
// request's state slot holds (zeros for a new request). The block of an entry's first token alone touches the slot's row:
// it reads it, then leaves the normed row of the entry's last token there. A block norms its own row and the row before
// (or the entry's last) by the same arithmetic, so n[t-1] has the same bits from the state as computed again.
//
// Per head, token by token, with S [dk, dv] float32 (row i belongs to key channel i), w = exp(-exp(x + w0)):
//     o = (S + diag(u) k v^T)^T r = S^T r + (sum_i r_i u_i k_i) v;     S <- diag(w) S + k v^T
// The decay travels as its distance from one, 1 - w = -expm1(-exp(.)), which float32 holds far more exactly for a channel
// that decays slowly than w itself: S <- S - (1 - w) S + k v.
//
//   dd_time_prepare   the operands of a step as float32 rows: r, k, v, 1 - w, and the bonus sum_i r_i u_i k_i per head
//   dd_time_scan      the recurrence over a step's entries. Column j of o depends on column j of S only: a block owns
//                     (entry, head, a run of columns); a column's rows are dealt out over neighbouring lanes, and a thread
//                     holds the same few rows of several columns in registers, so that an operand it reads from shared
//                     memory serves them all. No token's update waits for an exchange between lanes: only the read-outs
//                     are exchanged, those of four tokens together (spread_sums). Tokens are staged 16 at a time by
//                     cp.async, two buffers in turn.
//   dd_time_step      a step of single tokens in one kernel: operands, recurrence, and the read-out's norm, weight and gate;
//                     a block owns (entry, head), a thread eight rows of a column. The state's update is the scan's, bit for
//                     bit.
// The state is stored column by column ([slots, heads, dv, dkp], dkp = dk rounded up to 8 times a power of two; rows past dk stay zero).
#include "common.cuh"

namespace {
// Explicit roundings: a normed value has the same bits whether it is blended at once or kept in the state first.
__device__ __forceinline__ float tm_normed(float x, float r, float w) { return __fmul_rn(__fmul_rn(x, r), w); }
__device__ __forceinline__ float tm_blend(float n, float p, float mu) { return __fmaf_rn(__fsub_rn(p, n), mu, n); }

template <typename T> struct Pack4;
template <> struct Pack4<float> {
    __device__ static void store(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
};
template <> struct Pack4<__nv_bfloat16> {
    __device__ static void store(__nv_bfloat16* dst, float4 v) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        uint2 p;
        p.x = *reinterpret_cast<uint32_t*>(&lo);
        p.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(dst) = p;
    }
};

struct MixArgs {
    const float* x;              // [rows, width]
    const float* weight;         // [width]
    const float* weight2;        // [width] or null
    const float* mu;             // [n_mix, width]
    float* state;                // [slots, width] (n_mix > 0)
    const int* tok_entry;
    const int* entry_start;
    const int* entry_slot;
    int rows, width, n_mix;
    long long plane;             // elements between two blends' rows of token 0
    float eps, offset;
};

// Both sums over the block, in one order whatever the rows are (scratch: 2 * warps floats).
template <int THREADS>
__device__ __forceinline__ void tm_block_sums(float& a, float& b, float* scratch) {
    a = dd_warp_sum(a);
    b = dd_warp_sum(b);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __syncthreads();
    if (lane == 0) { scratch[warp] = a; scratch[THREADS / 32 + warp] = b; }
    __syncthreads();
    a = b = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) { a += scratch[w]; b += scratch[THREADS / 32 + w]; }
}

// Rows of width 4 * VPT * 256 at most, 16-byte aligned: a thread keeps its channels of the row and of the row before in
// registers. A block walks `per_block` consecutive tokens, so that the weights, and inside an entry the row before, are
// there already. S: the number of blends, -1: any number (their weights are read when they are used).
template <typename T, int VPT, int S>
__global__ void __launch_bounds__(256)
token_mix_vec_kernel(const MixArgs a, T* __restrict__ out1, T* __restrict__ out2, T* __restrict__ mixes, int per_block) {
    __shared__ float scratch[16];
    constexpr int SK = S > 0 ? S : 1;
    dd_launch_dependents();
    const int n4 = a.width >> 2;
    float4 w1[VPT], w2[VPT], mu[SK][VPT];
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * 256;
        const bool in = c < n4;
        w1[i] = in ? __ldg(reinterpret_cast<const float4*>(a.weight) + c) : zero;
        w2[i] = in && a.weight2 ? __ldg(reinterpret_cast<const float4*>(a.weight2) + c) : zero;
        w1[i].x += a.offset; w1[i].y += a.offset; w1[i].z += a.offset; w1[i].w += a.offset;
        w2[i].x += a.offset; w2[i].y += a.offset; w2[i].z += a.offset; w2[i].w += a.offset;
        if (S > 0) {
#pragma unroll
            for (int s = 0; s < SK; ++s) mu[s][i] = in ? __ldg(reinterpret_cast<const float4*>(a.mu + (size_t)s * a.width) + c) : zero;
        }
    }
    const int t0 = blockIdx.x * per_block, t1 = min(a.rows, t0 + per_block);
    dd_grid_wait();
    float4 prev[VPT];
    for (int t = t0; t < t1; ++t) {
        const float4* in4 = reinterpret_cast<const float4*>(a.x + (size_t)t * a.width);
        float4 v[VPT], other[VPT];
        float sq = 0.f, sq2 = 0.f;
        int first = -1, last = -1;
        float* kept = nullptr;
        if (S != 0) {
            const int e = a.tok_entry[t];
            first = a.entry_start[e];
            last = a.entry_start[e + 1] - 1;
            kept = a.state + (size_t)a.entry_slot[e] * a.width;
        }
        // the second row that is normed with this one: the entry's last row (it goes into the state) for the entry's first
        // token, the row before for the block's first token inside an entry, none where the walk has it already
        const bool is_first = S != 0 && t == first;
        const float* also = nullptr;
        if (S != 0) {
            if (is_first) also = last != t ? a.x + (size_t)last * a.width : nullptr;
            else if (t == t0) also = a.x + (size_t)(t - 1) * a.width;
        }
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + i * 256;
            v[i] = c < n4 ? in4[c] : zero;
            other[i] = also && c < n4 ? reinterpret_cast<const float4*>(also)[c] : zero;
            if (is_first) prev[i] = c < n4 ? reinterpret_cast<const float4*>(kept)[c] : zero;
        }
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            sq += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
            sq2 += (other[i].x * other[i].x + other[i].y * other[i].y) + (other[i].z * other[i].z + other[i].w * other[i].w);
        }
        tm_block_sums<256>(sq, sq2, scratch);
        const float r = 1.0f / sqrtf(sq / (float)a.width + a.eps), r2 = 1.0f / sqrtf(sq2 / (float)a.width + a.eps);
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + i * 256;
            if (c >= n4) continue;
            const float4 n = make_float4(tm_normed(v[i].x, r, w1[i].x), tm_normed(v[i].y, r, w1[i].y), tm_normed(v[i].z, r, w1[i].z), tm_normed(v[i].w, r, w1[i].w));
            if (out1) Pack4<T>::store(out1 + (size_t)t * a.width + 4 * c, n);
            if (out2)
                Pack4<T>::store(out2 + (size_t)t * a.width + 4 * c,
                                make_float4(tm_normed(v[i].x, r, w2[i].x), tm_normed(v[i].y, r, w2[i].y), tm_normed(v[i].z, r, w2[i].z), tm_normed(v[i].w, r, w2[i].w)));
            if (S != 0) {
                const float4 o = make_float4(tm_normed(other[i].x, r2, w1[i].x), tm_normed(other[i].y, r2, w1[i].y), tm_normed(other[i].z, r2, w1[i].z), tm_normed(other[i].w, r2, w1[i].w));
                if (!is_first && t == t0) prev[i] = o;
                const int count = S > 0 ? S : a.n_mix;
#pragma unroll
                for (int s = 0; s < count; ++s) {
                    const float4 m = S > 0 ? mu[S > 0 ? s : 0][i] : __ldg(reinterpret_cast<const float4*>(a.mu + (size_t)s * a.width) + c);
                    Pack4<T>::store(mixes + (size_t)s * a.plane + (size_t)t * a.width + 4 * c,
                                    make_float4(tm_blend(n.x, prev[i].x, m.x), tm_blend(n.y, prev[i].y, m.y), tm_blend(n.z, prev[i].z, m.z), tm_blend(n.w, prev[i].w, m.w)));
                }
                if (is_first) reinterpret_cast<float4*>(kept)[c] = also ? o : n;
                prev[i] = n;
            }
        }
    }
}

// Any width and alignment: a block a token, rows read twice.
template <typename T>
__global__ void __launch_bounds__(256)
token_mix_kernel(const MixArgs a, T* __restrict__ out1, T* __restrict__ out2, T* __restrict__ mixes) {
    __shared__ float scratch[16];
    dd_launch_dependents();
    dd_grid_wait();
    const int t = blockIdx.x;
    const float* in = a.x + (size_t)t * a.width;
    const float* also = nullptr;
    float* kept = nullptr;
    bool is_first = false;
    if (a.n_mix > 0) {
        const int e = a.tok_entry[t];
        const int last = a.entry_start[e + 1] - 1;
        is_first = t == a.entry_start[e];
        kept = a.state + (size_t)a.entry_slot[e] * a.width;
        also = is_first ? (last != t ? a.x + (size_t)last * a.width : nullptr) : in - a.width;
    }
    float sq = 0.f, sq2 = 0.f;
    for (int c = threadIdx.x; c < a.width; c += 256) {
        sq += in[c] * in[c];
        if (also) sq2 += also[c] * also[c];
    }
    tm_block_sums<256>(sq, sq2, scratch);
    const float r = 1.0f / sqrtf(sq / (float)a.width + a.eps), r2 = 1.0f / sqrtf(sq2 / (float)a.width + a.eps);
    for (int c = threadIdx.x; c < a.width; c += 256) {
        const float w = a.offset + a.weight[c];
        const float n = tm_normed(in[c], r, w), o = also ? tm_normed(also[c], r2, w) : 0.f;
        if (out1) out1[(size_t)t * a.width + c] = dd_from_f32<T>(n);
        if (out2) out2[(size_t)t * a.width + c] = dd_from_f32<T>(tm_normed(in[c], r, a.offset + a.weight2[c]));
        if (a.n_mix > 0) {
            const float p = is_first ? kept[c] : o;
            for (int s = 0; s < a.n_mix; ++s)
                mixes[(size_t)s * a.plane + (size_t)t * a.width + c] = dd_from_f32<T>(tm_blend(n, p, a.mu[(size_t)s * a.width + c]));
            if (is_first) kept[c] = also ? o : n;
        }
    }
}

template <typename T>
int launch_token_mix(const MixArgs& a, void* out1, void* out2, void* mixes, cudaStream_t s) {
    const bool wide = a.width % 4 == 0 && a.width <= 4096 && a.plane % 4 == 0 &&
                      !(((uintptr_t)a.x | (uintptr_t)a.weight | (uintptr_t)a.weight2 | (uintptr_t)a.mu | (uintptr_t)a.state |
                         (uintptr_t)out1 | (uintptr_t)out2 | (uintptr_t)mixes) & 15);
    if (!wide) {
        dd_launch(token_mix_kernel<T>, dim3(a.rows), dim3(256), 0, s, a, (T*)out1, (T*)out2, (T*)mixes);
        return dd_check_launch("dd_token_mix");
    }
    // many tokens: a few to a block, so that weights are fetched and rows normed once for them all
    const int per_block = a.rows >= 4 * 148 * 4 ? 4 : a.rows >= 2 * 148 * 4 ? 2 : 1;
    const int grid = dd_ceil_div(a.rows, per_block);
#define DD_MIX(V, S) dd_launch(token_mix_vec_kernel<T, V, S>, dim3(grid), dim3(256), 0, s, a, (T*)out1, (T*)out2, (T*)mixes, per_block)
#define DD_MIX_S(V)                                                        \
    do {                                                                   \
        if (a.n_mix == 0) DD_MIX(V, 0);                                    \
        else if (a.n_mix == 5) DD_MIX(V, 5);                               \
        else DD_MIX(V, -1);                                                \
    } while (0)
    if (a.width <= 1024) DD_MIX_S(1);
    else if (a.width <= 2048) DD_MIX_S(2);
    else DD_MIX_S(4);
#undef DD_MIX_S
#undef DD_MIX
    return dd_check_launch("dd_token_mix");
}

// ---------------------------------------------------------------- the recurrence

template <int BYTES> __device__ __forceinline__ void tm_cp_async(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// 1 - exp(-exp(x)), exact for small decays
__device__ __forceinline__ float tm_fade(float x) { return -expm1f(-expf(x)); }

// A warp a (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
time_prepare_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, int stride,
                    const float* __restrict__ decay_in, const float* __restrict__ w0, const float* __restrict__ u,
                    float* __restrict__ r_out, float* __restrict__ k_out, float* __restrict__ v_out, float* __restrict__ fade_out,
                    float* __restrict__ bonus_out, int n_tokens, int H, int dk, int dv) {
    dd_launch_dependents();
    dd_grid_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * 8 + warp;
    if (item >= (long long)n_tokens * H) return;
    const int t = (int)(item / H), h = (int)(item % H);
    const size_t in = (size_t)t * stride + (size_t)h * dk, at = (size_t)item * dk;
    float bonus = 0.f;
    for (int i = lane; i < dk; i += 32) {
        const float rv = dd_to_f32(r[in + i]), kv = dd_to_f32(k[in + i]);
        r_out[at + i] = rv;
        k_out[at + i] = kv;
        fade_out[at + i] = tm_fade(decay_in[at + i] + w0[h * dk + i]);
        bonus = __fmaf_rn(__fmul_rn(rv, u[h * dk + i]), kv, bonus);
    }
    bonus = dd_warp_sum(bonus);
    if (lane == 0) bonus_out[item] = bonus;
    for (int i = lane; i < dv; i += 32) v_out[(size_t)item * dv + i] = dd_to_f32(v[(size_t)t * stride + (size_t)h * dv + i]);
}

// One token for a thread's eight rows of its column: the part of S^T r, then the state.
__device__ __forceinline__ float time_token(float (&s)[8], const float* r, const float* k, const float* f, float v) {
    const float4 r0 = *reinterpret_cast<const float4*>(r), r1 = *reinterpret_cast<const float4*>(r + 4);
    const float4 k0 = *reinterpret_cast<const float4*>(k), k1 = *reinterpret_cast<const float4*>(k + 4);
    const float4 f0 = *reinterpret_cast<const float4*>(f), f1 = *reinterpret_cast<const float4*>(f + 4);
    const float rr[8] = {r0.x, r0.y, r0.z, r0.w, r1.x, r1.y, r1.z, r1.w};
    const float kk[8] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w};
    const float ff[8] = {f0.x, f0.y, f0.z, f0.w, f1.x, f1.y, f1.z, f1.w};
    float a = 0.f, b = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        a = __fmaf_rn(s[i], rr[i], a);
        b = __fmaf_rn(s[4 + i], rr[4 + i], b);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i] = __fmaf_rn(kk[i], v, __fmaf_rn(-ff[i], s[i], s[i]));
    return __fadd_rn(a, b);
}

// N sums, of which every one of a column's LPC lanes holds a part: at every exchange (O = 1, 2, 4, .. lanes apart) a lane gives
// away half of its sums and keeps the other half while it has more than one, so that all of them together take little more
// exchanges than one would. Returns the index of the first sum the lane is left with, in read[0].
template <int N, int O, int LPC>
__device__ __forceinline__ int spread_sums(float* read, int sub) {
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
        return (up ? N / 2 : 0) + spread_sums<N / 2, O * 2, LPC>(read, sub);
    } else {
        read[0] += __shfl_xor_sync(0xffffffffu, read[0], O);
        return spread_sums<1, O * 2, LPC>(read, sub);
    }
}

constexpr int TS_TOKENS = 16;          // tokens staged together

// R rows and C columns of the state a thread (R a multiple of 4, 16-byte pieces that lie a whole sweep of the column's LPC
// lanes apart, so that neighbouring lanes read neighbouring pieces); THREADS / LPC * C columns a block.
template <int R, int C, int LPC, int THREADS>
__global__ void __launch_bounds__(THREADS)
time_scan_kernel(const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v, const float* __restrict__ fade,
                 const float* __restrict__ bonus, const int* __restrict__ entry_start, const int* __restrict__ entry_slot,
                 float* __restrict__ state, float* __restrict__ out, int H, int dk, int dv) {
    constexpr int DKP = R * LPC, COLS = THREADS / LPC * C, P = R / 4;
    constexpr int BUF = TS_TOKENS * (3 * DKP + COLS) + TS_TOKENS;       // floats of one buffer: r, k, fade, v, bonus
    extern __shared__ __align__(16) float staged[];
    dd_launch_dependents();
    const int e = blockIdx.z, h = blockIdx.y;
    const int col0 = blockIdx.x * COLS;
    const int my_col = threadIdx.x / LPC * C, sub = threadIdx.x % LPC;
    const int start = entry_start[e], end = entry_start[e + 1];
    // rows past dk and columns past dv are never copied into: they stay the zeros written here, and so do the tokens past
    // an entry's last one in its last buffer (a token of zeros leaves the state as it is)
    for (int i = threadIdx.x; i < 2 * BUF; i += THREADS) staged[i] = 0.f;
    const bool wide = dk % 4 == 0 && dv % 4 == 0 && COLS % 4 == 0;
    auto stage = [&](int t0, int buf) {
        const int n = min(TS_TOKENS, end - t0);
        float* br = staged + buf * BUF;
        float* bk = br + TS_TOKENS * DKP;
        float* bf = bk + TS_TOKENS * DKP;
        float* bv = bf + TS_TOKENS * DKP;
        float* bb = bv + TS_TOKENS * COLS;
        if (wide) {
            for (int i = threadIdx.x; i < n * (DKP / 4); i += THREADS) {
                const int tt = i / (DKP / 4), c = (i % (DKP / 4)) * 4;
                if (c < dk) {
                    const size_t at = ((size_t)(t0 + tt) * H + h) * dk + c;
                    tm_cp_async<16>(br + tt * DKP + c, r + at);
                    tm_cp_async<16>(bk + tt * DKP + c, k + at);
                    tm_cp_async<16>(bf + tt * DKP + c, fade + at);
                }
            }
            for (int i = threadIdx.x; i < n * (COLS / 4); i += THREADS) {
                const int tt = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
                if (col0 + c < dv) tm_cp_async<16>(bv + tt * COLS + c, v + ((size_t)(t0 + tt) * H + h) * dv + col0 + c);
            }
        } else {
            for (int i = threadIdx.x; i < n * DKP; i += THREADS) {
                const int tt = i / DKP, c = i % DKP;
                if (c < dk) {
                    const size_t at = ((size_t)(t0 + tt) * H + h) * dk + c;
                    tm_cp_async<4>(br + i, r + at);
                    tm_cp_async<4>(bk + i, k + at);
                    tm_cp_async<4>(bf + i, fade + at);
                }
            }
            for (int i = threadIdx.x; i < n * COLS; i += THREADS) {
                const int tt = i / COLS, c = i % COLS;
                if (col0 + c < dv) tm_cp_async<4>(bv + i, v + ((size_t)(t0 + tt) * H + h) * dv + col0 + c);
            }
        }
        for (int i = threadIdx.x; i < n; i += THREADS) tm_cp_async<4>(bb + i, bonus + (size_t)(t0 + i) * H + h);
    };
    dd_grid_wait();
    float* sp = state + ((size_t)entry_slot[e] * H + h) * dv * DKP + sub * 4;
    float s[C][R];
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int col = min(col0 + my_col + c, dv - 1);
#pragma unroll
        for (int p = 0; p < P; ++p) {
            const float4 x = *reinterpret_cast<const float4*>(sp + (size_t)col * DKP + p * 4 * LPC);
            s[c][4 * p] = x.x; s[c][4 * p + 1] = x.y; s[c][4 * p + 2] = x.z; s[c][4 * p + 3] = x.w;
        }
    }
    __syncthreads();                                    // the zeros are written before any copy lands
    if (start < end) stage(start, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    int buf = 0;
    for (int t0 = start; t0 < end; t0 += TS_TOKENS, buf ^= 1) {
        const int n = min(TS_TOKENS, end - t0);
        if (t0 + TS_TOKENS < end) {
            if (t0 + 2 * TS_TOKENS > end) {             // the last, shorter run: its buffer holds older tokens behind it
                float* b = staged + (buf ^ 1) * BUF;
                const int left = end - t0 - TS_TOKENS;
                for (int i = threadIdx.x + left * DKP; i < TS_TOKENS * DKP; i += THREADS) {
                    b[i] = 0.f;
                    b[TS_TOKENS * DKP + i] = 0.f;
                    b[2 * TS_TOKENS * DKP + i] = 0.f;
                }
            }
            stage(t0 + TS_TOKENS, buf ^ 1);             // (that buffer's tokens were read before the last barrier)
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float* sr = staged + buf * BUF + sub * 4;
        const float* sv = staged + buf * BUF + 3 * TS_TOKENS * DKP + my_col;
        const float* sb = staged + buf * BUF + TS_TOKENS * (3 * DKP + COLS);
        // A token's operands are requested while the token before is worked through.
        float ops[2][3][R], vv[2][C];
        auto fetch = [&](int tt, int slot) {
#pragma unroll
            for (int w = 0; w < 3; ++w)
#pragma unroll
                for (int p = 0; p < P; ++p) {
                    const float4 x = *reinterpret_cast<const float4*>(sr + (w * TS_TOKENS + tt) * DKP + p * 4 * LPC);
                    ops[slot][w][4 * p] = x.x; ops[slot][w][4 * p + 1] = x.y; ops[slot][w][4 * p + 2] = x.z; ops[slot][w][4 * p + 3] = x.w;
                }
#pragma unroll
            for (int c = 0; c < C; ++c) vv[slot][c] = sv[tt * COLS + c];
        };
        fetch(0, 0);
        // (all sixteen, tokens of zeros among them: one group's exchanges then lie under the next group's products)
#pragma unroll
        for (int tt0 = 0; tt0 < TS_TOKENS; tt0 += 4) {
            float read[4 * C];                          // index token * C + column
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int slot = j & 1;
                fetch(min(tt0 + j + 1, TS_TOKENS - 1), slot ^ 1);
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    float part[P];
#pragma unroll
                    for (int p = 0; p < P; ++p) {
                        part[p] = 0.f;
#pragma unroll
                        for (int i = 4 * p; i < 4 * p + 4; ++i) part[p] = __fmaf_rn(s[c][i], ops[slot][0][i], part[p]);
                    }
                    read[j * C + c] = part[0];
#pragma unroll
                    for (int p = 1; p < P; ++p) read[j * C + c] = __fadd_rn(read[j * C + c], part[p]);
#pragma unroll
                    for (int i = 0; i < R; ++i)
                        s[c][i] = __fmaf_rn(ops[slot][1][i], vv[slot][c], __fmaf_rn(-ops[slot][2][i], s[c][i], s[c][i]));
                }
            }
            const int first = spread_sums<4 * C, 1, LPC>(read, sub);
            constexpr int MINE = 4 * C / LPC > 1 ? 4 * C / LPC : 1;      // sums a lane is left with
            const bool writes = LPC <= 4 * C || sub < 4 * C;            // (more lanes than sums: the others hold copies)
#pragma unroll
            for (int i = 0; i < MINE; ++i) {
                const int tt = tt0 + (first + i) / C, c = (first + i) % C;
                const int col = col0 + my_col + c;
                if (writes && tt < n && col < dv)
                    out[((size_t)(t0 + tt) * H + h) * dv + col] = __fmaf_rn(sb[tt], sv[tt * COLS + c], read[i]);
            }
        }
        __syncthreads();                                // all have read this buffer before the copies after next fill it
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (start < end) {
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int col = col0 + my_col + c;
            if (col >= dv) continue;
#pragma unroll
            for (int p = 0; p < P; ++p)
                *reinterpret_cast<float4*>(sp + (size_t)col * DKP + p * 4 * LPC) = make_float4(s[c][4 * p], s[c][4 * p + 1], s[c][4 * p + 2], s[c][4 * p + 3]);
        }
    }
}

// Single tokens: token t is entry t. A block owns (entry, head).
constexpr int ST_THREADS = 256, ST_AHEAD = 2;
template <typename T, int LPC>
__global__ void __launch_bounds__(ST_THREADS)
time_step_kernel(const T* __restrict__ r, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ gate, int stride,
                 const float* __restrict__ decay_in, const float* __restrict__ w0, const float* __restrict__ u,
                 const float* __restrict__ weight, float eps, const int* __restrict__ entry_slot, float* __restrict__ state,
                 T* __restrict__ out, int out_stride, int H, int dk, int dv) {
    constexpr int DKP = 8 * LPC, COLS = ST_THREADS / LPC;
    extern __shared__ __align__(16) float sh[];          // r, k, fade [DKP] each, then v and o [dv] each
    __shared__ float scratch[8];
    float *sr = sh, *sk = sr + DKP, *sf = sk + DKP, *sv = sf + DKP, *so = sv + dv;
    dd_launch_dependents();
    const int h = blockIdx.x, e = blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int my_col = tid / LPC, sub = tid % LPC;
    float* base = state + ((size_t)entry_slot[e] * H + h) * dv * DKP + sub * 8;
    for (int c = tid; c < dv * DKP / 32; c += ST_THREADS)      // the head's state on its way into L2 (one line a thread)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(base - sub * 8 + (size_t)c * 32));
    dd_grid_wait();
    const size_t row = (size_t)e * stride;
    float bonus = 0.f;
    for (int i = tid; i < DKP; i += ST_THREADS) {
        float rv = 0.f, kv = 0.f, fv = 0.f;
        if (i < dk) {
            rv = dd_to_f32(r[row + (size_t)h * dk + i]);
            kv = dd_to_f32(k[row + (size_t)h * dk + i]);
            fv = tm_fade(decay_in[((size_t)e * H + h) * dk + i] + w0[h * dk + i]);
        }
        sr[i] = rv; sk[i] = kv; sf[i] = fv;
    }
    for (int i = tid; i < dv; i += ST_THREADS) sv[i] = dd_to_f32(v[row + (size_t)h * dv + i]);
    __syncthreads();
    // every warp adds up the bonus for itself, in the order of the operands' kernel
    for (int i = lane; i < dk; i += 32) bonus = __fmaf_rn(__fmul_rn(sr[i], u[h * dk + i]), sk[i], bonus);
    bonus = dd_warp_sum(bonus);
    for (int c0 = my_col; c0 - my_col < dv; c0 += ST_AHEAD * COLS) {
        float s[ST_AHEAD][8];
#pragma unroll
        for (int a = 0; a < ST_AHEAD; ++a) {
            const int col = min(c0 + a * COLS, dv - 1);
            const float4 x = *reinterpret_cast<const float4*>(base + (size_t)col * DKP), y = *reinterpret_cast<const float4*>(base + (size_t)col * DKP + 4);
            s[a][0] = x.x; s[a][1] = x.y; s[a][2] = x.z; s[a][3] = x.w; s[a][4] = y.x; s[a][5] = y.y; s[a][6] = y.z; s[a][7] = y.w;
        }
#pragma unroll
        for (int a = 0; a < ST_AHEAD; ++a) {
            const int col = c0 + a * COLS;
            const float vv = sv[min(col, dv - 1)];
            float read = time_token(s[a], sr + sub * 8, sk + sub * 8, sf + sub * 8, vv);
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1) read += __shfl_xor_sync(0xffffffffu, read, o);
            if (col < dv) {
                float* sp = base + (size_t)col * DKP;
                *reinterpret_cast<float4*>(sp) = make_float4(s[a][0], s[a][1], s[a][2], s[a][3]);
                *reinterpret_cast<float4*>(sp + 4) = make_float4(s[a][4], s[a][5], s[a][6], s[a][7]);
                if (sub == 0) so[col] = __fmaf_rn(bonus, vv, read);
            }
        }
    }
    __syncthreads();
    float sq = 0.f;
    for (int i = tid; i < dv; i += ST_THREADS) sq = fmaf(so[i], so[i], sq);
    sq = dd_warp_sum(sq);
    if (lane == 0) scratch[warp] = sq;
    __syncthreads();
    sq = 0.f;
#pragma unroll
    for (int w = 0; w < ST_THREADS / 32; ++w) sq += scratch[w];
    const float inv = 1.0f / sqrtf(sq / (float)dv + eps);
    T* dst = out + (size_t)e * out_stride + (size_t)h * dv;
    for (int i = tid; i < dv; i += ST_THREADS) {
        const float z = dd_to_f32(gate[row + (size_t)h * dv + i]);
        dst[i] = dd_from_f32<T>(so[i] * inv * weight[h * dv + i] * (z / (1.0f + expf(-z))));
    }
}

int lanes_of(int dk) {
    int lpc = 1;
    while (lpc * 8 < dk) lpc *= 2;
    return lpc;
}
}  // namespace

// x: float32 [rows, width]; weight (and weight2 or null): float32 [width]; out1/out2: [rows, width] or null (out2 needs
// weight2); n_mix blends with weights mu float32 [n_mix, width] to mixes, `plane` elements apart. state: float32
// [slots, width], read and written (n_mix > 0).
DD_API int dd_token_mix(const float* x, const float* weight, const float* weight2, const float* mu, int n_mix, float* state,
                        const int* tok_entry, const int* entry_start, const int* entry_slot, void* out1, void* out2, void* mixes,
                        long long plane, int rows, int width, float eps, float offset, int out_dtype, void* stream) {
    if (rows <= 0) return 0;
    if (width <= 0 || n_mix < 0 || (out2 && !weight2)) return dd_fail("dd_token_mix: bad sizes (width %d, %d blends)", width, n_mix);
    if (n_mix > 0 && (!mu || !state || !mixes || !tok_entry || !entry_start || !entry_slot || plane < (long long)rows * width))
        return dd_fail("dd_token_mix: blends need their weights, the state and room for %d rows", rows);
    MixArgs a;
    a.x = x; a.weight = weight; a.weight2 = weight2; a.mu = mu; a.state = state; a.tok_entry = tok_entry;
    a.entry_start = entry_start; a.entry_slot = entry_slot; a.rows = rows; a.width = width; a.n_mix = n_mix;
    a.plane = n_mix > 0 ? plane : 0; a.eps = eps; a.offset = offset;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == DD_F32) return launch_token_mix<float>(a, out1, out2, mixes, s);
    if (out_dtype == DD_BF16) return launch_token_mix<__nv_bfloat16>(a, out1, out2, mixes, s);
    return dd_fail("dd_token_mix: unknown output dtype %d", out_dtype);
}

// r, k: [N] rows of `stride` elements with H heads of dk, v likewise with heads of dv (one type); decay_in: float32
// [N, H * dk]; w0, u: float32 [H * dk]. Outputs float32, contiguous: r, k, fade [N, H * dk], v [N, H * dv], bonus [N, H].
DD_API int dd_time_prepare(const void* r, const void* k, const void* v, int stride, const float* decay_in, const float* w0,
                           const float* u, float* r_out, float* k_out, float* v_out, float* fade_out, float* bonus_out, int n,
                           int H, int dk, int dv, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || dk <= 0 || dv <= 0) return dd_fail("dd_time_prepare: bad sizes");
    cudaStream_t s = (cudaStream_t)stream;
    const int grid = dd_ceil_div((long long)n * H, 8);
#define DD_PREP(T)                                                                                                        \
    dd_launch(time_prepare_kernel<T>, dim3(grid), dim3(256), 0, s, (const T*)r, (const T*)k, (const T*)v, stride, decay_in, w0, u, \
              r_out, k_out, v_out, fade_out, bonus_out, n, H, dk, dv)
    if (dtype == DD_F32) DD_PREP(float);
    else if (dtype == DD_BF16) DD_PREP(__nv_bfloat16);
    else return dd_fail("dd_time_prepare: unknown dtype %d", dtype);
#undef DD_PREP
    return dd_check_launch("dd_time_prepare");
}

// Operands as dd_time_prepare leaves them; state: float32 [slots, H, dv, dd_delta_state_rows(dk)], read and written;
// out: float32 [N, H * dv].
DD_API int dd_time_scan(const float* r, const float* k, const float* v, const float* fade, const float* bonus,
                        const int* entry_start, const int* entry_slot, int n_entries, float* state, float* out, int H, int dk,
                        int dv, void* stream) {
    if (n_entries <= 0) return 0;
    if (dk <= 0 || dk > 256 || dv <= 0 || H <= 0 || H > 65535 || n_entries > 65535)
        return dd_fail("dd_time_scan: %d heads of %d by %d are not supported (keys of at most 256)", H, dk, dv);
    if (((uintptr_t)r | (uintptr_t)k | (uintptr_t)v | (uintptr_t)fade | (uintptr_t)state) & 15)
        return dd_fail("dd_time_scan: operands must be 16-byte aligned");
    cudaStream_t s = (cudaStream_t)stream;
    // blocks of 16 columns (more where a warp holds more)
#define DD_SCAN(R, C, L)                                                                                                \
    do {                                                                                                                \
        constexpr int TH = L * 16 / C > 32 ? L * 16 / C : 32, COLS = TH / L * C;                                        \
        const size_t smem = (size_t)2 * (TS_TOKENS * (3 * R * L + COLS + 1)) * sizeof(float);                           \
        if (smem > 48 * 1024)                                                                                           \
            cudaFuncSetAttribute(time_scan_kernel<R, C, L, TH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        dd_launch_in_order(time_scan_kernel<R, C, L, TH>, dim3(dd_ceil_div(dv, COLS), H, n_entries), dim3(TH), smem, s, r, k, v, \
                           fade, bonus, entry_start, entry_slot, state, out, H, dk, dv);                                \
    } while (0)
    switch (8 * lanes_of(dk)) {
        case 8: DD_SCAN(4, 4, 2); break;
        case 16: DD_SCAN(4, 4, 4); break;
        case 32: DD_SCAN(4, 4, 8); break;
        case 64: DD_SCAN(4, 4, 16); break;
        case 128: DD_SCAN(4, 4, 32); break;
        default: DD_SCAN(8, 2, 32); break;
    }
#undef DD_SCAN
    return dd_check_launch("dd_time_scan");
}

// A step of single tokens (token t is entry t): r, k, v, gate: [N] rows of `stride` elements; weight: float32 [H * dv] of the
// read-out's norm; out: [N, out_stride] rows of H * dv in the same type.
DD_API int dd_time_step(const void* r, const void* k, const void* v, const void* gate, int stride, const float* decay_in,
                        const float* w0, const float* u, const float* weight, float eps, const int* entry_slot, int n_entries,
                        float* state, void* out, int out_stride, int H, int dk, int dv, int dtype, void* stream) {
    if (n_entries <= 0) return 0;
    if (dk <= 0 || dk > 256 || dv <= 0 || dv > 4096 || H <= 0 || n_entries > 65535)
        return dd_fail("dd_time_step: %d heads of %d by %d are not supported (keys of at most 256)", H, dk, dv);
    if ((uintptr_t)state & 15) return dd_fail("dd_time_step: the state must be 16-byte aligned");
    cudaStream_t s = (cudaStream_t)stream;
    const int lpc = lanes_of(dk);
    const size_t smem = (size_t)(3 * 8 * lpc + 2 * dv) * sizeof(float);
#define DD_STEP(T, L)                                                                                                   \
    dd_launch(time_step_kernel<T, L>, dim3(H, n_entries), dim3(ST_THREADS), smem, s, (const T*)r, (const T*)k, (const T*)v,     \
              (const T*)gate, stride, decay_in, w0, u, weight, eps, entry_slot, state, (T*)out, out_stride, H, dk, dv)
#define DD_STEP_L(T)                                                    \
    switch (lpc) {                                                      \
        case 1: DD_STEP(T, 1); break;                                   \
        case 2: DD_STEP(T, 2); break;                                   \
        case 4: DD_STEP(T, 4); break;                                   \
        case 8: DD_STEP(T, 8); break;                                   \
        case 16: DD_STEP(T, 16); break;                                 \
        default: DD_STEP(T, 32); break;                                 \
    }
    if (dtype == DD_F32) { DD_STEP_L(float) }
    else if (dtype == DD_BF16) { DD_STEP_L(__nv_bfloat16) }
    else return dd_fail("dd_time_step: unknown dtype %d", dtype);
#undef DD_STEP_L
#undef DD_STEP
    return dd_check_launch("dd_time_step");
}
