// A sublayer's result normed and added to the float32 stream, and the stream's rounding that the next sublayer reads, in one
// pass over the stream:
//     y[t] = a_scale a[t] + b_scale b[t],    or the sum over a token's rows y[t] = sum_k rows[pair_row[t, k]]
//     x[t] <- x[t] + factor * y[t] / sqrt(mean(y[t]^2) + eps) * w        (without a weight: x[t] <- x[t] + factor * y[t])
//     rounded[t] = x[t] in the engine's storage type (optional)
// All float32 inside. A block owns a token; a row of up to 4,096 elements stays in registers between the sum of squares
// and the update, a longer one is read again.
#include "common.cuh"

namespace {
constexpr int PN_THREADS = 256;

struct PostNormArgs {
    float* x;                    // [N, width]
    const float* a;              // [N, width], or rows of width (pair_row)
    const float* b;              // [N, width] or null
    const int* pair_row;         // [N, top] or null
    const float* weight;         // [width] or null
    float a_scale, b_scale, factor, eps;
    int width, top;
};

template <int V> struct Piece { float v[V]; };
template <int V> __device__ __forceinline__ Piece<V> pn_load(const float* p) {
    Piece<V> r;
    if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ void pn_store(float* p, const Piece<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void pn_store(__nv_bfloat16* p, const Piece<V>& r) {
    if constexpr (V == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&lo);
        u.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

template <typename T, int V, int KEEP>
__global__ void __launch_bounds__(PN_THREADS)
post_norm_kernel(const PostNormArgs a, T* __restrict__ rounded) {
    __shared__ float scratch[PN_THREADS / 32];
    dd_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x;
    Piece<V> w[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (tid + j * PN_THREADS) * V;
        if (a.weight && c < a.width) w[j] = pn_load<V>(a.weight + c);
    }
    dd_grid_wait();
    const size_t row = (size_t)t * a.width;
    auto load = [&](int c) {
        Piece<V> y;
        if (a.pair_row) {
#pragma unroll
            for (int i = 0; i < V; ++i) y.v[i] = 0.f;
            // the rows of four choices are looked up first and then requested together
            for (int k0 = 0; k0 < a.top; k0 += 4) {
                int at[4];
                Piece<V> r[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) at[u] = k0 + u < a.top ? a.pair_row[(size_t)t * a.top + k0 + u] : -1;
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    if (at[u] >= 0) r[u] = pn_load<V>(a.a + (size_t)at[u] * a.width + c);
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    if (at[u] >= 0)
#pragma unroll
                        for (int i = 0; i < V; ++i) y.v[i] += r[u].v[i];
            }
            return y;
        }
        y = pn_load<V>(a.a + row + c);
#pragma unroll
        for (int i = 0; i < V; ++i) y.v[i] *= a.a_scale;
        if (a.b) {
            const Piece<V> z = pn_load<V>(a.b + row + c);
#pragma unroll
            for (int i = 0; i < V; ++i) y.v[i] = fmaf(a.b_scale, z.v[i], y.v[i]);
        }
        return y;
    };
    Piece<V> kept[KEEP], x[KEEP];
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (tid + j * PN_THREADS) * V;
        if (c < a.width) {
            kept[j] = load(c);
            x[j] = pn_load<V>(a.x + row + c);
#pragma unroll
            for (int i = 0; i < V; ++i) sum = fmaf(kept[j].v[i], kept[j].v[i], sum);
        }
    }
    float r = a.factor;
    if (a.weight) {
        for (int c = (tid + KEEP * PN_THREADS) * V; c < a.width; c += PN_THREADS * V) {
            const Piece<V> y = load(c);
#pragma unroll
            for (int i = 0; i < V; ++i) sum = fmaf(y.v[i], y.v[i], sum);
        }
        sum = dd_warp_sum(sum);
        if ((tid & 31) == 0) scratch[tid >> 5] = sum;
        __syncthreads();
        sum = 0.f;
#pragma unroll
        for (int i = 0; i < PN_THREADS / 32; ++i) sum += scratch[i];
        r = a.factor * (1.0f / sqrtf(sum / (float)a.width + a.eps));
    }
    auto finish = [&](int c, const Piece<V>& y, Piece<V> now, const Piece<V>& wt) {
#pragma unroll
        for (int i = 0; i < V; ++i) now.v[i] = fmaf(y.v[i] * r, a.weight ? wt.v[i] : 1.0f, now.v[i]);
        pn_store<V>(a.x + row + c, now);
        if (rounded) pn_store<V>(rounded + row + c, now);
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int c = (tid + j * PN_THREADS) * V;
        if (c < a.width) finish(c, kept[j], x[j], w[j]);
    }
    for (int c = (tid + KEEP * PN_THREADS) * V; c < a.width; c += PN_THREADS * V) {
        Piece<V> wt = {};
        if (a.weight) wt = pn_load<V>(a.weight + c);
        finish(c, load(c), pn_load<V>(a.x + row + c), wt);
    }
}

template <int V>
__global__ void __launch_bounds__(256)
round_rows_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ out, long long n) {
    dd_launch_dependents();
    dd_grid_wait();
    const long long c = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
    if (c < n) pn_store<V>(out + c, pn_load<V>(x + c));
}

template <typename T>
int launch_post_norm(const PostNormArgs& a, void* rounded, int n_tokens, cudaStream_t s) {
    const bool wide = a.width % 4 == 0 && !(((uintptr_t)a.x | (uintptr_t)a.a | (uintptr_t)a.b | (uintptr_t)a.weight | (uintptr_t)rounded) & 15);
    const dim3 grid(n_tokens), block(PN_THREADS);
    T* out = (T*)rounded;
    if (!wide) dd_launch(post_norm_kernel<T, 1, 4>, grid, block, 0, s, a, out);
    else if (a.width <= PN_THREADS * 4) dd_launch(post_norm_kernel<T, 4, 1>, grid, block, 0, s, a, out);
    else if (a.width <= PN_THREADS * 8) dd_launch(post_norm_kernel<T, 4, 2>, grid, block, 0, s, a, out);
    else dd_launch(post_norm_kernel<T, 4, 4>, grid, block, 0, s, a, out);
    return dd_check_launch("dd_post_norm");
}
}  // namespace

// x: float32 [n_tokens, width], updated. a: float32 [n_tokens, width] (b the same or null), or, with pair_row (int32 [n_tokens,
// top]), rows of width elements of which those at a token's non-negative entries are added up in order. weight: float32
// [width] or null (no norm). rounded: [n_tokens, width] in out_dtype or null.
DD_API int dd_post_norm(float* x, const float* a, const float* b, float a_scale, float b_scale, const int* pair_row, int top,
                        const float* weight, float eps, float factor, void* rounded, int n_tokens, int width, int out_dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (width <= 0 || !a || (pair_row && (b || top <= 0 || a_scale != 1.0f))) return dd_fail("dd_post_norm: bad operands (width %d)", width);
    PostNormArgs p;
    p.x = x; p.a = a; p.b = b; p.pair_row = pair_row; p.weight = weight; p.a_scale = a_scale; p.b_scale = b_scale;
    p.factor = factor; p.eps = eps; p.width = width; p.top = top;
    if (out_dtype == DD_F32) return launch_post_norm<float>(p, rounded, n_tokens, (cudaStream_t)stream);
    if (out_dtype == DD_BF16) return launch_post_norm<__nv_bfloat16>(p, rounded, n_tokens, (cudaStream_t)stream);
    return dd_fail("dd_post_norm: unknown output dtype %d", out_dtype);
}

// out = x in bfloat16; n elements.
DD_API int dd_round_rows(const float* x, void* out, long long n, void* stream) {
    if (n <= 0) return 0;
    const bool wide = n % 4 == 0 && !(((uintptr_t)x | (uintptr_t)out) & 15);
    const int grid = dd_ceil_div(n, wide ? 1024 : 256);
    if (wide) dd_launch(round_rows_kernel<4>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, x, (__nv_bfloat16*)out, n);
    else dd_launch(round_rows_kernel<1>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, x, (__nv_bfloat16*)out, n);
    return dd_check_launch("dd_round_rows");
}
