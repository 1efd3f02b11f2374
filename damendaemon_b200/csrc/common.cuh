// Shared helpers for the hand-written sm_100a kernels: element types, warp
// reductions, the C ABI's error reporting. No PyTorch headers: the library is
// plain CUDA behind extern "C" launchers, loaded with ctypes.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define DD_API extern "C" __attribute__((visibility("default")))

enum DdDtype { DD_F32 = 0, DD_BF16 = 1 };
enum DdAct { DD_ACT_NONE = 0, DD_ACT_GELU_NEW = 1, DD_ACT_GELU_ERF = 2, DD_ACT_RELU2 = 3, DD_ACT_TANH = 4 };

// Records a message for dd_last_error() and returns a non-zero code.
int dd_fail(const char* fmt, ...);
// Returns 0 if the last launch was accepted, else records the CUDA error.
int dd_check_launch(const char* what);

template <typename T> struct DdType;
template <> struct DdType<float> { static constexpr int id = DD_F32; };
template <> struct DdType<__nv_bfloat16> { static constexpr int id = DD_BF16; };

__device__ __forceinline__ float dd_to_f32(float v) { return v; }
__device__ __forceinline__ float dd_to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T dd_from_f32(float v);
template <> __device__ __forceinline__ float dd_from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 dd_from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float dd_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float dd_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// gelu_new(u) = 0.5 u (1 + tanh(sqrt(2/pi) (u + 0.044715 u^3))); gelu(u) = 0.5 u (1 + erf(u / sqrt 2));
// relu2(u) = max(u, 0)^2; tanh.
__device__ __forceinline__ float dd_activation(float u, int act) {
    if (act == DD_ACT_GELU_NEW) {
        const float c = 0.7978845608028654f;
        return 0.5f * u * (1.0f + tanhf(c * (u + 0.044715f * u * u * u)));
    }
    if (act == DD_ACT_GELU_ERF) return 0.5f * u * (1.0f + erff(u * 0.7071067811865476f));
    if (act == DD_ACT_RELU2) { const float r = fmaxf(u, 0.f); return r * r; }
    if (act == DD_ACT_TANH) return tanhf(u);
    return u;
}

// The gated unit's value from its gate and up products, in float32. CLAMPED: g = min(gate, limit),
// u = clamp(up, -limit, limit), g * sigmoid(alpha g) * (u + 1); SILU: gate * sigmoid(gate) * up; GELU_TANH:
// gelu_new(gate) * up. FAST: the exponential of the special-function unit (for results that are rounded to bfloat16).
enum DdGated { DD_GATED_CLAMPED = 0, DD_GATED_SILU = 1, DD_GATED_GELU_TANH = 2 };
template <bool FAST>
__device__ __forceinline__ float dd_gated_value(float gate, float up, int form, float limit, float alpha) {
    if (form == DD_GATED_SILU) return gate * (1.0f / (1.0f + (FAST ? __expf(-gate) : expf(-gate)))) * up;
    if (form == DD_GATED_GELU_TANH) return dd_activation(gate, DD_ACT_GELU_NEW) * up;
    const float g = fminf(gate, limit);
    const float u = fminf(fmaxf(up, -limit), limit);
    return g * (1.0f / (1.0f + (FAST ? __expf(-alpha * g) : expf(-alpha * g)))) * (u + 1.0f);
}

// A rotation that `tail` elements undergo while they are copied: n_pairs pairs (neighbours, or one of each half of the first
// 2 * n_pairs elements) turned by positions[token] * freqs[pair], float32 inside; n_pairs = 0: a plain copy.
struct DdTailTurn {
    const float* freqs;
    const int* positions;
    int n_pairs, interleaved;
};
// Copies the tails of `n` consecutive rows (the first is token t0) by a block's threads.
template <typename T>
__device__ __forceinline__ void dd_copy_tail(const T* in, int in_stride, T* out, int out_stride, int n, int tail, int t0,
                                             const DdTailTurn& turn, int threads) {
    if (turn.n_pairs > 0)
        for (int i = threadIdx.x; i < n * turn.n_pairs; i += threads) {
            const int tt = i / turn.n_pairs, p = i % turn.n_pairs;
            const int c = turn.interleaved ? 2 * p : p, to = turn.interleaved ? 1 : turn.n_pairs;
            float sn, cs;
            sincosf((float)turn.positions[t0 + tt] * turn.freqs[p], &sn, &cs);
            const float a = dd_to_f32(in[(size_t)tt * in_stride + c]), b = dd_to_f32(in[(size_t)tt * in_stride + c + to]);
            out[(size_t)tt * out_stride + c] = dd_from_f32<T>(a * cs - b * sn);
            out[(size_t)tt * out_stride + c + to] = dd_from_f32<T>(b * cs + a * sn);
        }
    const int rest = tail - 2 * turn.n_pairs;
    for (int i = threadIdx.x; i < n * rest; i += threads) {
        const int tt = i / rest, c = 2 * turn.n_pairs + i % rest;
        out[(size_t)tt * out_stride + c] = in[(size_t)tt * in_stride + c];
    }
}

static inline int dd_ceil_div(long long a, long long b) { return (int)((a + b - 1) / b); }

// Programmatic dependent launch. Every kernel of this library is launched so that it may start
// while the kernel before it on the stream is still running: it does whatever does not depend
// on earlier kernels (barrier set-up, TMEM allocation, prefetching weights), lets its own
// successor start early (dd_launch_dependents) and then waits for the kernel before it to have
// finished and flushed its writes (dd_grid_wait) before it reads or writes anything else in
// global memory. Without the launch attribute both instructions do nothing.
__device__ __forceinline__ void dd_grid_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void dd_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

extern int dd_pdl_enabled;      // errors.cu; switched by dd_set_pdl()

// A launch in plain stream order, whatever dd_pdl_enabled says: for a kernel of few long-running blocks, which must be
// dealt out over an empty GPU (started early, its blocks go wherever the kernel before has just freed room, several to
// an SM while others stay empty, and stay there).
template <typename... KArgs, typename... Args>
static inline cudaError_t dd_launch_in_order(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                             Args... args) {
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = block;
    config.dynamicSmemBytes = smem;
    config.stream = stream;
    config.numAttrs = 0;
    return cudaLaunchKernelEx(&config, kernel, static_cast<KArgs>(args)...);
}

template <typename... KArgs, typename... Args>
static inline cudaError_t dd_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                    Args... args) {
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = block;
    config.dynamicSmemBytes = smem;
    config.stream = stream;
    cudaLaunchAttribute attribute[1];
    attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[0].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attribute;
    config.numAttrs = dd_pdl_enabled ? 1 : 0;
    return cudaLaunchKernelEx(&config, kernel, static_cast<KArgs>(args)...);
}
