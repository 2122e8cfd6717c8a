// Shared device helpers for the sm_100a kernel library.
//
// Every kernel is launched through an extern "C" function that takes raw device
// pointers and a stream, returns 0 or a negative MX_ERR_* / positive cudaError_t
// code, and never allocates. Activations are `float` (the 32-bit path) or
// `__nv_bfloat16` (serving); statistics, softmax, rotation angles and the
// residual stream are float in both.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define MX_OK 0
#define MX_ERR_UNSUPPORTED (-1)   // a size this kernel refuses (see mx_last_error_message)
#define MX_ERR_ARGUMENT (-2)

// Bits a kernel may set in the step's device status word; the host reads it after a step.
#define MX_STATUS_BAD_TOKEN_ID 1
#define MX_STATUS_BAD_SLOT 2
#define MX_STATUS_BAD_PAGE 4
#define MX_STATUS_WAIT_TIMEOUT 8

#define MX_DTYPE_F32 0
#define MX_DTYPE_BF16 1

extern "C" const char* mx_last_error_message();
void mx_set_error(const char* fmt, ...);

#define MX_REFUSE(...)              \
    do {                            \
        mx_set_error(__VA_ARGS__);  \
        return MX_ERR_UNSUPPORTED;  \
    } while (0)

static inline int mx_launch_status() {
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) {
        mx_set_error("CUDA launch failed: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return MX_OK;
}

// ---- programmatic dependent launch: a kernel launched with mx_launch_chained may start while the
// kernel before it in the stream is still running. It must call pdl_wait() before it reads anything
// an earlier kernel wrote and before it writes global memory at all; what it does before that
// (reading weights, setting up shared memory) overlaps the predecessor's tail. pdl_trigger() lets
// the NEXT kernel in the stream begin its own preamble.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;\n" ::); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
// A pointer to what the kernel before wrote, as it may be used after pdl_wait(): the compiler is told that it
// no longer knows the pointer, so no load through it can be moved above the wait. Without this a load through
// a `const __restrict__` parameter is fair game for the scheduler (the qualifiers promise that nothing writes
// the data while the kernel runs, which is not true of the time before the wait): LayerNorm read rows that
// the product before it had not finished when other loads were placed ahead of its wait.
template <typename T>
__device__ __forceinline__ T* after_wait(T* p) {
    asm volatile("" : "+l"(p)::"memory");
    return p;
}
__device__ __forceinline__ void prefetch_l2(const void* p) {
    asm volatile("prefetch.global.L2 [%0];\n" ::"l"(p));
}

bool mx_chained_launch_enabled();

template <typename... KArgs, typename... Args>
static inline cudaError_t mx_launch_chained(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                            cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = block;
    config.dynamicSmemBytes = smem;
    config.stream = stream;
    cudaLaunchAttribute attribute[1];
    attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[0].val.programmaticStreamSerializationAllowed = mx_chained_launch_enabled() ? 1 : 0;
    config.attrs = attribute;
    config.numAttrs = 1;
    return cudaLaunchKernelEx(&config, kernel, KArgs(args)...);
}

// The first key position that a query at `pos` may see, by the attention kernels' one mask parameter:
// window > 0: the last `window` positions (pos - window + 1, not below 0); window < 0: the start of the query's
// own block of -window positions, blocks counted from position 0 of the sequence (keys of earlier blocks are
// out of sight however near); 0: every earlier position. It never decreases with `pos`.
__device__ __forceinline__ int first_visible_key(int pos, int window) {
    if (window > 0) return max(0, pos - window + 1);
    if (window < 0) return pos >= 0 ? pos - pos % (-window) : 0;
    return 0;
}

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. `scratch` holds 32
// floats. The order of additions is fixed by the thread layout alone.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float total = 0.f;
    for (int w = 0; w < nwarps; ++w) total += scratch[w];
    return total;
}

// tanh from one ex2 and one reciprocal: 1 - 2 / (1 + e^(2x)), absolute error of a few 1e-7; for scores that are
// capped in float inside the tensor-core attention kernels (tanh.approx is good to 2^-11 only).
__device__ __forceinline__ float tanh_by_exp2(float x) {
    x = fminf(fmaxf(x, -15.f), 15.f);
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e) : "f"(x * 2.885390081777927f));
    return 1.f - __fdividef(2.f, 1.f + e);
}

__device__ __forceinline__ float fast_log2(float x) {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

// tanh of a small argument on the FMA pipe: the odd Taylor polynomial up to x^11, whose first dropped term is
// below 2e-8 of x for |x| <= TANH_SMALL. Scores under a cap are mostly that small (|score| <= 0.35 cap), and the
// special-function units that tanh_by_exp2 needs are what bounds a softmax.
#define TANH_SMALL 0.35f
__device__ __forceinline__ float tanh_small(float x) {
    const float x2 = x * x;
    float p = -1382.f / 155925.f;
    p = fmaf(p, x2, 62.f / 2835.f);
    p = fmaf(p, x2, -17.f / 315.f);
    p = fmaf(p, x2, 2.f / 15.f);
    p = fmaf(p, x2, -1.f / 3.f);
    return fmaf(x * x2, p, x);
}

// tanh-approximated GELU: 0.5 u (1 + tanh(sqrt(2/pi) (u + 0.044715 u^3))).
__device__ __forceinline__ float gelu_tanh(float u) {
    const float k0 = 0.7978845608028654f, k1 = 0.044715f;
    return 0.5f * u * (1.f + tanhf(k0 * (u + k1 * u * u * u)));
}
// Epilogue modes of every matrix product, with v = acc + bias: 0 out(T) = v; 1 out(T) = gelu_tanh(v);
// 2 out(f32) = residual + v; 3 out(f32) = v; 4 out(T) = max(v, 0)^2.
#define MX_MODE_NONE 0
#define MX_MODE_GELU 1
#define MX_MODE_RESIDUAL 2
#define MX_MODE_F32 3
#define MX_MODE_RELU2 4
#define MX_MODE_LAST 4
__host__ __device__ __forceinline__ bool mx_mode_is_float(int mode) {
    return mode == MX_MODE_RESIDUAL || mode == MX_MODE_F32;
}

// The same with the hardware tanh (relative error about 2^-11): for results that are rounded to
// bfloat16 (2^-9) right after; the 32-bit path keeps tanhf.
__device__ __forceinline__ float gelu_tanh_fast(float u) {
    const float k0 = 0.7978845608028654f, k1 = 0.044715f;
    float t;
    asm("tanh.approx.f32 %0, %1;\n" : "=f"(t) : "f"(k0 * (u + k1 * u * u * u)));
    return 0.5f * u * (1.f + t);
}

// The activation that an epilogue mode puts on a value (modes without one return it): exact, and with the hardware
// tanh for results that are rounded to bfloat16.
__device__ __forceinline__ float relu_squared(float v) {
    v = fmaxf(v, 0.f);
    return v * v;
}
__device__ __forceinline__ float mode_activation(float v, int mode) {
    return mode == MX_MODE_GELU ? gelu_tanh(v) : (mode == MX_MODE_RELU2 ? relu_squared(v) : v);
}
__device__ __forceinline__ float mode_activation_fast(float v, int mode) {
    return mode == MX_MODE_GELU ? gelu_tanh_fast(v) : (mode == MX_MODE_RELU2 ? relu_squared(v) : v);
}

// silu of a value that is rounded to T (or meets operands that were): exact for float, from the hardware's exponential
// and reciprocal (a few units in the last float place) for bfloat16. The argument stays where the quotient has digits:
// beyond -80 the result is below any bfloat16 step of what it is added to.
template <typename T> __device__ __forceinline__ float silu_of(float z);
template <> __device__ __forceinline__ float silu_of<float>(float z) { return z / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float silu_of<__nv_bfloat16>(float z) {
    return __fdividef(z, 1.f + __expf(fminf(-z, 80.f)));
}
