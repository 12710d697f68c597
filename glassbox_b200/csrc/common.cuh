// Shared declarations for the kernel library: element types, error reporting, small helpers.
//
// Every exported function is `extern "C"`, takes raw device pointers plus a CUDA stream, and
// returns 0 on success. On failure it returns a non-zero code and leaves a message that
// `gb_last_error()` returns; nothing is printed and nothing traps. Kernels never assert: a bad
// index (token id, cache slot) is recorded in a caller-supplied status word and the access is
// skipped, so a faulty batch cannot fault the GPU.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define GB_EXPORT extern "C" __attribute__((visibility("default")))

enum GbDtype : int { GB_F32 = 0, GB_BF16 = 1 };

// Bits of the device status word.
enum GbStatusBits : int {
    GB_STATUS_BAD_TOKEN = 1,      // a token id outside the vocabulary
    GB_STATUS_BAD_SLOT = 2,       // a cache slot or page id outside the pool
    GB_STATUS_BAD_POSITION = 4,   // a position outside the rotary table, or beyond what a block table covers
    GB_STATUS_WAIT_TIMEOUT = 8,   // a bounded wait inside a kernel gave up
};

void gb_set_error(const char* fmt, ...);
int gb_check_launch(const char* what);

#define GB_REQUIRE(cond, ...)                 \
    do {                                      \
        if (!(cond)) {                        \
            gb_set_error(__VA_ARGS__);        \
            return 1;                         \
        }                                     \
    } while (0)

__device__ __forceinline__ float gb_to_float(float v) { return v; }
__device__ __forceinline__ float gb_to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T gb_from_float(float v);
template <> __device__ __forceinline__ float gb_from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 gb_from_float<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

// The clamped gated unit: g * sigmoid(slope * g) * (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit).
__device__ __forceinline__ float gb_clamped_unit(float gate, float up, float limit, float slope) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-slope * g)) * (u + 1.0f);
}

// The tanh form of GELU: 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).
__device__ __forceinline__ float gb_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// The same through the identity 0.5 (1 + tanh(y)) = 1 / (1 + exp(-2 y)) with the hardware's exponential and division (a
// relative error near 1e-6): for epilogues that round the result to bfloat16.
__device__ __forceinline__ float gb_gelu_tanh_fast(float z) {
    return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

// GELU itself: z times the cumulative normal distribution, z / 2 (1 + erf(z / sqrt 2)).
__device__ __forceinline__ float gb_gelu(float z) { return 0.5f * z * (1.0f + erff(z * 0.7071067811865476f)); }

// The same with erf from the rational approximation 7.1.26 of Abramowitz and Stegun's handbook (an error of 1.5e-7) and the
// hardware's exponential and division: for epilogues that round the result to bfloat16.
__device__ __forceinline__ float gb_gelu_fast(float z) {
    const float x = fabsf(z) * 0.7071067811865476f;
    const float t = __fdividef(1.0f, fmaf(0.3275911f, x, 1.0f));
    float p = fmaf(1.061405429f, t, -1.453152027f);
    p = fmaf(p, t, 1.421413741f);
    p = fmaf(p, t, -0.284496736f);
    p = fmaf(p, t, 0.254829592f);
    const float tail = p * t * __expf(-x * x);           // 1 - erf(x), x >= 0
    return 0.5f * z * (z < 0.f ? tail : 2.0f - tail);
}

// cap * tanh(s / cap) through tanh(y) = 1 - 2 / (1 + exp(2 y)) with the hardware's exponential and division: an absolute
// error of a few 1e-7 * cap, for scores on their way into an exponential. inv2 = 2 / cap.
__device__ __forceinline__ float gb_cap_fast(float s, float cap, float inv2) {
    return fmaf(-2.0f * cap, __fdividef(1.0f, 1.0f + __expf(s * inv2)), cap);
}

// The same for four scores in place, which share one division: by the product of their denominators, each kept at or below
// 1 + e^20 (where the tanh is 1 to the last bit).
__device__ __forceinline__ void gb_cap_fast4(float (&s)[4], float cap, float inv2) {
    float e[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) e[i] = 1.0f + __expf(fminf(s[i] * inv2, 20.0f));
    const float a = e[0] * e[1], b = e[2] * e[3], r = __fdividef(1.0f, a * b), ra = r * b, rb = r * a;
    const float down = -2.0f * cap;
    s[0] = fmaf(down, e[1] * ra, cap);
    s[1] = fmaf(down, e[0] * ra, cap);
    s[2] = fmaf(down, e[3] * rb, cap);
    s[3] = fmaf(down, e[2] * rb, cap);
}

// The first key that a query at position `pos` sees. mask > 0: a sliding window of that many keys; mask < 0: chunks of -mask
// positions counted from position 0, a query sees the keys of its own chunk; 0: every key.
__device__ __forceinline__ int gb_first_key(int pos, int mask) {
    if (mask < 0) return pos - pos % -mask;
    return (mask > 0 && pos + 1 > mask) ? pos + 1 - mask : 0;
}

// ln(1 + e^z), accurate for any z (also as a factor: no cancellation where e^z is small).
__device__ __forceinline__ float gb_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// One gated unit, told apart by its two numbers: a negative slope selects gelu_tanh(gate) * up, a slope of zero
// silu(gate) * up (neither clamps anything), a positive one the clamped unit.
__device__ __forceinline__ float gb_gated_unit(float gate, float up, float limit, float slope) {
    if (slope > 0.f) return gb_clamped_unit(gate, up, limit, slope);
    return slope < 0.f ? gb_gelu_tanh(gate) * up : gate / (1.0f + expf(-gate)) * up;
}

__device__ __forceinline__ float gb_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float gb_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

static inline int gb_ceil_div(long long a, long long b) { return (int)((a + b - 1) / b); }

// Programmatic dependent launch. A kernel launched through gb_launch (while the switch is on) may start
// while its predecessor in the stream is still running: it does its set-up, lets its own successor start
// (gb_pdl_launch_dependents) and then waits (gb_pdl_wait) until the predecessor has completed and its
// writes are visible; nothing before the wait may read what earlier kernels wrote, or write anything.
// Launched any other way, both instructions do nothing.
int gb_pdl_enabled();

__device__ __forceinline__ void gb_pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void gb_pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

// How a kernel body that can run in several settings meets the work before it. A body calls start() first and
// wait() at the point from which it reads what earlier work wrote; before wait() it may only read what no kernel of
// the step writes (weights, step metadata). A bounded wait may give up: the body then returns at once, having written nothing. Stand-alone kernels use GbPdlSync (programmatic dependent launch); a
// persistent kernel passes an object whose wait() is its barrier's wait.
struct GbPdlSync {
    __device__ __forceinline__ void start() { gb_pdl_launch_dependents(); }
    __device__ __forceinline__ void wait() { gb_pdl_wait(); }
    __device__ __forceinline__ bool gave_up() const { return false; }   // after wait(): true = do nothing more
    // the threads that share one virtual block: here the whole thread block
    __device__ __forceinline__ int thread() const { return (int)threadIdx.x; }
    __device__ __forceinline__ void group_barrier() { __syncthreads(); }
};

enum { GB_PDL_ELEMENTWISE = 1, GB_PDL_GEMM = 2, GB_PDL_ATTENTION = 4 };   // bits of the switch

template <typename... KArgs, typename... Args>
static inline cudaError_t gb_launch(int family, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                    cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = (gb_pdl_enabled() & family) ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
