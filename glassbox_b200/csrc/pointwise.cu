// Small row-wise and element-wise kernels for layers that norm a branch before it joins the residual stream, for
// activations other than SwiGLU, and for a scaled head:
//   rmsnorm_add   x[r, :] += gain * y[r, :] / sqrt(mean(y[r, :]^2) + eps)   (float32 throughout); optionally y + bias in the
//                 place of y, and a copy of the new x[r, :] in the activation dtype
//   cast_rows     out[r, :] = x[rows[r], :] in the activation dtype
//   add_bias      y[r, :] += bias
//   clamped_glu   act[r, f] = g * sigmoid(slope * g) * (u + 1), g = min(gate + b, limit), u = clamp(up + b, -limit, limit)
//   relu2         out = max(in, 0)^2
//   gelu          out = gelu(in), the exact form
//   scale         t *= s
//   tanh_cap      t <- cap * tanh(t / cap)
//   gate_rows     y[r, :] *= sigmoid(gate[r, :])
//   gated_head_norm  out[r, h, :] = w * o[r, h, :] / sqrt(mean_v(o[r, h, :]^2) + eps) * sigmoid(gate[r, h, :])  (or * silu(gate))
//   gelu_glu      act[r, f] = gelu_tanh(gate[r, f]) * up[r, f]
//   scaled_sum    out (+)= a * x + b * y
//   post_norm     x[r, :] <- gain * t / rms(t), t = alpha * x[r, :] + y[r, :] (y stored, or a weighted sum, or two normed branches)
//   gate_group_norm  u = y * silu(z), each of equal parts of the row normed by its own root mean square, times a gain
#include "common.cuh"

// ----------------------------------------------------------------------------------------------
// A branch's output y (float32) is normalised and added into the residual x (float32). One block per row.
// ----------------------------------------------------------------------------------------------
template <int THREADS, typename T>
__global__ void __launch_bounds__(THREADS) rmsnorm_add_kernel(const float* __restrict__ y, long long ldy,
                                                              const float* __restrict__ gain, float* __restrict__ x,
                                                              long long ldx, int n, int d, float eps,
                                                              const float* __restrict__ bias, T* __restrict__ copy) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int r = blockIdx.x;
    if (r >= n) return;
    const float* src = y + (size_t)r * ldy;
    float* dst = x + (size_t)r * ldx;
    __shared__ float partial[THREADS / 32];
    __shared__ float total;
    constexpr int VMAX = 4;
    const bool quick = d % 4 == 0 && d <= THREADS * 4 * VMAX && ((uintptr_t)src & 15) == 0 && ((uintptr_t)dst & 15) == 0 &&
                       ((uintptr_t)gain & 15) == 0 && ((uintptr_t)bias & 15) == 0;
    T* cp = copy ? copy + (size_t)r * d : nullptr;
    float4 v[VMAX], o[VMAX];
    float ss = 0.f;
    if (quick) {
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * THREADS + threadIdx.x) * 4;
            v[i] = j < d ? *reinterpret_cast<const float4*>(src + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            o[i] = j < d ? *reinterpret_cast<const float4*>(dst + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (bias != nullptr && j < d) {
                const float4 b = *reinterpret_cast<const float4*>(bias + j);
                v[i].x += b.x; v[i].y += b.y; v[i].z += b.z; v[i].w += b.w;
            }
        }
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
            ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
        }
    } else {
        for (int j = threadIdx.x; j < d; j += THREADS) {
            const float t = src[j] + (bias ? bias[j] : 0.f);
            ss = fmaf(t, t, ss);
        }
    }
    ss = gb_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x == 0) {
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < THREADS / 32; ++w) t += partial[w];
        total = 1.0f / sqrtf(t / (float)d + eps);
    }
    __syncthreads();
    const float s = total;
    if (quick) {
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * THREADS + threadIdx.x) * 4;
            if (j < d) {
                const float4 g = *reinterpret_cast<const float4*>(gain + j);
                float4 w;
                w.x = o[i].x + g.x * (v[i].x * s);
                w.y = o[i].y + g.y * (v[i].y * s);
                w.z = o[i].z + g.z * (v[i].z * s);
                w.w = o[i].w + g.w * (v[i].w * s);
                *reinterpret_cast<float4*>(dst + j) = w;
                if (cp != nullptr) {
                    cp[j] = gb_from_float<T>(w.x); cp[j + 1] = gb_from_float<T>(w.y);
                    cp[j + 2] = gb_from_float<T>(w.z); cp[j + 3] = gb_from_float<T>(w.w);
                }
            }
        }
    } else {
        for (int j = threadIdx.x; j < d; j += THREADS) {
            const float w = dst[j] + gain[j] * ((src[j] + (bias ? bias[j] : 0.f)) * s);
            dst[j] = w;
            if (cp != nullptr) cp[j] = gb_from_float<T>(w);
        }
    }
}

// bias (optional, float32 [d]) is added to y first; copy (optional, [n, d] of dtype copy_dtype) receives the new x
GB_EXPORT int gb_rmsnorm_add(const float* y, long long ldy, const float* gain, float* x, long long ldx, int n, int d,
                             float eps, const float* bias, void* copy, int copy_dtype, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && d > 0, "gb_rmsnorm_add: bad sizes n=%d d=%d", n, d);
    GB_REQUIRE(copy == nullptr || copy_dtype == GB_F32 || copy_dtype == GB_BF16, "gb_rmsnorm_add: unsupported dtype %d", copy_dtype);
    if (n == 0) return 0;
    if (copy != nullptr && copy_dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, rmsnorm_add_kernel<128, __nv_bfloat16>, dim3(n), dim3(128), 0, stream, y, ldy, gain, x, ldx, n, d,
                  eps, bias, (__nv_bfloat16*)copy);
    else
        gb_launch(GB_PDL_ELEMENTWISE, rmsnorm_add_kernel<128, float>, dim3(n), dim3(128), 0, stream, y, ldy, gain, x, ldx, n, d, eps,
                  bias, (float*)copy);
    return gb_check_launch("gb_rmsnorm_add");
}

// ----------------------------------------------------------------------------------------------
// out[r, :] = x[rows ? rows[r] : r, :], float32 -> the activation dtype (a branch that reads the residual as it is).
// ----------------------------------------------------------------------------------------------
template <typename T>
__global__ void cast_rows_kernel(const float* __restrict__ x, long long ldx, const int* __restrict__ rows, T* __restrict__ out, int n,
                                 int d) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long total = (long long)n * d;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int r = (int)(idx / d), j = (int)(idx % d);
        const int src = rows ? rows[r] : r;
        out[idx] = gb_from_float<T>(src >= 0 ? x[(size_t)src * ldx + j] : 0.f);
    }
}

GB_EXPORT int gb_cast_rows(const float* x, long long ldx, const int* rows, void* out, int dtype, int n, int d, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && d > 0, "gb_cast_rows: bad sizes n=%d d=%d", n, d);
    if (n == 0) return 0;
    long long total = (long long)n * d;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, cast_rows_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, ldx, rows, (float*)out, n, d);
    else if (dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, cast_rows_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, x, ldx, rows,
                  (__nv_bfloat16*)out, n, d);
    else
        GB_REQUIRE(false, "gb_cast_rows: unsupported dtype %d", dtype);
    return gb_check_launch("gb_cast_rows");
}

// ----------------------------------------------------------------------------------------------
// y[r, :] += bias (float32): a product's bias where no later kernel takes it along.
// ----------------------------------------------------------------------------------------------
__global__ void add_bias_kernel(float* __restrict__ y, long long ldy, const float* __restrict__ bias, int n, int d) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long total = (long long)n * d;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int r = (int)(idx / d), j = (int)(idx % d);
        y[(size_t)r * ldy + j] += bias[j];
    }
}

GB_EXPORT int gb_add_bias(float* y, long long ldy, const float* bias, int n, int d, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && d > 0, "gb_add_bias: bad sizes n=%d d=%d", n, d);
    if (n == 0) return 0;
    long long total = (long long)n * d;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    gb_launch(GB_PDL_ELEMENTWISE, add_bias_kernel, dim3(blocks), dim3(256), 0, stream, y, ldy, bias, n, d);
    return gb_check_launch("gb_add_bias");
}

// ----------------------------------------------------------------------------------------------
// The clamped gated unit, from the sums of the stacked gate | up product (row r: ff gate sums, then ff up sums):
// g = min(gate + b_gate, limit), u = clamp(up + b_up, -limit, limit), act = g * sigmoid(slope * g) * (u + 1), in float32.
// ----------------------------------------------------------------------------------------------
template <typename TI, typename T>
__global__ void clamped_glu_kernel(const TI* __restrict__ gate_up, long long ld, const float* __restrict__ bias, float limit,
                                   float slope, T* __restrict__ act, int n, int ff) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long total = (long long)n * ff;
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int r = (int)(idx / ff), f = (int)(idx % ff);
        const TI* row = gate_up + (size_t)r * ld;
        act[idx] = gb_from_float<T>(gb_clamped_unit(gb_to_float(row[f]) + (bias ? bias[f] : 0.f),
                                                   gb_to_float(row[ff + f]) + (bias ? bias[ff + f] : 0.f), limit, slope));
    }
}

GB_EXPORT int gb_clamped_glu(const void* gate_up, int in_dtype, long long ld, const float* bias, float limit, float slope, void* act,
                             int dtype, int n, int ff, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && ff > 0 && limit > 0.f, "gb_clamped_glu: bad sizes n=%d ff=%d limit=%g", n, ff, (double)limit);
    if (n == 0) return 0;
    long long total = (long long)n * ff;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (in_dtype == GB_F32 && dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, clamped_glu_kernel<float, float>, dim3(blocks), dim3(256), 0, stream, (const float*)gate_up, ld,
                  bias, limit, slope, (float*)act, n, ff);
    else if (in_dtype == GB_F32 && dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, clamped_glu_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const float*)gate_up,
                  ld, bias, limit, slope, (__nv_bfloat16*)act, n, ff);
    else if (in_dtype == GB_BF16 && dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, clamped_glu_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream,
                  (const __nv_bfloat16*)gate_up, ld, bias, limit, slope, (__nv_bfloat16*)act, n, ff);
    else
        GB_REQUIRE(false, "gb_clamped_glu: unsupported dtypes %d -> %d", in_dtype, dtype);
    return gb_check_launch("gb_clamped_glu");
}

// ----------------------------------------------------------------------------------------------
// Squared ReLU.
// ----------------------------------------------------------------------------------------------
template <typename T>
__global__ void relu2_kernel(const T* __restrict__ in, T* __restrict__ out, long long total) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    for (; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const float v = fmaxf(gb_to_float(in[idx]), 0.f);
        out[idx] = gb_from_float<T>(v * v);
    }
}

GB_EXPORT int gb_relu2(const void* in, void* out, int dtype, long long total, cudaStream_t stream) {
    GB_REQUIRE(total >= 0, "gb_relu2: bad size");
    if (total == 0) return 0;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, relu2_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)in, (float*)out, total);
    else if (dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, relu2_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)in,
                  (__nv_bfloat16*)out, total);
    else
        GB_REQUIRE(false, "gb_relu2: unsupported dtype %d", dtype);
    return gb_check_launch("gb_relu2");
}

// ----------------------------------------------------------------------------------------------
// t *= s (float32): a head whose logits carry a constant factor.
// ----------------------------------------------------------------------------------------------
__global__ void scale_kernel(float* __restrict__ t, long long total, float s) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    for (; idx < total; idx += (long long)gridDim.x * blockDim.x) t[idx] *= s;
}

__global__ void tanh_cap_kernel(float* __restrict__ t, long long total, float cap, float inv_cap) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long stride = (long long)gridDim.x * blockDim.x;
    const long long quads = ((uintptr_t)t & 15) == 0 ? total / 4 : 0;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < quads; i += stride) {
        float4 v = reinterpret_cast<float4*>(t)[i];
        v.x = cap * tanhf(v.x * inv_cap); v.y = cap * tanhf(v.y * inv_cap);
        v.z = cap * tanhf(v.z * inv_cap); v.w = cap * tanhf(v.w * inv_cap);
        reinterpret_cast<float4*>(t)[i] = v;
    }
    for (long long i = 4 * quads + (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) t[i] = cap * tanhf(t[i] * inv_cap);
}

GB_EXPORT int gb_tanh_cap(float* t, long long total, float cap, cudaStream_t stream) {
    GB_REQUIRE(total >= 0 && cap > 0.f, "gb_tanh_cap: bad size or cap");
    if (total == 0) return 0;
    const long long blocks = (total / 4 + 255) / 256 + 1;
    gb_launch(GB_PDL_ELEMENTWISE, tanh_cap_kernel, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), 0, stream, t, total, cap, 1.0f / cap);
    return gb_check_launch("gb_tanh_cap");
}

template <typename T>
__global__ void gelu_kernel(const float* __restrict__ in, T* __restrict__ out, long long total) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) out[i] = gb_from_float<T>(gb_gelu(in[i]));
}

GB_EXPORT int gb_gelu(const float* in, void* out, int dtype, long long total, cudaStream_t stream) {
    GB_REQUIRE(total >= 0 && (dtype == GB_F32 || dtype == GB_BF16), "gb_gelu: bad size or dtype");
    if (total == 0) return 0;
    const long long blocks = (total + 255) / 256;
    const dim3 grid((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8));
    if (dtype == GB_F32) gb_launch(GB_PDL_ELEMENTWISE, gelu_kernel<float>, grid, dim3(256), 0, stream, in, (float*)out, total);
    else gb_launch(GB_PDL_ELEMENTWISE, gelu_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, in, (__nv_bfloat16*)out, total);
    return gb_check_launch("gb_gelu");
}

template <typename T, typename TG>
__global__ void gate_rows_kernel(T* __restrict__ y, const TG* __restrict__ gate, long long ld_gate, int n, int width) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long total = (long long)n * width, stride = (long long)gridDim.x * blockDim.x;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
        const long long r = i / width;
        y[i] = gb_from_float<T>(gb_to_float(y[i]) / (1.0f + expf(-gb_to_float(gate[r * ld_gate + (i - r * width)]))));
    }
}

GB_EXPORT int gb_gate_rows(void* y, int dtype, const void* gate, int gate_dtype, long long ld_gate, int n, int width, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && width > 0 && ld_gate >= width, "gb_gate_rows: bad sizes");
    GB_REQUIRE((dtype == GB_F32 || dtype == GB_BF16) && (gate_dtype == GB_F32 || gate_dtype == GB_BF16), "gb_gate_rows: unsupported dtype");
    if (n == 0) return 0;
    const long long blocks = ((long long)n * width + 255) / 256;
    const dim3 grid((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8));
#define GR_CASE(T, TG) gb_launch(GB_PDL_ELEMENTWISE, gate_rows_kernel<T, TG>, grid, dim3(256), 0, stream, (T*)y, (const TG*)gate, ld_gate, n, width)
    if (dtype == GB_F32 && gate_dtype == GB_F32) GR_CASE(float, float);
    else if (dtype == GB_F32) GR_CASE(float, __nv_bfloat16);
    else if (gate_dtype == GB_F32) GR_CASE(__nv_bfloat16, float);
    else GR_CASE(__nv_bfloat16, __nv_bfloat16);
#undef GR_CASE
    return gb_check_launch("gb_gate_rows");
}

GB_EXPORT int gb_scale(float* t, long long total, float s, cudaStream_t stream) {
    GB_REQUIRE(total >= 0, "gb_scale: bad size");
    if (total == 0) return 0;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    gb_launch(GB_PDL_ELEMENTWISE, scale_kernel, dim3(blocks), dim3(256), 0, stream, t, total, s);
    return gb_check_launch("gb_scale");
}

// ----------------------------------------------------------------------------------------------
// Per-head RMS norm of a mixer's read-out with an output gate: one warp per (row, head).
// o float32 [n, heads * v]; gate float32 (row stride ldg), logits of the gate; w float32 [v] shared by heads.
// ----------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                              long long ldg, const float* __restrict__ w, T* __restrict__ out,
                                                              int n, int heads, int v, float eps, int gate_silu) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long task = (long long)blockIdx.x * 4 + warp;
    if (task >= (long long)n * heads) return;
    const int row = (int)(task / heads), head = (int)(task % heads);
    const float* src = o + ((size_t)row * heads + head) * v;
    const float* g = gate + (size_t)row * ldg + (size_t)head * v;
    T* dst = out + ((size_t)row * heads + head) * v;
    float ss = 0.f;
    for (int j = lane; j < v; j += 32) ss = fmaf(src[j], src[j], ss);
    ss = gb_warp_sum(ss);
    const float s = 1.0f / sqrtf(ss / (float)v + eps);
    for (int j = lane; j < v; j += 32) {
        const float sig = 1.0f / (1.0f + expf(-g[j]));
        dst[j] = gb_from_float<T>(src[j] * s * w[j] * (gate_silu ? g[j] * sig : sig));
    }
}

// The same for long rows (a norm that spans all heads): one block per (row, head), the sum of squares meets in shared memory.
template <typename T>
__global__ void __launch_bounds__(256) gated_head_norm_wide_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                                   long long ldg, const float* __restrict__ w, T* __restrict__ out,
                                                                   int n, int heads, int v, float eps, int gate_silu) {
    __shared__ float partial[8];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int row = blockIdx.x / heads, head = blockIdx.x % heads;
    const float* src = o + ((size_t)row * heads + head) * v;
    const float* g = gate + (size_t)row * ldg + (size_t)head * v;
    T* dst = out + ((size_t)row * heads + head) * v;
    float ss = 0.f;
    for (int j = threadIdx.x; j < v; j += 256) ss = fmaf(src[j], src[j], ss);
    ss = gb_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += partial[i];
    const float s = 1.0f / sqrtf(ss / (float)v + eps);
    for (int j = threadIdx.x; j < v; j += 256) {
        const float sig = 1.0f / (1.0f + expf(-g[j]));
        dst[j] = gb_from_float<T>(src[j] * s * w[j] * (gate_silu ? g[j] * sig : sig));
    }
}

GB_EXPORT int gb_gated_head_norm(const float* o, const float* gate, long long ldg, const float* w, void* out, int out_dtype,
                                 int n, int heads, int v, float eps, int gate_silu, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && heads > 0 && v > 0, "gb_gated_head_norm: bad sizes");
    if (n == 0) return 0;
    if (v > 256) {
        if (out_dtype == GB_F32)
            gb_launch(GB_PDL_ELEMENTWISE, gated_head_norm_wide_kernel<float>, dim3(n * heads), dim3(256), 0, stream, o, gate, ldg, w,
                      (float*)out, n, heads, v, eps, gate_silu);
        else if (out_dtype == GB_BF16)
            gb_launch(GB_PDL_ELEMENTWISE, gated_head_norm_wide_kernel<__nv_bfloat16>, dim3(n * heads), dim3(256), 0, stream, o, gate, ldg, w,
                      (__nv_bfloat16*)out, n, heads, v, eps, gate_silu);
        else
            GB_REQUIRE(false, "gb_gated_head_norm: unsupported output dtype %d", out_dtype);
        return gb_check_launch("gb_gated_head_norm");
    }
    const int blocks = gb_ceil_div((long long)n * heads, 4);
    if (out_dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, gated_head_norm_kernel<float>, dim3(blocks), dim3(128), 0, stream, o, gate, ldg, w, (float*)out, n,
                  heads, v, eps, gate_silu);
    else if (out_dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, gated_head_norm_kernel<__nv_bfloat16>, dim3(blocks), dim3(128), 0, stream, o, gate, ldg, w,
                  (__nv_bfloat16*)out, n, heads, v, eps, gate_silu);
    else
        GB_REQUIRE(false, "gb_gated_head_norm: unsupported output dtype %d", out_dtype);
    return gb_check_launch("gb_gated_head_norm");
}

// ----------------------------------------------------------------------------------------------
// The gated unit whose gate passes the tanh form of GELU: act[r, f] = 0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))) * u with
// g = gate_up[r, f], u = gate_up[r, ff + f]; float32 arithmetic, any input and output dtype.
// ----------------------------------------------------------------------------------------------
template <typename TI, typename TO>
__global__ void __launch_bounds__(256) gelu_glu_kernel(const TI* __restrict__ gate_up, long long ld, TO* __restrict__ act, int n, int ff) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long long)n * ff) return;
    const int r = (int)(i / ff), f = (int)(i % ff);
    const float g = gb_to_float(gate_up[(size_t)r * ld + f]), u = gb_to_float(gate_up[(size_t)r * ld + ff + f]);
    act[i] = gb_from_float<TO>(gb_gelu_tanh(g) * u);
}

GB_EXPORT int gb_gelu_glu(const void* gate_up, int in_dtype, long long ld, void* act, int out_dtype, int n, int ff, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && ff > 0 && ld >= 2 * ff, "gb_gelu_glu: bad sizes");
    if (n == 0) return 0;
    const int blocks = gb_ceil_div((long long)n * ff, 256);
    if (in_dtype == GB_F32 && out_dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, gelu_glu_kernel<float, float>, dim3(blocks), dim3(256), 0, stream, (const float*)gate_up, ld, (float*)act, n, ff);
    else if (in_dtype == GB_F32 && out_dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, gelu_glu_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const float*)gate_up, ld,
                  (__nv_bfloat16*)act, n, ff);
    else if (in_dtype == GB_BF16 && out_dtype == GB_BF16)
        gb_launch(GB_PDL_ELEMENTWISE, gelu_glu_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream,
                  (const __nv_bfloat16*)gate_up, ld, (__nv_bfloat16*)act, n, ff);
    else
        GB_REQUIRE(false, "gb_gelu_glu: unsupported dtypes %d -> %d", in_dtype, out_dtype);
    return gb_check_launch("gb_gelu_glu");
}

// ----------------------------------------------------------------------------------------------
// out[r, :] (+)= a * x[r, :] + b * y[r, :]: two branches that share an input join with a weight each. Float32.
// ----------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) scaled_sum_kernel(const float* __restrict__ x, const float* __restrict__ y, float a, float b,
                                                         float* __restrict__ out, long long count, int accumulate) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= count) return;
    const float v = fmaf(a, x[i], b * y[i]);
    out[i] = accumulate ? out[i] + v : v;
}

GB_EXPORT int gb_scaled_sum(const float* x, const float* y, float a, float b, float* out, long long count, int accumulate,
                            cudaStream_t stream) {
    GB_REQUIRE(count >= 0, "gb_scaled_sum: bad size");
    if (count == 0) return 0;
    gb_launch(GB_PDL_ELEMENTWISE, scaled_sum_kernel, dim3(gb_ceil_div(count, 256)), dim3(256), 0, stream, x, y, a, b, out, count, accumulate);
    return gb_check_launch("gb_scaled_sum");
}

// ----------------------------------------------------------------------------------------------
// A residual that is normed after the sum: x[r, :] <- gain * t / sqrt(mean(t^2) + eps) with t = alpha * x[r, :] + y[r, :], and
// optionally a copy of the new row in the activation dtype. y comes as one of
//   rows     y[r, :] as it is stored
//   weighted sum_k weight[r, k] * pair[r, k, :] (+ gate[r] * shared[r, :]): a routed feed-forward's output in its parts
//   pair     a_scale * (ga * a[r, :] / rms(a[r, :])) + b_scale * (gb * b[r, :] / rms(b[r, :])): two branches side by side, each
//            normed over the row before they join
// so that a branch costs one launch beside its own. One block per row; float32 throughout; padding rows are skipped.
// ----------------------------------------------------------------------------------------------
struct PostNormArgs {
    float* x;
    long long ldx;
    const float* gain;
    float alpha, eps;
    const float* y;             // rows: y; pair: a
    const float* b;             // pair: b
    const float* ga;
    const float* gb;
    float a_scale, b_scale, pair_eps;
    const float* weighted;      // weighted: [n, top * d]
    const float* weight;
    const float* shared;
    const float* gate;
    int top;
    void* copy;
    const int* positions;
    int n, d;
};
enum { PN_ROWS = 0, PN_WEIGHTED = 1, PN_PAIR = 2 };
constexpr int PN_THREADS = 256, PN_VMAX = 4;

__device__ __forceinline__ float2 pn_block_sum2(float a, float b, float2* partial) {
    a = gb_warp_sum(a);
    b = gb_warp_sum(b);
    __syncthreads();                 // (an earlier use of `partial` is over)
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < PN_THREADS / 32; ++w) {
        t.x += partial[w].x;
        t.y += partial[w].y;
    }
    return t;
}

// four neighbours at once (the address is a multiple of four elements)
__device__ __forceinline__ void pn_store4(float* at, float4 v) { *reinterpret_cast<float4*>(at) = v; }
__device__ __forceinline__ void pn_store4(__nv_bfloat16* at, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(at) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}

template <int MODE, int VMAX, typename T>
__global__ void __launch_bounds__(PN_THREADS) post_norm_kernel(PostNormArgs p) {
    __shared__ float2 partial[PN_THREADS / 32];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int r = blockIdx.x;
    if (r >= p.n || (p.positions != nullptr && p.positions[r] < 0)) return;
    const int d = p.d, top = p.top;
    float* x = p.x + (size_t)r * p.ldx;
    T* cp = p.copy ? (T*)p.copy + (size_t)r * d : nullptr;
    const float* y = p.y ? p.y + (size_t)r * d : nullptr;
    const float* b = MODE == PN_PAIR ? p.b + (size_t)r * d : nullptr;
    const float* rows = MODE == PN_WEIGHTED ? p.weighted + (size_t)r * top * d : nullptr;
    const float* wt = MODE == PN_WEIGHTED ? p.weight + (size_t)r * top : nullptr;
    const float* sh = MODE == PN_WEIGHTED && p.shared ? p.shared + (size_t)r * d : nullptr;
    const float shg = MODE == PN_WEIGHTED && p.gate ? p.gate[r] : 1.0f;
    if constexpr (VMAX > 0) {            // rows of whole 16-byte pieces that fit the block's registers: one trip to memory
        float4 t[VMAX], v[VMAX], u[MODE == PN_PAIR ? VMAX : 1];
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * PN_THREADS + threadIdx.x) * 4;
            const bool in = j < d;
            t[i] = in ? *reinterpret_cast<const float4*>(x + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            if constexpr (MODE != PN_WEIGHTED) v[i] = in ? *reinterpret_cast<const float4*>(y + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            if constexpr (MODE == PN_PAIR) u[i] = in ? *reinterpret_cast<const float4*>(b + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if constexpr (MODE == PN_WEIGHTED) {
#pragma unroll
            for (int i = 0; i < VMAX; ++i) {
                const int j = (i * PN_THREADS + threadIdx.x) * 4;
                v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (j < d) {
#pragma unroll 4
                    for (int k = 0; k < top; ++k) {
                        const float w = wt[k];
                        const float4 q = *reinterpret_cast<const float4*>(rows + (size_t)k * d + j);
                        v[i].x = fmaf(w, q.x, v[i].x); v[i].y = fmaf(w, q.y, v[i].y);
                        v[i].z = fmaf(w, q.z, v[i].z); v[i].w = fmaf(w, q.w, v[i].w);
                    }
                    if (sh) {
                        const float4 q = *reinterpret_cast<const float4*>(sh + j);
                        v[i].x = fmaf(shg, q.x, v[i].x); v[i].y = fmaf(shg, q.y, v[i].y);
                        v[i].z = fmaf(shg, q.z, v[i].z); v[i].w = fmaf(shg, q.w, v[i].w);
                    }
                }
            }
        }
        if constexpr (MODE == PN_PAIR) {
            float sa = 0.f, sb = 0.f;
#pragma unroll
            for (int i = 0; i < VMAX; ++i) {
                sa = fmaf(v[i].x, v[i].x, sa); sa = fmaf(v[i].y, v[i].y, sa); sa = fmaf(v[i].z, v[i].z, sa); sa = fmaf(v[i].w, v[i].w, sa);
                sb = fmaf(u[i].x, u[i].x, sb); sb = fmaf(u[i].y, u[i].y, sb); sb = fmaf(u[i].z, u[i].z, sb); sb = fmaf(u[i].w, u[i].w, sb);
            }
            const float2 s = pn_block_sum2(sa, sb, partial);
            const float fa = p.a_scale / sqrtf(s.x / (float)d + p.pair_eps), fb = p.b_scale / sqrtf(s.y / (float)d + p.pair_eps);
#pragma unroll
            for (int i = 0; i < VMAX; ++i) {
                const int j = (i * PN_THREADS + threadIdx.x) * 4;
                if (j < d) {
                    const float4 g = *reinterpret_cast<const float4*>(p.ga + j), h = *reinterpret_cast<const float4*>(p.gb + j);
                    v[i].x = fmaf(g.x * fa, v[i].x, h.x * fb * u[i].x); v[i].y = fmaf(g.y * fa, v[i].y, h.y * fb * u[i].y);
                    v[i].z = fmaf(g.z * fa, v[i].z, h.z * fb * u[i].z); v[i].w = fmaf(g.w * fa, v[i].w, h.w * fb * u[i].w);
                }
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            t[i].x = fmaf(p.alpha, t[i].x, v[i].x); t[i].y = fmaf(p.alpha, t[i].y, v[i].y);
            t[i].z = fmaf(p.alpha, t[i].z, v[i].z); t[i].w = fmaf(p.alpha, t[i].w, v[i].w);
            ss = fmaf(t[i].x, t[i].x, ss); ss = fmaf(t[i].y, t[i].y, ss); ss = fmaf(t[i].z, t[i].z, ss); ss = fmaf(t[i].w, t[i].w, ss);
        }
        const float s = 1.0f / sqrtf(pn_block_sum2(ss, 0.f, partial).x / (float)d + p.eps);
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * PN_THREADS + threadIdx.x) * 4;
            if (j < d) {
                const float4 g = *reinterpret_cast<const float4*>(p.gain + j);
                const float4 w = make_float4(g.x * (t[i].x * s), g.y * (t[i].y * s), g.z * (t[i].z * s), g.w * (t[i].w * s));
                *reinterpret_cast<float4*>(x + j) = w;
                if (cp != nullptr) pn_store4(cp + j, w);
            }
        }
    } else {                             // any other row: a value is formed again in every pass
        float fa = 0.f, fb = 0.f;
        if constexpr (MODE == PN_PAIR) {
            float sa = 0.f, sb = 0.f;
            for (int j = threadIdx.x; j < d; j += PN_THREADS) {
                sa = fmaf(y[j], y[j], sa);
                sb = fmaf(b[j], b[j], sb);
            }
            const float2 s = pn_block_sum2(sa, sb, partial);
            fa = p.a_scale / sqrtf(s.x / (float)d + p.pair_eps);
            fb = p.b_scale / sqrtf(s.y / (float)d + p.pair_eps);
        }
        auto value = [&](int j) {
            float v;
            if constexpr (MODE == PN_ROWS) v = y[j];
            if constexpr (MODE == PN_PAIR) v = fmaf(p.ga[j] * fa, y[j], p.gb[j] * fb * b[j]);
            if constexpr (MODE == PN_WEIGHTED) {
                v = 0.f;
                for (int k = 0; k < top; ++k) v = fmaf(wt[k], rows[(size_t)k * d + j], v);
                if (sh) v = fmaf(shg, sh[j], v);
            }
            return fmaf(p.alpha, x[j], v);
        };
        float ss = 0.f;
        for (int j = threadIdx.x; j < d; j += PN_THREADS) {
            const float t = value(j);
            ss = fmaf(t, t, ss);
        }
        const float s = 1.0f / sqrtf(pn_block_sum2(ss, 0.f, partial).x / (float)d + p.eps);
        for (int j = threadIdx.x; j < d; j += PN_THREADS) {
            const float w = p.gain[j] * (value(j) * s);
            x[j] = w;
            if (cp != nullptr) cp[j] = gb_from_float<T>(w);
        }
    }
}

template <int MODE, typename T>
static void post_norm_launch(const PostNormArgs& p, bool vec, cudaStream_t stream) {
    const int pieces = gb_ceil_div(p.d, PN_THREADS * 4);
    if (!vec || pieces > PN_VMAX) gb_launch(GB_PDL_ELEMENTWISE, post_norm_kernel<MODE, 0, T>, dim3(p.n), dim3(PN_THREADS), 0, stream, p);
    else if (pieces == 1) gb_launch(GB_PDL_ELEMENTWISE, post_norm_kernel<MODE, 1, T>, dim3(p.n), dim3(PN_THREADS), 0, stream, p);
    else if (pieces == 2) gb_launch(GB_PDL_ELEMENTWISE, post_norm_kernel<MODE, 2, T>, dim3(p.n), dim3(PN_THREADS), 0, stream, p);
    else gb_launch(GB_PDL_ELEMENTWISE, post_norm_kernel<MODE, 4, T>, dim3(p.n), dim3(PN_THREADS), 0, stream, p);
}

// mode 0: y [n, d]; 1: weighted [n, top * d], weight [n, top], shared [n, d] or nullptr, gate [n] or nullptr; 2: y and b [n, d] with
// gains ga, gb [d]. All rows of y, b, weighted and shared are contiguous. copy: [n, d] of copy_dtype or nullptr.
GB_EXPORT int gb_post_norm(float* x, long long ldx, const float* gain, float alpha, float eps, int mode, const float* y, const float* b,
                           const float* ga, const float* gb, float a_scale, float b_scale, float pair_eps, const float* weighted,
                           const float* weight, int top, const float* shared, const float* gate, void* copy, int copy_dtype,
                           const int* positions, int n, int d, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && d > 0 && ldx >= d, "gb_post_norm: bad sizes n=%d d=%d", n, d);
    GB_REQUIRE(mode == PN_ROWS ? y != nullptr : mode == PN_WEIGHTED ? (weighted != nullptr && weight != nullptr && top > 0)
                                              : (mode == PN_PAIR && y != nullptr && b != nullptr && ga != nullptr && gb != nullptr),
               "gb_post_norm: mode %d lacks its operands", mode);
    GB_REQUIRE(copy == nullptr || copy_dtype == GB_F32 || copy_dtype == GB_BF16, "gb_post_norm: unsupported dtype %d", copy_dtype);
    if (n == 0) return 0;
    PostNormArgs p = {x, ldx, gain, alpha, eps, y, b, ga, gb, a_scale, b_scale, pair_eps, weighted, weight, shared, gate, top, copy,
                      positions, n, d};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)gain | (uintptr_t)y | (uintptr_t)b | (uintptr_t)ga | (uintptr_t)gb | (uintptr_t)weighted |
                          (uintptr_t)shared | (uintptr_t)copy;
    const bool vec = d % 4 == 0 && ldx % 4 == 0 && (all & 15) == 0;
    const bool half = copy != nullptr && copy_dtype == GB_BF16;
#define PN_GO(M)                                                                \
    if (mode == M) {                                                            \
        if (half) post_norm_launch<M, __nv_bfloat16>(p, vec, stream);           \
        else post_norm_launch<M, float>(p, vec, stream);                        \
    }
    PN_GO(PN_ROWS) PN_GO(PN_WEIGHTED) PN_GO(PN_PAIR)
#undef PN_GO
    return gb_check_launch("gb_post_norm");
}

// ----------------------------------------------------------------------------------------------
// A gate in front of a norm over equal parts of a row: u = y * silu(z), out = w * u / sqrt(mean over the part of u^2 + eps).
// y float32 [n, groups * size], z float32 logits (row stride ldz), w float32 [groups * size]. One block per (row, part).
// ----------------------------------------------------------------------------------------------
template <int THREADS, int VMAX, typename T>
__global__ void __launch_bounds__(THREADS) gate_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ldz,
                                                                  const float* __restrict__ w, T* __restrict__ out,
                                                                  const int* __restrict__ positions, int groups, int size, float eps) {
    __shared__ float partial[THREADS / 32];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int row = blockIdx.x / groups, g = blockIdx.x % groups;
    if (positions != nullptr && positions[row] < 0) return;
    const size_t at = (size_t)blockIdx.x * size;
    const float* src = y + at;
    const float* gz = z + (size_t)row * ldz + (size_t)g * size;
    const float* gw = w + (size_t)g * size;
    T* dst = out + at;
    // VMAX pieces of four numbers per thread in registers (rows of whole 16-byte pieces); VMAX 0: any row, in two passes
    float4 u[VMAX > 0 ? VMAX : 1];
    float ss = 0.f;
    auto gated = [](float a, float b) {
        if constexpr (sizeof(T) == 4) return a * (b / (1.0f + expf(-b)));
        else return __fdividef(a * b, 1.0f + __expf(-b));       // (the result is rounded to 16 bits in the end)
    };
    if constexpr (VMAX > 0) {
        float4 q[VMAX];
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * THREADS + threadIdx.x) * 4;
            u[i] = j < size ? *reinterpret_cast<const float4*>(src + j) : make_float4(0.f, 0.f, 0.f, 0.f);
            q[i] = j < size ? *reinterpret_cast<const float4*>(gz + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            u[i] = make_float4(gated(u[i].x, q[i].x), gated(u[i].y, q[i].y), gated(u[i].z, q[i].z), gated(u[i].w, q[i].w));
            ss = fmaf(u[i].x, u[i].x, ss); ss = fmaf(u[i].y, u[i].y, ss); ss = fmaf(u[i].z, u[i].z, ss); ss = fmaf(u[i].w, u[i].w, ss);
        }
    } else {
        for (int j = threadIdx.x; j < size; j += THREADS) {
            const float t = gated(src[j], gz[j]);
            ss = fmaf(t, t, ss);
        }
    }
    ss = gb_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; ++i) ss += partial[i];
    const float s = 1.0f / sqrtf(ss / (float)size + eps);
    if constexpr (VMAX > 0) {
#pragma unroll
        for (int i = 0; i < VMAX; ++i) {
            const int j = (i * THREADS + threadIdx.x) * 4;
            if (j < size) {
                const float4 g4 = *reinterpret_cast<const float4*>(gw + j);
                pn_store4(dst + j, make_float4(g4.x * (u[i].x * s), g4.y * (u[i].y * s), g4.z * (u[i].z * s), g4.w * (u[i].w * s)));
            }
        }
    } else {
        for (int j = threadIdx.x; j < size; j += THREADS) dst[j] = gb_from_float<T>(gw[j] * (gated(src[j], gz[j]) * s));
    }
}

GB_EXPORT int gb_gate_group_norm(const float* y, const float* z, long long ldz, const float* w, void* out, int out_dtype,
                                 const int* positions, int n, int groups, int size, float eps, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && groups > 0 && size > 0 && ldz >= (long long)groups * size, "gb_gate_group_norm: bad sizes");
    GB_REQUIRE(out_dtype == GB_F32 || out_dtype == GB_BF16, "gb_gate_group_norm: unsupported output dtype %d", out_dtype);
    if (n == 0) return 0;
    const bool vec = size % 4 == 0 && ldz % 4 == 0 && (((uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
#define GGN_GO(TH, VM)                                                                                                               \
    {                                                                                                                                \
        if (out_dtype == GB_F32)                                                                                                     \
            gb_launch(GB_PDL_ELEMENTWISE, gate_group_norm_kernel<TH, VM, float>, dim3(n * groups), dim3(TH), 0, stream, y, z, ldz, w, \
                      (float*)out, positions, groups, size, eps);                                                                    \
        else                                                                                                                         \
            gb_launch(GB_PDL_ELEMENTWISE, gate_group_norm_kernel<TH, VM, __nv_bfloat16>, dim3(n * groups), dim3(TH), 0, stream, y, z, \
                      ldz, w, (__nv_bfloat16*)out, positions, groups, size, eps);                                                    \
    }
    if (!vec || size > 256 * 4 * 4) GGN_GO(256, 0)
    else if (size <= 64 * 4) GGN_GO(64, 1)
    else if (size <= 128 * 4) GGN_GO(128, 1)
    else if (size <= 256 * 4) GGN_GO(256, 1)
    else if (size <= 256 * 8) GGN_GO(256, 2)
    else GGN_GO(256, 4)
#undef GGN_GO
    return gb_check_launch("gb_gate_group_norm");
}
