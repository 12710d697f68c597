// What lies between a mixer's stacked projection (float32 sums) and its attention when the norms span whole projections:
//
//   projection_norm_rope_write  q | k | v of grouped-query attention: RMS norm over ALL query channels at once (a gain per
//                               channel), the same over all key channels, rotation of the first `rot` channels of every query
//                               and key head (channel i with channel i + rot/2), q into the query buffer, k and v into the
//                               paged cache at the row's slot
//   latent_inputs               query latent | latent | shared key part of latent attention: RMS norm of the query latent into
//                               an activation buffer, RMS norm of the latent and rotation of the key part into the cache row
//
// Rotation: the angle is float32(position) * inv_freq[i]; sine and cosine are multiplied by `magnitude`. Everything is float32
// until it is stored.
#include "common.cuh"

__device__ __forceinline__ void pn_store2(float* at, float a, float c) { *reinterpret_cast<float2*>(at) = make_float2(a, c); }
__device__ __forceinline__ void pn_store2(__nv_bfloat16* at, float a, float c) {
    *reinterpret_cast<__nv_bfloat162*>(at) = __floats2bfloat162_rn(a, c);
}

constexpr int PJ_MAX_PAIRS = 512;      // rotated pairs of a head at most

// Sums of two numbers per thread over the block, to every thread. `red` holds 2 * 32 floats.
__device__ __forceinline__ float2 pn_block_sum2(float a, float b, float* red) {
    a = gb_warp_sum(a);
    b = gb_warp_sum(b);
    const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    if ((threadIdx.x & 31) == 0) {
        red[warp] = a;
        red[32 + warp] = b;
    }
    __syncthreads();
    float sa = 0.f, sb = 0.f;
    for (int w = 0; w < warps; ++w) {
        sa += red[w];
        sb += red[32 + w];
    }
    return make_float2(sa, sb);
}

// cos and sin of this row's angles, times the magnitude, into shared memory (the caller synchronises)
__device__ __forceinline__ void pn_angles(float2* cs, const float* inv_freq, int half, int pos, float magnitude) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, c;
        sincosf((float)pos * inv_freq[i], &sn, &c);
        cs[i] = make_float2(c * magnitude, sn * magnitude);
    }
}

// ----------------------------------------------------------------------------------------------
// One block per row. qkv [n, ld]: H*D query, G*D key, G*V value columns. Two neighbouring channels per step where the sizes
// allow (VEC: D, V, rot/2 and the row starts even), single channels otherwise.
// ----------------------------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(512) projection_norm_rope_write_kernel(
    const float* __restrict__ qkv, long long ld, const float* __restrict__ q_gain, const float* __restrict__ k_gain,
    const float* __restrict__ inv_freq, float magnitude, const int* __restrict__ positions, const int* __restrict__ slots,
    T* __restrict__ q_out, T* __restrict__ kcache, T* __restrict__ vcache, int n, int H, int G, int D, int V, int rot, float eps,
    int page_size, long long num_slots, int write_kv, int* __restrict__ status) {
    __shared__ float red[64];
    __shared__ float2 cs[PJ_MAX_PAIRS];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int row = blockIdx.x;
    if (row >= n) return;
    const int pos = positions[row];
    if (pos < 0) return;
    const float* src = qkv + (size_t)row * ld;
    const int qc = H * D, kc = G * D, half = rot / 2;
    bool store = write_kv != 0;
    const long long slot = slots[row];
    if (store && (slot < 0 || slot >= num_slots)) {
        if (threadIdx.x == 0) atomicOr(status, GB_STATUS_BAD_SLOT);
        store = false;
    }
    const long long page = slot / page_size;
    const int off = (int)(slot % page_size);
    pn_angles(cs, inv_freq, half, pos, magnitude);
    float sq = 0.f, sk = 0.f;
    if (VEC) {
        for (int c = 2 * threadIdx.x; c < qc; c += 2 * blockDim.x) {
            const float2 x = *reinterpret_cast<const float2*>(src + c);
            sq = fmaf(x.x, x.x, fmaf(x.y, x.y, sq));
        }
        for (int c = 2 * threadIdx.x; c < kc; c += 2 * blockDim.x) {
            const float2 x = *reinterpret_cast<const float2*>(src + qc + c);
            sk = fmaf(x.x, x.x, fmaf(x.y, x.y, sk));
        }
    } else {
        for (int c = threadIdx.x; c < qc; c += blockDim.x) sq = fmaf(src[c], src[c], sq);
        for (int c = threadIdx.x; c < kc; c += blockDim.x) sk = fmaf(src[qc + c], src[qc + c], sk);
    }
    const float2 ss = pn_block_sum2(sq, sk, red);      // (its barrier also publishes the angles)
    const float rq = q_gain ? 1.0f / sqrtf(ss.x / (float)qc + eps) : 1.f, rk = k_gain ? 1.0f / sqrtf(ss.y / (float)kc + eps) : 1.f;
    constexpr int STEP = VEC ? 2 : 1;
    const int qk_end = store ? qc + kc : qc;           // without a slot the keys go nowhere
    for (int c = STEP * threadIdx.x; c < qk_end; c += STEP * blockDim.x) {
        const bool is_q = c < qc;
        const int head = c / D, i = c - head * D;      // heads 0 .. H-1 are queries, then keys
        const float* gain = is_q ? q_gain : (k_gain ? k_gain - qc : nullptr);
        const float r = is_q ? rq : rk;
        // the other half of this channel's pair, and the sign with which it comes in
        const int other = i < rot ? (i < half ? c + half : c - half) : c;
        const int pair = i < rot ? (i < half ? i : i - half) : 0;
        const float sign = i < half ? -1.f : 1.f;
        T* dst = is_q ? q_out + (size_t)row * qc + c : kcache + ((page * G + (head - H)) * page_size + off) * D + i;
        if (VEC) {
            float2 x = *reinterpret_cast<const float2*>(src + c);
            x.x *= r; x.y *= r;
            if (gain) { const float2 g = *reinterpret_cast<const float2*>(gain + c); x.x *= g.x; x.y *= g.y; }
            if (i < rot) {
                float2 y = *reinterpret_cast<const float2*>(src + other);
                y.x *= r; y.y *= r;
                if (gain) { const float2 g = *reinterpret_cast<const float2*>(gain + other); y.x *= g.x; y.y *= g.y; }
                const float2 a = cs[pair], b = cs[pair + 1];
                x.x = x.x * a.x + sign * (y.x * a.y);
                x.y = x.y * b.x + sign * (y.y * b.y);
            }
            pn_store2(dst, x.x, x.y);
        } else {
            float x = src[c] * r;
            if (gain) x *= gain[c];
            if (i < rot) {
                float y = src[other] * r;
                if (gain) y *= gain[other];
                x = x * cs[pair].x + sign * (y * cs[pair].y);
            }
            *dst = gb_from_float<T>(x);
        }
    }
    if (!store) return;
    const float* v = src + qc + kc;
    for (int c = STEP * threadIdx.x; c < G * V; c += STEP * blockDim.x) {
        const int g = c / V, i = c - g * V;
        T* dst = vcache + ((page * G + g) * page_size + off) * V + i;
        if (VEC) {
            const float2 x = *reinterpret_cast<const float2*>(v + c);
            pn_store2(dst, x.x, x.y);
        } else {
            *dst = gb_from_float<T>(v[c]);
        }
    }
}

GB_EXPORT int gb_projection_norm_rope_write(const float* qkv, long long ld, const float* q_gain, const float* k_gain, const float* inv_freq,
                                            float magnitude, const int* positions, const int* slots, void* q_out, void* kcache, void* vcache,
                                            int dtype, int n, int H, int G, int D, int V, int rot, float eps, int page_size,
                                            long long num_slots, int write_kv, int* status, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && H > 0 && G > 0 && D > 0 && V > 0 && page_size > 0, "gb_projection_norm_rope_write: bad sizes");
    GB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D && rot / 2 <= PJ_MAX_PAIRS, "gb_projection_norm_rope_write: %d rotated channels of %d", rot, D);
    GB_REQUIRE(rot == 0 || inv_freq != nullptr, "gb_projection_norm_rope_write: a rotation needs its frequencies");
    GB_REQUIRE(dtype == GB_F32 || dtype == GB_BF16, "gb_projection_norm_rope_write: unsupported dtype %d", dtype);
    if (n == 0) return 0;
    const bool vec = D % 2 == 0 && V % 2 == 0 && rot % 4 == 0 && ld % 2 == 0 && ((uintptr_t)qkv & 7) == 0 && ((uintptr_t)q_gain & 7) == 0 &&
                     ((uintptr_t)k_gain & 7) == 0 && ((uintptr_t)q_out & 7) == 0;
    // few rows: wide blocks, so that a row's channels are few per thread; many rows fill the GPU with narrower ones
    const int threads = n > 296 ? 256 : 512;
#define PN_CASE(TT, VV)                                                                                                                       \
    gb_launch(GB_PDL_ELEMENTWISE, projection_norm_rope_write_kernel<TT, VV>, dim3(n), dim3(threads), 0, stream, qkv, ld, q_gain, k_gain, inv_freq, \
              magnitude, positions, slots, (TT*)q_out, (TT*)kcache, (TT*)vcache, n, H, G, D, V, rot, eps, page_size, num_slots, write_kv, status)
    if (dtype == GB_F32) {
        if (vec) PN_CASE(float, true); else PN_CASE(float, false);
    } else {
        if (vec) PN_CASE(__nv_bfloat16, true); else PN_CASE(__nv_bfloat16, false);
    }
#undef PN_CASE
    return gb_check_launch("gb_projection_norm_rope_write");
}

// ----------------------------------------------------------------------------------------------
// One block per row. proj [n, ld]: qr query-latent columns, c latent columns, r columns of the shared key part. cq [n, qr]
// receives the normed query latent; with write_kv the cache row [c | r] at the row's slot the normed latent and the rotated
// key part (channel i with channel i + rot_dims/2 over the first rot_dims of it).
// ----------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) latent_inputs_kernel(const float* __restrict__ proj, long long ld, const float* __restrict__ q_gain,
                                                            const float* __restrict__ latent_gain, const float* __restrict__ inv_freq,
                                                            float magnitude, const int* __restrict__ positions, const int* __restrict__ slots,
                                                            T* __restrict__ cq, T* __restrict__ cache, int n, int qr, int c, int r, int rot_dims,
                                                            long long num_slots, float eps, int write_kv, int* __restrict__ status) {
    __shared__ float red[64];
    __shared__ float2 cs[PJ_MAX_PAIRS];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int row = blockIdx.x;
    if (row >= n) return;
    const int pos = positions[row];
    T* qdst = cq + (size_t)row * qr;
    if (pos < 0) {      // a padding row goes on into the next product: zeros
        for (int j = threadIdx.x; j < qr; j += blockDim.x) qdst[j] = gb_from_float<T>(0.f);
        return;
    }
    const float* src = proj + (size_t)row * ld;
    const float* lat = src + qr;
    const int half = rot_dims / 2;
    bool store = write_kv != 0;
    const long long slot = slots[row];
    if (store && (slot < 0 || slot >= num_slots)) {
        if (threadIdx.x == 0) atomicOr(status, GB_STATUS_BAD_SLOT);
        store = false;
    }
    if (store) pn_angles(cs, inv_freq, half, pos, magnitude);
    float sq = 0.f, sl = 0.f;
    for (int j = threadIdx.x; j < qr; j += blockDim.x) sq = fmaf(src[j], src[j], sq);
    if (store)
        for (int j = threadIdx.x; j < c; j += blockDim.x) sl = fmaf(lat[j], lat[j], sl);
    const float2 ss = pn_block_sum2(sq, sl, red);
    const float rq = 1.0f / sqrtf(ss.x / (float)qr + eps);
    for (int j = threadIdx.x; j < qr; j += blockDim.x) qdst[j] = gb_from_float<T>(q_gain[j] * (src[j] * rq));
    if (!store) return;
    const float rl = 1.0f / sqrtf(ss.y / (float)c + eps);
    T* dst = cache + (size_t)slot * (c + r);
    for (int j = threadIdx.x; j < c; j += blockDim.x) dst[j] = gb_from_float<T>(latent_gain[j] * (lat[j] * rl));
    const float* key = lat + c;
    for (int j = threadIdx.x; j < r; j += blockDim.x) {
        float x = key[j];
        if (j < rot_dims) {
            const int i = j < half ? j : j - half;
            const float y = key[j < half ? j + half : j - half];
            x = j < half ? x * cs[i].x - y * cs[i].y : x * cs[i].x + y * cs[i].y;
        }
        dst[c + j] = gb_from_float<T>(x);
    }
}

GB_EXPORT int gb_latent_inputs(const float* proj, long long ld, const float* q_gain, const float* latent_gain, const float* inv_freq,
                               float magnitude, const int* positions, const int* slots, void* cq, void* cache, int dtype, int n, int qr, int c,
                               int r, int rot_dims, long long num_slots, float eps, int write_kv, int* status, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && qr > 0 && c > 0 && r >= 0, "gb_latent_inputs: bad sizes");
    GB_REQUIRE(rot_dims >= 0 && rot_dims <= r && rot_dims % 2 == 0 && rot_dims / 2 <= PJ_MAX_PAIRS,
               "gb_latent_inputs: %d rotated numbers do not fit a part of %d", rot_dims, r);
    GB_REQUIRE(!write_kv || latent_gain != nullptr, "gb_latent_inputs: a latent that is stored needs its gain");
    GB_REQUIRE(dtype == GB_F32 || dtype == GB_BF16, "gb_latent_inputs: unsupported dtype %d", dtype);
    if (n == 0) return 0;
    if (dtype == GB_F32)
        gb_launch(GB_PDL_ELEMENTWISE, latent_inputs_kernel<float>, dim3(n), dim3(256), 0, stream, proj, ld, q_gain, latent_gain, inv_freq,
                  magnitude, positions, slots, (float*)cq, (float*)cache, n, qr, c, r, rot_dims, num_slots, eps, write_kv, status);
    else
        gb_launch(GB_PDL_ELEMENTWISE, latent_inputs_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, stream, proj, ld, q_gain, latent_gain, inv_freq,
                  magnitude, positions, slots, (__nv_bfloat16*)cq, (__nv_bfloat16*)cache, n, qr, c, r, rot_dims, num_slots, eps, write_kv, status);
    return gb_check_launch("gb_latent_inputs");
}
