// A selective state-space mixer with one scalar decay per head and token (state-space duality), and the causal convolution in
// front of it. Per head the state S is an [N, V] matrix of float32 that lives in the request's state slot:
//     dt = softplus(dt_raw + dt_bias);  S <- exp(-exp(a_log) dt) S + dt B x^T;  y = S^T C + skip x
// Heads share B and C (N numbers each) in groups. x | B | C come out of one causal convolution with bias and SiLU.
//
//   gb_ring_conv     y[t, c] = silu(b[c] + sum_j w[c, j] x[t - (taps-1) + j, c]) along each request's rows. The slot keeps the
//                    last inputs in a RING of `taps` rows, the input of position p in row p mod taps: a single new token then
//                    writes a row that nobody reads in that step, so many blocks may share a request's inputs without a second
//                    kernel that moves them up.
//   gb_ssd_decode    steps of single tokens: convolution, step size, decay, update, read-out and skip in one kernel that reads
//                    and writes S once.
//   gb_ssd_chunks    prompt portions in bfloat16 on the tensor cores: chunks of 64 tokens side by side.
// (gb_ssd_walk, in delta_rule.cu, takes float32 portions and other sizes token by token.)
#include "common.cuh"

// ----------------------------------------------------------------------------------------------
// Convolution over portions. A thread takes RC_ROWS consecutive rows of VEC channels: every load is asked for before the first
// use, an input row is read once per thread. Rows of several requests, or rows that reach back before their portion, take the
// slow path row by row.
// ----------------------------------------------------------------------------------------------
constexpr int RC_ROWS = 8, RC_THREADS = 128;

struct RingConvArgs {
    const float* x;
    long long ldx;
    const float* w;             // [C, taps], the last column weighs the current token
    const float* bias;          // [C] or nullptr
    void* y;
    long long ldy;
    float* state;               // per slot `state_stride` numbers, of which [taps, C] from `state_off` on
    long long state_stride, state_off;
    const int* row_seq;
    const int* positions;
    const int* seq_first_row;
    const int* seq_slots;
    int row0, n, C, taps, num_slots;
    int* status;
};

__device__ __forceinline__ float rc_silu(float v) { return v / (1.0f + expf(-v)); }

template <int TAPS, typename T>
__global__ void __launch_bounds__(RC_THREADS) ring_conv_kernel(RingConvArgs p) {
    constexpr int VEC = 4, IN = RC_ROWS + TAPS - 1;
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int first = p.row0 + blockIdx.x * RC_ROWS, last = min(first + RC_ROWS, p.n) - 1;
    const int ch = (blockIdx.y * RC_THREADS + threadIdx.x) * VEC;
    if (ch >= p.C) return;
    float4 wv[TAPS];            // the weights of the four channels, one float4 per tap
    {
        float raw[VEC][TAPS];
#pragma unroll
        for (int c = 0; c < VEC; ++c)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) raw[c][j] = p.w[(size_t)(ch + c) * TAPS + j];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wv[j] = make_float4(raw[0][j], raw[1][j], raw[2][j], raw[3][j]);
    }
    const float4 b = p.bias ? *reinterpret_cast<const float4*>(p.bias + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
    const int seq = p.row_seq[first], r0 = p.seq_first_row[seq];
    auto store = [&](int row, float4 a) {
        T* dst = (T*)p.y + (size_t)row * p.ldy + ch;
        a = make_float4(rc_silu(a.x), rc_silu(a.y), rc_silu(a.z), rc_silu(a.w));
        if constexpr (sizeof(T) == 2) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(a.x, a.y), hi = __floats2bfloat162_rn(a.z, a.w);
            uint2 o;
            o.x = *reinterpret_cast<const unsigned*>(&lo);
            o.y = *reinterpret_cast<const unsigned*>(&hi);
            *reinterpret_cast<uint2*>(dst) = o;
        } else {
            *reinterpret_cast<float4*>(dst) = a;
        }
    };
    auto mac = [](float4 acc, float4 w, float4 v) {
        return make_float4(fmaf(w.x, v.x, acc.x), fmaf(w.y, v.y, acc.y), fmaf(w.z, v.z, acc.z), fmaf(w.w, v.w, acc.w));
    };
    if (p.row_seq[last] == seq && first - (TAPS - 1) >= r0) {
        if (p.positions[first] < 0) return;
        float4 in[IN];
#pragma unroll
        for (int i = 0; i < IN; ++i) {
            const int src = min(first - (TAPS - 1) + i, last);
            in[i] = *reinterpret_cast<const float4*>(p.x + (size_t)src * p.ldx + ch);
        }
#pragma unroll
        for (int i = 0; i < RC_ROWS; ++i) {
            if (first + i > last) break;
            float4 acc = b;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = mac(acc, wv[j], in[i + j]);
            store(first + i, acc);
        }
        return;
    }
    for (int row = first; row <= last; ++row) {
        const int pos = p.positions[row];
        if (pos < 0) continue;
        const int s = p.row_seq[row], begin = p.seq_first_row[s], slot = p.seq_slots[s];
        if (slot < 0 || slot >= p.num_slots) {
            atomicOr(p.status, GB_STATUS_BAD_SLOT);
            continue;
        }
        const float* ring = p.state + (size_t)slot * p.state_stride + p.state_off;
        float4 acc = b;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int back = TAPS - 1 - j;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (row - back >= begin) v = *reinterpret_cast<const float4*>(p.x + (size_t)(row - back) * p.ldx + ch);
            else if (pos - back >= 0) v = *reinterpret_cast<const float4*>(ring + (size_t)((pos - back) % TAPS) * p.C + ch);
            acc = mac(acc, wv[j], v);
        }
        store(row, acc);
    }
}

// Any number of taps, any alignment: a thread per (row, channel).
template <typename T>
__global__ void __launch_bounds__(256) ring_conv_plain_kernel(RingConvArgs p) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int row = p.row0 + blockIdx.x, ch = blockIdx.y * 256 + threadIdx.x;
    if (row >= p.n || ch >= p.C) return;
    const int pos = p.positions[row];
    if (pos < 0) return;
    const int s = p.row_seq[row], begin = p.seq_first_row[s], slot = p.seq_slots[s];
    if (slot < 0 || slot >= p.num_slots) {
        atomicOr(p.status, GB_STATUS_BAD_SLOT);
        return;
    }
    const float* ring = p.state + (size_t)slot * p.state_stride + p.state_off;
    float acc = p.bias ? p.bias[ch] : 0.f;
    for (int j = 0; j < p.taps; ++j) {
        const int back = p.taps - 1 - j;
        float v = 0.f;
        if (row - back >= begin) v = p.x[(size_t)(row - back) * p.ldx + ch];
        else if (pos - back >= 0) v = ring[(size_t)((pos - back) % p.taps) * p.C + ch];
        acc = fmaf(p.w[(size_t)ch * p.taps + j], v, acc);
    }
    ((T*)p.y)[(size_t)row * p.ldy + ch] = gb_from_float<T>(rc_silu(acc));
}

// After every reader: the last min(taps, rows) inputs of each request's portion go into its ring.
__global__ void __launch_bounds__(256) ring_conv_state_kernel(RingConvArgs p, const int* __restrict__ seq_start_pos, int seq0, int S) {
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int seq = seq0 + blockIdx.x, ch = blockIdx.y * 256 + threadIdx.x;
    if (seq >= S || ch >= p.C) return;
    const int start = seq_start_pos[seq];
    if (start < 0) return;
    const int slot = p.seq_slots[seq];
    if (slot < 0 || slot >= p.num_slots) return;
    const int r0 = p.seq_first_row[seq], len = p.seq_first_row[seq + 1] - r0;
    float* ring = p.state + (size_t)slot * p.state_stride + p.state_off;
    for (int i = max(0, len - p.taps); i < len; ++i) ring[(size_t)((start + i) % p.taps) * p.C + ch] = p.x[(size_t)(r0 + i) * p.ldx + ch];
}

// Rows row0 .. n-1 and requests seq0 .. S-1 (the ones before are not touched).
GB_EXPORT int gb_ring_conv(const float* x, long long ldx, const float* w, const float* bias, void* y, int y_dtype, long long ldy,
                           float* state, long long state_stride, long long state_off, const int* row_seq, const int* positions,
                           const int* seq_first_row, const int* seq_start_pos, const int* seq_slots, int row0, int n, int seq0, int S,
                           int C, int taps, int num_slots, int update_state, int* status, cudaStream_t stream) {
    GB_REQUIRE(n >= 0 && S >= 0 && row0 >= 0 && seq0 >= 0 && C > 0 && taps >= 1 && taps <= 64, "gb_ring_conv: bad sizes (taps %d)", taps);
    GB_REQUIRE(y_dtype == GB_F32 || y_dtype == GB_BF16, "gb_ring_conv: unsupported output dtype %d", y_dtype);
    if (n <= row0 || S <= seq0) return 0;
    RingConvArgs p = {x, ldx, w, bias, y, ldy, state, state_stride, state_off, row_seq, positions, seq_first_row, seq_slots, row0, n, C,
                      taps, num_slots, status};
    const bool vec = C % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 && taps <= 4 &&
                     (((uintptr_t)x | (uintptr_t)bias | (uintptr_t)state) & 15) == 0 && ((uintptr_t)y & (y_dtype == GB_F32 ? 15 : 7)) == 0;
    if (vec) {
        const dim3 grid(gb_ceil_div(n - row0, RC_ROWS), gb_ceil_div(C / 4, RC_THREADS));
#define RC_GO(K)                                                                                                                    \
    if (taps == K) {                                                                                                                \
        if (y_dtype == GB_F32) gb_launch(GB_PDL_ELEMENTWISE, ring_conv_kernel<K, float>, grid, dim3(RC_THREADS), 0, stream, p);      \
        else gb_launch(GB_PDL_ELEMENTWISE, ring_conv_kernel<K, __nv_bfloat16>, grid, dim3(RC_THREADS), 0, stream, p);                \
    }
        RC_GO(1) RC_GO(2) RC_GO(3) RC_GO(4)
#undef RC_GO
    } else {
        const dim3 grid(n - row0, gb_ceil_div(C, 256));
        if (y_dtype == GB_F32) gb_launch(GB_PDL_ELEMENTWISE, ring_conv_plain_kernel<float>, grid, dim3(256), 0, stream, p);
        else gb_launch(GB_PDL_ELEMENTWISE, ring_conv_plain_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, p);
    }
    int rc = gb_check_launch("gb_ring_conv");
    if (rc || !update_state) return rc;
    gb_launch(GB_PDL_ELEMENTWISE, ring_conv_state_kernel, dim3(S - seq0, gb_ceil_div(C, 256)), dim3(256), 0, stream, p, seq_start_pos, seq0, S);
    return gb_check_launch("gb_ring_conv (state)");
}

// ----------------------------------------------------------------------------------------------
// Single tokens. Grid (request, head, block of value columns); 256 threads: a thread owns VEC neighbouring columns of every
// `par`-th row of S, so a warp reads and writes whole row segments; the first SD_U rows' loads are in flight before the
// convolution of the block's channels begins. The rows' shares of the read-out meet in shared memory in a fixed order.
// ----------------------------------------------------------------------------------------------
constexpr int SD_THREADS = 256, SD_U = 8, SD_MAX_STATE = 1024;

struct SsdDecodeArgs {
    const float* xbc;           // [n, ldx]: x | B | C before the convolution
    long long ldx;
    const float* dt_raw;        // [n, ld_dt]
    long long ld_dt;
    const float* conv_w;        // [C, taps]
    const float* conv_b;        // [C]
    const float* dt_bias;
    const float* a_log;
    const float* skip;
    float* state;
    long long state_stride, conv_off;
    float* y;                   // [n, heads * V]
    const int* seq_first_row;
    const int* seq_start_pos;
    const int* seq_slots;
    int heads, groups, N, V, taps, num_slots, write_state, cols;
    int* status;
};

template <int VEC>
struct SdVec;
template <>
struct SdVec<1> { typedef float type; };
template <>
struct SdVec<4> { typedef float4 type; };

// One channel's convolution at a single new token: `own` is the token's input, the ring holds the ones before.
template <int TAPS>
__device__ __forceinline__ float sd_conv(const SsdDecodeArgs& p, const float* ring, int ch, int pos, int C, float own) {
    const int taps = TAPS > 0 ? TAPS : p.taps;
    float acc = p.conv_b[ch];
    if constexpr (TAPS > 0) {
        float w[TAPS], v[TAPS];           // every load before the first use
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            w[j] = p.conv_w[(size_t)ch * TAPS + j];
            const int q = pos - (TAPS - 1) + j;
            v[j] = j == TAPS - 1 ? own : q >= 0 ? ring[(size_t)(q % TAPS) * C + ch] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], v[j], acc);
    } else {
        for (int j = 0; j < taps; ++j) {
            const int q = pos - (taps - 1) + j;
            if (q >= 0) acc = fmaf(p.conv_w[(size_t)ch * taps + j], j == taps - 1 ? own : ring[(size_t)(q % taps) * C + ch], acc);
        }
    }
    return rc_silu(acc);
}

template <int VEC, int TAPS>
__global__ void __launch_bounds__(SD_THREADS, 3) ssd_decode_kernel(SsdDecodeArgs p) {
    typedef typename SdVec<VEC>::type vec_t;
    extern __shared__ __align__(16) float sd_smem[];
    float* Bs = sd_smem, *Cs = Bs + p.N, *xs = Cs + p.N, *part = xs + ((p.cols + 3) & ~3) + ((4 - (2 * p.N) % 4) & 3);
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int seq = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * p.cols, nc = min(p.cols, p.V - c0);
    const int pos = p.seq_start_pos[seq], slot = p.seq_slots[seq];
    const size_t row = (size_t)p.seq_first_row[seq];
    if (pos < 0) return;
    if (slot < 0 || slot >= p.num_slots) {
        if (threadIdx.x == 0) atomicOr(p.status, GB_STATUS_BAD_SLOT);
        return;
    }
    const int N = p.N, V = p.V, tid = threadIdx.x, taps = TAPS > 0 ? TAPS : p.taps;
    const int inner = p.heads * V, per = p.heads / p.groups, g = head / per, C = inner + 2 * p.groups * N;
    float* slot_state = p.state + (size_t)slot * p.state_stride;
    const int nvec = nc / VEC, par = SD_THREADS / nvec;         // (VEC divides nc: the launch sees to it)
    const int my_c = (tid % nvec) * VEC, my_r = tid / nvec;
    const bool active = my_r < par;
    float* S = slot_state + ((size_t)head * N) * V + c0 + my_c;
    vec_t first[SD_U];
#pragma unroll
    for (int u = 0; u < SD_U; ++u) {
        const int r = my_r + u * par;
        if (active && r < N) first[u] = *reinterpret_cast<const vec_t*>(S + (size_t)r * V);
    }
    const float dt_raw = p.dt_raw[row * p.ld_dt + head] + p.dt_bias[head], rate = p.a_log[head], skip = p.skip[head];
    // the token's B, C and this block's x: the convolution over the ring's last inputs and the token's own
    float* ring = slot_state + p.conv_off;
    const bool keeps_bc = head % per == 0 && blockIdx.z == 0;   // one block per group stores the shared channels' inputs
    const int channels = 2 * N + nc;
    auto channel = [&](int i) {
        return i < N ? inner + g * N + i : i < 2 * N ? inner + p.groups * N + g * N + (i - N) : head * V + c0 + (i - 2 * N);
    };
    for (int i0 = tid; i0 < channels; i0 += 2 * SD_THREADS) {   // two channels of a thread at a time
        const int i1 = i0 + SD_THREADS;
        const int ch0 = channel(i0), ch1 = i1 < channels ? channel(i1) : ch0;
        const float own0 = p.xbc[row * p.ldx + ch0], own1 = p.xbc[row * p.ldx + ch1];
        const float a0 = sd_conv<TAPS>(p, ring, ch0, pos, C, own0), a1 = i1 < channels ? sd_conv<TAPS>(p, ring, ch1, pos, C, own1) : 0.f;
        // (B, C and x lie one behind the other)
        Bs[i0] = a0;
        if (i1 < channels) Bs[i1] = a1;
        if (p.write_state) {
            if (i0 >= 2 * N || keeps_bc) ring[(size_t)(pos % taps) * C + ch0] = own0;
            if (i1 < channels && (i1 >= 2 * N || keeps_bc)) ring[(size_t)(pos % taps) * C + ch1] = own1;
        }
    }
    const float dt = gb_softplus(dt_raw);
    const float decay = expf(-expf(rate) * dt);
    __syncthreads();
    float x[VEC], acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        x[e] = active ? xs[my_c + e] * dt : 0.f;
        acc[e] = 0.f;
    }
    if (active) {
        for (int r0 = my_r; r0 < N; r0 += SD_U * par) {
            if (r0 != my_r) {
#pragma unroll
                for (int u = 0; u < SD_U; ++u) {
                    const int r = r0 + u * par;
                    if (r < N) first[u] = *reinterpret_cast<const vec_t*>(S + (size_t)r * V);
                }
            }
#pragma unroll
            for (int u = 0; u < SD_U; ++u) {
                const int r = r0 + u * par;
                if (r < N) {
                    const float b = Bs[r], c = Cs[r];
                    float* f = reinterpret_cast<float*>(&first[u]);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        f[e] = fmaf(decay, f[e], b * x[e]);
                        acc[e] = fmaf(c, f[e], acc[e]);
                    }
                    if (p.write_state) *reinterpret_cast<vec_t*>(S + (size_t)r * V) = first[u];
                }
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) part[my_r * nc + my_c + e] = acc[e];
    }
    __syncthreads();
    const int rows = min(par, N);
    for (int c = tid; c < nc; c += SD_THREADS) {
        float o = 0.f;
#pragma unroll 8
        for (int r = 0; r < rows; ++r) o += part[r * nc + c];
        p.y[row * inner + (size_t)head * V + c0 + c] = fmaf(skip, xs[c], o);
    }
}

// Every request of seq 0 .. S-1 brings exactly one row.
GB_EXPORT int gb_ssd_decode(const float* xbc, long long ldx, const float* dt_raw, long long ld_dt, const float* conv_w, const float* conv_b,
                            const float* dt_bias, const float* a_log, const float* skip, float* state, long long state_stride,
                            long long conv_off, float* y, const int* seq_first_row, const int* seq_start_pos, const int* seq_slots, int S,
                            int heads, int groups, int N, int V, int taps, int num_slots, int write_state, int* status,
                            cudaStream_t stream) {
    GB_REQUIRE(S >= 0 && heads > 0 && groups > 0 && heads % groups == 0, "gb_ssd_decode: heads %d must be a multiple of groups %d", heads, groups);
    GB_REQUIRE(N > 0 && N <= SD_MAX_STATE && V > 0 && taps >= 1 && taps <= 64, "gb_ssd_decode: state size %d (1..%d), value size %d, taps %d", N,
               SD_MAX_STATE, V, taps);
    if (S == 0) return 0;
    const bool vec = V % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    // columns per block: whole heads when there are enough (request, head) pairs to fill the GPU, parts of 32 or 16 when few
    int cols = V < 128 ? V : 128;
    if (vec) {
        while (cols > 16 && cols % 8 == 0 && (long long)S * heads * gb_ceil_div(V, cols) < 148) cols /= 2;
        if (cols % 4) cols = 4;
    }
    SsdDecodeArgs p = {xbc, ldx, dt_raw, ld_dt, conv_w, conv_b, dt_bias, a_log, skip, state, state_stride, conv_off, y, seq_first_row,
                       seq_start_pos, seq_slots, heads, groups, N, V, taps, num_slots, write_state, cols, status};
    const dim3 grid(S, heads, gb_ceil_div(V, cols));
    const size_t smem = ((size_t)2 * N + cols + 8 + SD_THREADS * (vec ? 4 : 1)) * sizeof(float);
    if (vec && taps == 4) gb_launch(GB_PDL_ATTENTION, ssd_decode_kernel<4, 4>, grid, dim3(SD_THREADS), smem, stream, p);
    else if (vec) gb_launch(GB_PDL_ATTENTION, ssd_decode_kernel<4, 0>, grid, dim3(SD_THREADS), smem, stream, p);
    else gb_launch(GB_PDL_ATTENTION, ssd_decode_kernel<1, 0>, grid, dim3(SD_THREADS), smem, stream, p);
    return gb_check_launch("gb_ssd_decode");
}

// ----------------------------------------------------------------------------------------------
// Prompt portions in bfloat16. With c_i the running sum of the log decays inside a chunk of SC_L tokens (inclusive), S_0 the
// state in front of the chunk and M_ij = (C_i . B_j) exp(c_i - c_j) dt_j for j <= i:
//     y_i = exp(c_i) C_i S_0 + sum_j M_ij x_j + skip x_i,      S_end = exp(c_last) S_0 + sum_j exp(c_last - c_j) dt_j B_j x_j^T
//   ssd_chunk_state   per (chunk, head): the chunk's own sum, from a zero state; dt_j and c_j
//   ssd_chain         per element of S: through the request's chunks in order, in float32; a chunk's own sum is replaced by the
//                     state in front of it, the request's slot receives the last state
//   ssd_chunk_out     per (chunk, head): the read-outs
// Logarithms of decays, their sums, exponentials and step sizes are float32. x, B and C are bfloat16 (the convolution's output);
// what they are multiplied with (the weights of the chunk's sum, S_0, M) is float32 and enters the products as a sum of two
// bfloat16 numbers, so that about 16 bits of it count. S_0 is handed over in that form already, one 32-bit word per element
// (the rounded value below, what the rounding left above it); as columns of a product the two halves of a word are neighbours,
// so the two sums that belong to one element end up in one thread. The words of eight neighbouring channels lie in the order
// 0 2 4 6 1 3 5 7: of two 8-column tiles the first then gives a thread an even channel and the second the odd one behind it,
// which are the two channels that the thread holds of M x.
// Chunk c of request s has the number seq_first_row[s] / SC_L + s + c: unique, and below n / SC_L + S.
// ----------------------------------------------------------------------------------------------
constexpr int SC_L = 64, SC_THREADS = 128, SC_OUT_THREADS = 256;

struct SsdChunkArgs {
    const __nv_bfloat16* xbc;   // [n, ldx]: x | B | C after the convolution
    long long ldx;
    const float* dt_raw;
    long long ld_dt;
    const float* dt_bias;
    const float* a_log;
    const float* skip;
    float* state;
    long long state_stride;
    float* y;                   // [n, heads * V]
    float* chunk_state;         // [chunks, heads, N, V]
    float* chunk_steps;         // [chunks, heads, 2, SC_L]: dt_j, c_j
    const int* seq_first_row;
    const int* seq_start_pos;
    const int* seq_slots;
    int S, tiles, heads, groups, N, V, num_slots, write_state, vec;
    int* status;
};

struct SsdChunk {
    int row0, len, number;
};

// which chunk this block works on; false: none
__device__ __forceinline__ bool ssd_find_chunk(const SsdChunkArgs& p, SsdChunk& c) {
    const int seq = blockIdx.x / p.tiles, tile = blockIdx.x % p.tiles;
    if (seq >= p.S || p.seq_start_pos[seq] < 0) return false;
    const int r0 = p.seq_first_row[seq], len = p.seq_first_row[seq + 1] - r0;
    if (tile * SC_L >= len) return false;
    c.row0 = r0 + tile * SC_L;
    c.len = min(SC_L, len - tile * SC_L);
    c.number = r0 / SC_L + seq + tile;
    return true;
}

// step sizes and the inclusive running sum of the log decays of a chunk (rows behind its end: step 0); threads 0 .. 63
__device__ __forceinline__ void ssd_steps(const SsdChunkArgs& p, const SsdChunk& c, int head, float* dt_s, float* cum_s, float* half) {
    float run = 0.f;
    const int t = threadIdx.x, lane = t & 31;
    if (t < SC_L) {
        const float dt = t < c.len ? gb_softplus(p.dt_raw[(size_t)(c.row0 + t) * p.ld_dt + head] + p.dt_bias[head]) : 0.f;
        dt_s[t] = dt;
        run = -expf(p.a_log[head]) * dt;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += v;
        }
        if (t == 31) *half = run;
    }
    __syncthreads();
    if (t < SC_L) cum_s[t] = t < 32 ? run : run + *half;
    __syncthreads();
}

__device__ __forceinline__ void ssd_ldm(unsigned (&r)[4], const __nv_bfloat16* at) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(at);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ssd_ldm_t(unsigned (&r)[4], const __nv_bfloat16* at) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(at);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ssd_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// two floats as the sum of two pairs of bfloat16: hi is the rounded value, lo what the rounding left
__device__ __forceinline__ void ssd_split(float a, float b, unsigned& hi, unsigned& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
    hi = *reinterpret_cast<const unsigned*>(&h);
    lo = *reinterpret_cast<const unsigned*>(&l);
}

__device__ __forceinline__ void ssd_cp16(void* smem, const void* gmem, bool valid) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;        // 0: the 16 bytes are filled with zeros, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void ssd_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void ssd_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

__device__ __forceinline__ int ssd_word_at(int channel) { return (channel & ~7) + (channel & 1) * 4 + ((channel & 7) >> 1); }
__device__ __forceinline__ unsigned ssd_word(float v) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v), l = __float2bfloat16_rn(v - __bfloat162float(h));
    return (unsigned)__bfloat16_as_ushort(h) | ((unsigned)__bfloat16_as_ushort(l) << 16);
}

// A block's threads over the elements of a table of `width` columns: element threadIdx.x, then every blockDim.x-th (no division
// inside the loop).
struct SsdCells {
    int r, c, dr, dc, width;
    __device__ __forceinline__ explicit SsdCells(int w) : width(w) {
        r = threadIdx.x / w;
        c = threadIdx.x - r * w;
        dr = blockDim.x / w;
        dc = blockDim.x - dr * w;
    }
    __device__ __forceinline__ void next() {
        r += dr;
        c += dc;
        if (c >= width) {
            c -= width;
            ++r;
        }
    }
};

// SC_L rows x `width` columns (of which `cols` exist, the rest and the rows behind the chunk's end are zero) into shared memory
__device__ __forceinline__ void ssd_stage(__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, long long lds, int rows, int cols, int width,
                                          bool vec) {
    const int pieces = width / 8;
    if (vec) {                   // (cols is then a multiple of 8 as well)
        for (SsdCells at(pieces); at.r < SC_L; at.next()) {
            const int r = at.r, c = at.c * 8;
            const bool in = r < rows && c < cols;
            ssd_cp16(dst + r * ld + c, in ? src + (size_t)r * lds + c : src, in);
        }
    } else {
        for (SsdCells at(width); at.r < SC_L; at.next()) {
            const int r = at.r, c = at.c;
            dst[r * ld + c] = r < rows && c < cols ? src[(size_t)r * lds + c] : __float2bfloat16_rn(0.f);
        }
    }
}

__global__ void __launch_bounds__(SC_THREADS) ssd_chunk_state_kernel(SsdChunkArgs p) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ float dt_s[SC_L], cum_s[SC_L], half;
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    SsdChunk c;
    if (!ssd_find_chunk(p, c)) return;
    const int head = blockIdx.y, g = head / (p.heads / p.groups), N = p.N, V = p.V, inner = p.heads * V;
    const int NW = (N + 15) & ~15, VW = (V + 15) & ~15, ldb = NW + 8, ldv = VW + 8;
    __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(ssd_smem);      // [L][ldb]
    __nv_bfloat16* Xh = Bs + SC_L * ldb, *Xl = Xh + SC_L * ldv;           // [L][ldv]: exp(c_last - c_j) dt_j x_j in two parts
    const __nv_bfloat16* base = p.xbc + (size_t)c.row0 * p.ldx;
    const __nv_bfloat16* xsrc = base + head * V;
    if (p.vec) ssd_stage(Xh, ldv, xsrc, p.ldx, c.len, V, VW, true);
    ssd_cp_commit();
    ssd_stage(Bs, ldb, base + inner + g * N, p.ldx, c.len, N, NW, p.vec);
    ssd_cp_commit();
    ssd_steps(p, c, head, dt_s, cum_s, &half);
    const float last = cum_s[SC_L - 1];
    float* steps = p.chunk_steps + ((size_t)c.number * p.heads + head) * 2 * SC_L;
    steps[threadIdx.x] = threadIdx.x < SC_L ? dt_s[threadIdx.x] : cum_s[threadIdx.x - SC_L];
    ssd_cp_wait<1>();                        // (a thread reads back the pieces that it asked for itself)
    if (p.vec) {
        for (SsdCells at(VW / 8); at.r < SC_L; at.next()) {
            const int r = at.r, v = at.c * 8;
            uint4 h, l;
            const uint4 raw = *reinterpret_cast<const uint4*>(Xh + r * ldv + v);
            const float w = expf(last - cum_s[r]) * dt_s[r];
            const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&raw);
            float2 f = __bfloat1622float2(q[0]);
            ssd_split(f.x * w, f.y * w, h.x, l.x);
            f = __bfloat1622float2(q[1]);
            ssd_split(f.x * w, f.y * w, h.y, l.y);
            f = __bfloat1622float2(q[2]);
            ssd_split(f.x * w, f.y * w, h.z, l.z);
            f = __bfloat1622float2(q[3]);
            ssd_split(f.x * w, f.y * w, h.w, l.w);
            *reinterpret_cast<uint4*>(Xh + r * ldv + v) = h;
            *reinterpret_cast<uint4*>(Xl + r * ldv + v) = l;
        }
    } else {
        for (SsdCells at(VW / 2); at.r < SC_L; at.next()) {
            const int r = at.r, v = at.c * 2;
            const float w = expf(last - cum_s[r]) * dt_s[r];
            float a = 0.f, b = 0.f;
            if (r < c.len && v < V) a = __bfloat162float(xsrc[(size_t)r * p.ldx + v]) * w;
            if (r < c.len && v + 1 < V) b = __bfloat162float(xsrc[(size_t)r * p.ldx + v + 1]) * w;
            unsigned h, l;
            ssd_split(a, b, h, l);
            *reinterpret_cast<unsigned*>(Xh + r * ldv + v) = h;
            *reinterpret_cast<unsigned*>(Xl + r * ldv + v) = l;
        }
    }
    ssd_cp_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int mt = NW / 16, vt = VW / 16;
    float* out = p.chunk_state + ((size_t)c.number * p.heads + head) * N * V;
    const int ks = (c.len + 15) / 16;                 // (rows behind the chunk's end are zero)
    for (int m = warp; m < mt; m += SC_THREADS / 32) {
        unsigned a[SC_L / 16][4];                     // B^T: 16 state channels x the chunk's tokens
#pragma unroll
        for (int k = 0; k < SC_L / 16; ++k) ssd_ldm_t(a[k], Bs + (k * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldb + m * 16 + ((lane >> 3) & 1) * 8);
        for (int v = 0; v < vt; ++v) {
            float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int k = 0; k < SC_L / 16; ++k) {
                if (k >= ks) break;
                unsigned h[4], l[4];
                const int at = (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + v * 16 + (lane >> 4) * 8;
                ssd_ldm_t(h, Xh + at);
                ssd_ldm_t(l, Xl + at);
                ssd_mma(acc[0], a[k], h[0], h[1]);
                ssd_mma(acc[1], a[k], h[2], h[3]);
                ssd_mma(acc[0], a[k], l[0], l[1]);
                ssd_mma(acc[1], a[k], l[2], l[3]);
            }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int r = m * 16 + (lane >> 2) + hf * 8, col = v * 16 + j * 8 + (lane & 3) * 2;
                    if (r >= N) continue;
                    float* o = out + (size_t)r * V + col;
                    if (col + 1 < V && (V & 1) == 0) *reinterpret_cast<float2*>(o) = make_float2(acc[j][hf * 2], acc[j][hf * 2 + 1]);
                    else {
                        if (col < V) o[0] = acc[j][hf * 2];
                        if (col + 1 < V) o[1] = acc[j][hf * 2 + 1];
                    }
                }
        }
    }
}

template <int VEC>
__global__ void __launch_bounds__(256) ssd_chain_kernel(SsdChunkArgs p) {
    typedef typename SdVec<VEC>::type vec_t;
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    const int seq = blockIdx.x, head = blockIdx.y;
    if (p.seq_start_pos[seq] < 0) return;
    const int slot = p.seq_slots[seq];
    if (slot < 0 || slot >= p.num_slots) {
        if (threadIdx.x == 0) atomicOr(p.status, GB_STATUS_BAD_SLOT);
        return;
    }
    const int numbers = p.N * p.V, e = (blockIdx.z * 256 + threadIdx.x) * VEC;
    if (e >= numbers) return;
    const int r0 = p.seq_first_row[seq], len = p.seq_first_row[seq + 1] - r0;
    const int lo = r0 / SC_L + seq, chunks = (len + SC_L - 1) / SC_L;
    float* mine = p.state + (size_t)slot * p.state_stride + (size_t)head * numbers + e;
    vec_t s = *reinterpret_cast<const vec_t*>(mine);
    float* sf = reinterpret_cast<float*>(&s);
    constexpr int U = 8;          // eight chunks' own sums are asked for before the chain through them starts
    for (int c0 = 0; c0 < chunks; c0 += U) {
        vec_t own[U];
        float f[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const size_t at = (size_t)(lo + min(c0 + u, chunks - 1)) * p.heads + head;
            own[u] = *reinterpret_cast<const vec_t*>(p.chunk_state + at * numbers + e);
            f[u] = expf(p.chunk_steps[(at * 2 + 1) * SC_L + SC_L - 1]);
        }
        __syncwarp();             // a thread's words go where its neighbour's sums were: both have read theirs
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u >= chunks) break;
            const size_t at = (size_t)(lo + c0 + u) * p.heads + head;
            unsigned* words = reinterpret_cast<unsigned*>(p.chunk_state) + at * numbers;       // the state in front of this chunk
            if constexpr (VEC == 4) {
                unsigned* eight = words + (e & ~7) + ((e >> 2) & 1) * 2;
                *reinterpret_cast<uint2*>(eight) = make_uint2(ssd_word(sf[0]), ssd_word(sf[2]));
                *reinterpret_cast<uint2*>(eight + 4) = make_uint2(ssd_word(sf[1]), ssd_word(sf[3]));
            } else {
                words[e] = ssd_word(sf[0]);                      // (in order: whoever reads it puts the words in theirs)
            }
            const float* of = reinterpret_cast<const float*>(&own[u]);
#pragma unroll
            for (int i = 0; i < VEC; ++i) sf[i] = fmaf(f[u], sf[i], of[i]);
        }
    }
    if (p.write_state) *reinterpret_cast<vec_t*>(mine) = s;
}

// Eight warps: a warp has 16 of the chunk's tokens and every second tile of 16 value channels (the two warps of the same
// tokens each form their C B^T).
__global__ void __launch_bounds__(SC_OUT_THREADS) ssd_chunk_out_kernel(SsdChunkArgs p) {
    extern __shared__ __align__(16) unsigned char ssd_smem[];
    __shared__ __align__(16) float steps[2 * SC_L];
    gb_pdl_launch_dependents();
    gb_pdl_wait();
    SsdChunk c;
    if (!ssd_find_chunk(p, c)) return;
    const int head = blockIdx.y, g = head / (p.heads / p.groups), N = p.N, V = p.V, inner = p.heads * V;
    const int NW = (N + 15) & ~15, VW = (V + 15) & ~15, ldb = NW + 8, ldv = VW + 8, lds = 2 * VW + 8;
    __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(ssd_smem);      // [L][ldb]
    __nv_bfloat16* Bs = Cs + SC_L * ldb;                                  // [L][ldb]
    __nv_bfloat16* Xs = Bs + SC_L * ldb;                                  // [L][ldv]
    __nv_bfloat16* Ss = Xs + SC_L * ldv;                                  // [NW][lds]: the words of S_0
    const __nv_bfloat16* base = p.xbc + (size_t)c.row0 * p.ldx;
    const size_t number = (size_t)c.number * p.heads + head;
    ssd_stage(Cs, ldb, base + inner + p.groups * N + g * N, p.ldx, c.len, N, NW, p.vec);
    ssd_stage(Bs, ldb, base + inner + g * N, p.ldx, c.len, N, NW, p.vec);
    if (threadIdx.x < SC_L / 2) ssd_cp16(steps + threadIdx.x * 4, p.chunk_steps + number * 2 * SC_L + threadIdx.x * 4, true);
    ssd_cp_commit();
    ssd_stage(Xs, ldv, base + head * V, p.ldx, c.len, V, VW, p.vec);
    const unsigned* S0 = reinterpret_cast<const unsigned*>(p.chunk_state) + number * N * V;
    if (p.vec) {
        for (SsdCells at(VW / 4); at.r < NW; at.next()) {
            const int r = at.r, v = at.c * 4;
            const bool in = r < N && v < V;
            ssd_cp16(Ss + r * lds + 2 * v, in ? S0 + (size_t)r * V + v : S0, in);
        }
    } else {
        for (SsdCells at(VW); at.r < NW; at.next()) {
            const int r = at.r, v = at.c;
            reinterpret_cast<unsigned*>(Ss + r * lds)[ssd_word_at(v)] = r < N && v < V ? S0[(size_t)r * V + v] : 0u;
        }
    }
    ssd_cp_commit();
    ssd_cp_wait<1>();
    __syncthreads();
    const int warp = (threadIdx.x >> 5) & 3, v0 = threadIdx.x >> 7, lane = threadIdx.x & 31;
    const int i0 = warp * 16;                          // this warp's 16 tokens
    const int kn = NW / 16;
    const bool busy = i0 < c.len;
    const __nv_bfloat16* crow = Cs + (i0 + (lane & 15)) * ldb + (lane >> 4) * 8;
    const float* dt_s = steps, *cum_s = steps + SC_L;
    const int ia = i0 + (lane >> 2), ib = ia + 8;
    const float ca = cum_s[ia], cb = cum_s[ib];
    unsigned mh[SC_L / 16][4], ml[SC_L / 16][4];
    if (busy) {
        // C_i . B_j for the tokens up to this warp's last
        float s[SC_L / 8][4];
#pragma unroll
        for (int j = 0; j < SC_L / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        for (int k = 0; k < kn; ++k) {
            unsigned a[4];
            ssd_ldm(a, crow + k * 16);
#pragma unroll
            for (int j2 = 0; j2 < SC_L / 16; ++j2) {
                if (j2 > warp) break;
                unsigned b[4];
                ssd_ldm(b, Bs + (j2 * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldb + k * 16 + ((lane >> 3) & 1) * 8);
                ssd_mma(s[2 * j2], a, b[0], b[1]);
                ssd_mma(s[2 * j2 + 1], a, b[2], b[3]);
            }
        }
        // M in two parts, as the A operand of M x
#pragma unroll
        for (int j = 0; j < SC_L / 8; ++j) {
            if ((j >> 1) > warp) break;
            const int t0 = j * 8 + (lane & 3) * 2, t1 = t0 + 1;
            const float d0 = dt_s[t0], d1 = dt_s[t1], c0 = cum_s[t0], c1 = cum_s[t1];
            const float w0 = t0 <= ia ? s[j][0] * (__expf(ca - c0) * d0) : 0.f, w1 = t1 <= ia ? s[j][1] * (__expf(ca - c1) * d1) : 0.f;
            const float w2 = t0 <= ib ? s[j][2] * (__expf(cb - c0) * d0) : 0.f, w3 = t1 <= ib ? s[j][3] * (__expf(cb - c1) * d1) : 0.f;
            ssd_split(w0, w1, mh[j >> 1][(j & 1) * 2], ml[j >> 1][(j & 1) * 2]);
            ssd_split(w2, w3, mh[j >> 1][(j & 1) * 2 + 1], ml[j >> 1][(j & 1) * 2 + 1]);
        }
    }
    ssd_cp_wait<0>();
    __syncthreads();
    if (!busy) return;
    const float fa = __expf(ca), fb = __expf(cb), skip = p.skip[head];
    for (int v = v0; v < VW / 16; v += 2) {
        float w[4][4];                                 // C S_0: four tiles of words, each an 8-column half of 16 channels
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j][0] = w[j][1] = w[j][2] = w[j][3] = 0.f;
#pragma unroll 4
        for (int k = 0; k < kn; ++k) {
            unsigned a[4], b0[4], b1[4];
            ssd_ldm(a, crow + k * 16);
            const __nv_bfloat16* srow = Ss + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * lds + v * 32 + (lane >> 4) * 8;
            ssd_ldm_t(b0, srow);
            ssd_ldm_t(b1, srow + 16);
            ssd_mma(w[0], a, b0[0], b0[1]);
            ssd_mma(w[1], a, b0[2], b0[3]);
            ssd_mma(w[2], a, b1[0], b1[1]);
            ssd_mma(w[3], a, b1[2], b1[3]);
        }
        float acc[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            acc[j][0] = fa * (w[2 * j][0] + w[2 * j][1]); acc[j][1] = fa * (w[2 * j + 1][0] + w[2 * j + 1][1]);
            acc[j][2] = fb * (w[2 * j][2] + w[2 * j][3]); acc[j][3] = fb * (w[2 * j + 1][2] + w[2 * j + 1][3]);
        }
#pragma unroll
        for (int k = 0; k < SC_L / 16; ++k) {          // + M x
            if (k > warp) break;
            unsigned b[4];
            ssd_ldm_t(b, Xs + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + v * 16 + (lane >> 4) * 8);
            ssd_mma(acc[0], mh[k], b[0], b[1]);
            ssd_mma(acc[1], mh[k], b[2], b[3]);
            ssd_mma(acc[0], ml[k], b[0], b[1]);
            ssd_mma(acc[1], ml[k], b[2], b[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = hf ? ib : ia, col = v * 16 + j * 8 + (lane & 3) * 2;
                if (i >= c.len) continue;
                const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(Xs + i * ldv + col);
                const float y0 = fmaf(skip, __low2float(x), acc[j][hf * 2]), y1 = fmaf(skip, __high2float(x), acc[j][hf * 2 + 1]);
                float* o = p.y + (size_t)(c.row0 + i) * inner + (size_t)head * V + col;
                if (col + 1 < V && (V & 1) == 0) *reinterpret_cast<float2*>(o) = make_float2(y0, y1);
                else {
                    if (col < V) o[0] = y0;
                    if (col + 1 < V) o[1] = y1;
                }
            }
    }
}

static size_t ssd_out_smem(int N, int V) {
    const int NW = (N + 15) & ~15, VW = (V + 15) & ~15;
    return ((size_t)2 * SC_L * (NW + 8) + (size_t)SC_L * (VW + 8) + (size_t)NW * (2 * VW + 8)) * 2;
}

GB_EXPORT int gb_ssd_chunk_rows() { return SC_L; }
// 1 if the chunked form takes these sizes
GB_EXPORT int gb_ssd_chunks_supported(int N, int V) { return N > 0 && V > 0 && N <= 256 && ssd_out_smem(N, V) <= 200 * 1024 ? 1 : 0; }

// chunk_state: float32 [chunks, heads * N * V], chunk_steps: float32 [chunks, heads * 2 * SC_L], chunks at least n / SC_L + S.
GB_EXPORT int gb_ssd_chunks(const void* xbc, long long ldx, const float* dt_raw, long long ld_dt, const float* dt_bias, const float* a_log,
                            const float* skip, float* state, long long state_stride, float* y, const int* seq_first_row,
                            const int* seq_start_pos, const int* seq_slots, int S, int n, int max_rows_per_seq, int heads, int groups, int N,
                            int V, int num_slots, int write_state, int chunks, float* chunk_state, float* chunk_steps, int* status,
                            cudaStream_t stream) {
    GB_REQUIRE(S >= 0 && n >= 0 && heads > 0 && groups > 0 && heads % groups == 0, "gb_ssd_chunks: heads %d must be a multiple of groups %d",
               heads, groups);
    GB_REQUIRE(gb_ssd_chunks_supported(N, V), "gb_ssd_chunks: state size %d and value size %d are not built", N, V);
    GB_REQUIRE(chunks >= n / SC_L + S && chunk_state && chunk_steps && max_rows_per_seq > 0, "gb_ssd_chunks: %d chunks are too few for %d rows of %d requests",
               chunks, n, S);
    if (S == 0 || n == 0) return 0;
    const int tiles = gb_ceil_div(max_rows_per_seq, SC_L);
    const int NW = (N + 15) & ~15, VW = (V + 15) & ~15;
    const int vec = N % 8 == 0 && V % 8 == 0 && ldx % 8 == 0 && (heads * V) % 8 == 0 && ((uintptr_t)xbc & 15) == 0 &&
                    (((uintptr_t)chunk_state | (uintptr_t)chunk_steps | (uintptr_t)state) & 15) == 0 && state_stride % 4 == 0;
    GB_REQUIRE(((uintptr_t)chunk_steps & 15) == 0, "gb_ssd_chunks: the steps' buffer must be 16-byte aligned");
    SsdChunkArgs p = {(const __nv_bfloat16*)xbc, ldx, dt_raw, ld_dt, dt_bias, a_log, skip, state, state_stride, y, chunk_state, chunk_steps,
                      seq_first_row, seq_start_pos, seq_slots, S, tiles, heads, groups, N, V, num_slots, write_state, vec, status};
    const size_t smem_state = ((size_t)SC_L * (NW + 8) + (size_t)2 * SC_L * (VW + 8)) * 2, smem_out = ssd_out_smem(N, V);
    cudaFuncSetAttribute(ssd_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_state);
    cudaFuncSetAttribute(ssd_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
    gb_launch(GB_PDL_ATTENTION, ssd_chunk_state_kernel, dim3(S * tiles, heads), dim3(SC_THREADS), smem_state, stream, p);
    int rc = gb_check_launch("gb_ssd_chunks (state)");
    if (rc) return rc;
    if (vec) gb_launch(GB_PDL_ATTENTION, ssd_chain_kernel<4>, dim3(S, heads, gb_ceil_div((long long)N * V, 1024)), dim3(256), 0, stream, p);
    else gb_launch(GB_PDL_ATTENTION, ssd_chain_kernel<1>, dim3(S, heads, gb_ceil_div((long long)N * V, 256)), dim3(256), 0, stream, p);
    rc = gb_check_launch("gb_ssd_chunks (chain)");
    if (rc) return rc;
    gb_launch(GB_PDL_ATTENTION, ssd_chunk_out_kernel, dim3(S * tiles, heads), dim3(SC_OUT_THREADS), smem_out, stream, p);
    return gb_check_launch("gb_ssd_chunks (out)");
}
