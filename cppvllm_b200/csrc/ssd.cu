// State-space recurrence with one decay per head and token (the dual of masked linear attention): a matrix S [N, P] per request
// and head, N the state size, P the value size,
//
//   [x | B | C] = silu(causal convolution of the projection's columns + bias)      x [H P], B and C [G N]; head h uses group h / (H / G)
//   dt = ln(1 + e^(z + dt_bias_h));   a = -e^(A_log_h) dt;   S <- e^a S + dt B x^T;   y = S^T C + D_h x
//
// A request's state row holds S [H, N, P] (float) and behind it, for K > 1 taps, a ring of the last K raw inputs of the convolution
// [K, H P + 2 G N]: the input at position q lies in row q mod K.  A ring of K rows (one more than the convolution looks back) lets
// the kernel for decoded tokens write its input while other blocks still read the others; inputs before position 0 are zeros by
// their position.
//
//   ssd_prep    : x, B, C, dt and a of every token.  By vectors where the channels allow it: a thread owns eight channels over four
//                 tokens and asks for all their rows together.
//   ssd_ring    : the last K - 1 raw inputs of every portion into the ring (behind ssd_prep, which reads the older ones).
//   ssd_scan    : portions in chunks of 64 tokens on the tensor cores (bf16 x, B, C; `mma.sync.m16n8k16`, float accumulation).  With
//                 l the running sum of a inside a chunk (never positive differences, so nothing overflows) and S0 the state in front:
//                   y_t = e^(l_t) S0^T C_t + sum_(s <= t) (C_t . B_s) e^(l_t - l_s) dt_s x_s + D x_t
//                   S   = e^(l_last) S0 + sum_s B_s (e^(l_last - l_s) dt_s x_s)^T
//                 The float factors (weights of the sums and S0) are split into two bf16 addends, so 16 bits of their significand
//                 reach the products; B, C and x are operands as they are.
//                   pass 1: per (chunk but the last, head, 64 columns): what the chunk adds to a state from zero; e^(l_last)
//                   pass 2: the states in front of the chunks, element by element
//                   pass 3: per (chunk, head, 64 columns): the outputs from the true state; a request's last chunk leaves the new state
//                 Where no request has more than one chunk only pass 3 runs.
//   ssd_step    : a step of decoded tokens (one per request) in one kernel, a block per (request, head): convolutions, ring, dt, the
//                 rule on S, y.
//   ssd_norm    : out = T( u / sqrt(mean(u^2) + eps) * w ), u = y silu(z), over equal parts of the row; a weight per element of the row.
#include "common.cuh"
#include "sm100.cuh"
#include "mma_tiles.cuh"

namespace cvb {

struct SsdShape {
    int H, G, N, P, C, taps;            // C = H P + 2 G N channels of the convolution
    int stride, u_off, dt_off;          // elements per row of the packed projection; columns where x | B | C and where dt begin
    int64_t state_floats;               // per slot
    int num_slots;
};

__device__ __forceinline__ float ssd_silu(float z) { return z / (1.f + expf(-z)); }
// with bf16 activations through the hardware's exponential and division
template <typename T> __device__ __forceinline__ float ssd_silu_of(float z) {
    if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
    else return ssd_silu(z);
}
__device__ __forceinline__ float ssd_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

constexpr int kSsdThreads = 128;
constexpr int kPrepRun = 4;                              // tokens per thread of the vector form

// The convolution of channel c for the token at packed row t: `local` tokens of its portion lie before it, it sits at position pos.
template <typename T>
__device__ __forceinline__ float ssd_conv_of(const T* __restrict__ packed, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                                             const float* __restrict__ ring, const SsdShape& sh, int64_t t, int local, int pos, int c) {
    float acc = conv_b[c];
    for (int m = 0; m < sh.taps; ++m) {
        const int back = sh.taps - 1 - m;
        float x = 0.f;
        if (local >= back) x = to_float(packed[(t - back) * sh.stride + sh.u_off + c]);
        else if (pos >= back) x = ring[static_cast<int64_t>((pos - back) % sh.taps) * sh.C + c];
        acc = fmaf(conv_w[static_cast<int64_t>(m) * sh.C + c], x, acc);
    }
    return acc;
}

// dt and the logarithm of the decay
template <typename T>
__device__ __forceinline__ float ssd_dt(const T* __restrict__ packed, const float* __restrict__ dt_bias, const SsdShape& sh, int64_t t, int h) {
    return ssd_softplus(to_float(packed[t * sh.stride + sh.dt_off + h]) + dt_bias[h]);
}

template <typename T, typename U>
__global__ void __launch_bounds__(kSsdThreads)
ssd_prep_kernel(U* __restrict__ u, float* __restrict__ dt, float* __restrict__ la, const T* __restrict__ packed, const float* __restrict__ conv_w,
                const float* __restrict__ conv_b, const float* __restrict__ dt_bias, const float* __restrict__ neg_a,
                const float* __restrict__ state, const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens,
                const int* __restrict__ state_slots, const int* __restrict__ positions, SsdShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int64_t t = blockIdx.x;
    if (blockIdx.y == 0) {
        for (int h = threadIdx.x; h < sh.H; h += kSsdThreads) {
            const float d = ssd_dt(packed, dt_bias, sh, t, h);
            dt[t * sh.H + h] = d;
            la[t * sh.H + h] = neg_a[h] * d;
        }
    }
    const int s = seq_of_token[t];
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    const int local = static_cast<int>(t) - cu_seqlens[s], pos = positions[t];
    const float* ring = state + static_cast<int64_t>(slot) * sh.state_floats + static_cast<int64_t>(sh.H) * sh.N * sh.P;
    for (int c = blockIdx.y * kSsdThreads + threadIdx.x; c < sh.C; c += gridDim.y * kSsdThreads)
        u[t * sh.C + c] = from_float<U>(ssd_silu_of<U>(ssd_conv_of(packed, conv_w, conv_b, ring, sh, t, local, pos, c)));
}

// eight elements of a row as they lie in memory
template <typename T> struct Row8;
template <> struct Row8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = *reinterpret_cast<const float4*>(p); b = *reinterpret_cast<const float4*>(p + 4); }
    __device__ __forceinline__ void get(float (&f)[8]) const { f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w; }
};
template <> struct Row8<__nv_bfloat16> {
    uint4 r;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { r = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void get(float (&f)[8]) const {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
    }
};

template <typename T, typename U, int K>
__global__ void __launch_bounds__(kSsdThreads)
ssd_prep_vec_kernel(U* __restrict__ u, float* __restrict__ dt, float* __restrict__ la, const T* __restrict__ packed, const float* __restrict__ conv_w,
                    const float* __restrict__ conv_b, const float* __restrict__ dt_bias, const float* __restrict__ neg_a,
                    const float* __restrict__ state, const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens,
                    const int* __restrict__ state_slots, const int* __restrict__ positions, int n_tokens, SsdShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.x * kPrepRun, t1 = min(t0 + kPrepRun, n_tokens);
    if (blockIdx.y == gridDim.y - 1) {                    // the last row of blocks: dt and the decays
        for (int i = threadIdx.x; i < (t1 - t0) * sh.H; i += kSsdThreads) {
            const int64_t t = t0 + i / sh.H;
            const int h = i % sh.H;
            const float d = ssd_dt(packed, dt_bias, sh, t, h);
            dt[t * sh.H + h] = d;
            la[t * sh.H + h] = neg_a[h] * d;
        }
        return;
    }
    const int c = (blockIdx.y * kSsdThreads + threadIdx.x) * 8;
    if (c >= sh.C) return;
    const T* base = packed + sh.u_off + c;
    Row8<T> x[K - 1 + kPrepRun];                          // rows t0 - K + 1 .. t1 - 1, asked for together
#pragma unroll
    for (int i = 0; i < K - 1 + kPrepRun; ++i) x[i].load(base + static_cast<int64_t>(min(max(t0 - K + 1 + i, 0), t1 - 1)) * sh.stride);
    int seq[kPrepRun], first[kPrepRun];
#pragma unroll
    for (int i = 0; i < kPrepRun; ++i) seq[i] = seq_of_token[min(t0 + i, t1 - 1)];
#pragma unroll
    for (int i = 0; i < kPrepRun; ++i) first[i] = cu_seqlens[seq[i]];
    float w[K][8], b[8];
    load8(b, conv_b + c);
#pragma unroll
    for (int m = 0; m < K; ++m) load8(w[m], conv_w + static_cast<int64_t>(m) * sh.C + c);
#pragma unroll
    for (int i = 0; i < kPrepRun; ++i) {
        const int t = t0 + i, local = t - first[i];
        if (t >= t1) break;
        float y[8];
        if (local >= K - 1) {
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = b[e];
#pragma unroll
            for (int m = 0; m < K; ++m) {
                float v[8];
                x[i + m].get(v);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[e] = fmaf(w[m][e], v[e], y[e]);
            }
        } else {                                          // the window reaches back before the portion
            const int slot = state_slots[seq[i]];
            if (slot < 0 || slot >= sh.num_slots) {
                atomicExch(err, 2);
                continue;
            }
            const float* ring = state + static_cast<int64_t>(slot) * sh.state_floats + static_cast<int64_t>(sh.H) * sh.N * sh.P;
#pragma unroll 1
            for (int e = 0; e < 8; ++e) {
                const float v = ssd_conv_of(packed, conv_w, conv_b, ring, sh, t, local, positions[t], c + e);
#pragma unroll
                for (int k = 0; k < 8; ++k)
                    if (k == e) y[k] = v;
            }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = ssd_silu_of<U>(y[e]);
        store8(u + static_cast<int64_t>(t) * sh.C + c, y);
    }
}

template <typename T>
__global__ void __launch_bounds__(kSsdThreads)
ssd_ring_kernel(float* __restrict__ state, const T* __restrict__ packed, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                const int* __restrict__ positions, SsdShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x;
    const int begin = cu_seqlens[s], end = cu_seqlens[s + 1];
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    float* ring = state + static_cast<int64_t>(slot) * sh.state_floats + static_cast<int64_t>(sh.H) * sh.N * sh.P;
    for (int c = blockIdx.y * kSsdThreads + threadIdx.x; c < sh.C; c += gridDim.y * kSsdThreads)
        for (int t = max(begin, end - sh.taps + 1); t < end; ++t)
            ring[static_cast<int64_t>(positions[t] % sh.taps) * sh.C + c] = to_float(packed[static_cast<int64_t>(t) * sh.stride + sh.u_off + c]);
}

// ---- portions on the tensor cores ---------------------------------------------------------------------------------------

constexpr int kChunk = 64;                               // tokens per chunk
constexpr int kCols = 64;                                // columns of S per block
constexpr int kOutThreads = 256;                         // pass 3: two warps per 16 tokens, 32 columns each
constexpr int kLdX = kCols + 8;                          // padded row of a tile of columns, in elements

struct SsdChunk { int seq, k, n_chunks, buf, begin, n; };

// Block x's chunk: chunk k of the n_chunks of a request; `buf`: where the request's chunks lie in the chunk buffers, which hold
// requests with more than one chunk only.
__device__ __forceinline__ bool ssd_locate(const int* __restrict__ cu_seqlens, int S, int x, SsdChunk& c) {
    int base = 0, held = 0;
    for (int s = 0; s < S; ++s) {
        const int a = cu_seqlens[s], tokens = cu_seqlens[s + 1] - a;
        const int chunks = (tokens + kChunk - 1) / kChunk;
        if (x < base + chunks) {
            c.seq = s; c.k = x - base; c.n_chunks = chunks; c.buf = held;
            c.begin = a + c.k * kChunk;
            c.n = min(kChunk, tokens - c.k * kChunk);
            return true;
        }
        base += chunks;
        if (chunks > 1) held += chunks;
    }
    return false;
}

// Running sums of the decays' logarithms and the step sizes of a chunk; tokens past its end count as 0.
__device__ __forceinline__ void chunk_sums(float* l, float* d, const float* __restrict__ la, const float* __restrict__ dt, int begin, int n,
                                           int H, int h) {
    const int tid = threadIdx.x;
    if (tid < kChunk) {
        l[tid] = tid < n ? la[static_cast<int64_t>(begin + tid) * H + h] : 0.f;
        d[tid] = tid < n ? dt[static_cast<int64_t>(begin + tid) * H + h] : 0.f;
    }
    __syncthreads();
    if (tid < 32) {
        const float a = l[2 * tid], b = l[2 * tid + 1];
        float run = a + b;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (tid >= o) run += up;
        }
        float before = __shfl_up_sync(0xffffffffu, run, 1);
        if (tid == 0) before = 0.f;
        l[2 * tid] = before + a;
        l[2 * tid + 1] = run;
    }
    __syncthreads();
}

// `width` columns (a multiple of 8) of a chunk's rows into shared rows of ld elements; rows past the chunk are zeros.
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* dst, int ld, const __nv_bfloat16* __restrict__ src, int64_t stride, int n, int width) {
    const int per = width >> 3;
    for (int i = threadIdx.x; i < kChunk * per; i += blockDim.x) {
        const int r = i / per, c = (i - r * per) * 8;
        cp_async16(dst + r * ld + c, r < n ? src + r * stride + c : src, r < n);
    }
}

// x times e^(l_last - l_s) dt_s, in two bf16 addends
__device__ __forceinline__ void weigh_rows(__nv_bfloat16* hi, __nv_bfloat16* lo, const __nv_bfloat16* x, const float* l, const float* d, int width) {
    const float last = l[kChunk - 1];
    for (int i = threadIdx.x; i < kChunk * (width >> 1); i += blockDim.x) {
        const int r = i / (width >> 1), c = (i - r * (width >> 1)) * 2;
        const float w = expf(last - l[r]) * d[r];
        float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x + r * kLdX + c));
        v.x *= w; v.y *= w;
        const __nv_bfloat162 h = __floats2bfloat162_rn(v.x, v.y);
        const float2 hf = __bfloat1622float2(h);
        *reinterpret_cast<__nv_bfloat162*>(hi + r * kLdX + c) = h;
        *reinterpret_cast<__nv_bfloat162*>(lo + r * kLdX + c) = __floats2bfloat162_rn(v.x - hf.x, v.y - hf.y);
    }
}

// What the chunk adds to S: sum_s B_s xw_s^T; the block's warps take slabs of 16 rows of S in turn.  put(row, column, two values).
template <typename F>
__device__ __forceinline__ void chunk_state(const __nv_bfloat16* sB, int ldb, const __nv_bfloat16* hi, const __nv_bfloat16* lo, int N, int width, F put) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int m0 = warp * 16; m0 < N; m0 += static_cast<int>(blockDim.x >> 5) * 16) {
        float acc[kCols / 8][4];
#pragma unroll
        for (int i = 0; i < kCols / 8; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll
        for (int kk = 0; kk < kChunk / 16; ++kk) {
            uint32_t a[4];
            ldm_x4_trans(a, sB + (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldb + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int dp = 0; dp < kCols / 16; ++dp) {
                if (dp * 16 >= width) break;
                const int at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdX + dp * 16 + ((lane >> 4) & 1) * 8;
                uint32_t b[4];
                ldm_x4_trans(b, hi + at);
                mma_16816(acc[dp * 2], a, b[0], b[1]);
                mma_16816(acc[dp * 2 + 1], a, b[2], b[3]);
                ldm_x4_trans(b, lo + at);
                mma_16816(acc[dp * 2], a, b[0], b[1]);
                mma_16816(acc[dp * 2 + 1], a, b[2], b[3]);
            }
        }
        const int r = m0 + (lane >> 2), c = (lane & 3) << 1;
#pragma unroll
        for (int i = 0; i < kCols / 8; ++i) {
            if (i * 8 >= width) break;
            put(r, i * 8 + c, make_float2(acc[i][0], acc[i][1]));
            put(r + 8, i * 8 + c, make_float2(acc[i][2], acc[i][3]));
        }
    }
}

// Pass 1.  ends[buf + k + 1] receives chunk k's addition (k < n_chunks - 1), decays[buf + k] its e^(l_last).
__global__ void __launch_bounds__(kSsdThreads)
ssd_chunk_kernel(const __nv_bfloat16* __restrict__ u, const float* __restrict__ dt, const float* __restrict__ la, float* __restrict__ ends,
                 float* __restrict__ decays, const int* __restrict__ cu_seqlens, int S, SsdShape sh) {
    pdl_trigger();
    pdl_wait();
    SsdChunk ck;
    if (!ssd_locate(cu_seqlens, S, blockIdx.x, ck) || ck.k == ck.n_chunks - 1) return;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float l[kChunk], d[kChunk];
    const int h = blockIdx.y, p0 = blockIdx.z * kCols, width = min(kCols, sh.P - p0);
    const int g = h / (sh.H / sh.G), ldb = sh.N + 8;
    __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* sX = sB + kChunk * ldb;
    __nv_bfloat16* hi = sX + kChunk * kLdX;
    __nv_bfloat16* lo = hi + kChunk * kLdX;
    const __nv_bfloat16* row = u + static_cast<int64_t>(ck.begin) * sh.C;
    fetch_rows(sX, kLdX, row + h * sh.P + p0, sh.C, ck.n, width);
    cp_async_commit();
    fetch_rows(sB, ldb, row + sh.H * sh.P + g * sh.N, sh.C, ck.n, sh.N);
    cp_async_commit();
    chunk_sums(l, d, la, dt, ck.begin, ck.n, sh.H, h);
    cp_async_wait<1>();
    __syncthreads();
    weigh_rows(hi, lo, sX, l, d, width);
    cp_async_wait<0>();
    __syncthreads();
    float* dst = ends + (static_cast<int64_t>(ck.buf + ck.k + 1) * sh.H + h) * sh.N * sh.P + p0;
    chunk_state(sB, ldb, hi, lo, sh.N, width, [&](int r, int c, float2 v) { *reinterpret_cast<float2*>(dst + static_cast<int64_t>(r) * sh.P + c) = v; });
    if (threadIdx.x == 0 && blockIdx.z == 0) decays[static_cast<int64_t>(ck.buf + ck.k) * sh.H + h] = expf(l[kChunk - 1]);
}

// Pass 2: ends[buf + k] becomes the state in front of chunk k of every request with more than one chunk.  Grid: (request, head, parts).
__global__ void __launch_bounds__(256)
ssd_carry_kernel(float* __restrict__ ends, const float* __restrict__ decays, const float* __restrict__ state, const int* __restrict__ cu_seqlens,
                 const int* __restrict__ state_slots, int S, SsdShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y;
    int buf = 0;
    for (int q = 0; q < s; ++q) {
        const int chunks = (cu_seqlens[q + 1] - cu_seqlens[q] + kChunk - 1) / kChunk;
        if (chunks > 1) buf += chunks;
    }
    const int nc = (cu_seqlens[s + 1] - cu_seqlens[s] + kChunk - 1) / kChunk;
    if (nc < 2) return;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    const int64_t mat = static_cast<int64_t>(sh.N) * sh.P, step = sh.H * mat;
    const float* from = state + static_cast<int64_t>(slot) * sh.state_floats + h * mat;
    float* e0 = ends + (static_cast<int64_t>(buf) * sh.H + h) * mat;
    const float* d0 = decays + static_cast<int64_t>(buf) * sh.H + h;
    for (int64_t i = (static_cast<int64_t>(blockIdx.z) * 256 + threadIdx.x) * 4; i < mat; i += static_cast<int64_t>(gridDim.z) * 1024) {
        float4 run = *reinterpret_cast<const float4*>(from + i);
        *reinterpret_cast<float4*>(e0 + i) = run;
#pragma unroll 8
        for (int k = 1; k < nc; ++k) {
            float4* e = reinterpret_cast<float4*>(e0 + k * step + i);
            const float a = d0[static_cast<int64_t>(k - 1) * sh.H];
            const float4 v = *e;
            run = make_float4(fmaf(a, run.x, v.x), fmaf(a, run.y, v.y), fmaf(a, run.z, v.z), fmaf(a, run.w, v.w));
            *e = run;
        }
    }
}

// Pass 3.  A warp owns 16 tokens of the chunk and half the block's columns; both warps of a pair make the 16 tokens' C . B.
__global__ void __launch_bounds__(kOutThreads)
ssd_out_kernel(float* __restrict__ y, const __nv_bfloat16* __restrict__ u, const float* __restrict__ dt, const float* __restrict__ la,
               const float* __restrict__ D, const float* __restrict__ ends, float* __restrict__ state, const int* __restrict__ cu_seqlens,
               const int* __restrict__ state_slots, int S, SsdShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    SsdChunk ck;
    if (!ssd_locate(cu_seqlens, S, blockIdx.x, ck)) return;
    const int slot = state_slots[ck.seq];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float l[kChunk], d[kChunk];
    const int h = blockIdx.y, p0 = blockIdx.z * kCols, width = min(kCols, sh.P - p0);
    const int g = h / (sh.H / sh.G), N = sh.N, ldb = N + 8;
    const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, col0 = (threadIdx.x >> 7) * (kCols / 2);
    const int s_rows = N > kChunk ? N : kChunk;           // the room of S0 also takes the chunk's weighted rows
    __nv_bfloat16* sC = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* sB = sC + kChunk * ldb;
    __nv_bfloat16* sX = sB + kChunk * ldb;
    __nv_bfloat16* hi = sX + kChunk * kLdX;
    __nv_bfloat16* lo = hi + s_rows * kLdX;
    const __nv_bfloat16* row = u + static_cast<int64_t>(ck.begin) * sh.C;
    fetch_rows(sC, ldb, row + sh.H * sh.P + (sh.G + g) * N, sh.C, ck.n, N);
    fetch_rows(sB, ldb, row + sh.H * sh.P + g * N, sh.C, ck.n, N);
    fetch_rows(sX, kLdX, row + h * sh.P + p0, sh.C, ck.n, width);
    cp_async_commit();
    const int64_t mat = static_cast<int64_t>(N) * sh.P;
    float* st = state + static_cast<int64_t>(slot) * sh.state_floats + h * mat + p0;
    const float* from = ck.n_chunks > 1 ? ends + (static_cast<int64_t>(ck.buf + ck.k) * sh.H + h) * mat + p0 : st;
    const int quads = width >> 2;
    for (int i = threadIdx.x; i < N * quads; i += kOutThreads) {
        const int r = i / quads, c = (i - r * quads) * 4;
        const float4 v = *reinterpret_cast<const float4*>(from + static_cast<int64_t>(r) * sh.P + c);
        const __nv_bfloat162 h0 = __floats2bfloat162_rn(v.x, v.y), h1 = __floats2bfloat162_rn(v.z, v.w);
        const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
        __nv_bfloat162* ph = reinterpret_cast<__nv_bfloat162*>(hi + r * kLdX + c);
        __nv_bfloat162* pl = reinterpret_cast<__nv_bfloat162*>(lo + r * kLdX + c);
        ph[0] = h0; ph[1] = h1;
        pl[0] = __floats2bfloat162_rn(v.x - f0.x, v.y - f0.y);
        pl[1] = __floats2bfloat162_rn(v.z - f1.x, v.w - f1.y);
    }
    chunk_sums(l, d, la, dt, ck.begin, ck.n, sh.H, h);
    cp_async_wait<0>();
    __syncthreads();

    const int r0 = warp * 16 + (lane >> 2), r1 = r0 + 8;  // the two tokens whose rows this thread holds
    float o[kCols / 16][4];
#pragma unroll
    for (int i = 0; i < kCols / 16; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    float m[kChunk / 8][4];
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i) { m[i][0] = m[i][1] = m[i][2] = m[i][3] = 0.f; }
    if (warp * 16 < ck.n && col0 < width) {
        for (int ks = 0; ks < N / 16; ++ks) {
            uint32_t a[4];
            ldm_x4(a, sC + (warp * 16 + (lane & 15)) * ldb + ks * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int dp = 0; dp < kCols / 32; ++dp) {     // S0^T C
                if (col0 + dp * 16 >= width) break;
                const int at = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdX + col0 + dp * 16 + ((lane >> 4) & 1) * 8;
                uint32_t b[4];
                ldm_x4_trans(b, hi + at);
                mma_16816(o[dp * 2], a, b[0], b[1]);
                mma_16816(o[dp * 2 + 1], a, b[2], b[3]);
                ldm_x4_trans(b, lo + at);
                mma_16816(o[dp * 2], a, b[0], b[1]);
                mma_16816(o[dp * 2 + 1], a, b[2], b[3]);
            }
#pragma unroll
            for (int np = 0; np < kChunk / 16; ++np) {    // C . B of the tokens up to the warp's own
                if (np > warp) break;
                uint32_t b[4];
                ldm_x4(b, sB + (np * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldb + ks * 16 + ((lane >> 3) & 1) * 8);
                mma_16816(m[np * 2], a, b[0], b[1]);
                mma_16816(m[np * 2 + 1], a, b[2], b[3]);
            }
        }
        const float l0 = l[r0], l1 = l[r1], e0 = expf(l0), e1 = expf(l1);
#pragma unroll
        for (int i = 0; i < kCols / 16; ++i) { o[i][0] *= e0; o[i][1] *= e0; o[i][2] *= e1; o[i][3] *= e1; }
#pragma unroll
        for (int nt = 0; nt < kChunk / 8; ++nt) {
            if (nt > warp * 2 + 1) break;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int s = nt * 8 + ((lane & 3) << 1) + (e & 1), t = e < 2 ? r0 : r1;
                m[nt][e] = s <= t ? m[nt][e] * expf((e < 2 ? l0 : l1) - l[s]) * d[s] : 0.f;
            }
        }
#pragma unroll
        for (int kk = 0; kk < kChunk / 16; ++kk) {
            if (kk > warp) break;
            uint32_t ah[4], al[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float v0 = m[kk * 2 + (q >> 1)][(q & 1) * 2], v1 = m[kk * 2 + (q >> 1)][(q & 1) * 2 + 1];
                const __nv_bfloat162 b2 = __floats2bfloat162_rn(v0, v1);
                const float2 f = __bfloat1622float2(b2);
                ah[q] = *reinterpret_cast<const uint32_t*>(&b2);
                al[q] = pack2(v0 - f.x, v1 - f.y);
            }
#pragma unroll
            for (int dp = 0; dp < kCols / 32; ++dp) {
                if (col0 + dp * 16 >= width) break;
                uint32_t b[4];
                ldm_x4_trans(b, sX + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdX + col0 + dp * 16 + ((lane >> 4) & 1) * 8);
                mma_16816(o[dp * 2], ah, b[0], b[1]);
                mma_16816(o[dp * 2 + 1], ah, b[2], b[3]);
                mma_16816(o[dp * 2], al, b[0], b[1]);
                mma_16816(o[dp * 2 + 1], al, b[2], b[3]);
            }
        }
        const float skip = D[h];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = half ? r1 : r0;
            if (r >= ck.n) continue;
            float* dst = y + (static_cast<int64_t>(ck.begin + r) * sh.H + h) * sh.P + p0;
#pragma unroll
            for (int i = 0; i < kCols / 16; ++i) {
                if (col0 + i * 8 >= width) break;
                const int c = col0 + i * 8 + ((lane & 3) << 1);
                const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + r * kLdX + c));
                *reinterpret_cast<float2*>(dst + c) = make_float2(fmaf(skip, x.x, o[i][half * 2]), fmaf(skip, x.y, o[i][half * 2 + 1]));
            }
        }
    }
    if (ck.k != ck.n_chunks - 1) return;                  // the whole block: the request's last chunk leaves the new state
    __syncthreads();
    weigh_rows(hi, lo, sX, l, d, width);
    __syncthreads();
    const float keep = expf(l[kChunk - 1]);
    chunk_state(sB, ldb, hi, lo, N, width, [&](int r, int c, float2 v) {
        const float2 s0 = *reinterpret_cast<const float2*>(from + static_cast<int64_t>(r) * sh.P + c);
        *reinterpret_cast<float2*>(st + static_cast<int64_t>(r) * sh.P + c) = make_float2(fmaf(keep, s0.x, v.x), fmaf(keep, s0.y, v.y));
    });
}

// ---- decoded tokens: one token per request -------------------------------------------------------------------------------
//
// The block's threads are laid out as rows of S by groups of V neighbouring columns (V = 4 where the value size allows 16-byte
// accesses): a thread updates its columns of every R-th row, adds its part of S^T C up in registers, and the R partial sums of a
// column meet in shared memory in a fixed order.
constexpr int kStepThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads)
ssd_step_kernel(float* __restrict__ y, const T* __restrict__ packed, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                const float* __restrict__ dt_bias, const float* __restrict__ neg_a, const float* __restrict__ D, float* __restrict__ state,
                const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, const int* __restrict__ positions, SsdShape sh,
                int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float smf[];
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int N = sh.N, P = sh.P, HP = sh.H * P, per = sh.H / sh.G, g = h / per;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (tid == 0) atomicExch(err, 2);
        return;
    }
    float* xs = smf;                                      // [P]
    float* bs = xs + P;                                   // [N]
    float* cs = bs + N;                                   // [N]
    float* part = cs + N;                                 // [R, P]
    const int nvec = (P + V - 1) / V;
    const bool narrow = nvec < kStepThreads;
    const int R = narrow ? kStepThreads / nvec : 1;       // rows worked on side by side
    const int64_t t = cu_seqlens[s];
    const int pos = positions[t];
    float* row = state + static_cast<int64_t>(slot) * sh.state_floats;
    float* ring = row + static_cast<int64_t>(sh.H) * N * P;
    const bool first_of_group = h % per == 0;             // writes the group's B and C into the ring
    float* st = row + static_cast<int64_t>(h) * N * P;
    const int rg = narrow ? tid / nvec : 0;
    // the thread's first rows of S are on their way before the convolutions
    constexpr int kAhead = V == 4 ? 8 : 1;
    float4 ahead[kAhead];
    if constexpr (V == 4) {
        if (narrow && rg < R) {
#pragma unroll
            for (int k = 0; k < kAhead; ++k)
                if (rg + k * R < N) ahead[k] = *reinterpret_cast<const float4*>(st + static_cast<int64_t>(rg + k * R) * P + (tid - rg * nvec) * 4);
        }
    }
    for (int c = tid; c < P + 2 * N; c += kStepThreads) {
        const int ch = c < P ? h * P + c : (c < P + N ? HP + g * N + c - P : HP + (sh.G + g) * N + c - P - N);
        smf[c] = ssd_silu(ssd_conv_of(packed, conv_w, conv_b, ring, sh, t, 0, pos, ch));
        if (sh.taps > 1 && (c < P || first_of_group))
            ring[static_cast<int64_t>(pos % sh.taps) * sh.C + ch] = to_float(packed[t * sh.stride + sh.u_off + ch]);
    }
    const float dt = ssd_dt(packed, dt_bias, sh, t, h), a = expf(neg_a[h] * dt), skip = D[h];
    __syncthreads();
    for (int cv = narrow ? tid - rg * nvec : tid; cv < nvec; cv += (narrow ? nvec : kStepThreads)) {
        if (rg >= R) break;
        float v[V], o[V];
#pragma unroll
        for (int j = 0; j < V; ++j) { v[j] = dt * xs[cv * V + j]; o[j] = 0.f; }
        int i = rg;
        if constexpr (V == 4) {
            if (narrow) {
#pragma unroll
                for (int k = 0; k < kAhead; ++k, i += R) {
                    if (i >= N) break;
                    const float b = bs[i], q = cs[i];
                    float4 x = ahead[k];
                    x.x = fmaf(a, x.x, b * v[0]); x.y = fmaf(a, x.y, b * v[1]); x.z = fmaf(a, x.z, b * v[2]); x.w = fmaf(a, x.w, b * v[3]);
                    o[0] = fmaf(q, x.x, o[0]); o[1] = fmaf(q, x.y, o[1]); o[2] = fmaf(q, x.z, o[2]); o[3] = fmaf(q, x.w, o[3]);
                    *reinterpret_cast<float4*>(st + static_cast<int64_t>(i) * P + cv * V) = x;
                }
            }
        }
#pragma unroll 8
        for (; i < N; i += R) {
            float* p = st + static_cast<int64_t>(i) * P + cv * V;
            const float k = bs[i], q = cs[i];
            if constexpr (V == 4) {
                float4 x = *reinterpret_cast<const float4*>(p);
                x.x = fmaf(a, x.x, k * v[0]); x.y = fmaf(a, x.y, k * v[1]); x.z = fmaf(a, x.z, k * v[2]); x.w = fmaf(a, x.w, k * v[3]);
                o[0] = fmaf(q, x.x, o[0]); o[1] = fmaf(q, x.y, o[1]); o[2] = fmaf(q, x.z, o[2]); o[3] = fmaf(q, x.w, o[3]);
                *reinterpret_cast<float4*>(p) = x;
            } else {
                const float x = fmaf(a, p[0], k * v[0]);
                o[0] = fmaf(q, x, o[0]);
                p[0] = x;
            }
        }
#pragma unroll
        for (int j = 0; j < V; ++j) part[rg * P + cv * V + j] = o[j];
    }
    __syncthreads();
    for (int j = tid; j < P; j += kStepThreads) {
        float o = 0.f;
        for (int r = 0; r < R; ++r) o += part[r * P + j];
        y[t * HP + h * P + j] = fmaf(skip, xs[j], o);
    }
}

// ---- the gate and the norm behind it ---------------------------------------------------------------------------------------

constexpr int kNormQuads = 8;                            // four-element pieces a thread keeps in registers

// A block (up to 512 elements: a warp, four to a block) per (token, part); rows in pieces of four that start on 16 bytes (8 bytes of bf16
// rows) stay in registers.
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS < 128 ? 128 : THREADS)
ssd_norm_vec_kernel(T* __restrict__ out, int out_stride, const float* __restrict__ y, const T* __restrict__ z, int z_stride, const float* __restrict__ w,
                    int64_t rows, int parts, int n, float eps, float scale) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[32];
    constexpr int kPer = THREADS < 128 ? 128 / THREADS : 1, kQuads = THREADS < 128 ? 4 : kNormQuads;
    const int64_t row = static_cast<int64_t>(blockIdx.x) * kPer + threadIdx.x / THREADS;
    if (row >= rows) return;
    const int64_t t = row / parts;
    const int c0 = static_cast<int>(row - t * parts) * n, lane = threadIdx.x % THREADS;
    const float* yr = y + t * parts * n + c0;
    const T* zr = z + t * z_stride + c0;
    float4 v[kQuads];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kQuads; ++k) {
        const int j = (lane + k * THREADS) * 4;
        if (j < n) {
            v[k] = *reinterpret_cast<const float4*>(yr + j);
            float g[4];
            if constexpr (sizeof(T) == 2) {
                const uint2 raw = *reinterpret_cast<const uint2*>(zr + j);
                const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                g[0] = a.x; g[1] = a.y; g[2] = b.x; g[3] = b.y;
            } else {
                const float4 a = *reinterpret_cast<const float4*>(zr + j);
                g[0] = a.x; g[1] = a.y; g[2] = a.z; g[3] = a.w;
            }
            v[k].x *= ssd_silu_of<T>(g[0]); v[k].y *= ssd_silu_of<T>(g[1]); v[k].z *= ssd_silu_of<T>(g[2]); v[k].w *= ssd_silu_of<T>(g[3]);
            ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
        }
    }
    ss = THREADS > 32 ? block_sum(ss, scratch) : warp_sum(ss);
    const float inv = scale / sqrtf(ss / static_cast<float>(n) + eps);
    T* dst = out + t * out_stride + c0;
#pragma unroll
    for (int k = 0; k < kQuads; ++k) {
        const int j = (lane + k * THREADS) * 4;
        if (j < n) {
            const float4 ww = *reinterpret_cast<const float4*>(w + c0 + j);
            const float r[4] = {v[k].x * inv * ww.x, v[k].y * inv * ww.y, v[k].z * inv * ww.z, v[k].w * inv * ww.w};
            if constexpr (sizeof(T) == 2) {
                uint2 raw;
                *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(r[0], r[1]);
                *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(r[2], r[3]);
                *reinterpret_cast<uint2*>(dst + j) = raw;
            } else {
                *reinterpret_cast<float4*>(dst + j) = make_float4(r[0], r[1], r[2], r[3]);
            }
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(kSsdThreads)
ssd_norm_kernel(T* __restrict__ out, int out_stride, const float* __restrict__ y, const T* __restrict__ z, int z_stride, const float* __restrict__ w,
                int parts, int n, float eps, float scale) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[32];
    const int64_t t = blockIdx.x;
    const int c0 = blockIdx.y * n;
    const float* yr = y + t * parts * n + c0;
    const T* zr = z + t * z_stride + c0;
    float ss = 0.f;
    for (int j = threadIdx.x; j < n; j += kSsdThreads) {
        const float v = yr[j] * ssd_silu_of<T>(to_float(zr[j]));
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = scale / sqrtf(ss / static_cast<float>(n) + eps);
    for (int j = threadIdx.x; j < n; j += kSsdThreads)
        out[t * out_stride + c0 + j] = from_float<T>(yr[j] * ssd_silu_of<T>(to_float(zr[j])) * inv * w[c0 + j]);
}

static bool ssd_al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

static int ssd_shape(SsdShape& sh, int H, int G, int N, int P, int taps, int stride, int u_off, int dt_off, int64_t state_floats, int num_slots) {
    if (H <= 0 || H > 65535 || G <= 0 || N <= 0 || P <= 0 || taps <= 0 || num_slots <= 0) return CVB_E_SIZE;
    const int64_t C = static_cast<int64_t>(H) * P + 2LL * G * N;
    if (H % G || C > (1 << 30)) return CVB_E_SHAPE;
    if (state_floats < static_cast<int64_t>(H) * N * P + (taps > 1 ? taps * C : 0)) return CVB_E_SHAPE;
    if (u_off < 0 || dt_off < 0 || stride < u_off + C || stride < dt_off + H) return CVB_E_SHAPE;
    sh = SsdShape{H, G, N, P, static_cast<int>(C), taps, stride, u_off, dt_off, state_floats, num_slots};
    return CVB_OK;
}

}  // namespace cvb

using namespace cvb;

// `u_dtype`: element type of u (float, or the packed rows' bf16).
extern "C" int cvb_ssd_prep(void* u, float* dt, float* la, const void* packed, int T, int stride, int u_off, int dt_off, const float* conv_w,
                            const float* conv_b, int taps, const float* dt_bias, const float* neg_a, const float* state, int64_t state_floats,
                            const int* seq_of_token, const int* cu_seqlens, const int* state_slots, const int* positions, int num_slots, int H,
                            int G, int N, int P, int dtype, int u_dtype, int* err_flag, cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    if (T < 0) return CVB_E_SIZE;
    SsdShape sh;
    const int rc = ssd_shape(sh, H, G, N, P, taps, stride, u_off, dt_off, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    const bool vec = sh.C % 8 == 0 && u_off % 8 == 0 && stride % 8 == 0 && taps >= 2 && taps <= 4 && ssd_al16(u) && ssd_al16(packed)
                     && ssd_al16(conv_w) && ssd_al16(conv_b);
    const dim3 vgrid((T + kPrepRun - 1) / kPrepRun, (sh.C / 8 + kSsdThreads - 1) / kSsdThreads + 1);
    const int per = (sh.C + kSsdThreads - 1) / kSsdThreads;
    const dim3 grid(T, per < 64 ? per : 64);
#define CALL_K(TY, UY, KK) launch_kernel(ssd_prep_vec_kernel<TY, UY, KK>, vgrid, dim3(kSsdThreads), 0, stream, (UY*)u, dt, la, (const TY*)packed, conv_w, \
                                         conv_b, dt_bias, neg_a, state, seq_of_token, cu_seqlens, state_slots, positions, T, sh, err_flag)
#define CALL_U(TY, UY)                                                                                                           \
    do {                                                                                                                         \
        if (vec && taps == 2) CALL_K(TY, UY, 2);                                                                                 \
        else if (vec && taps == 3) CALL_K(TY, UY, 3);                                                                            \
        else if (vec) CALL_K(TY, UY, 4);                                                                                         \
        else launch_kernel(ssd_prep_kernel<TY, UY>, grid, dim3(kSsdThreads), 0, stream, (UY*)u, dt, la, (const TY*)packed, conv_w, conv_b,  \
                           dt_bias, neg_a, state, seq_of_token, cu_seqlens, state_slots, positions, sh, err_flag);               \
    } while (0)
    if (dtype == CVB_DTYPE_F32 && u_dtype == CVB_DTYPE_F32) CALL_U(float, float);
    else if (dtype == CVB_DTYPE_BF16 && u_dtype == CVB_DTYPE_F32) CALL_U(__nv_bfloat16, float);
    else if (dtype == CVB_DTYPE_BF16 && u_dtype == CVB_DTYPE_BF16) CALL_U(__nv_bfloat16, __nv_bfloat16);
    else return CVB_E_DTYPE;
#undef CALL_U
#undef CALL_K
    return launch_status();
}

extern "C" int cvb_ssd_ring(float* state, int64_t state_floats, const void* packed, int stride, int u_off, int dt_off, int taps,
                            const int* cu_seqlens, const int* state_slots, const int* positions, int num_slots, int S, int H, int G, int N,
                            int P, int dtype, int* err_flag, cudaStream_t stream) {
    if (S == 0 || taps <= 1) return CVB_OK;
    if (S < 0) return CVB_E_SIZE;
    SsdShape sh;
    const int rc = ssd_shape(sh, H, G, N, P, taps, stride, u_off, dt_off, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    const int per = (sh.C + kSsdThreads - 1) / kSsdThreads;
#define CALL(TY) launch_kernel(ssd_ring_kernel<TY>, dim3(S, per < 65535 ? per : 65535), dim3(kSsdThreads), 0, stream, state, (const TY*)packed, cu_seqlens, \
                               state_slots, positions, sh, err_flag)
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
    return launch_status();
}

static size_t ssd_out_smem(int N) {
    return (static_cast<size_t>(2) * kChunk * (N + 8) + static_cast<size_t>(kChunk) * kLdX + static_cast<size_t>(2) * (N > kChunk ? N : kChunk) * kLdX)
           * sizeof(__nv_bfloat16);
}

// `chunks`: how many chunks of 64 tokens the step's requests have together; `held`: how many of them belong to requests with more than
// one (0: pass 3 alone runs); `ends` holds H N P floats and `decays` H floats per held chunk.  u: bf16 rows [x | B | C].
extern "C" int cvb_ssd_chunks(float* y, const void* u, const float* dt, const float* la, const float* D, float* ends, int64_t ends_floats,
                              float* decays, int64_t decays_floats, float* state, int64_t state_floats, int num_slots, const int* cu_seqlens,
                              const int* state_slots, int S, int chunks, int held, int H, int G, int N, int P, int* err_flag,
                              cudaStream_t stream) {
    if (S == 0) return CVB_OK;
    const int64_t C = static_cast<int64_t>(H) * P + 2LL * G * N;
    SsdShape sh;
    const int rc = ssd_shape(sh, H, G, N, P, 1, static_cast<int>(C) + H, 0, static_cast<int>(C), state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    if (S < 0 || chunks <= 0 || held < 0) return CVB_E_SIZE;
    if (N % 16 || P % 16 || N > 256) return CVB_E_UNSUPPORTED;
    if (!ssd_al16(u) || !ssd_al16(y) || !ssd_al16(state) || state_floats % 4 || (held > 0 && !ssd_al16(ends))) return CVB_E_ALIGN;
    const int64_t mat = static_cast<int64_t>(N) * P;
    if (held > 0 && (ends == nullptr || decays == nullptr || ends_floats < held * H * mat || decays_floats < static_cast<int64_t>(held) * H)) return CVB_E_SCRATCH;
    const int slices = (P + kCols - 1) / kCols;
    const size_t smem1 = (static_cast<size_t>(kChunk) * (N + 8) + static_cast<size_t>(3) * kChunk * kLdX) * sizeof(__nv_bfloat16);
    const size_t smem3 = ssd_out_smem(N);
    static bool raised = false;
    if (!raised) {
        if (cudaFuncSetAttribute(ssd_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024) != cudaSuccess
            || cudaFuncSetAttribute(ssd_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(ssd_out_smem(256))) != cudaSuccess)
            return launch_status();
        raised = true;
    }
    if (held > 0) {
        launch_kernel(ssd_chunk_kernel, dim3(chunks, H, slices), dim3(kSsdThreads), smem1, stream, (const __nv_bfloat16*)u, dt, la, ends, decays,
                      cu_seqlens, S, sh);
        const int64_t zs = (mat / 4 + 255) / 256;
        launch_kernel(ssd_carry_kernel, dim3(S, H, static_cast<unsigned>(zs < 64 ? zs : 64)), dim3(256), 0, stream, ends, decays, state, cu_seqlens,
                      state_slots, S, sh, err_flag);
    }
    launch_kernel(ssd_out_kernel, dim3(chunks, H, slices), dim3(kOutThreads), smem3, stream, y, (const __nv_bfloat16*)u, dt, la, D, ends, state,
                  cu_seqlens, state_slots, S, sh, err_flag);
    return launch_status();
}

extern "C" int cvb_ssd_step(float* y, const void* packed, int stride, int u_off, int dt_off, const float* conv_w, const float* conv_b, int taps,
                            const float* dt_bias, const float* neg_a, const float* D, float* state, int64_t state_floats, const int* cu_seqlens,
                            const int* state_slots, const int* positions, int num_slots, int S, int H, int G, int N, int P, int dtype,
                            int* err_flag, cudaStream_t stream) {
    if (S == 0) return CVB_OK;
    if (S < 0) return CVB_E_SIZE;
    SsdShape sh;
    const int rc = ssd_shape(sh, H, G, N, P, taps, stride, u_off, dt_off, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    const bool four = P % 4 == 0 && state_floats % 4 == 0 && ssd_al16(state);
    const int nvec = four ? P / 4 : P, R = nvec < kStepThreads ? kStepThreads / nvec : 1;
    const size_t smem = (static_cast<size_t>(P) + 2 * static_cast<size_t>(N) + static_cast<size_t>(R) * P) * sizeof(float);
    if (smem > 48 * 1024) return CVB_E_SIZE;
#define CALL_V(TY, VV) launch_kernel(ssd_step_kernel<TY, VV>, dim3(S, H), dim3(kStepThreads), smem, stream, y, (const TY*)packed, conv_w, conv_b, dt_bias, \
                                     neg_a, D, state, cu_seqlens, state_slots, positions, sh, err_flag)
#define CALL(TY) if (four) { CALL_V(TY, 4); } else { CALL_V(TY, 1); }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_V
    return launch_status();
}

extern "C" int cvb_ssd_norm(void* out, int out_stride, const float* y, const void* z, int z_stride, const float* w, int T, int parts, int n,
                            float eps, float scale, int dtype, cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    if (T < 0 || parts <= 0 || parts > 65535 || n <= 0) return CVB_E_SIZE;
    const int64_t rows = static_cast<int64_t>(T) * parts;
    if (rows > 2147483647LL) return CVB_E_SIZE;
    if (out_stride < parts * n || z_stride < parts * n) return CVB_E_SHAPE;
    const uintptr_t ab = dtype == CVB_DTYPE_BF16 ? 7 : 15;
    const bool vec = n % 4 == 0 && n <= 256 * kNormQuads * 4 && out_stride % 4 == 0 && z_stride % 4 == 0 && ssd_al16(y) && ssd_al16(w)
                     && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & ab) == 0;
#define CALL_N(TY, TH) launch_kernel(ssd_norm_vec_kernel<TY, TH>, dim3(static_cast<unsigned>(TH < 128 ? (rows + 3) / 4 : rows)), dim3(TH < 128 ? 128 : TH), 0, \
                                     stream, (TY*)out, out_stride, y, (const TY*)z, z_stride, w, rows, parts, n, eps, scale)
#define CALL(TY)                                                                                                              \
    if (vec && n <= 512) { CALL_N(TY, 32); }                                                                                  \
    else if (vec && n <= 4096) { CALL_N(TY, 128); }                                                                           \
    else if (vec) { CALL_N(TY, 256); }                                                                                        \
    else launch_kernel(ssd_norm_kernel<TY>, dim3(T, parts), dim3(kSsdThreads), 0, stream, (TY*)out, out_stride, y, (const TY*)z, z_stride, w, \
                       parts, n, eps, scale)
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_N
    return launch_status();
}
