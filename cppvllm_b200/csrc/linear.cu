// Gated linear attention: a matrix S [dk, dv] per request and head whose rows decay by a number per token and key channel,
//
//   g = sg(Wa2 a + b)^(1 / tau);   S <- diag(g) S + k v^T;   o = S^T (qk_scale q)
//
// float throughout; q, k, v (and the low-rank a, the output gate) are column ranges of a packed projection in the activations' type T.
//
//   linear_decay : g in place of the float product z = Wa2 a
//   linear_scan  : portions of prompts.  A block owns 64 (32 for more than 128 rows) columns of S of one (chunk of a request's tokens,
//                  head); eight lanes share four (two) columns, a lane four neighbouring rows of every 32.  Eight tokens a stage
//                  travel through registers into shared memory (converted on the way), so a token costs a lane three 16-byte reads
//                  of shared memory per four rows and four columns (the reads of shared memory are what bounds the kernel); the
//                  eight partial outputs of a stage are added up and handed out over the eight lanes by one transposing butterfly
//                  (seven shuffles a column).  Long portions are cut into chunks that run side by side:
//                    pass 1: every chunk but a request's last: the state it leaves and the product of its decays, from zero (a
//                            request's first chunk from the request's state); the last chunk's place receives the state in front
//                    pass 2: the states behind the chunks in turn, element by element: E_k <- diag(P_k) E_(k-1) + E_k
//                    pass 3: every chunk from its true state, with outputs; a request's last chunk leaves the new state
//                  Where no request has more than one chunk only pass 3 runs.
//   linear_step  : a step of decoded tokens (one per request) in one kernel, a block per (request, head): the low-rank decay product,
//                  the decay, the rule on S, the RMS norm of the head's output, its weight, silu of the gate and a constant, into a
//                  column range of wider rows.
#include "common.cuh"

namespace cvb {

__device__ __forceinline__ float linear_silu(float z) { return z / (1.f + expf(-z)); }
// sigmoid(z)^(1 / tau), through its logarithm min(z, 0) - ln(1 + e^-|z|)
__device__ __forceinline__ float root_of_sigmoid(float z, float inv_tau) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau); }

__global__ void __launch_bounds__(256)
linear_decay_kernel(float* __restrict__ z, const float* __restrict__ bias, float inv_tau, int n, int64_t total) {
    pdl_trigger();
    pdl_wait();
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < total; i += static_cast<int64_t>(gridDim.x) * 256)
        z[i] = root_of_sigmoid(z[i] + bias[i % n], inv_tau);
}
__global__ void __launch_bounds__(256)
linear_decay_vec_kernel(float* __restrict__ z, const float* __restrict__ bias, float inv_tau, int n4, int64_t total4) {
    pdl_trigger();
    pdl_wait();
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < total4; i += static_cast<int64_t>(gridDim.x) * 256) {
        float4 v = reinterpret_cast<float4*>(z)[i];
        const int c = static_cast<int>(i % n4) * 4;
        v.x = root_of_sigmoid(v.x + bias[c], inv_tau);
        v.y = root_of_sigmoid(v.y + bias[c + 1], inv_tau);
        v.z = root_of_sigmoid(v.z + bias[c + 2], inv_tau);
        v.w = root_of_sigmoid(v.w + bias[c + 3], inv_tau);
        reinterpret_cast<float4*>(z)[i] = v;
    }
}

constexpr int kLinThreads = 128;
constexpr int kLinTokens = 8;                            // tokens per stage: as many as lanes share a column
constexpr int lin_cols(int kpt) { return kpt <= 16 ? 4 : 2; }         // columns of S per eight lanes; 16 times that per block

struct LinearShape {
    int H, dk, dv, stride, q_off, k_off, v_off;
    float qk_scale;
    int64_t state_floats;
    int num_slots;
};

// Block x's chunk: chunk k of the n chunks of request s.  `buf`: where the request's chunks lie in the chunk buffers, which
// hold requests with more than one chunk only.
__device__ __forceinline__ bool linear_locate(const int* __restrict__ cu_seqlens, int S, int len, int x, int& s_out, int& k, int& n, int& buf) {
    int base = 0, held = 0;
    for (int s = 0; s < S; ++s) {
        const int tokens = cu_seqlens[s + 1] - cu_seqlens[s];
        const int chunks = (tokens + len - 1) / len;
        if (x < base + chunks) { s_out = s; k = x - base; n = chunks; buf = held; return true; }
        base += chunks;
        if (chunks > 1) held += chunks;
    }
    return false;
}

// 16 bytes of a row as floats
template <typename T> struct Raw16;
template <> struct Raw16<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void put(float* dst, const uint4& r, float s) {
        *reinterpret_cast<float4*>(dst) = make_float4(__uint_as_float(r.x) * s, __uint_as_float(r.y) * s, __uint_as_float(r.z) * s, __uint_as_float(r.w) * s);
    }
};
template <> struct Raw16<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void put(float* dst, const uint4& r, float s) {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
        const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]), c = __bfloat1622float2(h[2]), d = __bfloat1622float2(h[3]);
        *reinterpret_cast<float4*>(dst) = make_float4(a.x * s, a.y * s, b.x * s, b.y * s);
        *reinterpret_cast<float4*>(dst + 4) = make_float4(c.x * s, c.y * s, d.x * s, d.y * s);
    }
};

template <typename T, int KPT, bool OUT>
__global__ void __launch_bounds__(kLinThreads)
linear_scan_kernel(float* __restrict__ out, const T* __restrict__ packed, const float* __restrict__ gg, float* __restrict__ state,
                   float* __restrict__ ends, float* __restrict__ decays, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ state_slots, int n_seqs, int len, LinearShape sh, int vec, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    constexpr int dkp = KPT * 8;                          // rows, padded
    constexpr int NC = lin_cols(KPT), kLinCols = 16 * NC;
    constexpr int kArr = OUT ? 3 : 2;                     // k, g and, with outputs, q
    constexpr int kStage = kLinTokens * (kArr * dkp + kLinCols);
    extern __shared__ __align__(16) float sm[];           // two stages
    const int h = blockIdx.y, j0 = blockIdx.z * kLinCols, tid = threadIdx.x;
    const int part = tid & 7, col = (tid >> 3) * NC, j = j0 + col;
    const int dk = sh.dk, dv = sh.dv;
    int s, kc, nc, buf;
    if (!linear_locate(cu_seqlens, n_seqs, len, blockIdx.x, s, kc, nc, buf)) return;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (tid == 0) atomicExch(err, 2);
        return;
    }
    const int begin = cu_seqlens[s] + kc * len, end = min(begin + len, cu_seqlens[s + 1]);
    float* st = state + static_cast<int64_t>(slot) * sh.state_floats + static_cast<int64_t>(h) * dk * dv;
    const int64_t mat = static_cast<int64_t>(sh.H) * dk * dv;
    auto end_of = [&](int k) { return ends + (static_cast<int64_t>(buf) + k) * mat + static_cast<int64_t>(h) * dk * dv; };
    // row r of this lane's KPT rows
    auto row = [&](int r) { return (r >> 2) * 32 + part * 4 + (r & 3); };
    const float* from = OUT ? (nc == 1 ? st : (kc == 0 ? end_of(nc - 1) : end_of(kc - 1))) : st;
    const bool zero = !OUT && kc > 0;
    float S[KPT][NC];
#pragma unroll
    for (int r = 0; r < KPT; ++r)
#pragma unroll
        for (int c = 0; c < NC; ++c)
            S[r][c] = (row(r) < dk && j + c < dv && !(zero && kc < nc - 1)) ? from[static_cast<int64_t>(row(r)) * dv + j + c] : 0.f;
    auto put = [&](float* dst) {
#pragma unroll
        for (int r = 0; r < KPT; ++r)
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (row(r) < dk && j + c < dv) dst[static_cast<int64_t>(row(r)) * dv + j + c] = S[r][c];
    };
    if (!OUT && kc == nc - 1) {                           // the state in front of the portion, where the first chunk of pass 3 finds it
        if (nc > 1) put(end_of(kc));
        return;
    }
    for (int i = tid; i < 2 * kStage; i += kLinThreads) sm[i] = 0.f;         // rows past dk and columns past dv stay zero
    __syncthreads();

    // a stage: [tokens][dkp] of k, of g, (of q), [tokens][columns] of v
    constexpr int N = Raw16<T>::N;
    constexpr int kQK = (OUT ? 2 : 1) * kLinTokens * dkp / N;                // 16-byte pieces of k (and q) in a stage
    constexpr int kQKPer = (kQK + kLinThreads - 1) / kLinThreads;
    constexpr int kGPer = (kLinTokens * dkp / 4 + kLinThreads - 1) / kLinThreads;
    constexpr int kVPer = (kLinTokens * kLinCols / N + kLinThreads - 1) / kLinThreads;
    uint4 rq[kQKPer], rv[kVPer];
    float4 rg[kGPer];
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    auto fetch = [&](int t0) {
        const int n = end - t0;
#pragma unroll
        for (int u = 0; u < kQKPer; ++u) {
            const int idx = tid + u * kLinThreads;
            const int arr = idx / (kLinTokens * dkp / N), rem = idx - arr * (kLinTokens * dkp / N);
            const int tt = rem / (dkp / N), i = (rem - tt * (dkp / N)) * N;
            rq[u] = (idx < kQK && tt < n && i < dk)
                        ? *reinterpret_cast<const uint4*>(packed + static_cast<int64_t>(t0 + tt) * sh.stride + (arr ? sh.q_off : sh.k_off) + h * dk + i) : zero4;
        }
#pragma unroll
        for (int u = 0; u < kGPer; ++u) {
            const int idx = tid + u * kLinThreads;
            const int tt = idx / (dkp / 4), i = (idx - tt * (dkp / 4)) * 4;
            rg[u] = (tt < min(n, kLinTokens) && i < dk) ? *reinterpret_cast<const float4*>(gg + (static_cast<int64_t>(t0 + tt) * sh.H + h) * dk + i)
                                                        : make_float4(1.f, 1.f, 1.f, 1.f);
        }
#pragma unroll
        for (int u = 0; u < kVPer; ++u) {
            const int idx = tid + u * kLinThreads;
            const int tt = idx / (kLinCols / N), c = (idx - tt * (kLinCols / N)) * N;
            rv[u] = (tt < min(n, kLinTokens) && j0 + c < dv)
                        ? *reinterpret_cast<const uint4*>(packed + static_cast<int64_t>(t0 + tt) * sh.stride + sh.v_off + h * dv + j0 + c) : zero4;
        }
    };
    auto keep = [&](int stage) {
        float* base = sm + stage * kStage;
#pragma unroll
        for (int u = 0; u < kQKPer; ++u) {
            const int idx = tid + u * kLinThreads;
            const int arr = idx / (kLinTokens * dkp / N), rem = idx - arr * (kLinTokens * dkp / N);
            if (idx < kQK) Raw16<T>::put(base + (arr ? 2 : 0) * kLinTokens * dkp + rem * N, rq[u], arr ? sh.qk_scale : 1.f);
        }
#pragma unroll
        for (int u = 0; u < kGPer; ++u) {
            const int idx = tid + u * kLinThreads;
            if (idx < kLinTokens * dkp / 4) *reinterpret_cast<float4*>(base + kLinTokens * dkp + idx * 4) = rg[u];
        }
#pragma unroll
        for (int u = 0; u < kVPer; ++u) {
            const int idx = tid + u * kLinThreads;
            if (idx < kLinTokens * kLinCols / N) Raw16<T>::put(base + kArr * kLinTokens * dkp + idx * N, rv[u], 1.f);
        }
    };
    // rows that do not start on 16 bytes: element by element, straight into the stage
    auto direct = [&](int t0, int stage) {
        float* base = sm + stage * kStage;
        const int n = min(kLinTokens, end - t0);
        for (int idx = tid; idx < kLinTokens * dk; idx += kLinThreads) {
            const int tt = idx / dk, i = idx - tt * dk;
            const bool live = tt < n;
            const T* rp = packed + static_cast<int64_t>(t0 + (live ? tt : 0)) * sh.stride + h * dk + i;
            base[tt * dkp + i] = live ? to_float(rp[sh.k_off]) : 0.f;
            base[(kLinTokens + tt) * dkp + i] = live ? gg[(static_cast<int64_t>(t0 + tt) * sh.H + h) * dk + i] : 1.f;
            if (OUT) base[(2 * kLinTokens + tt) * dkp + i] = live ? to_float(rp[sh.q_off]) * sh.qk_scale : 0.f;
        }
        for (int idx = tid; idx < kLinTokens * kLinCols; idx += kLinThreads) {
            const int tt = idx / kLinCols, c = idx - tt * kLinCols;
            base[kArr * kLinTokens * dkp + idx] = (tt < n && j0 + c < dv) ? to_float(packed[static_cast<int64_t>(t0 + tt) * sh.stride + sh.v_off + h * dv + j0 + c]) : 0.f;
        }
    };

    float P[KPT];                                         // pass 1: the product of the chunk's decays (columns 0 and 1 of the block keep it)
    if (!OUT) {
#pragma unroll
        for (int r = 0; r < KPT; ++r) P[r] = 1.f;
    }
    if (vec) fetch(begin);
    int stage = 0;
    for (int t0 = begin; t0 < end; t0 += kLinTokens, stage ^= 1) {
        if (vec) keep(stage); else direct(t0, stage);
        __syncthreads();                                  // one barrier a stage: the other stage's readers passed the barrier before
        if (vec && t0 + kLinTokens < end) fetch(t0 + kLinTokens);
        const float* base = sm + stage * kStage;
        float o[kLinTokens][NC];
#pragma unroll
        for (int tt = 0; tt < kLinTokens; ++tt) {         // tokens past the end: k = 0 and g = 1 change nothing
            float v[NC];
            const float* vp = base + kArr * kLinTokens * dkp + tt * kLinCols + col;
            if constexpr (NC == 4) { const float4 x = *reinterpret_cast<const float4*>(vp); v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
            else { const float2 x = *reinterpret_cast<const float2*>(vp); v[0] = x.x; v[1] = x.y; }
#pragma unroll
            for (int c = 0; c < NC; ++c) o[tt][c] = 0.f;
#pragma unroll
            for (int m = 0; m < KPT / 4; ++m) {
                const int at = tt * dkp + m * 32 + part * 4;
                const float4 k4 = *reinterpret_cast<const float4*>(base + at);
                const float4 g4 = *reinterpret_cast<const float4*>(base + kLinTokens * dkp + at);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, g[4] = {g4.x, g4.y, g4.z, g4.w};
                float qq[4] = {0.f, 0.f, 0.f, 0.f};
                if (OUT) {
                    const float4 q4 = *reinterpret_cast<const float4*>(base + 2 * kLinTokens * dkp + at);
                    qq[0] = q4.x; qq[1] = q4.y; qq[2] = q4.z; qq[3] = q4.w;
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        float& x = S[m * 4 + e][c];
                        x = fmaf(g[e], x, kk[e] * v[c]);
                        if (OUT) o[tt][c] = fmaf(x, qq[e], o[tt][c]);
                    }
                    if (!OUT) P[m * 4 + e] *= g[e];
                }
            }
        }
        if (OUT) {
            // lane `part` of the eight receives the sums of token `part`
#pragma unroll
            for (int half = kLinTokens / 2; half > 0; half >>= 1) {
                const bool up = (part & half) != 0;
#pragma unroll
                for (int i = 0; i < half; ++i)
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const float away = up ? o[i][c] : o[i + half][c], own = up ? o[i + half][c] : o[i][c];
                        o[i][c] = own + __shfl_xor_sync(0xffffffffu, away, half);
                    }
            }
            const int t = t0 + part;
            if (t < end) {
                float* dst = out + (static_cast<int64_t>(t) * sh.H + h) * dv + j;
                if (NC == 4 && j + 3 < dv && (dv & 3) == 0) {
                    *reinterpret_cast<float4*>(dst) = make_float4(o[0][0], o[0][1], o[0][NC - 2], o[0][NC - 1]);
                } else {
#pragma unroll
                    for (int c = 0; c < NC; ++c)
                        if (j + c < dv) dst[c] = o[0][c];
                }
            }
        }
    }
    if (!OUT || kc == nc - 1) put(OUT ? st : end_of(kc));
    if (!OUT && j0 == 0 && col == 0) {
        float* pd = decays + ((static_cast<int64_t>(buf) + kc) * sh.H + h) * dk;
#pragma unroll
        for (int r = 0; r < KPT; ++r)
            if (row(r) < dk) pd[row(r)] = P[r];
    }
}

// E_k <- diag(P_k) E_(k-1) + E_k for the chunks 1 .. n - 2 of every request with more than one chunk.  Grid: (request, head, rows).
__global__ void __launch_bounds__(256)
linear_carry_kernel(float* __restrict__ ends, const float* __restrict__ decays, const int* __restrict__ cu_seqlens, int n_seqs, int len, int H,
                    int dk, int dv) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y;
    int buf = 0;
    for (int q = 0; q < s; ++q) {
        const int chunks = (cu_seqlens[q + 1] - cu_seqlens[q] + len - 1) / len;
        if (chunks > 1) buf += chunks;
    }
    const int nc = (cu_seqlens[s + 1] - cu_seqlens[s] + len - 1) / len;
    if (nc < 3) return;
    const int64_t mat = static_cast<int64_t>(H) * dk * dv;
    for (int i = blockIdx.z * 256 + threadIdx.x; i < dk * dv; i += gridDim.z * 256) {
        float* e = ends + buf * mat + static_cast<int64_t>(h) * dk * dv + i;
        const float* p = decays + (static_cast<int64_t>(buf) * H + h) * dk + i / dv;
        float run = e[0];
#pragma unroll 4
        for (int k = 1; k < nc - 1; ++k) {
            run = fmaf(p[static_cast<int64_t>(k) * H * dk], run, e[k * mat]);
            e[k * mat] = run;
        }
    }
}

// One token per request.  The block's threads are laid out as rows of S by groups of V neighbouring columns (V = 4 where the
// value size allows 16-byte accesses): a thread updates its columns of every R-th row, adds its part of S^T q up in registers,
// and the R partial sums of a column meet in shared memory in a fixed order.
constexpr int kLinearThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kLinearThreads)
linear_step_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ packed, int g_off, int a_off, int rank,
                   const T* __restrict__ wa2, const float* __restrict__ a2_bias, float inv_tau, const float* __restrict__ norm_w, float eps,
                   float out_scale, float* __restrict__ state, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                   LinearShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int dk = sh.dk, dv = sh.dv;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (tid == 0) atomicExch(err, 2);
        return;
    }
    float* qs = sm;                                      // [dk] each
    float* ks = qs + dk;
    float* as = ks + dk;
    float* lo = as + dk;                                 // [rank]
    float* part = lo + rank;                             // [R, dv]
    const int nvec = (dv + V - 1) / V;
    const bool narrow = nvec < kLinearThreads;
    const int R = narrow ? kLinearThreads / nvec : 1;    // rows worked on side by side
    const int64_t t = cu_seqlens[s];
    const T* row = packed + t * sh.stride;
    for (int i = tid; i < rank; i += kLinearThreads) lo[i] = to_float(row[a_off + i]);
    for (int i = tid; i < dk; i += kLinearThreads) {
        qs[i] = to_float(row[sh.q_off + h * dk + i]) * sh.qk_scale;
        ks[i] = to_float(row[sh.k_off + h * dk + i]);
    }
    __syncthreads();
    for (int i = tid; i < dk; i += kLinearThreads) {
        const T* w = wa2 + static_cast<int64_t>(h * dk + i) * rank;
        float z = 0.f;
#pragma unroll 8
        for (int r = 0; r < rank; ++r) z = fmaf(to_float(w[r]), lo[r], z);
        as[i] = root_of_sigmoid(z + a2_bias[h * dk + i], inv_tau);
    }
    __syncthreads();
    float* st = state + static_cast<int64_t>(slot) * sh.state_floats + static_cast<int64_t>(h) * dk * dv;
    const int rg = narrow ? tid / nvec : 0;
    for (int cv = narrow ? tid - rg * nvec : tid; cv < nvec; cv += (narrow ? nvec : kLinearThreads)) {
        if (rg >= R) break;
        float v[V], o[V];
#pragma unroll
        for (int j = 0; j < V; ++j) { v[j] = to_float(row[sh.v_off + h * dv + cv * V + j]); o[j] = 0.f; }
#pragma unroll 8
        for (int i = rg; i < dk; i += R) {
            float* p = st + static_cast<int64_t>(i) * dv + cv * V;
            const float a = as[i], k = ks[i], q = qs[i];
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
        for (int j = 0; j < V; ++j) part[rg * dv + cv * V + j] = o[j];
    }
    __syncthreads();
    float ss = 0.f;
    for (int j = tid; j < dv; j += kLinearThreads) {
        float o = 0.f;
        for (int r = 0; r < R; ++r) o += part[r * dv + j];
        part[j] = o;                                     // a column is added up and read back by one thread
        ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = out_scale / sqrtf(ss / static_cast<float>(dv) + eps);
    for (int j = tid; j < dv; j += kLinearThreads) {
        const float g = to_float(row[g_off + h * dv + j]);
        out[t * out_stride + h * dv + j] = from_float<T>(part[j] * inv * norm_w[j] * linear_silu(g));
    }
}

static int linear_shape(LinearShape& sh, int H, int dk, int dv, int stride, int q_off, int k_off, int v_off, float qk_scale, int64_t state_floats,
                        int num_slots) {
    if (H <= 0 || H > 65535 || dk <= 0 || dv <= 0 || num_slots <= 0) return CVB_E_SIZE;
    if (state_floats < static_cast<int64_t>(H) * dk * dv) return CVB_E_SHAPE;
    if (q_off < 0 || k_off < 0 || v_off < 0 || stride < q_off + H * dk || stride < k_off + H * dk || stride < v_off + H * dv) return CVB_E_SHAPE;
    sh = LinearShape{H, dk, dv, stride, q_off, k_off, v_off, qk_scale, state_floats, num_slots};
    return CVB_OK;
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int KPT, bool OUT>
static void launch_linear(float* out, const T* packed, const float* gg, float* state, float* ends, float* decays, const int* cu_seqlens,
                          const int* state_slots, int S, int len, int chunks, const LinearShape& sh, int vec, int* err, cudaStream_t stream) {
    constexpr int cols = 16 * lin_cols(KPT);
    const size_t smem = static_cast<size_t>(2) * kLinTokens * ((OUT ? 3 : 2) * KPT * 8 + cols) * sizeof(float);
    static bool raised = false;
    if (smem > 48 * 1024 && !raised) {
        if (cudaFuncSetAttribute(linear_scan_kernel<T, KPT, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) return;
        raised = true;
    }
    launch_kernel(linear_scan_kernel<T, KPT, OUT>, dim3(chunks, sh.H, (sh.dv + cols - 1) / cols), dim3(kLinThreads), smem, stream, out, packed,
                  gg, state, ends, decays, cu_seqlens, state_slots, S, len, sh, vec, err);
}

template <typename T, int KPT>
static int run_linear(float* out, const T* packed, const float* gg, float* state, float* ends, float* decays, const int* cu_seqlens,
                      const int* state_slots, int S, int len, int chunks, int single, const LinearShape& sh, int vec, int* err, cudaStream_t stream) {
    if (!single) {
        launch_linear<T, KPT, false>(out, packed, gg, state, ends, decays, cu_seqlens, state_slots, S, len, chunks, sh, vec, err, stream);
        const int zs = (sh.dk * sh.dv + 255) / 256;
        launch_kernel(linear_carry_kernel, dim3(S, sh.H, zs < 64 ? zs : 64), dim3(256), 0, stream, ends, decays, cu_seqlens, S, len, sh.H, sh.dk, sh.dv);
    }
    launch_linear<T, KPT, true>(out, packed, gg, state, ends, decays, cu_seqlens, state_slots, S, len, chunks, sh, vec, err, stream);
    return launch_status();
}

}  // namespace cvb

using namespace cvb;

extern "C" int cvb_linear_decay(float* z, const float* bias, float inv_tau, int T, int n, cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    if (T < 0 || n <= 0) return CVB_E_SIZE;
    const int64_t total = static_cast<int64_t>(T) * n;
    const bool four = n % 4 == 0 && al16(z);
    const int64_t want = ((four ? total / 4 : total) + 255) / 256;
    const unsigned blocks = static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16);
    if (four) launch_kernel(linear_decay_vec_kernel, dim3(blocks), dim3(256), 0, stream, z, bias, inv_tau, n / 4, total / 4);
    else launch_kernel(linear_decay_kernel, dim3(blocks), dim3(256), 0, stream, z, bias, inv_tau, n, total);
    return launch_status();
}

// `chunks`: how many chunks of `len` tokens (a multiple of eight) the step's requests have together; `held`: how many of them belong to
// requests with more than one (0: pass 3 alone runs); `ends` holds H dk dv floats and `decays` H dk floats per held chunk.
extern "C" int cvb_linear_scan(float* out, const void* packed, int stride, int q_off, int k_off, int v_off, float qk_scale, const float* gg,
                               float* state, int64_t state_floats, int num_slots, float* ends, int64_t ends_floats, float* decays,
                               int64_t decays_floats, const int* cu_seqlens, const int* state_slots, int S, int len, int chunks, int held,
                               int H, int dk, int dv, int dtype, int* err_flag, cudaStream_t stream) {
    if (S == 0) return CVB_OK;
    LinearShape sh;
    const int rc = linear_shape(sh, H, dk, dv, stride, q_off, k_off, v_off, qk_scale, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    if (S < 0 || dk > 512 || len <= 0 || len % kLinTokens || chunks <= 0 || (dv + 31) / 32 > 65535) return CVB_E_SIZE;
    if (held > 0 && (ends == nullptr || decays == nullptr || ends_floats < static_cast<int64_t>(held) * H * dk * dv
                     || decays_floats < static_cast<int64_t>(held) * H * dk)) return CVB_E_SCRATCH;
    const int n = dtype == CVB_DTYPE_BF16 ? 8 : 4;
    if (!al16(out)) return CVB_E_ALIGN;
    const int vec = dk % n == 0 && dv % n == 0 && stride % n == 0 && q_off % n == 0 && k_off % n == 0 && v_off % n == 0 && al16(packed) && al16(gg);
#define CALL_K(TY, KPT) return run_linear<TY, KPT>(out, (const TY*)packed, gg, state, ends, decays, cu_seqlens, state_slots, S, len, chunks,    \
                                                   held == 0, sh, vec, err_flag, stream)
#define CALL(TY)                                                                                                              \
    if (dk <= 32) { CALL_K(TY, 4); }                                                                                          \
    else if (dk <= 64) { CALL_K(TY, 8); }                                                                                     \
    else if (dk <= 128) { CALL_K(TY, 16); }                                                                                   \
    else if (dk <= 256) { CALL_K(TY, 32); }                                                                                   \
    else { CALL_K(TY, 64); }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_K
}

extern "C" int cvb_linear_step(void* out, int out_stride, const void* packed, int stride, int q_off, int k_off, int v_off, int g_off, int a_off,
                               int rank, const void* wa2, const float* a2_bias, float qk_scale, float inv_tau, const float* norm_w, float eps,
                               float out_scale, float* state, int64_t state_floats, const int* cu_seqlens, const int* state_slots,
                               int num_slots, int S, int H, int dk, int dv, int dtype, int* err_flag, cudaStream_t stream) {
    if (S == 0) return CVB_OK;
    LinearShape sh;
    const int rc = linear_shape(sh, H, dk, dv, stride, q_off, k_off, v_off, qk_scale, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    if (S < 0 || rank <= 0) return CVB_E_SIZE;
    if (out_stride < H * dv || g_off < 0 || stride < g_off + H * dv || a_off < 0 || stride < a_off + rank) return CVB_E_SHAPE;
    const bool four = dv % 4 == 0 && (state_floats & 3) == 0 && al16(state);
    const int V = four ? 4 : 1, nvec = (dv + V - 1) / V, R = nvec < kLinearThreads ? kLinearThreads / nvec : 1;
    const size_t smem = (static_cast<size_t>(3) * dk + rank + static_cast<size_t>(R) * dv) * sizeof(float);
    if (smem > 48 * 1024) return CVB_E_SIZE;
#define CALL_V(TY, VV)                                                                                                        \
    launch_kernel(linear_step_kernel<TY, VV>, dim3(S, H), dim3(kLinearThreads), smem, stream, (TY*)out, out_stride, (const TY*)packed, g_off,  \
                  a_off, rank, (const TY*)wa2, a2_bias, inv_tau, norm_w, eps, out_scale, state, cu_seqlens, state_slots, sh, err_flag)
#define CALL(TY) if (four) { CALL_V(TY, 4); } else { CALL_V(TY, 1); }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_V
    return launch_status();
}
