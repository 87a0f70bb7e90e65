// Kernels of the selective scan (Mamba): a recurrence with one decay per channel and
// state number.  Per channel c and state n, with a step size of every channel's own,
//
//     dt_c = softplus(raw_c + bias_c)
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n          (A negative)
//     y_c = sum_n S[c, n] C_n + D_c x_c,      out_c = y_c * silu(z_c)
//
// B and C are shared by all channels of a token.  The kernels serve a step of packed
// rows: sequence b owns rows cu_seqlens[b]..cu_seqlens[b+1], continues from the state
// kept for its cache slot and leaves the state for its next step; a prompt, a portion
// of one and a single token are the same case.  Step sizes, decays, the state and the
// sums are float whatever the activation type is.
#include "common.cuh"
#include <math.h>

namespace {
constexpr float kLog2e = 1.4426950408889634f;

// log(1 + exp(x)) without overflow and without a cut-off
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }

// The decay exp(dt A): the accurate function in the float32 path; in the bfloat16 path
// the hardware's exponential of two, `rate` then holding A log2(e).
template <typename T> __device__ __forceinline__ float decay_of(float dt, float rate);
template <> __device__ __forceinline__ float decay_of<float>(float dt, float rate) { return expf(dt * rate); }
template <> __device__ __forceinline__ float decay_of<bf16>(float dt, float rate) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(dt * rate));
    return y;
}
template <typename T> __device__ __forceinline__ float rate_scale() { return sizeof(T) == 4 ? 1.0f : kLog2e; }

// L lanes share a channel, each owning NP neighbouring states; a block of `kThreads` serves
// kThreads / L neighbouring channels of one sequence.  A tile of TT tokens at a time is
// staged in shared memory as floats: (dt, dt x) per token and channel, (B, C) side by side
// per token and state.  The loads of the next tile are in flight while this one is computed;
// x and z of a tile stay in the registers of the threads that write its outputs.  Tokens are
// walked strictly in order and a token's sum over the states has one order (a lane's NP states,
// then a butterfly over the lanes), so the cut into steps does not show.
template <int NP, int L, int kThreads> struct Tile {
    static constexpr int kStates = NP * L;
    static constexpr int kChannels = kThreads / L;
    static constexpr int TT = kStates <= 128 ? 32 : kStates == 256 ? 16 : 8;
    static constexpr int kPerX = (TT * kChannels + kThreads - 1) / kThreads;        // (token, channel) pairs a thread stages
    static constexpr int kPerB = (TT * kStates + kThreads - 1) / kThreads;          // (B, C) pairs a thread stages
    static_assert(TT % 4 == 0 && L >= 4 && L <= 32, "a tile is whole groups of four tokens, four lanes at least a channel");
};

template <typename T, int NP, int L, int kThreads>
__global__ void __launch_bounds__(kThreads)
selective_scan_kernel(const T* __restrict__ x, int ld_x, const T* __restrict__ bc, int ld_bc,
                      const float* __restrict__ dt_raw, int ld_dt, const float* __restrict__ dt_bias,
                      const float* __restrict__ rates, const float* __restrict__ skip,
                      const T* __restrict__ z, int ld_z, float* __restrict__ state, T* __restrict__ out, int ld_out,
                      const int* __restrict__ cu_seqlens, const int* __restrict__ slots, int C, int N) {
    chain_release();
    chain_wait();
    using G = Tile<NP, L, kThreads>;
    constexpr int TT = G::TT, CB = G::kChannels, NS = G::kStates, PX = G::kPerX, PB = G::kPerB;
    __shared__ __align__(16) float2 sbc[TT * NS];
    __shared__ __align__(16) float2 sd[TT * CB];
    __shared__ float sy[TT * CB];
    const int tid = threadIdx.x;
    const int ch = tid / L, l = tid % L;
    const int c0 = blockIdx.x * CB, c = c0 + ch;
    const int b = blockIdx.y;
    const int first = cu_seqlens[b], last = cu_seqlens[b + 1];
    if (first >= last) return;
    const bool live = c < C;
    float* S = state + ((size_t)slots[b] * C + (live ? c : 0)) * N;
    const bool by_four = N % 4 == 0 && NP % 4 == 0;
    float s[NP], rate[NP];
#pragma unroll
    for (int k = 0; k < NP; ++k) {
        const int n = l * NP + k;
        s[k] = (live && n < N) ? S[n] : 0.f;
        rate[k] = (live && n < N) ? rates[(size_t)c * N + n] * rate_scale<T>() : 0.f;
    }

    // staging: element e of this thread is (token, channel) number tid + e kThreads of the tile
    T rx[PX], rz[PX], rb[PB], rc[PB];
    float rdt[PX];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int e = 0; e < PX; ++e) {
            const int idx = tid + e * kThreads, tt = idx / CB, cc = c0 + idx % CB;
            const bool ok = tt < TT && t0 + tt < last && cc < C;
            const size_t row = ok ? (size_t)(t0 + tt) : 0;
            rx[e] = ok ? x[row * ld_x + cc] : from_f32<T>(0.f);
            rz[e] = ok ? z[row * ld_z + cc] : from_f32<T>(0.f);
            rdt[e] = ok ? dt_raw[row * ld_dt + cc] : 0.f;
        }
#pragma unroll
        for (int e = 0; e < PB; ++e) {
            const int idx = tid + e * kThreads, tt = idx / NS, n = idx % NS;
            const bool ok = tt < TT && t0 + tt < last && n < N;
            const T* row = bc + (ok ? (size_t)(t0 + tt) * ld_bc + n : 0);
            rb[e] = ok ? row[0] : from_f32<T>(0.f);
            rc[e] = ok ? row[N] : from_f32<T>(0.f);
        }
    };
    fetch(first);
    float bias[PX];
#pragma unroll
    for (int e = 0; e < PX; ++e) {
        const int cc = c0 + (tid + e * kThreads) % CB;
        bias[e] = cc < C ? dt_bias[cc] : 0.f;
    }
    for (int t0 = first; t0 < last; t0 += TT) {
        const int nt = min(TT, last - t0);
        float x_now[PX], z_now[PX];
#pragma unroll
        for (int e = 0; e < PX; ++e) {
            const int idx = tid + e * kThreads, tt = idx / CB;
            x_now[e] = to_f32<T>(rx[e]);
            z_now[e] = to_f32<T>(rz[e]);
            if (idx < TT * CB) {
                // a token beyond the last takes a step of nothing: the state stays as it is
                const float dt = tt < nt ? softplus_f(rdt[e] + bias[e]) : 0.f;
                sd[idx] = make_float2(dt, dt * x_now[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < PB; ++e) {
            const int idx = tid + e * kThreads;
            if (TT * NS % kThreads == 0 || idx < TT * NS) sbc[idx] = make_float2(to_f32<T>(rb[e]), to_f32<T>(rc[e]));
        }
        __syncthreads();
        if (t0 + TT < last) fetch(t0 + TT);
#pragma unroll 2
        for (int tq = 0; tq < nt; tq += 4) {
            float acc[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float2 d = sd[(tq + u) * CB + ch];
                const float2* row = sbc + (tq + u) * NS + l * NP;
                float2 v[NP];
                if constexpr (NP % 2 == 0) {
#pragma unroll
                    for (int k = 0; k < NP; k += 2) *reinterpret_cast<float4*>(v + k) = *reinterpret_cast<const float4*>(row + k);
                } else {
#pragma unroll
                    for (int k = 0; k < NP; ++k) v[k] = row[k];
                }
                acc[u] = 0.f;
#pragma unroll
                for (int k = 0; k < NP; ++k) {
                    s[k] = fmaf(decay_of<T>(d.x, rate[k]), s[k], d.y * v[k].x);
                    acc[u] = fmaf(s[k], v[k].y, acc[u]);
                }
            }
            // four sums over L lanes: after two exchanges lane l holds token (l & 3)'s sum over its four lanes
            const bool odd = l & 1, high = l & 2;
            const float p01 = (odd ? acc[1] : acc[0]) + __shfl_xor_sync(0xffffffffu, odd ? acc[0] : acc[1], 1);
            const float p23 = (odd ? acc[3] : acc[2]) + __shfl_xor_sync(0xffffffffu, odd ? acc[2] : acc[3], 1);
            float sum = (high ? p23 : p01) + __shfl_xor_sync(0xffffffffu, high ? p01 : p23, 2);
#pragma unroll
            for (int o = 4; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            if (l < 4) sy[(tq + l) * CB + ch] = sum;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < PX; ++e) {
            const int idx = tid + e * kThreads, tt = idx / CB, cc = c0 + idx % CB;
            if (tt < nt && cc < C)
                out[(size_t)(t0 + tt) * ld_out + cc] = from_f32<T>(fmaf(__ldg(skip + cc), x_now[e], sy[idx]) * silu_f(z_now[e]));
        }
    }
    if (live) {
        if (by_four) {
#pragma unroll
            for (int k = 0; k + 3 < NP; k += 4)
                if (l * NP + k < N) *reinterpret_cast<float4*>(S + l * NP + k) = make_float4(s[k], s[k + 1], s[k + 2], s[k + 3]);
        } else {
#pragma unroll
            for (int k = 0; k < NP; ++k)
                if (l * NP + k < N) S[l * NP + k] = s[k];
        }
    }
}

// The same recurrence for a step in which every sequence brings one token (row b is
// sequence b's): the state is read and written once, four numbers an access where N allows it.
constexpr int kStepThreads = 128;

template <typename T, int NP, int L>
__global__ void __launch_bounds__(kStepThreads)
selective_step_kernel(const T* __restrict__ x, int ld_x, const T* __restrict__ bc, int ld_bc,
                      const float* __restrict__ dt_raw, int ld_dt, const float* __restrict__ dt_bias,
                      const float* __restrict__ rates, const float* __restrict__ skip,
                      const T* __restrict__ z, int ld_z, float* __restrict__ state, T* __restrict__ out, int ld_out,
                      const int* __restrict__ slots, int C, int N) {
    chain_release();
    constexpr int CB = kStepThreads / L;
    const int ch = threadIdx.x / L, l = threadIdx.x % L;
    const int c = blockIdx.x * CB + ch, b = blockIdx.y;
    const bool live = c < C, by_four = N % 4 == 0;
    float rate[NP], s[NP], bb[NP], cc[NP];
    // four numbers of this lane's run of a row of N
    auto four = [&](const float* p, int k) {
        if (by_four) return (live && l * NP + k < N) ? *reinterpret_cast<const float4*>(p + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        auto one = [&](int i) { return (live && l * NP + k + i < N) ? p[k + i] : 0.f; };
        return make_float4(one(0), one(1), one(2), one(3));
    };
    // what no kernel of this step writes is read before the wait
    const float* rate_row = rates + (size_t)(live ? c : 0) * N + l * NP;
#pragma unroll
    for (int k = 0; k < NP; k += 4) {
        const float4 v = four(rate_row, k);
        rate[k] = v.x * rate_scale<T>(); rate[k + 1] = v.y * rate_scale<T>();
        rate[k + 2] = v.z * rate_scale<T>(); rate[k + 3] = v.w * rate_scale<T>();
    }
    const float bias = live ? dt_bias[c] : 0.f, d_skip = live ? skip[c] : 0.f;
    chain_wait();
    float* S = state + ((size_t)slots[b] * C + (live ? c : 0)) * N + l * NP;
    const T* row = bc + (size_t)b * ld_bc;
#pragma unroll
    for (int k = 0; k < NP; k += 4) {
        const float4 v = four(S, k);
        s[k] = v.x; s[k + 1] = v.y; s[k + 2] = v.z; s[k + 3] = v.w;
    }
#pragma unroll
    for (int k = 0; k < NP; ++k) {
        const int n = l * NP + k;
        bb[k] = n < N ? to_f32<T>(row[n]) : 0.f;
        cc[k] = n < N ? to_f32<T>(row[N + n]) : 0.f;
    }
    const float xv = live ? to_f32<T>(x[(size_t)b * ld_x + c]) : 0.f;
    const float zv = live ? to_f32<T>(z[(size_t)b * ld_z + c]) : 0.f;
    const float dt = softplus_f((live ? dt_raw[(size_t)b * ld_dt + c] : 0.f) + bias), dx = dt * xv;
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < NP; ++k) {
        s[k] = fmaf(decay_of<T>(dt, rate[k]), s[k], dx * bb[k]);
        sum = fmaf(s[k], cc[k], sum);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (!live) return;
#pragma unroll
    for (int k = 0; k < NP; ++k) {
        if (l * NP + k >= N) continue;
        if (by_four) {
            if (k % 4 == 0) *reinterpret_cast<float4*>(S + k) = make_float4(s[k], s[k + 1], s[k + 2], s[k + 3]);
        } else {
            S[k] = s[k];
        }
    }
    if (l == 0) out[(size_t)b * ld_out + c] = from_f32<T>(fmaf(d_skip, xv, sum) * silu_f(zv));
}

struct Args {
    const void* x; int ld_x; const void* bc; int ld_bc; const float* dt_raw; int ld_dt; const float* dt_bias;
    const float* rates; const float* skip; const void* z; int ld_z; float* state; void* out; int ld_out;
    const int* cu_seqlens; const int* slots; int n_seqs, C, N, one_token_each; cudaStream_t stream;
};

template <typename T, int NP, int L, int kThreads>
int launch_scan(const Args& a) {
    constexpr int CB = kThreads / L;
    return launch_chained(selective_scan_kernel<T, NP, L, kThreads>, dim3((a.C + CB - 1) / CB, a.n_seqs), dim3(kThreads), 0, a.stream,
                          (const T*)a.x, a.ld_x, (const T*)a.bc, a.ld_bc, a.dt_raw, a.ld_dt, a.dt_bias, a.rates, a.skip, (const T*)a.z,
                          a.ld_z, a.state, (T*)a.out, a.ld_out, a.cu_seqlens, a.slots, a.C, a.N);
}
template <typename T, int NP, int L>
int launch_step(const Args& a) {
    constexpr int CB = kStepThreads / L;
    return launch_chained(selective_step_kernel<T, NP, L>, dim3((a.C + CB - 1) / CB, a.n_seqs), dim3(kStepThreads), 0, a.stream,
                          (const T*)a.x, a.ld_x, (const T*)a.bc, a.ld_bc, a.dt_raw, a.ld_dt, a.dt_bias, a.rates, a.skip, (const T*)a.z,
                          a.ld_z, a.state, (T*)a.out, a.ld_out, a.slots, a.C, a.N);
}

// Measurements and tests may fix the states of a lane (1, 2 or 4); 0: the launcher chooses.
static int g_states = 0;

template <typename T>
int dispatch(const Args& a) {
    if (a.one_token_each) {
        if (a.N <= 16) return launch_step<T, 4, 4>(a);
        if (a.N <= 32) return launch_step<T, 4, 8>(a);
        if (a.N <= 64) return launch_step<T, 4, 16>(a);
        if (a.N <= 128) return launch_step<T, 4, 32>(a);
        if (a.N <= 256) return launch_step<T, 8, 32>(a);
        return launch_step<T, 16, 32>(a);
    }
    // states a lane: many lanes a channel where the step brings few states, so that a scheduler has several warps to
    // turn to (measured with 16 states a channel: one prompt of 2,048 tokens and 4,096 channels 162 / 186 / 219 us at
    // 1 / 2 / 4, 8,192 channels 270 / 240 / 258; eight prompts of 4,096 channels 870 / 691 / 652)
    const long long states = (long long)a.C * a.N * a.n_seqs;
    int np = states > 400000 ? 4 : states > 90000 ? 2 : 1;
    if (g_states == 1 || g_states == 2 || g_states == 4) np = g_states;
    if (a.N <= 16) return np == 1 ? launch_scan<T, 1, 16, 256>(a) : np == 2 ? launch_scan<T, 2, 8, 256>(a) : launch_scan<T, 4, 4, 128>(a);
    if (a.N <= 32) return np == 1 ? launch_scan<T, 1, 32, 512>(a) : np == 2 ? launch_scan<T, 2, 16, 256>(a) : launch_scan<T, 4, 8, 256>(a);
    if (a.N <= 64) return launch_scan<T, 2, 32, 512>(a);
    if (a.N <= 128) return launch_scan<T, 4, 32, 512>(a);
    if (a.N <= 256) return launch_scan<T, 8, 32, 256>(a);
    return launch_scan<T, 16, 32, 256>(a);
}
}  // namespace

GTG_API void gtg_selective_scan_shape(int states) { g_states = states; }

// Most states a channel may have.
GTG_API int gtg_selective_scan_max_states() { return 512; }

// x, z [n, C], bc [n, B: N | C: N] and out of the activation type (dtype 0 float, 1 bfloat16); dt_raw float
// [n, C]; rates float [C, N], the negative A; state float [slots, C, N].  `one_token_each`: row b is
// sequence b's only token.
GTG_API int gtg_selective_scan(int dtype, const void* x, int ld_x, const void* bc, int ld_bc, const float* dt_raw, int ld_dt,
                               const float* dt_bias, const float* rates, const float* skip, const void* z, int ld_z,
                               float* state, void* out, int ld_out, const int* cu_seqlens, const int* slots, int n_seqs,
                               int C, int N, int one_token_each, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (C <= 0 || N <= 0 || ld_x < C || ld_z < C || ld_dt < C || ld_out < C || ld_bc < 2 * N) return kErrBadArgument;
    if (N > gtg_selective_scan_max_states() || n_seqs > 65535 || ((uintptr_t)state % 16) || ((uintptr_t)rates % 16)) return kErrUnsupported;
    const Args a{x, ld_x, bc, ld_bc, dt_raw, ld_dt, dt_bias, rates, skip, z, ld_z, state, out, ld_out, cu_seqlens, slots,
                 n_seqs, C, N, one_token_each, stream};
    if (dtype == 0) return dispatch<float>(a);
    if (dtype == 1) return dispatch<bf16>(a);
    return kErrBadArgument;
}
