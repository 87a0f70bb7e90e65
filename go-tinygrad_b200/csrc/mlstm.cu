// Kernels of the matrix memory (mLSTM): a recurrent mixer whose per-sequence state is,
// per head, a matrix S of d x dv floats, a vector n of d floats and the running maximum
// m of the logarithms of its gates.  With a log input gate i and a log forget gate f,
//
//     i = cap tanh((raw_i + bias_i) / cap),  f = log sigmoid(cap tanh((raw_f + bias_f) / cap))
//     m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone
//     o = S^T (q q_scale) / (max(|n . q q_scale|, exp(-m')) + 1e-6)
//
// S, n and m are zero at the start.  The kernels leave the numerators S^T q and the
// denominators; `head_norm_gate` (delta.cu) divides, norms and gates.  They serve a step
// of packed rows: sequence b owns rows cu_seqlens[b]..cu_seqlens[b+1], continues from the
// state kept for its cache slot and leaves the state for its next step; a prompt, a
// portion of one and a single token are the same case.  Gates, their logarithms and
// exponentials, the maximum, the state and the sums are float whatever the activation
// type is.
//
// The columns of S never meet, and n is one more column whose value is always 1: column
// dv of a head stands for it.  The running maximum is kept once per column, dv + 1 equal
// copies per head, so that blocks that serve different columns of a head share nothing.
#include "common.cuh"
#include <math.h>

namespace {
// log(sigmoid(x)) without overflow and without a cut-off
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float capped(float x, float cap) { return cap * tanhf(x / cap); }

// two floats in one register pair: products and sums of both in one instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair_of(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 parts_of(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// ------------------------------------------------ prompts: the recurrence token by token
// One block per (head, slice of columns, sequence).  RG lanes share kCP neighbouring columns,
// each owning kKR rows of them in registers: rows 4 (r + RG j) .. + 4 for lane r of the RG, so
// that k and q of a token arrive by 16-byte reads from shared memory (rows beyond d are zeros
// there).  A warp serves 32 / RG such groups.  What a token costs a lane is kKR kCP products and
// two fused multiply-adds each, on pairs of rows; the sums of four tokens and kCP columns meet in
// one butterfly in which every exchange halves what a lane still carries.
//
// Tiles of kTT tokens are double-buffered in shared memory as floats.  While the columns' warps
// compute a tile, four warps of helpers store the next one (its loads were issued a tile earlier)
// and write the results of the one before to memory, and one warp works out the gates of the next.
// A token beyond the last is staged as zeros with a step that changes nothing.  Tokens are walked
// strictly in order: the result does not depend on the cut of the sequence into steps, on the
// batch or on the slices.
constexpr int kTT = 16;
constexpr int kKR = 16;                    // rows a lane owns
constexpr int kCP = 2;                     // columns a lane owns
constexpr int kMaxWarps = 8;               // warps of columns a block may have
constexpr int kHelpers = 128;              // threads that move tiles
constexpr int kMaxCols = 64;               // columns a block may serve

template <typename T, int RG>
__global__ void __launch_bounds__(kMaxWarps * 32 + 32 + kHelpers)
mlstm_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int ld,
                  const float* __restrict__ gates, int ld_gates, const float* __restrict__ gate_bias, float cap, float q_scale,
                  float* __restrict__ S_all, float* __restrict__ n_all, float* __restrict__ m_all,
                  float* __restrict__ num, int ld_num, float* __restrict__ den,
                  const int* __restrict__ cu_seqlens, const int* __restrict__ slots, int heads, int d, int dv, int warps, int slices, int vec) {
    chain_release();
    chain_wait();
    constexpr int D = RG * kKR, WC = 32 / RG * kCP;
    extern __shared__ __align__(16) float smem[];
    const int cols = warps * WC;
    float* sk = smem;                              // [2][kTT][D]
    float* sq = sk + 2 * kTT * D;                  // [2][kTT][D]
    float* sv = sq + 2 * kTT * D;                  // [2][kTT][cols]
    float* sy = sv + 2 * kTT * cols;               // [2][kTT][cols]
    float4* sg = reinterpret_cast<float4*>(sy + 2 * kTT * cols);     // [2][kTT] (keep, add, exp(-m), m)
    const int h = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
    const int first = cu_seqlens[b], last = cu_seqlens[b + 1];
    if (first >= last) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int j0 = slice * cols;                   // the block's first column
    const int tiles = (last - first + kTT - 1) / kTT;
    const size_t head = (size_t)slots[b] * heads + h;
    float* mm = m_all + head * (dv + 1);

    if (warp == warps) {
        // ---------------------------------------------------------------- the gates' warp
        float m = mm[j0];
        const float bi = gate_bias[h], bf = gate_bias[heads + h];
        float ri = 0.f, rf = 0.f;
        auto read = [&](int t0) {
            const bool ok = lane < kTT && t0 + lane < last;
            const float* g = gates + (size_t)(ok ? t0 + lane : first) * ld_gates;
            ri = ok ? g[h] : 0.f;
            rf = ok ? g[heads + h] : 0.f;
        };
        auto work = [&](int t0, int stage) {
            const float i = capped(ri + bi, cap), f = log_sigmoid_f(capped(rf + bf, cap));
            const int nt = min(kTT, last - t0);
            float m_before = 0.f, m_after = 0.f;
#pragma unroll
            for (int t = 0; t < kTT; ++t) {
                const float ft = __shfl_sync(0xffffffffu, f, t), it = __shfl_sync(0xffffffffu, i, t);
                const float next = t < nt ? fmaxf(ft + m, it) : m;
                if (lane == t) { m_before = m; m_after = next; }
                m = next;
            }
            if (lane < kTT)                        // a token beyond the last changes nothing
                sg[stage * kTT + lane] = lane < nt ? make_float4(expf(f + m_before - m_after), expf(i - m_after), expf(-m_after), m_after)
                                                   : make_float4(1.f, 0.f, 1.f, 0.f);
        };
        read(first);
        work(first, 0);
        read(first + kTT);
        __syncthreads();
        for (int t = 0; t < tiles; ++t) {
            if (t + 1 < tiles) {
                work(first + (t + 1) * kTT, (t + 1) & 1);
                read(first + (t + 2) * kTT);
            }
            __syncthreads();
        }
        for (int c = lane; c < cols; c += 32)
            if (j0 + c <= dv) mm[j0 + c] = m;
        return;
    }

    if (warp > warps) {
        // --------------------------------------------------------------- the helpers' warps
        const int tid = threadIdx.x - (warps + 1) * 32;
        constexpr int kPieces = 2 * kTT * (D / 8) / kHelpers;      // 8 elements each: k rows of the tile, then q rows
        constexpr int kValues = kTT * kMaxCols / kHelpers;
        uint4 raw[kPieces];
        T rv[kValues];
        // (token, column) of this thread's first value, and what the next one adds
        const int v_tt = tid / cols, v_c = tid % cols, v_dt = kHelpers / cols, v_dc = kHelpers % cols;
        auto fetch = [&](int t0) {
            int tt = v_tt, c = v_c;
#pragma unroll
            for (int e = 0; e < kValues; ++e) {
                if (tt < kTT) {
                    const int col = j0 + c;
                    rv[e] = (t0 + tt < last && col < dv) ? v[(size_t)(t0 + tt) * ld + (size_t)h * dv + col] : from_f32<T>(col == dv ? 1.f : 0.f);
                }
                tt += v_dt;
                c += v_dc;
                if (c >= cols) { c -= cols; ++tt; }
            }
            if constexpr (sizeof(T) == 2) {
                if (!vec) return;
#pragma unroll
                for (int e = 0; e < kPieces; ++e) {
                    const int idx = tid + e * kHelpers, which = idx / (kTT * (D / 8)), rest = idx % (kTT * (D / 8));
                    const int tt = rest / (D / 8), at = (rest % (D / 8)) * 8;
                    raw[e] = (t0 + tt < last && at < d) ? *reinterpret_cast<const uint4*>((which ? q : k) + (size_t)(t0 + tt) * ld + (size_t)h * d + at)
                                                        : make_uint4(0u, 0u, 0u, 0u);
                }
            }
        };
        auto store = [&](int t0, int stage) {
            float* dk = sk + stage * kTT * D;
            float* dq = sq + stage * kTT * D;
#pragma unroll
            for (int e = 0; e < kValues; ++e) {
                const int idx = tid + e * kHelpers;
                if (idx < kTT * cols) sv[stage * kTT * cols + idx] = to_f32<T>(rv[e]);
            }
            if constexpr (sizeof(T) == 2) {
                if (vec) {
#pragma unroll
                    for (int e = 0; e < kPieces; ++e) {
                        const int idx = tid + e * kHelpers, which = idx / (kTT * (D / 8)), rest = idx % (kTT * (D / 8));
                        float* dst = (which ? dq : dk) + rest * 8;
                        const float factor = which ? q_scale : 1.f;
                        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[e]);
                        const float2 a0 = __bfloat1622float2(h2[0]), a1 = __bfloat1622float2(h2[1]);
                        const float2 a2 = __bfloat1622float2(h2[2]), a3 = __bfloat1622float2(h2[3]);
                        reinterpret_cast<float4*>(dst)[0] = make_float4(a0.x * factor, a0.y * factor, a1.x * factor, a1.y * factor);
                        reinterpret_cast<float4*>(dst)[1] = make_float4(a2.x * factor, a2.y * factor, a3.x * factor, a3.y * factor);
                    }
                    return;
                }
            }
            for (int idx = tid; idx < kTT * D; idx += kHelpers) {
                const int tt = idx / D, at = idx % D;
                const bool ok = t0 + tt < last && at < d;
                const size_t where = ok ? (size_t)(t0 + tt) * ld + (size_t)h * d + at : 0;
                dk[idx] = ok ? to_f32<T>(k[where]) : 0.f;
                dq[idx] = ok ? to_f32<T>(q[where]) * q_scale : 0.f;
            }
        };
        auto show = [&](int t) {                   // tile t's results to memory
            const int t0 = first + t * kTT, nt = min(kTT, last - t0);
            int tt = v_tt, c = v_c;
            for (int idx = tid; idx < nt * cols; idx += kHelpers) {
                const size_t row = (size_t)(t0 + tt);
                const float x = sy[(t & 1) * kTT * cols + idx];
                if (j0 + c < dv) num[row * ld_num + (size_t)h * dv + j0 + c] = x;
                else if (j0 + c == dv) den[row * heads + h] = x;
                tt += v_dt;
                c += v_dc;
                if (c >= cols) { c -= cols; ++tt; }
            }
        };
        fetch(first);
        store(first, 0);
        if (tiles > 1) fetch(first + kTT);
        __syncthreads();
        for (int t = 0; t < tiles; ++t) {
            if (t + 1 < tiles) {
                store(first + (t + 1) * kTT, (t + 1) & 1);
                if (t + 2 < tiles) fetch(first + (t + 2) * kTT);
            }
            if (t > 0) show(t - 1);
            __syncthreads();
        }
        show(tiles - 1);
        return;
    }

    // ------------------------------------------------------------------ the columns' warps
    const int r = lane % RG, wc = warp * WC + lane / RG * kCP;       // the lane's rows, its first column within the slice
    float* S = S_all + head * d * dv;
    float* nn = n_all + head * d;
    f32x2 s[kCP][kKR / 2];
#pragma unroll
    for (int c = 0; c < kCP; ++c) {
        const int col = j0 + wc + c;
#pragma unroll
        for (int p = 0; p < kKR / 2; ++p) {
            float e[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = 2 * p + x, row = i / 4 * 4 * RG + r * 4 + i % 4;
                e[x] = (row < d && col < dv) ? S[(size_t)row * dv + col] : (row < d && col == dv) ? nn[row] : 0.f;
            }
            s[c][p] = pair_of(e[0], e[1]);
        }
    }
    __syncthreads();
    for (int t = 0; t < tiles; ++t) {
        const int stage = t & 1;
        const float* tk = sk + stage * kTT * D + r * 4;
        const float* tq = sq + stage * kTT * D + r * 4;
        const float* tv = sv + stage * kTT * cols + wc;
        const float4* tg = sg + stage * kTT;
#pragma unroll 1
        for (int t4 = 0; t4 < kTT; t4 += 4) {
            constexpr int kSums = 4 * kCP;
            float part[kSums];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float4 g = tg[t4 + u];
                const f32x2 keep = pair_of(g.x, g.x);
                f32x2 val[kCP], acc[kCP];
                float vv[kCP];
                *reinterpret_cast<float2*>(vv) = *reinterpret_cast<const float2*>(tv + (t4 + u) * cols);
#pragma unroll
                for (int c = 0; c < kCP; ++c) {
                    const float x = vv[c] * g.y;
                    val[c] = pair_of(x, x);
                    acc[c] = pair_of(0.f, 0.f);
                }
#pragma unroll
                for (int j = 0; j < kKR / 4; ++j) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(tk + (t4 + u) * D + j * 4 * RG);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(tq + (t4 + u) * D + j * 4 * RG);
#pragma unroll
                    for (int c = 0; c < kCP; ++c) {
                        s[c][2 * j] = fma2(keep, s[c][2 * j], mul2(kk.x, val[c]));
                        acc[c] = fma2(s[c][2 * j], qq.x, acc[c]);
                        s[c][2 * j + 1] = fma2(keep, s[c][2 * j + 1], mul2(kk.y, val[c]));
                        acc[c] = fma2(s[c][2 * j + 1], qq.y, acc[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < kCP; ++c) {
                    const float2 a = parts_of(acc[c]);
                    part[u * kCP + c] = a.x + a.y;
                }
            }
            // every exchange halves the sums a lane carries, while there are lanes and sums to halve: afterwards lane r
            // holds the sums whose number is r modulo kHalved, kSums / kHalved of them
            constexpr int kHalved = kSums < RG ? kSums : RG;
#pragma unroll
            for (int o = 1, left = kSums; o < kHalved; o <<= 1, left >>= 1) {
                const bool up = r & o;
#pragma unroll
                for (int i = 0; i < left / 2; ++i) {
                    const float mine = up ? part[2 * i + 1] : part[2 * i], theirs = up ? part[2 * i] : part[2 * i + 1];
                    part[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
                }
            }
#pragma unroll
            for (int o = kHalved; o < RG; o <<= 1) part[0] += __shfl_xor_sync(0xffffffffu, part[0], o);
            if (r < kHalved) {
#pragma unroll
                for (int i = 0; i < kSums / kHalved; ++i) {
                    const int number = i * kHalved + r, tt = t4 + number / kCP, c = wc + number % kCP;
                    float sum = part[i];
                    if (j0 + c == dv) sum = fmaxf(fabsf(sum), tg[tt].z) + 1e-6f;
                    sy[stage * kTT * cols + tt * cols + c] = sum;
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < kCP; ++c) {
        const int col = j0 + wc + c;
        if (col > dv) continue;
#pragma unroll
        for (int p = 0; p < kKR / 2; ++p) {
            const float2 e = parts_of(s[c][p]);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = 2 * p + x, row = i / 4 * 4 * RG + r * 4 + i % 4;
                if (row >= d) continue;
                if (col < dv) S[(size_t)row * dv + col] = x ? e.y : e.x;
                else nn[row] = x ? e.y : e.x;
            }
        }
    }
}

// --------------------------------------------- a step in which every sequence brings one token
// What costs is reading and writing the state once: one block per (head, slice of `cols`
// columns, sequence), a thread owns four neighbouring columns (16-byte accesses; a row of the
// slice is one contiguous run of the block's threads) for the rows rs, rs + RS, ...; the RS
// partial sums of a column meet in shared memory and are added in a fixed order.  Slice 0
// serves n as well.
constexpr int kStepThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kStepThreads)
mlstm_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int ld,
                  const float* __restrict__ gates, int ld_gates, const float* __restrict__ gate_bias, float cap, float q_scale,
                  float* __restrict__ S_all, float* __restrict__ n_all, float* __restrict__ m_all,
                  float* __restrict__ num, int ld_num, float* __restrict__ den,
                  const int* __restrict__ slots, int heads, int d, int dv, int cols, int slices) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float smem[];
    const int h = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
    const int tid = threadIdx.x;
    const int CG = cols / 4, RS = kStepThreads / CG;
    float* red = smem;                             // [RS][cols]
    float* sk = red + RS * cols;                   // [d]
    float* sq = sk + d;                            // [d]
    float* scratch = sq + d;                       // 33
    const size_t head = (size_t)slots[b] * heads + h;
    const int j0 = slice * cols;
    const int cg = tid % CG, rs = tid / CG;
    const bool live = rs < RS && j0 + 4 * cg < dv;
    const size_t row0 = (size_t)b * ld;
    for (int i = tid; i < d; i += kStepThreads) {
        sk[i] = to_f32<T>(k[row0 + (size_t)h * d + i]);
        sq[i] = to_f32<T>(q[row0 + (size_t)h * d + i]) * q_scale;
    }
    const float* g = gates + (size_t)b * ld_gates;
    const float ig = capped(g[h] + gate_bias[h], cap), fg = log_sigmoid_f(capped(g[heads + h] + gate_bias[heads + h], cap));
    float* mm = m_all + head * (dv + 1);
    const float m = mm[j0], m_new = fmaxf(fg + m, ig);
    const float keep = expf(fg + m - m_new), add = expf(ig - m_new);
    float4 val = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live) {
        const T* vp = v + row0 + (size_t)h * dv + j0 + 4 * cg;
        val = make_float4(to_f32<T>(vp[0]) * add, to_f32<T>(vp[1]) * add, to_f32<T>(vp[2]) * add, to_f32<T>(vp[3]) * add);
    }
    __syncthreads();                               // k and q stand; every thread has read the maximum
    if (live) {
        const size_t pitch = (size_t)dv / 4;
        float4* S = reinterpret_cast<float4*>(S_all + head * d * dv + j0) + cg;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        int row = rs;
        for (; row + 3 * RS < d; row += 4 * RS) {  // four rows in flight
            float4 s[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) s[u] = S[(size_t)(row + u * RS) * pitch];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float kk = sk[row + u * RS], qq = sq[row + u * RS];
                s[u].x = fmaf(keep, s[u].x, kk * val.x); s[u].y = fmaf(keep, s[u].y, kk * val.y);
                s[u].z = fmaf(keep, s[u].z, kk * val.z); s[u].w = fmaf(keep, s[u].w, kk * val.w);
                acc.x = fmaf(s[u].x, qq, acc.x); acc.y = fmaf(s[u].y, qq, acc.y);
                acc.z = fmaf(s[u].z, qq, acc.z); acc.w = fmaf(s[u].w, qq, acc.w);
                S[(size_t)(row + u * RS) * pitch] = s[u];
            }
        }
        for (; row < d; row += RS) {
            float4 s = S[(size_t)row * pitch];
            const float kk = sk[row], qq = sq[row];
            s.x = fmaf(keep, s.x, kk * val.x); s.y = fmaf(keep, s.y, kk * val.y);
            s.z = fmaf(keep, s.z, kk * val.z); s.w = fmaf(keep, s.w, kk * val.w);
            acc.x = fmaf(s.x, qq, acc.x); acc.y = fmaf(s.y, qq, acc.y);
            acc.z = fmaf(s.z, qq, acc.z); acc.w = fmaf(s.w, qq, acc.w);
            S[(size_t)row * pitch] = s;
        }
        *reinterpret_cast<float4*>(red + rs * cols + 4 * cg) = acc;
    }
    for (int c = tid; c < cols; c += kStepThreads)
        if (j0 + c < dv) mm[j0 + c] = m_new;
    if (slice == 0) {
        if (tid == 0) mm[dv] = m_new;
        float* nn = n_all + head * d;
        float part = 0.f;
        for (int i = tid; i < d; i += kStepThreads) {
            const float x = fmaf(keep, nn[i], sk[i] * add);
            nn[i] = x;
            part = fmaf(x, sq[i], part);
        }
        const float total = block_sum(part, scratch);
        if (tid == 0) den[(size_t)b * heads + h] = fmaxf(fabsf(total), expf(-m_new)) + 1e-6f;
    }
    __syncthreads();
    for (int c = tid; c < cols; c += kStepThreads) {
        if (j0 + c >= dv) continue;
        float sum = 0.f;
        for (int r = 0; r < RS; ++r) sum += red[r * cols + c];
        num[(size_t)b * ld_num + (size_t)h * dv + j0 + c] = sum;
    }
}

struct Args {
    const void *q, *k, *v; int ld; const float* gates; int ld_gates; const float* gate_bias; float cap, q_scale;
    float *S, *n, *m, *num; int ld_num; float* den; const int *cu_seqlens, *slots; int n_seqs, heads, d, dv; cudaStream_t stream;
};

// Measurements and tests may fix the warps of columns of a block (1, 2, 4 or 8); 0: the launcher chooses.
static int g_warps = 0;

template <typename T, int RG>
int launch_scan(const Args& a, int vec) {
    static int n_sm = 0;
    if (n_sm == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n_sm, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n_sm <= 0)
            n_sm = 148;
    }
    constexpr int D = RG * kKR, WC = 32 / RG * kCP;
    // as many warps a block as still give most multiprocessors a block (every block stages the head's k and q again); four
    // where those give every multiprocessor two and the staged rows are short (measured at heads of 128 x 256: eight prompts
    // 1,510 / 1,090 / 1,250 us at 2 / 4 / 8 warps, one prompt 246 / 277 / 424; heads of 256 x 512: eight prompts 6.1 / 4.9 /
    // 3.7 ms, one 881 / 662 / 477 us)
    const long long all = (long long)a.n_seqs * a.heads * ((a.dv + WC) / WC);        // warps of dv + 1 columns a head
    int warps = kMaxWarps;
    while (warps > 1 && all / warps < 4LL * n_sm / 5) warps /= 2;
    if (warps == 8 && RG <= 8 && all / 4 >= 2LL * n_sm) warps = 4;
    if (g_warps == 1 || g_warps == 2 || g_warps == 4 || g_warps == 8) warps = g_warps;
    while (warps * WC > kMaxCols) warps /= 2;
    const int cols = warps * WC, slices = (a.dv + cols) / cols;
    const size_t smem = (size_t)(4 * kTT * D + 4 * kTT * cols + 2 * kTT * 4) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<T, RG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return launch_chained(mlstm_scan_kernel<T, RG>, dim3(a.heads * slices, a.n_seqs), dim3((warps + 1) * 32 + kHelpers), smem, a.stream,
                          (const T*)a.q, (const T*)a.k, (const T*)a.v, a.ld, a.gates, a.ld_gates, a.gate_bias, a.cap, a.q_scale,
                          a.S, a.n, a.m, a.num, a.ld_num, a.den, a.cu_seqlens, a.slots, a.heads, a.d, a.dv, warps, slices, vec);
}

template <typename T>
int dispatch_scan(const Args& a, int vec) {
    if (a.d <= 64) return launch_scan<T, 4>(a, vec);
    if (a.d <= 128) return launch_scan<T, 8>(a, vec);
    if (a.d <= 256) return launch_scan<T, 16>(a, vec);
    return launch_scan<T, 32>(a, vec);
}
}  // namespace

GTG_API void gtg_mlstm_scan_shape(int warps) { g_warps = warps; }

// Most key channels a head may have.
GTG_API int gtg_mlstm_max_key_dim() { return 512; }

// q, k [n, heads * d] and v [n, heads * dv]: columns of one matrix of row stride ld, of the activation type
// (dtype 0 float, 1 bfloat16); gates float [n, i: heads | f: heads]; gate_bias float [2 heads]; S float
// [slots, heads, d, dv], n float [slots, heads, d], m float [slots, heads, dv + 1]; num float [n, heads * dv],
// den float [n, heads].  `one_token_each`: row b is sequence b's only token.
GTG_API int gtg_mlstm_scan(int dtype, const void* q, const void* k, const void* v, int ld, const float* gates, int ld_gates,
                           const float* gate_bias, float cap, float q_scale, float* S, float* n, float* m, float* num, int ld_num,
                           float* den, const int* cu_seqlens, const int* slots, int n_seqs, int heads, int d, int dv,
                           int one_token_each, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (heads <= 0 || d <= 0 || dv <= 0 || !(cap > 0.f)) return kErrBadArgument;
    if (ld < heads * d || ld < heads * dv || ld_gates < 2 * heads || ld_num < heads * dv) return kErrBadArgument;
    if (d > gtg_mlstm_max_key_dim() || n_seqs > 65535 || (long long)heads * (dv + 1) > 0x7fffffffLL) return kErrUnsupported;
    if (dtype != 0 && dtype != 1) return kErrBadArgument;
    const Args a{q, k, v, ld, gates, ld_gates, gate_bias, cap, q_scale, S, n, m, num, ld_num, den, cu_seqlens, slots, n_seqs, heads, d, dv, stream};
    if (one_token_each && dv % 4 == 0 && ((uintptr_t)S % 16) == 0) {
        int cols = 4;                              // the widest slice up to 128 columns that is a power of two
        while (cols < 128 && cols < dv) cols *= 2;
        const int slices = (dv + cols - 1) / cols;
        const size_t smem = (size_t)((kStepThreads / (cols / 4)) * cols + 2 * d + 36) * sizeof(float);
        const dim3 grid(heads * slices, n_seqs);
        if (dtype == 0)
            return launch_chained(mlstm_step_kernel<float>, grid, dim3(kStepThreads), smem, stream, (const float*)q, (const float*)k, (const float*)v,
                                  ld, gates, ld_gates, gate_bias, cap, q_scale, S, n, m, num, ld_num, den, slots, heads, d, dv, cols, slices);
        return launch_chained(mlstm_step_kernel<bf16>, grid, dim3(kStepThreads), smem, stream, (const bf16*)q, (const bf16*)k, (const bf16*)v,
                              ld, gates, ld_gates, gate_bias, cap, q_scale, S, n, m, num, ld_num, den, slots, heads, d, dv, cols, slices);
    }
    const int vec = dtype == 1 && d % 8 == 0 && ld % 8 == 0 && ((uintptr_t)q % 16) == 0 && ((uintptr_t)k % 16) == 0;
    return dtype == 0 ? dispatch_scan<float>(a, vec) : dispatch_scan<bf16>(a, vec);
}
