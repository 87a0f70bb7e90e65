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
// One block per (head, slice of columns, sequence).  A warp serves CP neighbouring columns
// over all rows: lane l owns KR rows in runs of V = min(KR, 4), rows V (l + 32 j) .. + V,
// so that k and q of a token arrive by 8- or 16-byte reads from shared memory (rows beyond
// d are zeros there).  Tiles of kTT tokens are staged as floats, the loads of the next tile
// in flight meanwhile; a warp of its own works out the gates of the tile ahead.  The sums of
// four tokens and CP columns meet in one butterfly in which every exchange halves what a
// lane still carries.  Tokens are walked strictly in order: the result does not depend on
// the cut of the sequence into steps, on the batch or on the slices.
constexpr int kTT = 16;
constexpr int kMaxWarps = 8;

template <typename T, int KR, int CP>
__global__ void __launch_bounds__((kMaxWarps + 1) * 32)
mlstm_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int ld,
                  const float* __restrict__ gates, int ld_gates, const float* __restrict__ gate_bias, float cap, float q_scale,
                  float* __restrict__ S_all, float* __restrict__ n_all, float* __restrict__ m_all,
                  float* __restrict__ num, int ld_num, float* __restrict__ den,
                  const int* __restrict__ cu_seqlens, const int* __restrict__ slots, int heads, int d, int dv, int slices, int vec) {
    chain_release();
    chain_wait();
    constexpr int D = 32 * KR, V = KR < 4 ? KR : 4, P = KR / 2;
    extern __shared__ __align__(16) float smem[];
    const int warps = (blockDim.x >> 5) - 1, cols = warps * CP, threads = warps * 32;
    float* sk = smem;                              // [kTT][D]
    float* sq = sk + kTT * D;                      // [kTT][D]
    float* sv = sq + kTT * D;                      // [kTT][cols], times the token's input factor
    float* sy = sv + kTT * cols;                   // [kTT][cols]
    float4* sg = reinterpret_cast<float4*>(sy + kTT * cols);     // two tiles of [kTT] (keep, add, exp(-m), m)
    const int h = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
    const int first = cu_seqlens[b], last = cu_seqlens[b + 1];
    if (first >= last) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int j0 = slice * cols;                   // the block's first column
    const size_t head = (size_t)slots[b] * heads + h;
    float* S = S_all + head * d * dv;
    float* nn = n_all + head * d;
    float* mm = m_all + head * (dv + 1);

    if (warp == warps) {
        // ---------------------------------------------------------------- the gates' warp
        float m = mm[j0];
        const float bi = gate_bias[h], bf = gate_bias[heads + h];
        auto read = [&](int t0, float& ri, float& rf) {
            const bool ok = lane < kTT && t0 + lane < last;
            const float* g = gates + (size_t)(ok ? t0 + lane : first) * ld_gates;
            ri = ok ? g[h] : 0.f;
            rf = ok ? g[heads + h] : 0.f;
        };
        auto work = [&](int t0, int stage, float ri, float rf) {
            const float i = capped(ri + bi, cap), f = log_sigmoid_f(capped(rf + bf, cap));
            const int nt = min(kTT, last - t0);
            float m_before = 0.f, m_after = 0.f;
            for (int t = 0; t < nt; ++t) {
                const float ft = __shfl_sync(0xffffffffu, f, t), it = __shfl_sync(0xffffffffu, i, t);
                const float next = fmaxf(ft + m, it);
                if (lane == t) { m_before = m; m_after = next; }
                m = next;
            }
            if (lane < kTT)                        // a token beyond the last changes nothing
                sg[stage * kTT + lane] = lane < nt ? make_float4(expf(f + m_before - m_after), expf(i - m_after), expf(-m_after), m_after)
                                                   : make_float4(1.f, 0.f, 1.f, 0.f);
        };
        float ri, rf;
        read(first, ri, rf);
        work(first, 0, ri, rf);
        int stage = 0;
        read(first + kTT, ri, rf);
        for (int t0 = first; t0 < last; t0 += kTT, stage ^= 1) {
            __syncthreads();                       // (1) the tile before has been computed; this tile's gates stand
            __syncthreads();                       // (2) this tile is staged
            if (t0 + kTT < last) {
                work(t0 + kTT, stage ^ 1, ri, rf);
                read(t0 + 2 * kTT, ri, rf);
            }
        }
        for (int c = lane; c < cols; c += 32)
            if (j0 + c <= dv) mm[j0 + c] = m;
        return;
    }

    // ------------------------------------------------------------------ the columns' warps
    const int wc = warp * CP;                      // the warp's first column within the slice
    f32x2 s[CP][P];
#pragma unroll
    for (int c = 0; c < CP; ++c) {
        const int col = j0 + wc + c;
#pragma unroll
        for (int p = 0; p < P; ++p) {
            float e[2];
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = 2 * p + x, row = (i / V) * 32 * V + lane * V + i % V;
                e[x] = (row < d && col < dv) ? S[(size_t)row * dv + col] : (row < d && col == dv) ? nn[row] : 0.f;
            }
            s[c][p] = pair_of(e[0], e[1]);
        }
    }
    // staging by pieces of 8 elements (16 bytes of bfloat16): piece e of this thread is number tid + e threads
    // of the tile's k rows, then of its q rows
    constexpr int kMaxPieces = 2 * kTT * D / 8 / 128;        // (with four warps; half of them with eight)
    uint4 raw[kMaxPieces];
    T rv[CP / 2];                                  // the tile's values: kTT cols of them over all threads
    auto fetch = [&](int t0) {
#pragma unroll
        for (int e = 0; e < CP / 2; ++e) {
            const int idx = tid + e * threads, tt = idx / cols, col = j0 + idx % cols;
            rv[e] = (t0 + tt < last && col < dv) ? v[(size_t)(t0 + tt) * ld + (size_t)h * dv + col]
                                                 : from_f32<T>(t0 + tt < last && col == dv ? 1.f : 0.f);
        }
        if constexpr (sizeof(T) == 2) {
            if (!vec) return;
#pragma unroll
            for (int e = 0; e < kMaxPieces; ++e) {
                const int idx = tid + e * threads;
                raw[e] = make_uint4(0u, 0u, 0u, 0u);
                if (idx >= 2 * kTT * (D / 8)) continue;
                const int which = idx / (kTT * (D / 8)), rest = idx % (kTT * (D / 8));
                const int tt = rest / (D / 8), at = (rest % (D / 8)) * 8;
                if (t0 + tt < last && at < d)
                    raw[e] = *reinterpret_cast<const uint4*>((which ? q : k) + (size_t)(t0 + tt) * ld + (size_t)h * d + at);
            }
        }
    };
    fetch(first);
    int stage = 0, shown = first, shown_n = 0;     // the tile whose results lie in sy
    auto show = [&]() {
        for (int idx = tid; idx < shown_n * cols; idx += threads) {
            const int tt = idx / cols, c = idx % cols;
            const size_t row = (size_t)(shown + tt);
            if (j0 + c < dv) num[row * ld_num + (size_t)h * dv + j0 + c] = sy[idx];
            else if (j0 + c == dv) den[row * heads + h] = sy[idx];
        }
    };
    for (int t0 = first; t0 < last; t0 += kTT, stage ^= 1) {
        const int nt = min(kTT, last - t0);
        __syncthreads();                           // (1)
        show();
        if constexpr (sizeof(T) == 2) {
            if (vec) {
#pragma unroll
                for (int e = 0; e < kMaxPieces; ++e) {
                    const int idx = tid + e * threads;
                    if (idx >= 2 * kTT * (D / 8)) continue;
                    const int which = idx / (kTT * (D / 8)), rest = idx % (kTT * (D / 8));
                    float* dst = (which ? sq : sk) + rest * 8;
                    const float factor = which ? q_scale : 1.f;
                    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[e]);
                    const float2 a = __bfloat1622float2(h2[0]), bb = __bfloat1622float2(h2[1]);
                    const float2 c = __bfloat1622float2(h2[2]), dd = __bfloat1622float2(h2[3]);
                    reinterpret_cast<float4*>(dst)[0] = make_float4(a.x * factor, a.y * factor, bb.x * factor, bb.y * factor);
                    reinterpret_cast<float4*>(dst)[1] = make_float4(c.x * factor, c.y * factor, dd.x * factor, dd.y * factor);
                }
            }
        }
        if (sizeof(T) == 4 || !vec) {
            for (int idx = tid; idx < kTT * D; idx += threads) {
                const int tt = idx / D, at = idx % D;
                const bool ok = tt < nt && at < d;
                const size_t where = ok ? (size_t)(t0 + tt) * ld + (size_t)h * d + at : 0;
                sk[idx] = ok ? to_f32<T>(k[where]) : 0.f;
                sq[idx] = ok ? to_f32<T>(q[where]) * q_scale : 0.f;
            }
        }
#pragma unroll
        for (int e = 0; e < CP / 2; ++e) {
            const int idx = tid + e * threads;
            sv[idx] = to_f32<T>(rv[e]) * sg[stage * kTT + idx / cols].y;
        }
        __syncthreads();                           // (2)
        if (t0 + kTT < last) fetch(t0 + kTT);
        for (int tq = 0; tq < nt; tq += 4) {
            float part[4 * CP];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float keep = sg[stage * kTT + tq + u].x;
                const f32x2 keep2 = pair_of(keep, keep);
                f32x2 val[CP], acc[CP];
#pragma unroll
                for (int c = 0; c < CP; ++c) {
                    const float x = sv[(tq + u) * cols + wc + c];
                    val[c] = pair_of(x, x);
                    acc[c] = pair_of(0.f, 0.f);
                }
#pragma unroll
                for (int run = 0; run < KR / V; ++run) {
                    f32x2 kk[V / 2], qq[V / 2];
                    const int at = (tq + u) * D + run * 32 * V + lane * V;
                    if constexpr (V == 4) {
                        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(sk + at), e = *reinterpret_cast<const ulonglong2*>(sq + at);
                        kk[0] = a.x; kk[1] = a.y; qq[0] = e.x; qq[1] = e.y;
                    } else {
                        kk[0] = *reinterpret_cast<const f32x2*>(sk + at);
                        qq[0] = *reinterpret_cast<const f32x2*>(sq + at);
                    }
#pragma unroll
                    for (int p = 0; p < V / 2; ++p) {
#pragma unroll
                        for (int c = 0; c < CP; ++c) {
                            f32x2& x = s[c][run * (V / 2) + p];
                            x = fma2(keep2, x, mul2(kk[p], val[c]));
                            acc[c] = fma2(x, qq[p], acc[c]);
                        }
                    }
                }
#pragma unroll
                for (int c = 0; c < CP; ++c) {
                    const float2 a = parts_of(acc[c]);
                    part[u * CP + c] = a.x + a.y;
                }
            }
            // every exchange halves the sums a lane carries: after log2(4 CP) of them lane l holds number l mod (4 CP)
            int o = 1;
#pragma unroll
            for (int left = 4 * CP; left > 1; left >>= 1, o <<= 1) {
                const bool up = lane & o;
#pragma unroll
                for (int i = 0; i < left / 2; ++i) {
                    const float mine = up ? part[2 * i + 1] : part[2 * i], theirs = up ? part[2 * i] : part[2 * i + 1];
                    part[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
                }
            }
            float sum = part[0];
#pragma unroll
            for (int o2 = 4 * CP; o2 < 32; o2 <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o2);
            if (lane < 4 * CP) {
                const int tt = tq + lane / CP, c = wc + lane % CP;
                if (j0 + c == dv) sum = fmaxf(fabsf(sum), sg[stage * kTT + tt].z) + 1e-6f;
                sy[tt * cols + c] = sum;
            }
        }
        shown = t0;
        shown_n = nt;
    }
    // the last tile's results: only the columns' warps still run, and they meet at a barrier of their own
    asm volatile("bar.sync 1, %0;\n" ::"r"(threads) : "memory");
    show();
#pragma unroll
    for (int c = 0; c < CP; ++c) {
        const int col = j0 + wc + c;
        if (col > dv) continue;
#pragma unroll
        for (int p = 0; p < P; ++p) {
            const float2 e = parts_of(s[c][p]);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int i = 2 * p + x, row = (i / V) * 32 * V + lane * V + i % V;
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

template <typename T, int KR, int CP>
int launch_scan(const Args& a, int warps, int vec) {
    const int cols = warps * CP, slices = (a.dv + cols) / cols;              // dv + 1 columns
    const size_t smem = (size_t)(2 * kTT * 32 * KR + 2 * kTT * cols + 2 * kTT * 4) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<T, KR, CP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return launch_chained(mlstm_scan_kernel<T, KR, CP>, dim3(a.heads * slices, a.n_seqs), dim3((warps + 1) * 32), smem, a.stream,
                          (const T*)a.q, (const T*)a.k, (const T*)a.v, a.ld, a.gates, a.ld_gates, a.gate_bias, a.cap, a.q_scale,
                          a.S, a.n, a.m, a.num, a.ld_num, a.den, a.cu_seqlens, a.slots, a.heads, a.d, a.dv, slices, vec);
}

// Measurements may fix the warps of a block (4 or 8) and the columns of a warp (2 or 4); 0: the launcher chooses.
static int g_warps = 0, g_columns = 0;

template <typename T>
int dispatch_scan(const Args& a, int vec) {
    static int n_sm = 0;
    if (n_sm == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n_sm, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n_sm <= 0)
            n_sm = 148;
    }
    // wide blocks (every block stages the head's k and q again) while they still give each multiprocessor one
    const long long columns = (long long)a.n_seqs * a.heads * a.dv;
    int cp = columns / 32 >= 4LL * n_sm / 5 ? 4 : 2, warps = columns / (8 * cp) >= 4LL * n_sm / 5 ? 8 : 4;
    if (g_warps == 4 || g_warps == 8) warps = g_warps;
    if (g_columns == 2 || g_columns == 4) cp = g_columns;
    if (a.d <= 64) return cp == 4 ? launch_scan<T, 2, 4>(a, warps, vec) : launch_scan<T, 2, 2>(a, warps, vec);
    if (a.d <= 128) return cp == 4 ? launch_scan<T, 4, 4>(a, warps, vec) : launch_scan<T, 4, 2>(a, warps, vec);
    if (a.d <= 256) return cp == 4 ? launch_scan<T, 8, 4>(a, warps, vec) : launch_scan<T, 8, 2>(a, warps, vec);
    return launch_scan<T, 16, 2>(a, warps, vec);
}
}  // namespace

GTG_API void gtg_mlstm_scan_shape(int warps, int columns) { g_warps = warps; g_columns = columns; }

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
