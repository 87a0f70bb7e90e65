// Kernels of linear attention with a fixed decay per head (lightning attention): a recurrent mixer whose
// per-sequence state is, per head, a matrix S of d x dv floats,
//
//     S_t = a S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   S zero at the start,
//
// a the head's decay, a number of the model.  They serve a step of packed rows: sequence b owns rows
// cu_seqlens[b]..cu_seqlens[b+1], continues from the state kept for its cache slot and leaves the state for
// its next step; a prompt, a portion of one and a single token are the same case.  q, k and v are of the
// activation type; the state, the decays and the sums are float.
//
//   scan     token by token, any size and either type;
//   step     a step in which every sequence brings one token.
#include "mma_helpers.cuh"
#include <math.h>

namespace {
// ---------------------------------------------------------------- token by token
// The columns of S never meet.  One block serves (head, a slice of columns, sequence); R lanes of a warp
// share a column, lane r owning rows r, r + R, ... (up to kRows of them) in registers; their partial sums
// meet by shuffles.  q, k and v of a tile of tokens at a time are staged in shared memory as floats.
// Tokens are walked strictly in order: the result does
// not depend on the cut of the sequence into steps, on the batch or on the slices.
constexpr int kRows = 16;
constexpr int kScanThreads = 128;
constexpr int kTile = 8;

template <typename T>
__global__ void __launch_bounds__(kScanThreads)
lightning_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int ld,
                      const float* __restrict__ decay, float* __restrict__ state, float* __restrict__ out, int ld_out,
                      const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
                      int heads, int d, int dv, int R, int slices) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float smem[];
    const int cols = kScanThreads / R;
    float* sq = smem;                                        // [kTile][d]
    float* sk = sq + kTile * d;
    float* sv = sk + kTile * d;                              // [kTile][cols]
    const int h = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
    const int row0 = cu_seqlens[b], n_rows = cu_seqlens[b + 1] - row0;
    if (n_rows <= 0) return;
    const int tid = threadIdx.x, r = tid % R, jj = tid / R;
    const int j = slice * cols + jj;
    const bool col_ok = j < dv;
    const float a = decay[h];
    float* S = state + ((size_t)slots[b] * heads + h) * (size_t)d * dv;
    float s[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
        const int row = r + i * R;
        s[i] = (col_ok && row < d) ? S[(size_t)row * dv + j] : 0.f;
    }
    for (int t0 = 0; t0 < n_rows; t0 += kTile) {
        const int nt = min(kTile, n_rows - t0);
        for (int idx = tid; idx < nt * d; idx += kScanThreads) {
            const int t = idx / d, i = idx - t * d;
            const size_t at = (size_t)(row0 + t0 + t) * ld + (size_t)h * d + i;
            sq[idx] = to_f32<T>(q[at]);
            sk[idx] = to_f32<T>(k[at]);
        }
        for (int idx = tid; idx < nt * cols; idx += kScanThreads) {
            const int t = idx / cols, c = idx - t * cols;
            const int col = slice * cols + c;
            sv[idx] = col < dv ? to_f32<T>(v[(size_t)(row0 + t0 + t) * ld + (size_t)h * dv + col]) : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float* kt = sk + t * d;
            const float* qt = sq + t * d;
            const float vt = sv[t * cols + jj];
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < kRows; ++i) {
                const int row = r + i * R;
                if (row < d) {
                    s[i] = fmaf(a, s[i], kt[row] * vt);
                    acc = fmaf(s[i], qt[row], acc);
                }
            }
            for (int o = 1; o < R; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (r == 0 && col_ok) out[(size_t)(row0 + t0 + t) * ld_out + (size_t)h * dv + j] = acc;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
        const int row = r + i * R;
        if (col_ok && row < d) S[(size_t)row * dv + j] = s[i];
    }
}

// ------------------------------------------- a step in which every sequence brings one token
// What costs is reading and writing the state once: one block per (head, slice of `cols` columns,
// sequence), a thread owns four neighbouring columns (16-byte accesses; a row of the slice is one
// contiguous run of the block's threads) for the rows rs, rs + RS, ...; the RS partial sums of a column
// meet in shared memory and are added in a fixed order.
constexpr int kStepThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kStepThreads)
lightning_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int ld,
                      const float* __restrict__ decay, float* __restrict__ state, float* __restrict__ out, int ld_out,
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
    const int j0 = slice * cols;
    const int cg = tid % CG, rs = tid / CG;
    const bool live = j0 + 4 * cg < dv;
    const size_t row0 = (size_t)b * ld;
    for (int i = tid; i < d; i += kStepThreads) {
        sk[i] = to_f32<T>(k[row0 + (size_t)h * d + i]);
        sq[i] = to_f32<T>(q[row0 + (size_t)h * d + i]);
    }
    const float a = decay[h];
    float4 val = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live) {
        const T* vp = v + row0 + (size_t)h * dv + j0 + 4 * cg;
        val = make_float4(to_f32<T>(vp[0]), to_f32<T>(vp[1]), to_f32<T>(vp[2]), to_f32<T>(vp[3]));
    }
    __syncthreads();
    if (live) {
        const size_t pitch = (size_t)dv / 4;
        float4* S = reinterpret_cast<float4*>(state + ((size_t)slots[b] * heads + h) * d * dv + j0) + cg;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        auto advance = [&](float4& s, int row) {
            const float kk = sk[row], qq = sq[row];
            s.x = fmaf(a, s.x, kk * val.x); s.y = fmaf(a, s.y, kk * val.y);
            s.z = fmaf(a, s.z, kk * val.z); s.w = fmaf(a, s.w, kk * val.w);
            acc.x = fmaf(s.x, qq, acc.x); acc.y = fmaf(s.y, qq, acc.y);
            acc.z = fmaf(s.z, qq, acc.z); acc.w = fmaf(s.w, qq, acc.w);
            S[(size_t)row * pitch] = s;
        };
        int row = rs;
        for (; row + 7 * RS < d; row += 8 * RS) {  // eight rows in flight
            float4 s[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) s[u] = S[(size_t)(row + u * RS) * pitch];
#pragma unroll
            for (int u = 0; u < 8; ++u) advance(s[u], row + u * RS);
        }
        for (; row < d; row += RS) {
            float4 s = S[(size_t)row * pitch];
            advance(s, row);
        }
        *reinterpret_cast<float4*>(red + rs * cols + 4 * cg) = acc;
    }
    __syncthreads();
    for (int c = tid; c < cols; c += kStepThreads) {
        if (j0 + c >= dv) continue;
        float sum = 0.f;
        for (int r = 0; r < RS; ++r) sum += red[r * cols + c];
        out[(size_t)b * ld_out + (size_t)h * dv + j0 + c] = sum;
    }
}
}  // namespace

// Most key channels a head may have.
GTG_API int gtg_lightning_max_key_dim() { return 32 * kRows; }

// q, k [n, heads * d] and v [n, heads * dv]: columns of one matrix of row stride ld, of the activation type
// (dtype 0 float, 1 bfloat16); decay float [heads]; state float [slots, heads, d, dv]; out float
// [n, heads * dv].  `one_token_each`: row b is sequence b's only token.
GTG_API int gtg_lightning_scan(int dtype, const void* q, const void* k, const void* v, int ld, const float* decay, float* state,
                               float* out, int ld_out, const int* cu_seqlens, const int* slots, int n_seqs, int heads, int d,
                               int dv, int one_token_each, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (heads <= 0 || d <= 0 || dv <= 0 || ld < heads * d || ld < heads * dv || ld_out < heads * dv) return kErrBadArgument;
    if (dtype != 0 && dtype != 1) return kErrBadArgument;
    if (d > gtg_lightning_max_key_dim() || n_seqs > 65535 || (long long)heads * dv > 0x7fffffffLL) return kErrUnsupported;
#define GTG_LIGHTNING(KERNEL, T, ...)                                                                                \
    return launch_chained(KERNEL<T>, grid, dim3(threads), smem, stream, (const T*)q, (const T*)k, (const T*)v, ld, decay, state, out, \
                          ld_out, __VA_ARGS__)
    if (one_token_each && dv % 4 == 0 && ((uintptr_t)state % 16) == 0) {
        int cols = 4;                              // the widest slice up to 128 columns that is a power of two
        while (cols < 128 && cols < dv) cols *= 2;
        const int slices = (dv + cols - 1) / cols, threads = kStepThreads;
        const size_t smem = (size_t)((kStepThreads / (cols / 4)) * cols + 2 * d) * sizeof(float);
        const dim3 grid(heads * slices, n_seqs);
        if (dtype == 0) GTG_LIGHTNING(lightning_step_kernel, float, slots, heads, d, dv, cols, slices);
        GTG_LIGHTNING(lightning_step_kernel, bf16, slots, heads, d, dv, cols, slices);
    }
    int R = 1;                                     // lanes a column: the fewest that leave a lane at most kRows rows
    while (R < 32 && (d + R - 1) / R > kRows) R *= 2;
    const int cols = kScanThreads / R, slices = (dv + cols - 1) / cols, threads = kScanThreads;
    const size_t smem = (size_t)kTile * (2 * d + cols) * sizeof(float);
    const dim3 grid(heads * slices, n_seqs);
    if (dtype == 0) GTG_LIGHTNING(lightning_scan_kernel, float, cu_seqlens, slots, heads, d, dv, R, slices);
    GTG_LIGHTNING(lightning_scan_kernel, bf16, cu_seqlens, slots, heads, d, dv, R, slices);
#undef GTG_LIGHTNING
}
