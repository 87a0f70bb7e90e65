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
//   step     a step in which every sequence brings one token;
//   chunks   bfloat16 prompts on the tensor cores, two kernels: `states` walks a sequence's chunks of
//            kChunk tokens and leaves the state each chunk starts from, `outputs` serves every tile of
//            tokens by itself from that state and the chunk's own keys and values.
#include "mma_helpers.cuh"
#include <math.h>

namespace {
// ---------------------------------------------------------------- token by token
// The columns of S never meet.  One block serves (head, a slice of columns, sequence); R lanes of a warp
// share a column, lane r owning rows r, r + R, ... (up to kRows of them) in registers; their partial sums
// meet by shuffles.  q, k and v of a tile of tokens at a time are staged in shared memory as floats.
// Tokens are walked strictly in order: the result does not depend on the cut of the sequence into steps, on
// the batch or on the slices.
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
// ---------------------------------------------------------------- prompts, chunk by chunk
// A sequence's tokens of the step are cut into chunks of kChunk, counted from its first row.  With S the state
// a chunk of L tokens starts from, and t, s its tokens counted from 0,
//
//     S' = a^L S + sum_s a^(L-1-s) k_s v_s^T,   o_t = a^(t+1) S^T q_t + sum_(s<=t) a^(t-s) (q_t . k_s) v_s.
//
// All products run on the warp-level tensor cores (mma.sync.m16n8k16, float sums).  q, k and v are bfloat16 and
// enter as they are; what is float and would have to be rounded (S, the scaled values, the decayed scores)
// enters as the sum of two bfloat16 numbers, which keeps 16 bits of it, by two products.
constexpr int kChunk = 128;
constexpr int kTileTokens = 64;
constexpr int kChunkThreads = 128;

__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = pack_bf16(x - f.x, y - f.y);
}
// where chunk 0 of sequence b lies among all sequences' chunks: no two sequences' chunks meet, and there are at most
// tokens / kChunk + sequences of them
__device__ __forceinline__ int first_chunk(int row0, int b) { return row0 / kChunk + b; }

// One block of four warps per (head, slice of NC columns of S, sequence) walks the chunks.  S lives in the
// accumulators: warp w owns rows [w DP/4, (w+1) DP/4).  A chunk's keys arrive one chunk ahead by asynchronous
// copies, its values one ahead in registers.  `chunks` receives, per chunk and head, the state it starts from
// as two planes of bfloat16 numbers [2][d][dv] whose sum it is.
template <int DP, int NC>
__global__ void __launch_bounds__(kChunkThreads)
lightning_states_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v, int ld, const float* __restrict__ decay,
                        float* __restrict__ state, bf16* __restrict__ chunks, const int* __restrict__ cu_seqlens,
                        const int* __restrict__ slots, int heads, int d, int dv, int slices) {
    chain_release();
    chain_wait();
    constexpr int MT = DP / 64, NT = NC / 8, KCPR = DP / 8, KTILE = kChunk * DP * 2, VTILE = kChunk * NC * 2;
    constexpr int kPieces = kChunk * (NC / 8) / kChunkThreads;     // 8 values each
    extern __shared__ __align__(128) unsigned char chunk_smem[];
    __shared__ float pw[kChunk + 1];                         // a^i
    const uint32_t sK = smem_u32(chunk_smem);                // two stages
    const uint32_t sV = sK + 2 * KTILE;                      // high part, low part
    const int h = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
    const int row0 = cu_seqlens[b], n_rows = cu_seqlens[b + 1] - row0;
    if (n_rows <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int j0 = slice * NC;
    const int n_chunks = (n_rows + kChunk - 1) / kChunk;
    float* S = state + ((size_t)slots[b] * heads + h) * (size_t)d * dv;
    for (int i = tid; i <= kChunk; i += kChunkThreads) pw[i] = powf(decay[h], (float)i);

    auto load_keys = [&](int stage, int c) {
        for (int id = tid; id < kChunk * KCPR; id += kChunkThreads) {
            const int r = id / KCPR, p = id % KCPR;
            const bool ok = c * kChunk + r < n_rows && p * 8 < d;
            cp_async16(sK + stage * KTILE + swz_offset<DP>(r, p), ok ? k + (size_t)(row0 + c * kChunk + r) * ld + (size_t)h * d + p * 8 : k, ok ? 16 : 0);
        }
        cp_async_commit();
    };
    uint4 raw[kPieces];
    auto load_values = [&](int c) {
#pragma unroll
        for (int e = 0; e < kPieces; ++e) {
            const int id = tid + e * kChunkThreads, r = id / (NC / 8), p = id % (NC / 8);
            const bool ok = c * kChunk + r < n_rows && j0 + p * 8 < dv;
            raw[e] = ok ? *reinterpret_cast<const uint4*>(v + (size_t)(row0 + c * kChunk + r) * ld + (size_t)h * dv + j0 + p * 8) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    load_keys(0, 0);
    load_values(0);
    float acc[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = (warp * MT + mt) * 16 + g + (e >> 1) * 8, col = j0 + nt * 8 + t4 * 2 + (e & 1);
                acc[mt][nt][e] = (row < d && col < dv) ? S[(size_t)row * dv + col] : 0.f;
            }
    __syncthreads();                                         // the powers stand
    const size_t plane = (size_t)d * dv;
    for (int c = 0; c < n_chunks; ++c) {
        const int L = min(kChunk, n_rows - c * kChunk);
        bf16* dst = chunks + ((size_t)(first_chunk(row0, b) + c) * heads + h) * 2 * plane;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int row = (warp * MT + mt) * 16 + g + r * 8, col = j0 + nt * 8 + t4 * 2;
                    if (row < d && col < dv) {
                        uint32_t hi, lo;
                        split_pair(acc[mt][nt][r * 2], acc[mt][nt][r * 2 + 1], hi, lo);
                        *reinterpret_cast<uint32_t*>(dst + (size_t)row * dv + col) = hi;
                        *reinterpret_cast<uint32_t*>(dst + plane + (size_t)row * dv + col) = lo;
                    }
                }
        // the chunk's values, scaled to the chunk's end
#pragma unroll
        for (int e = 0; e < kPieces; ++e) {
            const int id = tid + e * kChunkThreads, r = id / (NC / 8), p = id % (NC / 8);
            const float f = r < L ? pw[L - 1 - r] : 0.f;
            const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw[e]);
            uint4 hi, lo;
            uint32_t* hp = reinterpret_cast<uint32_t*>(&hi);
            uint32_t* lp = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 y = __bfloat1622float2(x[i]);
                split_pair(y.x * f, y.y * f, hp[i], lp[i]);
            }
            *reinterpret_cast<uint4*>(chunk_smem + 2 * KTILE + swz_offset<NC>(r, p)) = hi;
            *reinterpret_cast<uint4*>(chunk_smem + 2 * KTILE + VTILE + swz_offset<NC>(r, p)) = lo;
        }
        if (c + 1 < n_chunks) {
            load_keys((c + 1) & 1, c + 1);
            load_values(c + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const float keep = pw[L];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[mt][nt][e] *= keep;
        const uint32_t kb = sK + (c & 1) * KTILE;
#pragma unroll
        for (int kk = 0; kk < kChunk / 16; ++kk) {
            if (kk * 16 >= L) break;
            uint32_t bh[NT][2], bl[NT][2];
#pragma unroll
            for (int nn = 0; nn < NT / 2; ++nn) {
                const int r = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), p = nn * 2 + (lane >> 4);
                ldmatrix_x4_trans(bh[nn * 2][0], bh[nn * 2][1], bh[nn * 2 + 1][0], bh[nn * 2 + 1][1], sV + swz_offset<NC>(r, p));
                ldmatrix_x4_trans(bl[nn * 2][0], bl[nn * 2][1], bl[nn * 2 + 1][0], bl[nn * 2 + 1][1], sV + VTILE + swz_offset<NC>(r, p));
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                // K^T: rows of S are key channels, the product runs over tokens
                uint32_t a[4];
                const int r = kk * 16 + (lane >> 4) * 8 + (lane & 7), p = (warp * MT + mt) * 2 + ((lane >> 3) & 1);
                ldmatrix_x4_trans(a[0], a[1], a[2], a[3], kb + swz_offset<DP>(r, p));
#pragma unroll
                for (int nt = 0; nt < NT; ++nt) {
                    mma_bf16_16816(acc[mt][nt], a, bh[nt][0], bh[nt][1]);
                    mma_bf16_16816(acc[mt][nt], a, bl[nt][0], bl[nt][1]);
                }
            }
        }
        __syncthreads();                                     // the scaled values and this chunk's keys have been read
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = (warp * MT + mt) * 16 + g + (e >> 1) * 8, col = j0 + nt * 8 + t4 * 2 + (e & 1);
                if (row < d && col < dv) S[(size_t)row * dv + col] = acc[mt][nt][e];
            }
}

// One block of four warps per (tile of 64 tokens, head and slice of DVP columns, sequence), a warp sixteen tokens.
// Stages of 64 rows: first the state's DP / 64 (its two planes), then the chunk's key tiles up to the tokens' own
// (keys and values), double-buffered by asynchronous copies.
template <int DP, int DVP>
__global__ void __launch_bounds__(kChunkThreads)
lightning_outputs_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, int ld,
                         const float* __restrict__ decay, const bf16* __restrict__ chunks, float* __restrict__ out, int ld_out,
                         const int* __restrict__ cu_seqlens, int heads, int d, int dv, int slices) {
    chain_release();
    chain_wait();
    constexpr int QTILE = kTileTokens * DP * 2, XTILE = 64 * DVP * 2, YTILE = 64 * (DP > DVP ? DP : DVP) * 2, STAGE = XTILE + YTILE;
    constexpr int kStateStages = DP / 64;
    extern __shared__ __align__(128) unsigned char chunk_smem[];
    __shared__ float pw[kChunk + 1];
    const uint32_t sQ = smem_u32(chunk_smem), sX = sQ + QTILE;       // stage s at sX + s STAGE: [64][DVP], then [64][DP or DVP]
    const int b = blockIdx.z, h = blockIdx.y / slices, j0 = blockIdx.y % slices * DVP;
    const int row0 = cu_seqlens[b], n_rows = cu_seqlens[b + 1] - row0;
    const int tile0 = blockIdx.x * kTileTokens;
    if (tile0 >= n_rows) return;
    const int chunk = tile0 / kChunk, inside = tile0 % kChunk / kTileTokens;      // which tile of its chunk
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    for (int i = tid; i <= kChunk; i += kChunkThreads) pw[i] = powf(decay[h], (float)i);
    const size_t plane = (size_t)d * dv;
    const bf16* S = chunks + ((size_t)(first_chunk(row0, b) + chunk) * heads + h) * 2 * plane;

    for (int id = tid; id < kTileTokens * (DP / 8); id += kChunkThreads) {
        const int r = id / (DP / 8), p = id % (DP / 8);
        const bool ok = tile0 + r < n_rows && p * 8 < d;
        cp_async16(sQ + swz_offset<DP>(r, p), ok ? q + (size_t)(row0 + tile0 + r) * ld + (size_t)h * d + p * 8 : q, ok ? 16 : 0);
    }
    auto load_stage = [&](int i) {
        const uint32_t x = sX + (i & 1) * STAGE, y = x + XTILE;
        if (i < kStateStages) {
            for (int id = tid; id < 64 * (DVP / 8); id += kChunkThreads) {
                const int r = id / (DVP / 8), p = id % (DVP / 8), row = i * 64 + r;
                const bool ok = row < d && j0 + p * 8 < dv;
                const size_t at = ok ? (size_t)row * dv + j0 + p * 8 : 0;
                cp_async16(x + swz_offset<DVP>(r, p), S + at, ok ? 16 : 0);
                cp_async16(y + swz_offset<DVP>(r, p), S + plane + at, ok ? 16 : 0);
            }
        } else {
            const int first = chunk * kChunk + (i - kStateStages) * 64;
            for (int id = tid; id < 64 * (DVP / 8); id += kChunkThreads) {
                const int r = id / (DVP / 8), p = id % (DVP / 8);
                const bool ok = first + r < n_rows && j0 + p * 8 < dv;
                cp_async16(x + swz_offset<DVP>(r, p), ok ? v + (size_t)(row0 + first + r) * ld + (size_t)h * dv + j0 + p * 8 : v, ok ? 16 : 0);
            }
            for (int id = tid; id < 64 * (DP / 8); id += kChunkThreads) {
                const int r = id / (DP / 8), p = id % (DP / 8);
                const bool ok = first + r < n_rows && p * 8 < d;
                cp_async16(y + swz_offset<DP>(r, p), ok ? k + (size_t)(row0 + first + r) * ld + (size_t)h * d + p * 8 : k, ok ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    load_stage(0);                                           // its group holds the queries too
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    auto q_fragment = [&](int kk, uint32_t* a) {
        const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, p = kk * 2 + (lane >> 4);
        ldmatrix_x4(a[0], a[1], a[2], a[3], sQ + swz_offset<DP>(r, p));
    };
    auto multiply = [&](const uint32_t* a, uint32_t tile, int kk) {       // o += a . rows [16 kk, 16 kk + 16) of a tile of DVP columns
#pragma unroll
        for (int dd = 0; dd < DVP / 16; ++dd) {
            uint32_t b0, b1, b2, b3;
            const int r = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), p = dd * 2 + (lane >> 4);
            ldmatrix_x4_trans(b0, b1, b2, b3, tile + swz_offset<DVP>(r, p));
            mma_bf16_16816(o[dd * 2], a, b0, b1);
            mma_bf16_16816(o[dd * 2 + 1], a, b2, b3);
        }
    };
    const int t_row[2] = {inside * 64 + warp * 16 + g, inside * 64 + warp * 16 + g + 8};       // this thread's two tokens, within the chunk
    const int n_stages = kStateStages + inside + 1;
    for (int i = 0; i < n_stages; ++i) {
        if (i + 1 < n_stages) {
            load_stage(i + 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t x = sX + (i & 1) * STAGE, y = x + XTILE;
        if (i < kStateStages) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t a[4];
                q_fragment(i * 4 + kk, a);
                multiply(a, x, kk);
                multiply(a, y, kk);
            }
            if (i == kStateStages - 1) {
                const float f0 = pw[t_row[0] + 1], f1 = pw[t_row[1] + 1];
#pragma unroll
                for (int n = 0; n < DVP / 8; ++n) { o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1; }
            }
        } else {
            float s[8][4];
#pragma unroll
            for (int n = 0; n < 8; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
#pragma unroll
            for (int kk = 0; kk < DP / 16; ++kk) {
                uint32_t a[4];
                q_fragment(kk, a);
#pragma unroll
                for (int jj = 0; jj < 4; ++jj) {
                    uint32_t b0, b1, b2, b3;
                    const int r = jj * 16 + (lane & 7) + (lane >> 4) * 8, p = kk * 2 + ((lane >> 3) & 1);
                    ldmatrix_x4(b0, b1, b2, b3, y + swz_offset<DP>(r, p));
                    mma_bf16_16816(s[jj * 2], a, b0, b1);
                    mma_bf16_16816(s[jj * 2 + 1], a, b2, b3);
                }
            }
            const int key0 = (i - kStateStages) * 64;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int half = 0; half < 2; ++half)         // keys 8 half .. of the sixteen
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const int n = 2 * kk + half, back = t_row[r] - (key0 + n * 8 + t4 * 2);
                        const float s0 = back >= 0 ? s[n][r * 2] * pw[back] : 0.f, s1 = back >= 1 ? s[n][r * 2 + 1] * pw[back - 1] : 0.f;
                        split_pair(s0, s1, hi[half * 2 + r], lo[half * 2 + r]);
                    }
                multiply(hi, x, kk);
                multiply(lo, x, kk);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int t = tile0 + warp * 16 + g + r * 8;
        if (t >= n_rows) continue;
        float* dst = out + (size_t)(row0 + t) * ld_out + (size_t)h * dv + j0 + t4 * 2;
#pragma unroll
        for (int n = 0; n < DVP / 8; ++n)
            if (j0 + n * 8 < dv) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][r * 2], o[n][r * 2 + 1]);
    }
}

struct ChunkArgs {
    const bf16 *q, *k, *v; int ld; const float* decay; float* state; bf16* chunks; float* out; int ld_out;
    const int *cu_seqlens, *slots; int n_seqs, max_q_len, heads, d, dv; cudaStream_t stream;
};

template <int DP, int NC>
int launch_states(const ChunkArgs& a) {
    const int slices = (a.dv + NC - 1) / NC;
    constexpr int smem = 2 * kChunk * DP * 2 + 2 * kChunk * NC * 2;
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(lightning_states_kernel<DP, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_chained(lightning_states_kernel<DP, NC>, dim3(a.heads * slices, a.n_seqs), dim3(kChunkThreads), smem, a.stream, a.k, a.v, a.ld,
                          a.decay, a.state, a.chunks, a.cu_seqlens, a.slots, a.heads, a.d, a.dv, slices);
}

template <int DP, int DVP>
int launch_outputs(const ChunkArgs& a) {
    const int slices = (a.dv + DVP - 1) / DVP;
    constexpr int smem = kTileTokens * DP * 2 + 2 * (64 * DVP * 2 + 64 * (DP > DVP ? DP : DVP) * 2);
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(lightning_outputs_kernel<DP, DVP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_chained(lightning_outputs_kernel<DP, DVP>, dim3((a.max_q_len + kTileTokens - 1) / kTileTokens, a.heads * slices, a.n_seqs),
                          dim3(kChunkThreads), smem, a.stream, a.q, a.k, a.v, a.ld, a.decay, (const bf16*)a.chunks, a.out, a.ld_out, a.cu_seqlens,
                          a.heads, a.d, a.dv, slices);
}

template <int DP>
int run_chunks(const ChunkArgs& a) {
    // sixteen columns a block of `states` where blocks of 32 would leave multiprocessors idle
    const int st = (long long)a.n_seqs * a.heads * ((a.dv + 31) / 32) < 148 ? launch_states<DP, 16>(a) : launch_states<DP, 32>(a);
    if (st != 0) return st;
    return a.dv <= 64 ? launch_outputs<DP, 64>(a) : launch_outputs<DP, 128>(a);
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

// bfloat16 values that `gtg_lightning_chunks` needs beside its operands for so many tokens and sequences.
GTG_API long long gtg_lightning_chunk_values(int n_tokens, int n_seqs, int heads, int d, int dv) {
    return ((long long)n_tokens / kChunk + n_seqs) * heads * 2 * d * dv;
}
GTG_API int gtg_lightning_chunks_supports(int d, int dv) { return d > 0 && d % 8 == 0 && d <= 256 && dv > 0 && dv % 8 == 0; }

// The recurrence of bfloat16 prompts chunk by chunk; arguments as in gtg_lightning_scan; `chunks`:
// gtg_lightning_chunk_values bfloat16 values.
GTG_API int gtg_lightning_chunks(const void* q, const void* k, const void* v, int ld, const float* decay, float* state, void* chunks,
                                 float* out, int ld_out, const int* cu_seqlens, const int* slots, int n_seqs, int max_q_len, int heads,
                                 int d, int dv, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return 0;
    if (heads <= 0 || ld < heads * d || ld < heads * dv || ld_out < heads * dv || !chunks) return kErrBadArgument;
    if (!gtg_lightning_chunks_supports(d, dv)) return kErrUnsupported;
    if (ld % 8 || ld_out % 2 || ((uintptr_t)q % 16) || ((uintptr_t)k % 16) || ((uintptr_t)v % 16) || ((uintptr_t)out % 8) || ((uintptr_t)chunks % 16))
        return kErrUnsupported;
    if (n_seqs > 65535 || (long long)heads * ((dv + 63) / 64) > 65535) return kErrUnsupported;
    const ChunkArgs a{(const bf16*)q, (const bf16*)k, (const bf16*)v, ld, decay, state, (bf16*)chunks, out, ld_out, cu_seqlens, slots, n_seqs,
                      max_q_len, heads, d, dv, stream};
    return d <= 64 ? run_chunks<64>(a) : d <= 128 ? run_chunks<128>(a) : run_chunks<256>(a);
}
