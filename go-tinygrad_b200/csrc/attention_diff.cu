// Differential attention over the paged cache: every query and key head has two parts ("maps") side by
// side, each pair of parts is a causal softmax attention of its own over the same values, and with a1 and
// a2 the two maps' outputs a head's output is
//
//     o = a1 - lambda a2,   out = o / sqrt(mean(o^2) + eps) * out_scale
//
// the mean over the head's vd channels.  Cache rows: a key row holds both maps, 2 d channels; a value row
// vd.  Query head h reads key/value head h / (n_heads / n_kv).  The token at position p sees the keys
// lo(p)..p of its own sequence, lo(p) = max(0, p - window + 1) (window 0: all of them).  Scores, weights,
// both outputs, their difference and the norm are float; in bfloat16 the weights are rounded for their
// product with the values.
//
// Two kernels: a plain one (a warp per token and head; either type, any width) and one on the warp-level
// tensor cores for bfloat16.  Both serve prompts, portions of one and decode steps.
#include "mma_helpers.cuh"
#include <math.h>

namespace {
// ---------------------------------------------------------------- the plain kernel
// Keys are walked 32 at a time from lo: the result for a (token, head) depends on nothing but its own
// keys, not on the batch, not on how the tokens were cut into steps.
constexpr int kWarps = 4;

// PER: value channels a lane (vd <= 32 PER)
template <typename T, int PER>
__global__ void __launch_bounds__(kWarps * 32)
attention_diff_simple_kernel(const T* __restrict__ q, int ldq, T* __restrict__ out, int ldo,
                             const T* __restrict__ kc, const T* __restrict__ vc, long long page_stride,
                             const int* __restrict__ block_table, int table_stride,
                             const int* __restrict__ token_seq, const int* __restrict__ slots,
                             const int* __restrict__ positions, int N, int n_heads, int n_kv, int d, int vd,
                             float scale, int window, float lambda, float out_scale, float eps) {
    chain_release();
    chain_wait();
    extern __shared__ float rows_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long wid = (long long)blockIdx.x * kWarps + warp;
    if (wid >= (long long)N * n_heads) return;
    const int n = (int)(wid / n_heads), h = (int)(wid % n_heads);
    const int kvh = h / (n_heads / n_kv);
    const int pos = positions[n];
    const int* table = block_table + (size_t)slots[token_seq[n]] * table_stride;
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;

    float* qs = rows_smem + warp * 2 * d;
    for (int i = lane; i < 2 * d; i += 32) qs[i] = to_f32<T>(q[(size_t)n * ldq + (size_t)h * 2 * d + i]);
    __syncwarp();

    float acc[2][PER], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < PER; ++j) acc[0][j] = acc[1][j] = 0.f;
    for (int t0 = lo; t0 <= pos; t0 += 32) {
        const int t = t0 + lane;
        const bool valid = t <= pos;
        int page = 0;
        float score[2] = {-INFINITY, -INFINITY};
        if (valid) {
            page = table[t / kPageTokens];
            const T* kp = kc + (size_t)page * page_stride + ((size_t)kvh * kPageTokens + (t % kPageTokens)) * 2 * d;
#pragma unroll
            for (int map = 0; map < 2; ++map) {
                float s = 0.f;
                for (int i = 0; i < d; ++i) s = fmaf(qs[map * d + i], to_f32<T>(kp[map * d + i]), s);
                score[map] = s * scale;
            }
        }
        float p[2];
#pragma unroll
        for (int map = 0; map < 2; ++map) {
            const float m_new = fmaxf(m[map], warp_max(score[map]));
            p[map] = valid ? expf(score[map] - m_new) : 0.f;
            const float corr = expf(m[map] - m_new);         // 0 on the first keys (m = -inf)
            l[map] = l[map] * corr + warp_sum(p[map]);
#pragma unroll
            for (int j = 0; j < PER; ++j) acc[map][j] *= corr;
            m[map] = m_new;
        }
        const int count = min(32, pos - t0 + 1);
        for (int src = 0; src < count; ++src) {
            const float p1 = __shfl_sync(0xffffffffu, p[0], src), p2 = __shfl_sync(0xffffffffu, p[1], src);
            const int pg = __shfl_sync(0xffffffffu, page, src);
            const T* vp = vc + (size_t)pg * page_stride + ((size_t)kvh * kPageTokens + ((t0 + src) % kPageTokens)) * vd;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int c = lane + 32 * j;
                if (c < vd) {
                    const float v = to_f32<T>(vp[c]);
                    acc[0][j] = fmaf(p1, v, acc[0][j]);
                    acc[1][j] = fmaf(p2, v, acc[1][j]);
                }
            }
        }
    }
    const float f1 = 1.0f / l[0], f2 = lambda / l[1];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        if (lane + 32 * j < vd) {
            acc[0][j] = acc[0][j] * f1 - acc[1][j] * f2;
            ss = fmaf(acc[0][j], acc[0][j], ss);
        }
    }
    const float inv = out_scale / sqrtf(warp_sum(ss) / (float)vd + eps);
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = lane + 32 * j;
        if (c < vd) out[(size_t)n * ldo + (size_t)h * vd + c] = from_f32<T>(acc[0][j] * inv);
    }
}

// ---------------------------------------------------------------- warp-level tensor cores
// Rows are (token, query head of the group) pairs: all query heads that share a key/value head meet the
// same keys, so a block of 64 rows reads every page once for the group and for both maps.  One block of
// eight warps per (64-row tile, key/value head, sequence) and, for steps that bring few rows (decode), per
// share of the pages the tile sees (`n_splits`): warps 0-3 compute map 1 of the rows (sixteen each), warps
// 4-7 map 2.  At the end map 2's warps leave their part in shared memory and map 1's combine, norm and
// store; a share instead leaves both maps' unnormalised outputs with their maxima and sums, and the merge
// kernel does the rest in a fixed order.  Scores are exponentiated with exp2 on log2(e)-scaled values.
// Key rows of 2 d and value rows of vd channels (d and vd multiples of 8) are zero-padded in shared memory
// to two tiles of DKP and one of DVP channels.
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kTileRows = 64;
constexpr int kThreads = 256;

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ int first_seen(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }

template <int DKP, int DVP>
constexpr int diff_smem_bytes() {
    return 6 * kTileRows * DKP * 2 + 2 * kTileRows * DVP * 2;    // queries of both maps, two stages of keys and values
}

template <int DKP, int DVP>
__global__ void __launch_bounds__(kThreads)
attention_diff_mma_kernel(const bf16* __restrict__ q, int ldq, bf16* __restrict__ out, int ldo,
                          const bf16* __restrict__ kc, const bf16* __restrict__ vc, long long page_stride,
                          const int* __restrict__ block_table, int table_stride,
                          const int* __restrict__ cu_seqlens, const int* __restrict__ slots, const int* __restrict__ start_pos,
                          int n_heads, int n_kv, int d, int vd, float scale, int window,
                          float lambda, float out_scale, float eps, int n_splits,
                          float* __restrict__ part_o, float* __restrict__ part_ml) {
    chain_release();
    chain_wait();
    constexpr int KCPR = DKP / 8, VCPR = DVP / 8;          // 16-byte pieces per staged row
    constexpr int KTILE = kTileRows * DKP * 2, VTILE = kTileRows * DVP * 2;
    constexpr int OPITCH = DVP + 4;                        // floats per row of map 2's output
    extern __shared__ __align__(128) unsigned char smem[];
    const uint32_t sQ = smem_u32(smem);                    // [map]
    const uint32_t sK = sQ + 2 * KTILE;                    // [stage][map]
    const uint32_t sV = sK + 4 * KTILE;                    // [stage]

    const int b = blockIdx.z, kvh = blockIdx.y;
    // the longest tiles first
    const int n_tiles = gridDim.x / n_splits;
    const int tile = n_tiles - 1 - blockIdx.x / n_splits, split = blockIdx.x % n_splits;
    const int group = n_heads / n_kv;
    const int q_begin = cu_seqlens[b];
    const int q_len = cu_seqlens[b + 1] - q_begin;
    const int n_rows = q_len * group;                      // (token, head of the group) pairs of this sequence
    if (tile * kTileRows >= n_rows) return;
    const int start = start_pos[b];
    const int* table = block_table + (size_t)slots[b] * table_stride;
    const int tid = threadIdx.x, map = tid >> 7, warp = (tid >> 5) & 3, lane = tid & 31;
    const int g = lane >> 2, t4 = lane & 3;

    const int rows_here = min(kTileRows, n_rows - tile * kTileRows);
    const int tok_first = (tile * kTileRows) / group, tok_last = (tile * kTileRows + rows_here - 1) / group;
    const int kv_total = start + q_len;                    // keys that exist after this step
    const int p_first = first_seen(start + tok_first, window) / kPageTokens, p_last = (start + tok_last) / kPageTokens;
    const int per_split = (p_last - p_first + n_splits) / n_splits;
    const int j_lo = p_first + split * per_split;
    const int j_hi = min(p_last, j_lo + per_split - 1);

    // this thread's two rows of the warp's sixteen
    int row_tok[2], row_head[2], row_pos[2];
    bool row_ok[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = warp * 16 + g + r * 8;
        row_ok[r] = row < rows_here;
        const int rr = tile * kTileRows + (row_ok[r] ? row : rows_here - 1);
        row_tok[r] = rr / group;
        row_head[r] = kvh * group + rr % group;
        row_pos[r] = start + row_tok[r];
    }
    auto part_index = [&](int r) { return (((size_t)(q_begin + row_tok[r]) * n_heads + row_head[r]) * 2 + map) * n_splits + split; };
    if (j_lo > j_hi) {
        // nothing of this tile falls to this share: say so (the merge passes over it)
        if (t4 == 0) {
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                if (!row_ok[r]) continue;
                part_ml[part_index(r) * 2] = -INFINITY;
                part_ml[part_index(r) * 2 + 1] = 0.f;
            }
        }
        return;
    }

    // ---- stage the query rows of both maps, then page by page the keys and values
    for (int id = tid; id < 2 * kTileRows * KCPR; id += kThreads) {
        const int mp = id / (kTileRows * KCPR), r = id / KCPR % kTileRows, c = id % KCPR;
        const bool ok = r < rows_here && c * 8 < d;
        const int rr = tile * kTileRows + r;
        const bf16* src = ok ? q + (size_t)(q_begin + rr / group) * ldq + (size_t)(kvh * group + rr % group) * 2 * d + mp * d + c * 8 : q;
        cp_async16(sQ + mp * KTILE + swz_offset<DKP>(r, c), src, ok ? 16 : 0);
    }
    auto load_kv = [&](int stage, int j) {
        const size_t page = (size_t)table[j] * page_stride;
        const size_t kbase = page + (size_t)kvh * kPageTokens * 2 * d, vbase = page + (size_t)kvh * kPageTokens * vd;
        for (int id = tid; id < 2 * kTileRows * KCPR; id += kThreads) {
            const int r = id / (2 * KCPR), mp = id / KCPR % 2, c = id % KCPR;
            const bool ok = (j * kPageTokens + r) < kv_total && c * 8 < d;
            cp_async16(sK + (stage * 2 + mp) * KTILE + swz_offset<DKP>(r, c), kc + (ok ? kbase + (size_t)r * 2 * d + mp * d + c * 8 : 0), ok ? 16 : 0);
        }
        for (int id = tid; id < kTileRows * VCPR; id += kThreads) {
            const int r = id / VCPR, c = id % VCPR;
            const bool ok = (j * kPageTokens + r) < kv_total && c * 8 < vd;
            cp_async16(sV + stage * VTILE + swz_offset<DVP>(r, c), vc + (ok ? vbase + (size_t)r * vd + c * 8 : 0), ok ? 16 : 0);
        }
    };
    load_kv(0, j_lo);
    cp_async_commit();

    uint32_t qf[DKP / 16][4];
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    float m_row[2] = {-INFINITY, -INFINITY};   // running max of scaled scores (log2 domain)
    float l_row[2] = {0.f, 0.f};               // this thread's share of the running sum
    const float s_in = scale * kLog2e;
    const int w_first = tile * kTileRows + warp * 16, w_last = min(w_first + 15, tile * kTileRows + rows_here - 1);
    const int warp_pos_lo = start + w_first / group;
    const int warp_seen_hi = w_last >= w_first ? first_seen(start + w_last / group, window) : 0;
    const bool warp_live = warp * 16 < rows_here;          // a warp none of whose rows exists stages pages and computes nothing
    for (int j = j_lo, it = 0; j <= j_hi; ++j, ++it) {
        const int stage = it & 1;
        if (j + 1 <= j_hi) {
            load_kv(stage ^ 1, j + 1);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        if (warp_live) {
            if (it == 0) {
#pragma unroll
                for (int kk = 0; kk < DKP / 16; ++kk) {
                    const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                    const int c = kk * 2 + (lane >> 4);
                    ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], sQ + map * KTILE + swz_offset<DKP>(r, c));
                }
            }
            // ---- S = Q K^T of this warp's map and 16 rows with the page's 64 keys
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
            const uint32_t kbase = sK + (stage * 2 + map) * KTILE, vbase = sV + stage * VTILE;
#pragma unroll
            for (int kk = 0; kk < DKP / 16; ++kk) {
#pragma unroll
                for (int jj = 0; jj < 4; ++jj) {
                    uint32_t b0, b1, b2, b3;
                    const int r = jj * 16 + (lane & 7) + (lane >> 4) * 8;
                    const int c = kk * 2 + ((lane >> 3) & 1);
                    ldmatrix_x4(b0, b1, b2, b3, kbase + swz_offset<DKP>(r, c));
                    mma_bf16_16816(s[jj * 2], qf[kk], b0, b1);
                    mma_bf16_16816(s[jj * 2 + 1], qf[kk], b2, b3);
                }
            }
            // ---- mask by position (only pages that cross an edge for some row of this warp)
            const bool all_visible = (j * kPageTokens + kPageTokens - 1 <= warp_pos_lo) && (j * kPageTokens >= warp_seen_hi);
            if (!all_visible) {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int key = j * kPageTokens + i * 8 + t4 * 2 + (e & 1);
                        const int r = e >> 1;
                        if (key > row_pos[r] || key < first_seen(row_pos[r], window)) s[i][e] = -INFINITY;
                    }
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
#pragma unroll
                for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
            }
            float corr[2], m_use[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float m_new = fmaxf(m_row[r], mx[r] * s_in);         // scale > 0: max commutes with it
                m_use[r] = m_new == -INFINITY ? 0.f : m_new;
                corr[r] = fast_exp2(m_row[r] - m_use[r]);
                m_row[r] = m_new;
                l_row[r] *= corr[r];
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float p = fast_exp2(fmaf(s[i][e], s_in, -m_use[e >> 1]));
                    s[i][e] = p;
                    l_row[e >> 1] += p;
                }
            }
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) {
                o[i][0] *= corr[0]; o[i][1] *= corr[0];
                o[i][2] *= corr[1]; o[i][3] *= corr[1];
            }
            // ---- O += P V
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t pa[4];
                pa[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
                pa[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
                pa[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
                pa[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
                for (int dd = 0; dd < DVP / 16; ++dd) {
                    uint32_t b0, b1, b2, b3;
                    const int r = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
                    const int c = dd * 2 + (lane >> 4);
                    ldmatrix_x4_trans(b0, b1, b2, b3, vbase + swz_offset<DVP>(r, c));
                    mma_bf16_16816(o[dd * 2], pa, b0, b1);
                    mma_bf16_16816(o[dd * 2 + 1], pa, b2, b3);
                }
            }
        }
        __syncthreads();
    }

    // ---- the rows' sums; then this share of the output, or the combination of the two maps
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 1);
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 2);
    }
    if (n_splits > 1) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            if (!row_ok[r]) continue;
            const size_t pidx = part_index(r);
            float* po = part_o + pidx * DVP;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i)
                *reinterpret_cast<float2*>(po + i * 8 + t4 * 2) = make_float2(o[i][r * 2], o[i][r * 2 + 1]);
            if (t4 == 0) { part_ml[pidx * 2] = m_row[r]; part_ml[pidx * 2 + 1] = l_row[r]; }
        }
        return;
    }
    float* second = reinterpret_cast<float*>(smem);        // [64][OPITCH]; the pages have been read
    if (map == 1) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float f = l_row[r] > 0.f ? lambda / l_row[r] : 0.f;
            float* dst = second + (warp * 16 + g + r * 8) * OPITCH + t4 * 2;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[i][r * 2] * f, o[i][r * 2 + 1] * f);
        }
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const float f = l_row[r] > 0.f ? 1.0f / l_row[r] : 0.f;
        const float* src = second + (warp * 16 + g + r * 8) * OPITCH + t4 * 2;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) {                // channels beyond vd are zero in both
            const float2 b2 = *reinterpret_cast<const float2*>(src + i * 8);
            const float x = o[i][r * 2] * f - b2.x, y = o[i][r * 2 + 1] * f - b2.y;
            o[i][r * 2] = x;
            o[i][r * 2 + 1] = y;
            ss = fmaf(x, x, fmaf(y, y, ss));
        }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if (!row_ok[r]) continue;
        const float inv = out_scale / sqrtf(ss / (float)vd + eps);
        bf16* dst = out + (size_t)(q_begin + row_tok[r]) * ldo + (size_t)row_head[r] * vd + t4 * 2;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i)
            if (i * 8 + t4 * 2 < vd)
                *reinterpret_cast<__nv_bfloat162*>(dst + i * 8) = __floats2bfloat162_rn(o[i][r * 2] * inv, o[i][r * 2 + 1] * inv);
    }
}

// ---------------------------------------------------------------- decode steps
// A step in which every sequence brings one token: the (head of the group) rows of a block are at most sixteen, one
// fragment, so the eight warps share the page instead: warp (map, quarter) scores its map's rows against the page's keys
// 16 quarter .. + 16 and keeps a running maximum, sum and output of its own; nothing meets across warps until the last
// page.  One block per (share of the pages, key/value head, sequence); pages arrive kRing - 1 ahead.  At the end the four
// quarters of a map are added up in order, scaled to their common maximum.
constexpr int kRing = 3;

template <int DKP, int DVP>
constexpr int diff_decode_smem_bytes() {
    constexpr int ring = kRing * kTileRows * (2 * DKP + DVP) * 2, parts = 8 * 16 * (DVP + 4) * 4 + 8 * 16 * 8;
    return 2 * 16 * DKP * 2 + (ring > parts ? ring : parts);
}

template <int DKP, int DVP>
__global__ void __launch_bounds__(kThreads, DVP > 128 ? 1 : 2)
attention_diff_decode_kernel(const bf16* __restrict__ q, int ldq, bf16* __restrict__ out, int ldo,
                             const bf16* __restrict__ kc, const bf16* __restrict__ vc, long long page_stride,
                             const int* __restrict__ block_table, int table_stride,
                             const int* __restrict__ slots, const int* __restrict__ start_pos,
                             int n_heads, int n_kv, int d, int vd, float scale, int window,
                             float lambda, float out_scale, float eps, int n_splits,
                             float* __restrict__ part_o, float* __restrict__ part_ml) {
    chain_release();
    chain_wait();
    constexpr int KCPR = DKP / 8, VCPR = DVP / 8;
    constexpr int KTILE = kTileRows * DKP * 2, STAGE = 2 * KTILE + kTileRows * DVP * 2, QTILE = 16 * DKP * 2;
    constexpr int OPITCH = DVP + 4;
    extern __shared__ __align__(128) unsigned char smem[];
    const uint32_t sQ = smem_u32(smem);                    // [map]
    const uint32_t sR = sQ + 2 * QTILE;                    // [stage]: keys of both maps, values
    const int b = blockIdx.z, kvh = blockIdx.y, split = blockIdx.x;
    const int group = n_heads / n_kv, pos = start_pos[b];
    const int* table = block_table + (size_t)slots[b] * table_stride;
    const int tid = threadIdx.x, warp = tid >> 5, map = warp >> 2, quarter = warp & 3, lane = tid & 31;
    const int g = lane >> 2, t4 = lane & 3;
    const int lo = first_seen(pos, window);
    const int p_first = lo / kPageTokens, p_last = pos / kPageTokens;
    const int per_split = (p_last - p_first + n_splits) / n_splits;
    const int j_lo = p_first + split * per_split;
    const int j_hi = min(p_last, j_lo + per_split - 1);
    const size_t th0 = (size_t)b * n_heads + kvh * group;  // (token, head) of row 0
    if (j_lo > j_hi) {
        if (tid < 2 * group) {
            const size_t pidx = ((th0 + tid % group) * 2 + tid / group) * n_splits + split;
            part_ml[pidx * 2] = -INFINITY;
            part_ml[pidx * 2 + 1] = 0.f;
        }
        return;
    }
    for (int id = tid; id < 2 * 16 * KCPR; id += kThreads) {
        const int mp = id / (16 * KCPR), r = id / KCPR % 16, c = id % KCPR;
        const bool ok = r < group && c * 8 < d;
        cp_async16(sQ + mp * QTILE + swz_offset<DKP>(r, c), ok ? q + (size_t)b * ldq + (size_t)(kvh * group + r) * 2 * d + mp * d + c * 8 : q, ok ? 16 : 0);
    }
    auto load_page = [&](int stage, int j) {
        const size_t page = (size_t)table[j] * page_stride;
        const size_t kbase = page + (size_t)kvh * kPageTokens * 2 * d, vbase = page + (size_t)kvh * kPageTokens * vd;
        const uint32_t sK = sR + stage * STAGE, sV = sK + 2 * KTILE;
        for (int id = tid; id < 2 * kTileRows * KCPR; id += kThreads) {
            const int r = id / (2 * KCPR), mp = id / KCPR % 2, c = id % KCPR;
            const bool ok = j * kPageTokens + r <= pos && c * 8 < d;
            cp_async16(sK + mp * KTILE + swz_offset<DKP>(r, c), kc + (ok ? kbase + (size_t)r * 2 * d + mp * d + c * 8 : 0), ok ? 16 : 0);
        }
        for (int id = tid; id < kTileRows * VCPR; id += kThreads) {
            const int r = id / VCPR, c = id % VCPR;
            const bool ok = j * kPageTokens + r <= pos && c * 8 < vd;
            cp_async16(sV + swz_offset<DVP>(r, c), vc + (ok ? vbase + (size_t)r * vd + c * 8 : 0), ok ? 16 : 0);
        }
    };
#pragma unroll
    for (int s = 0; s < kRing - 1; ++s) {                  // the first group holds the queries too; empty groups keep the count
        if (j_lo + s <= j_hi) load_page(s, j_lo + s);
        cp_async_commit();
    }
    uint32_t qf[DKP / 16][4];
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
    float m_row[2] = {-INFINITY, -INFINITY}, l_row[2] = {0.f, 0.f};
    const float s_in = scale * kLog2e;
    for (int j = j_lo, it = 0; j <= j_hi; ++j, ++it) {
        cp_async_wait<kRing - 2>();
        __syncthreads();                                   // this page stands; the page before it has been read
        if (j + kRing - 1 <= j_hi) load_page((it + kRing - 1) % kRing, j + kRing - 1);
        cp_async_commit();
        if (it == 0) {
#pragma unroll
            for (int kk = 0; kk < DKP / 16; ++kk) {
                const int r = (lane & 7) + ((lane >> 3) & 1) * 8, c = kk * 2 + (lane >> 4);
                ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], sQ + map * QTILE + swz_offset<DKP>(r, c));
            }
        }
        const int key0 = j * kPageTokens + quarter * 16;
        if (key0 > pos || key0 + 15 < lo) continue;        // none of the warp's sixteen keys is seen
        const uint32_t kbase = sR + (it % kRing) * STAGE + map * KTILE, vbase = sR + (it % kRing) * STAGE + 2 * KTILE;
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
#pragma unroll
        for (int kk = 0; kk < DKP / 16; ++kk) {
            uint32_t b0, b1, b2, b3;
            const int r = quarter * 16 + (lane & 7) + (lane >> 4) * 8, c = kk * 2 + ((lane >> 3) & 1);
            ldmatrix_x4(b0, b1, b2, b3, kbase + swz_offset<DKP>(r, c));
            mma_bf16_16816(s[0], qf[kk], b0, b1);
            mma_bf16_16816(s[1], qf[kk], b2, b3);
        }
        if (key0 + 15 > pos || key0 < lo) {
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = key0 + i * 8 + t4 * 2 + (e & 1);
                    if (key > pos || key < lo) s[i][e] = -INFINITY;
                }
        }
        float corr[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float mx = fmaxf(fmaxf(s[0][r * 2], s[0][r * 2 + 1]), fmaxf(s[1][r * 2], s[1][r * 2 + 1]));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_new = fmaxf(m_row[r], mx * s_in);        // finite: at least one of the keys is seen
            corr[r] = fast_exp2(m_row[r] - m_new);
            m_row[r] = m_new;
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float p = fast_exp2(fmaf(s[i][r * 2 + e], s_in, -m_new));
                    s[i][r * 2 + e] = p;
                    sum += p;
                }
            l_row[r] = l_row[r] * corr[r] + sum;
        }
        const uint32_t pa[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
        for (int dd = 0; dd < DVP / 16; ++dd) {
            uint32_t b0, b1, b2, b3;
            const int r = quarter * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), c = dd * 2 + (lane >> 4);
            ldmatrix_x4_trans(b0, b1, b2, b3, vbase + swz_offset<DVP>(r, c));
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                float* oo = o[dd * 2 + x];
                oo[0] *= corr[0]; oo[1] *= corr[0]; oo[2] *= corr[1]; oo[3] *= corr[1];
            }
            mma_bf16_16816(o[dd * 2], pa, b0, b1);
            mma_bf16_16816(o[dd * 2 + 1], pa, b2, b3);
        }
    }
    cp_async_wait<0>();
    __syncthreads();                                       // the ring has been read: its place takes the warps' parts
    float* po = reinterpret_cast<float*>(smem + 2 * QTILE);                // [warp][16][OPITCH]
    float2* pml = reinterpret_cast<float2*>(po + 8 * 16 * OPITCH);         // [warp][16]
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 1);
        l_row[r] += __shfl_xor_sync(0xffffffffu, l_row[r], 2);
        const int row = g + r * 8;
        if (row >= group) continue;
        float* dst = po + (warp * 16 + row) * OPITCH + t4 * 2;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[i][r * 2], o[i][r * 2 + 1]);
        if (t4 == 0) pml[warp * 16 + row] = make_float2(m_row[r], l_row[r]);
    }
    __syncthreads();
    // a warp a row: the quarters of both maps, then the share or the finished head
    for (int row = warp; row < group; row += 8) {
        float f[2][4], M[2], L[2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            M[mp] = -INFINITY;
            L[mp] = 0.f;
#pragma unroll
            for (int k = 0; k < 4; ++k) M[mp] = fmaxf(M[mp], pml[(mp * 4 + k) * 16 + row].x);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 ml = pml[(mp * 4 + k) * 16 + row];
                f[mp][k] = ml.x == -INFINITY ? 0.f : exp2f(ml.x - M[mp]);
                L[mp] += f[mp][k] * ml.y;
            }
        }
        const size_t th = th0 + row;
        constexpr int PER = DVP / 32;
        float a[2][PER];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp)
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                a[mp][i] = 0.f;
#pragma unroll
                for (int k = 0; k < 4; ++k) a[mp][i] = fmaf(f[mp][k], po[((mp * 4 + k) * 16 + row) * OPITCH + lane + 32 * i], a[mp][i]);
            }
        if (n_splits > 1) {
#pragma unroll
            for (int mp = 0; mp < 2; ++mp) {
                const size_t pidx = (th * 2 + mp) * n_splits + split;
#pragma unroll
                for (int i = 0; i < PER; ++i) part_o[pidx * DVP + lane + 32 * i] = a[mp][i];
                if (lane == 0) { part_ml[pidx * 2] = M[mp]; part_ml[pidx * 2 + 1] = L[mp]; }
            }
            continue;
        }
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            a[0][i] = a[0][i] / L[0] - lambda * (a[1][i] / L[1]);
            ss = fmaf(a[0][i], a[0][i], ss);
        }
        const float inv = out_scale / sqrtf(warp_sum(ss) / (float)vd + eps);
        bf16* dst = out + (size_t)b * ldo + (size_t)(kvh * group + row) * vd;
#pragma unroll
        for (int i = 0; i < PER; ++i)
            if (lane + 32 * i < vd) dst[lane + 32 * i] = __float2bfloat16_rn(a[0][i] * inv);
    }
}

// One block per (token, query head), a thread per channel: each map's shares in order, scaled to their
// common maximum; then the difference and its norm.
__global__ void attention_diff_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                            bf16* __restrict__ out, int ldo, int n_heads, int vd, int dvp, int n_splits,
                                            float lambda, float out_scale, float eps) {
    chain_release();
    chain_wait();
    __shared__ float scratch[33];
    const size_t th = blockIdx.x;
    const int n = (int)(th / n_heads), h = (int)(th % n_heads), c = threadIdx.x;
    float a[2];
#pragma unroll
    for (int map = 0; map < 2; ++map) {
        const size_t base = (th * 2 + map) * n_splits;
        float M = -INFINITY;
        for (int s = 0; s < n_splits; ++s) M = fmaxf(M, part_ml[(base + s) * 2]);
        const float Mu = M == -INFINITY ? 0.f : M;
        float acc = 0.f, L = 0.f;
        for (int s = 0; s < n_splits; ++s) {
            const float m = part_ml[(base + s) * 2];
            if (m == -INFINITY) continue;                  // a share without keys wrote no output
            const float f = exp2f(m - Mu);
            if (c < vd) acc += f * part_o[(base + s) * dvp + c];
            L += f * part_ml[(base + s) * 2 + 1];
        }
        a[map] = L > 0.f ? acc / L : 0.f;
    }
    const float o = a[0] - lambda * a[1];
    const float inv = out_scale / sqrtf(block_sum(o * o, scratch) / (float)vd + eps);
    if (c < vd) out[(size_t)n * ldo + (size_t)h * vd + c] = __float2bfloat16_rn(o * inv);
}

inline int padded(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : 256; }

struct DiffArgs {
    const bf16* q; int ldq; bf16* out; int ldo; const bf16 *kc, *vc; long long page_stride; const int* block_table; int table_stride;
    const int *cu_seqlens, *slots, *start_pos; int n_seqs, max_q_len, tiles, n_heads, n_kv, d, vd; float scale; int window;
    float lambda, out_scale, eps; int n_splits; float *part_o, *part_ml; cudaStream_t stream;
};

template <int DKP, int DVP>
int launch_diff_decode(const DiffArgs& a) {
    auto kernel = attention_diff_decode_kernel<DKP, DVP>;
    constexpr int smem = diff_decode_smem_bytes<DKP, DVP>();
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_chained(kernel, dim3(a.n_splits, a.n_kv, a.n_seqs), dim3(kThreads), smem, a.stream, a.q, a.ldq, a.out, a.ldo,
                          a.kc, a.vc, a.page_stride, a.block_table, a.table_stride, a.slots, a.start_pos, a.n_heads, a.n_kv,
                          a.d, a.vd, a.scale, a.window, a.lambda, a.out_scale, a.eps, a.n_splits, a.part_o, a.part_ml);
}

template <int DKP, int DVP>
int launch_diff(const DiffArgs& a) {
    if (a.max_q_len == 1 && a.n_heads / a.n_kv <= 16) return launch_diff_decode<DKP, DVP>(a);
    auto kernel = attention_diff_mma_kernel<DKP, DVP>;
    constexpr int smem = diff_smem_bytes<DKP, DVP>();
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_chained(kernel, dim3(a.tiles * a.n_splits, a.n_kv, a.n_seqs), dim3(kThreads), smem, a.stream, a.q, a.ldq, a.out, a.ldo,
                          a.kc, a.vc, a.page_stride, a.block_table, a.table_stride, a.cu_seqlens, a.slots, a.start_pos, a.n_heads, a.n_kv,
                          a.d, a.vd, a.scale, a.window, a.lambda, a.out_scale, a.eps, a.n_splits, a.part_o, a.part_ml);
}
}  // namespace

// q: [N, n_heads * 2 d] (a head's map 1, then its map 2), out: [N, n_heads * vd]; a key row holds 2 d
// channels, a value row vd.  dtype 0: float, 1: bfloat16.
GTG_API int gtg_attention_diff_simple(int dtype, const void* q, int ldq, void* out, int ldo, const void* kc, const void* vc,
                                      long long page_stride, const int* block_table, int table_stride, const int* token_seq,
                                      const int* slots, const int* positions, int N, int n_heads, int n_kv, int d, int vd,
                                      float scale, int window, float lambda, float out_scale, float eps, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (n_heads <= 0 || n_kv <= 0 || n_heads % n_kv || d <= 0 || vd <= 0 || window < 0) return kErrBadArgument;
    if (ldq < n_heads * 2 * d || ldo < n_heads * vd) return kErrBadArgument;
    const size_t smem = (size_t)kWarps * 2 * d * sizeof(float);
    if (d > 1024 || vd > 1024 || smem > 48 * 1024) return kErrUnsupported;
    const long long blocks = ((long long)N * n_heads + kWarps - 1) / kWarps;
    if (blocks > 0x7fffffffLL) return kErrUnsupported;
#define GTG_DIFF_SIMPLE(T, PER)                                                                                     \
    return launch_chained(attention_diff_simple_kernel<T, PER>, dim3((unsigned)blocks), dim3(kWarps * 32), smem, stream, (const T*)q, \
                          ldq, (T*)out, ldo, (const T*)kc, (const T*)vc, page_stride, block_table, table_stride, token_seq, slots,    \
                          positions, N, n_heads, n_kv, d, vd, scale, window, lambda, out_scale, eps)
    if (dtype == 0) { if (vd <= 128) GTG_DIFF_SIMPLE(float, 4); if (vd <= 256) GTG_DIFF_SIMPLE(float, 8); GTG_DIFF_SIMPLE(float, 32); }
    if (dtype == 1) { if (vd <= 128) GTG_DIFF_SIMPLE(bf16, 4); if (vd <= 256) GTG_DIFF_SIMPLE(bf16, 8); GTG_DIFF_SIMPLE(bf16, 32); }
#undef GTG_DIFF_SIMPLE
    return kErrBadArgument;
}

// Whether the tensor-core kernel takes maps of d and values of vd channels (else: the plain kernel).
GTG_API int gtg_attention_diff_supports(int d, int vd) {
    return d > 0 && vd > 0 && d % 8 == 0 && vd % 8 == 0 && d <= 128 && vd <= 256;
}

// Floats of scratch that `n_splits` shares need: per (token, head, map, share) the padded output, maximum and sum.
GTG_API long long gtg_attention_diff_scratch_floats(int n_tokens, int n_heads, int vd, int n_splits) {
    if (n_splits <= 1) return 0;
    return (long long)n_tokens * n_heads * 2 * n_splits * (padded(vd) + 2);
}

// Into how many shares the pages of a step's tiles are cut: the number for which the waves of blocks (two to a
// multiprocessor) times the pages a block walks, plus what a block costs beyond its pages, is least; a second kernel
// merges the shares, which counts too.  It depends on the step's sizes only.
GTG_API int gtg_attention_diff_splits(int n_seqs, int max_q_len, int n_heads, int n_kv, int max_kv_len, int window) {
    if (n_seqs <= 0 || n_kv <= 0) return 1;
    int device = 0, sms = 148;
    if (cudaGetDevice(&device) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    const long long tiles = ((long long)max_q_len * (n_heads / n_kv) + kTileRows - 1) / kTileRows;
    const long long blocks = tiles * n_kv * n_seqs;
    const int keys = window > 0 ? min(max_kv_len, window + max_q_len) : max_kv_len;
    const int pages = (keys + kPageTokens - 1) / kPageTokens + (window > 0 ? 1 : 0);
    constexpr long long kBlockPages = 2, kMergePages = 4;  // a block's start and end, and the merge, in pages' time
    int best = 1;
    long long least = -1;
    for (int n = 1; n <= min(32, pages); ++n) {
        const long long waves = (blocks * n + 2LL * sms - 1) / (2LL * sms);
        const long long cost = waves * ((pages + n - 1) / n + kBlockPages) + (n > 1 ? kMergePages : 0);
        if (least < 0 || cost < least) { least = cost; best = n; }
    }
    return best;
}

GTG_API int gtg_attention_diff_bf16(const void* q, int ldq, void* out, int ldo, const void* kc, const void* vc,
                                    long long page_stride, const int* block_table, int table_stride, const int* cu_seqlens,
                                    const int* slots, const int* start_pos, int n_seqs, int max_q_len, int n_tokens, int n_heads,
                                    int n_kv, int d, int vd, float scale, int window, float lambda, float out_scale, float eps,
                                    int n_splits, float* scratch, cudaStream_t stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return 0;
    if (n_heads <= 0 || n_kv <= 0 || n_heads % n_kv || window < 0 || n_splits < 1 || !(scale > 0.f)) return kErrBadArgument;
    if (ldq < n_heads * 2 * d || ldo < n_heads * vd || (n_splits > 1 && !scratch)) return kErrBadArgument;
    if (!gtg_attention_diff_supports(d, vd)) return kErrUnsupported;
    if (ldq % 8 || page_stride % 8 || ((uintptr_t)q % 16) || ((uintptr_t)kc % 16) || ((uintptr_t)vc % 16) || ldo % 2 ||
        ((uintptr_t)out % 4)) return kErrUnsupported;
    const long long tiles = ((long long)max_q_len * (n_heads / n_kv) + kTileRows - 1) / kTileRows;
    if (tiles * n_splits > 0x7fffffffLL || n_seqs > 65535 || n_kv > 65535) return kErrUnsupported;
    const int dvp = padded(vd);
    const DiffArgs a{(const bf16*)q, ldq, (bf16*)out, ldo, (const bf16*)kc, (const bf16*)vc, page_stride, block_table, table_stride,
                     cu_seqlens, slots, start_pos, n_seqs, max_q_len, (int)tiles, n_heads, n_kv, d, vd, scale, window, lambda, out_scale, eps,
                     n_splits, scratch, scratch ? scratch + (size_t)n_tokens * n_heads * 2 * n_splits * dvp : nullptr, stream};
    int st;
    if (d <= 64) st = dvp == 64 ? launch_diff<64, 64>(a) : dvp == 128 ? launch_diff<64, 128>(a) : launch_diff<64, 256>(a);
    else st = dvp == 64 ? launch_diff<128, 64>(a) : dvp == 128 ? launch_diff<128, 128>(a) : launch_diff<128, 256>(a);
    if (st != 0 || n_splits == 1) return st;
    return launch_chained(attention_diff_merge_kernel, dim3((unsigned)((long long)n_tokens * n_heads)), dim3(dvp), 0, stream,
                          (const float*)a.part_o, (const float*)a.part_ml, (bf16*)out, ldo, n_heads, vd, dvp, n_splits, lambda, out_scale, eps);
}
