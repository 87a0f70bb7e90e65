// Differential attention of prompts on the fifth-generation tensor cores, for maps of 64 channels over values
// of 128, over the paged cache (what a head computes: see attention_diff.cu).
//
// One CTA per (128-query tile, query head, sequence) computes both maps of its head.  Per step of two cache pages
// (128 keys) and map m:
//   S_m  = Q_m K_m^T   tcgen05.mma 128 x 128 x 64; queries and the map's half of the key rows in shared memory
//                      (TMA, 128-byte swizzle, K-major), S_m in TMEM
//   P_m  = softmax     four warps a map, one thread per query row: its 128 scores out of TMEM, masked where the step
//                      crosses an edge, running maximum and sum in float; P_m back to TMEM as packed bfloat16, where
//                      S_m was
//   O_m += P_m V       tcgen05.mma 128 x 128 x 128 with A = P_m from TMEM and the value pages as the MN-major B
//                      operand, which both maps share; O_m stays in TMEM
// The two maps take turns on the tensor pipe: while one map's warps are in their softmax, the other's products run.
// Products of one CTA complete in the order they are issued, S_m of the next step behind O_m of this one, so a
// complete S_m means that O_m holds every step before it and that P_m has been read: the softmax warps may then
// rescale O_m and overwrite P_m.  As in attention_tcgen05.cu the running maximum only follows jumps above 2^8.
// At the end map 2's warps leave lambda O_2 / l_2 in shared memory and map 1's take it off theirs, norm the
// difference (a thread holds a query's whole row) and store it.  Roles: warps 0-3 map 1, warps 4-7 map 2, warp 8
// issues the TMA loads (a ring of three steps), warp 9 allocates TMEM and issues the MMAs.  One CTA an SM (all 512
// columns of TMEM).  Every mbarrier wait is bounded.
#include "tcgen05_attention.cuh"

namespace {
constexpr int BQ = 128, BK = 128, D = 64, VD = 128;
constexpr int kThreads = 320;
constexpr int kStages = 3;
constexpr int kPages = BK / kPageTokens;
constexpr int kBlockBytes = kPageTokens * 64 * 2;            // 64 tokens x 64 channels: one swizzled block of a page
constexpr int kQBytes = 2 * BQ * D * 2;                      // both maps
constexpr int kKeyBytes = BK * D * 2;                        // one map's keys of a step
constexpr int kStageBytes = 2 * kKeyBytes + BK * VD * 2;
constexpr int kOffKV = kQBytes, kOffBar = kOffKV + kStages * kStageBytes;
constexpr int kSmemBytes = kOffBar + 256;
constexpr int kTmemCols = 512;                               // S_1, S_2 (128 floats each; P_m in the first 64 of S_m), O_1, O_2
constexpr int kColO = 2 * BK;
constexpr int kPitch = VD + 4;                               // floats a row of the exchange
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRaiseBy = 8.0f;
static_assert(BQ * kPitch * 4 <= kStages * kStageBytes, "the exchange takes the ring's place");

// map_q: the step's [tokens, row width] queries, boxes of 64 channels x 128 rows.  map_kv: one cache entry as rows
// of 128 channels, row = ((page*2 + k|v)*n_kv + head)*64 + token; boxes of 64 channels x 64 rows.
// grid: (query heads, sequences, query tiles), the longest tiles first.
template <bool kTest>
__global__ void __launch_bounds__(kThreads, 1)
attention_diff_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                         bf16* __restrict__ out, int ldo, const int* __restrict__ block_table, int table_stride,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ slots, const int* __restrict__ start_pos,
                         int n_heads, int n_kv, float scale, int window, float lambda, float out_scale, float eps) {
    extern __shared__ __align__(1024) unsigned char smem[];
    const int h = blockIdx.x, b = blockIdx.y;
    const int tile = gridDim.z - 1 - blockIdx.z;
    const int q_begin = cu_seqlens[b];
    const int q_len = cu_seqlens[b + 1] - q_begin;
    if (tile * BQ >= q_len) return;                              // before any barrier or TMEM use
    const uint32_t base = smem_addr(smem);
    if (base & 1023u) {                                          // the swizzled tiles need this alignment
        if (threadIdx.x == 0) atomicExch(&g_status, 2);
        return;
    }
    const uint32_t bars = base + kOffBar;
    const uint32_t q_full = bars;
    auto s_full = [&](int m) { return bars + 8u + 8u * m; };
    auto p_full = [&](int m) { return bars + 24u + 8u * m; };
    const uint32_t all_done = bars + 40u;
    auto kv_full = [&](int s) { return bars + 48u + 8u * s; };
    auto kv_empty = [&](int s) { return bars + 48u + 8u * kStages + 8u * s; };
    uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(smem + kOffBar + 160);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + kOffBar + 168);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int start = start_pos[b];
    const int kvh = h / (n_heads / n_kv);
    const int* table = block_table + (size_t)slots[b] * table_stride;
    const int rows_here = min(BQ, q_len - tile * BQ);
    const int k_max = start + tile * BQ + rows_here - 1;         // last key any row of the tile sees
    const int k_min = window > 0 ? max(0, start + tile * BQ - window + 1) : 0;
    const int j_lo = k_min / kPageTokens, j_hi = k_max / kPageTokens;
    const int n_steps = (j_hi - j_lo + kPages) / kPages;

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int m = 0; m < 2; ++m) { mbar_init(s_full(m), 1); mbar_init(p_full(m), 4); }      // one arrival per softmax warp
        mbar_init(all_done, 1);
        for (int s = 0; s < kStages; ++s) { mbar_init(kv_full(s), 1); mbar_init(kv_empty(s), 1); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::);
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n"
                     ::"r"(smem_addr(tmem_holder)), "r"(kTmemCols));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::);
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
    const uint32_t tmem = *tmem_holder;
    chain_wait();                                                // queries, keys and values come from the kernel before
    chain_release();

    if (warp == 8) {
        // ------------------------------------------------------------ TMA producer
        if (lane == 0) {
            mbar_expect_tx(q_full, kQBytes);
            for (int m = 0; m < 2; ++m) tma_load_2d<kTest>(base + m * (BQ * 128), &map_q, (h * 2 + m) * D, q_begin + tile * BQ, q_full);
            for (int i = 0; i < n_steps; ++i) {
                const int s = i % kStages;
                if (!mbar_wait<kTest>(kv_empty(s), (((uint32_t)i / kStages) & 1u) ^ 1u, abort_flag)) break;
                const uint32_t dst = base + kOffKV + s * kStageBytes;
                mbar_expect_tx(kv_full(s), kStageBytes);
                for (int pg = 0; pg < kPages; ++pg) {
                    // a page beyond the last one is the step's first page again: finite values under keys that no row sees
                    const int first = j_lo + i * kPages, j = first + pg;
                    const int page = table[j <= j_hi ? j : first];
                    for (int kv = 0; kv < 2; ++kv) {
                        const int row = ((page * 2 + kv) * n_kv + kvh) * kPageTokens;
                        for (int half = 0; half < 2; ++half)     // of a key row: the maps; of a value row: its channels
                            tma_load_2d<kTest>(dst + (kv * 2 + half) * kKeyBytes + pg * kBlockBytes, &map_kv, 64 * half, row, kv_full(s));
                    }
                }
            }
        }
    } else if (warp == 9) {
        // ------------------------------------------------------------ MMA issuer
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc(BQ, BK, 0);               // S[128 x 128 keys], keys K-major
            const uint32_t idesc_pv = umma_idesc(BQ, VD, 1);              // O[128 x 128 channels], values MN-major
            bool ok = mbar_wait<kTest>(q_full, 0, abort_flag);
            auto issue_s = [&](int i, int m) {
                const uint32_t kbase = base + kOffKV + (i % kStages) * kStageBytes + m * kKeyBytes;
#pragma unroll
                for (int kk = 0; kk < D / 16; ++kk)
                    umma_ss(tmem + m * BK, umma_desc(base + m * (BQ * 128)) + 2 * kk, umma_desc(kbase) + 2 * kk, idesc_s, kk > 0 ? 1u : 0u);
                umma_commit(s_full(m));
            };
            if (ok) ok = mbar_wait<kTest>(kv_full(0), 0, abort_flag);
            if (ok) {
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
                issue_s(0, 0);
                issue_s(0, 1);
            }
            for (int i = 0; i < n_steps && ok; ++i) {
                const int s = i % kStages;
                const uint64_t dv = umma_desc(base + kOffKV + s * kStageBytes + 2 * kKeyBytes, BK * 128);
                for (int m = 0; m < 2; ++m) {
                    ok = mbar_wait<kTest>(p_full(m), (uint32_t)i & 1u, abort_flag);     // P_m is in TMEM, O_m rescaled if it had to be
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
#pragma unroll
                    for (int kk = 0; kk < BK / 16; ++kk)                  // 16 keys: 8 columns of P, two 8-key groups of V
                        umma_ts(tmem + kColO + m * VD, tmem + m * BK + 8 * kk, dv + (uint64_t)(2 * 1024 >> 4) * kk, idesc_pv, (i > 0 || kk > 0) ? 1u : 0u);
                    if (m == 1) umma_commit(kv_empty(s));                 // keys and values of the step have been read
                    if (i + 1 < n_steps) {
                        if (m == 0) {
                            ok = mbar_wait<kTest>(kv_full((i + 1) % kStages), ((uint32_t)(i + 1) / kStages) & 1u, abort_flag);
                            if (!ok) break;
                            asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
                        }
                        issue_s(i + 1, m);
                    }
                }
            }
            if (ok) umma_commit(all_done);
        }
    } else {
        // ------------------------------------------------------------ softmax + output (thread = query row of one map)
        const unsigned full = 0xffffffffu;
        const int m = warp >> 2;
        const int r = (warp & 3) * 32 + lane;                    // row of the tile, TMEM lane
        const int pos = start + tile * BQ + r;
        const uint32_t lane_off = (uint32_t)((warp & 3) * 32) << 16;
        const uint32_t tmem_s = tmem + m * BK + lane_off, tmem_o = tmem + kColO + m * VD + lane_off;
        const float s_in = scale * kLog2e;
        float m_run = -INFINITY, l_run = 0.f;
        uint32_t sv[BK];
        bool ok = true;
        for (int i = 0; i < n_steps; ++i) {
            const int key0 = (j_lo + i * kPages) * kPageTokens;
            ok = __all_sync(full, mbar_wait<kTest>(s_full(m), (uint32_t)i & 1u, abort_flag));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
#pragma unroll
            for (int c = 0; c < BK / 32; ++c) tmem_ld32(tmem_s + 32 * c, sv + 32 * c);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
            const bool all_visible = (key0 + BK - 1 <= pos) && (window <= 0 || key0 > pos - window);
            if (!all_visible) {
#pragma unroll
                for (int c = 0; c < BK; ++c) {
                    const int key = key0 + c;
                    if (!(key <= pos && (window <= 0 || key > pos - window))) sv[c] = __float_as_uint(-INFINITY);
                }
            }
            float mx[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) mx[e] = -INFINITY;
#pragma unroll
            for (int c = 0; c < BK; c += 8) {
#pragma unroll
                for (int e = 0; e < 8; ++e) mx[e] = fmaxf(mx[e], __uint_as_float(sv[c + e]));
            }
            const float m_step = fmaxf(fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])), fmaxf(fmaxf(mx[4], mx[5]), fmaxf(mx[6], mx[7]))) * s_in;
            if (i == 0) {
                m_run = m_step;                                  // the first product overwrites O_m
            } else {
                const bool raise = m_step > m_run + kRaiseBy;    // also: the first visible key of a row
                if (__any_sync(full, raise)) {
                    float corr = 1.0f;
                    if (raise) {
                        corr = fast_exp2(m_run - m_step);        // 0 when the row had seen nothing
                        m_run = m_step;
                        l_run *= corr;
                    }
                    uint32_t ov[8];                              // few registers: the scores are live
#pragma unroll 1
                    for (int part = 0; part < VD / 8; ++part) {
                        tmem_ld8(tmem_o + 8 * part, ov);
                        asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
#pragma unroll
                        for (int e = 0; e < 8; ++e) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * corr);
                        tmem_st8(tmem_o + 8 * part, ov);
                    }
                }
            }
            const float m_use = m_run == -INFINITY ? 0.f : m_run;
            float l0 = 0.f, l1 = 0.f;
            // the row of P: 128 bfloat16 as 64 packed columns (packed in place); eight exponentials are issued back to back
#pragma unroll
            for (int c = 0; c < BK / 2; c += 4) {
                float p[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) p[e] = fmaf(__uint_as_float(sv[2 * c + e]), s_in, -m_use);
#pragma unroll
                for (int e = 0; e < 8; ++e) p[e] = exp2_in_order(p[e]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    l0 += p[2 * e];
                    l1 += p[2 * e + 1];
                    __nv_bfloat162 hh = __floats2bfloat162_rn(p[2 * e], p[2 * e + 1]);
                    sv[c + e] = *reinterpret_cast<uint32_t*>(&hh);   // the scores at and below this index are done with
                }
            }
#pragma unroll
            for (int c = 0; c < BK / 64; ++c) tmem_st32(tmem_s + 32 * c, sv + 32 * c);
            l_run += l0 + l1;
            asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::);
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full(m));
        }
        if (ok) ok = __all_sync(full, mbar_wait<kTest>(all_done, 0u, abort_flag));
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
        float* second = reinterpret_cast<float*>(smem + kOffKV) + r * kPitch;      // the ring has been read
        if (ok) {
#pragma unroll
            for (int c = 0; c < VD / 32; ++c) tmem_ld32(tmem_o + 32 * c, sv + 32 * c);
            asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
        }
        if (ok && m == 1) {
            const float f = l_run > 0.f ? lambda / l_run : 0.f;
#pragma unroll
            for (int c = 0; c < VD; c += 4)
                *reinterpret_cast<float4*>(second + c) = make_float4(__uint_as_float(sv[c]) * f, __uint_as_float(sv[c + 1]) * f,
                                                                     __uint_as_float(sv[c + 2]) * f, __uint_as_float(sv[c + 3]) * f);
        }
        asm volatile("bar.sync 1, 256;\n" ::: "memory");         // the softmax warps of both maps
        if (ok && m == 0 && r < rows_here) {
            const float f = l_run > 0.f ? 1.0f / l_run : 0.f;
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < VD; c += 4) {
                const float4 t = *reinterpret_cast<const float4*>(second + c);
                const float x[4] = {fmaf(__uint_as_float(sv[c]), f, -t.x), fmaf(__uint_as_float(sv[c + 1]), f, -t.y),
                                    fmaf(__uint_as_float(sv[c + 2]), f, -t.z), fmaf(__uint_as_float(sv[c + 3]), f, -t.w)};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    sv[c + e] = __float_as_uint(x[e]);
                    ss = fmaf(x[e], x[e], ss);
                }
            }
            const float inv = out_scale / sqrtf(ss / (float)VD + eps);
            bf16* dst = out + (size_t)(q_begin + tile * BQ + r) * ldo + (size_t)h * VD;
#pragma unroll
            for (int c = 0; c < VD; c += 8) {
                uint32_t o4[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    __nv_bfloat162 hh = __floats2bfloat162_rn(__uint_as_float(sv[c + 2 * e]) * inv, __uint_as_float(sv[c + 2 * e + 1]) * inv);
                    o4[e] = *reinterpret_cast<uint32_t*>(&hh);
                }
                *reinterpret_cast<uint4*>(dst + c) = make_uint4(o4[0], o4[1], o4[2], o4[3]);
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::);
    __syncthreads();
    if (warp == 9) {
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::);
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(kTmemCols));
    }
}

template <bool kTest>
int launch(const CUtensorMap& map_q, const CUtensorMap& map_kv, bf16* out, int ldo, const int* block_table, int table_stride,
           const int* cu_seqlens, const int* slots, const int* start_pos, int B, int max_q_len, int n_heads, int n_kv, float scale,
           int window, float lambda, float out_scale, float eps, cudaStream_t stream) {
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(attention_diff_tc_kernel<kTest>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBytes);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_chained(attention_diff_tc_kernel<kTest>, dim3(n_heads, B, (max_q_len + BQ - 1) / BQ), dim3(kThreads), (size_t)kSmemBytes, stream,
                          map_q, map_kv, out, ldo, block_table, table_stride, cu_seqlens, slots, start_pos, n_heads, n_kv, scale, window, lambda,
                          out_scale, eps);
}
}  // namespace

GTG_API int gtg_attention_diff_tcgen05_status() {
    int v = 0;
    if (cudaMemcpyFromSymbol(&v, g_status, sizeof(int)) != cudaSuccess) return -1;
    return v;
}

// What this kernel serves: maps of 64 and values of 128 channels, keys and values of a page side by side.
GTG_API int gtg_attention_diff_tcgen05_supports(int d, int vd) { return d == D && vd == VD; }

// Arguments as in gtg_attention_diff_bf16; n_pages: pages of the entry's pool.
GTG_API int gtg_attention_diff_tcgen05(const void* q, int ldq, int n_tokens, void* out, int ldo, const void* kc, const void* vc,
                                       long long page_stride, int n_pages, const int* block_table, int table_stride,
                                       const int* cu_seqlens, const int* slots, const int* start_pos, int B, int max_q_len, int n_heads,
                                       int n_kv, int d, int vd, float scale, int window, float lambda, float out_scale, float eps,
                                       cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0) return 0;
    if (n_heads <= 0 || n_kv <= 0 || n_heads % n_kv || window < 0 || !(scale > 0.f)) return kErrBadArgument;
    if (d != D || vd != VD) return kErrUnsupported;
    if (ldq < n_heads * 2 * D || ldo < n_heads * VD) return kErrBadArgument;
    if (ldq % 8 || ldo % 8 || ((uintptr_t)q % 16) || ((uintptr_t)out % 16) || ((uintptr_t)kc % 16)) return kErrUnsupported;
    // keys then values of a page, contiguous and alike in width: the layout the row arithmetic above assumes
    const long long kv_rows = 2LL * n_kv * kPageTokens;
    if (page_stride != kv_rows * VD || (const bf16*)vc != (const bf16*)kc + (long long)n_kv * kPageTokens * VD) return kErrUnsupported;
    if (B > 65535 || (max_q_len + BQ - 1) / BQ > 65535 || (long long)n_pages * kv_rows > 0x7fffffffLL) return kErrUnsupported;
    CUtensorMap map_q, map_kv;
    int st = make_map(&map_q, q, n_tokens, n_heads * 2 * D, ldq, BQ);
    if (st != 0) return st;
    st = make_map(&map_kv, kc, (long long)n_pages * kv_rows, VD, VD, kPageTokens);
    if (st != 0) return st;
#define GTG_ARGS map_q, map_kv, (bf16*)out, ldo, block_table, table_stride, cu_seqlens, slots, start_pos, B, max_q_len, n_heads, n_kv, \
                 scale, window, lambda, out_scale, eps, stream
    return g_test_waits ? launch<true>(GTG_ARGS) : launch<false>(GTG_ARGS);
#undef GTG_ARGS
}

// Test hook: see attention_tcgen05.cu.
GTG_API int gtg_attention_diff_tcgen05_test_hooks(int test_waits) {
    const int zero = 0;
    cudaError_t e = cudaDeviceSynchronize();
    g_test_waits = test_waits != 0;
    if (e == cudaSuccess) e = cudaMemcpyToSymbol(g_status, &zero, sizeof(zero));
    return (int)e;
}
