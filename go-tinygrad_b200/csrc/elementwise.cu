// Bandwidth-bound kernels around the matrix products: embedding gather, the
// residual add fused with RMSNorm, SwiGLU, the rotary table of a step and the
// rotation of queries and keys fused with the write into the paged cache.
// Each is templated on the activation type (float for the 32-bit path,
// __nv_bfloat16 for the serving path); sums, the reciprocal root, the rotation
// and the residual stream are float in both.
#include "common.cuh"

// ---------------------------------------------------------------- embedding
// out[n,:] = table[tokens[n],:] widened to float (the residual stream), times
// `scale` (1: no scaling, as in model/inference_helpers.go:9-34).  Token ids are validated by the
// host; an id outside the table is clamped so the kernel never reads outside.
// `turns` (or null): double [(H + 1) / 2], whole turns a position; channel 2i gets
// sin(2 pi positions[n] turns[i]) added, channel 2i + 1 the cosine.  The angle is reduced to
// a fraction of a turn in double, so that far positions lose nothing.
template <typename T>
__global__ void embed_kernel(const int* __restrict__ tokens, const T* __restrict__ table,
                             float* __restrict__ out, int H, int V, float scale,
                             const int* __restrict__ positions, const double* __restrict__ turns) {
    chain_wait();        // the step's metadata is written here or just before: nothing later may start early
    chain_release();
    const int n = blockIdx.x;
    int tok = tokens[n];
    tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
    const T* src = table + (size_t)tok * H;
    float* dst = out + (size_t)n * H;
    if (!turns) {
        for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = to_f32<T>(src[i]) * scale;
        return;
    }
    const double p = (double)positions[n];
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const double t = p * turns[i >> 1];
        const float half_turns = (float)(2.0 * (t - rint(t)));
        dst[i] = to_f32<T>(src[i]) * scale + ((i & 1) ? cospif(half_turns) : sinpif(half_turns));
    }
}

GTG_API int gtg_embed(int dtype, const int* tokens, const void* table, float* out,
                      int N, int H, int V, float scale, const int* positions, const double* turns, cudaStream_t stream) {
    int st = 0;
    if (N <= 0) return 0;
    const int threads = H >= 1024 ? 256 : 128;
    if (dtype == 0) st = launch_chained(embed_kernel<float>, dim3(N), dim3(threads), 0, stream, tokens, (const float*)table, out, H, V, scale, positions, turns);
    else if (dtype == 1) st = launch_chained(embed_kernel<bf16>, dim3(N), dim3(threads), 0, stream, tokens, (const bf16*)table, out, H, V, scale, positions, turns);
    else return kErrBadArgument;
    return st;
}

// ------------------------------------------------- residual add + RMSNorm
// x = residual[r,:] (+ pending[r,:]);  out[i,:] = weight * x * (1/sqrt(mean(x^2)+eps))
// with r = rows ? rows[i] : i.  Without `rows` the sum is written back to the
// residual stream.  eps is added to the mean inside the root, and the product
// is (w*x)*s (backends/simd/vec.go:72-85).  kTwo: a second weight over the same row gives
// a second output, for layers whose sublayers read two norms of one hidden state.
template <typename T, bool kTwo>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const T* __restrict__ pending,
                                   const float* __restrict__ weight, float eps,
                                   T* __restrict__ out, const int* __restrict__ rows, int H,
                                   const float* __restrict__ weight2, T* __restrict__ out2) {
    chain_release();
    chain_wait();
    extern __shared__ float smem[];
    float* row = smem;          // H floats
    float* scratch = smem + H;  // 33 floats
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    float* res = residual + (size_t)r * H;
    const T* pen = pending ? pending + (size_t)r * H : nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float x = res[i];
        if (pen) {
            x += to_f32<T>(pen[i]);
            if (!rows) res[i] = x;
        }
        row[i] = x;
        ss += x * x;
    }
    const float total = block_sum(ss, scratch);
    const float s = 1.0f / sqrtf(total / (float)H + eps);
    T* o = out + (size_t)i_out * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x)
        o[i] = from_f32<T>((weight[i] * row[i]) * s);
    if (kTwo) {
        T* o2 = out2 + (size_t)i_out * H;
        for (int i = threadIdx.x; i < H; i += blockDim.x)
            o2[i] = from_f32<T>((weight2[i] * row[i]) * s);
    }
}

// The same for bfloat16 rows whose width is a multiple of 8 and at most 8192:
// every thread owns 8 consecutive channels, moved with 16- and 32-byte accesses
// and kept in registers between the sum of squares and the scaling.
template <bool kTwo>
__global__ void __launch_bounds__(1024)
add_rmsnorm_bf16_vec_kernel(float* __restrict__ residual, const bf16* __restrict__ pending,
                            const float* __restrict__ weight, float eps, bf16* __restrict__ out,
                            const int* __restrict__ rows, int H,
                            const float* __restrict__ weight2, bf16* __restrict__ out2) {
    chain_release();
    chain_wait();
    __shared__ float scratch[33];
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    const int c = threadIdx.x * 8;
    const bool active = c < H;
    float x[8];
    float w[8];
    float ss = 0.f;
    if (active) {
        const float4* wp = reinterpret_cast<const float4*>(weight + c);
        const float4 w0 = wp[0], w1 = wp[1];
        w[0] = w0.x; w[1] = w0.y; w[2] = w0.z; w[3] = w0.w; w[4] = w1.x; w[5] = w1.y; w[6] = w1.z; w[7] = w1.w;
        float4* rp = reinterpret_cast<float4*>(residual + (size_t)r * H + c);
        const float4 a = rp[0], b = rp[1];
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
        if (pending) {
            const uint4 p = *reinterpret_cast<const uint4*>(pending + (size_t)r * H + c);
            const __nv_bfloat162* ph = reinterpret_cast<const __nv_bfloat162*>(&p);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(ph[j]);
                x[2 * j] += f.x;
                x[2 * j + 1] += f.y;
            }
            if (!rows) {
                rp[0] = make_float4(x[0], x[1], x[2], x[3]);
                rp[1] = make_float4(x[4], x[5], x[6], x[7]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
    }
    const float total = block_sum(ss, scratch);
    const float s = 1.0f / sqrtf(total / (float)H + eps);
    if (active) {
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            oh[j] = __floats2bfloat162_rn((w[2 * j] * x[2 * j]) * s, (w[2 * j + 1] * x[2 * j + 1]) * s);
        *reinterpret_cast<uint4*>(out + (size_t)i_out * H + c) = o;
        if (kTwo) {
            const float4* wp = reinterpret_cast<const float4*>(weight2 + c);
            const float4 w0 = wp[0], w1 = wp[1];
            oh[0] = __floats2bfloat162_rn((w0.x * x[0]) * s, (w0.y * x[1]) * s);
            oh[1] = __floats2bfloat162_rn((w0.z * x[2]) * s, (w0.w * x[3]) * s);
            oh[2] = __floats2bfloat162_rn((w1.x * x[4]) * s, (w1.y * x[5]) * s);
            oh[3] = __floats2bfloat162_rn((w1.z * x[6]) * s, (w1.w * x[7]) * s);
            *reinterpret_cast<uint4*>(out2 + (size_t)i_out * H + c) = o;
        }
    }
}

// weight2 and out2: a second norm of the same rows (both null: none).
GTG_API int gtg_add_rmsnorm(int dtype, float* residual, const void* pending, const float* weight,
                            float eps, void* out, const int* rows, int R, int H, const float* weight2, void* out2,
                            cudaStream_t stream) {
    int st = 0;
    if (R <= 0) return 0;
    if ((weight2 == nullptr) != (out2 == nullptr)) return kErrBadArgument;
    if (dtype == 1 && H % 8 == 0 && H <= 8192 && ((uintptr_t)residual % 16) == 0 && ((uintptr_t)out % 16) == 0 &&
        ((uintptr_t)weight % 16) == 0 && ((uintptr_t)pending % 16) == 0 && ((uintptr_t)weight2 % 16) == 0 && ((uintptr_t)out2 % 16) == 0) {
        int t = ((H / 8) + 31) / 32 * 32;
        if (out2)
            return launch_chained(add_rmsnorm_bf16_vec_kernel<true>, dim3(R), dim3(t), 0, stream, residual, (const bf16*)pending, weight, eps, (bf16*)out, rows, H, weight2, (bf16*)out2);
        st = launch_chained(add_rmsnorm_bf16_vec_kernel<false>, dim3(R), dim3(t), 0, stream, residual, (const bf16*)pending, weight, eps, (bf16*)out, rows, H, nullptr, nullptr);
        return st;
    }
    int threads = 32;
    while (threads < 1024 && threads * 4 < H) threads *= 2;
    const size_t smem = (size_t)(H + 33) * sizeof(float);
    if (smem > 200 * 1024) return kErrUnsupported;
#define GTG_RMSNORM(T, TWO)                                                                                          \
    do {                                                                                                             \
        if (smem > 48 * 1024) {                                                                                      \
            const cudaError_t e = cudaFuncSetAttribute(add_rmsnorm_kernel<T, TWO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        return launch_chained(add_rmsnorm_kernel<T, TWO>, dim3(R), dim3(threads), smem, stream, residual, (const T*)pending, weight, eps, \
                              (T*)out, rows, H, weight2, (T*)out2);                                                  \
    } while (0)
    if (dtype == 0) { if (out2) GTG_RMSNORM(float, true); GTG_RMSNORM(float, false); }
    if (dtype == 1) { if (out2) GTG_RMSNORM(bf16, true); GTG_RMSNORM(bf16, false); }
#undef GTG_RMSNORM
    return kErrBadArgument;
}

// ------------------------------------------------------------------ SwiGLU
// out[m,i] = act(gu[m,i]) * gu[m,I+i]; act is silu, g / (1 + exp(-g))
// (backends/simd/vec.go:52-59), or another of the pointwise activations (`kind`; from
// kEpiClamped on it is the clamped gated product's code instead).
// `gu` holds the gate columns then the up columns.
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, T* __restrict__ out, int ldo, int M, int I, int kind) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * I;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / I;
        const int i = (int)(idx - m * I);
        const float g = to_f32<T>(gu[m * 2 * I + i]);
        const float u = to_f32<T>(gu[m * 2 * I + I + i]);
        out[m * ldo + i] = from_f32<T>(kind == 2 ? g / (1.0f + expf(-g)) * u : epi_is_clamped(kind) ? gated_value(g, u, kind) : activate(g, kind) * u);
    }
}

GTG_API int gtg_swiglu(int dtype, const void* gu, void* out, int ldo, int M, int I, int kind, cudaStream_t stream) {
    int st = 0;
    if (M <= 0 || I <= 0) return 0;
    if (kind < 0 || (kind >= kActivations && !epi_is_clamped(kind)) || ldo < I) return kErrBadArgument;
    const size_t total = (size_t)M * I;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == 0) st = launch_chained(swiglu_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)gu, (float*)out, ldo, M, I, kind);
    else if (dtype == 1) st = launch_chained(swiglu_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)gu, (bf16*)out, ldo, M, I, kind);
    else return kErrBadArgument;
    return st;
}

// ------------------------------------------------------------ rotary table
// cos_sin[n,i] = (cos, sin)(positions[n] * inv_freq[i]); the angle is a double
// product and the functions are evaluated in double, then rounded to float
// (model/llama.go:855-862).  Computed once per step for the step's tokens.
// `amplitude` multiplies both (1 for a plain rotation; frequency scalings that
// lengthen the context may grow queries and keys a little with it).
__global__ void rope_table_kernel(const int* __restrict__ positions, const double* __restrict__ inv_freq,
                                  float2* __restrict__ cos_sin, int N, int half, double amplitude) {
    chain_release();
    chain_wait();
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= N * half) return;
    const int n = idx / half, i = idx - n * half;
    const double ang = (double)positions[n] * inv_freq[i];
    double s, c;
    sincos(ang, &s, &c);
    cos_sin[idx] = make_float2((float)(c * amplitude), (float)(s * amplitude));
}

GTG_API int gtg_rope_table(const int* positions, const double* inv_freq, float* cos_sin,
                           int N, int half, double amplitude, cudaStream_t stream) {
    int st = 0;
    if (N <= 0 || half <= 0) return 0;
    const int total = N * half;
    st = launch_chained(rope_table_kernel, dim3((total + 127) / 128), dim3(128), 0, stream, positions, inv_freq, (float2*)cos_sin, N, half, amplitude);
    return st;
}

// ------------------------------------------- rotation + write into the cache
// For token n with fused projections qkv[n] = [q heads | k heads | v heads]:
// rotate q in place and k on its way into the cache, a' = a*c - b*s,
// b' = a*s + b*c; copy v into the cache.  Keys are stored after rotation
// (model/llama.go:1253-1254).  Which channels (a, b) form pair i is the
// encoding's layout: half-split, (i, i + rot/2) (model/llama.go:1556-1589), or
// interleaved, (2i, 2i+1); `rot` <= hd channels of a head rotate, the rest pass
// unchanged.  cos_sin holds rot/2 (cos, sin) per token.  With n_kv_store == 0
// only the queries are rotated (a layer that reads another layer's cache).
// cos_sin == nullptr means no rotation.  With `v_from_k` the row has no value
// heads: the value stored for a key/value head is its key as projected, before
// the rotation (a mixer without a value projection).
template <typename T>
__global__ void rope_kv_store_kernel(T* __restrict__ qkv, int ld, const float2* __restrict__ cos_sin,
                                     int n_heads, int n_kv_store, int hd, int rot, int interleaved, int v_from_k,
                                     T* __restrict__ kc, T* __restrict__ vc, long long page_stride,
                                     const int* __restrict__ block_table, int table_stride,
                                     const int* __restrict__ token_seq, const int* __restrict__ slots,
                                     const int* __restrict__ positions) {
    chain_release();
    chain_wait();
    const int n = blockIdx.x;
    const int half = hd >> 1, rhalf = rot >> 1;
    const int pos = positions[n];
    T* row = qkv + (size_t)n * ld;
    size_t cache_off = 0;
    if (n_kv_store > 0) {
        const int slot = slots[token_seq[n]];
        const int page = block_table[(size_t)slot * table_stride + pos / kPageTokens];
        cache_off = (size_t)page * page_stride + (size_t)(pos % kPageTokens) * hd;
    }
    // one item = two channels of one head: pair i of the rotated part, or two
    // consecutive channels of what passes unchanged
    const int items = (n_heads + 2 * n_kv_store) * half;
    for (int it = threadIdx.x; it < items; it += blockDim.x) {
        const int head = it / half, i = it - head * half;
        T* src = row + (v_from_k && head >= n_heads + n_kv_store ? head - n_kv_store : head) * hd;
        int ia, ib;
        if (i < rhalf) { ia = interleaved ? 2 * i : i; ib = interleaved ? 2 * i + 1 : i + rhalf; }
        else { ia = rot + 2 * (i - rhalf); ib = ia + 1; }
        const float a = to_f32<T>(src[ia]), b = to_f32<T>(src[ib]);
        if (head < n_heads + n_kv_store) {
            float c = 1.f, s = 0.f;
            if (cos_sin && i < rhalf) { const float2 cs = cos_sin[(size_t)n * rhalf + i]; c = cs.x; s = cs.y; }
            const float ra = a * c - b * s, rb = a * s + b * c;
            if (head < n_heads) {
                if (i < rhalf) { src[ia] = from_f32<T>(ra); src[ib] = from_f32<T>(rb); }
            } else {
                T* dst = kc + cache_off + (size_t)(head - n_heads) * kPageTokens * hd;
                dst[ia] = i < rhalf ? from_f32<T>(ra) : src[ia];
                dst[ib] = i < rhalf ? from_f32<T>(rb) : src[ib];
            }
        } else {
            T* dst = vc + cache_off + (size_t)(head - n_heads - n_kv_store) * kPageTokens * hd;
            dst[ia] = src[ia];
            dst[ib] = src[ib];
        }
    }
}

// The same for bfloat16 with head sizes that are multiples of 16 and 16-byte
// aligned rows: one thread rotates 8 consecutive pairs with 16-byte accesses.
__global__ void rope_kv_store_bf16_vec_kernel(bf16* __restrict__ qkv, int ld, const float2* __restrict__ cos_sin,
                                              int n_heads, int n_kv_store, int hd, int v_from_k,
                                              bf16* __restrict__ kc, bf16* __restrict__ vc, long long page_stride,
                                              const int* __restrict__ block_table, int table_stride,
                                              const int* __restrict__ token_seq, const int* __restrict__ slots,
                                              const int* __restrict__ positions) {
    chain_release();
    chain_wait();
    const int n = blockIdx.x;
    const int half = hd >> 1, chunks = half >> 3;
    const int pos = positions[n];
    bf16* row = qkv + (size_t)n * ld;
    size_t cache_off = 0;
    if (n_kv_store > 0) {
        const int slot = slots[token_seq[n]];
        const int page = block_table[(size_t)slot * table_stride + pos / kPageTokens];
        cache_off = (size_t)page * page_stride + (size_t)(pos % kPageTokens) * hd;
    }
    const int items = (n_heads + 2 * n_kv_store) * chunks;
    for (int it = threadIdx.x; it < items; it += blockDim.x) {
        const int head = it / chunks, i = (it - head * chunks) * 8;
        bf16* src = row + (v_from_k && head >= n_heads + n_kv_store ? head - n_kv_store : head) * hd;
        const uint4 av = *reinterpret_cast<const uint4*>(src + i);
        const uint4 bv = *reinterpret_cast<const uint4*>(src + i + half);
        if (head >= n_heads + n_kv_store) {                       // a value head: copy
            bf16* dst = vc + cache_off + (size_t)(head - n_heads - n_kv_store) * kPageTokens * hd;
            *reinterpret_cast<uint4*>(dst + i) = av;
            *reinterpret_cast<uint4*>(dst + i + half) = bv;
            continue;
        }
        uint4 ra = av, rb = bv;
        if (cos_sin) {
            const float4* cs = reinterpret_cast<const float4*>(cos_sin + (size_t)n * half + i);   // (c0,s0,c1,s1) x 4
            const __nv_bfloat162* ah = reinterpret_cast<const __nv_bfloat162*>(&av);
            const __nv_bfloat162* bh = reinterpret_cast<const __nv_bfloat162*>(&bv);
            __nv_bfloat162* rah = reinterpret_cast<__nv_bfloat162*>(&ra);
            __nv_bfloat162* rbh = reinterpret_cast<__nv_bfloat162*>(&rb);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float4 t = cs[j];
                const float2 a = __bfloat1622float2(ah[j]), b = __bfloat1622float2(bh[j]);
                rah[j] = __floats2bfloat162_rn(a.x * t.x - b.x * t.y, a.y * t.z - b.y * t.w);
                rbh[j] = __floats2bfloat162_rn(a.x * t.y + b.x * t.x, a.y * t.w + b.y * t.z);
            }
        }
        bf16* dst = head < n_heads ? src : kc + cache_off + (size_t)(head - n_heads) * kPageTokens * hd;
        *reinterpret_cast<uint4*>(dst + i) = ra;
        *reinterpret_cast<uint4*>(dst + i + half) = rb;
    }
}

GTG_API int gtg_rope_kv_store(int dtype, void* qkv, int ld, const float* cos_sin,
                              int n_heads, int n_kv_store, int hd, int rot, int interleaved, int v_from_k,
                              void* kc, void* vc, long long page_stride,
                              const int* block_table, int table_stride,
                              const int* token_seq, const int* slots, const int* positions,
                              int N, cudaStream_t stream) {
    int st = 0;
    if (N <= 0) return 0;
    if (hd <= 0 || (hd & 1) || rot <= 0 || (rot & 1) || rot > hd) return kErrBadArgument;
    if (dtype == 1 && rot == hd && !interleaved && hd % 16 == 0 && ld % 8 == 0 && page_stride % 8 == 0 && ((uintptr_t)qkv % 16) == 0 &&
        ((uintptr_t)kc % 16) == 0 && ((uintptr_t)vc % 16) == 0 && ((uintptr_t)cos_sin % 16) == 0) {
        const int vec_items = (n_heads + 2 * n_kv_store) * (hd / 16);
        int t = 32;
        while (t < 256 && t < vec_items) t *= 2;
        st = launch_chained(rope_kv_store_bf16_vec_kernel, dim3(N), dim3(t), 0, stream, (bf16*)qkv, ld, (const float2*)cos_sin, n_heads, n_kv_store, hd, v_from_k,
            (bf16*)kc, (bf16*)vc, page_stride, block_table, table_stride, token_seq, slots, positions);
        return st;
    }
    const int items = (n_heads + 2 * n_kv_store) * (hd / 2);
    int threads = 64;
    while (threads < 512 && threads < items) threads *= 2;
    if (dtype == 0)
        st = launch_chained(rope_kv_store_kernel<float>, dim3(N), dim3(threads), 0, stream, (float*)qkv, ld, (const float2*)cos_sin, n_heads, n_kv_store, hd, rot, interleaved, v_from_k,
            (float*)kc, (float*)vc, page_stride, block_table, table_stride, token_seq, slots, positions);
    else if (dtype == 1)
        st = launch_chained(rope_kv_store_kernel<bf16>, dim3(N), dim3(threads), 0, stream, (bf16*)qkv, ld, (const float2*)cos_sin, n_heads, n_kv_store, hd, rot, interleaved, v_from_k,
            (bf16*)kc, (bf16*)vc, page_stride, block_table, table_stride, token_seq, slots, positions);
    else return kErrBadArgument;
    return st;
}

// --------------------------------------------------- advance a decode batch
// Between two decode steps that never leave the device: the sampled token
// becomes the next input, every position moves on by one and so does every
// sequence's count of generated tokens (which keys its next random draw).
__global__ void advance_kernel(int* tokens, int* positions, int* steps, const int* sampled, int B) {
    chain_wait();        // the step's metadata is written here or just before: nothing later may start early
    chain_release();
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < B) { tokens[b] = sampled[b]; positions[b] += 1; steps[b] += 1; }
}

GTG_API int gtg_advance(int* tokens, int* positions, int* steps, const int* sampled, int B,
                        cudaStream_t stream) {
    int st = 0;
    if (B <= 0) return 0;
    st = launch_chained(advance_kernel, dim3((B + 127) / 128), dim3(128), 0, stream, tokens, positions, steps, sampled, B);
    return st;
}

// ------------------------------------------- a step's cache addresses, checked
// The debug pass that stands in for a memory checker: before a kernel that finds
// its keys and values through (sequence -> slot -> block table -> page), walk the
// same indices and record the first one that would leave its array -- in a flag
// the host reads, never by trapping -- so that the host can refuse the launch.
//   mode 0  per token:    item n has sequence token_seq[n], position positions[n]
//   mode 1  per sequence: item b is read up to position positions[b] (a decode step)
//   mode 2  per sequence: item b is read up to start_pos[b] + its run in cu_seqlens (a prompt step)
// flag[0]: 0 or what is wrong (1 sequence index, 2 slot, 3 negative position or run,
// 4 position beyond the block table's row, 5 page index outside the cache);
// flag[1]: the item.
__global__ void check_cache_access_kernel(int mode, int n_items, const int* __restrict__ token_seq,
                                          const int* __restrict__ slots, const int* __restrict__ positions,
                                          const int* __restrict__ start_pos, const int* __restrict__ cu_seqlens,
                                          int n_seqs, const int* __restrict__ block_table, int table_stride,
                                          int n_slots, int n_pages, int* __restrict__ flag) {
    const int item = blockIdx.x * blockDim.x + threadIdx.x;
    if (item >= n_items) return;
    int bad = 0;
    int seq = item, first_page = 0, last_pos = 0;
    if (mode == 0) {
        seq = token_seq[item];
        if (seq < 0 || seq >= n_seqs) bad = 1;
        last_pos = positions[item];
        first_page = last_pos >= 0 ? last_pos / kPageTokens : 0;          // earlier pages were other tokens' to check
    } else if (mode == 1) {
        last_pos = positions[item];
    } else {
        const int run = cu_seqlens[item + 1] - cu_seqlens[item];
        if (run < 0 || start_pos[item] < 0) bad = 3;
        last_pos = start_pos[item] + run - 1;
        if (run == 0) last_pos = -2;                                      // nothing is read
    }
    if (!bad && last_pos != -2) {
        const int slot = slots[seq];
        if (slot < 0 || slot >= n_slots) bad = 2;
        else if (last_pos < 0) bad = 3;
        else if (last_pos / kPageTokens >= table_stride) bad = 4;
        else {
            for (int p = first_page; p <= last_pos / kPageTokens; ++p) {
                const int page = block_table[(size_t)slot * table_stride + p];
                if (page < 0 || page >= n_pages) { bad = 5; break; }
            }
        }
    }
    if (bad && atomicCAS(&flag[0], 0, bad) == 0) flag[1] = item;
}

GTG_API int gtg_check_cache_access(int mode, int n_items, const int* token_seq, const int* slots,
                                   const int* positions, const int* start_pos, const int* cu_seqlens, int n_seqs,
                                   const int* block_table, int table_stride, int n_slots, int n_pages, int* flag,
                                   cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (mode < 0 || mode > 2 || flag == nullptr || slots == nullptr || block_table == nullptr) return kErrBadArgument;
    check_cache_access_kernel<<<(n_items + 127) / 128, 128, 0, stream>>>(mode, n_items, token_seq, slots, positions,
        start_pos, cu_seqlens, n_seqs, block_table, table_stride, n_slots, n_pages, flag);
    return launch_status();
}

// ------------------------------------------------- residual add + LayerNorm
// x = residual[r,:] (+ pending[r,:]);  out[i,:] = (x - mean) / sqrt(var + eps) * weight + bias,
// var the mean of the squared deviations from the mean (two passes over the row,
// which is kept in shared memory), everything in float.  Rows as in add_rmsnorm.
template <typename T>
__global__ void add_layernorm_kernel(float* __restrict__ residual, const T* __restrict__ pending,
                                     const float* __restrict__ weight, const float* __restrict__ bias, float eps,
                                     T* __restrict__ out, const int* __restrict__ rows, int H) {
    chain_release();
    chain_wait();
    extern __shared__ float smem[];
    float* row = smem;          // H floats
    float* scratch = smem + H;  // 33 floats
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    float* res = residual + (size_t)r * H;
    const T* pen = pending ? pending + (size_t)r * H : nullptr;
    float sum = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float x = res[i];
        if (pen) {
            x += to_f32<T>(pen[i]);
            if (!rows) res[i] = x;
        }
        row[i] = x;
        sum += x;
    }
    const float mean = block_sum(sum, scratch) / (float)H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float d = row[i] - mean;
        ss += d * d;
    }
    const float var = block_sum(ss, scratch) / (float)H;
    const float s = 1.0f / sqrtf(var + eps);
    T* o = out + (size_t)i_out * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x)
        o[i] = from_f32<T>((row[i] - mean) * s * weight[i] + (bias ? bias[i] : 0.f));
}

// The same for bfloat16 rows whose width is a multiple of 8 and at most 8192:
// every thread owns 8 consecutive channels, kept in registers through both passes.
__global__ void __launch_bounds__(1024)
add_layernorm_bf16_vec_kernel(float* __restrict__ residual, const bf16* __restrict__ pending,
                              const float* __restrict__ weight, const float* __restrict__ bias, float eps,
                              bf16* __restrict__ out, const int* __restrict__ rows, int H) {
    chain_release();
    chain_wait();
    __shared__ float scratch[33];
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    const int c = threadIdx.x * 8;
    const bool active = c < H;
    float x[8];
    float sum = 0.f;
    if (active) {
        float4* rp = reinterpret_cast<float4*>(residual + (size_t)r * H + c);
        const float4 a = rp[0], b = rp[1];
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
        if (pending) {
            const uint4 p = *reinterpret_cast<const uint4*>(pending + (size_t)r * H + c);
            const __nv_bfloat162* ph = reinterpret_cast<const __nv_bfloat162*>(&p);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(ph[j]);
                x[2 * j] += f.x;
                x[2 * j + 1] += f.y;
            }
            if (!rows) {
                rp[0] = make_float4(x[0], x[1], x[2], x[3]);
                rp[1] = make_float4(x[4], x[5], x[6], x[7]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) sum += x[j];
    }
    const float mean = block_sum(sum, scratch) / (float)H;
    float ss = 0.f;
    if (active) {
#pragma unroll
        for (int j = 0; j < 8; ++j) { x[j] -= mean; ss += x[j] * x[j]; }
    }
    const float var = block_sum(ss, scratch) / (float)H;
    const float s = 1.0f / sqrtf(var + eps);
    if (active) {
        const float4* wp = reinterpret_cast<const float4*>(weight + c);
        const float4 w0 = wp[0], w1 = wp[1];
        const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
        float bb[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (bias) {
            const float4* bp = reinterpret_cast<const float4*>(bias + c);
            const float4 b0 = bp[0], b1 = bp[1];
            bb[0] = b0.x; bb[1] = b0.y; bb[2] = b0.z; bb[3] = b0.w; bb[4] = b1.x; bb[5] = b1.y; bb[6] = b1.z; bb[7] = b1.w;
        }
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            oh[j] = __floats2bfloat162_rn(x[2 * j] * s * w[2 * j] + bb[2 * j], x[2 * j + 1] * s * w[2 * j + 1] + bb[2 * j + 1]);
        *reinterpret_cast<uint4*>(out + (size_t)i_out * H + c) = o;
    }
}

GTG_API int gtg_add_layernorm(int dtype, float* residual, const void* pending, const float* weight,
                              const float* bias, float eps, void* out, const int* rows, int R, int H,
                              cudaStream_t stream) {
    if (R <= 0) return 0;
    if (dtype == 1 && H % 8 == 0 && H <= 8192 && ((uintptr_t)residual % 16) == 0 && ((uintptr_t)out % 16) == 0 &&
        ((uintptr_t)weight % 16) == 0 && ((uintptr_t)bias % 16) == 0 && ((uintptr_t)pending % 16) == 0) {
        const int t = ((H / 8) + 31) / 32 * 32;
        return launch_chained(add_layernorm_bf16_vec_kernel, dim3(R), dim3(t), 0, stream, residual, (const bf16*)pending, weight, bias, eps, (bf16*)out, rows, H);
    }
    int threads = 32;
    while (threads < 1024 && threads * 4 < H) threads *= 2;
    const size_t smem = (size_t)(H + 33) * sizeof(float);
    if (smem > 200 * 1024) return kErrUnsupported;
    cudaError_t e;
    if (dtype == 0) {
        if (smem > 48 * 1024) {
            e = cudaFuncSetAttribute(add_layernorm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        return launch_chained(add_layernorm_kernel<float>, dim3(R), dim3(threads), smem, stream, residual, (const float*)pending, weight, bias, eps, (float*)out, rows, H);
    }
    if (dtype == 1) {
        if (smem > 48 * 1024) {
            e = cudaFuncSetAttribute(add_layernorm_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        return launch_chained(add_layernorm_kernel<bf16>, dim3(R), dim3(threads), smem, stream, residual, (const bf16*)pending, weight, bias, eps, (bf16*)out, rows, H);
    }
    return kErrBadArgument;
}

// ----------------------------- a normed update joins the hidden state, which is normed again
// x = residual[r,:] + LN(update[r,:]; weight_u);  out[i,:] = LN(x; weight) + bias, LN(x; w) =
// (x - mean) / sqrt(var + eps) * w, var the mean of the squared deviations: the arrangement in which a
// sublayer stands between two norms, the second of which meets the first of the next sublayer here.
// U is the update's type (float from a product that kept its sums).  Rows as in add_rmsnorm: with `rows`
// nothing is written back.  Everything in float.
//
// With `ex.top` > 0 the update is that of a mixture of experts and is summed here: of row r, the weighted sum of its
// experts' rows ex.y[ex.item_row[r top + k],:] (an item without a row: of the mixture's input ex.x[r,:]), k in order, and
// ex.base[r,:] last; `update` is then not read.
struct ExpertRows {
    const float* y;
    int ldy;
    const int* item_row;
    const float* weights;
    const void* x;               // of the output's type, or null
    int ldx;
    const float* base;           // or null
    int top;
};
template <typename U, typename T>
__global__ void layernorm_add_layernorm_kernel(float* __restrict__ residual, const U* __restrict__ update,
                                               const float* __restrict__ weight_u, float eps_u,
                                               const float* __restrict__ weight, const float* __restrict__ bias, float eps,
                                               T* __restrict__ out, const int* __restrict__ rows, int H, ExpertRows ex) {
    chain_release();
    chain_wait();
    extern __shared__ float smem[];
    float* row = smem;          // H floats
    float* scratch = smem + H;  // 33 floats
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    float* res = residual + (size_t)r * H;
    const U* up = update + (size_t)r * H;
    auto deviation = [&](float sum, float& mean) {          // of the row in shared memory: its mean and its variance
        mean = block_sum(sum, scratch) / (float)H;
        float ss = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            const float d = row[i] - mean;
            ss += d * d;
        }
        return block_sum(ss, scratch) / (float)H;
    };
    float sum = 0.f, mean;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float u = 0.f;
        if (ex.top > 0) {
            for (int k = 0; k < ex.top; ++k) {
                const int er = ex.item_row[(size_t)r * ex.top + k];
                const float v = er >= 0 ? ex.y[(size_t)er * ex.ldy + i] : to_f32<T>(reinterpret_cast<const T*>(ex.x)[(size_t)r * ex.ldx + i]);
                u = fmaf(ex.weights[(size_t)r * ex.top + k], v, u);
            }
            if (ex.base) u += ex.base[(size_t)r * H + i];
        } else {
            u = to_f32<U>(up[i]);
        }
        row[i] = u;
        sum += u;
    }
    float s = 1.0f / sqrtf(deviation(sum, mean) + eps_u);
    sum = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float x = res[i] + (row[i] - mean) * s * weight_u[i];
        if (!rows) res[i] = x;
        row[i] = x;
        sum += x;
    }
    s = 1.0f / sqrtf(deviation(sum, mean) + eps);
    T* o = out + (size_t)i_out * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x)
        o[i] = from_f32<T>((row[i] - mean) * s * weight[i] + (bias ? bias[i] : 0.f));
}

// Sum over the block with one barrier: every warp leaves its sum in `part` and every thread adds them up.
// Sums that follow one another use different `part`s (32 floats each).
__device__ __forceinline__ float block_sum_once(float v, float* part) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    const int n = blockDim.x >> 5;
    float t = 0.f;
    for (int w = 0; w < n; ++w) t += part[w];
    return t;
}

__device__ __forceinline__ void load_eight(const float* p, float* x) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}
__device__ __forceinline__ void load_eight(const bf16* p, float* x) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(h[j]);
        x[2 * j] = f.x;
        x[2 * j + 1] = f.y;
    }
}

// The same for bfloat16 rows whose width is a multiple of 8 and at most 8192: every thread owns 8
// consecutive channels, kept in registers from the first read to the last write.
template <typename U, bool kExperts>
__global__ void __launch_bounds__(1024)
layernorm_add_layernorm_vec_kernel(float* __restrict__ residual, const U* __restrict__ update,
                                   const float* __restrict__ weight_u, float eps_u,
                                   const float* __restrict__ weight, const float* __restrict__ bias, float eps,
                                   bf16* __restrict__ out, const int* __restrict__ rows, int H, ExpertRows ex) {
    chain_release();
    chain_wait();        // before every load: one through a restricted pointer to const may be moved over a later wait
    __shared__ float part[4][32];
    const int c = threadIdx.x * 8;
    const bool active = c < H;
    float wu[8], w[8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (active) {
        load_eight(weight_u + c, wu);
        load_eight(weight + c, w);
        if (bias) load_eight(bias + c, b);
    }
    const int i_out = blockIdx.x;
    const int r = rows ? rows[i_out] : i_out;
    float u[8], x[8];
    float* rp = residual + (size_t)r * H + c;
    float sum = 0.f;
    if (active) {
        load_eight(rp, x);
        if constexpr (kExperts) {
#pragma unroll
            for (int j = 0; j < 8; ++j) u[j] = 0.f;
#pragma unroll 4
            for (int k = 0; k < ex.top; ++k) {
                const int er = ex.item_row[(size_t)r * ex.top + k];
                const float f = ex.weights[(size_t)r * ex.top + k];
                float v[8];
                if (er >= 0) load_eight(ex.y + (size_t)er * ex.ldy + c, v);
                else load_eight(reinterpret_cast<const bf16*>(ex.x) + (size_t)r * ex.ldx + c, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) u[j] = fmaf(f, v[j], u[j]);
            }
            if (ex.base) {
                float v[8];
                load_eight(ex.base + (size_t)r * H + c, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) u[j] += v[j];
            }
        } else {
            load_eight(update + (size_t)r * H + c, u);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) sum += u[j];
    }
    float mean = block_sum_once(sum, part[0]) / (float)H;
    float ss = 0.f;
    if (active) {
#pragma unroll
        for (int j = 0; j < 8; ++j) { u[j] -= mean; ss += u[j] * u[j]; }
    }
    float s = 1.0f / sqrtf(block_sum_once(ss, part[1]) / (float)H + eps_u);
    sum = 0.f;
    if (active) {
#pragma unroll
        for (int j = 0; j < 8; ++j) { x[j] += u[j] * s * wu[j]; sum += x[j]; }
        if (!rows) {
            reinterpret_cast<float4*>(rp)[0] = make_float4(x[0], x[1], x[2], x[3]);
            reinterpret_cast<float4*>(rp)[1] = make_float4(x[4], x[5], x[6], x[7]);
        }
    }
    mean = block_sum_once(sum, part[2]) / (float)H;
    ss = 0.f;
    if (active) {
#pragma unroll
        for (int j = 0; j < 8; ++j) { x[j] -= mean; ss += x[j] * x[j]; }
    }
    s = 1.0f / sqrtf(block_sum_once(ss, part[3]) / (float)H + eps);
    if (active) {
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            oh[j] = __floats2bfloat162_rn(x[2 * j] * s * w[2 * j] + b[2 * j], x[2 * j + 1] * s * w[2 * j + 1] + b[2 * j + 1]);
        *reinterpret_cast<uint4*>(out + (size_t)i_out * H + c) = o;
    }
}

GTG_API int gtg_layernorm_add_layernorm(int dtype, int update_f32, float* residual, const void* update, const float* weight_u,
                                        float eps_u, const float* weight, const float* bias, float eps, void* out,
                                        const int* rows, int R, int H, const float* y, int ldy, const int* item_row,
                                        const float* expert_weights, const void* x, int ldx, const float* base, int top,
                                        cudaStream_t stream) {
    if (R <= 0) return 0;
    if (H <= 0 || (!update && top <= 0) || !weight_u || !weight) return kErrBadArgument;
    if (top > 0 && (!y || ldy < H || !item_row || !expert_weights || (x && ldx < H))) return kErrBadArgument;
    const ExpertRows ex{y, ldy, item_row, expert_weights, x, ldx, base, top};
    const bool ex_wide = top <= 0 || (ldy % 4 == 0 && ldx % 8 == 0 && ((uintptr_t)y % 16) == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)base % 16) == 0);
    if (ex_wide && dtype == 1 && H % 8 == 0 && H <= 8192 && ((uintptr_t)residual % 16) == 0 && ((uintptr_t)out % 16) == 0 &&
        ((uintptr_t)weight % 16) == 0 && ((uintptr_t)weight_u % 16) == 0 && ((uintptr_t)bias % 16) == 0 && ((uintptr_t)update % 16) == 0) {
        const int t = ((H / 8) + 31) / 32 * 32;
#define GTG_NORM_ADD_NORM_VEC(U, EX)                                                                             \
        return launch_chained(layernorm_add_layernorm_vec_kernel<U, EX>, dim3(R), dim3(t), 0, stream, residual, (const U*)update, \
                              weight_u, eps_u, weight, bias, eps, (bf16*)out, rows, H, ex)
        if (top > 0) GTG_NORM_ADD_NORM_VEC(float, true);
        if (update_f32) GTG_NORM_ADD_NORM_VEC(float, false);
        GTG_NORM_ADD_NORM_VEC(bf16, false);
#undef GTG_NORM_ADD_NORM_VEC
    }
    int threads = 32;
    while (threads < 1024 && threads * 4 < H) threads *= 2;
    const size_t smem = (size_t)(H + 33) * sizeof(float);
    if (smem > 200 * 1024) return kErrUnsupported;
#define GTG_NORM_ADD_NORM(U, T)                                                                                  \
    do {                                                                                                         \
        if (smem > 48 * 1024) {                                                                                  \
            const cudaError_t e = cudaFuncSetAttribute(layernorm_add_layernorm_kernel<U, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                 \
        }                                                                                                        \
        return launch_chained(layernorm_add_layernorm_kernel<U, T>, dim3(R), dim3(threads), smem, stream, residual, (const U*)update, \
                              weight_u, eps_u, weight, bias, eps, (T*)out, rows, H, ex);                         \
    } while (0)
    if (dtype == 0) GTG_NORM_ADD_NORM(float, float);
    if (dtype == 1 && update_f32) GTG_NORM_ADD_NORM(float, bf16);
    if (dtype == 1) GTG_NORM_ADD_NORM(bf16, bf16);
#undef GTG_NORM_ADD_NORM
    return kErrBadArgument;
}

// ------------------------------------------------------ pointwise activations
// x <- f(x) in place, evaluated in float.  kind 0: relu(x)^2; 1: gelu in its tanh
// form, 0.5 x (1 + tanh(sqrt(2/pi) (x + 0.044715 x^3))); 2: silu, x / (1 + exp(-x)).
template <typename T>
__global__ void activation_kernel(T* __restrict__ x, int ld, int M, int I, int kind) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * I;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / I;
        T* p = x + m * ld + (idx - m * I);
        *p = from_f32<T>(activate(to_f32<T>(*p), kind));
    }
}

// The same for bfloat16 rows of 16-byte aligned runs: 8 values per thread and access.
__global__ void activation_bf16_vec_kernel(bf16* __restrict__ x, int ld, int M, int I8, int kind) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * I8;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / I8;
        uint4* p = reinterpret_cast<uint4*>(x + m * ld + (idx - m * I8) * 8);
        uint4 v = *p;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(h[e]);
            h[e] = __floats2bfloat162_rn(activate(f.x, kind), activate(f.y, kind));
        }
        *p = v;
    }
}

GTG_API int gtg_activation(int dtype, void* x, int ld, int M, int I, int kind, cudaStream_t stream) {
    if (M <= 0 || I <= 0) return 0;
    if (kind < 0 || kind > 2 || ld < I) return kErrBadArgument;
    if (dtype == 1 && I % 8 == 0 && ld % 8 == 0 && ((uintptr_t)x % 16) == 0) {
        const size_t total8 = (size_t)M * (I / 8);
        const int blocks8 = (int)((total8 + 255) / 256 > 148 * 16 ? 148 * 16 : (total8 + 255) / 256);
        return launch_chained(activation_bf16_vec_kernel, dim3(blocks8), dim3(256), 0, stream, (bf16*)x, ld, M, I / 8, kind);
    }
    const size_t total = (size_t)M * I;
    int blocks = (int)((total + 255) / 256 > 148 * 16 ? 148 * 16 : (total + 255) / 256);
    if (dtype == 0) return launch_chained(activation_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)x, ld, M, I, kind);
    if (dtype == 1) return launch_chained(activation_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (bf16*)x, ld, M, I, kind);
    return kErrBadArgument;
}

// ------------------------------------------------------------- soft cap
// x <- cap * tanh(x / cap) on float logits, in place.
__global__ void softcap_kernel(float* __restrict__ x, size_t total, float cap) {
    chain_release();
    chain_wait();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x)
        x[idx] = cap * tanhf(x[idx] / cap);
}

GTG_API int gtg_softcap(float* x, long long total, float cap, cudaStream_t stream) {
    if (total <= 0) return 0;
    if (!(cap > 0.f)) return kErrBadArgument;
    const long long want = (total + 255) / 256;
    const int blocks = (int)(want > 148 * 16 ? 148 * 16 : want);
    return launch_chained(softcap_kernel, dim3(blocks), dim3(256), 0, stream, x, (size_t)total, cap);
}

// ---------------------------------------- hidden state beside a kept tensor
// out[n, 0:H] = residual[n,:] (+ pending[n,:]);  out[n, H:2H] = other[n,:]: the
// operand of a projection that mixes the hidden state with a tensor kept from
// earlier in the step (the embedding output).  The sum is float; out is the
// compute type.
template <typename T>
__global__ void hidden_concat_kernel(const float* __restrict__ residual, const T* __restrict__ pending,
                                     const float* __restrict__ other, T* __restrict__ out, int H) {
    chain_release();
    chain_wait();
    const size_t n = blockIdx.x;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float x = residual[n * H + i];
        if (pending) x += to_f32<T>(pending[n * H + i]);
        out[n * 2 * H + i] = from_f32<T>(x);
        out[n * 2 * H + H + i] = from_f32<T>(other[n * H + i]);
    }
}

GTG_API int gtg_hidden_concat(int dtype, const float* residual, const void* pending, const float* other,
                              void* out, int N, int H, cudaStream_t stream) {
    if (N <= 0 || H <= 0) return 0;
    const int threads = H >= 1024 ? 256 : 128;
    if (dtype == 0) return launch_chained(hidden_concat_kernel<float>, dim3(N), dim3(threads), 0, stream, residual, (const float*)pending, other, (float*)out, H);
    if (dtype == 1) return launch_chained(hidden_concat_kernel<bf16>, dim3(N), dim3(threads), 0, stream, residual, (const bf16*)pending, other, (bf16*)out, H);
    return kErrBadArgument;
}

// ---- the norm of an update, added to the hidden state ---------------------------
// residual[r,:] += rmsnorm(update[r,:] (+ bias)) * weight, everything in float; the
// arrangement in which a sublayer's output is normed and the sublayers read the
// hidden state itself.  `image`, if given, receives the new hidden state rounded
// to T: what the next sublayer's products read.  U is the update's type (the
// activation type, or float from a product that kept its sums).
template <typename U, typename T>
__global__ void rmsnorm_add_kernel(const U* __restrict__ update, const float* __restrict__ bias,
                                   const float* __restrict__ weight, float eps, float* __restrict__ residual,
                                   T* __restrict__ image, int H) {
    chain_release();
    chain_wait();
    extern __shared__ float dyn_smem[];
    float* row = dyn_smem;
    float* scratch = dyn_smem + H;
    const size_t base = (size_t)blockIdx.x * H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float u = to_f32<U>(update[base + i]);
        if (bias) u += bias[i];
        row[i] = u;
        ss += u * u;
    }
    const float total = block_sum(ss, scratch);
    const float s = 1.0f / sqrtf(total / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float x = residual[base + i] + (weight[i] * row[i]) * s;
        residual[base + i] = x;
        if (image) image[base + i] = from_f32<T>(x);
    }
}

// The same for rows of a multiple of 8 channels, at most 8192, with a bfloat16 image: every
// thread owns 8 consecutive channels, moved by 16- and 32-byte accesses and kept in registers
// between the sum of squares and the addition.
template <typename U>
__global__ void __launch_bounds__(1024)
rmsnorm_add_vec_kernel(const U* __restrict__ update, const float* __restrict__ bias, const float* __restrict__ weight,
                       float eps, float* __restrict__ residual, bf16* __restrict__ image, int H) {
    chain_release();
    chain_wait();
    __shared__ float scratch[33];
    const int c = threadIdx.x * 8;
    const bool active = c < H;
    const size_t base = (size_t)blockIdx.x * H + c;
    float u[8];
    float ss = 0.f;
    if (active) {
        if (sizeof(U) == 4) {
            const float4* up = reinterpret_cast<const float4*>(update + base);
            const float4 a = up[0], b = up[1];
            u[0] = a.x; u[1] = a.y; u[2] = a.z; u[3] = a.w; u[4] = b.x; u[5] = b.y; u[6] = b.z; u[7] = b.w;
        } else {
            const uint4 p = *reinterpret_cast<const uint4*>(update + base);
            const __nv_bfloat162* ph = reinterpret_cast<const __nv_bfloat162*>(&p);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = __bfloat1622float2(ph[j]);
                u[2 * j] = f.x;
                u[2 * j + 1] = f.y;
            }
        }
        if (bias) {
#pragma unroll
            for (int j = 0; j < 8; ++j) u[j] += bias[c + j];
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += u[j] * u[j];
    }
    const float total = block_sum(ss, scratch);
    const float s = 1.0f / sqrtf(total / (float)H + eps);
    if (active) {
        const float4* wp = reinterpret_cast<const float4*>(weight + c);
        const float4 w0 = wp[0], w1 = wp[1];
        const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
        float4* rp = reinterpret_cast<float4*>(residual + base);
        const float4 a = rp[0], b = rp[1];
        float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] += (w[j] * u[j]) * s;
        rp[0] = make_float4(x[0], x[1], x[2], x[3]);
        rp[1] = make_float4(x[4], x[5], x[6], x[7]);
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j) oh[j] = __floats2bfloat162_rn(x[2 * j], x[2 * j + 1]);
        *reinterpret_cast<uint4*>(image + base) = o;
    }
}

GTG_API int gtg_rmsnorm_add(int dtype, int update_f32, const void* update, const float* bias, const float* weight,
                            float eps, float* residual, void* image, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    if (H <= 0) return kErrBadArgument;
    if (dtype == 1 && image && H % 8 == 0 && H <= 8192 && ((uintptr_t)update % 16) == 0 && ((uintptr_t)residual % 16) == 0 &&
        ((uintptr_t)image % 16) == 0 && ((uintptr_t)weight % 16) == 0) {
        const int t = ((H / 8) + 31) / 32 * 32;
        if (update_f32)
            return launch_chained(rmsnorm_add_vec_kernel<float>, dim3(R), dim3(t), 0, stream, (const float*)update, bias, weight,
                                  eps, residual, (bf16*)image, H);
        return launch_chained(rmsnorm_add_vec_kernel<bf16>, dim3(R), dim3(t), 0, stream, (const bf16*)update, bias, weight,
                              eps, residual, (bf16*)image, H);
    }
    int threads = 32;
    while (threads < 1024 && threads * 4 < H) threads *= 2;
    const size_t smem = (size_t)(H + 33) * sizeof(float);
    if (smem > 200 * 1024) return kErrUnsupported;
    cudaError_t e = cudaSuccess;
#define GTG_NORM_ADD(U, T)                                                                                       \
    do {                                                                                                         \
        if (smem > 48 * 1024)                                                                                    \
            e = cudaFuncSetAttribute(rmsnorm_add_kernel<U, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) return (int)e;                                                                     \
        return launch_chained(rmsnorm_add_kernel<U, T>, dim3(R), dim3(threads), smem, stream, (const U*)update,  \
                              bias, weight, eps, residual, (T*)image, H);                                        \
    } while (0)
    if (dtype == 0) GTG_NORM_ADD(float, float);
    if (dtype == 1 && update_f32) GTG_NORM_ADD(float, bf16);
    if (dtype == 1) GTG_NORM_ADD(bf16, bf16);
#undef GTG_NORM_ADD
    return kErrBadArgument;
}

// out[r,:] = T(x[r,:]): the hidden state rounded to the activation type.
template <typename T>
__global__ void round_rows_kernel(const float* __restrict__ x, T* __restrict__ out, size_t total) {
    chain_release();
    chain_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
        out[i] = from_f32<T>(x[i]);
}

GTG_API int gtg_round_rows(int dtype, const float* x, void* out, long long total, cudaStream_t stream) {
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 1023) / 1024 > 4096 ? 4096 : (total + 1023) / 1024);
    if (dtype == 0) return launch_chained(round_rows_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, (float*)out, (size_t)total);
    if (dtype == 1) return launch_chained(round_rows_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, x, (bf16*)out, (size_t)total);
    return kErrBadArgument;
}

// ---- biases ------------------------------------------------------------------------
// out[m,i] = silu(gu[m,i] + bg[i]) * (gu[m,I+i] + bu[i]) from a product's float sums; with another gated
// epilogue's `code` than 1, that product of the two in silu's place.
template <typename T>
__global__ void swiglu_bias_kernel(const float* __restrict__ gu, const float* __restrict__ bg,
                                   const float* __restrict__ bu, T* __restrict__ out, int ldo, int M, int I, int code) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * I;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / I;
        const int i = (int)(idx % I);
        const float g = gu[m * 2 * I + i] + (bg ? bg[i] : 0.f);
        const float u = gu[m * 2 * I + I + i] + (bu ? bu[i] : 0.f);
        out[m * ldo + i] = from_f32<T>(gated_value(g, u, code));
    }
}

GTG_API int gtg_swiglu_bias(int dtype, const float* gu, const float* bg, const float* bu, void* out, int ldo,
                            int M, int I, int code, cudaStream_t stream) {
    if (M <= 0 || I <= 0) return 0;
    if (!epi_is_gated(code)) return kErrBadArgument;
    const size_t total = (size_t)M * I;
    const unsigned blocks = (unsigned)((total + 255) / 256 > 8192 ? 8192 : (total + 255) / 256);
    if (dtype == 0) return launch_chained(swiglu_bias_kernel<float>, dim3(blocks), dim3(256), 0, stream, gu, bg, bu, (float*)out, ldo, M, I, code);
    if (dtype == 1) return launch_chained(swiglu_bias_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, gu, bg, bu, (bf16*)out, ldo, M, I, code);
    return kErrBadArgument;
}

// out[m,n] = T(x[m,n] + b[n]) from a product's float sums.
template <typename T>
__global__ void add_bias_kernel(const float* __restrict__ x, const float* __restrict__ b, T* __restrict__ out,
                                int M, int N) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * N;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x)
        out[idx] = from_f32<T>(x[idx] + b[idx % N]);
}

GTG_API int gtg_add_bias(int dtype, const float* x, const float* b, void* out, int M, int N, cudaStream_t stream) {
    if (M <= 0 || N <= 0) return 0;
    const size_t total = (size_t)M * N;
    const unsigned blocks = (unsigned)((total + 255) / 256 > 8192 ? 8192 : (total + 255) / 256);
    if (dtype == 0) return launch_chained(add_bias_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, b, (float*)out, M, N);
    if (dtype == 1) return launch_chained(add_bias_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, x, b, (bf16*)out, M, N);
    return kErrBadArgument;
}

// x[m,n] *= sigmoid(g[m,n]), the product evaluated in float: a gate on a mixer's heads.  The logits g
// are of x's type or float (a projection's sums).
template <typename T, typename G>
__global__ void sigmoid_gate_kernel(T* __restrict__ x, int ldx, const G* __restrict__ g, int ldg, int M, int N) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * N;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / N;
        const int n = (int)(idx % N);
        const float gate = 1.0f / (1.0f + expf(-to_f32<G>(g[m * ldg + n])));
        x[m * ldx + n] = from_f32<T>(to_f32<T>(x[m * ldx + n]) * gate);
    }
}

// The same for bfloat16 rows and float logits whose rows allow 16-byte accesses: eight channels a thread.
__global__ void sigmoid_gate_bf16_f32_vec_kernel(bf16* __restrict__ x, int ldx, const float* __restrict__ g, int ldg, int M, int N8) {
    chain_release();
    chain_wait();
    const size_t total = (size_t)M * N8;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t m = idx / N8;
        const int c = (int)(idx % N8) * 8;
        uint4 xv = *reinterpret_cast<const uint4*>(x + m * ldx + c);
        const float4 g0 = *reinterpret_cast<const float4*>(g + m * ldg + c), g1 = *reinterpret_cast<const float4*>(g + m * ldg + c + 4);
        const float gg[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
        __nv_bfloat162* xh = reinterpret_cast<__nv_bfloat162*>(&xv);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(xh[e]);
            xh[e] = __floats2bfloat162_rn(f.x * (1.0f / (1.0f + expf(-gg[2 * e]))), f.y * (1.0f / (1.0f + expf(-gg[2 * e + 1]))));
        }
        *reinterpret_cast<uint4*>(x + m * ldx + c) = xv;
    }
}

GTG_API int gtg_sigmoid_gate(int dtype, void* x, int ldx, const void* g, int ldg, int M, int N, int gate_f32, cudaStream_t stream) {
    if (M <= 0 || N <= 0) return 0;
    if (dtype == 1 && gate_f32 && N % 8 == 0 && ldx % 8 == 0 && ldg % 4 == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)g % 16) == 0) {
        const size_t total8 = (size_t)M * (N / 8);
        const unsigned blocks8 = (unsigned)((total8 + 255) / 256 > 148 * 16 ? 148 * 16 : (total8 + 255) / 256);
        return launch_chained(sigmoid_gate_bf16_f32_vec_kernel, dim3(blocks8), dim3(256), 0, stream, (bf16*)x, ldx, (const float*)g, ldg, M, N / 8);
    }
    const size_t total = (size_t)M * N;
    const unsigned blocks = (unsigned)((total + 255) / 256 > 8192 ? 8192 : (total + 255) / 256);
    if (dtype == 0) return launch_chained(sigmoid_gate_kernel<float, float>, dim3(blocks), dim3(256), 0, stream, (float*)x, ldx, (const float*)g, ldg, M, N);
    if (dtype == 1 && gate_f32) return launch_chained(sigmoid_gate_kernel<bf16, float>, dim3(blocks), dim3(256), 0, stream, (bf16*)x, ldx, (const float*)g, ldg, M, N);
    if (dtype == 1) return launch_chained(sigmoid_gate_kernel<bf16, bf16>, dim3(blocks), dim3(256), 0, stream, (bf16*)x, ldx, (const bf16*)g, ldg, M, N);
    return kErrBadArgument;
}

// ---- a norm of the float hidden state in place, a factor on float rows -------------
// x[n,:] <- x[n,:] / sqrt(mean(x[n,:]^2) + eps) * w, float throughout: the norm that
// stands directly behind the token embedding and changes the hidden state itself.
__global__ void rmsnorm_rows_kernel(float* __restrict__ x, const float* __restrict__ w, float eps, int H) {
    chain_release();
    chain_wait();
    __shared__ float scratch[33];
    float* row = x + (size_t)blockIdx.x * H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
    const float total = block_sum(ss, scratch);
    const float s = 1.0f / sqrtf(total / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = row[i] * s * w[i];
}

GTG_API int gtg_rmsnorm_rows(float* x, const float* w, float eps, int N, int H, cudaStream_t stream) {
    if (N <= 0 || H <= 0) return 0;
    const int threads = H >= 1024 ? 256 : H >= 256 ? 128 : 64;
    return launch_chained(rmsnorm_rows_kernel, dim3(N), dim3(threads), 0, stream, x, w, eps, H);
}

__global__ void scale_kernel(float* __restrict__ x, size_t total, float factor) {
    chain_release();
    chain_wait();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x)
        x[idx] *= factor;
}

// x <- factor * x, float (a multiplier on the logits).
GTG_API int gtg_scale(float* x, long long total, float factor, cudaStream_t stream) {
    if (total <= 0) return 0;
    const long long want = (total + 255) / 256;
    const int blocks = (int)(want > 148 * 16 ? 148 * 16 : want);
    return launch_chained(scale_kernel, dim3(blocks), dim3(256), 0, stream, x, (size_t)total, factor);
}

// ---- two updates, each normed, averaged and added --------------------------------
// v = factor * (a / sqrt(mean(a^2) + eps) * wa + b / sqrt(mean(b^2) + eps) * wb), float
// throughout, per row of two sublayers' outputs; v joins the float rows `residual`, or,
// where that is null, goes to `out`.
template <typename T>
__global__ void normed_pair_kernel(const T* __restrict__ a, const T* __restrict__ b, const float* __restrict__ wa,
                                   const float* __restrict__ wb, float eps, float factor, float* __restrict__ residual,
                                   T* __restrict__ out, int H) {
    chain_release();
    chain_wait();
    extern __shared__ float smem[];
    float* ra = smem;
    float* rb = smem + H;
    float* scratch = smem + 2 * H;
    const size_t base = (size_t)blockIdx.x * H;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float x = to_f32<T>(a[base + i]), y = to_f32<T>(b[base + i]);
        ra[i] = x;
        rb[i] = y;
        sa += x * x;
        sb += y * y;
    }
    sa = factor / sqrtf(block_sum(sa, scratch) / (float)H + eps);
    sb = factor / sqrtf(block_sum(sb, scratch) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = ra[i] * sa * wa[i] + rb[i] * sb * wb[i];
        if (residual) residual[base + i] += v;
        else out[base + i] = from_f32<T>(v);
    }
}

// The same for bfloat16 rows of a multiple of 8 channels, at most 8192: a thread owns 8
// neighbouring channels of both rows in registers.
__global__ void __launch_bounds__(1024)
normed_pair_bf16_vec_kernel(const bf16* __restrict__ a, const bf16* __restrict__ b, const float* __restrict__ wa,
                            const float* __restrict__ wb, float eps, float factor, float* __restrict__ residual,
                            bf16* __restrict__ out, int H) {
    chain_release();
    chain_wait();
    __shared__ float part[2][32];
    const int c = threadIdx.x * 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const bool active = c < H;
    const size_t base = (size_t)blockIdx.x * H + c;
    float x[8], y[8], r[8];
    float sa = 0.f, sb = 0.f;
    if (active) {
        const uint4 ua = *reinterpret_cast<const uint4*>(a + base), ub = *reinterpret_cast<const uint4*>(b + base);
        if (residual) {
            const float4 r0 = reinterpret_cast<const float4*>(residual + base)[0], r1 = reinterpret_cast<const float4*>(residual + base)[1];
            r[0] = r0.x; r[1] = r0.y; r[2] = r0.z; r[3] = r0.w; r[4] = r1.x; r[5] = r1.y; r[6] = r1.z; r[7] = r1.w;
        }
        const __nv_bfloat162* ha = reinterpret_cast<const __nv_bfloat162*>(&ua);
        const __nv_bfloat162* hb = reinterpret_cast<const __nv_bfloat162*>(&ub);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(ha[j]), g = __bfloat1622float2(hb[j]);
            x[2 * j] = f.x; x[2 * j + 1] = f.y;
            y[2 * j] = g.x; y[2 * j + 1] = g.y;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) { sa += x[j] * x[j]; sb += y[j] * y[j]; }
    }
    sa = warp_sum(sa);
    sb = warp_sum(sb);
    if (lane == 0) { part[0][warp] = sa; part[1][warp] = sb; }
    __syncthreads();
    if (!active) return;
    sa = sb = 0.f;
    for (int w = 0; w < warps; ++w) { sa += part[0][w]; sb += part[1][w]; }
    sa = factor / sqrtf(sa / (float)H + eps);
    sb = factor / sqrtf(sb / (float)H + eps);
    const float4 a0 = reinterpret_cast<const float4*>(wa + c)[0], a1 = reinterpret_cast<const float4*>(wa + c)[1];
    const float4 b0 = reinterpret_cast<const float4*>(wb + c)[0], b1 = reinterpret_cast<const float4*>(wb + c)[1];
    const float ua[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
    const float ub[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
    float v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = x[j] * sa * ua[j] + y[j] * sb * ub[j];
    if (residual) {
        reinterpret_cast<float4*>(residual + base)[0] = make_float4(r[0] + v[0], r[1] + v[1], r[2] + v[2], r[3] + v[3]);
        reinterpret_cast<float4*>(residual + base)[1] = make_float4(r[4] + v[4], r[5] + v[5], r[6] + v[6], r[7] + v[7]);
    } else {
        uint4 o;
        __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int j = 0; j < 4; ++j) oh[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
        *reinterpret_cast<uint4*>(out + base) = o;
    }
}

GTG_API int gtg_normed_pair(int dtype, const void* a, const void* b, const float* wa, const float* wb, float eps, float factor,
                            float* residual, void* out, int N, int H, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (H <= 0 || (residual == nullptr) == (out == nullptr)) return kErrBadArgument;
    if (dtype == 1 && H % 8 == 0 && H <= 8192 && ((uintptr_t)a % 16) == 0 && ((uintptr_t)b % 16) == 0 && ((uintptr_t)wa % 16) == 0 &&
        ((uintptr_t)wb % 16) == 0 && ((uintptr_t)residual % 16) == 0 && ((uintptr_t)out % 16) == 0)
        return launch_chained(normed_pair_bf16_vec_kernel, dim3(N), dim3((H / 8 + 31) / 32 * 32), 0, stream, (const bf16*)a, (const bf16*)b,
                              wa, wb, eps, factor, residual, (bf16*)out, H);
    int threads = 32;
    while (threads < 1024 && threads * 4 < H) threads *= 2;
    const size_t smem = (size_t)(2 * H + 33) * sizeof(float);
    if (smem > 200 * 1024) return kErrUnsupported;
#define GTG_PAIR(T)                                                                                                  \
    do {                                                                                                             \
        if (smem > 48 * 1024) {                                                                                      \
            const cudaError_t e = cudaFuncSetAttribute(normed_pair_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                     \
        }                                                                                                            \
        return launch_chained(normed_pair_kernel<T>, dim3(N), dim3(threads), smem, stream, (const T*)a, (const T*)b, wa, wb, eps, factor, \
                              residual, (T*)out, H);                                                                 \
    } while (0)
    if (dtype == 0) GTG_PAIR(float);
    if (dtype == 1) GTG_PAIR(bf16);
#undef GTG_PAIR
    return kErrBadArgument;
}
