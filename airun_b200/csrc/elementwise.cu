// Embedding gather, RMSNorm with the residual add (and a row gather) fused in,
// and the SwiGLU product.  All arithmetic is float32; storage may be bfloat16.
//
// Formulas as the reference computes them:
//   embedding  x[t] = E[token[t]], an id outside the table reads row 0
//              (crates/airun-cuda/kernels/ops.cu:227-252);
//   RMSNorm    out = x * rsqrt(sum(x^2)/n + eps) * w   (ops.cu:12-41);
//   add+norm   x += delta, then the norm of the sum    (ops.cu:47-78);
//   SwiGLU     out = g / (1 + exp(-g)) * u             (ops.cu:191-200).
#include "common.cuh"
#include <type_traits>

template <typename TTab>
__global__ void embed_kernel(const TTab* __restrict__ table, const int32_t* __restrict__ ids,
                             float* __restrict__ out, int H, int V, float scale, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    if (id < 0 || id >= V) {
        if (threadIdx.x == 0 && err) atomicOr(err, AIRUN_DEV_BAD_TOKEN);
        id = 0;
    }
    const TTab* src = table + (size_t)id * H;
    float* dst = out + (size_t)t * H;
    // scale 1 (no scaling, as the reference) leaves the value as it is: x * 1.0f is exact
    if ((H & 3) == 0 && ((uintptr_t)src & (4 * sizeof(TTab) - 1)) == 0 && ((uintptr_t)dst & 15) == 0) {
#pragma unroll 4
        for (int i = 4 * threadIdx.x; i < H; i += 4 * blockDim.x) {
            __align__(16) TTab v[4];
            if (sizeof(TTab) == 2) *reinterpret_cast<uint2*>(v) = *reinterpret_cast<const uint2*>(src + i);
            else *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(src + i);
            *reinterpret_cast<float4*>(dst + i) = make_float4(to_f32<TTab>(v[0]) * scale, to_f32<TTab>(v[1]) * scale,
                                                              to_f32<TTab>(v[2]) * scale, to_f32<TTab>(v[3]) * scale);
        }
        return;
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = to_f32<TTab>(src[i]) * scale;
}

AIRUN_EXPORT int airun_embed(const void* table, int table_dtype, const int32_t* ids, float* out,
                             int T, int H, int V, float scale, int* err, cudaStream_t stream) {
    if (T < 0 || H <= 0 || V <= 0) return AIRUN_ERR_ARG;
    if (T == 0) return AIRUN_OK;
    const int threads = H >= 1024 ? 256 : 128;
    if (table_dtype == AIRUN_DT_F32)
        airun_launch(embed_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table, ids, out, H, V, scale, err);
    else if (table_dtype == AIRUN_DT_BF16)
        airun_launch(embed_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const __nv_bfloat16*)table, ids, out, H, V, scale, err);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// One block per output row.  Source row = rows ? rows[r] : r.  With `delta` the
// sum x + delta is normed; it is written back to x only when write_back is set
// (a gathered final norm leaves x alone).  VEC = 4 reads float4 (n % 4 == 0) and keeps up to
// KEEP vectors per thread in registers between the two passes; longer rows are read again.
#define KEEP 4
template <typename TOut, int VEC>
__global__ void rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ delta,
                               const float* __restrict__ w, TOut* __restrict__ out,
                               const int32_t* __restrict__ rows, int n, float eps, int write_back,
                               const float* __restrict__ w2, TOut* __restrict__ out2) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[33];
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* xr = x + (size_t)src * n;
    const float* dr = delta ? delta + (size_t)src * n : nullptr;
    TOut* outr = out + (size_t)r * n;
    TOut* outr2 = out2 ? out2 + (size_t)r * n : nullptr;      // the same row under a second weight
    const int nv = n / VEC;                       // vectors in the row
    float keep[KEEP][VEC];
    float ss = 0.0f;
    // All loads of x and delta first, then the sums and the stores: a load issued after a store through the
    // same pointer waits for it, and four such round trips in turn were most of this kernel's time at a
    // few rows (3.9 us of a decode layer's two norms each).
    float dk[KEEP][VEC];
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
#pragma unroll
        for (int e = 0; e < VEC; ++e) { keep[k][e] = 0.0f; dk[k][e] = 0.0f; }
        if (i < nv) {
            if (VEC == 4) {
                const float4 v = reinterpret_cast<const float4*>(xr)[i];
                keep[k][0] = v.x; keep[k][1 % VEC] = v.y; keep[k][2 % VEC] = v.z; keep[k][3 % VEC] = v.w;
                if (dr) {
                    const float4 d = reinterpret_cast<const float4*>(dr)[i];
                    dk[k][0] = d.x; dk[k][1 % VEC] = d.y; dk[k][2 % VEC] = d.z; dk[k][3 % VEC] = d.w;
                }
            } else {
                keep[k][0] = xr[i];
                if (dr) dk[k][0] = dr[i];
            }
        }
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i < nv) {
            if (dr) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) keep[k][e] += dk[k][e];
                if (write_back) {
                    if (VEC == 4) reinterpret_cast<float4*>(xr)[i] = make_float4(keep[k][0], keep[k][1 % VEC], keep[k][2 % VEC], keep[k][3 % VEC]);
                    else xr[i] = keep[k][0];
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(keep[k][e], keep[k][e], ss);
        }
    }
    for (int i = threadIdx.x + KEEP * blockDim.x; i < nv; i += blockDim.x) {       // the rest of a long row
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float v = xr[i * VEC + e];
            if (dr) { v += dr[i * VEC + e]; if (write_back) xr[i * VEC + e] = v; }
            ss = fmaf(v, v, ss);
        }
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)n + eps);
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i < nv) {
#pragma unroll
            for (int e = 0; e < VEC; ++e)
                outr[i * VEC + e] = from_f32<TOut>(keep[k][e] * inv * (w ? w[i * VEC + e] : 1.0f));
            if (outr2) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) outr2[i * VEC + e] = from_f32<TOut>(keep[k][e] * inv * w2[i * VEC + e]);
            }
        }
    }
    for (int i = threadIdx.x + KEEP * blockDim.x; i < nv; i += blockDim.x) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float v = xr[i * VEC + e];
            if (dr && !write_back) v += dr[i * VEC + e];
            outr[i * VEC + e] = from_f32<TOut>(v * inv * (w ? w[i * VEC + e] : 1.0f));
            if (outr2) outr2[i * VEC + e] = from_f32<TOut>(v * inv * w2[i * VEC + e]);
        }
    }
}

// Many rows: one warp per row, no block-wide synchronisation.  The loads of a batch of RB float4 per
// lane (and as many of delta) are all issued before the first of them is used or anything is stored:
// a load after a store through the same pointer would otherwise wait for it.  The sum x + delta is
// written back and read again (from cache) for the second pass.
#define RB 8
template <typename TOut>
__global__ __launch_bounds__(256) void rmsnorm_rows_kernel(float* __restrict__ x, const float* __restrict__ delta,
                                                           const float* __restrict__ w, TOut* __restrict__ out,
                                                           int n_rows, int n, float eps, int write_back,
                                                           const float* __restrict__ w2, TOut* __restrict__ out2) {
    pdl_trigger();
    pdl_wait();
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (row >= n_rows) return;
    float4* xr = reinterpret_cast<float4*>(x + (size_t)row * n);
    const float4* dr = delta ? reinterpret_cast<const float4*>(delta + (size_t)row * n) : nullptr;
    const float4* w4 = reinterpret_cast<const float4*>(w);
    TOut* outr = out + (size_t)row * n;
    TOut* outr2 = out2 ? out2 + (size_t)row * n : nullptr;
    const float4* w24 = reinterpret_cast<const float4*>(w2);
    const int nv = n >> 2;
    float ss = 0.0f;
    const bool rewrite = dr && write_back;
    for (int i0 = lane; i0 < nv; i0 += 32 * RB) {
        float4 v[RB], d[RB];
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int i = i0 + 32 * u;
            v[u] = i < nv ? xr[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        if (dr) {
#pragma unroll
            for (int u = 0; u < RB; ++u) {
                const int i = i0 + 32 * u;
                d[u] = i < nv ? dr[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
#pragma unroll
            for (int u = 0; u < RB; ++u) { v[u].x += d[u].x; v[u].y += d[u].y; v[u].z += d[u].z; v[u].w += d[u].w; }
        }
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int i = i0 + 32 * u;
            if (rewrite && i < nv) xr[i] = v[u];
            ss = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, ss))));
        }
    }
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / (float)n + eps);
    for (int i0 = lane; i0 < nv; i0 += 32 * RB) {
        float4 v[RB], g[RB];
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int i = i0 + 32 * u;
            v[u] = i < nv ? xr[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            g[u] = (w && i < nv) ? w4[i] : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
        }
        if (dr && !rewrite) {
#pragma unroll
            for (int u = 0; u < RB; ++u) {
                const int i = i0 + 32 * u;
                if (i < nv) { const float4 d = dr[i]; v[u].x += d.x; v[u].y += d.y; v[u].z += d.z; v[u].w += d.w; }
            }
        }
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int i = i0 + 32 * u;
            if (i >= nv) continue;
            const float a = v[u].x * inv * g[u].x, b = v[u].y * inv * g[u].y, c = v[u].z * inv * g[u].z, d2 = v[u].w * inv * g[u].w;
            if (sizeof(TOut) == 4) {
                reinterpret_cast<float4*>(outr)[i] = make_float4(a, b, c, d2);
            } else {
                __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d2);
                uint2 pk;
                pk.x = *reinterpret_cast<uint32_t*>(&lo);
                pk.y = *reinterpret_cast<uint32_t*>(&hi);
                reinterpret_cast<uint2*>(outr)[i] = pk;
            }
            if (outr2) {
                const float4 g2 = w24[i];
                const float a2 = v[u].x * inv * g2.x, b2 = v[u].y * inv * g2.y, c2 = v[u].z * inv * g2.z, e2 = v[u].w * inv * g2.w;
                if (sizeof(TOut) == 4) {
                    reinterpret_cast<float4*>(outr2)[i] = make_float4(a2, b2, c2, e2);
                } else {
                    __nv_bfloat162 lo = __floats2bfloat162_rn(a2, b2), hi = __floats2bfloat162_rn(c2, e2);
                    uint2 pk;
                    pk.x = *reinterpret_cast<uint32_t*>(&lo);
                    pk.y = *reinterpret_cast<uint32_t*>(&hi);
                    reinterpret_cast<uint2*>(outr2)[i] = pk;
                }
            }
        }
    }
}

static int rmsnorm_launch(float* x, const float* delta, const float* w, void* out, int out_dtype,
                          const int32_t* rows, int n_rows, int n, float eps, int write_back,
                          const float* w2, void* out2, cudaStream_t stream) {
    if (n_rows < 0 || n <= 0 || ((w2 == nullptr) != (out2 == nullptr))) return AIRUN_ERR_ARG;
    if (rows && write_back) return AIRUN_ERR_ARG;
    if (n_rows == 0) return AIRUN_OK;
    const bool vec = n % 4 == 0 && (((uintptr_t)x | (uintptr_t)delta) & 15) == 0;
    if (vec && !rows && n_rows >= 256 && n >= 512 && (((uintptr_t)out | (uintptr_t)w | (uintptr_t)out2 | (uintptr_t)w2) & 15) == 0) {
        // enough warps per block that the blocks still cover the SMs twice
        const int wpb = n_rows >= 2368 ? 8 : n_rows >= 1184 ? 4 : 2;
        const int blocks = (n_rows + wpb - 1) / wpb;
        if (out_dtype == AIRUN_DT_F32)
            airun_launch(rmsnorm_rows_kernel<float>, dim3(blocks), dim3(32 * wpb), 0, stream, x, delta, w, (float*)out, n_rows, n, eps, write_back, w2, (float*)out2);
        else if (out_dtype == AIRUN_DT_BF16)
            airun_launch(rmsnorm_rows_kernel<__nv_bfloat16>, dim3(blocks), dim3(32 * wpb), 0, stream, x, delta, w, (__nv_bfloat16*)out, n_rows, n, eps, write_back, w2, (__nv_bfloat16*)out2);
        else
            return AIRUN_ERR_UNSUPPORTED;
        return airun_launch_status();
    }
    const int nv = vec ? n / 4 : n;
    int threads = (nv + 31) / 32 * 32;
    if (threads > 1024) threads = 1024;
    if (threads < 32) threads = 32;
    if (n_rows <= 64 && threads > 256 && vec) threads = 256;      // few rows: more loads in flight per thread
#define LAUNCH(TOut, VEC) \
    airun_launch(rmsnorm_kernel<TOut, VEC>, dim3(n_rows), dim3(threads), 0, stream, x, delta, w, (TOut*)out, rows, n, eps, write_back, w2, (TOut*)out2)
    if (out_dtype == AIRUN_DT_F32) { if (vec) LAUNCH(float, 4); else LAUNCH(float, 1); }
    else if (out_dtype == AIRUN_DT_BF16) { if (vec) LAUNCH(__nv_bfloat16, 4); else LAUNCH(__nv_bfloat16, 1); }
    else return AIRUN_ERR_UNSUPPORTED;
#undef LAUNCH
    return airun_launch_status();
}

AIRUN_EXPORT int airun_rmsnorm(float* x, const float* delta, const float* w, void* out, int out_dtype,
                               const int32_t* rows, int n_rows, int n, float eps, int write_back,
                               cudaStream_t stream) {
    return rmsnorm_launch(x, delta, w, out, out_dtype, rows, n_rows, n, eps, write_back, nullptr, nullptr, stream);
}

// The same row normed once and written under two weights: out = v / rms(v) * w and out2 = v / rms(v) * w2, the
// inputs of two sub-layers that read the residual stream side by side through norms of their own.
AIRUN_EXPORT int airun_rmsnorm_pair(float* x, const float* delta, const float* w, void* out, const float* w2, void* out2,
                                    int out_dtype, const int32_t* rows, int n_rows, int n, float eps, int write_back,
                                    cudaStream_t stream) {
    if (!w2 || !out2) return AIRUN_ERR_ARG;
    return rmsnorm_launch(x, delta, w, out, out_dtype, rows, n_rows, n, eps, write_back, w2, out2, stream);
}

// in: [T][2*I] where blocks of `group` gate columns alternate with blocks of
// `group` up columns (group == I means plain [gate | up] halves).  out: [T][I].
template <typename TIn, typename TOut>
__global__ void swiglu_kernel(const TIn* __restrict__ in, TOut* __restrict__ out,
                              long long total, int I, int group) {
    pdl_trigger();
    pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const long long t = idx / I;
    const int i = (int)(idx - t * I);
    const int b = i / group, o = i - b * group;
    const TIn* row = in + t * 2 * (long long)I;
    const float g = to_f32<TIn>(row[(size_t)(2 * b) * group + o]);
    const float u = to_f32<TIn>(row[(size_t)(2 * b + 1) * group + o]);
    out[idx] = from_f32<TOut>(g / (1.0f + expf(-g)) * u);
}

AIRUN_EXPORT int airun_swiglu(const void* in, int in_dtype, void* out, int out_dtype,
                              int T, int I, int group, cudaStream_t stream) {
    if (T < 0 || I <= 0 || group <= 0 || I % group != 0) return AIRUN_ERR_ARG;
    const long long total = (long long)T * I;
    if (total == 0) return AIRUN_OK;
    const int threads = 256;
    const int blocks = ceil_div_i(total, threads);
    if (in_dtype == AIRUN_DT_F32 && out_dtype == AIRUN_DT_F32)
        airun_launch(swiglu_kernel<float, float>, dim3(blocks), dim3(threads), 0, stream, (const float*)in, (float*)out, total, I, group);
    else if (in_dtype == AIRUN_DT_F32 && out_dtype == AIRUN_DT_BF16)
        airun_launch(swiglu_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(threads), 0, stream, (const float*)in, (__nv_bfloat16*)out, total, I, group);
    else if (in_dtype == AIRUN_DT_BF16 && out_dtype == AIRUN_DT_BF16)
        airun_launch(swiglu_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(blocks), dim3(threads), 0, stream, (const __nv_bfloat16*)in, (__nv_bfloat16*)out, total, I, group);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// out[r] = in[rows[r]] for rows of n elements of `elt` bytes (n*elt a multiple of 4).
__global__ void gather_rows_kernel(const uint32_t* __restrict__ in, uint32_t* __restrict__ out,
                                   const int32_t* __restrict__ rows, int words) {
    pdl_trigger();
    pdl_wait();
    const uint32_t* s = in + (size_t)rows[blockIdx.x] * words;
    uint32_t* d = out + (size_t)blockIdx.x * words;
    for (int i = threadIdx.x; i < words; i += blockDim.x) d[i] = s[i];
}

AIRUN_EXPORT int airun_gather_rows(const void* in, void* out, const int32_t* rows, int n_rows,
                                   int row_bytes, cudaStream_t stream) {
    if (n_rows < 0 || row_bytes <= 0 || row_bytes % 4 != 0) return AIRUN_ERR_ARG;
    if (n_rows == 0) return AIRUN_OK;
    airun_launch(gather_rows_kernel, dim3(n_rows), dim3(256), 0, stream, (const uint32_t*)in, (uint32_t*)out, rows, row_bytes / 4);
    return airun_launch_status();
}

// Random weights from a counter: element i of a tensor with key k is a function of (k, i) alone, so
// the host and the device fill the same tensor bit for bit and no generator state is carried.
//   h(c)  = mix(k + c * 0x9E3779B97F4A7C15), mix = the finaliser of splitmix64;
//   z     = (sum of the twelve 16-bit fields of h(3i), h(3i+1), h(3i+2) - 393210) / 65536:
//           integers up to there, so exact; mean 0, variance 1 - 2^-32, |z| <= 6;
//   kind 0: w = z * scale            (one float32 product)
//   kind 1: w = 1 + z * scale        (product, then sum: two roundings, never fused)
//   kind 2: w = h(3i) & 0x7fff       (int32)
// The reference has no random-weights mode; its benchmark makes token ids from a seeded xorshift the
// same stateless way (crates/airun-cli/src/bench.rs:177-187).
__device__ __forceinline__ unsigned long long fill_mix(unsigned long long z) {
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return z ^ (z >> 31);
}

template <typename TOut>
__global__ void fill_random_kernel(TOut* __restrict__ out, long long n, unsigned long long key, int kind, float scale) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const unsigned long long c = 3ull * (unsigned long long)i;
    const unsigned long long h0 = fill_mix(key + c * 0x9E3779B97F4A7C15ull);
    if constexpr (std::is_same<TOut, int32_t>::value) {
        out[i] = (int32_t)(h0 & 0x7fffull);
    } else {
        const unsigned long long h1 = fill_mix(key + (c + 1) * 0x9E3779B97F4A7C15ull);
        const unsigned long long h2 = fill_mix(key + (c + 2) * 0x9E3779B97F4A7C15ull);
        int s = 0;
#pragma unroll
        for (int f = 0; f < 4; ++f)
            s += (int)((h0 >> (16 * f)) & 0xffff) + (int)((h1 >> (16 * f)) & 0xffff) + (int)((h2 >> (16 * f)) & 0xffff);
        const float z = (float)(s - 393210) * (1.0f / 65536.0f);
        float w = __fmul_rn(z, scale);
        if (kind == 1) w = __fadd_rn(1.0f, w);
        out[i] = from_f32<TOut>(w);
    }
}

AIRUN_EXPORT int airun_fill_random(void* out, int out_dtype, long long n, unsigned long long key, int kind, float scale,
                                   cudaStream_t stream) {
    if (n < 0 || kind < 0 || kind > 2) return AIRUN_ERR_ARG;
    if (n == 0) return AIRUN_OK;
    const int threads = 256;
    const long long blocks = (n + threads - 1) / threads;
    if (blocks > 0x7fffffffll) return AIRUN_ERR_ARG;
    if (kind == 2) {
        if (out_dtype != 2) return AIRUN_ERR_UNSUPPORTED;
        fill_random_kernel<int32_t><<<(unsigned)blocks, threads, 0, stream>>>((int32_t*)out, n, key, kind, scale);
    } else if (out_dtype == AIRUN_DT_F32) {
        fill_random_kernel<float><<<(unsigned)blocks, threads, 0, stream>>>((float*)out, n, key, kind, scale);
    } else if (out_dtype == AIRUN_DT_BF16) {
        fill_random_kernel<__nv_bfloat16><<<(unsigned)blocks, threads, 0, stream>>>((__nv_bfloat16*)out, n, key, kind, scale);
    } else {
        return AIRUN_ERR_UNSUPPORTED;
    }
    return airun_launch_status();
}


// x = cap * tanh(x / cap), in place: a soft limit on logits.  The dense Qwen3 head has none (the
// reference applies no cap, crates/airun-core/src/runtime.rs:2632-2651); a head part may ask for one.
__global__ void soft_cap_kernel(float* __restrict__ x, long long n, float cap) {
    pdl_trigger();
    pdl_wait();
    const long long i = 4 * ((long long)blockIdx.x * blockDim.x + threadIdx.x);
    if (i + 4 <= n && ((uintptr_t)x & 15) == 0) {
        float4 v = *reinterpret_cast<float4*>(x + i);
        v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap); v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap);
        *reinterpret_cast<float4*>(x + i) = v;
    } else {
        for (long long j = i; j < n && j < i + 4; ++j) x[j] = cap * tanhf(x[j] / cap);
    }
}

AIRUN_EXPORT int airun_soft_cap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n < 0 || !(cap > 0.0f)) return AIRUN_ERR_ARG;
    if (n == 0) return AIRUN_OK;
    const long long blocks = (n + 1023) / 1024;
    if (blocks > 0x7fffffffll) return AIRUN_ERR_ARG;
    airun_launch(soft_cap_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, n, cap);
    return airun_launch_status();
}

// Copies whole cache pages inside the pools of one cache group: for every pair (src, dst) and every
// owner layer, page dst = page src.  pool: [owners][pages][page_words] 16-byte words.  Pairs whose
// ids are outside the pool set the bad-page bit and are skipped.
__global__ void copy_pages_kernel(uint4* __restrict__ pool, long long owner_words, long long page_words,
                                  const int32_t* __restrict__ pairs, int num_pages, int* __restrict__ err) {
    const int src = pairs[2 * blockIdx.x], dst = pairs[2 * blockIdx.x + 1];
    if (src < 0 || src >= num_pages || dst < 0 || dst >= num_pages) {
        if (threadIdx.x == 0 && err) atomicOr(err, AIRUN_DEV_BAD_PAGE);
        return;
    }
    const uint4* s = pool + (long long)blockIdx.y * owner_words + (long long)src * page_words;
    uint4* d = pool + (long long)blockIdx.y * owner_words + (long long)dst * page_words;
    for (long long i = threadIdx.x; i < page_words; i += blockDim.x) d[i] = s[i];
}

AIRUN_EXPORT int airun_copy_pages(void* pool, int owners, int num_pages, long long page_bytes, const int32_t* pairs,
                                  int n_pairs, int* err, cudaStream_t stream) {
    if (owners <= 0 || num_pages <= 0 || page_bytes <= 0 || page_bytes % 16 != 0 || n_pairs < 0 || ((uintptr_t)pool & 15))
        return AIRUN_ERR_ARG;
    if (n_pairs == 0) return AIRUN_OK;
    if (owners > 65535) return AIRUN_ERR_ARG;
    copy_pages_kernel<<<dim3(n_pairs, owners), 256, 0, stream>>>((uint4*)pool, (long long)num_pages * (page_bytes / 16),
                                                                 page_bytes / 16, pairs, num_pages, err);
    return airun_launch_status();
}

// Dynamic Tanh norm, which takes no statistic of the row: out = tanh(alpha * v) * w + b with
// v = x [+ delta] [+ vec], alpha one number for the whole norm (read from device memory), w and b
// vectors.  `vec` is one row added to every token (a per-pass offset of the residual stream).  With
// write_back the sum v becomes the new x.  Source row = rows ? rows[r] : r.  The accurate tanhf is used.
template <typename TOut>
__global__ void dyt_norm_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ vec,
                                const float* __restrict__ alpha, const float* __restrict__ w, const float* __restrict__ b,
                                TOut* __restrict__ out, const int32_t* __restrict__ rows, int n, int write_back) {
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    const float a = alpha[0];
    float* xr = x + (size_t)src * n;
    const float* dr = delta ? delta + (size_t)src * n : nullptr;
    TOut* outr = out + (size_t)r * n;
    if (n % 4 == 0) {                    // rows of float4 (the row pointers are then 16-byte aligned like their bases)
        for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n / 4; i += gridDim.y * blockDim.x) {
            float4 v = reinterpret_cast<const float4*>(xr)[i];
            if (dr) { const float4 d = reinterpret_cast<const float4*>(dr)[i]; v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w; }
            if (vec) { const float4 d = reinterpret_cast<const float4*>(vec)[i]; v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w; }
            if (write_back) reinterpret_cast<float4*>(xr)[i] = v;
            const float4 ww = reinterpret_cast<const float4*>(w)[i], bb = reinterpret_cast<const float4*>(b)[i];
            outr[4 * i + 0] = from_f32<TOut>(fmaf(tanhf(a * v.x), ww.x, bb.x));
            outr[4 * i + 1] = from_f32<TOut>(fmaf(tanhf(a * v.y), ww.y, bb.y));
            outr[4 * i + 2] = from_f32<TOut>(fmaf(tanhf(a * v.z), ww.z, bb.z));
            outr[4 * i + 3] = from_f32<TOut>(fmaf(tanhf(a * v.w), ww.w, bb.w));
        }
        return;
    }
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n; i += gridDim.y * blockDim.x) {
        float v = xr[i];
        if (dr) v += dr[i];
        if (vec) v += vec[i];
        if (write_back) xr[i] = v;
        outr[i] = from_f32<TOut>(fmaf(tanhf(a * v), w[i], b[i]));
    }
}

AIRUN_EXPORT int airun_dyt_norm(float* x, const float* delta, const float* vec, const float* alpha, const float* w,
                                const float* b, void* out, int out_dtype, const int32_t* rows, int n_rows, int n,
                                int write_back, cudaStream_t stream) {
    if (n_rows < 0 || n <= 0 || !alpha || !w || !b) return AIRUN_ERR_ARG;
    if (n_rows == 0) return AIRUN_OK;
    const int threads = 256;
    if (n % 4 == 0 && ((((uintptr_t)x | (uintptr_t)delta | (uintptr_t)vec | (uintptr_t)w | (uintptr_t)b) & 15) != 0)) return AIRUN_ERR_ARG;
    dim3 grid(n_rows, min(ceil_div_i(n % 4 == 0 ? n / 4 : n, threads), 64));
    if (out_dtype == AIRUN_DT_F32)
        airun_launch(dyt_norm_kernel<float>, grid, dim3(threads), 0, stream, x, delta, vec, alpha, w, b, (float*)out, rows, n, write_back);
    else if (out_dtype == AIRUN_DT_BF16)
        airun_launch(dyt_norm_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, x, delta, vec, alpha, w, b, (__nv_bfloat16*)out, rows, n, write_back);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// x[t] += delta[t] + vec for every row t (delta and vec may each be absent), and a += b elementwise
// (vec == nullptr, delta = b): the plain forms of adds that norms otherwise carry out on the way.
__global__ void add_rows_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ vec,
                                long long total, int n) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    float v = x[i];
    if (delta) v += delta[i];
    if (vec) v += vec[i % n];
    x[i] = v;
}

AIRUN_EXPORT int airun_add_rows(float* x, const float* delta, const float* vec, int T, int n, cudaStream_t stream) {
    if (T < 0 || n <= 0) return AIRUN_ERR_ARG;
    const long long total = (long long)T * n;
    if (total == 0 || (!delta && !vec)) return AIRUN_OK;
    airun_launch(add_rows_kernel, dim3(ceil_div_i(total, 256)), dim3(256), 0, stream, x, delta, vec, total, n);
    return airun_launch_status();
}

// Gated unit with clamped factors: g = min(gate, limit), u = clamp(up, -limit, limit),
// out = g * sigmoid(slope * g) * (u + 1).  Gate and up columns alternate in blocks of `group` (as for
// SwiGLU above); the output rows may be strided (a slice of a wider activation buffer).
template <typename TIn, typename TOut>
__global__ void glu_clamped_kernel(const TIn* __restrict__ in, TOut* __restrict__ out, long long total, int I, int group,
                                   long long out_stride, float limit, float slope) {
    pdl_trigger();
    pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const long long t = idx / I;
    const int i = (int)(idx - t * I);
    const int blk = i / group, o = i - blk * group;
    const TIn* row = in + t * 2 * (long long)I;
    const float g = fminf(to_f32<TIn>(row[(size_t)(2 * blk) * group + o]), limit);
    const float u = fminf(fmaxf(to_f32<TIn>(row[(size_t)(2 * blk + 1) * group + o]), -limit), limit);
    out[t * out_stride + i] = from_f32<TOut>(g / (1.0f + expf(-slope * g)) * (u + 1.0f));
}

AIRUN_EXPORT int airun_glu_clamped(const void* in, int in_dtype, void* out, int out_dtype, int T, int I, int group,
                                   long long out_stride, float limit, float slope, cudaStream_t stream) {
    if (T < 0 || I <= 0 || group <= 0 || I % group != 0 || out_stride < I || !(limit > 0.0f)) return AIRUN_ERR_ARG;
    const long long total = (long long)T * I;
    if (total == 0) return AIRUN_OK;
    const int threads = 256;
    const int blocks = ceil_div_i(total, threads);
    if (in_dtype == AIRUN_DT_F32 && out_dtype == AIRUN_DT_F32)
        airun_launch(glu_clamped_kernel<float, float>, dim3(blocks), dim3(threads), 0, stream, (const float*)in, (float*)out, total, I, group, out_stride, limit, slope);
    else if (in_dtype == AIRUN_DT_F32 && out_dtype == AIRUN_DT_BF16)
        airun_launch(glu_clamped_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(threads), 0, stream, (const float*)in, (__nv_bfloat16*)out, total, I, group, out_stride, limit, slope);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// Norm on a sub-layer's OUTPUT: x[t] += mult * y[t] / sqrt(mean(y[t]^2) + eps) * w, and, when `cast` is given,
// cast[t] = x[t] in the compute type (the input of the sub-layer that follows, which reads x itself).  One block
// per row; the row of y stays in registers between the two passes while it is short enough.
template <typename TCast>
__global__ __launch_bounds__(256) void postnorm_add_kernel(float* __restrict__ x, const float* __restrict__ y,
                                                           const float* __restrict__ w, TCast* __restrict__ cast,
                                                           int n, float eps, float mult) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[33];
    const int r = blockIdx.x;
    float* xr = x + (size_t)r * n;
    const float* yr = y + (size_t)r * n;
    float keep[8];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const int i = threadIdx.x + k * 256;
        keep[k] = i < n ? yr[i] : 0.0f;
        ss = fmaf(keep[k], keep[k], ss);
    }
    for (int i = threadIdx.x + 8 * 256; i < n; i += 256) ss = fmaf(yr[i], yr[i], ss);
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < n) {
            const float v = xr[i] + mult * (keep[k] * inv * w[i]);
            xr[i] = v;
            if (cast) cast[(size_t)r * n + i] = from_f32<TCast>(v);
        }
    }
    for (int i = threadIdx.x + 8 * 256; i < n; i += 256) {
        const float v = xr[i] + mult * (yr[i] * inv * w[i]);
        xr[i] = v;
        if (cast) cast[(size_t)r * n + i] = from_f32<TCast>(v);
    }
}

AIRUN_EXPORT int airun_postnorm_add(float* x, const float* y, const float* w, void* cast, int cast_dtype, int T, int n,
                                    float eps, float mult, cudaStream_t stream) {
    if (T < 0 || n <= 0 || !x || !y || !w) return AIRUN_ERR_ARG;
    if (T == 0) return AIRUN_OK;
    if (!cast || cast_dtype == AIRUN_DT_F32)
        airun_launch(postnorm_add_kernel<float>, dim3(T), dim3(256), 0, stream, x, y, w, (float*)cast, n, eps, mult);
    else if (cast_dtype == AIRUN_DT_BF16)
        airun_launch(postnorm_add_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, x, y, w, (__nv_bfloat16*)cast, n, eps, mult);
    else
        return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// What lies between two sub-layers whose inputs AND outputs are normed, in one pass over the residual row:
//     v = x[src] + y[src] / rms(y[src]) * w_post                 the result of the sub-layer before (without y: v = x[src])
//     x[src] = v                                                 when `write_back` is set
//     out[r]  by `mode`:  SANDWICH_NORM   v / rms(v) * w_pre     the input of the sub-layer after, in TOut
//                         SANDWICH_COPY   v                      float32
//                         SANDWICH_SPLIT  [hi | lo], 2n bfloat16 numbers with hi + lo = v to 16 bits of mantissa: a product
//                                         over them reads v without rounding it to bfloat16
// src = rows ? rows[r] : r.  One block per row; up to KEEP vectors a thread stay in registers between the passes, and
// the weights, which no kernel writes, are read before the kernel in front has finished.
#define SANDWICH_NORM 0
#define SANDWICH_COPY 1
#define SANDWICH_SPLIT 2
template <typename TOut>
__device__ __forceinline__ void sandwich_put(TOut* __restrict__ out, int i, int n, int mode, float v, float inv, float w) {
    if (mode == SANDWICH_NORM) {
        out[i] = from_f32<TOut>(v * inv * w);
    } else if (mode == SANDWICH_COPY) {
        out[i] = from_f32<TOut>(v);
    } else {
        const TOut hi = from_f32<TOut>(v);
        out[i] = hi;
        out[n + i] = from_f32<TOut>(v - to_f32<TOut>(hi));
    }
}

// PAIR: two results join at once, x + mult * (y / rms(y) * w_post + y2 / rms(y2) * w_post2); without it mult is not read.
template <typename TOut, int VEC, bool PAIR>
__global__ __launch_bounds__(512) void sandwich_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w_post,
                                     const float* __restrict__ y2, const float* __restrict__ w_post2, float mult,
                                     const float* __restrict__ w_pre, TOut* __restrict__ out, const int32_t* __restrict__ rows,
                                     int n, float eps_post, float eps_pre, int write_back, int mode) {
    pdl_trigger();
    __shared__ float red[33];
    const int nv = n / VEC;
    float v[KEEP][VEC], yk[KEEP][VEC], wa[KEEP][VEC], wb[KEEP][VEC];
    auto load = [&](const float* __restrict__ p, float (&d)[VEC], int i, float none) {
        if (!p || i >= nv) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) d[e] = none;
        } else if (VEC == 4) {
            const float4 f = reinterpret_cast<const float4*>(p)[i];
            d[0] = f.x; d[1 % VEC] = f.y; d[2 % VEC] = f.z; d[3 % VEC] = f.w;
        } else {
            d[0] = p[i];
        }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        load(y ? w_post : nullptr, wa[k], threadIdx.x + k * blockDim.x, 0.0f);
        load(mode == SANDWICH_NORM ? w_pre : nullptr, wb[k], threadIdx.x + k * blockDim.x, 1.0f);
    }
    float y2k[PAIR ? KEEP : 1][VEC], wa2[PAIR ? KEEP : 1][VEC];
    if (PAIR) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k) load(w_post2, wa2[PAIR ? k : 0], threadIdx.x + k * blockDim.x, 0.0f);
    }
    pdl_wait();
    const int r = blockIdx.x, src = rows ? rows[r] : r;
    float* xr = x + (size_t)src * n;
    const float* yr = y ? y + (size_t)src * n : nullptr;
    const float* y2r = PAIR ? y2 + (size_t)src * n : nullptr;
    TOut* outr = out ? out + (size_t)r * (mode == SANDWICH_SPLIT ? 2 * n : n) : nullptr;
    const int tail0 = (threadIdx.x + KEEP * blockDim.x) * VEC, tstep = blockDim.x * VEC;       // a row longer than the registers hold
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        load(xr, v[k], threadIdx.x + k * blockDim.x, 0.0f);
        load(yr, yk[k], threadIdx.x + k * blockDim.x, 0.0f);
        if (PAIR) load(y2r, y2k[PAIR ? k : 0], threadIdx.x + k * blockDim.x, 0.0f);
    }
    float inv_y = 0.0f, inv_y2 = 0.0f;
    if (yr) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(yk[k][e], yk[k][e], ss);
        for (int i = tail0; i < n; i += tstep)
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(yr[i + e], yr[i + e], ss);
        inv_y = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps_post);
        if (PAIR) {
            float s2 = 0.0f;
#pragma unroll
            for (int k = 0; k < KEEP; ++k)
#pragma unroll
                for (int e = 0; e < VEC; ++e) s2 = fmaf(y2k[PAIR ? k : 0][e], y2k[PAIR ? k : 0][e], s2);
            for (int i = tail0; i < n; i += tstep)
#pragma unroll
                for (int e = 0; e < VEC; ++e) s2 = fmaf(y2r[i + e], y2r[i + e], s2);
            inv_y2 = mult / sqrtf(block_sum(s2, red) / (float)n + eps_post);
            inv_y *= mult;
        }
    }
    ss = 0.0f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            v[k][e] += yk[k][e] * inv_y * wa[k][e];
            if (PAIR) v[k][e] += y2k[PAIR ? k : 0][e] * inv_y2 * wa2[PAIR ? k : 0][e];
            ss = fmaf(v[k][e], v[k][e], ss);
        }
        if (yr && write_back && i < nv) {
            if (VEC == 4) reinterpret_cast<float4*>(xr)[i] = make_float4(v[k][0], v[k][1 % VEC], v[k][2 % VEC], v[k][3 % VEC]);
            else xr[i] = v[k][0];
        }
    }
    for (int i = tail0; i < n; i += tstep)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float u = xr[i + e] + (yr ? yr[i + e] * inv_y * w_post[i + e] : 0.0f);
            if (PAIR) u += y2r[i + e] * inv_y2 * w_post2[i + e];
            if (yr && write_back) xr[i + e] = u;
            ss = fmaf(u, u, ss);
        }
    if (!outr) return;
    const float inv = mode == SANDWICH_NORM ? 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps_pre) : 1.0f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i >= nv) continue;
        if (VEC == 4 && sizeof(TOut) == 2 && mode == SANDWICH_NORM) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(v[k][0] * inv * wb[k][0], v[k][1 % VEC] * inv * wb[k][1 % VEC]);
            __nv_bfloat162 hi = __floats2bfloat162_rn(v[k][2 % VEC] * inv * wb[k][2 % VEC], v[k][3 % VEC] * inv * wb[k][3 % VEC]);
            reinterpret_cast<uint2*>(outr)[i] = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
        } else if (VEC == 4 && sizeof(TOut) == 4 && mode == SANDWICH_NORM) {
            reinterpret_cast<float4*>(outr)[i] = make_float4(v[k][0] * inv * wb[k][0], v[k][1 % VEC] * inv * wb[k][1 % VEC],
                                                             v[k][2 % VEC] * inv * wb[k][2 % VEC], v[k][3 % VEC] * inv * wb[k][3 % VEC]);
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) sandwich_put<TOut>(outr, i * VEC + e, n, mode, v[k][e], inv, wb[k][e]);
        }
    }
    for (int i = tail0; i < n; i += tstep)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float u = xr[i + e] + (yr && !write_back ? yr[i + e] * inv_y * w_post[i + e] : 0.0f);
            if (PAIR && !write_back) u += y2r[i + e] * inv_y2 * w_post2[i + e];
            sandwich_put<TOut>(outr, i + e, n, mode, u, inv, mode == SANDWICH_NORM ? w_pre[i + e] : 1.0f);
        }
}

AIRUN_EXPORT int airun_sandwich_norm(float* x, const float* y, const float* w_post, const float* y2, const float* w_post2, float mult,
                                     const float* w_pre, void* out, int out_dtype, const int32_t* rows, int n_rows, int n, float eps_post, float eps_pre, int write_back,
                                     int mode, cudaStream_t stream) {
    if (n_rows < 0 || n <= 0 || !x || (y && !w_post) || (y2 && (!y || !w_post2)) || (!y && !out) || mode < 0 || mode > 2 || (mode == SANDWICH_NORM && out && !w_pre) ||
        (rows && write_back) || (mode == SANDWICH_SPLIT && out_dtype != AIRUN_DT_BF16) || (mode == SANDWICH_COPY && out_dtype != AIRUN_DT_F32))
        return AIRUN_ERR_ARG;
    if (n_rows == 0) return AIRUN_OK;
    const bool vec = n % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)w_post | (uintptr_t)y2 | (uintptr_t)w_post2 | (uintptr_t)w_pre | (uintptr_t)out) & 15) == 0;
    const int nv = vec ? n / 4 : n;
    // many rows: as few threads as hold the row in registers; few rows: more of them, with fewer loads each
    int threads = ((n_rows > 64 ? (nv + KEEP - 1) / KEEP : (nv + 1) / 2) + 31) / 32 * 32;
    if (threads > 512) threads = 512;
    if (threads < 32) threads = 32;
#define SW_PAIR(TOut, VEC, PAIR) \
    airun_launch(sandwich_norm_kernel<TOut, VEC, PAIR>, dim3(n_rows), dim3(threads), 0, stream, x, y, w_post, y2, w_post2, mult, w_pre, \
                 (TOut*)out, rows, n, eps_post, eps_pre, write_back, mode)
#define SW_LAUNCH(TOut, VEC) do { if (y2) SW_PAIR(TOut, VEC, true); else SW_PAIR(TOut, VEC, false); } while (0)
    if (out_dtype == AIRUN_DT_F32) { if (vec) SW_LAUNCH(float, 4); else SW_LAUNCH(float, 1); }
    else if (out_dtype == AIRUN_DT_BF16) { if (vec) SW_LAUNCH(__nv_bfloat16, 4); else SW_LAUNCH(__nv_bfloat16, 1); }
    else return AIRUN_ERR_UNSUPPORTED;
#undef SW_LAUNCH
#undef SW_PAIR
    return airun_launch_status();
}

// out = in in another type (float32 -> bfloat16 or a plain copy), n elements.
template <typename TOut>
__global__ void cast_kernel(const float* __restrict__ in, TOut* __restrict__ out, long long n) {
    pdl_trigger();
    pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        out[i] = from_f32<TOut>(in[i]);
}

AIRUN_EXPORT int airun_cast_f32(const float* in, void* out, int out_dtype, long long n, cudaStream_t stream) {
    if (n < 0 || !in || !out) return AIRUN_ERR_ARG;
    if (n == 0) return AIRUN_OK;
    const int blocks = (int)((n + 1023) / 1024 > 148 * 8 ? 148 * 8 : (n + 1023) / 1024);
    if (out_dtype == AIRUN_DT_F32) airun_launch(cast_kernel<float>, dim3(blocks), dim3(256), 0, stream, in, (float*)out, n);
    else if (out_dtype == AIRUN_DT_BF16) airun_launch(cast_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, in, (__nv_bfloat16*)out, n);
    else return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// out = f(in) element by element, in: float32 [T][n] -> out's type (rows of `out` may be strided).
//   0: relu(z)^2   1: z * sigmoid(z)   2: 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))   3: relu(z)
//   4: 0.5 z (1 + erf(z / sqrt(2)))
__device__ __forceinline__ float unit_act(float z, int mode) {
    if (mode == 4) return 0.5f * z * (1.0f + erff(z * 0.7071067811865476f));
    if (mode == 0) { const float r = fmaxf(z, 0.0f); return r * r; }
    if (mode == 1) return z / (1.0f + expf(-z));
    if (mode == 2) return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    return fmaxf(z, 0.0f);
}

template <typename TOut>
__global__ void act_kernel(const float* __restrict__ in, TOut* __restrict__ out, long long total, int n, long long out_stride,
                           int mode) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long long t = i / n;
    out[t * out_stride + (i - t * n)] = from_f32<TOut>(unit_act(in[i], mode));
}

AIRUN_EXPORT int airun_act(const float* in, void* out, int out_dtype, int T, int n, long long out_stride, int mode,
                           cudaStream_t stream) {
    if (T < 0 || n <= 0 || mode < 0 || mode > 4 || out_stride < n) return AIRUN_ERR_ARG;
    const long long total = (long long)T * n;
    if (total == 0) return AIRUN_OK;
    const long long blocks = (total + 255) / 256;
    if (blocks > 0x7fffffffll) return AIRUN_ERR_ARG;
    if (out_dtype == AIRUN_DT_F32) airun_launch(act_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, in, (float*)out, total, n, out_stride, mode);
    else if (out_dtype == AIRUN_DT_BF16) airun_launch(act_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, in, (__nv_bfloat16*)out, total, n, out_stride, mode);
    else return AIRUN_ERR_UNSUPPORTED;
    return airun_launch_status();
}

// What two gated, scaled sub-layers add to the residual stream:
//   out = s1 * sigmoid(g1 + c1) * y1 [+ s2 * sigmoid(g2 + c2) * y2]
// y: a sub-layer's result [T][n], g: its gate's product [T][gate stride] (a column slice of a wider buffer is fine), c:
// the gate's bias [n], s: the sub-layer's scale per channel [n]; gates and scales may each be absent (null).  All float32.
__global__ void gated_sum_kernel(const float* __restrict__ y1, const float* __restrict__ g1, long long g1_stride,
                                 const float* __restrict__ c1, const float* __restrict__ s1, const float* __restrict__ y2,
                                 const float* __restrict__ g2, long long g2_stride, const float* __restrict__ c2,
                                 const float* __restrict__ s2, float* __restrict__ out, long long total, int n) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long long t = i / n;
    const int c = (int)(i - t * n);
    float v = y1[i];
    if (g1) v *= 1.0f / (1.0f + expf(-(g1[t * g1_stride + c] + (c1 ? c1[c] : 0.0f))));
    if (s1) v *= s1[c];
    if (y2) {
        float u = y2[i];
        if (g2) u *= 1.0f / (1.0f + expf(-(g2[t * g2_stride + c] + (c2 ? c2[c] : 0.0f))));
        if (s2) u *= s2[c];
        v += u;
    }
    out[i] = v;
}

AIRUN_EXPORT int airun_gated_sum(const float* y1, const float* g1, long long g1_stride, const float* c1, const float* s1,
                                 const float* y2, const float* g2, long long g2_stride, const float* c2, const float* s2,
                                 float* out, int T, int n, cudaStream_t stream) {
    if (T < 0 || n <= 0 || !y1 || !out || (g1 && g1_stride < n) || (g2 && g2_stride < n)) return AIRUN_ERR_ARG;
    const long long total = (long long)T * n;
    if (total == 0) return AIRUN_OK;
    const long long blocks = (total + 255) / 256;
    if (blocks > 0x7fffffffll) return AIRUN_ERR_ARG;
    airun_launch(gated_sum_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, y1, g1, g1_stride, c1, s1, y2, g2, g2_stride, c2, s2,
                 out, total, n);
    return airun_launch_status();
}

// x *= factor, in place (a head whose logits carry a fixed factor).
__global__ void scale_kernel(float* __restrict__ x, long long n, float factor) {
    pdl_trigger();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] *= factor;
}

AIRUN_EXPORT int airun_scale(float* x, long long n, float factor, cudaStream_t stream) {
    if (n < 0) return AIRUN_ERR_ARG;
    if (n == 0) return AIRUN_OK;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffll) return AIRUN_ERR_ARG;
    airun_launch(scale_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, n, factor);
    return airun_launch_status();
}
