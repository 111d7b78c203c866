// The norm after the sum, the norm on a sublayer's output before the sum, the gated activation of a two-matrix feed-forward as a pass of its own, and the rounding of
// the residual stream to the activation dtype.
//
//   post norm:   y = alpha x + ca a + cb b;   x <- y / sqrt(mean(y^2) + eps) * w      (x: the fp32 residual stream, in place)
//
//   output norm: y = ca a + cb g b;             x <- x + m y / sqrt(mean(y^2) + eps) * w    (g: a number per token)
//
// a and b are a layer's branch outputs (either may be absent); the new stream is also written in the activation dtype,
// which is what the next sublayer's products read.  In the output norm `a` may also be the rows of a token's chosen
// experts, which are weighed and added on the way.
#include "common.cuh"

template <typename TB, typename TO>
__global__ void __launch_bounds__(256) post_norm_kernel(float* __restrict__ x, const TB* __restrict__ a, const TB* __restrict__ b,
                                                        const float* __restrict__ w, TO* __restrict__ out, int D, float alpha, float ca, float cb,
                                                        float eps) {
    extern __shared__ float pn_row[];
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    float* xr = x + t * D;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float y = alpha * xr[i];
        if (a) y = fmaf(ca, to_f32<TB>(a[t * D + i]), y);
        if (b) y = fmaf(cb, to_f32<TB>(b[t * D + i]), y);
        pn_row[i] = y;
        ss = fmaf(y, y, ss);
    }
    ss = block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)D + eps);
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        const float y = pn_row[i] * r * w[i];
        xr[i] = y;
        if (out) out[t * D + i] = from_f32<TO>(y);
    }
}

// Eight numbers at a time (16-byte words of bfloat16, two of fp32): the same arithmetic in the same order per element.
__device__ __forceinline__ void pn_load8(const float* p, float* v) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void pn_load8(const __nv_bfloat16* p, float* v) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void pn_store8(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void pn_store8(__nv_bfloat16* p, const float* v) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

template <typename TB, typename TO>
__global__ void __launch_bounds__(256) post_norm8_kernel(float* __restrict__ x, const TB* __restrict__ a, const TB* __restrict__ b,
                                                         const float* __restrict__ w, TO* __restrict__ out, int D, float alpha, float ca, float cb,
                                                         float eps) {
    extern __shared__ __align__(16) float pn_row[];
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    float* xr = x + t * D;
    float ss = 0.0f;
    for (int i = threadIdx.x * 8; i < D; i += blockDim.x * 8) {
        float y[8], u[8];
        pn_load8(xr + i, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] *= alpha;
        if (a) {
            pn_load8(a + t * D + i, u);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = fmaf(ca, u[e], y[e]);
        }
        if (b) {
            pn_load8(b + t * D + i, u);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = fmaf(cb, u[e], y[e]);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
        pn_store8(pn_row + i, y);
    }
    ss = block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)D + eps);
    for (int i = threadIdx.x * 8; i < D; i += blockDim.x * 8) {
        float y[8], wv[8];
        pn_load8(pn_row + i, y);
        pn_load8(w + i, wv);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = y[e] * r * wv[e];
        pn_store8(xr + i, y);
        if (out) pn_store8(out + t * D + i, y);
    }
}

// x [n, D] fp32 residual (in place); a, b [n, D] of dtype `b_dtype` or null; w fp32 [D]; out [n, D] of `out_dtype` or null.
MM_EXPORT int mm_post_norm(void* x, const void* a, const void* b, int b_dtype, const void* w, void* out, int out_dtype, int n, int D, float alpha,
                           float ca, float cb, float eps, void* stream) {
    MM_REQUIRE(n >= 0 && D > 0 && D <= 51200, "post norm: widths above 51200 are not supported");
    MM_REQUIRE(x != nullptr && w != nullptr, "post norm: the stream and the weight are needed");
    if (n == 0) return MM_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)D * sizeof(float);
    typedef __nv_bfloat16 bf;
    const bool by8 = D % 8 == 0 && (((uintptr_t)x | (uintptr_t)a | (uintptr_t)b | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
#define PN_LAUNCH(TB, TO)                                                                                                         \
    do {                                                                                                                          \
        auto kernel = by8 ? post_norm8_kernel<TB, TO> : post_norm_kernel<TB, TO>;                                                 \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
        mm_launch(kernel, dim3(n), dim3(256), smem, s, (float*)x, (const TB*)a, (const TB*)b, (const float*)w, (TO*)out, D, alpha, ca, cb, eps); \
    } while (0)
    if (b_dtype == MM_F32 && out_dtype == MM_F32) PN_LAUNCH(float, float);
    else if (b_dtype == MM_BF16 && out_dtype == MM_BF16) PN_LAUNCH(bf, bf);
    else if (b_dtype == MM_F32 && out_dtype == MM_BF16) PN_LAUNCH(float, bf);
    else MM_REQUIRE(false, "post norm: this combination of dtypes is not built");
#undef PN_LAUNCH
    MM_CHECK_LAUNCH();
    return MM_OK;
}

// V numbers of a row at a time (V 8: 16-byte words; V 1: any width and alignment), the same arithmetic per element.
template <int V, typename T>
__device__ __forceinline__ void pn_load(const T* p, float* v) {
    if constexpr (V == 8) pn_load8(p, v);
    else v[0] = to_f32<T>(p[0]);
}
template <int V, typename T>
__device__ __forceinline__ void pn_store(T* p, const float* v) {
    if constexpr (V == 8) pn_store8(p, v);
    else p[0] = from_f32<T>(v[0]);
}

// top > 0: a holds a token's chosen rows, row(t, c) = place[t * top + c] (place null: t * top + c), weight wts[t * top + c]
template <int V, typename TA, typename TB, typename TO>
__global__ void __launch_bounds__(256) output_norm_kernel(float* __restrict__ x, const TA* __restrict__ a, const float* __restrict__ wts,
                                                          const int32_t* __restrict__ place, int top, const TB* __restrict__ b,
                                                          const float* __restrict__ gate, const float* __restrict__ w, TO* __restrict__ out, int D,
                                                          float m, float ca, float cb, float eps) {
    extern __shared__ __align__(16) float pn_row[];
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    const float fb = b ? (gate ? cb * gate[t] : cb) : 0.0f;
    float ss = 0.0f;
    for (int i = threadIdx.x * V; i < D; i += blockDim.x * V) {
        float y[V], u[V];
        if (top > 0) {
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = 0.0f;
            for (int c = 0; c < top; ++c) {
                const size_t row = place ? (size_t)place[t * top + c] : t * top + c;
                const float wt = wts[t * top + c];
                pn_load<V>(a + row * D + i, u);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = fmaf(wt, u[e], y[e]);
            }
        } else {
            pn_load<V>(a + t * D + i, y);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] *= ca;
        if (b) {
            pn_load<V>(b + t * D + i, u);
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = fmaf(fb, u[e], y[e]);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(y[e], y[e], ss);
        pn_store<V>(pn_row + i, y);
    }
    ss = block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)D + eps);
    float* xr = x + t * D;
    for (int i = threadIdx.x * V; i < D; i += blockDim.x * V) {
        float y[V], wv[V], xv[V];
        pn_load<V>(pn_row + i, y);
        pn_load<V>(w + i, wv);
        pn_load<V>(xr + i, xv);
#pragma unroll
        for (int e = 0; e < V; ++e) xv[e] = fmaf(m, y[e] * r * wv[e], xv[e]);
        pn_store<V>(xr + i, xv);
        if (out) pn_store<V>(out + t * D + i, xv);
    }
}

// x [n, D] fp32 residual (in place); a [n, D], or with top > 0 the chosen experts' rows [n * top, D] with wts fp32 [n, top] and
// place int32 [n, top] (or null); b [n, D] or null with gate fp32 [n] or null; w fp32 [D]; out [n, D] of `out_dtype` or null.
MM_EXPORT int mm_output_norm(void* x, const void* a, int a_dtype, const void* wts, const void* place, int top, const void* b, int b_dtype,
                             const void* gate, const void* w, void* out, int out_dtype, int n, int D, float m, float ca, float cb, float eps,
                             void* stream) {
    MM_REQUIRE(n >= 0 && D > 0 && D <= 51200, "output norm: widths above 51200 are not supported");
    MM_REQUIRE(x != nullptr && a != nullptr && w != nullptr, "output norm: the stream, a branch and the weight are needed");
    MM_REQUIRE(top >= 0 && (top == 0 || wts != nullptr), "output norm: chosen rows need their weights");
    if (n == 0) return MM_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)D * sizeof(float);
    typedef __nv_bfloat16 bf;
    const bool by8 = D % 8 == 0 && (((uintptr_t)x | (uintptr_t)a | (uintptr_t)b | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
    const int threads = by8 ? (D >= 2048 ? 256 : (D >= 1024 ? 128 : 64)) : 256;
#define ON_LAUNCH(TA, TB, TO)                                                                                                     \
    do {                                                                                                                          \
        auto kernel = by8 ? output_norm_kernel<8, TA, TB, TO> : output_norm_kernel<1, TA, TB, TO>;                                \
        if (smem > 40 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
        mm_launch(kernel, dim3(n), dim3(threads), smem, s, (float*)x, (const TA*)a, (const float*)wts, (const int32_t*)place, top, (const TB*)b, \
                  (const float*)gate, (const float*)w, (TO*)out, D, m, ca, cb, eps);                                              \
    } while (0)
    if (b == nullptr) b_dtype = out ? out_dtype : a_dtype;
    if (out == nullptr) out_dtype = b_dtype;
    if (a_dtype == MM_F32 && b_dtype == MM_F32 && out_dtype == MM_F32) ON_LAUNCH(float, float, float);
    else if (a_dtype == MM_BF16 && b_dtype == MM_BF16 && out_dtype == MM_BF16) ON_LAUNCH(bf, bf, bf);
    else if (a_dtype == MM_F32 && b_dtype == MM_BF16 && out_dtype == MM_BF16) ON_LAUNCH(float, bf, bf);
    else MM_REQUIRE(false, "output norm: this combination of dtypes is not built");
#undef ON_LAUNCH
    MM_CHECK_LAUNCH();
    return MM_OK;
}

// out [n, F] = glu_act(gate * s, up * s): gu holds the gate's columns, then the up columns, or with `interleave` (8) both in
// blocks of that many columns in turn; row_scale fp32 [n] or null.
template <typename TI, typename TO>
__global__ void glu_rows_kernel(const TI* __restrict__ gu, long long ld, TO* __restrict__ out, long long total, int F, int act, float limit,
                                const float* __restrict__ row_scale, int interleave) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long long t = i / F;
    const int c = (int)(i - t * F);
    const TI* row = gu + t * ld;
    const int g = interleave ? 2 * c - c % interleave : c, u = interleave ? g + interleave : F + c;
    out[i] = from_f32<TO>(glu_act<false>(to_f32<TI>(row[g]), to_f32<TI>(row[u]), act, limit, row_scale ? row_scale[t] : 1.0f));
}

MM_EXPORT int mm_glu_rows(const void* gu, int in_dtype, long long ld, void* out, int out_dtype, int n, int F, int act, float limit,
                          const void* row_scale, int interleave, void* stream) {
    MM_REQUIRE(n >= 0 && F > 0 && ld >= 2 * (long long)F, "gated activation: bad sizes");
    MM_REQUIRE(act >= MM_GLU_SILU && act <= MM_GLU_GELU_TANH, "gated activation: unknown kind");
    MM_REQUIRE(interleave == 0 || (interleave > 0 && F % interleave == 0), "gated activation: the blocks must divide the width");
    if (n == 0) return MM_OK;
    const long long total = (long long)n * F;
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
    const dim3 grid(ceil_div(total, 256));
    if (in_dtype == MM_F32 && out_dtype == MM_F32)
        mm_launch(glu_rows_kernel<float, float>, grid, dim3(256), 0, s, (const float*)gu, ld, (float*)out, total, F, act, limit, (const float*)row_scale, interleave);
    else if (in_dtype == MM_BF16 && out_dtype == MM_BF16)
        mm_launch(glu_rows_kernel<bf, bf>, grid, dim3(256), 0, s, (const bf*)gu, ld, (bf*)out, total, F, act, limit, (const float*)row_scale, interleave);
    else if (in_dtype == MM_F32 && out_dtype == MM_BF16)
        mm_launch(glu_rows_kernel<float, bf>, grid, dim3(256), 0, s, (const float*)gu, ld, (bf*)out, total, F, act, limit, (const float*)row_scale, interleave);
    else
        MM_REQUIRE(false, "gated activation: this combination of dtypes is not built");
    MM_CHECK_LAUNCH();
    return MM_OK;
}

// fp32 rows to the activation dtype
template <typename TO>
__global__ void cast_rows_kernel(const float* __restrict__ x, TO* __restrict__ out, long long total) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) out[i] = from_f32<TO>(x[i]);
}

__global__ void cast_rows8_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ out, long long total8) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    float v[8];
    pn_load8(x + i * 8, v);
    pn_store8(out + i * 8, v);
}

MM_EXPORT int mm_cast_rows(const void* x, void* out, int out_dtype, long long total, void* stream) {
    MM_REQUIRE(total >= 0, "cast: bad size");
    if (total == 0) return MM_OK;
    if (out_dtype == MM_BF16 && total % 8 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15) == 0) {
        mm_launch(cast_rows8_kernel, dim3(ceil_div(total / 8, 256)), dim3(256), 0, (cudaStream_t)stream, (const float*)x, (__nv_bfloat16*)out, total / 8);
        MM_CHECK_LAUNCH();
        return MM_OK;
    }
    const dim3 grid(ceil_div(total, 256));
    if (out_dtype == MM_F32)
        mm_launch(cast_rows_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)x, (float*)out, total);
    else if (out_dtype == MM_BF16)
        mm_launch(cast_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)x, (__nv_bfloat16*)out, total);
    else
        MM_REQUIRE(false, "cast: dtype must be float32 or bfloat16");
    MM_CHECK_LAUNCH();
    return MM_OK;
}

// out = ca a + cb g b, element by element (two branches as one where nothing downstream adds them itself); g: a number per
// row of D (null: 1)
template <typename T>
__global__ void scaled_sum2_kernel(const T* __restrict__ a, const T* __restrict__ b, T* __restrict__ out, long long total, float ca, float cb,
                                   const float* __restrict__ gate, int D) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) out[i] = from_f32<T>(fmaf(gate ? cb * gate[i / D] : cb, to_f32<T>(b[i]), ca * to_f32<T>(a[i])));
}

MM_EXPORT int mm_scaled_sum2(const void* a, const void* b, void* out, int dtype, long long total, float ca, float cb, const void* gate, int D,
                             void* stream) {
    MM_REQUIRE(total >= 0 && (gate == nullptr || D > 0), "scaled sum: bad size");
    if (total == 0) return MM_OK;
    const dim3 grid(ceil_div(total, 256));
    if (dtype == MM_F32)
        mm_launch(scaled_sum2_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)a, (const float*)b, (float*)out, total, ca, cb,
                  (const float*)gate, D);
    else if (dtype == MM_BF16)
        mm_launch(scaled_sum2_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, (const __nv_bfloat16*)a, (const __nv_bfloat16*)b,
                  (__nv_bfloat16*)out, total, ca, cb, (const float*)gate, D);
    else
        MM_REQUIRE(false, "scaled sum: dtype must be float32 or bfloat16");
    MM_CHECK_LAUNCH();
    return MM_OK;
}
