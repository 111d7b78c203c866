// A norm without statistics, number by number: N(x) = w tanh(alpha x) + b with one slope per tensor and a weight and an offset per
// channel; and the chain "norm a branch, add it to the residual stream, norm the sum" in one launch:
//
//   if branch:  residual += post ? N_post(branch) : branch     (fp32, in place)
//   if next:    out = N_next(residual)                          (activation dtype)
//
// The branch may still be in pieces: sum_c wts[t, c] y[place[t, c]], the chosen experts' rows with their weights.  With `rows`,
// output row i is made from source row rows[i] and nothing is added.  Also the soft cap of logits, c tanh(x / c).
// A thread keeps the channels' numbers of its columns in registers and walks over several tokens.  For steps of a
// few tokens the same chain is an epilogue of the products that make the branch (gemv_bf16.cu, gemm_skinny_tcgen05.cu).
#include "common.cuh"

template <int V, typename T>
__device__ __forceinline__ void tn_load(const T* p, float* v) {
    if constexpr (V == 1) {
        v[0] = to_f32<T>(p[0]);
    } else if constexpr (sizeof(T) == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 c = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = a.x; v[1] = a.y; v[2] = c.x; v[3] = c.y;
    }
}
template <int V, typename T>
__device__ __forceinline__ void tn_store(T* p, const float* v) {
    if constexpr (V == 1) {
        p[0] = from_f32<T>(v[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), c = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&c));
    }
}

// V columns per thread (1 or 4); blockIdx.x: columns, blockIdx.y: runs of `run` tokens
template <int V, typename TB, typename TO>
__global__ void __launch_bounds__(128) tanh_norm_chain_kernel(float* __restrict__ residual, const TB* __restrict__ branch, const float* __restrict__ wts,
                                                              const int32_t* __restrict__ place, int top, const TanhNorm post, const TanhNorm next,
                                                              const int32_t* __restrict__ rows, TO* __restrict__ out, int n, int D, int run) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (c >= D) return;
    float w1[V], b1[V], w2[V], b2[V];
    if (post.w != nullptr) {
        tn_load<V>(post.w + c, w1);
        tn_load<V>(post.b + c, b1);
    }
    if (next.w != nullptr) {
        tn_load<V>(next.w + c, w2);
        tn_load<V>(next.b + c, b2);
    }
    const int t1 = min(n, ((int)blockIdx.y + 1) * run);
    for (int t = blockIdx.y * run; t < t1; ++t) {
        float x[V];
        const size_t r = rows ? (size_t)rows[t] : (size_t)t;
        tn_load<V>(residual + r * D + c, x);
        if (branch != nullptr) {
            float y[V];
            if (top > 0) {
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = 0.0f;
#pragma unroll 4
                for (int k = 0; k < top; ++k) {
                    const int i = t * top + k;
                    float p[V];
                    tn_load<V>(branch + (size_t)(place ? place[i] : i) * D + c, p);
                    const float g = wts[i];
#pragma unroll
                    for (int e = 0; e < V; ++e) y[e] = fmaf(g, p[e], y[e]);
                }
            } else {
                tn_load<V>(branch + (size_t)t * D + c, y);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] += post.w != nullptr ? tanh_norm(y[e], post.alpha, w1[e], b1[e]) : y[e];
            tn_store<V>(residual + r * D + c, x);
        }
        if (next.w != nullptr) {
            float o[V];
#pragma unroll
            for (int e = 0; e < V; ++e) o[e] = tanh_norm(x[e], next.alpha, w2[e], b2[e]);
            tn_store<V>(out + (size_t)t * D + c, o);
        }
    }
}

MM_EXPORT int mm_tanh_norm_chain(void* residual, const void* branch, int branch_dtype, const void* wts, const void* place, int top, const void* post_w,
                                 const void* post_b, float post_alpha, const void* next_w, const void* next_b, float next_alpha, const void* rows,
                                 void* out, int out_dtype, int n, int D, void* stream) {
    MM_REQUIRE(n >= 0 && D > 0 && residual != nullptr, "tanh norm: bad sizes");
    MM_REQUIRE(branch == nullptr || rows == nullptr, "tanh norm: a gathered call adds nothing");
    MM_REQUIRE(branch != nullptr || next_w != nullptr, "tanh norm: nothing to do");
    MM_REQUIRE((post_w == nullptr) == (post_b == nullptr) && (next_w == nullptr) == (next_b == nullptr) && (next_w == nullptr || out != nullptr),
               "tanh norm: a norm has a weight and an offset, and the second one an output");
    MM_REQUIRE(top >= 0 && (top == 0 || wts != nullptr), "tanh norm: chosen rows need their weights");
    if (n == 0) return MM_OK;
    const bool vec = D % 4 == 0 && (((uintptr_t)residual | (uintptr_t)branch | (uintptr_t)post_w | (uintptr_t)post_b | (uintptr_t)next_w |
                                     (uintptr_t)next_b | (uintptr_t)out) & 15) == 0;
    const int V = vec ? 4 : 1, threads = 128;
    const int cols = ceil_div(ceil_div(D, V), threads);
    // as many tokens per thread as leave some 16 blocks per SM
    int run = (int)((long long)cols * n / (16 * 148));
    run = run < 1 ? 1 : (run > 16 ? 16 : run);
    if ((n + run - 1) / run > 65535) run = ceil_div(n, 65535);
    const dim3 grid(cols, ceil_div(n, run));
    cudaStream_t s = (cudaStream_t)stream;
    const TanhNorm post = {(const float*)post_w, (const float*)post_b, post_alpha}, next = {(const float*)next_w, (const float*)next_b, next_alpha};
    typedef __nv_bfloat16 bf;
    if (branch == nullptr) branch_dtype = out_dtype;
    if (out == nullptr) out_dtype = branch_dtype;
#define TN_LAUNCH(TB, TO)                                                                                                              \
    do {                                                                                                                               \
        auto kernel = vec ? tanh_norm_chain_kernel<4, TB, TO> : tanh_norm_chain_kernel<1, TB, TO>;                                     \
        mm_launch(kernel, grid, dim3(threads), 0, s, (float*)residual, (const TB*)branch, (const float*)wts, (const int32_t*)place, top, post, next, \
                  (const int32_t*)rows, (TO*)out, n, D, run);                                                                          \
    } while (0)
    if (branch_dtype == MM_F32 && out_dtype == MM_F32) TN_LAUNCH(float, float);
    else if (branch_dtype == MM_BF16 && out_dtype == MM_BF16) TN_LAUNCH(bf, bf);
    else if (branch_dtype == MM_F32 && out_dtype == MM_BF16) TN_LAUNCH(float, bf);
    else MM_REQUIRE(false, "tanh norm: this combination of dtypes is not built");
#undef TN_LAUNCH
    MM_CHECK_LAUNCH();
    return MM_OK;
}

__global__ void soft_cap_kernel(float* __restrict__ x, long long total, float cap) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) x[i] = cap * tanhf(x[i] / cap);
}

// x <- cap tanh(x / cap), in place
MM_EXPORT int mm_soft_cap(void* x, long long total, float cap, void* stream) {
    MM_REQUIRE(total >= 0 && cap > 0.0f, "soft cap: the cap must be positive");
    if (total == 0) return MM_OK;
    mm_launch(soft_cap_kernel, dim3(ceil_div(total, 256)), dim3(256), 0, (cudaStream_t)stream, (float*)x, total, cap);
    MM_CHECK_LAUNCH();
    return MM_OK;
}
