// Between the q/k/v projection of an attention and its kernel: norms of queries and keys, rotation, cache write.
//
//   rows [n, ld]: q at q_off (H heads of dk), k at k_off (G heads of dk), v at v_off (G heads of dv);
//   1. span norm (wq / wk given): all H dk numbers of q (all G dk of k) are divided by sqrt(their mean square + eps) together and
//      multiplied by a weight per number;
//   2. rotation of the half-split pairs (i, i + rot_dims / 2) of every head by the step's table of (cos, sin);
//   3. unit norm (unit): every q and k head is divided by sqrt(mean square of its dk numbers + eps).
//
// q goes to q_out [n, H dk], k and v into their pages.  A layer that reads another layer's keys has k_pages null: q alone is made.
// All arithmetic is fp32, and a token's numbers depend on its own row only.
#include "common.cuh"

#define PREP_THREADS 256

struct PrepArgs {
    int ld, q_off, k_off, v_off;
    const float* wq;            // [H * dk] or null
    const float* wk;            // [G * dk] or null
    float eps;
    const float2* rot;          // [n, rot_dims / 2] or null
    int rot_dims, unit;
    const int32_t* slots;       // page * page_size + place (negative: nothing to write)
    int page_size, H, G, dk, dv;
};

template <typename T>
__device__ __forceinline__ void prep_load4(const T* p, float* v);
template <>
__device__ __forceinline__ void prep_load4<float>(const float* p, float* v) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <>
__device__ __forceinline__ void prep_load4<__nv_bfloat16>(const __nv_bfloat16* p, float* v) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T>
__device__ __forceinline__ void prep_store4(T* p, const float* v);
template <>
__device__ __forceinline__ void prep_store4<float>(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
template <>
__device__ __forceinline__ void prep_store4<__nv_bfloat16>(__nv_bfloat16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

// 1 / root mean square of `count` consecutive numbers, by the whole block
template <typename TI>
__device__ __forceinline__ float span_inverse_rms(const TI* p, int count, float eps, float* scratch) {
    float ss = 0.0f;
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
        const float x = to_f32<TI>(p[i]);
        ss = fmaf(x, x, ss);
    }
    return 1.0f / sqrtf(block_sum(ss, scratch) / (float)count + eps);
}

// Two sums over the block at once (a fixed order: lanes, then warps)
__device__ __forceinline__ float2 block_sum2(float x, float y, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
    x = warp_sum(x);
    y = warp_sum(y);
    if (lane == 0) scratch[warp] = make_float2(x, y);
    __syncthreads();
    const float2 t = lane < nwarps ? scratch[lane] : make_float2(0.0f, 0.0f);
    return make_float2(warp_sum(t.x), warp_sum(t.y));
}

// Head sizes of which every piece is a multiple of four numbers: a head is dk / 8 units of eight numbers (four pairs, or eight
// numbers that do not turn), one lane each, `lanes` (a power of two) lanes per head, TURNS heads per group of lanes (a compile-time
// number, so that all of a row's loads are under way before the first is used, and the sums of the span norms come from the
// registers the row stands in).
template <typename TI, typename T, int TURNS>
__global__ void __launch_bounds__(TURNS == 1 ? 1024 : PREP_THREADS) qk_prep_vec_kernel(const TI* __restrict__ rows, T* __restrict__ q_out,
                                                                                       T* __restrict__ k_pages, T* __restrict__ v_pages, const PrepArgs a,
                                                                                       int lanes) {
    __shared__ float2 scratch[32];
    const int t = blockIdx.x, H = a.H, G = k_pages != nullptr ? a.G : 0, dk = a.dk, dv = a.dv, half = a.rot_dims / 2;
    const TI* row = rows + (size_t)t * a.ld;
    const int lane = threadIdx.x & (lanes - 1), groups = blockDim.x / lanes, head0 = threadIdx.x / lanes;
    const bool spans = a.wq != nullptr || (a.wk != nullptr && G > 0), turns = lane * 4 < half, unit_lane = lane < dk / 8;
    const int at0 = turns ? lane * 4 : a.rot_dims + (lane - half / 4) * 8, at1 = turns ? at0 + half : at0 + 4;
    float x[TURNS][8];
    float sq = 0.0f, sk = 0.0f;
#pragma unroll
    for (int u = 0; u < TURNS; ++u) {
        const int head = head0 + u * groups;
#pragma unroll
        for (int e = 0; e < 8; ++e) x[u][e] = 0.0f;
        if (unit_lane && head < H + G) {
            const TI* p = row + (head < H ? a.q_off + head * dk : a.k_off + (head - H) * dk);
            prep_load4<TI>(p + at0, x[u]);
            prep_load4<TI>(p + at1, x[u] + 4);
        }
    }
    float cs[4], sn[4];
    if (turns) {
        const float4* c = reinterpret_cast<const float4*>(a.rot + (size_t)t * half + at0);
        const float4 c01 = c[0], c23 = c[1];
        cs[0] = c01.x; sn[0] = c01.y; cs[1] = c01.z; sn[1] = c01.w;
        cs[2] = c23.x; sn[2] = c23.y; cs[3] = c23.z; sn[3] = c23.w;
    }
    const long long slot = G > 0 ? (long long)a.slots[t] : -1;
    const long long page = slot >= 0 ? slot / a.page_size : -1;
    const int place = slot >= 0 ? (int)(slot - page * a.page_size) : 0;
    if (page >= 0) {
        for (int i = threadIdx.x * 4; i < G * dv; i += blockDim.x * 4) {
            const int g = i / dv, e = i - g * dv;
            float v[4];
            prep_load4<TI>(row + a.v_off + i, v);
            prep_store4<T>(v_pages + (((size_t)page * G + g) * a.page_size + place) * dv + e, v);
        }
    }
    float rq = 1.0f, rk = 1.0f;
    if (spans) {
#pragma unroll
        for (int u = 0; u < TURNS; ++u) {
            float ss = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[u][e], x[u][e], ss);
            if (head0 + u * groups < H) sq += ss;
            else sk += ss;
        }
        const float2 s = block_sum2(sq, sk, scratch);
        rq = 1.0f / sqrtf(s.x / (float)(H * dk) + a.eps);
        rk = 1.0f / sqrtf(s.y / (float)(a.G * dk) + a.eps);
    }
#pragma unroll
    for (int u = 0; u < TURNS; ++u) {                          // every thread takes every turn: the lanes of a head add up
        const int head = head0 + u * groups;
        const bool live = unit_lane && head < H + G, is_q = head < H;
        if (live) {
            const float* w = is_q ? a.wq : a.wk;
            if (w != nullptr) {
                const int off = is_q ? head * dk : (head - H) * dk;
                float wv[8];
                prep_load4<float>(w + off + at0, wv);
                prep_load4<float>(w + off + at1, wv + 4);
                const float r = is_q ? rq : rk;
#pragma unroll
                for (int e = 0; e < 8; ++e) x[u][e] = x[u][e] * r * wv[e];
            }
            if (turns) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float p = x[u][e], v = x[u][4 + e];
                    x[u][e] = p * cs[e] - v * sn[e];
                    x[u][4 + e] = v * cs[e] + p * sn[e];
                }
            }
        }
        if (a.unit) {
            float ss = 0.0f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[u][e], x[u][e], ss);
            for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float r = 1.0f / sqrtf(ss / (float)dk + a.eps);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[u][e] *= r;
        }
        if (!live) continue;
        T* dst = is_q ? q_out + ((size_t)t * H + head) * dk : (page >= 0 ? k_pages + (((size_t)page * G + (head - H)) * a.page_size + place) * dk : nullptr);
        if (dst != nullptr) {
            prep_store4<T>(dst + at0, x[u]);
            prep_store4<T>(dst + at1, x[u] + 4);
        }
    }
}

// any sizes: a warp per head
template <typename TI, typename T>
__global__ void __launch_bounds__(PREP_THREADS) qk_prep_kernel(const TI* __restrict__ rows, T* __restrict__ q_out, T* __restrict__ k_pages,
                                                               T* __restrict__ v_pages, const PrepArgs a) {
    __shared__ float scratch[32];
    const int t = blockIdx.x, H = a.H, G = k_pages != nullptr ? a.G : 0, dk = a.dk, dv = a.dv, half = a.rot_dims / 2;
    const TI* row = rows + (size_t)t * a.ld;
    float rq = 1.0f, rk = 1.0f;
    if (a.wq != nullptr) rq = span_inverse_rms<TI>(row + a.q_off, H * dk, a.eps, scratch);
    if (a.wk != nullptr && G > 0) rk = span_inverse_rms<TI>(row + a.k_off, G * dk, a.eps, scratch);
    const long long slot = G > 0 ? (long long)a.slots[t] : -1;
    const long long page = slot >= 0 ? slot / a.page_size : -1;
    const int place = slot >= 0 ? (int)(slot - page * a.page_size) : 0;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int head = warp; head < H + G; head += warps) {
        const bool is_q = head < H;
        const int off = is_q ? head * dk : (head - H) * dk;
        const TI* p = row + (is_q ? a.q_off : a.k_off) + off;
        const float* w = is_q ? a.wq : a.wk;
        const float r = is_q ? rq : rk;
        auto normed = [&](int i) -> float { return w != nullptr ? to_f32<TI>(p[i]) * r * w[off + i] : to_f32<TI>(p[i]); };
        auto value = [&](int i) -> float {
            if (i >= a.rot_dims) return normed(i);
            const int pair = i < half ? i : i - half;
            const float2 c = a.rot[(size_t)t * half + pair];
            const float u = normed(pair), v = normed(pair + half);
            return i < half ? u * c.x - v * c.y : v * c.x + u * c.y;
        };
        float inv = 1.0f;
        if (a.unit) {
            float ss = 0.0f;
            for (int i = lane; i < dk; i += 32) {
                const float x = value(i);
                ss = fmaf(x, x, ss);
            }
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)dk + a.eps);
        }
        T* dst = is_q ? q_out + ((size_t)t * H + head) * dk : (page >= 0 ? k_pages + (((size_t)page * G + (head - H)) * a.page_size + place) * dk : nullptr);
        if (dst != nullptr)
            for (int i = lane; i < dk; i += 32) dst[i] = from_f32<T>(value(i) * inv);
    }
    if (page < 0) return;
    for (int i = threadIdx.x; i < G * dv; i += blockDim.x) {
        const int g = i / dv, e = i - g * dv;
        v_pages[(((size_t)page * G + g) * a.page_size + place) * dv + e] = from_f32<T>(to_f32<TI>(row[a.v_off + i]));
    }
}

template <typename TI, typename T>
static void prep_launch(const void* rows, void* q_out, void* k_pages, void* v_pages, const PrepArgs& a, int n, bool vec, cudaStream_t s) {
    int lanes = 1;
    while (lanes < a.dk / 8) lanes *= 2;
    const int all = ((a.H + (k_pages ? a.G : 0)) * lanes + 31) / 32 * 32;
    // A lane for every unit of a row where a step's tokens have an SM to themselves (one such block fits an SM); with more tokens,
    // smaller blocks side by side.  A 32-bit run keeps to the latter: its sums then have one order whatever else is in the step.
    int turns = sizeof(T) == 2 && n <= 296 && all <= 1024 ? 1 : 2;
    while (turns > 1 && turns < 8 && all > turns * PREP_THREADS) turns += turns < 4 ? 1 : 2;
    if (!vec || all > 8 * PREP_THREADS) {
        mm_launch(qk_prep_kernel<TI, T>, dim3(n), dim3(PREP_THREADS), 0, s, (const TI*)rows, (T*)q_out, (T*)k_pages, (T*)v_pages, a);
        return;
    }
    auto kernel = turns == 1 ? qk_prep_vec_kernel<TI, T, 1> : turns == 2 ? qk_prep_vec_kernel<TI, T, 2> : turns == 3 ? qk_prep_vec_kernel<TI, T, 3>
                  : turns == 4 ? qk_prep_vec_kernel<TI, T, 4> : turns == 6 ? qk_prep_vec_kernel<TI, T, 6> : qk_prep_vec_kernel<TI, T, 8>;
    // as few threads as the turns allow, so that none of them idles
    const int threads = turns == 1 ? all : ((all + turns - 1) / turns + 31) / 32 * 32;
    mm_launch(kernel, dim3(n), dim3(threads), 0, s, (const TI*)rows, (T*)q_out, (T*)k_pages, (T*)v_pages, a, lanes);
}

MM_EXPORT int mm_qk_prep(const void* rows, int rows_dtype, int ld, int q_off, int k_off, int v_off, const void* wq, const void* wk, float eps,
                         const void* rot, int rot_dims, int unit, void* q_out, void* k_pages, void* v_pages, int dtype, const void* slots,
                         int page_size, int n_tokens, int H, int G, int dk, int dv, void* stream) {
    MM_REQUIRE(n_tokens >= 0 && H > 0 && G > 0 && dk > 0 && dv > 0 && ld > 0, "qk prep: bad sizes");
    MM_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dk && (rot_dims == 0 || rot != nullptr),
               "qk prep: the rotated dimensions must be even, at most the key size, and have their table");
    MM_REQUIRE(q_out != nullptr && (k_pages == nullptr || (page_size > 0 && slots != nullptr && v_pages != nullptr)), "qk prep: bad page geometry");
    if (n_tokens == 0) return MM_OK;
    PrepArgs a;
    a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off;
    a.wq = (const float*)wq; a.wk = (const float*)wk; a.eps = eps;
    a.rot = (const float2*)rot; a.rot_dims = rot_dims; a.unit = unit;
    a.slots = (const int32_t*)slots; a.page_size = page_size; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
    const bool vec = dk % 8 == 0 && dk <= 256 && rot_dims % 8 == 0 && dv % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                     (((uintptr_t)rows | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)wq | (uintptr_t)wk | (uintptr_t)rot) & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
    if (rows_dtype == MM_F32 && dtype == MM_F32) prep_launch<float, float>(rows, q_out, k_pages, v_pages, a, n_tokens, vec, s);
    else if (rows_dtype == MM_F32 && dtype == MM_BF16) prep_launch<float, bf>(rows, q_out, k_pages, v_pages, a, n_tokens, vec, s);
    else if (rows_dtype == MM_BF16 && dtype == MM_BF16) prep_launch<bf, bf>(rows, q_out, k_pages, v_pages, a, n_tokens, vec, s);
    else MM_REQUIRE(false, "qk prep: this combination of dtypes is not built");
    MM_CHECK_LAUNCH();
    return MM_OK;
}
