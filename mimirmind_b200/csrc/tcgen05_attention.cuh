// What the tcgen05 attention kernels share: tensor-memory reads and writes of softmax rows, and a softmax thread's work on one
// tile of 128 keys.
#pragma once

#include "tcgen05.cuh"

namespace tc {

constexpr float RESCALE_STEP = 8.0f;            // log2 of how far a row's maximum may run ahead of its reference

__device__ __forceinline__ void tmem_ld32_nowait(uint32_t taddr, uint32_t* r) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
        "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
          "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
          "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr));
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t* r) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
                   "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr));
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t* r) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
                   "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
                 : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// 2^x on the special-function unit in one instruction (relative error 2^-22, far below the bf16 rounding of P)
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// Every lane has done its part (and its fences); one lane arrives for the warp.
__device__ __forceinline__ void warp_arrive(uint32_t bar, int lane) {
    __syncwarp();
    if (lane == 0) mbar_arrive(bar);
}

// The barriers between a softmax group and the tensor core (shared-memory addresses)
struct SoftmaxBars {
    uint32_t s_full;      // S of the tile is there
    uint32_t s_free;      // ... has been read, one arrival per softmax warp
    uint32_t p_full;      // P of the tile is written and fenced, one arrival per softmax warp
    uint32_t pv_done;     // P V of the group's previous tile has been added into O
};

// One thread's row of one tile of 128 keys, the group's tile number `u` (`first`: its first): S from tensor memory into `sreg`,
// masked by position, O (O_COLS columns at o_addr) rescaled when the row's maximum has outgrown its reference by RESCALE_STEP,
// P rounded to bf16 into p_tile (two halves of 64 keys, 128-byte swizzle), the row's sum added to l.  The row sees keys wlo .. pos and
// the first `keep` ones.  False: a wait ran out.
template <int O_COLS>
__device__ __forceinline__ bool softmax_tile(const SoftmaxBars& bars, volatile int* abort_flag, uint32_t s_addr, uint32_t o_addr, unsigned char* p_tile,
                                             uint32_t half_bytes, int row, int lane, bool row_valid, int pos, int wlo, int key0, uint32_t u, bool first,
                                             float scale_log2, uint32_t (&sreg)[128], float& m_ref, float& l, int keep = 0) {
    constexpr int BN = 128;
    if (!mbar_wait(bars.s_full, u & 1, abort_flag)) return false;
    tc_fence_after();
#pragma unroll
    for (int c = 0; c < 4; ++c) tmem_ld32_nowait(s_addr + c * 32, sreg + c * 32);
    tmem_ld_wait();
    tc_fence_before();
    warp_arrive(bars.s_free, lane);                // S of this tile is in registers
    // a tile every key of which this row sees needs no mask
    const bool interior = row_valid && key0 + BN - 1 <= pos && key0 >= wlo;
    float mx = -INFINITY;
    if (interior) {
#pragma unroll
        for (int i = 0; i < BN; ++i) mx = fmaxf(mx, __uint_as_float(sreg[i]));
    } else if (key0 < keep) {                      // a tile with kept tokens (uniform over the CTA)
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int key = key0 + i;
            if (!(row_valid && key <= pos && (key >= wlo || key < keep))) sreg[i] = 0xff800000u;
            mx = fmaxf(mx, __uint_as_float(sreg[i]));
        }
    } else {
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int key = key0 + i;
            if (!(row_valid && key <= pos && key >= wlo)) sreg[i] = 0xff800000u;      // -inf
            mx = fmaxf(mx, __uint_as_float(sreg[i]));
        }
    }
    // P V of the group's previous tile is done: its P buffer is free and its O is at rest until this tile's P is published
    if (!first && !mbar_wait(bars.pv_done, (u - 1) & 1, abort_flag)) return false;
    // Move the reference only when the maximum has outgrown it by RESCALE_STEP (or there was none).  O of a row without a
    // reference is still zero.
    const bool move = mx > m_ref && (m_ref == -INFINITY || (mx - m_ref) * scale_log2 > RESCALE_STEP);
    const bool scale_o = move && m_ref != -INFINITY;
    if (__any_sync(0xffffffffu, scale_o)) {
        tc_fence_after();
        const float alpha = scale_o ? fast_exp2((m_ref - mx) * scale_log2) : 1.0f;
#pragma unroll 1
        for (int c = 0; c < O_COLS / 16; ++c) {
            uint32_t oreg[16];
            tmem_ld16(o_addr + c * 16, oreg);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) oreg[i] = __float_as_uint(__uint_as_float(oreg[i]) * alpha);
            tmem_st16(o_addr + c * 16, oreg);
        }
        tmem_st_wait();
        l *= alpha;
    }
    if (move) m_ref = mx;
    const float use = (m_ref == -INFINITY) ? 0.0f : m_ref * scale_log2;
    // probabilities, rounded to bf16 as the tensor core will read them: the row of P is two halves of 64 keys, each 8 chunks
    // of 16 bytes, chunk index xor-ed with row % 8
    float sum = 0.0f;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        unsigned char* prow = p_tile + hf * half_bytes + row * 128;
#pragma unroll
        for (int ch = 0; ch < 8; ++ch) {
            uint32_t packed[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float p0 = fast_exp2(fmaf(__uint_as_float(sreg[hf * 64 + ch * 8 + 2 * i]), scale_log2, -use));
                const float p1 = fast_exp2(fmaf(__uint_as_float(sreg[hf * 64 + ch * 8 + 2 * i + 1]), scale_log2, -use));
                sum += p0 + p1;
                packed[i] = pack_bf16x2(p0, p1);
            }
            *reinterpret_cast<uint4*>(prow + ((ch ^ (row & 7)) << 4)) = make_uint4(packed[0], packed[1], packed[2], packed[3]);
        }
    }
    l += sum;
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      // P is read by the tensor core (async proxy)
    tc_fence_before();                                                // ... and O, if it was rescaled, is in tensor memory
    warp_arrive(bars.p_full, lane);
    return true;
}

}  // namespace tc
