// What the tensor-core attention kernels over the paged cache share (attention_mma.cu,
// attention_decode.cu): tile constants for the head size they are compiled for (-DHEAD_DIM=d),
// the work item, and the cp.async / ldmatrix / mma.sync wrappers.
#pragma once

#include "common.cuh"

#ifndef HEAD_DIM
#define HEAD_DIM 64
#endif

// 1: the softmax weights enter their product with the values as two bfloat16 terms instead of one,
// so that they keep 16 bits of mantissa (attention_mma.cu only)
#ifndef SPLIT_WEIGHTS
#define SPLIT_WEIGHTS 0
#endif

// 1: soft cap, sink and a factor of the results (attention_mma.cu only)
#ifndef SCORE_EXTRAS
#define SCORE_EXTRAS 0
#endif

namespace {

constexpr int D = HEAD_DIM;
constexpr int KT = 64;                 // keys per tile
constexpr int LDS = D + 8;             // shared-memory row stride in elements: conflict-free ldmatrix
constexpr int THREADS = 128;
static_assert(D % 16 == 0 && D >= 16 && D <= 256, "head size must be a multiple of 16 up to 256");

// first_partial, chunks and tile name the tile an item belongs to: its partial slots, how many of
// its items hold keys, and its index in the step (the decode kernel's merge uses them).
struct WorkItem {
    int seq, row0, kv_begin, kv_end, partial, first_partial, chunks, tile;
};

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool pred) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = pred ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}

__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* p) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0,
                                         unsigned b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
        "{%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float fast_exp2(float x) {          // ex2.approx: exp2(-inf) = 0
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}
// x and y as sums of two bfloat16 numbers each (16 bits of mantissa).
__device__ __forceinline__ void split_bf16(float x, float y, unsigned& hi, unsigned& low) {
    hi = pack_bf16(x, y);
    low = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

}  // namespace
