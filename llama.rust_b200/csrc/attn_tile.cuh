// Device helpers of the attention kernels over a step's segments and lists of cells.
#pragma once
#include "dense.cuh"

namespace b200 {

constexpr int ERR_CELL = 2, ERR_POS = 3;   // error codes: a cell outside the cache or the list, a position outside the rotary table

__device__ __forceinline__ void cp16(void *dst, const void *src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}

// shared-memory row of a key in 16-byte units: odd, so that eight lanes reading eight rows touch different banks
template <typename T>
__host__ __device__ inline int key_units(int n) { return ((n * (int)sizeof(T) + 15) / 16) | 1; }

// tile ti of 64 (or `per`) rows -> its segment, first row inside it and rows; false past the last
__device__ __forceinline__ const int32_t *find_tile(const int32_t *seg, int64_t n_seg, int64_t n_rows, int per, int ti, int *r0, int *rows, int *err) {
    for (int s = 0; s < (int)n_seg; s++) {
        const int32_t *sg = seg + s * SEG_FIELDS;
        const int n = sg[SEG_ROWS], k = (n + per - 1) / per;
        if (ti < k) {
            *r0 = ti * per;
            *rows = min(per, n - ti * per);
            if (sg[SEG_ROW0] >= 0 && (int64_t)sg[SEG_ROW0] + n <= n_rows) return sg;
            atomicExch(err, ERR_SEGMENT);
            return nullptr;
        }
        ti -= k;
    }
    return nullptr;
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void *p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void *p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}

}  // namespace b200
