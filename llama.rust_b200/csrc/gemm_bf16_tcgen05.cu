// BF16 x BF16 mat-mul on the tensor cores for many activation rows: y[m][n] = act(w[n][k] x[m][k] + bias) + addend, F32 sums.
//
// Output tiles of 128 weight rows x NC activation rows (64, 128 or 256), walked by persistent CTAs, one per SM, the column blocks of a
// weight row block next to each other so that the weights cross HBM once.  Per tile a pipeline of K = 64 steps: one thread moves the
// two operand boxes with TMA (128-byte swizzle; the hardware fills what lies outside either matrix with zeros), one thread issues four
// M 128 x N NC x K 16 MMAs per step into one of two tensor-memory stages, four warps drain the other stage: lane = weight row, so a
// store of one activation row's 32 outputs is one contiguous piece.  The activation function and the residual add are done there;
// a gated one takes neighbouring weight rows (gate, up), which neighbouring lanes exchange, each keeping every other activation row.
// Every wait is bounded; a wait that runs out raises the CTA's abort flag and the device error word.
#include <cuda.h>

#include "dense.cuh"

namespace b200 {

namespace {

constexpr int GB_ROWS = 128, GB_K = 64, GB_THREADS = 256, GB_EPI_WARP0 = 4, GB_TSTAGES = 2;
constexpr uint32_t GB_WAIT_LIMIT = 1u << 22;
constexpr int GB_ERR_WAIT = 4;

template <int NC>
struct GbCfg {
    static constexpr int A_BYTES = GB_ROWS * GB_K * 2, B_BYTES = NC * GB_K * 2, STAGE = A_BYTES + B_BYTES;
    static constexpr int STAGES = NC == 256 ? 4 : NC == 128 ? 6 : 8;
    static constexpr int SMEM = STAGES * STAGE + 1024;
    // kind::f16 instruction descriptor: F32 accumulator, BF16 x BF16, both operands K-major, N = NC, M = 128
    static constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NC >> 3) << 17) | ((uint32_t)(GB_ROWS >> 4) << 24);
};
struct GbBars {
    uint64_t full[8], empty[8], tfull[GB_TSTAGES], tempty[GB_TSTAGES];
    uint32_t tmem_base;
    int abort_flag;
};
struct GbOut {
    void *y;
    int y_type;
    int64_t ldy;
    const float *addend;
    int64_t ld_addend;
    const float *bias;
    int act;
    float act_limit, act_alpha;
    int n, m;
};

__device__ __forceinline__ uint32_t gb_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ uint64_t gb_desc(uint32_t addr) {   // K-major, 128-byte swizzle, 8-row groups 1024 bytes apart
    return (uint64_t)((addr >> 4) & 0x3fffu) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void gb_bar_init(uint32_t bar, uint32_t count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void gb_bar_arrive(uint32_t bar) {
    asm volatile("{ .reg .b64 st; mbarrier.arrive.shared::cta.b64 st, [%0]; }" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void gb_bar_expect(uint32_t bar, uint32_t bytes) {
    asm volatile("{ .reg .b64 st; mbarrier.arrive.expect_tx.shared::cta.b64 st, [%0], %1; }" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool gb_bar_wait(uint32_t bar, uint32_t parity, volatile int *abort_flag) {
    for (uint32_t it = 0; it < GB_WAIT_LIMIT; it++) {
        uint32_t ok;
        asm volatile("{ .reg .pred p; mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2; selp.u32 %0, 1, 0, p; }" : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
        if (ok) return true;
        if ((it & 255) == 255 && *abort_flag) return false;
    }
    *abort_flag = 1;
    return false;
}
__device__ __forceinline__ void gb_tma_load(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst), "l"(map), "r"(x),
                 "r"(y), "r"(bar)
                 : "memory");
}
__device__ __forceinline__ void gb_mma(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, int accumulate) {
    asm volatile("{ .reg .pred p; setp.ne.b32 p, %4, 0; tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }" ::"r"(d_tmem), "l"(adesc), "l"(bdesc),
                 "r"(idesc), "r"(accumulate)
                 : "memory");
}
__device__ __forceinline__ void gb_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void gb_tmem_ld32(uint32_t (&r)[32], uint32_t taddr) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
          "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]),
          "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr)
        : "memory");
}

template <int NC>
__global__ void __launch_bounds__(GB_THREADS, 1)
gemm_bf16_tcgen05_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, GbOut o, int ksteps, int col_blocks, int tiles, int *err) {
    using C = GbCfg<NC>;
    constexpr int S = C::STAGES;
    extern __shared__ uint8_t gb_raw[];
    __shared__ GbBars bars;
    pdl_trigger();
    const uint32_t smem = (gb_smem(gb_raw) + 1023u) & ~1023u;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    volatile int *abort_flag = &bars.abort_flag;
    if (threadIdx.x == 0) {
        for (int i = 0; i < S; i++) {
            gb_bar_init(gb_smem(&bars.full[i]), 1);
            gb_bar_init(gb_smem(&bars.empty[i]), 1);
        }
        for (int i = 0; i < GB_TSTAGES; i++) {
            gb_bar_init(gb_smem(&bars.tfull[i]), 1);
            gb_bar_init(gb_smem(&bars.tempty[i]), 4);
        }
        bars.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 2) {
        // both accumulator stages; the operand stages fill the SM's shared memory, so no second CTA competes for the columns
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(gb_smem(&bars.tmem_base)), "r"(GB_TSTAGES * NC) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = bars.tmem_base;
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            int step = 0, issued = -1;
            for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
                const int rb = t / col_blocks, cb = t - rb * col_blocks;
                bool ok = true;
                for (int ks = 0; ks < ksteps; ks++, step++) {
                    const int s = step % S;
                    if (!gb_bar_wait(gb_smem(&bars.empty[s]), ((uint32_t)(step / S) & 1u) ^ 1u, abort_flag)) {
                        ok = false;
                        break;
                    }
                    const uint32_t bar = gb_smem(&bars.full[s]), stage = smem + (uint32_t)(s * C::STAGE);
                    gb_bar_expect(bar, C::STAGE);
                    gb_tma_load(stage, &wmap, ks * GB_K, rb * GB_ROWS, bar);
                    gb_tma_load(stage + C::A_BYTES, &xmap, ks * GB_K, cb * NC, bar);
                    issued = step;
                }
                if (!ok) break;
            }
            // a CTA that gives up still waits (bounded) for the copies it has in flight
            if (*abort_flag)
                for (int p = issued - S + 1 < 0 ? 0 : issued - S + 1; p <= issued; p++) {
                    for (uint32_t it = 0; it < GB_WAIT_LIMIT; it++) {
                        uint32_t ok;
                        asm volatile("{ .reg .pred p; mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2; selp.u32 %0, 1, 0, p; }"
                                     : "=r"(ok) : "r"(gb_smem(&bars.full[p % S])), "r"((uint32_t)(p / S) & 1u) : "memory");
                        if (ok) break;
                    }
                }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int step = 0, j = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, j++) {
                const int ts = j % GB_TSTAGES;
                if (!gb_bar_wait(gb_smem(&bars.tempty[ts]), ((uint32_t)(j / GB_TSTAGES) & 1u) ^ 1u, abort_flag)) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t d_acc = tmem + (uint32_t)(ts * NC);
                for (int ks = 0; ks < ksteps; ks++, step++) {
                    const int s = step % S;
                    if (!gb_bar_wait(gb_smem(&bars.full[s]), (uint32_t)(step / S) & 1u, abort_flag)) {
                        ok = false;
                        break;
                    }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t stage = smem + (uint32_t)(s * C::STAGE);
                    const uint64_t ad = gb_desc(stage), bd = gb_desc(stage + C::A_BYTES);
#pragma unroll
                    for (int i = 0; i < GB_K / 16; i++) gb_mma(d_acc, ad + 2 * i, bd + 2 * i, C::IDESC, (ks | i) != 0);   // 32 bytes on per K = 16
                    gb_commit(gb_smem(&bars.empty[s]));
                }
                if (ok) gb_commit(gb_smem(&bars.tfull[ts]));
            }
        }
    } else if (warp >= GB_EPI_WARP0) {
        const int q = warp - GB_EPI_WARP0;   // tensor-memory lanes 32 q ..
        int j = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x, j++) {
            const int rb = t / col_blocks, cb = t - rb * col_blocks, ts = j % GB_TSTAGES;
            if (!__all_sync(0xffffffffu, gb_bar_wait(gb_smem(&bars.tfull[ts]), (uint32_t)(j / GB_TSTAGES) & 1u, abort_flag))) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int row = rb * GB_ROWS + 32 * q + lane, col0 = cb * NC;
            const bool row_ok = row < o.n;
            const float bias = o.bias && row_ok ? o.bias[row] : 0.0f;
            const uint32_t trow = tmem + ((uint32_t)(32 * q) << 16) + (uint32_t)(ts * NC);
#pragma unroll 1
            for (int c0 = 0; c0 < NC; c0 += 32) {
                uint32_t v[32];
                float ad[32];
                gb_tmem_ld32(v, trow + (uint32_t)c0);
                if (o.addend) {
#pragma unroll
                    for (int c = 0; c < 32; c++) {
                        const int col = col0 + c0 + c;
                        ad[c] = row_ok && col < o.m ? o.addend[(int64_t)col * o.ld_addend + row] : 0.0f;
                    }
                }
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (c0 + 32 == NC) {
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                    __syncwarp();
                    if (lane == 0) gb_bar_arrive(gb_smem(&bars.tempty[ts]));
                }
                if (o.act == ACT_CLAMPED_GATE) {
                    const int odd = lane & 1;
#pragma unroll
                    for (int c = 0; c < 32; c += 2) {
                        const float x0 = __uint_as_float(v[c]) + bias, x1 = __uint_as_float(v[c + 1]) + bias;
                        const float other = __shfl_xor_sync(0xffffffffu, odd ? x0 : x1, 1);
                        const float r = clamped_gate(odd ? other : x0, odd ? x1 : other, o.act_limit, o.act_alpha);
                        const int col = col0 + c0 + c + odd;
                        if (!row_ok || col >= o.m) continue;
                        if (o.y_type == B200_TYPE_F32) ((float *)o.y)[(int64_t)col * o.ldy + (row >> 1)] = r;
                        else ((__nv_bfloat16 *)o.y)[(int64_t)col * o.ldy + (row >> 1)] = __float2bfloat16_rn(r);
                    }
                    continue;
                }
                if (!row_ok) continue;
#pragma unroll
                for (int c = 0; c < 32; c++) {
                    const int col = col0 + c0 + c;
                    if (col >= o.m) break;
                    float r = dense_act(o.act, __uint_as_float(v[c]) + bias);
                    if (o.addend) r += ad[c];
                    if (o.y_type == B200_TYPE_F32) ((float *)o.y)[(int64_t)col * o.ldy + row] = r;
                    else ((__nv_bfloat16 *)o.y)[(int64_t)col * o.ldy + row] = __float2bfloat16_rn(r);
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 2) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(GB_TSTAGES * NC) : "memory");
    }
    if (threadIdx.x == 0 && bars.abort_flag) atomicExch(err, GB_ERR_WAIT);
}

typedef CUresult (*encode_fn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                              const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
encode_fn tensor_map_encoder() {
    static encode_fn fn = nullptr;
    if (!fn) {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &p, 12000, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
            fn = (encode_fn)p;
        else cudaGetLastError();
    }
    return fn;
}
// rows of k BF16 elements ld apart, in boxes of 64 elements x box_rows
int rows_map(CUtensorMap *map, const void *base, int64_t k, int64_t rows, int64_t ld, int box_rows) {
    encode_fn enc = tensor_map_encoder();
    B200_REQUIRE(enc != nullptr, "gemm: the driver has no tensor-map encoder");
    const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)GB_K, (cuuint32_t)box_rows}, es[2] = {1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    B200_REQUIRE(r == CUDA_SUCCESS, "gemm: tensor map of %lld x %lld (stride %lld) refused (%d)", (long long)rows, (long long)k, (long long)ld, (int)r);
    return B200_STATUS_SUCCESS;
}

template <int NC>
int launch_nc(const DenseMm &d, int sms, cudaStream_t s) {
    using C = GbCfg<NC>;
    static bool attr_done[64] = {false};
    int dev = 0;
    B200_CUDA(cudaGetDevice(&dev));
    B200_REQUIRE(dev >= 0 && dev < 64, "gemm: device index %d out of range", dev);
    if (!attr_done[dev]) {
        B200_CUDA(cudaFuncSetAttribute(gemm_bf16_tcgen05_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM));
        attr_done[dev] = true;
    }
    CUtensorMap wmap, xmap;
    int rc = rows_map(&wmap, d.w, d.k, d.n, d.ldw, GB_ROWS);
    if (rc == B200_STATUS_SUCCESS) rc = rows_map(&xmap, d.x, d.k, d.m, d.ldx, NC);
    if (rc != B200_STATUS_SUCCESS) return rc;
    int *err = nullptr;
    rc = device_error_word(&err);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const int64_t rb = (d.n + GB_ROWS - 1) / GB_ROWS, cb = (d.m + NC - 1) / NC;
    B200_REQUIRE(rb * cb < (1ll << 31), "gemm: too many tiles");
    const GbOut o = {d.y, d.y_type, d.ldy, d.addend, d.ld_addend, d.bias, d.act, d.act_limit, d.act_alpha, (int)d.n, (int)d.m};
    const int tiles = (int)(rb * cb);
    return launch_pdl(gemm_bf16_tcgen05_kernel<NC>, dim3((unsigned)(tiles < sms ? tiles : sms)), dim3(GB_THREADS), (size_t)C::SMEM, s, wmap, xmap, o,
                      (int)((d.k + GB_K - 1) / GB_K), (int)cb, tiles, err);
}

}  // namespace

// what the tensor maps can describe: 16-byte aligned bases and row strides
bool gemm_bf16_takes(const DenseMm &d) {
    return d.w_type == B200_TYPE_BF16 && d.x_type == B200_TYPE_BF16 && d.k % 8 == 0 && d.ldx % 8 == 0 && d.ldw % 8 == 0 && (((uintptr_t)d.w | (uintptr_t)d.x) & 15) == 0 &&
           d.n < (1ll << 31) - 256 && d.m < (1ll << 31) - 256 && d.norm_w == nullptr;
}

int launch_gemm_bf16(const DenseMm &d, cudaStream_t s) {
    int dev = 0, sms = 148;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
    if (d.m <= 64) return launch_nc<64>(d, sms, s);
    const int64_t rb = (d.n + GB_ROWS - 1) / GB_ROWS;
    const auto waves = [&](int nc) { return (rb * ((d.m + nc - 1) / nc) + sms - 1) / sms; };
    // a 256-wide tile takes about 1.8 times a 128-wide one
    if (d.m <= 128 || 10 * waves(128) <= 18 * waves(256)) return launch_nc<128>(d, sms, s);
    return launch_nc<256>(d, sms, s);
}

}  // namespace b200
