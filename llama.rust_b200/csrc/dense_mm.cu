// Mat-muls over dense F32 / BF16 weights, the weighted RMS norm in front of them and row gathers.
//
// Few activation rows (a decode step): one pass over the weights, a warp per pair (or four) of weight rows, the activations read
// through L1 by every warp; no barrier unless several warps share a row group to fill the GPU.  The norm in front of the mat-mul
// rides along: w' = norm weight folds into the activation as it is read, and the row's root mean square, a factor of the whole
// result, comes from the same pass.  The weights' first loads are issued before the wait for the previous kernel.
// Many rows: BF16 x BF16 on the tensor cores (gemm_bf16_tcgen05.cu); everything else (F32 weights, row lengths a tensor map cannot
// describe) on the tiled kernel here, in F32.
#include "dense.cuh"

namespace b200 {

namespace {

constexpr int DV_WARPS = 4;

template <typename W>
struct WLoad;   // a lane's 16-byte piece of a weight row
template <>
struct WLoad<__nv_bfloat16> {
    static constexpr int E = 8;
    static __device__ __forceinline__ void unpack(const uint4 &r, float (&f)[8]) {
        f[0] = bf16_lo(r.x); f[1] = bf16_hi(r.x); f[2] = bf16_lo(r.y); f[3] = bf16_hi(r.y);
        f[4] = bf16_lo(r.z); f[5] = bf16_hi(r.z); f[6] = bf16_lo(r.w); f[7] = bf16_hi(r.w);
    }
};
template <>
struct WLoad<float> {
    static constexpr int E = 4;
    static __device__ __forceinline__ void unpack(const uint4 &r, float (&f)[4]) {
        f[0] = __uint_as_float(r.x); f[1] = __uint_as_float(r.y); f[2] = __uint_as_float(r.z); f[3] = __uint_as_float(r.w);
    }
};

// RPW weight rows per warp group, NCOL activation rows; wpr warps share a row group (pieces dealt out in turn)
template <typename W, int RPW, int NCOL, bool VEC>
__global__ void __launch_bounds__(DV_WARPS * 32, NCOL == 1 ? 8 : 4)
dense_rows_kernel(DenseMm d, int m0, int wpr) {
    constexpr int E = VEC ? WLoad<W>::E : 1;
    constexpr int U = 2;   // pieces per row in flight
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int groups = DV_WARPS / wpr, grp = warp / wpr, sub = warp % wpr;
    const int64_t row0 = ((int64_t)blockIdx.x * groups + grp) * RPW;
    const int64_t k = d.k;
    const W *w[RPW];
#pragma unroll
    for (int r = 0; r < RPW; r++) w[r] = (const W *)d.w + (row0 + r < d.n ? row0 + r : d.n - 1) * d.ldw;
    const float *x = (const float *)d.x + (int64_t)m0 * d.ldx;
    const int64_t step = (int64_t)32 * E * wpr;
    int64_t i = ((int64_t)sub * 32 + lane) * E;
    float acc[RPW][NCOL], sq[NCOL];
#pragma unroll
    for (int c = 0; c < NCOL; c++) {
        sq[c] = 0.0f;
#pragma unroll
        for (int r = 0; r < RPW; r++) acc[r][c] = 0.0f;
    }
    if constexpr (VEC) {
        uint4 q[U][RPW];
        // the first pieces: weights do not depend on the previous kernel
#pragma unroll
        for (int u = 0; u < U; u++)
#pragma unroll
            for (int r = 0; r < RPW; r++)
                q[u][r] = i + u * step < k ? ld_stream16(w[r] + i + u * step) : make_uint4(0, 0, 0, 0);
        pdl_wait();
        while (i < k) {
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int64_t at = i + u * step;
                float f[RPW][E];
#pragma unroll
                for (int r = 0; r < RPW; r++) WLoad<W>::unpack(q[u][r], f[r]);
                const int64_t nx = at + U * step;
#pragma unroll
                for (int r = 0; r < RPW; r++) q[u][r] = nx < k ? ld_stream16(w[r] + nx) : make_uint4(0, 0, 0, 0);
                if (at < k) {
                    float nw[E];
                    if (d.norm_w) {
#pragma unroll
                        for (int e = 0; e < E; e += 4) *reinterpret_cast<float4 *>(nw + e) = *reinterpret_cast<const float4 *>(d.norm_w + at + e);
                    }
#pragma unroll
                    for (int c = 0; c < NCOL; c++) {
                        float xv[E];
#pragma unroll
                        for (int e = 0; e < E; e += 4) *reinterpret_cast<float4 *>(xv + e) = *reinterpret_cast<const float4 *>(x + c * d.ldx + at + e);
                        if (d.norm_w) {
#pragma unroll
                            for (int e = 0; e < E; e++) {
                                sq[c] = fmaf(xv[e], xv[e], sq[c]);
                                xv[e] *= nw[e];
                            }
                        }
#pragma unroll
                        for (int e = 0; e < E; e++)
#pragma unroll
                            for (int r = 0; r < RPW; r++) acc[r][c] = fmaf(f[r][e], xv[e], acc[r][c]);
                    }
                }
            }
            i += U * step;
        }
    } else {
        pdl_wait();
        for (; i < k; i += step) {
            const float nw = d.norm_w ? d.norm_w[i] : 1.0f;
#pragma unroll
            for (int c = 0; c < NCOL; c++) {
                float xv = x[c * d.ldx + i];
                if (d.norm_w) {
                    sq[c] = fmaf(xv, xv, sq[c]);
                    xv *= nw;
                }
#pragma unroll
                for (int r = 0; r < RPW; r++) acc[r][c] = fmaf(to_f32(w[r][i]), xv, acc[r][c]);
            }
        }
    }
    __shared__ float part[DV_WARPS][(RPW + 1) * NCOL];
#pragma unroll
    for (int c = 0; c < NCOL; c++) {
        sq[c] = d.norm_w ? warp_sum(sq[c]) : 0.0f;
#pragma unroll
        for (int r = 0; r < RPW; r++) acc[r][c] = warp_sum(acc[r][c]);
    }
    if (lane == 0) {
#pragma unroll
        for (int c = 0; c < NCOL; c++) {
            part[warp][RPW * NCOL + c] = sq[c];
#pragma unroll
            for (int r = 0; r < RPW; r++) part[warp][r * NCOL + c] = acc[r][c];
        }
    }
    if (wpr > 1) __syncthreads();
    else __syncwarp();
    if (sub != 0 || lane >= RPW * NCOL) return;
    const int r = lane / NCOL, c = lane % NCOL;
    const bool gated = d.act == ACT_CLAMPED_GATE;
    float v = 0.0f, v2 = 0.0f, s = 0.0f;
    for (int p = 0; p < wpr; p++) {
        v += part[warp + p][r * NCOL + c];
        if (gated && !(r & 1)) v2 += part[warp + p][(r + 1) * NCOL + c];
        s += part[warp + p][RPW * NCOL + c];
    }
    int64_t row = row0 + r;
    const int64_t col = m0 + c;
    if (row >= d.n || (gated && (r & 1))) return;
    if (d.norm_w) {
        const float f = 1.0f / sqrtf(s / (float)k + d.eps);
        v *= f;
        v2 *= f;
    }
    if (d.bias) v += d.bias[row];
    if (gated) {
        if (d.bias) v2 += d.bias[row + 1];
        v = clamped_gate(v, v2, d.act_limit, d.act_alpha);
        row >>= 1;
    } else {
        v = dense_act(d.act, v);
    }
    if (d.addend) v += d.addend[col * d.ld_addend + row];
    if (d.y_type == B200_TYPE_F32) ((float *)d.y)[col * d.ldy + row] = v;
    else ((__nv_bfloat16 *)d.y)[col * d.ldy + row] = __float2bfloat16_rn(v);
}

template <typename W, int RPW, int NCOL>
int launch_rows(const DenseMm &d, int m0, bool vec, int sms, cudaStream_t s) {
    const int64_t rg = (d.n + RPW - 1) / RPW;
    int wpr = 1;
    const int64_t pieces = (d.k + (vec ? 32 * WLoad<W>::E : 32) - 1) / (vec ? 32 * WLoad<W>::E : 32);
    while (wpr < DV_WARPS && rg * wpr < (int64_t)sms * 24 && pieces > 2 * wpr) wpr *= 2;
    const int64_t groups = DV_WARPS / wpr, blocks = (rg + groups - 1) / groups;
    B200_REQUIRE(blocks < 0x7fffffffLL, "dense mat-mul: too many rows");
    return vec ? launch_pdl(dense_rows_kernel<W, RPW, NCOL, true>, dim3((unsigned)blocks), dim3(DV_WARPS * 32), 0, s, d, m0, wpr)
               : launch_pdl(dense_rows_kernel<W, RPW, NCOL, false>, dim3((unsigned)blocks), dim3(DV_WARPS * 32), 0, s, d, m0, wpr);
}

template <typename W>
int launch_few(const DenseMm &d, cudaStream_t s) {
    int dev = 0, sms = 148;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
    const bool vec = d.k % WLoad<W>::E == 0 && d.ldw % WLoad<W>::E == 0 && d.k % 4 == 0 && d.ldx % 4 == 0 && (((uintptr_t)d.w | (uintptr_t)d.x | (uintptr_t)d.norm_w) & 15) == 0;
    int rc = B200_STATUS_SUCCESS;
    for (int64_t m0 = 0; m0 < d.m && rc == B200_STATUS_SUCCESS;) {
        const int64_t left = d.m - m0;
        if (left >= 4) { rc = launch_rows<W, 4, 4>(d, (int)m0, vec, sms, s); m0 += 4; }
        else if (left >= 2) { rc = launch_rows<W, 4, 2>(d, (int)m0, vec, sms, s); m0 += 2; }
        else { rc = launch_rows<W, 2, 1>(d, (int)m0, vec, sms, s); m0 += 1; }
    }
    return rc;
}

// Tiled F32 arithmetic for any types and sizes: 64 x 64 outputs per CTA, 4 x 4 per thread
constexpr int DT = 64, DTK = 16;
template <typename W, typename X>
__global__ void __launch_bounds__(256)
dense_tiled_kernel(DenseMm d) {
    __shared__ float sw[DTK][DT + 4], sx[DTK][DT + 4];
    pdl_trigger();
    pdl_wait();
    const int64_t n0 = (int64_t)blockIdx.x * DT, m0 = (int64_t)blockIdx.y * DT;
    const int tn = (threadIdx.x & 15) * 4, tm = (threadIdx.x >> 4) * 4;
    float acc[4][4] = {};
    for (int64_t k0 = 0; k0 < d.k; k0 += DTK) {
        for (int i = threadIdx.x; i < DT * DTK; i += 256) {
            const int r = i / DTK, kk = i % DTK;
            const bool in = k0 + kk < d.k;
            sw[kk][r] = in && n0 + r < d.n ? to_f32(((const W *)d.w)[(n0 + r) * d.ldw + k0 + kk]) : 0.0f;
            sx[kk][r] = in && m0 + r < d.m ? to_f32(((const X *)d.x)[(m0 + r) * d.ldx + k0 + kk]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < DTK; kk++) {
            float a[4], b[4];
#pragma unroll
            for (int e = 0; e < 4; e++) {
                a[e] = sw[kk][tn + e];
                b[e] = sx[kk][tm + e];
            }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[j], b[i], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            int64_t row = n0 + tn + j;
            const int64_t col = m0 + tm + i;
            if (row >= d.n || col >= d.m) continue;
            float v = acc[i][j] + (d.bias ? d.bias[row] : 0.0f);
            if (d.act == ACT_CLAMPED_GATE) {
                if (j & 1) continue;
                v = clamped_gate(v, acc[i][j | 1] + (d.bias ? d.bias[row + 1] : 0.0f), d.act_limit, d.act_alpha);
                row >>= 1;
            } else {
                v = dense_act(d.act, v);
            }
            if (d.addend) v += d.addend[col * d.ld_addend + row];
            if (d.y_type == B200_TYPE_F32) ((float *)d.y)[col * d.ldy + row] = v;
            else ((__nv_bfloat16 *)d.y)[col * d.ldy + row] = __float2bfloat16_rn(v);
        }
}

template <typename Y>
__global__ void __launch_bounds__(256)
rms_norm_w_kernel(const float *__restrict__ x, int64_t ldx, const float *__restrict__ w, Y *y, int64_t ldy, int ne0, float eps) {
    __shared__ float part[32];
    pdl_trigger();
    pdl_wait();
    const float *xr = x + (int64_t)blockIdx.x * ldx;
    Y *yr = y + (int64_t)blockIdx.x * ldy;
    float sum = 0.0f;
    for (int i = threadIdx.x; i < ne0; i += 256) sum = fmaf(xr[i], xr[i], sum);
    const float scale = 1.0f / sqrtf(block_sum(sum, part) / (float)ne0 + eps);
    for (int i = threadIdx.x; i < ne0; i += 256) yr[i] = from_f32<Y>(xr[i] * scale * w[i]);
}
// rows of whole 16-byte pieces, up to 8 of four elements per thread, read once
template <typename Y>
__global__ void __launch_bounds__(256)
rms_norm_w_vec_kernel(const float *__restrict__ x, int64_t ldx, const float *__restrict__ w, Y *y, int64_t ldy, int ne0, float eps) {
    __shared__ float part[32];
    pdl_trigger();
    pdl_wait();
    const float4 *xr = (const float4 *)(x + (int64_t)blockIdx.x * ldx);
    const int n4 = ne0 / 4;
    float4 v[8];
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < 8; j++) {
        const int i = threadIdx.x + 256 * j;
        v[j] = i < n4 ? xr[i] : make_float4(0, 0, 0, 0);
        sum += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float scale = 1.0f / sqrtf(block_sum(sum, part) / (float)ne0 + eps);
#pragma unroll
    for (int j = 0; j < 8; j++) {
        const int i = threadIdx.x + 256 * j;
        if (i >= n4) break;
        const float4 g = ((const float4 *)w)[i];
        const float4 o = make_float4(v[j].x * scale * g.x, v[j].y * scale * g.y, v[j].z * scale * g.z, v[j].w * scale * g.w);
        if constexpr (sizeof(Y) == 4) ((float4 *)(y + (int64_t)blockIdx.x * ldy))[i] = o;
        else ((uint2 *)(y + (int64_t)blockIdx.x * ldy))[i] = make_uint2(bf16_pack(o.x, o.y), bf16_pack(o.z, o.w));
    }
}

template <typename T, typename Y>
__global__ void __launch_bounds__(256)
take_rows_kernel(const T *__restrict__ table, int64_t ld_table, int64_t table_rows, const int32_t *__restrict__ ids, Y *y, int64_t ldy, int ne0, float factor,
                 int *err) {
    pdl_trigger();
    pdl_wait();
    const int64_t row = ids[blockIdx.x];
    if (row < 0 || row >= table_rows) {
        if (threadIdx.x == 0) atomicExch(err, 1);
        return;
    }
    const T *t = table + row * ld_table;
    Y *o = y + (int64_t)blockIdx.x * ldy;
    if constexpr (sizeof(T) == sizeof(Y)) {
        const int per = 16 / (int)sizeof(T);
        if (factor == 1.0f && ne0 % per == 0 && (((uintptr_t)t | (uintptr_t)o) & 15) == 0) {
            for (int i = threadIdx.x; i < ne0 / per; i += 256) ((uint4 *)o)[i] = ((const uint4 *)t)[i];
            return;
        }
    }
    for (int i = threadIdx.x; i < ne0; i += 256) o[i] = from_f32<Y>(to_f32(t[i]) * factor);
}

bool dense_type(int t) { return t == B200_TYPE_F32 || t == B200_TYPE_BF16; }

}  // namespace

int launch_dense_mm(const DenseMm &d, cudaStream_t s) {
    B200_REQUIRE(d.w && d.x && d.y && dense_type(d.w_type) && dense_type(d.x_type) && dense_type(d.y_type), "dense mat-mul: operands must be F32 or BF16");
    B200_REQUIRE(d.n > 0 && d.k > 0 && d.m >= 0 && d.k < (1ll << 31) && d.m < (1ll << 31), "dense mat-mul: bad shape");
    B200_REQUIRE(d.ldw >= d.k, "dense mat-mul: weight rows overlap");
    B200_REQUIRE(d.act != ACT_CLAMPED_GATE || (d.n % 2 == 0 && d.addend == nullptr), "dense mat-mul: a gated result takes pairs of rows and no addend");
    if (d.m == 0) return B200_STATUS_SUCCESS;
    if (d.m <= DENSE_FEW_ROWS && d.x_type == B200_TYPE_F32) return d.w_type == B200_TYPE_F32 ? launch_few<float>(d, s) : launch_few<__nv_bfloat16>(d, s);
    B200_REQUIRE(d.norm_w == nullptr, "dense mat-mul: the norm rides along with up to %d F32 rows only", DENSE_FEW_ROWS);
    if (gemm_bf16_takes(d)) return launch_gemm_bf16(d, s);
    const dim3 grid((unsigned)((d.n + DT - 1) / DT), (unsigned)((d.m + DT - 1) / DT));
    B200_REQUIRE(grid.y <= 65535, "dense mat-mul: too many rows for one launch");
    if (d.w_type == B200_TYPE_F32)
        return d.x_type == B200_TYPE_F32 ? launch_pdl(dense_tiled_kernel<float, float>, grid, dim3(256), 0, s, d)
                                         : launch_pdl(dense_tiled_kernel<float, __nv_bfloat16>, grid, dim3(256), 0, s, d);
    return d.x_type == B200_TYPE_F32 ? launch_pdl(dense_tiled_kernel<__nv_bfloat16, float>, grid, dim3(256), 0, s, d)
                                     : launch_pdl(dense_tiled_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, s, d);
}

int launch_rms_norm_w(const float *x, int64_t ldx, const float *w, void *y, int y_type, int64_t ldy, int64_t ne0, int64_t nrows, float eps, cudaStream_t s) {
    B200_REQUIRE(x && w && y && dense_type(y_type) && ne0 > 0 && ne0 < (1 << 30) && nrows < 0x7fffffffLL, "rms_norm_w: bad argument");
    if (nrows == 0) return B200_STATUS_SUCCESS;
    const dim3 grid((unsigned)nrows);
    const bool vec = ne0 % 4 == 0 && ne0 <= 8192 && ldx % 4 == 0 && ldy % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)y) & 15) == 0;
    if (y_type == B200_TYPE_F32)
        return vec ? launch_pdl(rms_norm_w_vec_kernel<float>, grid, dim3(256), 0, s, x, ldx, w, (float *)y, ldy, (int)ne0, eps)
                   : launch_pdl(rms_norm_w_kernel<float>, grid, dim3(256), 0, s, x, ldx, w, (float *)y, ldy, (int)ne0, eps);
    return vec ? launch_pdl(rms_norm_w_vec_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, x, ldx, w, (__nv_bfloat16 *)y, ldy, (int)ne0, eps)
               : launch_pdl(rms_norm_w_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, x, ldx, w, (__nv_bfloat16 *)y, ldy, (int)ne0, eps);
}

int launch_take_rows(const void *table, int table_type, int64_t ld_table, int64_t table_rows, const int32_t *ids, int64_t n, void *y, int y_type, int64_t ldy,
                     int64_t ne0, float factor, cudaStream_t s) {
    B200_REQUIRE(table && ids && y && dense_type(table_type) && dense_type(y_type) && ne0 > 0 && ne0 < (1 << 30) && n < 0x7fffffffLL, "take_rows: bad argument");
    if (n == 0) return B200_STATUS_SUCCESS;
    int *err = nullptr;
    int rc = device_error_word(&err);
    if (rc != B200_STATUS_SUCCESS) return rc;
    typedef __nv_bfloat16 bf;
    const dim3 g((unsigned)n), b(256);
    const int e = (int)ne0;
    if (table_type == B200_TYPE_F32)
        return y_type == B200_TYPE_F32 ? launch_pdl(take_rows_kernel<float, float>, g, b, 0, s, (const float *)table, ld_table, table_rows, ids, (float *)y, ldy, e, factor, err)
                                       : launch_pdl(take_rows_kernel<float, bf>, g, b, 0, s, (const float *)table, ld_table, table_rows, ids, (bf *)y, ldy, e, factor, err);
    return y_type == B200_TYPE_F32 ? launch_pdl(take_rows_kernel<bf, float>, g, b, 0, s, (const bf *)table, ld_table, table_rows, ids, (float *)y, ldy, e, factor, err)
                                   : launch_pdl(take_rows_kernel<bf, bf>, g, b, 0, s, (const bf *)table, ld_table, table_rows, ids, (bf *)y, ldy, e, factor, err);
}

}  // namespace b200
