// Row kernels around the residual stream: layer norms on both sides of a residual sum as one launch, and token embeddings with a
// second table indexed by (previous token, token).
//
// norm_sum: x' = x + norm(y) scale, h = norm'(x').  A block owns a row; means and variances are taken in two passes over registers
// (deviations from the mean, so a large mean costs no precision).  A norm alone is the case without y.
#include "dense.cuh"

namespace b200 {

namespace {

constexpr int NS_VEC = 2;   // pieces of four elements a thread of the vector form holds

// sum over a block of whole warps, the same value in every thread; part: 32 floats of shared memory
__device__ __forceinline__ float row_sum(float v, float *part) {
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    if (nw == 1) return v;
    if (lane == 0) part[warp] = v;
    __syncthreads();
    v = warp_sum(lane < nw ? part[lane] : 0.0f);
    __syncthreads();
    return v;
}

// rows of whole 16-byte pieces, read once: blockDim.x * VEC * 4 elements at most.  AHEAD: the weights are fetched before the wait for the
// previous kernel (a few rows, where a block's latency is what counts)
template <typename Y, int VEC, bool AHEAD>
__global__ void __launch_bounds__(1024)
norm_sum_vec_kernel(NormSum a) {
    __shared__ float part[32];
    const int n4 = (int)a.ne0 / 4;
    const int64_t row = blockIdx.x;
    const float inv = 1.0f / (float)a.ne0;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f), one = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
    float4 v[VEC], x[VEC], w1[VEC], b1[VEC], sc[VEC], w2[VEC], b2[VEC];
    bool in[VEC];
    int at[VEC];
#pragma unroll
    for (int j = 0; j < VEC; j++) {
        at[j] = threadIdx.x + j * blockDim.x;
        in[j] = at[j] < n4;
        if (!in[j]) at[j] = 0;
    }
    const auto fetch = [&](float4 (&r)[VEC], const float *p, const float4 &none) {
#pragma unroll
        for (int j = 0; j < VEC; j++) r[j] = p ? ((const float4 *)p)[at[j]] : none;
    };
    const auto fetch_first = [&]() {
        fetch(w1, a.w1, one);
        fetch(b1, a.b1, zero);
        fetch(sc, a.scale, one);
    };
    const auto fetch_second = [&]() {
        fetch(w2, a.w2, one);
        fetch(b2, a.b2, zero);
    };
    const auto normed = [&](float4 (&r)[VEC], const float4 (&w)[VEC], const float4 (&b)[VEC]) {
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < VEC; j++)
            if (in[j]) s += (r[j].x + r[j].y) + (r[j].z + r[j].w);
        const float mean = row_sum(s, part) * inv;
        float q = 0.0f;
#pragma unroll
        for (int j = 0; j < VEC; j++) {
            r[j] = make_float4(r[j].x - mean, r[j].y - mean, r[j].z - mean, r[j].w - mean);
            if (in[j]) q += (r[j].x * r[j].x + r[j].y * r[j].y) + (r[j].z * r[j].z + r[j].w * r[j].w);
        }
        const float f = 1.0f / sqrtf(row_sum(q, part) * inv + a.eps);
#pragma unroll
        for (int j = 0; j < VEC; j++)
            r[j] = make_float4(fmaf(r[j].x * f, w[j].x, b[j].x), fmaf(r[j].y * f, w[j].y, b[j].y), fmaf(r[j].z * f, w[j].z, b[j].z), fmaf(r[j].w * f, w[j].w, b[j].w));
    };
    pdl_trigger();
    if constexpr (AHEAD) {
        fetch_first();
        fetch_second();
    }
    pdl_wait();
#pragma unroll
    for (int j = 0; j < VEC; j++) {
        x[j] = ((const float4 *)(a.x + row * a.ldx))[at[j]];
        if (a.y) v[j] = ((const float4 *)(a.y + row * a.ldy))[at[j]];
    }
    if (a.y) {
        if constexpr (!AHEAD) fetch_first();
        normed(v, w1, b1);
#pragma unroll
        for (int j = 0; j < VEC; j++) {
            x[j] = make_float4(fmaf(v[j].x, sc[j].x, x[j].x), fmaf(v[j].y, sc[j].y, x[j].y), fmaf(v[j].z, sc[j].z, x[j].z), fmaf(v[j].w, sc[j].w, x[j].w));
            if (in[j]) ((float4 *)(a.sum + row * a.ld_sum))[at[j]] = x[j];
        }
    }
    if (!a.h) return;
    if (a.w2) {
        if constexpr (!AHEAD) fetch_second();
        normed(x, w2, b2);
    }
#pragma unroll
    for (int j = 0; j < VEC; j++) {
        if (!in[j]) continue;
        if constexpr (sizeof(Y) == 4) ((float4 *)((float *)a.h + row * a.ldh))[at[j]] = x[j];
        else ((uint2 *)((__nv_bfloat16 *)a.h + row * a.ldh))[at[j]] = make_uint2(bf16_pack(x[j].x, x[j].y), bf16_pack(x[j].z, x[j].w));
    }
}

template <typename Y>
__global__ void __launch_bounds__(256)
norm_sum_kernel(NormSum a) {
    __shared__ float part[32];
    const int n = (int)a.ne0;
    const int64_t row = blockIdx.x;
    const float inv = 1.0f / (float)n;
    const auto stats = [&](const float *r, float *mean, float *f) {
        float s = 0.0f, q = 0.0f;
        for (int i = threadIdx.x; i < n; i += 256) s += r[i];
        *mean = row_sum(s, part) * inv;
        for (int i = threadIdx.x; i < n; i += 256) q = fmaf(r[i] - *mean, r[i] - *mean, q);
        *f = 1.0f / sqrtf(row_sum(q, part) * inv + a.eps);
    };
    pdl_trigger();
    pdl_wait();
    const float *x = a.x + row * a.ldx;
    float mean, f;
    if (a.y) {
        const float *y = a.y + row * a.ldy;
        float *o = a.sum + row * a.ld_sum;
        stats(y, &mean, &f);
        for (int i = threadIdx.x; i < n; i += 256)   // (a thread comes back to the elements it wrote itself)
            o[i] = fmaf(fmaf((y[i] - mean) * f, a.w1[i], a.b1 ? a.b1[i] : 0.0f), a.scale ? a.scale[i] : 1.0f, x[i]);
        x = o;
    }
    if (!a.h) return;
    if (a.w2) stats(x, &mean, &f);
    Y *h = (Y *)a.h + row * a.ldh;
    for (int i = threadIdx.x; i < n; i += 256) h[i] = from_f32<Y>(a.w2 ? fmaf((x[i] - mean) * f, a.w2[i], a.b2 ? a.b2[i] : 0.0f) : x[i]);
}

template <typename T, typename Y>
__global__ void __launch_bounds__(256)
pair_embed_kernel(PairEmbed a, bool vec, int *err) {
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x, token = a.tokens[row];
    if (token < 0 || token >= a.table_rows) {
        if (threadIdx.x == 0) atomicExch(err, 1);
        return;
    }
    const T *t = (const T *)a.table + token * a.ld_table, *p = nullptr;
    if (a.pairs) {
        const int64_t prev = a.prev[row];
        p = (const T *)a.pairs + (prev < 0 ? a.buckets : (prev * a.mul_prev + token * a.mul_cur) % a.buckets) * a.ld_pairs;
    }
    if (vec) {   // four elements at a time, all of a thread's loads ahead of its stores
        const auto four = [](const T *q) {
            if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float4 *>(q);
            else {
                const uint2 w = *reinterpret_cast<const uint2 *>(q);
                return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
            }
        };
        constexpr int U = 4;
        for (int i0 = 4 * threadIdx.x; i0 < (int)a.ne0; i0 += 4 * 256 * U) {
            float4 v[U];
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int i = i0 + 4 * 256 * u;
                if (i >= (int)a.ne0) break;
                const float4 e = four(t + i), q = p ? four(p + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                v[u] = make_float4(e.x * a.factor + q.x, e.y * a.factor + q.y, e.z * a.factor + q.z, e.w * a.factor + q.w);
            }
#pragma unroll
            for (int u = 0; u < U; u++) {
                const int i = i0 + 4 * 256 * u;
                if (i >= (int)a.ne0) break;
                *reinterpret_cast<float4 *>(a.y + row * a.ldy + i) = v[u];
                if (!a.h) continue;
                if constexpr (sizeof(Y) == 4) *reinterpret_cast<float4 *>((Y *)a.h + row * a.ldh + i) = v[u];
                else *reinterpret_cast<uint2 *>((Y *)a.h + row * a.ldh + i) = make_uint2(bf16_pack(v[u].x, v[u].y), bf16_pack(v[u].z, v[u].w));
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < (int)a.ne0; i += 256) {
        const float v = to_f32(t[i]) * a.factor + (p ? to_f32(p[i]) : 0.0f);
        a.y[row * a.ldy + i] = v;
        if (a.h) ((Y *)a.h)[row * a.ldh + i] = from_f32<Y>(v);
    }
}

}  // namespace

int launch_norm_sum(const NormSum &a, cudaStream_t s) {
    B200_REQUIRE(a.x && (a.y || a.h) && (!a.y || (a.w1 && a.sum)) && a.ne0 > 0 && a.ne0 < (1 << 30) && a.n < 0x7fffffffLL, "norm_sum: bad argument");
    B200_REQUIRE(!a.h || a.h_type == B200_TYPE_F32 || a.h_type == B200_TYPE_BF16, "norm_sum: the second result must be F32 or BF16");
    if (a.n == 0) return B200_STATUS_SUCCESS;
    const uintptr_t all = (uintptr_t)a.x | (uintptr_t)a.y | (uintptr_t)a.w1 | (uintptr_t)a.b1 | (uintptr_t)a.scale | (uintptr_t)a.sum | (uintptr_t)a.w2 | (uintptr_t)a.b2 |
                          (uintptr_t)a.h;
    const bool vec = (a.ne0 | a.ldx | a.ldy | a.ld_sum | a.ldh) % 4 == 0 && (all & 15) == 0 && a.ne0 <= 1024 * NS_VEC * 4;
    const bool half = a.h && a.h_type == B200_TYPE_BF16;
    const dim3 grid((unsigned)a.n);
    if (!vec) return half ? launch_pdl(norm_sum_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, a) : launch_pdl(norm_sum_kernel<float>, grid, dim3(256), 0, s, a);
    const int64_t pieces = a.ne0 / 4;
    if (a.n <= DENSE_FEW_ROWS && pieces <= 1024) {   // one piece per thread: a row's chain of sums is then shortest
        const dim3 block((unsigned)((pieces + 31) / 32 * 32));
        return half ? launch_pdl(norm_sum_vec_kernel<__nv_bfloat16, 1, true>, grid, block, 0, s, a) : launch_pdl(norm_sum_vec_kernel<float, 1, true>, grid, block, 0, s, a);
    }
    const dim3 block((unsigned)(((pieces + NS_VEC - 1) / NS_VEC + 31) / 32 * 32));
    return half ? launch_pdl(norm_sum_vec_kernel<__nv_bfloat16, NS_VEC, false>, grid, block, 0, s, a) : launch_pdl(norm_sum_vec_kernel<float, NS_VEC, false>, grid, block, 0, s, a);
}

int launch_pair_embed(const PairEmbed &a, cudaStream_t s) {
    B200_REQUIRE(a.table && a.tokens && a.y && (a.type == B200_TYPE_F32 || a.type == B200_TYPE_BF16) && a.ne0 > 0 && a.ne0 < (1 << 30) && a.n < 0x7fffffffLL,
                 "pair_embed: bad argument");
    B200_REQUIRE(!a.pairs || (a.prev && a.buckets > 0 && a.mul_prev >= 0 && a.mul_cur >= 0), "pair_embed: bad table of pairs");
    B200_REQUIRE(!a.h || a.h_type == B200_TYPE_F32 || a.h_type == B200_TYPE_BF16, "pair_embed: the copy must be F32 or BF16");
    if (a.n == 0) return B200_STATUS_SUCCESS;
    int *err = nullptr;
    int rc = device_error_word(&err);
    if (rc != B200_STATUS_SUCCESS) return rc;
    typedef __nv_bfloat16 bf;
    const dim3 g((unsigned)a.n), b(256);
    const bool half = a.h && a.h_type == B200_TYPE_BF16;
    const bool vec = (a.ne0 | a.ld_table | a.ld_pairs | a.ldy | a.ldh) % 4 == 0 && (((uintptr_t)a.table | (uintptr_t)a.pairs | (uintptr_t)a.y | (uintptr_t)a.h) & 15) == 0;
    if (a.type == B200_TYPE_F32) return half ? launch_pdl(pair_embed_kernel<float, bf>, g, b, 0, s, a, vec, err) : launch_pdl(pair_embed_kernel<float, float>, g, b, 0, s, a, vec, err);
    return half ? launch_pdl(pair_embed_kernel<bf, bf>, g, b, 0, s, a, vec, err) : launch_pdl(pair_embed_kernel<bf, float>, g, b, 0, s, a, vec, err);
}

}  // namespace b200
