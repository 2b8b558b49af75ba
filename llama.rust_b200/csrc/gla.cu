// Gated linear attention: per head a state S [dim][vdim] in F32 with
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   a_t = sigmoid(decay logit)^(1 / tau)  per key channel,
// each head's o then RMS-normed over vdim, weighted, and multiplied by silu(g).  All of it in F32.
//
// Two forms.  Token by token (decode steps, short stretches): one launch, the value columns of a head split over the blocks of a
// cluster, every thread owning the same state elements for all tokens, the head's norm summed through distributed shared memory.
// Chunks of C tokens (prompts), four launches:
//   gla_chunk_kernel   per (chunk, head): decays; the C x C matrix A of key weights inside the chunk; q scaled to the chunk's start;
//                      the chunk's own contribution to the state, with keys scaled to its end
//   gla_scan_kernel    per state element: the state in front of every chunk, and behind the last
//   gla_out_kernel     per (chunk, head, 64 value columns): o = q~ S + A v
//   gla_gate_kernel    per (row, head): norm and gate
// Decays only ever multiply (products over the tokens between two places), so no exponent can overflow however strong a decay is:
// inside a 16-token block A comes from running products, between blocks q carries the product since its block's start and k the
// product to its block's end, and the keys are carried on from block to block as the products grow.
#include <cooperative_groups.h>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace b200 {

// decode_ctx.h's segment fields
enum { GSEG_ROW0 = 0, GSEG_ROWS = 1, GSEG_SLOT = 2, GSEG_FRESH = 3, GSEG_FIELDS = 8 };

namespace {

constexpr int GLA_THREADS = 256, GLA_SUB = 16, GLA_VT = 64;

// log of the decay: log(sigmoid(z)) / tau
__device__ __forceinline__ float gla_log_decay(float z, float inv_tau) { return -(fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z)))) * inv_tau; }

// ---- token by token ------------------------------------------------------------------------------------------
template <typename W, typename Y, int VEC>
__global__ void __launch_bounds__(GLA_THREADS)
gla_step_kernel(GlaArgs a, int lanes, int cols) {
    extern __shared__ float gla_sm[];
    __shared__ float part[32], mine;
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, h = blockIdx.y;
    const int v0 = blockIdx.x * cols, vn = min(cols, a.vdim - v0);   // this block's value columns (may be none)
    const int groups = GLA_THREADS / lanes, grp = tid / lanes, c0 = (tid % lanes) * VEC;
    float *s_a = gla_sm, *s_k = s_a + a.dim, *s_q = s_k + a.dim, *s_red = s_q + a.dim;   // s_red [groups][cols]
    pdl_trigger();
    pdl_wait();
    const int32_t *sg = a.seg + (int64_t)blockIdx.z * GSEG_FIELDS;
    const int row0 = sg[GSEG_ROW0], rows = sg[GSEG_ROWS];
    bool fresh = sg[GSEG_FRESH] != 0;
    float *S = a.state + (((int64_t)sg[GSEG_SLOT] * a.heads + h) * a.dim) * a.vdim + v0;
    const W *a2 = (const W *)a.a2 + (int64_t)h * a.dim * a.rank;
    const bool active = c0 < vn;
    for (int t = 0; t < rows; t++) {
        const float *p = a.proj + (int64_t)(row0 + t) * a.ldp;
        for (int d = tid; d < a.dim; d += GLA_THREADS) {
            float z = a.a2_bias[h * a.dim + d];
            const W *w = a2 + (int64_t)d * a.rank;
            for (int r = 0; r < a.rank; r++) z = fmaf(to_f32(w[r]), p[a.off_a + r], z);
            s_a[d] = expf(gla_log_decay(z, a.inv_tau));
            s_k[d] = p[a.off_k + h * a.dim + d];
            s_q[d] = p[a.off_q + h * a.dim + d] * a.q_factor;
        }
        float v[VEC], o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) {
            v[e] = active ? p[a.off_v + h * a.vdim + v0 + c0 + e] : 0.0f;
            o[e] = 0.0f;
        }
        __syncthreads();
        if (active) {
            constexpr int U = 8;
            for (int d0 = grp; d0 < a.dim; d0 += U * groups) {
                float s[U][VEC];
#pragma unroll
                for (int u = 0; u < U; u++) {
                    const int d = d0 + u * groups;
                    if (d < a.dim && !fresh) {
                        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(s[u]) = *reinterpret_cast<const float4 *>(S + (int64_t)d * a.vdim + c0);
                        else s[u][0] = S[(int64_t)d * a.vdim + c0];
                    } else {
#pragma unroll
                        for (int e = 0; e < VEC; e++) s[u][e] = 0.0f;
                    }
                }
#pragma unroll
                for (int u = 0; u < U; u++) {
                    const int d = d0 + u * groups;
                    if (d < a.dim) {
                        const float al = s_a[d], kk = s_k[d], qq = s_q[d];
#pragma unroll
                        for (int e = 0; e < VEC; e++) {
                            s[u][e] = fmaf(al, s[u][e], kk * v[e]);
                            o[e] = fmaf(qq, s[u][e], o[e]);
                        }
                        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(S + (int64_t)d * a.vdim + c0) = *reinterpret_cast<const float4 *>(s[u]);
                        else S[(int64_t)d * a.vdim + c0] = s[u][0];
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; e++) s_red[grp * cols + c0 + e] = o[e];
        }
        fresh = false;
        __syncthreads();
        float sq = 0.0f;
        for (int c = tid; c < vn; c += GLA_THREADS) {
            float sum = 0.0f;
            for (int g = 0; g < groups; g++) sum += s_red[g * cols + c];
            s_red[c] = sum;   // only this thread reads or writes column c from here on
            sq = fmaf(sum, sum, sq);
        }
        sq = block_sum(sq, part);
        if (cluster.num_blocks() > 1) {
            if (tid == 0) mine = sq;
            cluster.sync();
            sq = 0.0f;
            for (unsigned b = 0; b < cluster.num_blocks(); b++) sq += *cluster.map_shared_rank(&mine, b);
            cluster.sync();   // nobody overwrites or leaves before everyone has read
        }
        const float scale = 1.0f / sqrtf(sq / (float)a.vdim + a.eps);
        for (int c = tid; c < vn; c += GLA_THREADS) {
            const float g = p[a.off_g + h * a.vdim + v0 + c];
            ((Y *)a.y)[(int64_t)(row0 + t) * a.ldy + h * a.vdim + v0 + c] = from_f32<Y>(s_red[c] * scale * a.norm_w[v0 + c] * silu_f32(g));
        }
        __syncthreads();
    }
}

// ---- chunks ------------------------------------------------------------------------------------------------
struct GlaScratch {
    float *q;        // [chunk][head][C][dim]   q times the decay since the chunk's start
    float *A;        // [chunk][head][C][C]
    float *dC;       // [chunk][head][dim]      the chunk's whole decay
    float *S;        // [chunk][head][dim][vdim] the chunk's contribution, then the state in front of it
    float *o;        // [n][heads][vdim]
    int chunks;      // bound: n / C + n_seg
};
// chunk ci of the step -> its segment, first row and rows; false past the last
__device__ __forceinline__ bool gla_find_chunk(const int32_t *seg, int n_seg, int C, int ci, int *row0, int *rows) {
    for (int s = 0; s < n_seg; s++) {
        const int n = seg[s * GSEG_FIELDS + GSEG_ROWS], k = (n + C - 1) / C;
        if (ci < k) {
            *row0 = seg[s * GSEG_FIELDS + GSEG_ROW0] + ci * C;
            *rows = min(C, n - ci * C);
            return true;
        }
        ci -= k;
    }
    return false;
}

template <typename W, int C>
__global__ void __launch_bounds__(GLA_THREADS)
gla_chunk_kernel(GlaArgs a, GlaScratch sc) {
    constexpr int NB = C / GLA_SUB;
    extern __shared__ float gla_sm[];
    const int dim = a.dim, DP = (dim + 3) / 4 * 4 + 4;
    float *sQ = gla_sm, *sK = sQ + C * DP, *sD = sK + C * DP, *sT = sD + C * DP, *sV = sT + NB * DP;   // sD: decays; sT: per 16-token block; sV [C][VT + 4]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, ci = blockIdx.x;
    pdl_trigger();
    pdl_wait();
    int row0, rows;
    if (!gla_find_chunk(a.seg, (int)a.n_seg, C, ci, &row0, &rows)) return;
    const float *proj = a.proj + (int64_t)row0 * a.ldp;
    const int64_t ch = (int64_t)ci * a.heads + h;

    for (int i = tid; i < C * DP; i += GLA_THREADS) {
        const int t = i / DP, d = i - t * DP;
        const bool in = t < rows && d < dim;
        sQ[i] = in ? proj[(int64_t)t * a.ldp + a.off_q + h * dim + d] * a.q_factor : 0.0f;
        sK[i] = in ? proj[(int64_t)t * a.ldp + a.off_k + h * dim + d] : 0.0f;
        if (d >= dim) sD[i] = 1.0f;
    }
    for (int i = tid; i < NB * (DP - dim); i += GLA_THREADS) sT[i / (DP - dim) * DP + dim + i % (DP - dim)] = 1.0f;
    // decays of 16 tokens of a channel per thread
    const W *a2 = (const W *)a.a2 + (int64_t)h * dim * a.rank;
    for (int i = tid; i < dim * NB; i += GLA_THREADS) {
        const int sb = i / dim, d = i - sb * dim;
        float z[GLA_SUB];
        const float bias = a.a2_bias[h * dim + d];
#pragma unroll
        for (int t = 0; t < GLA_SUB; t++) z[t] = bias;
        for (int r = 0; r < a.rank; r++) {
            const float w = to_f32(a2[(int64_t)d * a.rank + r]);
#pragma unroll
            for (int t = 0; t < GLA_SUB; t++)
                if (sb * GLA_SUB + t < rows) z[t] = fmaf(w, proj[(int64_t)(sb * GLA_SUB + t) * a.ldp + a.off_a + r], z[t]);
        }
#pragma unroll
        for (int t = 0; t < GLA_SUB; t++) sD[(sb * GLA_SUB + t) * DP + d] = sb * GLA_SUB + t < rows ? expf(gla_log_decay(z[t], a.inv_tau)) : 1.0f;
    }
    __syncthreads();

    // A inside the 16-token blocks: a warp per column j, its key carried on token by token
    float *A = sc.A + ch * C * C;
    for (int col = warp; col < C; col += GLA_THREADS / 32) {
        const int sb = col / GLA_SUB, j = col % GLA_SUB;
        float acc[GLA_SUB];
#pragma unroll
        for (int i = 0; i < GLA_SUB; i++) acc[i] = 0.0f;
        for (int d = lane; d < dim; d += 32) {
            float k = sK[col * DP + d];
#pragma unroll
            for (int i = 0; i < GLA_SUB; i++) {
                if (i < j) continue;
                const int at = (sb * GLA_SUB + i) * DP + d;
                if (i > j) k *= sD[at];
                acc[i] = fmaf(sQ[at], k, acc[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < GLA_SUB; i++) {
            const float v = warp_sum(acc[i]);
            if (lane == 0) A[(sb * GLA_SUB + i) * C + col] = i >= j ? v : 0.0f;
        }
    }
    __syncthreads();
    // q carries the decay since its block's start, k the decay to its block's end
    for (int i = tid; i < dim * NB; i += GLA_THREADS) {
        const int sb = i / dim, d = i - sb * dim;
        float p = 1.0f, s = 1.0f;
        for (int t = 0; t < GLA_SUB; t++) {
            const int at = (sb * GLA_SUB + t) * DP + d, bt = (sb * GLA_SUB + GLA_SUB - 1 - t) * DP + d;
            p *= sD[at];
            sQ[at] *= p;
            sK[bt] *= s;
            s *= sD[bt];
        }
        sT[sb * DP + d] = p;
    }
    __syncthreads();
    // A between blocks: row block I against the columns before it; then those keys go on over block I
    for (int I = 1; I <= NB; I++) {
        if (I < NB) {
            const int i = tid >> 4, j = tid & 15;
            float acc[NB];
#pragma unroll
            for (int J = 0; J < NB; J++) acc[J] = 0.0f;
            const float *q = sQ + (I * GLA_SUB + i) * DP;
            for (int d = 0; d < DP - 4; d += 4) {
                const float4 qv = *reinterpret_cast<const float4 *>(q + d);
#pragma unroll
                for (int J = 0; J < NB; J++) {
                    if (J >= I) break;
                    const float4 kv = *reinterpret_cast<const float4 *>(sK + (J * GLA_SUB + j) * DP + d);
                    acc[J] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, acc[J]))));
                }
            }
#pragma unroll
            for (int J = 0; J < NB; J++)
                if (J < I) A[(I * GLA_SUB + i) * C + J * GLA_SUB + j] = acc[J];
            __syncthreads();
        }
        if (I < NB) {
            for (int i = tid; i < I * GLA_SUB * dim; i += GLA_THREADS) {
                const int t = i / dim, d = i - t * dim;
                sK[t * DP + d] *= sT[I * DP + d];
            }
            __syncthreads();
        }
    }
    // q to the chunk's start; the chunk's decay
    for (int i = tid; i < C * dim; i += GLA_THREADS) {
        const int t = i / dim, d = i - t * dim;
        float v = sQ[t * DP + d];
        for (int s = t / GLA_SUB - 1; s >= 0; s--) v *= sT[s * DP + d];
        sc.q[ch * C * dim + i] = v;
    }
    for (int d = tid; d < dim; d += GLA_THREADS) {
        float v = 1.0f;
        for (int s = 0; s < NB; s++) v *= sT[s * DP + d];
        sc.dC[ch * dim + d] = v;
    }
    // the chunk's contribution to the state: k^T v, 64 x 64 tiles, 4 x 4 per thread
    float *dS = sc.S + ch * dim * a.vdim;
    const int ty = tid >> 4, tx = tid & 15;
    for (int v0 = 0; v0 < a.vdim; v0 += GLA_VT) {
        __syncthreads();
        for (int i = tid; i < C * GLA_VT; i += GLA_THREADS) {
            const int t = i / GLA_VT, c = i % GLA_VT;
            sV[t * (GLA_VT + 4) + c] = t < rows && v0 + c < a.vdim ? proj[(int64_t)t * a.ldp + a.off_v + h * a.vdim + v0 + c] : 0.0f;
        }
        __syncthreads();
        for (int d0 = 0; d0 < dim; d0 += 64) {
            const int d = d0 + 4 * ty;
            if (d >= dim) continue;
            float acc[4][4] = {};
#pragma unroll 4
            for (int t = 0; t < C; t++) {
                const float4 k = *reinterpret_cast<const float4 *>(sK + t * DP + d), v = *reinterpret_cast<const float4 *>(sV + t * (GLA_VT + 4) + 4 * tx);
                const float kk[4] = {k.x, k.y, k.z, k.w}, vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
#pragma unroll
                    for (int f = 0; f < 4; f++) acc[e][f] = fmaf(kk[e], vv[f], acc[e][f]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++)
#pragma unroll
                for (int f = 0; f < 4; f++)
                    if (d + e < dim && v0 + 4 * tx + f < a.vdim) dS[(int64_t)(d + e) * a.vdim + v0 + 4 * tx + f] = acc[e][f];
        }
    }
}

// one state element per thread, over the chunks of a segment
__global__ void __launch_bounds__(GLA_THREADS)
gla_scan_kernel(GlaArgs a, GlaScratch sc, int C) {
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, sidx = blockIdx.z;
    const int64_t per = (int64_t)a.dim * a.vdim, i = (int64_t)blockIdx.x * GLA_THREADS + threadIdx.x;
    if (i >= per) return;
    int first = 0;
    for (int s = 0; s < sidx; s++) first += (a.seg[s * GSEG_FIELDS + GSEG_ROWS] + C - 1) / C;
    const int32_t *sg = a.seg + sidx * GSEG_FIELDS;
    const int chunks = (sg[GSEG_ROWS] + C - 1) / C, d = (int)(i / a.vdim);
    float *state = a.state + ((int64_t)sg[GSEG_SLOT] * a.heads + h) * per + i;
    float s = sg[GSEG_FRESH] ? 0.0f : *state;
    float *p = sc.S + ((int64_t)first * a.heads + h) * per + i;
    const float *dc = sc.dC + ((int64_t)first * a.heads + h) * a.dim + d;
    const int64_t pstep = (int64_t)a.heads * per, dstep = (int64_t)a.heads * a.dim;
    int c = 0;
    for (; c + 4 <= chunks; c += 4) {
        float x[4], g[4];
#pragma unroll
        for (int u = 0; u < 4; u++) {
            x[u] = p[u * pstep];
            g[u] = dc[u * dstep];
        }
#pragma unroll
        for (int u = 0; u < 4; u++) {
            p[u * pstep] = s;
            s = fmaf(g[u], s, x[u]);
        }
        p += 4 * pstep;
        dc += 4 * dstep;
    }
    for (; c < chunks; c++, p += pstep, dc += dstep) {
        const float x = *p;
        *p = s;
        s = fmaf(*dc, s, x);
    }
    *state = s;
}

// o [C][64] = q~ [C][dim] S [dim][64] + A [C][C] v [C][64], slabs of 16 through shared memory
template <int C>
__global__ void __launch_bounds__(GLA_THREADS)
gla_out_kernel(GlaArgs a, GlaScratch sc) {
    constexpr int RT = C / 16, KS = 16;
    __shared__ float sl[KS][C + 4], sr[KS][GLA_VT + 4];
    pdl_trigger();
    pdl_wait();
    const int tid = threadIdx.x, h = blockIdx.y, ci = blockIdx.x, v0 = blockIdx.z * GLA_VT;
    int row0, rows;
    if (!gla_find_chunk(a.seg, (int)a.n_seg, C, ci, &row0, &rows)) return;
    const int64_t ch = (int64_t)ci * a.heads + h;
    const float *q = sc.q + ch * C * a.dim, *S = sc.S + ch * a.dim * a.vdim, *A = sc.A + ch * C * C;
    const int ty = tid >> 4, tx = tid & 15;
    float acc[RT][4] = {};
    const auto slab = [&]() {
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KS; k++) {
            float l[RT];
#pragma unroll
            for (int e = 0; e < RT; e++) l[e] = sl[k][RT * ty + e];
            const float4 r = *reinterpret_cast<const float4 *>(&sr[k][4 * tx]);
#pragma unroll
            for (int e = 0; e < RT; e++) {
                acc[e][0] = fmaf(l[e], r.x, acc[e][0]);
                acc[e][1] = fmaf(l[e], r.y, acc[e][1]);
                acc[e][2] = fmaf(l[e], r.z, acc[e][2]);
                acc[e][3] = fmaf(l[e], r.w, acc[e][3]);
            }
        }
        __syncthreads();
    };
    for (int d0 = 0; d0 < a.dim; d0 += KS) {
        for (int i = tid; i < C * KS; i += GLA_THREADS) {
            const int t = i / KS, k = i % KS;
            sl[k][t] = d0 + k < a.dim ? q[(int64_t)t * a.dim + d0 + k] : 0.0f;
        }
        for (int i = tid; i < KS * GLA_VT; i += GLA_THREADS) {
            const int k = i / GLA_VT, c = i % GLA_VT;
            sr[k][c] = d0 + k < a.dim && v0 + c < a.vdim ? S[(int64_t)(d0 + k) * a.vdim + v0 + c] : 0.0f;
        }
        slab();
    }
    for (int t0 = 0; t0 < rows; t0 += KS) {
        for (int i = tid; i < C * KS; i += GLA_THREADS) {
            const int t = i / KS, k = i % KS;
            sl[k][t] = t0 + k <= t ? A[t * C + t0 + k] : 0.0f;
        }
        for (int i = tid; i < KS * GLA_VT; i += GLA_THREADS) {
            const int k = i / GLA_VT, c = i % GLA_VT;
            sr[k][c] = t0 + k < rows && v0 + c < a.vdim ? a.proj[(int64_t)(row0 + t0 + k) * a.ldp + a.off_v + h * a.vdim + v0 + c] : 0.0f;
        }
        slab();
    }
#pragma unroll
    for (int e = 0; e < RT; e++) {
        const int t = RT * ty + e;
        if (t >= rows) continue;
        float *o = sc.o + ((int64_t)(row0 + t) * a.heads + h) * a.vdim;
#pragma unroll
        for (int f = 0; f < 4; f++)
            if (v0 + 4 * tx + f < a.vdim) o[v0 + 4 * tx + f] = acc[e][f];
    }
}

// a warp per (row, head)
template <typename Y>
__global__ void __launch_bounds__(GLA_THREADS)
gla_gate_kernel(GlaArgs a, const float *o) {
    pdl_trigger();
    pdl_wait();
    const int64_t item = (int64_t)blockIdx.x * (GLA_THREADS / 32) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= a.n * a.heads) return;
    const int64_t row = item / a.heads;
    const int h = (int)(item - row * a.heads);
    const float *x = o + item * a.vdim, *g = a.proj + row * a.ldp + a.off_g + h * a.vdim;
    Y *y = (Y *)a.y + row * a.ldy + h * a.vdim;
    float sq = 0.0f;
    for (int c = lane; c < a.vdim; c += 32) sq = fmaf(x[c], x[c], sq);
    const float scale = 1.0f / sqrtf(warp_sum(sq) / (float)a.vdim + a.eps);
    for (int c = lane; c < a.vdim; c += 32) y[c] = from_f32<Y>(x[c] * scale * a.norm_w[c] * silu_f32(g[c]));
}

int gla_chunk_rows(int64_t dim) { return dim <= 128 ? 64 : dim <= 256 ? 32 : dim <= 1024 ? 16 : 0; }

size_t round4(size_t n) { return (n + 3) / 4 * 4; }

template <typename W, typename Y, int VEC>
int launch_step(const GlaArgs &a, cudaStream_t s) {
    // enough blocks to fill the GPU, at least 32 columns each
    int vs = 1;
    while (vs < 8 && a.n_seg * a.heads * vs < 148 && (a.vdim + 2 * vs - 1) / (2 * vs) >= 32) vs *= 2;
    const int cols = ((a.vdim + vs - 1) / vs + VEC - 1) / VEC * VEC;
    int lanes = 1;
    while (lanes * VEC < cols) lanes *= 2;
    B200_REQUIRE(lanes <= GLA_THREADS, "gla: value size %d is too large", a.vdim);
    const size_t smem = (3 * (size_t)a.dim + (size_t)(GLA_THREADS / lanes) * cols) * 4;
    B200_REQUIRE(smem <= 200 * 1024 && a.n_seg <= 65535 && a.heads <= 65535, "gla: head size %d x %d is too large", a.dim, a.vdim);
    if (smem > 48 * 1024) B200_CUDA(cudaFuncSetAttribute(gla_step_kernel<W, Y, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_pdl_cluster(gla_step_kernel<W, Y, VEC>, dim3((unsigned)vs, (unsigned)a.heads, (unsigned)a.n_seg), dim3(GLA_THREADS), (unsigned)vs, smem, s, a, lanes, cols);
}

template <typename W, int C>
int launch_chunks(const GlaArgs &a, cudaStream_t s) {
    GlaScratch sc;
    sc.chunks = (int)((a.n + C - 1) / C + a.n_seg);
    const size_t nh = (size_t)sc.chunks * a.heads;
    sc.q = a.scratch;
    sc.A = sc.q + round4(nh * C * a.dim);
    sc.dC = sc.A + round4(nh * C * C);
    sc.S = sc.dC + round4(nh * a.dim);
    sc.o = sc.S + round4(nh * a.dim * a.vdim);
    const int DP = (a.dim + 3) / 4 * 4 + 4;
    const size_t smem = ((size_t)(3 * C + C / GLA_SUB) * DP + (size_t)C * (GLA_VT + 4)) * 4;
    B200_REQUIRE(a.heads <= 65535 && a.n_seg <= 65535, "gla: too many heads or sequences");
    if (smem > 48 * 1024) B200_CUDA(cudaFuncSetAttribute(gla_chunk_kernel<W, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    int rc = launch_pdl(gla_chunk_kernel<W, C>, dim3((unsigned)sc.chunks, (unsigned)a.heads), dim3(GLA_THREADS), smem, s, a, sc);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const int64_t per = (int64_t)a.dim * a.vdim;
    rc = launch_pdl(gla_scan_kernel, dim3((unsigned)((per + GLA_THREADS - 1) / GLA_THREADS), (unsigned)a.heads, (unsigned)a.n_seg), dim3(GLA_THREADS), 0, s, a, sc, C);
    if (rc != B200_STATUS_SUCCESS) return rc;
    rc = launch_pdl(gla_out_kernel<C>, dim3((unsigned)sc.chunks, (unsigned)a.heads, (unsigned)((a.vdim + GLA_VT - 1) / GLA_VT)), dim3(GLA_THREADS), 0, s, a, sc);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const dim3 grid((unsigned)((a.n * a.heads + GLA_THREADS / 32 - 1) / (GLA_THREADS / 32)));
    return a.y_type == B200_TYPE_F32 ? launch_pdl(gla_gate_kernel<float>, grid, dim3(GLA_THREADS), 0, s, a, (const float *)sc.o)
                                     : launch_pdl(gla_gate_kernel<__nv_bfloat16>, grid, dim3(GLA_THREADS), 0, s, a, (const float *)sc.o);
}

template <typename W>
int launch_typed(const GlaArgs &a, cudaStream_t s) {
    const int C = gla_chunk_rows(a.dim);
    if (a.scratch && C == 64) return launch_chunks<W, 64>(a, s);
    if (a.scratch && C == 32) return launch_chunks<W, 32>(a, s);
    if (a.scratch && C == 16) return launch_chunks<W, 16>(a, s);
    const bool vec = a.vdim % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    if (a.y_type == B200_TYPE_F32) return vec ? launch_step<W, float, 4>(a, s) : launch_step<W, float, 1>(a, s);
    return vec ? launch_step<W, __nv_bfloat16, 4>(a, s) : launch_step<W, __nv_bfloat16, 1>(a, s);
}

}  // namespace

size_t gla_scratch_floats(int64_t heads, int64_t dim, int64_t vdim, int64_t n, int64_t n_seg) {
    const int64_t C = gla_chunk_rows(dim);
    if (C == 0) return 4;
    const size_t nh = (size_t)((n + C - 1) / C + n_seg) * heads;
    return round4(nh * C * dim) + round4(nh * C * C) + round4(nh * dim) + round4(nh * dim * vdim) + (size_t)n * heads * vdim;
}

int launch_gla(const GlaArgs &a, cudaStream_t s) {
    B200_REQUIRE(a.proj && a.a2 && a.a2_bias && a.norm_w && a.state && a.seg && a.y, "gla: null operand");
    B200_REQUIRE(a.heads > 0 && a.dim > 0 && a.vdim > 0 && a.rank > 0 && a.n_seg > 0, "gla: bad shape");
    return a.a2_type == B200_TYPE_F32 ? launch_typed<float>(a, s) : launch_typed<__nv_bfloat16>(a, s);
}

}  // namespace b200
