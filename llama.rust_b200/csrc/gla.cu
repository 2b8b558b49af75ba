// Gated linear attention: a head keeps a state S [dim][vdim]; a token first fades it, row d by its decay a[d] (the decay logit's
// sigmoid to the power 1 / tau), then adds its key times its value, and reads it with its query:
//     S[d][e] <- a[d] S[d][e] + k[d] v[e],      o[e] = sum_d q[d] S[d][e]
// The head's o goes through an RMS norm with a weight and is gated by silu(g).  All of it in F32.
//
// Two forms.  Token by token (decode steps, short stretches): one launch, the value columns of a head split over the blocks of a
// cluster, every thread owning the same state elements for all tokens, the head's norm summed through distributed shared memory.
// Chunks of C tokens (prompts), four launches:
//   gla_chunk_kernel   per (chunk, head): decays; the C x C matrix A of key weights inside the chunk; q scaled to the chunk's start,
//                      k to its end
//   gla_mm_kernel      the chunk's own contribution to the state, k^T v
//   gla_scan_kernel    per state element: the state in front of every chunk, and behind the last
//   gla_mm_kernel      o = q S + A v, with the head's norm and gate where one block holds the whole head (vdim up to 256;
//                      gla_gate_kernel otherwise)
// Decays only ever multiply (products over the tokens between two places), so no exponent can overflow however strong a decay is:
// inside a 16-token block A comes from running products, between blocks q carries the product since its block's start and k the
// product to its block's end, and the keys are carried on from block to block as the products grow.
#include <cooperative_groups.h>

#include "dense.cuh"

namespace cg = cooperative_groups;

namespace b200 {

namespace {

constexpr int GLA_THREADS = 256, GLA_SUB = 16;

// log of the decay: log(sigmoid(z)) / tau
__device__ __forceinline__ float gla_log_decay(float z, float inv_tau) { return -(fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z)))) * inv_tau; }

__device__ __forceinline__ bool gla_segment_ok(const GlaArgs &a, const int32_t *sg) {
    return sg[SEG_ROW0] >= 0 && sg[SEG_ROWS] >= 0 && (int64_t)sg[SEG_ROW0] + sg[SEG_ROWS] <= a.n && sg[SEG_SLOT] >= 0 && sg[SEG_SLOT] < a.n_slots;
}

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
    // the step's inputs are in place before its first kernel starts
    const int32_t *sg = a.seg + (int64_t)blockIdx.z * SEG_FIELDS;
    const int row0 = sg[SEG_ROW0], rows = sg[SEG_ROWS];
    if (!gla_segment_ok(a, sg)) {   // (the same for every block of the cluster)
        if (tid == 0) atomicExch(a.err, ERR_SEGMENT);
        return;
    }
    bool fresh = sg[SEG_FRESH] != 0;
    float *S = a.state + (((int64_t)sg[SEG_SLOT] * a.heads + h) * a.dim) * a.vdim + v0;
    const W *a2 = (const W *)a.a2 + (int64_t)h * a.dim * a.rank;
    for (int d = tid; d < a.dim; d += GLA_THREADS) {
        for (int c = 0; c < vn; c += 32) l2_prefetch(S + (int64_t)d * a.vdim + c);
        l2_prefetch(a2 + (int64_t)d * a.rank);
    }
    pdl_wait();
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
    float *q;        // [chunk][head][dim][C]   q times the decay since the chunk's start, transposed
    float *k;        // [chunk][head][C][dim]   k times the decay to the chunk's end
    float *A;        // [chunk][head][C keys][C rows]
    float *dC;       // [chunk][head][dim]      the chunk's whole decay
    float *S;        // [chunk][head][dim][vdim] the chunk's contribution, then the state in front of it
    float *o;        // [n][heads][vdim], when a head's values do not fit one block
    int chunks;      // there is room for
};
// chunk ci of the step -> its segment, first row and rows; false past the last
__device__ __forceinline__ bool gla_find_chunk(const GlaArgs &a, int C, int ci, int *row0, int *rows) {
    for (int s = 0; s < (int)a.n_seg; s++) {
        const int n = a.seg[s * SEG_FIELDS + SEG_ROWS], k = (n + C - 1) / C;
        if (ci < k) {
            *row0 = a.seg[s * SEG_FIELDS + SEG_ROW0] + ci * C;
            *rows = min(C, n - ci * C);
            return gla_segment_ok(a, a.seg + s * SEG_FIELDS);   // (the scan reports one that is not)
        }
        ci -= k;
    }
    return false;
}
// BYTES of 4 or 16 from global to shared memory, zeros when !in
template <int BYTES>
__device__ __forceinline__ void gla_cp(float *dst, const float *src, bool in) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if constexpr (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(in ? 16 : 0) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(in ? 4 : 0) : "memory");
}

constexpr int GLA_RANK = 16;   // ranks of the decay input staged at a time

template <typename W, int C, int VEC>
__global__ void __launch_bounds__(GLA_THREADS)
gla_chunk_kernel(GlaArgs a, GlaScratch sc) {
    constexpr int NB = C / GLA_SUB;
    extern __shared__ __align__(16) float gla_sm[];
    const int dim = a.dim, DP = (dim + 3) / 4 * 4 + 4;
    float *sQ = gla_sm, *sK = sQ + C * DP, *sD = sK + C * DP, *sT = sD + C * DP, *sA = sT + NB * DP;   // sD: decays; sT: per 16-token block; sA [C][GLA_RANK]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, ci = blockIdx.x;
    pdl_trigger();
    pdl_wait();
    int row0, rows;
    if (!gla_find_chunk(a, C, ci, &row0, &rows)) return;
    const float *proj = a.proj + (int64_t)row0 * a.ldp;
    const int64_t ch = (int64_t)ci * a.heads + h;

    // q and k; what pads a row is zero (decays: one)
    for (int t = warp; t < C; t += GLA_THREADS / 32)
        for (int d = lane * VEC; d < DP; d += 32 * VEC) {
            const bool in = t < rows && d < dim;
            const float *p = proj + (in ? (int64_t)t * a.ldp + h * dim + d : 0);
            gla_cp<4 * VEC>(sQ + t * DP + d, p + a.off_q, in);
            gla_cp<4 * VEC>(sK + t * DP + d, p + a.off_k, in);
        }
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < C * (DP - dim); i += GLA_THREADS) sD[i / (DP - dim) * DP + dim + i % (DP - dim)] = 1.0f;
    for (int i = tid; i < NB * (DP - dim); i += GLA_THREADS) sT[i / (DP - dim) * DP + dim + i % (DP - dim)] = 1.0f;
    // decays of 16 tokens of a channel per thread; the low-rank input through shared memory, 16 ranks at a time
    const W *a2 = (const W *)a.a2 + (int64_t)h * dim * a.rank;
    for (int i0 = 0; i0 < dim * NB; i0 += GLA_THREADS) {
        const int i = i0 + tid, sb = min(i / dim, NB - 1), d = i - sb * dim;
        const bool mine = i < dim * NB;
        float z[GLA_SUB];
        const float bias = mine ? a.a2_bias[h * dim + d] : 0.0f;
#pragma unroll
        for (int t = 0; t < GLA_SUB; t++) z[t] = bias;
        for (int r0 = 0; r0 < a.rank; r0 += GLA_RANK) {
            if (i0 > 0 || r0 > 0) __syncthreads();
            if (i0 == 0 || a.rank > GLA_RANK)
                for (int j = tid; j < C * GLA_RANK; j += GLA_THREADS) {
                    const int t = j / GLA_RANK, r = r0 + j % GLA_RANK;
                    sA[j] = t < rows && r < a.rank ? proj[(int64_t)t * a.ldp + a.off_a + r] : 0.0f;
                }
            float w[GLA_RANK];
#pragma unroll
            for (int r = 0; r < GLA_RANK; r++) w[r] = mine && r0 + r < a.rank ? to_f32(a2[(int64_t)d * a.rank + r0 + r]) : 0.0f;
            __syncthreads();
#pragma unroll
            for (int t = 0; t < GLA_SUB; t++) {
                const float4 *x = reinterpret_cast<const float4 *>(sA + (sb * GLA_SUB + t) * GLA_RANK);
#pragma unroll
                for (int r = 0; r < GLA_RANK; r += 4) {
                    const float4 v = x[r / 4];
                    z[t] = fmaf(w[r], v.x, fmaf(w[r + 1], v.y, fmaf(w[r + 2], v.z, fmaf(w[r + 3], v.w, z[t]))));
                }
            }
        }
        if (mine) {
#pragma unroll
            for (int t = 0; t < GLA_SUB; t++) sD[(sb * GLA_SUB + t) * DP + d] = sb * GLA_SUB + t < rows ? expf(gla_log_decay(z[t], a.inv_tau)) : 1.0f;
        }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();

    // A inside the 16-token blocks: half a warp per column j, its key carried on token by token, four channels at a time
    float *A = sc.A + ch * C * C;
    for (int pair = warp; pair < C / 2; pair += GLA_THREADS / 32) {
        const int col = 2 * pair + (lane >> 4), l16 = lane & 15, sb = col / GLA_SUB, j = col % GLA_SUB, j0 = j & ~1;
        float acc[GLA_SUB];
#pragma unroll
        for (int i = 0; i < GLA_SUB; i++) acc[i] = 0.0f;
        for (int d = 4 * l16; d < DP - 4; d += 64) {   // what pads a row is a zero query and key
            float4 k = *reinterpret_cast<const float4 *>(sK + col * DP + d);
#pragma unroll
            for (int i = 0; i < GLA_SUB; i++) {
                if (i < j0) continue;
                const int at = (sb * GLA_SUB + i) * DP + d;
                if (i > j0) {
                    float4 w = *reinterpret_cast<const float4 *>(sD + at);
                    if (i == j) w = make_float4(1.0f, 1.0f, 1.0f, 1.0f);   // the pair's second column, at its own token
                    k = make_float4(k.x * w.x, k.y * w.y, k.z * w.z, k.w * w.w);
                }
                const float4 q = *reinterpret_cast<const float4 *>(sQ + at);
                acc[i] = fmaf(q.x, k.x, fmaf(q.y, k.y, fmaf(q.z, k.z, fmaf(q.w, k.w, acc[i]))));
            }
        }
        // 16 sums over 16 lanes: each step halves both, lane i ends with row i
#pragma unroll
        for (int o = GLA_SUB / 2; o > 0; o >>= 1) {
            const bool up = (l16 & o) != 0;
#pragma unroll
            for (int i = 0; i < o; i++) {
                const float keep = up ? acc[i + o] : acc[i], send = up ? acc[i] : acc[i + o];
                acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        // the column: zero above its token, these 16 rows; the rows below come from the other blocks
        for (int i = l16; i < sb * GLA_SUB; i += 16) A[col * C + i] = 0.0f;
        A[col * C + sb * GLA_SUB + l16] = l16 >= j ? acc[0] * a.q_factor : 0.0f;
    }
    __syncthreads();
    // q carries the decay since its block's start, k the decay to its block's end
    for (int i = tid; i < dim * NB; i += GLA_THREADS) {
        const int sb = i / dim, d = i - sb * dim;
        float p = a.q_factor, s = 1.0f, w = 1.0f;
#pragma unroll
        for (int t = 0; t < GLA_SUB; t++) {
            const int at = (sb * GLA_SUB + t) * DP + d, bt = (sb * GLA_SUB + GLA_SUB - 1 - t) * DP + d;
            p *= sD[at];
            w *= sD[at];
            sQ[at] *= p;
            sK[bt] *= s;
            s *= sD[bt];
        }
        sT[sb * DP + d] = w;
    }
    __syncthreads();
    // A between blocks: row block I against the columns before it; then those keys go on over block I
#pragma unroll 1
    for (int I = 1; I < NB; I++) {
        const int i = tid & 15, j = tid >> 4;
        float acc[NB];
#pragma unroll
        for (int J = 0; J < NB; J++) acc[J] = 0.0f;
        const float *q = sQ + (I * GLA_SUB + i) * DP;
        for (int d = 0; d < DP - 4; d += 4) {
            const float4 qv = *reinterpret_cast<const float4 *>(q + d);
#pragma unroll
            for (int J = 0; J < NB - 1; J++) {
                if (J >= I) break;
                const float4 kv = *reinterpret_cast<const float4 *>(sK + (J * GLA_SUB + j) * DP + d);
                acc[J] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, acc[J]))));
            }
        }
#pragma unroll
        for (int J = 0; J < NB; J++)
            if (J < I) A[(J * GLA_SUB + j) * C + I * GLA_SUB + i] = acc[J];
        __syncthreads();
        for (int d = lane * 4; d < DP; d += 128) {
            const float4 w = *reinterpret_cast<const float4 *>(sT + I * DP + d);
            for (int t = warp; t < I * GLA_SUB; t += GLA_THREADS / 32) {
                float4 *k = reinterpret_cast<float4 *>(sK + t * DP + d);
                const float4 v = *k;
                *k = make_float4(v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w);
            }
        }
        __syncthreads();
    }
    // out: keys at the chunk's end, queries at its start (transposed), the chunk's decay
    for (int t = warp; t < C; t += GLA_THREADS / 32)
        for (int d = lane * VEC; d < dim; d += 32 * VEC) {
            float *p = sc.k + ch * C * dim + t * dim + d;
            if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = *reinterpret_cast<const float4 *>(sK + t * DP + d);
            else *p = sK[t * DP + d];
        }
    // (a thread: one channel, every 16th token's block in turn, so that the decay in front of a block is carried along)
    for (int i = tid; i < GLA_SUB * dim; i += GLA_THREADS) {
        const int d = i / GLA_SUB, t = i % GLA_SUB;
        float w = 1.0f;
#pragma unroll
        for (int s = 0; s < NB; s++) {
            sc.q[ch * C * dim + d * C + s * GLA_SUB + t] = sQ[(s * GLA_SUB + t) * DP + d] * w;
            w *= sT[s * DP + d];
        }
    }
    for (int d = tid; d < dim; d += GLA_THREADS) {
        float v = 1.0f;
        for (int s = 0; s < NB; s++) v *= sT[s * DP + d];
        sc.dC[ch * dim + d] = v;
    }
}

// two F32 fused multiply-adds in one instruction
__device__ __forceinline__ float2 gla_fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(*reinterpret_cast<unsigned long long *>(&d)) : "l"(*reinterpret_cast<unsigned long long *>(&a)),
        "l"(*reinterpret_cast<unsigned long long *>(&b)), "l"(*reinterpret_cast<unsigned long long *>(&c)));
    return d;
}

// The two matrix products of a chunk, out[m][v] = sum_k L[k][m] R[k][v] in F32 over 16-deep slabs (double buffered):
//   OUT = false  the chunk's contribution to the state: L = keys [token][channel], R = values; 64 channels per block
//   OUT = true   the chunk's outputs: L = queries [channel][token], R = the state in front of the chunk, then L = A [key][token],
//                R = values; when one block holds a head's values (FUSED) the norm and the gate follow in place
// A warp owns RW rows (of the C of a chunk or of 64 channels), a lane 4 NV columns (128 apart): left operands are broadcasts, right ones contiguous.
template <typename Y, int RW, int NV, bool OUT, bool FUSED, int VEC>
__global__ void __launch_bounds__(GLA_THREADS, 2)
gla_mm_kernel(GlaArgs a, GlaScratch sc, int C) {
    constexpr int KS = 16, TM = RW * (GLA_THREADS / 32), TN = 128 * NV;
    __shared__ __align__(16) float sl[2][KS][TM], sr[2][KS][TN];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, ci = blockIdx.x;
    const int tiles_v = (a.vdim + TN - 1) / TN, v0 = (blockIdx.z % tiles_v) * TN, m0 = (blockIdx.z / tiles_v) * TM;
    pdl_trigger();
    pdl_wait();
    int row0, rows;
    if (!gla_find_chunk(a, C, ci, &row0, &rows)) return;
    const int64_t ch = (int64_t)ci * a.heads + h;
    const float *values = a.proj + (int64_t)row0 * a.ldp + a.off_v + h * a.vdim;
    const int n_state = OUT ? (a.dim + KS - 1) / KS : 0, slabs = n_state + (rows + KS - 1) / KS;
    const auto load = [&](int s) {
        const bool st = s < n_state;
        const int k0 = (st ? s : s - n_state) * KS, kn = st ? a.dim : rows;
        const float *L = st ? sc.q + ch * C * a.dim : OUT ? sc.A + ch * C * C : sc.k + ch * C * a.dim;
        const int ldl = OUT ? C : a.dim, mn = OUT ? C : a.dim;
        const float *R = st ? sc.S + ch * a.dim * a.vdim : values;
        const int64_t ldr = st ? a.vdim : a.ldp;
        constexpr int LV = OUT ? 4 : VEC;
        for (int i = tid; i < KS * (TM / LV); i += GLA_THREADS) {
            const int k = i / (TM / LV), m = (i - k * (TM / LV)) * LV;
            const bool in = k0 + k < kn && m0 + m < mn;
            gla_cp<4 * LV>(&sl[s & 1][k][m], L + (in ? (int64_t)(k0 + k) * ldl + m0 + m : 0), in);
        }
        for (int i = tid; i < KS * (TN / VEC); i += GLA_THREADS) {
            const int k = i / (TN / VEC), c = (i - k * (TN / VEC)) * VEC;
            const bool in = k0 + k < kn && v0 + c < a.vdim;
            gla_cp<4 * VEC>(&sr[s & 1][k][c], R + (in ? (int64_t)(k0 + k) * ldr + v0 + c : 0), in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float2 acc[RW][2 * NV];
#pragma unroll
    for (int r = 0; r < RW; r++)
#pragma unroll
        for (int c = 0; c < 2 * NV; c++) acc[r][c] = make_float2(0.0f, 0.0f);
    load(0);
    for (int s = 0; s < slabs; s++) {
        if (s + 1 < slabs) {
            load(s + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        // A is zero where the key comes after the row
        if (!OUT || s < n_state || (s - n_state) * KS <= warp * RW + RW - 1) {
#pragma unroll
            for (int k = 0; k < KS; k++) {
                float l[RW];
#pragma unroll
                for (int r = 0; r < RW; r++) l[r] = sl[s & 1][k][warp * RW + r];
#pragma unroll
                for (int g = 0; g < NV; g++) {
                    const float4 x = *reinterpret_cast<const float4 *>(&sr[s & 1][k][128 * g + 4 * lane]);
#pragma unroll
                    for (int r = 0; r < RW; r++) {
                        const float2 ll = make_float2(l[r], l[r]);
                        acc[r][2 * g] = gla_fma2(ll, make_float2(x.x, x.y), acc[r][2 * g]);
                        acc[r][2 * g + 1] = gla_fma2(ll, make_float2(x.z, x.w), acc[r][2 * g + 1]);
                    }
                }
            }
        }
        __syncthreads();
    }
    const auto at = [&](int r, int g, int e) { return e < 2 ? (e ? acc[r][2 * g].y : acc[r][2 * g].x) : (e == 3 ? acc[r][2 * g + 1].y : acc[r][2 * g + 1].x); };
#pragma unroll
    for (int r = 0; r < RW; r++) {
        const int m = m0 + warp * RW + r;
        if (m >= (OUT ? rows : a.dim)) continue;
        float *dst = OUT ? sc.o + ((int64_t)(row0 + m) * a.heads + h) * a.vdim : sc.S + (ch * a.dim + m) * a.vdim;
        float scale = 1.0f;
        if constexpr (FUSED) {
            float sq = 0.0f;   // columns past the head's values hold zero
#pragma unroll
            for (int g = 0; g < NV; g++)
#pragma unroll
                for (int e = 0; e < 4; e++) sq = fmaf(at(r, g, e), at(r, g, e), sq);
            scale = 1.0f / sqrtf(warp_sum(sq) / (float)a.vdim + a.eps);
        }
#pragma unroll
        for (int g = 0; g < NV; g++) {
            const int c = v0 + 128 * g + 4 * lane;
            if constexpr (FUSED) {
                Y *y = (Y *)a.y + (int64_t)(row0 + m) * a.ldy + h * a.vdim;
                const float *gate = a.proj + (int64_t)(row0 + m) * a.ldp + a.off_g + h * a.vdim;
                if constexpr (VEC == 4) {
                    if (c >= a.vdim) continue;
                    const float4 gv = *reinterpret_cast<const float4 *>(gate + c), w = *reinterpret_cast<const float4 *>(a.norm_w + c);
                    const float4 o = make_float4(at(r, g, 0) * scale * w.x * silu_f32(gv.x), at(r, g, 1) * scale * w.y * silu_f32(gv.y),
                                                 at(r, g, 2) * scale * w.z * silu_f32(gv.z), at(r, g, 3) * scale * w.w * silu_f32(gv.w));
                    if constexpr (sizeof(Y) == 4) *reinterpret_cast<float4 *>(y + c) = o;
                    else *reinterpret_cast<uint2 *>(y + c) = make_uint2(bf16_pack(o.x, o.y), bf16_pack(o.z, o.w));
                } else {
#pragma unroll
                    for (int e = 0; e < 4; e++)
                        if (c + e < a.vdim) y[c + e] = from_f32<Y>(at(r, g, e) * scale * a.norm_w[c + e] * silu_f32(gate[c + e]));
                }
            } else if constexpr (VEC == 4) {
                if (c < a.vdim) *reinterpret_cast<float4 *>(dst + c) = make_float4(at(r, g, 0), at(r, g, 1), at(r, g, 2), at(r, g, 3));
            } else {
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (c + e < a.vdim) dst[c + e] = at(r, g, e);
            }
        }
    }
}

// VEC neighbouring state elements per thread, over the chunks of a segment
template <int VEC>
__global__ void __launch_bounds__(GLA_THREADS)
gla_scan_kernel(GlaArgs a, GlaScratch sc, int C) {
    constexpr int U = 8;
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, sidx = blockIdx.z;
    const int64_t per = (int64_t)a.dim * a.vdim, i = ((int64_t)blockIdx.x * GLA_THREADS + threadIdx.x) * VEC;
    if (i >= per) return;
    int first = 0;
    for (int s = 0; s < sidx; s++) first += (a.seg[s * SEG_FIELDS + SEG_ROWS] + C - 1) / C;
    const int32_t *sg = a.seg + sidx * SEG_FIELDS;
    const int chunks = (sg[SEG_ROWS] + C - 1) / C, d = (int)(i / a.vdim);
    if (!gla_segment_ok(a, sg) || first + chunks > sc.chunks) {
        if (i == 0) atomicExch(a.err, ERR_SEGMENT);
        return;
    }
    float *state = a.state + ((int64_t)sg[SEG_SLOT] * a.heads + h) * per + i;
    const auto ld = [](const float *p, float (&f)[VEC]) {
        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(f) = *reinterpret_cast<const float4 *>(p);
        else f[0] = *p;
    };
    const auto st = [](float *p, const float (&f)[VEC]) {
        if constexpr (VEC == 4) *reinterpret_cast<float4 *>(p) = *reinterpret_cast<const float4 *>(f);
        else *p = f[0];
    };
    float s[VEC];
    ld(state, s);
    if (sg[SEG_FRESH])
#pragma unroll
        for (int e = 0; e < VEC; e++) s[e] = 0.0f;
    float *p = sc.S + ((int64_t)first * a.heads + h) * per + i;
    const float *dc = sc.dC + ((int64_t)first * a.heads + h) * a.dim + d;
    const int64_t pstep = (int64_t)a.heads * per, dstep = (int64_t)a.heads * a.dim;
    for (int c = 0; c < chunks; c += U, p += U * pstep, dc += U * dstep) {
        float x[U][VEC], g[U];
#pragma unroll
        for (int u = 0; u < U; u++)
            if (c + u < chunks) {
                ld(p + u * pstep, x[u]);
                g[u] = dc[u * dstep];
            }
#pragma unroll
        for (int u = 0; u < U; u++)
            if (c + u < chunks) {
                st(p + u * pstep, s);
#pragma unroll
                for (int e = 0; e < VEC; e++) s[e] = fmaf(g[u], s[e], x[u][e]);
            }
    }
    st(state, s);
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

template <int C, int VEC, typename Y>
int launch_out(const GlaArgs &a, const GlaScratch &sc, unsigned chunks, cudaStream_t s) {
    constexpr int RW = C / (GLA_THREADS / 32);
    const dim3 b(GLA_THREADS);
    if (a.vdim <= 128) return launch_pdl(gla_mm_kernel<Y, RW, 1, true, true, VEC>, dim3(chunks, (unsigned)a.heads, 1), b, 0, s, a, sc, C);
    if (a.vdim <= 256) return launch_pdl(gla_mm_kernel<Y, RW, 2, true, true, VEC>, dim3(chunks, (unsigned)a.heads, 1), b, 0, s, a, sc, C);
    int rc = launch_pdl(gla_mm_kernel<float, RW, 2, true, false, VEC>, dim3(chunks, (unsigned)a.heads, (unsigned)((a.vdim + 255) / 256)), b, 0, s, a, sc, C);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl(gla_gate_kernel<Y>, dim3((unsigned)((a.n * a.heads + GLA_THREADS / 32 - 1) / (GLA_THREADS / 32))), b, 0, s, a, (const float *)sc.o);
}

template <typename W, int C, int VEC>
int launch_chunks(const GlaArgs &a, cudaStream_t s) {
    GlaScratch sc;
    const unsigned chunks = (unsigned)((a.n + C - 1) / C + a.n_seg);
    const size_t nh = (size_t)chunks * a.heads;
    sc.chunks = (int)chunks;
    sc.q = a.scratch;
    sc.k = sc.q + round4(nh * C * a.dim);
    sc.A = sc.k + round4(nh * C * a.dim);
    sc.dC = sc.A + round4(nh * C * C);
    sc.S = sc.dC + round4(nh * a.dim);
    sc.o = sc.S + round4(nh * a.dim * a.vdim);
    const int DP = (a.dim + 3) / 4 * 4 + 4;
    const size_t smem = ((size_t)(3 * C + C / GLA_SUB) * DP + (size_t)C * GLA_RANK) * 4;
    B200_REQUIRE(a.heads <= 65535 && a.n_seg <= 65535, "gla: too many heads or sequences");
    if (smem > 48 * 1024) B200_CUDA(cudaFuncSetAttribute(gla_chunk_kernel<W, C, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const dim3 b(GLA_THREADS);
    const unsigned H = (unsigned)a.heads;
    int rc = launch_pdl(gla_chunk_kernel<W, C, VEC>, dim3(chunks, H), b, smem, s, a, sc);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const unsigned md = (unsigned)((a.dim + 63) / 64);
    rc = a.vdim <= 128 ? launch_pdl(gla_mm_kernel<float, 8, 1, false, false, VEC>, dim3(chunks, H, md), b, 0, s, a, sc, C)
                       : launch_pdl(gla_mm_kernel<float, 8, 2, false, false, VEC>, dim3(chunks, H, md * (unsigned)((a.vdim + 255) / 256)), b, 0, s, a, sc, C);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const int64_t per = (int64_t)a.dim * a.vdim / VEC;
    rc = launch_pdl(gla_scan_kernel<VEC>, dim3((unsigned)((per + GLA_THREADS - 1) / GLA_THREADS), H, (unsigned)a.n_seg), b, 0, s, a, sc, C);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return a.y_type == B200_TYPE_F32 ? launch_out<C, VEC, float>(a, sc, chunks, s) : launch_out<C, VEC, __nv_bfloat16>(a, sc, chunks, s);
}

// rows the vector forms can read and write in pieces of four
bool gla_rows_of_four(const GlaArgs &a) {
    const int64_t all = a.dim | a.vdim | a.ldp | a.ldy | a.off_q | a.off_k | a.off_v | a.off_g;
    return all % 4 == 0 && (((uintptr_t)a.proj | (uintptr_t)a.y | (uintptr_t)a.state | (uintptr_t)a.norm_w | (uintptr_t)a.scratch) & 15) == 0;
}

template <typename W>
int launch_typed(const GlaArgs &a, cudaStream_t s) {
    const int C = gla_chunk_rows(a.dim);
    const bool four = gla_rows_of_four(a);
    if (a.scratch && C == 64) return four ? launch_chunks<W, 64, 4>(a, s) : launch_chunks<W, 64, 1>(a, s);
    if (a.scratch && C == 32) return four ? launch_chunks<W, 32, 4>(a, s) : launch_chunks<W, 32, 1>(a, s);
    if (a.scratch && C == 16) return four ? launch_chunks<W, 16, 4>(a, s) : launch_chunks<W, 16, 1>(a, s);
    const bool vec = a.vdim % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    if (a.y_type == B200_TYPE_F32) return vec ? launch_step<W, float, 4>(a, s) : launch_step<W, float, 1>(a, s);
    return vec ? launch_step<W, __nv_bfloat16, 4>(a, s) : launch_step<W, __nv_bfloat16, 1>(a, s);
}

}  // namespace

size_t gla_scratch_floats(int64_t heads, int64_t dim, int64_t vdim, int64_t n, int64_t n_seg) {
    const int64_t C = gla_chunk_rows(dim);
    if (C == 0) return 4;
    const size_t nh = (size_t)((n + C - 1) / C + n_seg) * heads;
    return 2 * round4(nh * C * dim) + round4(nh * C * C) + round4(nh * dim) + round4(nh * dim * vdim) + (vdim > 256 ? (size_t)n * heads * vdim : 0);
}

int launch_gla(const GlaArgs &args, cudaStream_t s) {
    GlaArgs a = args;
    int rc = device_error_word(&a.err);
    if (rc != B200_STATUS_SUCCESS) return rc;
    B200_REQUIRE(a.proj && a.a2 && a.a2_bias && a.norm_w && a.state && a.seg && a.y, "gla: null operand");
    B200_REQUIRE(a.heads > 0 && a.dim > 0 && a.vdim > 0 && a.rank > 0 && a.n_seg > 0, "gla: bad shape");
    return a.a2_type == B200_TYPE_F32 ? launch_typed<float>(a, s) : launch_typed<__nv_bfloat16>(a, s);
}

}  // namespace b200
