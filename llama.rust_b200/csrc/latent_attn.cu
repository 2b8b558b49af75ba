// Latent attention: keys and values of all heads come from one cached vector per token, the normed latent c (rank numbers) and a
// rotated key part shared by the heads (rot numbers).  Per head the unrotated key is Uk c, the value Uv c; the score is (q . k) *
// factor over both parts, the softmax has a learned sink in its denominator (exp(sink): no key, no value, not scaled), keys are
// limited to a window of positions, and each head's output is multiplied by sigmoid of a gate.
//
// Cells of a sequence's positions are listed in `tab` (segment field TAB0: its first entry, KEY0: that entry's position).
// Few rows per sequence: Uk moves to the query's side, so that attention reads the cached rows themselves, once for all heads:
//   latent_query_kernel    queries through Uk and rotated; the rows' own latents normed, rotated and stored (one more block per row)
//   latent_decode_kernel   per (split of keys, 8 heads, row): running softmax over 32-key tiles in shared memory, F32 arithmetic
//   latent_value_kernel    splits and sink merged, Uv, gate
// Many rows: keys and values expanded for every listed cell by one mat-mul, then
//   latent_attn_mma_kernel  64 rows x 64-key tiles on mma.sync (BF16 operands, F32 scores and sums; a weight goes in as two BF16
//                           parts, so that it keeps its 32-bit value to 2^-17), or
//   latent_attn_kernel      a warp per (row, head), F32 arithmetic, any type and size
#include "attn_tile.cuh"

namespace b200 {

namespace {

constexpr int LT = 256;             // threads per block
constexpr int LK = 32, LH = 8;      // keys per tile, heads (one per warp) per block of the few-rows kernel
constexpr int LRB = 512;            // latent elements a block of it accumulates
constexpr int LV_ROWS = 32;         // value rows per block of the merge

// element j of a rotated part at x, by the position's row of (cos, sin) pairs
__device__ __forceinline__ float rotated(const float *x, const float *rope, int rot_dims, int j) {
    if (j >= rot_dims) return x[j];
    const float c = rope[j & ~1], s = rope[j | 1];
    return (j & 1) ? fmaf(x[j], c, x[j - 1] * s) : fmaf(x[j], c, -(x[j + 1] * s));
}
__device__ __forceinline__ const float *rope_row(const LatentArgs &a, int pos, int *err) {
    if (a.rot_dims > 0 && (pos < 0 || pos >= a.rope_rows)) {
        if (threadIdx.x == 0) atomicExch(err, ERR_POS);
        return nullptr;
    }
    return a.rot_dims > 0 ? a.rope + (int64_t)pos * a.rot_dims : a.proj;   // (nothing is read when nothing rotates)
}

template <typename T>
__device__ __forceinline__ void store_row(const LatentArgs &a, int64_t row, float *part, int *err) {
    const float *x = a.proj + row * a.ldp + a.off_c;
    const int64_t cell = a.cells[row];
    const float *rope = rope_row(a, a.pos[row], err);
    if (cell < 0 || cell >= a.n_cells || !rope) {
        if (threadIdx.x == 0 && rope) atomicExch(err, ERR_CELL);
        return;
    }
    float sq = 0.0f;
    for (int r = threadIdx.x; r < a.rank; r += LT) sq = fmaf(x[r], x[r], sq);
    const float scale = 1.0f / sqrtf(block_sum(sq, part) / (float)a.rank + a.eps);
    T *c = (T *)a.cache + cell * a.ldc;
    for (int r = threadIdx.x; r < a.rank; r += LT) c[r] = from_f32<T>(x[r] * scale * a.norm_w[r]);
    for (int j = threadIdx.x; j < a.rot; j += LT) c[a.rank + j] = from_f32<T>(rotated(x + a.rank, rope, a.rot_dims, j));
}

template <typename T>
__global__ void __launch_bounds__(LT)
latent_store_kernel(LatentArgs a, int *err) {
    __shared__ float part[32];
    pdl_trigger();
    pdl_wait();
    store_row<T>(a, blockIdx.x, part, err);
}

// VEC elements of a weight row (16 bytes) or one
template <typename T, int VEC>
__device__ __forceinline__ void load_piece(const T *p, float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        f[0] = to_f32(*p);
    } else {
        const uint4 q = ld_stream16(p);
        if constexpr (sizeof(T) == 2) {
            f[0] = bf16_lo(q.x); f[1] = bf16_hi(q.x); f[2] = bf16_lo(q.y); f[3] = bf16_hi(q.y);
            f[4] = bf16_lo(q.z); f[5] = bf16_hi(q.z); f[6] = bf16_lo(q.w); f[7] = bf16_hi(q.w);
        } else {
            f[0] = __uint_as_float(q.x); f[1] = __uint_as_float(q.y); f[2] = __uint_as_float(q.z); f[3] = __uint_as_float(q.w);
        }
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(LT)
latent_query_kernel(LatentArgs a, int lanes, int *err) {
    extern __shared__ float l_sm[];
    __shared__ float part[32];
    const int tid = threadIdx.x, h = blockIdx.x;
    const int64_t row = blockIdx.y;
    pdl_trigger();
    if (h < a.heads) {
        // this block's columns of the head's key rows
        const int r0 = blockIdx.z * lanes * VEC, lines = (min(lanes * VEC, a.rank - r0) * (int)sizeof(T) + 127) / 128;
        const T *uk = (const T *)a.ukv + (int64_t)h * a.dim * a.rank + r0;
        for (int i = tid; i < a.dim * lines; i += LT) l2_prefetch((const char *)(uk + (int64_t)(i / lines) * a.rank) + 128 * (i % lines));
    }
    pdl_wait();
    if (h == a.heads) {
        if (blockIdx.z == 0) store_row<T>(a, row, part, err);
        return;
    }
    const float *q = a.proj + row * a.ldp + a.off_q + h * (a.dim + a.rot);
    float *out = a.queries + (row * a.heads + h) * (a.rank + a.rot);
    const float *rope = rope_row(a, a.pos[row], err);
    if (!rope) return;
    float *sq = l_sm, *red = sq + (a.dim + 3) / 4 * 4;   // red [groups][lanes * VEC]
    for (int d = tid; d < a.dim; d += LT) sq[d] = q[d];
    __syncthreads();
    const int groups = LT / lanes, g = tid / lanes, l = tid % lanes;
    const T *uk = (const T *)a.ukv + (int64_t)h * a.dim * a.rank;
    {
        const int r0 = blockIdx.z * lanes * VEC, r = r0 + l * VEC;
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[e] = 0.0f;
        if (r < a.rank) {
#pragma unroll 8
            for (int d = g; d < a.dim; d += groups) {
                float f[VEC];
                load_piece<T, VEC>(uk + (int64_t)d * a.rank + r, f);
                const float s = sq[d];
#pragma unroll
                for (int e = 0; e < VEC; e++) acc[e] = fmaf(s, f[e], acc[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; e++) red[(g * lanes + l) * VEC + e] = acc[e];
        __syncthreads();
        for (int i = tid; i < lanes * VEC && r0 + i < a.rank; i += LT) {
            float v = 0.0f;
            for (int k = 0; k < groups; k++) v += red[k * lanes * VEC + i];
            out[r0 + i] = v;
        }
    }
    if (blockIdx.z == 0)
        for (int j = tid; j < a.rot; j += LT) out[a.rank + j] = rotated(q + a.dim, rope, a.rot_dims, j);
}

// the keys a row sees: positions [lo, hi]
__device__ __forceinline__ int first_key(const LatentArgs &a, int pos) { return a.window > 0 ? max(0, pos - a.window + 1) : 0; }

template <typename T>
__global__ void __launch_bounds__(LT)
latent_decode_kernel(LatentArgs a, int head_groups, int *err) {
    constexpr int PE = 16 / (int)sizeof(T);   // elements of a piece
    extern __shared__ __align__(16) uint8_t l_raw[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int D = a.rank + a.rot, pieces = (D + PE - 1) / PE, qs = pieces * PE, units = key_units<T>(D);
    T *sk = (T *)l_raw;                                              // [LK][units] pieces
    float *sq = (float *)(l_raw + (size_t)LK * units * 16);          // [LH][qs]
    float *sp = sq + LH * qs;                                        // [LK][LH] weights
    float *scorr = sp + LK * LH;                                     // [LH] what this tile's maximum makes of the sums so far
    const int split = blockIdx.x, h0 = (blockIdx.y % head_groups) * LH, rb0 = (blockIdx.y / head_groups) * LRB;
    const int64_t row = blockIdx.z;
    const int nh = min(LH, a.heads - h0);
    pdl_trigger();
    pdl_wait();
    const int pos = a.pos[row];
    const int lo = first_key(a, pos) + split * a.per_split, hi = min(lo + a.per_split, pos + 1);
    if (lo >= hi) return;
    const int si = a.row_seg[row];
    if (si < 0 || si >= a.n_seg) {
        if (tid == 0) atomicExch(err, ERR_SEGMENT);
        return;
    }
    const int32_t *sg = a.seg + (int64_t)si * SEG_FIELDS;
    const int tab0 = sg[SEG_TAB0] - sg[SEG_KEY0];
    for (int i = tid; i < LH * qs; i += LT) {
        const int h = i / qs, d = i - h * qs;
        sq[i] = h < nh && d < D ? a.queries[(row * a.heads + h0 + h) * D + d] : 0.0f;
    }
    float acc[LH][2], m = -INFINITY, l = 0.0f;   // m, l: of the warp's head
#pragma unroll
    for (int h = 0; h < LH; h++) acc[h][0] = acc[h][1] = 0.0f;
    const int r = rb0 + 2 * tid;
    for (int k0 = lo; k0 < hi; k0 += LK) {
        const int kn = min(LK, hi - k0);
        __syncthreads();
        // rows of cells, a warp four at a time: 16-byte pieces (a cell's row is padded to whole ones)
        for (int k = warp; k < LK; k += LT / 32) {
            const int64_t at = (int64_t)tab0 + k0 + k;
            const int64_t cell = k < kn && at >= 0 && at < a.n_tab ? a.tab[at] : -1;
            const bool in = cell >= 0 && cell < a.n_cells;
            if (k < kn && !in && lane == 0) atomicExch(err, ERR_CELL);
            const T *src = (const T *)a.cache + (in ? cell * a.ldc : 0);
            for (int p = lane; p < pieces; p += 32) cp16(sk + ((size_t)k * units + p) * PE, src + p * PE, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // scores: lane = key, warp = head
        {
            const T *kr = sk + (size_t)lane * units * PE;
            const float *qa = sq + warp * qs;
            float s4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 4
            for (int p = 0; p < pieces; p++) {
                const uint4 w = *reinterpret_cast<const uint4 *>(kr + p * PE);
                float f[PE];
                if constexpr (sizeof(T) == 2) {
                    f[0] = bf16_lo(w.x); f[1] = bf16_hi(w.x); f[2] = bf16_lo(w.y); f[3] = bf16_hi(w.y);
                    f[4] = bf16_lo(w.z); f[5] = bf16_hi(w.z); f[6] = bf16_lo(w.w); f[7] = bf16_hi(w.w);
                } else {
                    f[0] = __uint_as_float(w.x); f[1] = __uint_as_float(w.y); f[2] = __uint_as_float(w.z); f[3] = __uint_as_float(w.w);
                }
#pragma unroll
                for (int e = 0; e < PE; e += 4) {
                    const float4 x = *reinterpret_cast<const float4 *>(qa + p * PE + e);
                    s4[0] = fmaf(x.x, f[e], s4[0]);
                    s4[1] = fmaf(x.y, f[e + 1], s4[1]);
                    s4[2] = fmaf(x.z, f[e + 2], s4[2]);
                    s4[3] = fmaf(x.w, f[e + 3], s4[3]);
                }
            }
            const float s = lane < kn ? ((s4[0] + s4[1]) + (s4[2] + s4[3])) * a.scale : -INFINITY;
            const float mn = fmaxf(m, warp_max(s)), corr = m == -INFINITY ? 0.0f : expf(m - mn), p = lane < kn ? expf(s - mn) : 0.0f;
            l = l * corr + warp_sum(p);
            m = mn;
            sp[lane * LH + warp] = p;
            if (lane == 0) scorr[warp] = corr;
        }
        __syncthreads();
        if (r < a.rank) {
#pragma unroll
            for (int h = 0; h < LH; h++) {
                const float c = scorr[h];
                acc[h][0] *= c;
                acc[h][1] *= c;
            }
            const T *kc = sk + r;
#pragma unroll 4
            for (int k = 0; k < kn; k++) {
                float x, y;
                if constexpr (sizeof(T) == 2) {
                    const uint32_t w = *reinterpret_cast<const uint32_t *>(kc + (size_t)k * units * PE);
                    x = bf16_lo(w);
                    y = bf16_hi(w);
                } else {
                    const float2 w = *reinterpret_cast<const float2 *>(kc + (size_t)k * units * PE);
                    x = w.x;
                    y = w.y;
                }
#pragma unroll
                for (int h = 0; h < LH; h += 4) {
                    const float4 p = *reinterpret_cast<const float4 *>(sp + k * LH + h);
                    acc[h][0] = fmaf(p.x, x, acc[h][0]);         acc[h][1] = fmaf(p.x, y, acc[h][1]);
                    acc[h + 1][0] = fmaf(p.y, x, acc[h + 1][0]); acc[h + 1][1] = fmaf(p.y, y, acc[h + 1][1]);
                    acc[h + 2][0] = fmaf(p.z, x, acc[h + 2][0]); acc[h + 2][1] = fmaf(p.z, y, acc[h + 2][1]);
                    acc[h + 3][0] = fmaf(p.w, x, acc[h + 3][0]); acc[h + 3][1] = fmaf(p.w, y, acc[h + 3][1]);
                }
            }
        }
    }
    float *out = a.partial + ((row * a.n_splits + split) * a.heads + h0) * (int64_t)(a.rank + 2);
#pragma unroll
    for (int h = 0; h < LH; h++) {
        if (h >= nh) break;
        if (r < a.rank) out[(int64_t)h * (a.rank + 2) + r] = acc[h][0];
        if (r + 1 < a.rank) out[(int64_t)h * (a.rank + 2) + r + 1] = acc[h][1];
    }
    if (rb0 == 0 && lane == 0 && warp < nh) {
        out[(int64_t)warp * (a.rank + 2) + a.rank] = m;
        out[(int64_t)warp * (a.rank + 2) + a.rank + 1] = l;
    }
}

template <typename T, typename Y, int VEC>
__global__ void __launch_bounds__(LT)
latent_value_kernel(LatentArgs a) {
    extern __shared__ float l_sm[];   // [rank], then [n_splits]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x;
    const int64_t row = blockIdx.y;
    const T *uv = (const T *)a.ukv + ((int64_t)a.heads * a.dim + (int64_t)h * a.vdim) * a.rank;
    pdl_trigger();
    {
        const int e0 = blockIdx.z * LV_ROWS, en = min(a.vdim, e0 + LV_ROWS);
        const char *w0 = (const char *)(uv + (int64_t)e0 * a.rank), *w1 = (const char *)(uv + (int64_t)en * a.rank);
        for (const char *w = w0 + 128 * tid; w < w1; w += 128 * LT) l2_prefetch(w);
    }
    pdl_wait();
    const int pos = a.pos[row], keys = pos + 1 - first_key(a, pos);
    const int splits = min(a.n_splits, (keys + a.per_split - 1) / a.per_split);
    const int64_t step = (int64_t)a.heads * (a.rank + 2);
    const float *p = a.partial + (row * a.n_splits * a.heads + h) * (int64_t)(a.rank + 2);
    float *sw = l_sm + (a.rank + 3) / 4 * 4;   // [splits] what each split counts
    if (warp == 0) {
        float m = a.sink[h];
        for (int s = lane; s < splits; s += 32) m = fmaxf(m, p[s * step + a.rank]);
        m = warp_max(m);
        float l = 0.0f;
        for (int s = lane; s < splits; s += 32) {
            const float w = expf(p[s * step + a.rank] - m);
            sw[s] = w;
            l = fmaf(p[s * step + a.rank + 1], w, l);
        }
        l = 1.0f / (warp_sum(l) + expf(a.sink[h] - m));
        for (int s = lane; s < splits; s += 32) sw[s] *= l;
    }
    __syncthreads();
    for (int r = tid; r < a.rank; r += LT) {
        float v = 0.0f;
#pragma unroll 8
        for (int s = 0; s < splits; s++) v = fmaf(p[s * step + r], sw[s], v);
        l_sm[r] = v;
    }
    __syncthreads();
    const float gate = sigmoid_f32(a.proj[row * a.ldp + a.off_g + h]);
    for (int e = blockIdx.z * LV_ROWS + warp; e < min(a.vdim, (int)(blockIdx.z + 1) * LV_ROWS); e += LT / 32) {
        const T *w = uv + (int64_t)e * a.rank;
        float acc = 0.0f;
#pragma unroll 4
        for (int r = lane * VEC; r < a.rank; r += 32 * VEC) {
            float f[VEC];
            load_piece<T, VEC>(w + r, f);
#pragma unroll
            for (int i = 0; i < VEC; i++) acc = fmaf(f[i], l_sm[r + i], acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) ((Y *)a.y)[row * a.ldy + h * a.vdim + e] = from_f32<Y>(acc * gate);
    }
}

// ---- many rows ---------------------------------------------------------------------------------------------
template <typename T, typename Y>
__global__ void __launch_bounds__(LT)
latent_attn_kernel(LatentArgs a, int *err) {
    extern __shared__ float l_sm[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.y, D = a.dim + a.rot;
    float *q = l_sm + warp * (D + a.vdim), *o = q + D;
    pdl_trigger();
    pdl_wait();
    int r0, rows;
    const int32_t *sg = find_tile(a.seg, a.n_seg, a.n, LT / 32, blockIdx.x, &r0, &rows, err);
    if (!sg || warp >= rows) return;
    const int64_t row = sg[SEG_ROW0] + r0 + warp;
    const int pos = sg[SEG_POS0] + r0 + warp, lo = first_key(a, pos);
    if (a.rot_dims > 0 && pos >= a.rope_rows) {
        if (lane == 0) atomicExch(err, ERR_POS);
        return;
    }
    const float *x = a.proj + row * a.ldp + a.off_q + h * D, *rope = a.rope + (int64_t)pos * a.rot_dims;
    for (int d = lane; d < a.dim; d += 32) q[d] = x[d];
    for (int j = lane; j < a.rot; j += 32) q[a.dim + j] = rotated(x + a.dim, rope, a.rot_dims, j);
    for (int c = lane; c < a.vdim; c += 32) o[c] = 0.0f;
    __syncwarp();
    float m = -INFINITY, l = 0.0f;
    const int64_t base = (int64_t)sg[SEG_TAB0] - sg[SEG_KEY0];
    if (base + lo < 0 || base + pos >= a.n_tab) {
        if (lane == 0) atomicExch(err, ERR_CELL);
        return;
    }
    for (int k0 = lo; k0 <= pos; k0 += 32) {
        const int k = k0 + lane;
        float s = -INFINITY;
        if (k <= pos) {
            const T *kn = (const T *)a.kv + (base + k) * a.ldkv + h * a.dim, *kr = (const T *)a.cache + (base + k) * a.ldc + a.rank;
            s = 0.0f;
            for (int d = 0; d < a.dim; d++) s = fmaf(q[d], to_f32(kn[d]), s);
            for (int j = 0; j < a.rot; j++) s = fmaf(q[a.dim + j], to_f32(kr[j]), s);
            s *= a.scale;
        }
        const float mn = fmaxf(m, warp_max(s)), corr = m == -INFINITY ? 0.0f : expf(m - mn), p = k <= pos ? expf(s - mn) : 0.0f;
        l = l * corr + warp_sum(p);
        m = mn;
        const int kn = min(32, pos + 1 - k0);
        for (int c0 = 0; c0 < a.vdim; c0 += 32) {
            const int c = c0 + lane;
            float v = c < a.vdim ? o[c] * corr : 0.0f;
            for (int i = 0; i < kn; i++) {
                const float w = __shfl_sync(0xffffffffu, p, i);
                if (c < a.vdim) v = fmaf(w, to_f32(((const T *)a.kv)[(base + k0 + i) * a.ldkv + a.heads * a.dim + h * a.vdim + c]), v);
            }
            if (c < a.vdim) o[c] = v;
        }
    }
    const float mf = fmaxf(m, a.sink[h]), w = expf(m - mf), den = l * w + expf(a.sink[h] - mf);
    const float f = w / den * sigmoid_f32(a.proj[row * a.ldp + a.off_g + h]);
    for (int c = lane; c < a.vdim; c += 32) ((Y *)a.y)[row * a.ldy + h * a.vdim + c] = from_f32<Y>(o[c] * f);
}

// tensor-core form: 4 warps x 16 rows, DK = dim + rot and DV = vdim padded
constexpr int MT = 128, MQ = 64, MK = 64;

// One buffer each for keys and values: the next keys land while the weights meet the values, the next values while the queries meet
// the keys; three blocks per SM cover each other's waits.
template <typename Y, int DK, int DV, bool ALIGNED>
__global__ void __launch_bounds__(MT, DK <= 192 ? 3 : 2)
latent_attn_mma_kernel(LatentArgs a, int *err) {
    typedef __nv_bfloat16 bf;
    constexpr int KS = DK + 8, VS = DV + 8;   // row strides: an odd number of 16-byte units
    extern __shared__ __align__(16) uint8_t l_raw[];
    bf *sQ = (bf *)l_raw, *sK = sQ + MQ * KS, *sV = sK + MK * KS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, D = a.dim + a.rot;
    pdl_trigger();
    pdl_wait();
    int r0, rows;
    // later tiles of a prompt see more keys: they go first
    const int32_t *sg = find_tile(a.seg, a.n_seg, a.n, MQ, gridDim.x - 1 - blockIdx.x, &r0, &rows, err);
    if (!sg) return;
    const int64_t row0 = sg[SEG_ROW0] + r0;
    const int pos0 = sg[SEG_POS0] + r0, last = pos0 + rows - 1;
    const int lo = first_key(a, pos0);
    const int64_t base = (int64_t)sg[SEG_TAB0] - sg[SEG_KEY0];
    if ((a.rot_dims > 0 && last >= a.rope_rows) || base + lo < 0 || base + last >= a.n_tab) {
        if (tid == 0) atomicExch(err, a.rot_dims > 0 && last >= a.rope_rows ? ERR_POS : ERR_CELL);
        return;
    }
    const int tiles = (last - lo) / MK + 1;
    const bf *kn = (const bf *)a.kv + (base + lo) * a.ldkv + h * a.dim, *kr = (const bf *)a.cache + (base + lo) * a.ldc + a.rank;
    const bf *vp = (const bf *)a.kv + (base + lo) * a.ldkv + a.heads * a.dim + h * a.vdim;
    const int ldkv = (int)a.ldkv, ldc = (int)a.ldc;
    // key j of the sequence stands at lo + j; rows past the last key and channels past the head's are zero
    const auto load_keys = [&](int t) {
        const int j0 = t * MK, jn = last - lo - j0;   // keys 0 .. jn of the tile exist
        if (t < tiles) {
            if constexpr (ALIGNED) {
                constexpr int KP = DK / 8;
                const int np = a.dim / 8, dp = D / 8;
                for (int i = tid; i < MK * KP; i += MT) {
                    const int j = i / KP, p = i - j * KP;
                    const bool in = j <= jn && p < dp;
                    const int at = in ? j0 + j : 0, q = in ? p : 0;
                    cp16(sK + j * KS + p * 8, q < np ? kn + (int64_t)at * ldkv + q * 8 : kr + (int64_t)at * ldc + (q - np) * 8, in);
                }
            } else {
                for (int i = tid; i < MK * DK; i += MT) {
                    const int j = i / DK, d = i - j * DK;
                    bf x = __float2bfloat16_rn(0.0f);
                    if (j <= jn && d < D) x = d < a.dim ? kn[(int64_t)(j0 + j) * ldkv + d] : kr[(int64_t)(j0 + j) * ldc + d - a.dim];
                    sK[j * KS + d] = x;
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const auto load_values = [&](int t) {
        const int j0 = t * MK, jn = last - lo - j0;
        if (t < tiles) {
            if constexpr (ALIGNED) {
                constexpr int VP = DV / 8;
                const int np = a.vdim / 8;
                for (int i = tid; i < MK * VP; i += MT) {
                    const int j = i / VP, p = i - j * VP;
                    const bool in = j <= jn && p < np;
                    cp16(sV + j * VS + p * 8, vp + (in ? (int64_t)(j0 + j) * ldkv + p * 8 : 0), in);
                }
            } else {
                for (int i = tid; i < MK * DV; i += MT) {
                    const int j = i / DV, c = i - j * DV;
                    sV[j * VS + c] = j <= jn && c < a.vdim ? vp[(int64_t)(j0 + j) * ldkv + c] : __float2bfloat16_rn(0.0f);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_keys(0);
    load_values(0);
    if constexpr (ALIGNED) {
        // four channels at a time (two pairs of a rotated part), several pieces in flight
        constexpr int QP = DK / 4;
#pragma unroll 4
        for (int i = tid; i < MQ * QP; i += MT) {
            const int t = i / QP, d = (i - t * QP) * 4;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (t < rows && d < D) {
                x = *reinterpret_cast<const float4 *>(a.proj + (row0 + t) * a.ldp + a.off_q + h * D + d);
                const int j = d - a.dim;
                if (j >= 0 && j < a.rot_dims) {
                    const float4 w = *reinterpret_cast<const float4 *>(a.rope + (int64_t)(pos0 + t) * a.rot_dims + j);   // cos, sin, cos, sin
                    x = make_float4(fmaf(x.x, w.x, -(x.y * w.y)), fmaf(x.y, w.x, x.x * w.y), fmaf(x.z, w.z, -(x.w * w.w)), fmaf(x.w, w.z, x.z * w.w));
                }
            }
            *reinterpret_cast<uint2 *>(sQ + t * KS + d) = make_uint2(bf16_pack(x.x, x.y), bf16_pack(x.z, x.w));
        }
    } else {
        for (int i = tid; i < MQ * DK; i += MT) {
            const int t = i / DK, d = i - t * DK;
            float x = 0.0f;
            if (t < rows && d < D) {
                const float *q = a.proj + (row0 + t) * a.ldp + a.off_q + h * D;
                x = d < a.dim ? q[d] : rotated(q + a.dim, a.rope + (int64_t)(pos0 + t) * a.rot_dims, a.rot_dims, d - a.dim);
            }
            sQ[t * KS + d] = __float2bfloat16_rn(x);
        }
    }
    // this lane's two rows of the warp's 16
    const int ra = warp * 16 + (lane >> 2), rb = ra + 8, pa = pos0 + ra, pb = pos0 + rb;
    float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = a.scale * 1.4426950408889634f;   // powers of two
    const int window = a.window > 0 ? a.window : 0x7fffffff;
    const bf *qp = sQ + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8;
    const bf *kp = sK + ((lane >> 4) * 8 + (lane & 7)) * KS + ((lane >> 3) & 1) * 8;
    const bf *vq = sV + (((lane >> 3) & 1) * 8 + (lane & 7)) * VS + (lane >> 4) * 8;
    for (int t = 0; t < tiles; t++) {
        const int k0 = lo + t * MK;
        asm volatile("cp.async.wait_group 1;" ::: "memory");   // the keys; the values may still be on their way
        __syncthreads();
        float s[MK / 8][4];
#pragma unroll
        for (int i = 0; i < MK / 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++) {
            uint32_t qa[4];
            ldsm4(qa, qp + kk * 16);
#pragma unroll
            for (int j = 0; j < MK / 16; j++) {
                uint32_t kb[4];   // keys 16 j .. + 7 and + 8 .. + 15, both halves of the 16 channels
                ldsm4(kb, kp + j * 16 * KS + kk * 16);
                mma_bf16(s[2 * j], qa, kb[0], kb[1]);
                mma_bf16(s[2 * j + 1], qa, kb[2], kb[3]);
            }
        }
        __syncthreads();
        load_keys(t + 1);
        // powers of two of the scaled scores; only tiles at an edge of what the rows see need the mask
        float mx[2] = {m[0], m[1]};
        if (k0 + MK - 1 > pos0 || pos0 + MQ - 1 - k0 >= window) {
#pragma unroll
            for (int i = 0; i < MK / 8; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int key = k0 + i * 8 + 2 * (lane & 3) + (e & 1), p = e < 2 ? pa : pb;
                    s[i][e] = key <= p && p - key < window ? s[i][e] * sc : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
                }
        } else {
#pragma unroll
            for (int i = 0; i < MK / 8; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    s[i][e] *= sc;
                    mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
                }
        }
        float corr[2], mm[2];
#pragma unroll
        for (int u = 0; u < 2; u++) {
            mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 1));
            mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 2));
            corr[u] = m[u] == -INFINITY ? 0.0f : exp2f(m[u] - mx[u]);
            m[u] = mx[u];
            mm[u] = mx[u] == -INFINITY ? 0.0f : mx[u];   // a row that has seen nothing yet: every power below is of minus infinity
            l[u] *= corr[u];
        }
#pragma unroll
        for (int i = 0; i < DV / 8; i++) {
            o[i][0] *= corr[0];
            o[i][1] *= corr[0];
            o[i][2] *= corr[1];
            o[i][3] *= corr[1];
        }
        asm volatile("cp.async.wait_group 1;" ::: "memory");   // the values; the next keys may still be on their way
        __syncthreads();
#pragma unroll
        for (int j = 0; j < MK / 16; j++) {
            uint32_t ph[4], pl[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {   // fragment registers: (rows a, keys low), (rows b, low), (a, high), (b, high)
                const int i = 2 * j + (u >> 1), e = 2 * (u & 1);
                const float x = exp2f(s[i][e] - mm[u & 1]), y = exp2f(s[i][e + 1] - mm[u & 1]);
                l[u & 1] += x + y;
                ph[u] = bf16_pack(x, y);
                pl[u] = bf16_pack(x - bf16_lo(ph[u]), y - bf16_hi(ph[u]));
            }
#pragma unroll
            for (int c = 0; c < DV / 16; c += 2) {
                uint32_t va[4], vb[4];
                ldsm4_t(va, vq + j * 16 * VS + c * 16);
                ldsm4_t(vb, vq + j * 16 * VS + c * 16 + 16);
                mma_bf16(o[2 * c], ph, va[0], va[1]);
                mma_bf16(o[2 * c + 1], ph, va[2], va[3]);
                mma_bf16(o[2 * c + 2], ph, vb[0], vb[1]);
                mma_bf16(o[2 * c + 3], ph, vb[2], vb[3]);
                mma_bf16(o[2 * c], pl, va[0], va[1]);
                mma_bf16(o[2 * c + 1], pl, va[2], va[3]);
                mma_bf16(o[2 * c + 2], pl, vb[0], vb[1]);
                mma_bf16(o[2 * c + 3], pl, vb[2], vb[3]);
            }
        }
        __syncthreads();
        load_values(t + 1);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    const float sink = a.sink[h] * 1.4426950408889634f;
#pragma unroll
    for (int u = 0; u < 2; u++) {
        float lt = l[u];
        lt += __shfl_xor_sync(0xffffffffu, lt, 1);
        lt += __shfl_xor_sync(0xffffffffu, lt, 2);
        const int r = u ? rb : ra;
        if (r >= rows) continue;
        const float mf = fmaxf(m[u], sink), w = exp2f(m[u] - mf), den = lt * w + exp2f(sink - mf);
        const float f = w / den * sigmoid_f32(a.proj[(row0 + r) * a.ldp + a.off_g + h]);
        Y *y = (Y *)a.y + (row0 + r) * a.ldy + h * a.vdim;
#pragma unroll
        for (int i = 0; i < DV / 8; i++) {
            const int c = i * 8 + 2 * (lane & 3);
            if (c < a.vdim) y[c] = from_f32<Y>(o[i][2 * u] * f);
            if (c + 1 < a.vdim) y[c + 1] = from_f32<Y>(o[i][2 * u + 1] * f);
        }
    }
}

int check(const LatentArgs &a, int **err) {
    B200_REQUIRE(a.heads > 0 && a.heads < 65535 && a.dim > 0 && a.rank > 0 && a.vdim > 0 && a.rot >= 0 && a.rot_dims % 2 == 0 && a.rot_dims <= a.rot && a.n <= 65535 &&
                     (a.type == B200_TYPE_F32 || a.type == B200_TYPE_BF16) && a.proj && a.pos,
                 "latent attention: bad argument");
    return device_error_word(err);
}

template <typename K>
int allow_smem(K kernel, size_t smem) {
    B200_REQUIRE(smem <= 220 * 1024, "latent attention: head or latent size too large (%zu bytes of shared memory)", smem);
    if (smem > 48 * 1024) B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return B200_STATUS_SUCCESS;
}

template <typename T, int VEC>
int run_query(const LatentArgs &a, int *err, cudaStream_t s) {
    // a block takes 16 pieces of the rank: enough blocks for one row
    int lanes = 1;
    while (lanes < 16 && lanes * VEC < a.rank) lanes *= 2;
    const unsigned blocks = (unsigned)((a.rank + lanes * VEC - 1) / (lanes * VEC));
    B200_REQUIRE(blocks <= 65535, "latent attention: rank %d is too large", a.rank);
    const size_t smem = ((size_t)(a.dim + 3) / 4 * 4 + (size_t)LT * VEC) * 4;
    int rc = allow_smem(latent_query_kernel<T, VEC>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl(latent_query_kernel<T, VEC>, dim3((unsigned)a.heads + 1, (unsigned)a.n, blocks), dim3(LT), smem, s, a, lanes, err);
}
template <typename T>
int run_decode(const LatentArgs &a, int *err, cudaStream_t s) {
    const int D = a.rank + a.rot, pe = 16 / (int)sizeof(T), qs = (D + pe - 1) / pe * pe;
    const size_t smem = (size_t)LK * key_units<T>(D) * 16 + ((size_t)LH * qs + LK * LH + LH) * 4;
    int rc = allow_smem(latent_decode_kernel<T>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const int hg = (a.heads + LH - 1) / LH, rb = (a.rank + LRB - 1) / LRB;
    return launch_pdl(latent_decode_kernel<T>, dim3((unsigned)a.n_splits, (unsigned)(hg * rb), (unsigned)a.n), dim3(LT), smem, s, a, hg, err);
}
template <typename T, int VEC>
int run_value(const LatentArgs &a, cudaStream_t s) {
    const dim3 g((unsigned)a.heads, (unsigned)a.n, (unsigned)((a.vdim + LV_ROWS - 1) / LV_ROWS));
    const size_t smem = ((size_t)a.rank + 4 + a.n_splits) * 4;
    if (a.y_type == B200_TYPE_F32) {
        int rc = allow_smem(latent_value_kernel<T, float, VEC>, smem);
        return rc != B200_STATUS_SUCCESS ? rc : launch_pdl(latent_value_kernel<T, float, VEC>, g, dim3(LT), smem, s, a);
    }
    int rc = allow_smem(latent_value_kernel<T, __nv_bfloat16, VEC>, smem);
    return rc != B200_STATUS_SUCCESS ? rc : launch_pdl(latent_value_kernel<T, __nv_bfloat16, VEC>, g, dim3(LT), smem, s, a);
}
template <typename T, typename Y>
int run_attn_any(const LatentArgs &a, int *err, cudaStream_t s) {
    const size_t smem = (size_t)(LT / 32) * (a.dim + a.rot + a.vdim) * 4;
    int rc = allow_smem(latent_attn_kernel<T, Y>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl(latent_attn_kernel<T, Y>, dim3((unsigned)((a.n + LT / 32 - 1) / (LT / 32) + a.n_seg), (unsigned)a.heads), dim3(LT), smem, s, a, err);
}
template <typename Y, int DK, int DV, bool ALIGNED>
int run_attn_mma(const LatentArgs &a, int *err, cudaStream_t s) {
    const size_t smem = ((size_t)MQ * (DK + 8) + (size_t)MK * (DK + 8 + DV + 8)) * 2;
    int rc = allow_smem(latent_attn_mma_kernel<Y, DK, DV, ALIGNED>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl(latent_attn_mma_kernel<Y, DK, DV, ALIGNED>, dim3((unsigned)((a.n + MQ - 1) / MQ + a.n_seg), (unsigned)a.heads), dim3(MT), smem, s, a, err);
}
template <typename Y>
int run_attn_bf16(const LatentArgs &a, int *err, cudaStream_t s) {
    const int D = a.dim + a.rot;
    const bool al = a.dim % 8 == 0 && a.rot % 8 == 0 && a.vdim % 8 == 0 && a.rank % 8 == 0 && a.ldkv % 8 == 0 && a.ldc % 8 == 0 &&
                    a.ldp % 4 == 0 && a.off_q % 4 == 0 && a.rot_dims % 4 == 0 && (((uintptr_t)a.kv | (uintptr_t)a.cache | (uintptr_t)a.proj | (uintptr_t)a.rope) & 15) == 0;
    if (D <= 128 && a.vdim <= 64) return al ? run_attn_mma<Y, 128, 64, true>(a, err, s) : run_attn_mma<Y, 128, 64, false>(a, err, s);
    if (D <= 192 && a.vdim <= 128) return al ? run_attn_mma<Y, 192, 128, true>(a, err, s) : run_attn_mma<Y, 192, 128, false>(a, err, s);
    if (D <= 256 && a.vdim <= 128) return al ? run_attn_mma<Y, 256, 128, true>(a, err, s) : run_attn_mma<Y, 256, 128, false>(a, err, s);
    return run_attn_any<__nv_bfloat16, Y>(a, err, s);
}

}  // namespace

int launch_latent_store(const LatentArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.cells && a.norm_w && a.cache, "latent store: null operand");
    return a.type == B200_TYPE_F32 ? launch_pdl(latent_store_kernel<float>, dim3((unsigned)a.n), dim3(LT), 0, s, a, err)
                                   : launch_pdl(latent_store_kernel<__nv_bfloat16>, dim3((unsigned)a.n), dim3(LT), 0, s, a, err);
}
int launch_latent_query(const LatentArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.cells && a.norm_w && a.cache && a.ukv && a.queries, "latent query: null operand");
    const bool al = ((uintptr_t)a.ukv & 15) == 0;
    if (a.type == B200_TYPE_F32) return al && a.rank % 4 == 0 ? run_query<float, 4>(a, err, s) : run_query<float, 1>(a, err, s);
    return al && a.rank % 8 == 0 ? run_query<__nv_bfloat16, 8>(a, err, s) : run_query<__nv_bfloat16, 1>(a, err, s);
}
int launch_latent_decode(const LatentArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.queries && a.cache && a.row_seg && a.seg && a.tab && a.partial && a.per_split > 0 && a.n_splits > 0, "latent decode: null operand");
    B200_REQUIRE(a.ldc % 8 == 0 && ((uintptr_t)a.cache & 15) == 0, "latent decode: cell rows must be whole 16-byte pieces");
    return a.type == B200_TYPE_F32 ? run_decode<float>(a, err, s) : run_decode<__nv_bfloat16>(a, err, s);
}
int launch_latent_value(const LatentArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.partial && a.ukv && a.sink && a.y && a.per_split > 0 && a.n_splits > 0, "latent value: null operand");
    const bool al = ((uintptr_t)a.ukv & 15) == 0;
    if (a.type == B200_TYPE_F32) return al && a.rank % 4 == 0 ? run_value<float, 4>(a, s) : run_value<float, 1>(a, s);
    return al && a.rank % 8 == 0 ? run_value<__nv_bfloat16, 8>(a, s) : run_value<__nv_bfloat16, 1>(a, s);
}
int launch_latent_attn(const LatentArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.kv && a.cache && a.sink && a.seg && a.y && a.n_seg > 0, "latent attention: null operand");
    if (a.type == B200_TYPE_F32) return a.y_type == B200_TYPE_F32 ? run_attn_any<float, float>(a, err, s) : run_attn_any<float, __nv_bfloat16>(a, err, s);
    return a.y_type == B200_TYPE_F32 ? run_attn_bf16<float>(a, err, s) : run_attn_bf16<__nv_bfloat16>(a, err, s);
}

}  // namespace b200
