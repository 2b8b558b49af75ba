// Grouped-query attention: query head h reads key head h / (heads / kv_heads); keys and values of a position stand in its cell.  A row
// at position i sees the positions j <= i of its sequence with i - j < window or j < keep; the softmax can have a learned sink in its
// denominator (exp(sink): no key, no value, not scaled).  Queries and keys are rotated in the layout of halves (channel i with i +
// dims / 2).  proj holds q of all heads, k and v of all key heads, one after the other, before the rotation.
//
// What a row sees is walked as a list of entries: its kept first positions, then the window's.  An entry's position leads to a cell
// through the segment's part of `tab` (KEPT first positions, then the positions from KEY0 on).
//   grouped_decode_kernel     few rows per sequence: a cluster per (row, key head, up to 8 query heads), its blocks share the entries and
//                             merge through distributed shared memory.  Positions of this step come from proj (and the row's own is
//                             stored in its cell on the way), earlier ones from the cells
//   grouped_store_kernel      keys and values of a prompt's rows into their cells, then
//   grouped_attn_mma_kernel   64 rows x 64-entry tiles on mma.sync (BF16 operands, F32 scores and sums; a weight goes in as two BF16
//                             parts, so that it keeps its 32-bit value to 2^-17), or
//   grouped_attn_kernel       a warp per (row, head), F32 arithmetic, any type and size
#include <cooperative_groups.h>

#include "attn_tile.cuh"

namespace b200 {

namespace {

namespace cg = cooperative_groups;

constexpr int GT = 256;            // threads per block, at most
constexpr int GK = 16;             // entries per tile of a warp of the few-rows kernel
constexpr int GH = 8;              // query heads per block of it
constexpr int SPLITS_MAX = 8;      // blocks that share a row's entries

__host__ __device__ inline int pad8(int n) { return (n + 7) / 8 * 8; }

// channel j of a rotated head at x, by the position's row of (cos, sin) pairs
__device__ __forceinline__ float rotated_half(const float *x, const float *rope, int rot_dims, int j) {
    if (j >= rot_dims) return x[j];
    const int half = rot_dims >> 1, i = j < half ? j : j - half;
    const float c = rope[2 * i], s = rope[2 * i + 1];
    return j < half ? fmaf(x[j], c, -(x[j + half] * s)) : fmaf(x[j], c, x[j - half] * s);
}

// the entries a row at `pos` sees when the first of its block of rows is at `first`: kept positions 0 .. kept - 1, then lo .. pos
struct Entries {
    int kept, lo, total;
    __device__ __forceinline__ Entries(const GroupedArgs &a, int first, int pos) {
        kept = a.window > 0 ? min(a.keep, pos + 1) : 0;
        lo = a.window > 0 ? max(a.keep, first - a.window + 1) : 0;
        total = kept + max(0, pos + 1 - lo);
    }
    __device__ __forceinline__ int position(int e) const { return e < kept ? e : lo + e - kept; }
};
// the cell of a position of the segment, -1 when the lists do not have it
__device__ __forceinline__ int64_t cell_of(const GroupedArgs &a, const int32_t *sg, int p) {
    const int kept = sg[SEG_KEPT], key0 = sg[SEG_KEY0];
    if (p >= kept && p < key0) return -1;
    const int64_t at = (int64_t)sg[SEG_TAB0] + (p < kept ? p : kept + p - key0);
    if (at < 0 || at >= a.n_tab) return -1;
    const int64_t cell = a.tab[at];
    return cell >= 0 && cell < a.n_cells ? cell : -1;
}
__device__ __forceinline__ bool segment_ok(const GroupedArgs &a, int si) {
    if (si < 0 || si >= a.n_seg) return false;
    const int32_t *sg = a.seg + (int64_t)si * SEG_FIELDS;
    return sg[SEG_ROW0] >= 0 && sg[SEG_ROWS] >= 0 && (int64_t)sg[SEG_ROW0] + sg[SEG_ROWS] <= a.n;
}

template <typename T>
__global__ void __launch_bounds__(GT)
grouped_store_kernel(GroupedArgs a, int *err) {
    pdl_trigger();
    pdl_wait();
    const int64_t row = blockIdx.x, cell = a.cells[row];
    const int pos = a.pos[row], per = pad8(a.dim) + pad8(a.vdim);
    if (cell < 0 || cell >= a.n_cells || (a.rot_dims > 0 && (pos < 0 || pos >= a.rope_rows))) {
        if (threadIdx.x == 0) atomicExch(err, cell < 0 || cell >= a.n_cells ? ERR_CELL : ERR_POS);
        return;
    }
    const float *rope = a.rope + (int64_t)pos * a.rot_dims;
    const float *k = a.proj + row * a.ldp + (int64_t)a.heads * a.dim, *v = k + (int64_t)a.kv_heads * a.dim;
    T *c = (T *)a.cache + cell * a.ldc;
    for (int i = threadIdx.x; i < a.kv_heads * a.dim; i += GT) {
        const int g = i / a.dim, j = i - g * a.dim;
        c[g * per + j] = from_f32<T>(rotated_half(k + g * a.dim, rope, a.rot_dims, j));
    }
    for (int i = threadIdx.x; i < a.kv_heads * a.vdim; i += GT) {
        const int g = i / a.vdim, j = i - g * a.vdim;
        c[g * per + pad8(a.dim) + j] = from_f32<T>(v[i]);
    }
}

// ---- few rows ------------------------------------------------------------------------------------------------
template <typename T>
struct Piece;   // 16 bytes of a cell's row
template <>
struct Piece<__nv_bfloat16> {
    static constexpr int E = 8;
    static __device__ __forceinline__ void unpack(const uint4 &w, float (&f)[8]) {
        f[0] = bf16_lo(w.x); f[1] = bf16_hi(w.x); f[2] = bf16_lo(w.y); f[3] = bf16_hi(w.y);
        f[4] = bf16_lo(w.z); f[5] = bf16_hi(w.z); f[6] = bf16_lo(w.w); f[7] = bf16_hi(w.w);
    }
    static __device__ __forceinline__ float2 pair(const __nv_bfloat16 *p) {
        const uint32_t w = *reinterpret_cast<const uint32_t *>(p);
        return make_float2(bf16_lo(w), bf16_hi(w));
    }
};
template <>
struct Piece<float> {
    static constexpr int E = 4;
    static __device__ __forceinline__ void unpack(const uint4 &w, float (&f)[4]) {
        f[0] = __uint_as_float(w.x); f[1] = __uint_as_float(w.y); f[2] = __uint_as_float(w.z); f[3] = __uint_as_float(w.w);
    }
    static __device__ __forceinline__ float2 pair(const float *p) { return *reinterpret_cast<const float2 *>(p); }
};

// shared memory of a block of nw warps: each warp's own tiles (when they are done, the warps' sums), then floats at the offsets
struct DecodeSmem {
    int units, tile;                       // 16-byte units of an entry's row, bytes of a tile
    size_t tiles;                          // bytes of the part ahead of the floats
    int q, p, m, l, w, out, ml, floats;    // offsets
    __host__ __device__ DecodeSmem(int dim, int vdim, int es, int hw, int nw, int stages) {
        const int d = pad8(dim), e = pad8(vdim);
        units = (d + e) * es / 16;
        while (units % 4 != 2) units++;    // the two lanes of four neighbouring entries meet eight different bank groups
        tile = GK * units * 16;
        const size_t sums = (size_t)nw * hw * e * 4;
        tiles = (size_t)nw * stages * tile;
        if (tiles < sums) tiles = sums;
        q = 0;
        p = q + hw * d;
        m = p + nw * GK * hw;
        l = m + nw * hw;
        w = l + nw * hw;
        out = (w + 8 * hw + 3) / 4 * 4;
        ml = out + hw * e;
        floats = ml + 2 * hw;
    }
    __host__ __device__ size_t bytes() const { return tiles + (size_t)floats * 4; }
};

// A warp owns a stretch of the entries from load to weighted sum (no barrier until the end): two lanes share an entry's scores, then a
// lane owns NP pairs of value channels.
template <typename T, int HW, int NP>
__global__ void __launch_bounds__(GT, 1)
grouped_decode_kernel(GroupedArgs a, int head_groups, int stages, int *err) {
    constexpr int PE = Piece<T>::E;
    extern __shared__ __align__(16) uint8_t g_raw[];
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const int dim = pad8(a.dim), vdim = pad8(a.vdim), kp = dim / PE, vp = vdim / PE;
    const DecodeSmem L(a.dim, a.vdim, (int)sizeof(T), HW, nw, stages);
    float *f32 = (float *)(g_raw + L.tiles);
    float *sq = f32 + L.q, *sp = f32 + L.p + warp * GK * HW, *sm = f32 + L.m, *sl = f32 + L.l, *sw = f32 + L.w, *sout = f32 + L.out, *sml = f32 + L.ml;
    const int rep = a.heads / a.kv_heads, g = blockIdx.y / head_groups, hg = blockIdx.y % head_groups, h0 = hg * GH, nh = min(HW, rep - h0);
    const int64_t row = blockIdx.z;
    pdl_trigger();
    // the step's inputs and the cells of earlier steps are in place before its first kernel starts
    const int pos = a.pos[row], si = a.row_seg[row];
    const bool seg_ok = segment_ok(a, si), pos_ok = pos >= 0 && (a.rot_dims == 0 || pos < a.rope_rows);
    if (!seg_ok || !pos_ok) {   // (the same for every block of the cluster)
        if (tid == 0) atomicExch(err, seg_ok ? ERR_POS : ERR_SEGMENT);
        return;
    }
    const int32_t *sg = a.seg + (int64_t)si * SEG_FIELDS;
    const int step0 = sg[SEG_POS0], step_n = sg[SEG_ROWS], step_row = sg[SEG_ROW0];
    const Entries en(a, pos, pos);
    const int owners = (int)gridDim.x * nw, per = (en.total + owners - 1) / owners;
    const int e0 = min(en.total, ((int)blockIdx.x * nw + warp) * per), e1 = min(en.total, e0 + per), tiles = (e1 - e0 + GK - 1) / GK;
    const int head_row = dim + vdim;
    const float *kx = a.proj + (int64_t)a.heads * a.dim + (int64_t)g * a.dim, *vx = a.proj + (int64_t)(a.heads + a.kv_heads) * a.dim + (int64_t)g * a.vdim;
    uint8_t *mine = g_raw + (size_t)warp * stages * L.tile;
    // what stands behind entry lane % GK of tile t: a cell, -1 - r for row r of this step, NOTHING past the last or when the lists lack it
    constexpr int64_t NOTHING = INT64_MIN;
    const auto look_up = [&](int t) -> int64_t {
        const int e = e0 + t * GK + lane % GK;
        if (e >= e1) return NOTHING;
        const int p = en.position(e);
        if (p >= step0) {
            if (p - step0 < step_n) return -1 - (int64_t)(step_row + (p - step0));
            atomicExch(err, ERR_SEGMENT);
            return NOTHING;
        }
        const int64_t cell = cell_of(a, sg, p);
        if (cell < 0) atomicExch(err, ERR_CELL);
        return cell < 0 ? NOTHING : cell;
    };
    // an entry's row: key channels, then value channels.  cells: those of earlier steps (what is missing is zero), fresh: this step's
    const auto load_tile = [&](int t, int64_t found, bool cells, bool fresh) {
        T *dst0 = (T *)(mine + (size_t)(t % stages) * L.tile);
#pragma unroll 4
        for (int k = 0; k < GK; k++) {
            const int64_t at = __shfl_sync(0xffffffffu, found, k);
            T *dst = dst0 + (size_t)k * L.units * PE;
            if (at >= 0 || at == NOTHING) {
                if (!cells) continue;
                const T *src = (const T *)a.cache + (at < 0 ? 0 : at * a.ldc) + (int64_t)g * head_row;
                for (int c = lane; c < kp + vp; c += 32) cp16(dst + c * PE, src + c * PE, at >= 0);
            } else if (fresh) {
                const int64_t r = -1 - at;
                const int p = step0 + (int)(r - step_row);
                const float *rope = a.rope + (int64_t)p * a.rot_dims;
                T *keep = nullptr;
                if (p == pos && hg == 0) {
                    const int64_t cell = a.cells[row];
                    if (cell >= 0 && cell < a.n_cells) keep = (T *)a.cache + cell * a.ldc + (int64_t)g * head_row;
                    else if (lane == 0) atomicExch(err, ERR_CELL);
                }
#pragma unroll 4
                for (int c = lane; c < dim + vdim; c += 32) {
                    float x = 0.0f;
                    if (c < a.dim) x = rotated_half(kx + r * a.ldp, rope, a.rot_dims, c);
                    else if (c >= dim && c - dim < a.vdim) x = vx[r * a.ldp + c - dim];
                    dst[c] = from_f32<T>(x);
                    if (keep) keep[c] = from_f32<T>(x);
                }
            }
        }
    };
    const auto commit = []() { asm volatile("cp.async.commit_group;" ::: "memory"); };
    const int64_t found0 = look_up(0), found1 = look_up(1);
    if (tiles > 0) load_tile(0, found0, true, false);
    commit();
    if (stages > 1) {
        if (tiles > 1) load_tile(1, found1, true, false);
        commit();
    }
    int64_t found = stages > 1 ? look_up(2) : found1;   // of the next tile to load
    pdl_wait();
    if (tiles > 0) load_tile(0, found0, false, true);
    if (stages > 1 && tiles > 1) load_tile(1, found1, false, true);
    {
        const float *q = a.proj + row * a.ldp + (int64_t)(g * rep + h0) * a.dim, *rope = a.rope + (int64_t)pos * a.rot_dims;
        for (int i = tid; i < HW * dim; i += (int)blockDim.x) {
            const int h = i / dim, d = i - h * dim;
            sq[i] = h < nh && d < a.dim ? rotated_half(q + (int64_t)h * a.dim, rope, a.rot_dims, d) * a.scale : 0.0f;
        }
    }
    __syncthreads();
    float acc[HW][2 * NP], m[HW], l[HW];   // m: the warp's, l: this lane's share
#pragma unroll
    for (int h = 0; h < HW; h++) {
        m[h] = -INFINITY;
        l[h] = 0.0f;
#pragma unroll
        for (int i = 0; i < 2 * NP; i++) acc[h][i] = 0.0f;
    }
    const int entry = lane >> 1, part = lane & 1;
    for (int t = 0; t < tiles; t++) {
        const int kn = min(GK, e1 - e0 - t * GK);
        if (stages > 1) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncwarp();
        const T *tile = (const T *)(mine + (size_t)(t % stages) * L.tile);
        float s[HW];
        {
            const T *kr = tile + (size_t)entry * L.units * PE;
#pragma unroll
            for (int h = 0; h < HW; h++) s[h] = 0.0f;
#pragma unroll 2
            for (int p = part; p < kp; p += 2) {
                float f[PE];
                Piece<T>::unpack(*reinterpret_cast<const uint4 *>(kr + p * PE), f);
#pragma unroll
                for (int h = 0; h < HW; h++) {
#pragma unroll
                    for (int e = 0; e < PE; e += 4) {
                        const float4 x = *reinterpret_cast<const float4 *>(sq + h * dim + p * PE + e);
                        s[h] = fmaf(x.x, f[e], s[h]);
                        s[h] = fmaf(x.y, f[e + 1], s[h]);
                        s[h] = fmaf(x.z, f[e + 2], s[h]);
                        s[h] = fmaf(x.w, f[e + 3], s[h]);
                    }
                }
            }
        }
#pragma unroll
        for (int h = 0; h < HW; h++) {
            s[h] += __shfl_xor_sync(0xffffffffu, s[h], 1);
            const bool in = entry < kn;
            float mx = in ? s[h] : -INFINITY;
#pragma unroll
            for (int o = 2; o < 32; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[h], mx), corr = expf(m[h] - mn), p = in ? expf(s[h] - mn) : 0.0f;   // (a tile has an entry: mn is finite)
            m[h] = mn;
            l[h] = l[h] * corr + (part == 0 ? p : 0.0f);
            if (part == 0) sp[entry * HW + h] = p;
#pragma unroll
            for (int i = 0; i < 2 * NP; i++) acc[h][i] *= corr;
        }
        __syncwarp();
        const T *vc = tile + dim + 2 * lane;
#pragma unroll 4
        for (int k = 0; k < kn; k++) {
            float w[HW];
            if constexpr (HW % 4 == 0) {
#pragma unroll
                for (int h = 0; h < HW; h += 4) *reinterpret_cast<float4 *>(w + h) = *reinterpret_cast<const float4 *>(sp + k * HW + h);
            } else {
#pragma unroll
                for (int h = 0; h < HW; h++) w[h] = sp[k * HW + h];
            }
#pragma unroll
            for (int i = 0; i < NP; i++) {
                if (2 * lane + 64 * i >= vdim) break;
                const float2 v = Piece<T>::pair(vc + (size_t)k * L.units * PE + 64 * i);
#pragma unroll
                for (int h = 0; h < HW; h++) {
                    acc[h][2 * i] = fmaf(w[h], v.x, acc[h][2 * i]);
                    acc[h][2 * i + 1] = fmaf(w[h], v.y, acc[h][2 * i + 1]);
                }
            }
        }
        __syncwarp();   // the tile and the weights may be overwritten
        if (t + stages < tiles) load_tile(t + stages, found, true, true);
        commit();
        found = look_up(t + stages + 1);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // the warps' sums, where the tiles were
    float *sacc = (float *)g_raw;
#pragma unroll
    for (int h = 0; h < HW; h++) {
        l[h] = warp_sum(l[h]);
#pragma unroll
        for (int i = 0; i < NP; i++)
            if (2 * lane + 64 * i < vdim) *reinterpret_cast<float2 *>(sacc + ((size_t)warp * HW + h) * vdim + 2 * lane + 64 * i) = make_float2(acc[h][2 * i], acc[h][2 * i + 1]);
        if (lane == 0) {
            sm[warp * HW + h] = m[h];
            sl[warp * HW + h] = l[h];
        }
    }
    __syncthreads();
    for (int h = warp; h < HW; h += nw) {   // what each warp counts
        const float wm = lane < nw ? sm[lane * HW + h] : -INFINITY, mx = warp_max(wm), w = wm == -INFINITY ? 0.0f : expf(wm - mx);
        const float sum = warp_sum(lane < nw ? sl[lane * HW + h] * w : 0.0f);
        if (lane < nw) sw[lane * HW + h] = w;
        if (lane == 0) {
            sml[2 * h] = mx;
            sml[2 * h + 1] = sum;
        }
    }
    __syncthreads();
    for (int i = tid; i < HW * vdim; i += (int)blockDim.x) {
        const int h = i / vdim;
        float v = 0.0f;
#pragma unroll 8
        for (int k = 0; k < nw; k++) v = fmaf(sacc[(size_t)k * HW * vdim + i], sw[k * HW + h], v);
        sout[i] = v;
    }
    const int blocks = (int)cluster.num_blocks();
    cluster.sync();
    for (int h = warp; h < HW; h += nw) {   // what each block counts, the sink in the denominator
        const float sink = a.sink && h < nh ? a.sink[g * rep + h0 + h] : -INFINITY;
        float2 ml = make_float2(-INFINITY, 0.0f);
        if (lane < blocks) ml = *reinterpret_cast<const float2 *>(cluster.map_shared_rank(sml, lane) + 2 * h);
        const float mx = fmaxf(sink, warp_max(ml.x)), w = ml.x == -INFINITY ? 0.0f : expf(ml.x - mx);
        const float den = warp_sum(ml.y * w) + expf(sink - mx);
        if (lane < blocks) sw[lane * HW + h] = w / den;
    }
    __syncthreads();
    for (int i = (int)cluster.block_rank() * (int)blockDim.x + tid; i < nh * vdim; i += blocks * (int)blockDim.x) {
        const int h = i / vdim, c = i - h * vdim;
        if (c >= a.vdim) continue;
        float part_of[SPLITS_MAX], v = 0.0f;
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++) part_of[b] = b < blocks ? cluster.map_shared_rank(sout, b)[i] : 0.0f;
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++)
            if (b < blocks) v = fmaf(part_of[b], sw[b * HW + h], v);
        const int64_t at = row * a.ldy + (int64_t)(g * rep + h0 + h) * a.vdim + c;
        if (a.y_type == B200_TYPE_F32) ((float *)a.y)[at] = v;
        else ((__nv_bfloat16 *)a.y)[at] = __float2bfloat16_rn(v);
    }
    cluster.sync();   // nobody leaves before everyone has read
}

// ---- many rows -------------------------------------------------------------------------------------------------
template <typename T, typename Y>
__global__ void __launch_bounds__(GT)
grouped_attn_kernel(GroupedArgs a, int *err) {
    extern __shared__ float g_sm[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.y, g = h / (a.heads / a.kv_heads);
    float *q = g_sm + warp * (a.dim + a.vdim), *o = q + a.dim;
    const int64_t row = (int64_t)blockIdx.x * (GT / 32) + warp;
    pdl_trigger();
    pdl_wait();
    if (row >= a.n) return;
    const int pos = a.pos[row], si = a.row_seg[row];
    const bool seg_ok = segment_ok(a, si);
    if (!seg_ok || pos < 0 || (a.rot_dims > 0 && pos >= a.rope_rows)) {
        if (lane == 0) atomicExch(err, seg_ok ? ERR_POS : ERR_SEGMENT);
        return;
    }
    const int32_t *sg = a.seg + (int64_t)si * SEG_FIELDS;
    const Entries en(a, pos, pos);
    const int head_row = pad8(a.dim) + pad8(a.vdim);
    const float *x = a.proj + row * a.ldp + (int64_t)h * a.dim, *rope = a.rope + (int64_t)pos * a.rot_dims;
    for (int d = lane; d < a.dim; d += 32) q[d] = rotated_half(x, rope, a.rot_dims, d);
    for (int c = lane; c < a.vdim; c += 32) o[c] = 0.0f;
    __syncwarp();
    float m = -INFINITY, l = 0.0f;
    for (int e0 = 0; e0 < en.total; e0 += 32) {
        const int e = e0 + lane;
        float s = -INFINITY;
        int64_t cell = 0;
        if (e < en.total) {
            cell = cell_of(a, sg, en.position(e));
            if (cell < 0) {
                atomicExch(err, ERR_CELL);
                cell = 0;
            }
            const T *k = (const T *)a.cache + cell * a.ldc + (int64_t)g * head_row;
            s = 0.0f;
            for (int d = 0; d < a.dim; d++) s = fmaf(q[d], to_f32(k[d]), s);
            s *= a.scale;
        }
        const float mn = fmaxf(m, warp_max(s)), corr = m == -INFINITY ? 0.0f : expf(m - mn), p = e < en.total ? expf(s - mn) : 0.0f;
        l = l * corr + warp_sum(p);
        m = mn;
        const int kn = min(32, en.total - e0);
        for (int c0 = 0; c0 < a.vdim; c0 += 32) {
            const int c = c0 + lane;
            float v = c < a.vdim ? o[c] * corr : 0.0f;
            for (int i = 0; i < kn; i++) {
                const float w = __shfl_sync(0xffffffffu, p, i);
                const int64_t at = __shfl_sync(0xffffffffu, cell, i);
                if (c < a.vdim) v = fmaf(w, to_f32(((const T *)a.cache)[at * a.ldc + (int64_t)g * head_row + pad8(a.dim) + c]), v);
            }
            if (c < a.vdim) o[c] = v;
        }
    }
    const float sink = a.sink ? a.sink[h] : -INFINITY, mf = fmaxf(m, sink), w = expf(m - mf), f = w / (l * w + expf(sink - mf));
    for (int c = lane; c < a.vdim; c += 32) ((Y *)a.y)[row * a.ldy + (int64_t)h * a.vdim + c] = from_f32<Y>(o[c] * f);
}

// tensor-core form: 4 warps x 16 rows, DK and DV the padded head sizes
constexpr int MT = 128, MQ = 64, MK = 64;

// One buffer each for keys and values: the next keys land while the weights meet the values, the next values while the queries meet
// the keys; several blocks per SM cover each other's waits.  The cells of a tile's entries are looked up two tiles ahead.
template <typename Y, int DK, int DV>
__global__ void __launch_bounds__(MT, DK + DV <= 256 ? 3 : 2)
grouped_attn_mma_kernel(GroupedArgs a, bool vec_q, int *err) {
    typedef __nv_bfloat16 bf;
    constexpr int KS = DK + 8, VS = DV + 8;   // row strides: an odd number of 16-byte units
    extern __shared__ __align__(16) uint8_t g_raw[];
    __shared__ int scell[3][MK];
    bf *sQ = (bf *)g_raw, *sK = sQ + MQ * KS, *sV = sK + MK * KS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const int dim = pad8(a.dim), vdim = pad8(a.vdim), head_row = dim + vdim;
    pdl_trigger();
    pdl_wait();
    int r0, rows;
    // later tiles of a prompt see more keys: they go first
    const int32_t *sg = find_tile(a.seg, a.n_seg, a.n, MQ, gridDim.x - 1 - blockIdx.x, &r0, &rows, err);
    if (!sg) return;
    const int64_t row0 = sg[SEG_ROW0] + r0;
    const int pos0 = sg[SEG_POS0] + r0, last = pos0 + rows - 1;
    if (a.rot_dims > 0 && (pos0 < 0 || last >= a.rope_rows)) {
        if (tid == 0) atomicExch(err, ERR_POS);
        return;
    }
    const Entries en(a, pos0, last);
    const int tiles = (en.total + MK - 1) / MK;
    const bf *cache = (const bf *)a.cache + (int64_t)g * head_row;
    // the cells of a tile's entries, -1 past the last
    const auto find_cells = [&](int t) {
        if (tid >= MK) return;
        const int e = t * MK + tid;
        int64_t cell = -1;
        if (e < en.total) {
            cell = cell_of(a, sg, en.position(e));
            if (cell < 0) atomicExch(err, ERR_CELL);
        }
        scell[t % 3][tid] = (int)cell;
    };
    const auto load_part = [&](bf *dst, int stride, int pieces, int channels, int from, int t) {
        if (t < tiles) {
            const int np = channels / 8;
            for (int i = tid; i < MK * pieces; i += MT) {
                const int j = i / pieces, p = i - j * pieces, cell = scell[t % 3][j];
                const bool in = cell >= 0 && p < np;
                cp16(dst + j * stride + p * 8, cache + (in ? (int64_t)cell * a.ldc + from + p * 8 : 0), in);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const auto load_keys = [&](int t) { load_part(sK, KS, DK / 8, dim, 0, t); };
    const auto load_values = [&](int t) { load_part(sV, VS, DV / 8, vdim, dim, t); };
    find_cells(0);
    find_cells(1);
    __syncthreads();
    load_keys(0);
    load_values(0);
    const float *q0 = a.proj + row0 * a.ldp + (int64_t)h * a.dim;
    if (vec_q) {   // four channels at a time, their partners half the rotated part away
        constexpr int QP = DK / 4;
        const int half = a.rot_dims >> 1;
#pragma unroll 4
        for (int i = tid; i < MQ * QP; i += MT) {
            const int t = i / QP, d = (i - t * QP) * 4;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (t < rows && d < a.dim) {
                const float *q = q0 + (int64_t)t * a.ldp;
                x = *reinterpret_cast<const float4 *>(q + d);
                if (d < a.rot_dims) {
                    const bool low = d < half;
                    const float4 y = *reinterpret_cast<const float4 *>(q + (low ? d + half : d - half));
                    const float *rope = a.rope + (int64_t)(pos0 + t) * a.rot_dims + 2 * (low ? d : d - half);
                    const float4 u = *reinterpret_cast<const float4 *>(rope), w = *reinterpret_cast<const float4 *>(rope + 4);   // cos, sin, cos, sin
                    const float sg1 = low ? -1.0f : 1.0f;
                    x = make_float4(fmaf(x.x, u.x, sg1 * (y.x * u.y)), fmaf(x.y, u.z, sg1 * (y.y * u.w)), fmaf(x.z, w.x, sg1 * (y.z * w.y)), fmaf(x.w, w.z, sg1 * (y.w * w.w)));
                }
            }
            *reinterpret_cast<uint2 *>(sQ + t * KS + d) = make_uint2(bf16_pack(x.x, x.y), bf16_pack(x.z, x.w));
        }
    } else {
        for (int i = tid; i < MQ * DK; i += MT) {
            const int t = i / DK, d = i - t * DK;
            const bool in = t < rows && d < a.dim;
            sQ[t * KS + d] = __float2bfloat16_rn(in ? rotated_half(q0 + (int64_t)t * a.ldp, a.rope + (int64_t)(pos0 + t) * a.rot_dims, a.rot_dims, d) : 0.0f);
        }
    }
    // this lane's two rows of the warp's 16
    const int ra = warp * 16 + (lane >> 2), rb = ra + 8, pa = pos0 + ra, pb = pos0 + rb;
    float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < DV / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = a.scale * 1.4426950408889634f;   // powers of two
    const int window = a.window > 0 ? a.window : 0x7fffffff, keep = a.window > 0 ? a.keep : 0;
    const bf *qp = sQ + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8;
    const bf *kp = sK + ((lane >> 4) * 8 + (lane & 7)) * KS + ((lane >> 3) & 1) * 8;
    const bf *vq = sV + (((lane >> 3) & 1) * 8 + (lane & 7)) * VS + (lane >> 4) * 8;
    for (int t = 0; t < tiles; t++) {
        const int k0 = t * MK;
        asm volatile("cp.async.wait_group 1;" ::: "memory");   // the keys; the values may still be on their way
        __syncthreads();
        find_cells(t + 2);   // (read after two more barriers; the tile that had the place is done)
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
        const int pfirst = en.position(k0), plast = en.position(k0 + MK - 1);
        if (k0 + MK > en.total || plast > pos0 || (plast >= keep && last - pfirst >= window)) {
#pragma unroll
            for (int i = 0; i < MK / 8; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int key = k0 + i * 8 + 2 * (lane & 3) + (e & 1), kpos = en.position(key), p = e < 2 ? pa : pb;
                    s[i][e] = key < en.total && kpos <= p && (p - kpos < window || kpos < keep) ? s[i][e] * sc : -INFINITY;
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
    const float sink = a.sink ? a.sink[h] * 1.4426950408889634f : -INFINITY;
#pragma unroll
    for (int u = 0; u < 2; u++) {
        float lt = l[u];
        lt += __shfl_xor_sync(0xffffffffu, lt, 1);
        lt += __shfl_xor_sync(0xffffffffu, lt, 2);
        const int r = u ? rb : ra;
        if (r >= rows) continue;
        const float mf = fmaxf(m[u], sink), w = exp2f(m[u] - mf), f = w / (lt * w + exp2f(sink - mf));
        Y *y = (Y *)a.y + (row0 + r) * a.ldy + (int64_t)h * a.vdim;
#pragma unroll
        for (int i = 0; i < DV / 8; i++) {
            const int c = i * 8 + 2 * (lane & 3);
            if (c < a.vdim) y[c] = from_f32<Y>(o[i][2 * u] * f);
            if (c + 1 < a.vdim) y[c + 1] = from_f32<Y>(o[i][2 * u + 1] * f);
        }
    }
}

// ---- launches --------------------------------------------------------------------------------------------------
int check(const GroupedArgs &a, int **err) {
    B200_REQUIRE(a.heads > 0 && a.heads <= 65535 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= 65536 && a.vdim > 0 && a.vdim <= 65536 &&
                     a.window >= 0 && a.keep >= 0 && a.rot_dims >= 0 && a.rot_dims % 2 == 0 && a.rot_dims <= a.dim && (a.rot_dims == 0 || a.rope) && a.n <= 65535 &&
                     (a.type == B200_TYPE_F32 || a.type == B200_TYPE_BF16) && a.proj && a.pos && a.cache,
                 "grouped attention: bad argument");
    const int64_t row = (int64_t)a.kv_heads * (grouped_pad(a.dim) + grouped_pad(a.vdim));
    B200_REQUIRE(a.ldc >= row && a.ldc % 8 == 0 && ((uintptr_t)a.cache & 15) == 0, "grouped attention: cell rows must be whole 16-byte pieces");
    return device_error_word(err);
}
template <typename K>
int allow_smem(K kernel, size_t smem) {
    if (smem > 48 * 1024) B200_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return B200_STATUS_SUCCESS;
}
constexpr size_t SMEM_MAX = 220 * 1024;

// warps and tiles per warp that fit: eight warps with two tiles if possible; 0 warps: none do
DecodeSmem decode_plan(const GroupedArgs &a, int es, int hw, int *warps, int *stages) {
    for (*warps = GT / 32; *warps >= 1; *warps /= 2)
        for (*stages = 2; *stages >= 1; --*stages) {
            const DecodeSmem L(a.dim, a.vdim, es, hw, *warps, *stages);
            if (L.bytes() <= SMEM_MAX) return L;
        }
    *warps = 0;
    return DecodeSmem(1, 1, es, hw, 1, 1);
}
template <typename T, int HW, int NP>
int run_decode(const GroupedArgs &a, int *err, cudaStream_t s) {
    int warps = 0, stages = 0;
    const DecodeSmem L = decode_plan(a, (int)sizeof(T), HW, &warps, &stages);
    B200_REQUIRE(warps > 0, "grouped decode: head size too large");
    const int rep = a.heads / a.kv_heads, hg = (rep + GH - 1) / GH;
    int rc = allow_smem(grouped_decode_kernel<T, HW, NP>, L.bytes());
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl_cluster(grouped_decode_kernel<T, HW, NP>, dim3((unsigned)a.splits, (unsigned)(a.kv_heads * hg), (unsigned)a.n), dim3((unsigned)(32 * warps)),
                              (unsigned)a.splits, L.bytes(), s, a, hg, stages, err);
}
template <typename T, int HW>
int run_decode_channels(const GroupedArgs &a, int *err, cudaStream_t s) {
    return a.vdim <= 64 ? run_decode<T, HW, 1>(a, err, s) : a.vdim <= 128 ? run_decode<T, HW, 2>(a, err, s) : run_decode<T, HW, 4>(a, err, s);
}
template <typename T>
int run_decode_heads(const GroupedArgs &a, int *err, cudaStream_t s) {
    const int rep = a.heads / a.kv_heads;
    return rep > 4 ? run_decode_channels<T, 8>(a, err, s) : rep > 2 ? run_decode_channels<T, 4>(a, err, s) : rep > 1 ? run_decode_channels<T, 2>(a, err, s) : run_decode_channels<T, 1>(a, err, s);
}
template <typename T, typename Y>
int run_any(const GroupedArgs &a, int *err, cudaStream_t s) {
    const size_t smem = (size_t)(GT / 32) * (a.dim + a.vdim) * 4;
    B200_REQUIRE(smem <= SMEM_MAX, "grouped attention: head size too large (%zu bytes of shared memory)", smem);
    int rc = allow_smem(grouped_attn_kernel<T, Y>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl(grouped_attn_kernel<T, Y>, dim3((unsigned)((a.n + GT / 32 - 1) / (GT / 32)), (unsigned)a.heads), dim3(GT), smem, s, a, err);
}
template <typename Y, int DK, int DV>
int run_mma(const GroupedArgs &a, int *err, cudaStream_t s) {
    const size_t smem = ((size_t)MQ * (DK + 8) + (size_t)MK * (DK + 8 + DV + 8)) * 2;
    int rc = allow_smem(grouped_attn_mma_kernel<Y, DK, DV>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    const bool vec_q = a.dim % 4 == 0 && a.ldp % 4 == 0 && a.rot_dims % 8 == 0 && (((uintptr_t)a.proj | (uintptr_t)a.rope) & 15) == 0;
    return launch_pdl(grouped_attn_mma_kernel<Y, DK, DV>, dim3((unsigned)((a.n + MQ - 1) / MQ + a.n_seg), (unsigned)a.heads), dim3(MT), smem, s, a, vec_q, err);
}
template <typename Y>
int run_bf16(const GroupedArgs &a, int *err, cudaStream_t s) {
    const int d = a.dim, e = a.vdim;
    if (a.n_cells > 0x7fffffffLL) return run_any<__nv_bfloat16, Y>(a, err, s);
    if (d <= 64 && e <= 64) return run_mma<Y, 64, 64>(a, err, s);
    if (d <= 96 && e <= 96) return run_mma<Y, 96, 96>(a, err, s);
    if (d <= 128 && e <= 128) return run_mma<Y, 128, 128>(a, err, s);
    if (d <= 192 && e <= 128) return run_mma<Y, 192, 128>(a, err, s);
    if (d <= 256 && e <= 256) return run_mma<Y, 256, 256>(a, err, s);
    return run_any<__nv_bfloat16, Y>(a, err, s);
}

}  // namespace

int launch_grouped_store(const GroupedArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.cells, "grouped store: null operand");
    return a.type == B200_TYPE_F32 ? launch_pdl(grouped_store_kernel<float>, dim3((unsigned)a.n), dim3(GT), 0, s, a, err)
                                   : launch_pdl(grouped_store_kernel<__nv_bfloat16>, dim3((unsigned)a.n), dim3(GT), 0, s, a, err);
}
int launch_grouped_attn(const GroupedArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.seg && a.row_seg && a.tab && a.y && a.n_seg > 0, "grouped attention: null operand");
    if (a.type == B200_TYPE_F32) return a.y_type == B200_TYPE_F32 ? run_any<float, float>(a, err, s) : run_any<float, __nv_bfloat16>(a, err, s);
    return a.y_type == B200_TYPE_F32 ? run_bf16<float>(a, err, s) : run_bf16<__nv_bfloat16>(a, err, s);
}
int launch_grouped_decode(const GroupedArgs &a, cudaStream_t s) {
    int *err = nullptr;
    int rc = check(a, &err);
    if (rc != B200_STATUS_SUCCESS || a.n == 0) return rc;
    B200_REQUIRE(a.cells && a.seg && a.row_seg && a.tab && a.y && a.n_seg > 0 && a.splits >= 1 && a.splits <= SPLITS_MAX, "grouped decode: bad operand");
    int warps = 0, stages = 0;
    decode_plan(a, a.type == B200_TYPE_F32 ? 4 : 2, GH, &warps, &stages);
    if (a.vdim > 256 || warps == 0) {   // heads a block cannot hold
        rc = launch_grouped_store(a, s);
        return rc != B200_STATUS_SUCCESS ? rc : launch_grouped_attn(a, s);
    }
    return a.type == B200_TYPE_F32 ? run_decode_heads<float>(a, err, s) : run_decode_heads<__nv_bfloat16>(a, err, s);
}

}  // namespace b200
