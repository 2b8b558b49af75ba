// Grouped-query attention: query head h reads key head h / (heads / kv_heads); keys and values of a position stand in its cell.  A row
// at position i sees the positions j <= i of its sequence with i - j < window or j < keep; the softmax can have a learned sink in its
// denominator (exp(sink): no key, no value, not scaled).  Queries and keys are rotated in the layout of halves (channel i with i +
// dims / 2).  proj holds q of all heads, k and v of all key heads, one after the other, before the rotation.
//
// What a row sees is walked as a list of entries: its kept first positions, then the window's.  An entry's position leads to a cell
// through the segment's part of `tab` (KEPT first positions, then the positions from KEY0 on).
//   grouped_decode_mma_kernel, grouped_decode_kernel   few rows per sequence, BF16 and F32 cells: a cluster per (row, key head, up to 8
//                             query heads), its blocks share the entries and merge through distributed shared memory.  Positions of this
//                             step come from proj (and the row's own is stored in its cell on the way), earlier ones from the cells
//   grouped_store_kernel      keys and values of a prompt's rows into their cells, then
//   grouped_attn_mma_kernel   64 rows x 64-entry tiles on mma.sync (BF16 operands, F32 scores and sums; a weight goes in as two BF16
//                             parts, so that it keeps its 32-bit value to 2^-17), or
//   grouped_attn_kernel       a warp per (row, head), F32 arithmetic, any type and size
#include <cooperative_groups.h>

#include "attn_tile.cuh"

namespace b200 {

namespace {

namespace cg = cooperative_groups;

constexpr int GT = 256;            // threads per block
constexpr int GK = 16;             // entries per tile of a warp of the few-rows kernel
constexpr int GH = 8;              // query heads per block of it
__host__ __device__ constexpr int decode_threads(int hw, int np) { return hw * np >= 16 ? 256 : 512; }   // of that kernel, at most
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
// shared memory of a block of nw warps: each warp's own tiles (when they are done, the warps' sums), then floats at the offsets
struct DecodeSmem {
    int units, tile;                       // 16-byte units of an entry's row, bytes of a tile
    size_t tiles;                          // bytes of the part ahead of the floats
    int q, p, m, l, w, out, ml, floats;    // offsets
    __host__ __device__ DecodeSmem(int dim, int vdim, int hw, int nw, int stages) {
        const int d = pad8(dim), e = pad8(vdim);
        units = (d + e) / 4;
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
        out = (w + (nw > 8 ? nw : 8) * hw + 3) / 4 * 4;
        ml = out + hw * e;
        floats = ml + 2 * hw;
    }
    __host__ __device__ size_t bytes() const { return tiles + (size_t)floats * 4; }
};

// keys and values of a row of this step, as its cell holds them, into `dst` (a warp; values `gap` elements further on) and, if given, into
// the cell
template <typename T>
__device__ __noinline__ void fresh_row(const float *k, const float *v, const float *rope, int rot_dims, int dim, int vdim, T *dst, int gap, T *keep) {
    constexpr int U = 8;
    const int d = pad8(dim), n = d + pad8(vdim), half = rot_dims >> 1;
    for (int c0 = threadIdx.x & 31; c0 < n; c0 += 32 * U) {
        float x[U], y[U], cs[U], sn[U];
#pragma unroll
        for (int u = 0; u < U; u++) {   // all the loads, then the stores
            const int c = c0 + 32 * u;
            const bool turns = c < rot_dims, low = c < half;
            const float *at = c < dim ? k + c : c >= d && c - d < vdim ? v + (c - d) : k, *other = turns ? (low ? at + half : at - half) : at;
            const float *turn = turns ? rope + 2 * (low ? c : c - half) : at;
            x[u] = *at;
            y[u] = *other;
            cs[u] = turns ? turn[0] : 1.0f;
            sn[u] = turns ? (low ? -turn[1] : turn[1]) : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < U; u++) {
            const int c = c0 + 32 * u;
            if (c >= n) break;
            const T r = from_f32<T>(c < dim || (c >= d && c - d < vdim) ? (c < rot_dims ? fmaf(x[u], cs[u], y[u] * sn[u]) : x[u]) : 0.0f);
            dst[c < d ? c : c + gap] = r;
            if (keep) keep[c] = r;
        }
    }
}

// F32 cells.  A warp owns a stretch of the entries from load to weighted sum (no barrier until the end): two lanes share an entry's scores, then a
// lane owns NP pairs of value channels.
template <int HW, int NP>
__global__ void __launch_bounds__(decode_threads(HW, NP), 1)
grouped_decode_kernel(GroupedArgs a, int head_groups, int stages, int *err) {
    typedef float T;
    constexpr int PE = 4;   // elements of 16 bytes
    extern __shared__ __align__(16) uint8_t g_raw[];
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const int dim = pad8(a.dim), vdim = pad8(a.vdim), kp = dim / PE, vp = vdim / PE;
    const DecodeSmem L(a.dim, a.vdim, HW, nw, stages);
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
    // what stands behind entry lane % GK of tile t: a cell, -2 - r for row r of this step, -1 past the last entry
    const auto look_up = [&](int t) -> int {
        const int e = e0 + t * GK + lane % GK;
        if (e >= e1) return -1;
        const int p = en.position(e);
        if (p >= step0 && p - step0 < step_n) return -2 - (step_row + (p - step0));
        const int64_t cell = p < step0 ? cell_of(a, sg, p) : -1;
        if (cell < 0) atomicExch(err, ERR_CELL);
        return cell < 0 ? 0 : (int)cell;
    };
    // an entry's row: key channels, then value channels.  First what cells hold, then this step's own rows
    const T *cache = (const T *)a.cache + (int64_t)g * head_row;
    const auto load_cells = [&](int t, int found) {
        const int kn = min(GK, e1 - e0 - t * GK);
        T *dst = (T *)(mine + (size_t)(t % stages) * L.tile) + lane * PE;
#pragma unroll 4
        for (int k = 0; k < kn; k++, dst += L.units * PE) {
            const int at = __shfl_sync(0xffffffffu, found, k);
            const T *src = cache + (int64_t)at * a.ldc;
            if (at >= 0)
                for (int c = lane; c < kp + vp; c += 32) cp16(dst + (c - lane) * PE, src + c * PE, true);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const auto load_fresh = [&](int t, int found) {
        for (uint32_t todo = __ballot_sync(0xffffffffu, lane < GK && found < -1); todo; todo &= todo - 1) {
            const int k = __ffs(todo) - 1;
            const int64_t r = -2 - __shfl_sync(0xffffffffu, found, k);
            const int32_t *cell = hg == 0 && r == row ? a.cells + row : nullptr;
            T *keep = nullptr;
            if (cell && *cell >= 0 && *cell < a.n_cells) keep = (T *)a.cache + (int64_t)*cell * a.ldc + (int64_t)g * head_row;
            else if (cell && lane == 0) atomicExch(err, ERR_CELL);
            fresh_row<T>(kx + r * a.ldp, vx + r * a.ldp, a.rope + (int64_t)(step0 + (int)(r - step_row)) * a.rot_dims, a.rot_dims, a.dim, a.vdim,
                         (T *)(mine + (size_t)(t % stages) * L.tile) + (size_t)k * L.units * PE, 0, keep);
        }
    };
    const int found0 = look_up(0), found1 = tiles > 1 ? look_up(1) : -1;
    load_cells(0, found0);
    if (stages > 1) load_cells(1, found1);
    int found = stages > 1 && tiles > 2 ? look_up(2) : found1;   // of the next tile to load
    pdl_wait();
    load_fresh(0, found0);
    if (stages > 1) load_fresh(1, found1);
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
                const float4 f = *reinterpret_cast<const float4 *>(kr + p * PE);
#pragma unroll
                for (int h = 0; h < HW; h++) {
                    const float4 x = *reinterpret_cast<const float4 *>(sq + h * dim + p * PE);
                    s[h] = fmaf(x.x, f.x, s[h]);
                    s[h] = fmaf(x.y, f.y, s[h]);
                    s[h] = fmaf(x.z, f.z, s[h]);
                    s[h] = fmaf(x.w, f.w, s[h]);
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
                const float2 v = *reinterpret_cast<const float2 *>(vc + (size_t)k * L.units * PE + 64 * i);
#pragma unroll
                for (int h = 0; h < HW; h++) {
                    acc[h][2 * i] = fmaf(w[h], v.x, acc[h][2 * i]);
                    acc[h][2 * i + 1] = fmaf(w[h], v.y, acc[h][2 * i + 1]);
                }
            }
        }
        __syncwarp();   // the tile and the weights may be overwritten
        load_cells(t + stages, found);
        if (t + stages < tiles) {
            load_fresh(t + stages, found);
            found = look_up(t + stages + 1);
        }
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
#pragma unroll 4
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

// The same over BF16 cells on the tensor cores: a warp's tile of 16 entries meets up to 8 heads' queries in m16n8k16 products whose 16 rows
// are the heads' high BF16 parts and the remainders (their sum keeps 16 bits of the query), then the weights, high parts and remainders
// likewise, meet the values.  A block pushes its sums to the block of the cluster that owns them.
constexpr int DW = 8;   // warps of a block, at most
struct DecodeMmaSmem {
    int kq, vq, units, tile;                  // channels of a key and a value in an entry's row, its 16-byte units, bytes of a tile
    int q, m, l, w, recv, recv_ml, bytes;     // byte offsets
    __host__ __device__ DecodeMmaSmem(int dim, int vdim, int nw, int stages) {
        kq = (dim + 15) / 16 * 16;
        vq = (vdim + 15) / 16 * 16;
        units = (kq + vq) / 8 + 1;            // odd: eight rows of a matrix in different banks
        tile = GK * units * 16;
        q = nw * stages * tile;               // (the warps' sums take the tiles' place)
        m = q + 16 * (kq + 8) * 2;
        l = m + nw * GH * 4;
        w = l + nw * GH * 4;
        recv = w + SPLITS_MAX * GH * 4;
        recv_ml = recv + (GH * vq + SPLITS_MAX) * 4;
        bytes = recv_ml + SPLITS_MAX * GH * 8;
    }
};
__device__ __forceinline__ void cluster_arrive_relaxed() { asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// a bulk copy whose bytes count at the barrier, and the wait for them, bounded (a second time if the first ran out: the copies may still
// be on their way); false when it ran out
constexpr int ERR_BULK = 4;
constexpr uint32_t BULK_WAIT_LIMIT = 1u << 20;
__device__ __forceinline__ void bulk_copy(void *dst, const void *src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes), "r"(bar)
                 : "memory");
}
__device__ __forceinline__ bool bulk_wait(uint32_t bar, uint32_t parity) {
    for (int attempt = 0; attempt < 2; attempt++)
        for (uint32_t it = 0; it < BULK_WAIT_LIMIT; it++) {
            uint32_t ok;
            asm volatile("{ .reg .pred p; mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2; selp.u32 %0, 1, 0, p; }" : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
            if (ok) return attempt == 0;
        }
    return false;
}

template <int NT>   // pairs of value channel groups of 8: 16 NT channels at most
__global__ void __launch_bounds__(32 * DW, 1)
grouped_decode_mma_kernel(GroupedArgs a, int head_groups, int stages, int *err) {
    typedef __nv_bfloat16 bf;
    extern __shared__ __align__(16) uint8_t g_raw[];
    __shared__ uint64_t bars[DW][2];   // a warp's tiles
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5, blocks = (int)gridDim.x;
    const int dim = pad8(a.dim), vdim = pad8(a.vdim);
    const DecodeMmaSmem L(a.dim, a.vdim, nw, stages);
    bf *sQ = (bf *)(g_raw + L.q);
    float *sm = (float *)(g_raw + L.m), *sl = (float *)(g_raw + L.l), *sw = (float *)(g_raw + L.w), *recv = (float *)(g_raw + L.recv);
    float2 *recv_ml = (float2 *)(g_raw + L.recv_ml);
    const int rep = a.heads / a.kv_heads, g = blockIdx.y / head_groups, hg = blockIdx.y % head_groups, h0 = hg * GH, nh = min(GH, rep - h0);
    const int64_t row = blockIdx.z;
    const int KS = L.units * 8, QS = L.kq + 8;   // strides of an entry's and a query's row in elements
    pdl_trigger();
    // the step's inputs and the cells of earlier steps are in place before its first kernel starts
    const int pos = a.pos[row], si = a.row_seg[row];
    const bool seg_ok = segment_ok(a, si), pos_ok = pos >= 0 && (a.rot_dims == 0 || pos < a.rope_rows);
    if (!seg_ok || !pos_ok) {   // (the same for every block of the cluster)
        if (tid == 0) atomicExch(err, seg_ok ? ERR_POS : ERR_SEGMENT);
        return;
    }
    cluster_arrive_relaxed();   // waited for before anything goes to another block
    const int32_t *sg = a.seg + (int64_t)si * SEG_FIELDS;
    const int step0 = sg[SEG_POS0], step_n = sg[SEG_ROWS], step_row = sg[SEG_ROW0];
    const Entries en(a, pos, pos);
    const int owners = blocks * nw, per = (en.total + owners - 1) / owners;
    const int e0 = min(en.total, ((int)blockIdx.x * nw + warp) * per), e1 = min(en.total, e0 + per), tiles = (e1 - e0 + GK - 1) / GK;
    const int head_row = dim + vdim;
    bf *mine = (bf *)(g_raw + (size_t)warp * stages * L.tile);
    const bf *cache = (const bf *)a.cache + (int64_t)g * head_row;
    // what stands behind entry lane % GK of tile t: a cell, -2 - r for row r of this step, -1 past the last entry
    const auto look_up = [&](int t) -> int {
        const int e = e0 + t * GK + lane % GK;
        if (e >= e1) return -1;
        const int p = en.position(e);
        if (p >= step0 && p - step0 < step_n) return -2 - (step_row + (p - step0));
        const int64_t cell = p < step0 ? cell_of(a, sg, p) : -1;
        if (cell < 0) atomicExch(err, ERR_CELL);
        return cell < 0 ? 0 : (int)cell;
    };
    // bulk copies by the entry's lane; values past the last entry are zero
    const auto load_cells = [&](int t, int found) {
        if (t >= tiles) return;
        bf *dst = mine + (size_t)(t % stages) * (L.tile / 2);
        const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&bars[warp][t % stages]);
        const uint32_t cells = __ballot_sync(0xffffffffu, lane < GK && found >= 0);
        if (lane == 0)
            asm volatile("{ .reg .b64 st; mbarrier.arrive.expect_tx.shared::cta.b64 st, [%0], %1; }" ::"r"(bar), "r"((uint32_t)__popc(cells) * (uint32_t)head_row * 2) : "memory");
        __syncwarp();
        if (lane < GK && found >= 0) {
            const bf *src = cache + (int64_t)found * a.ldc;
            if (L.kq == dim) {
                bulk_copy(dst + lane * KS, src, (uint32_t)head_row * 2, bar);
            } else {
                bulk_copy(dst + lane * KS, src, (uint32_t)dim * 2, bar);
                bulk_copy(dst + lane * KS + L.kq, src + dim, (uint32_t)vdim * 2, bar);
            }
        }
        const int kn = e1 - e0 - t * GK;   // (their scores are masked, so the keys need not be)
        for (int k = kn + (lane >> 3); k < GK; k += 4)
            for (int c = lane & 7; c < L.vq / 8; c += 8) *reinterpret_cast<uint4 *>(dst + k * KS + L.kq + 8 * c) = make_uint4(0, 0, 0, 0);
    };
    const auto load_fresh = [&](int t, int found) {
        for (uint32_t todo = __ballot_sync(0xffffffffu, lane < GK && found < -1); todo; todo &= todo - 1) {
            const int k = __ffs(todo) - 1;
            const int64_t r = -2 - __shfl_sync(0xffffffffu, found, k);
            const int32_t *cell = hg == 0 && r == row ? a.cells + row : nullptr;
            bf *keep = nullptr;
            if (cell && *cell >= 0 && *cell < a.n_cells) keep = (bf *)a.cache + (int64_t)*cell * a.ldc + (int64_t)g * head_row;
            else if (cell && lane == 0) atomicExch(err, ERR_CELL);
            const float *x = a.proj + r * a.ldp + (int64_t)a.heads * a.dim;
            fresh_row<bf>(x + g * a.dim, x + (int64_t)a.kv_heads * a.dim + (int64_t)g * a.vdim, a.rope + (int64_t)(step0 + (int)(r - step_row)) * a.rot_dims, a.rot_dims, a.dim, a.vdim,
                          mine + (size_t)(t % stages) * (L.tile / 2) + k * KS, L.kq - dim, keep);
        }
    };
    if (lane == 0) {
        for (int i = 0; i < stages; i++) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"((uint32_t)__cvta_generic_to_shared(&bars[warp][i])) : "memory");
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    const int found0 = look_up(0), found1 = tiles > 1 ? look_up(1) : -1;
    load_cells(0, found0);
    if (stages > 1) load_cells(1, found1);
    int found = stages > 1 && tiles > 2 ? look_up(2) : found1;   // of the next tile to load
    // channels between a head's and the next multiple of 16 stay zero
    if (L.kq != dim || L.vq != vdim)
        for (int i = lane; i < stages * GK * 2; i += 32) {
            bf *r = mine + (i >> 1) * KS;
            if (!(i & 1) && L.kq != dim) *reinterpret_cast<uint4 *>(r + dim) = make_uint4(0, 0, 0, 0);
            if ((i & 1) && L.vq != vdim) *reinterpret_cast<uint4 *>(r + L.kq + vdim) = make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    if (tiles > 0) load_fresh(0, found0);
    if (stages > 1 && tiles > 1) load_fresh(1, found1);
    {   // queries in powers of two: high parts in rows 0 .. 7, remainders in rows 8 .. 15
        const float *q = a.proj + row * a.ldp + (int64_t)(g * rep + h0) * a.dim, *rope = a.rope + (int64_t)pos * a.rot_dims;
        for (int h = warp; h < GH; h += nw)
            for (int d = lane; d < L.kq; d += 32) {
                const float x = h < nh && d < a.dim ? rotated_half(q + (int64_t)h * a.dim, rope, a.rot_dims, d) * (a.scale * 1.4426950408889634f) : 0.0f;
                const bf hi = __float2bfloat16_rn(x);
                sQ[h * QS + d] = hi;
                sQ[(h + 8) * QS + d] = __float2bfloat16_rn(x - __bfloat162float(hi));
            }
    }
    __syncthreads();
    // this lane's head is lane / 4; of a product's 8 columns it has two, high parts and remainders
    float acc[2 * NT][4], m = -INFINITY, l = 0.0f;
#pragma unroll
    for (int i = 0; i < 2 * NT; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    const bf *qp = sQ + (lane & 15) * QS + (lane >> 4) * 8;
    const int koff = ((lane >> 4) * 8 + (lane & 7)) * KS + ((lane >> 3) & 1) * 8, voff = (((lane >> 3) & 1) * 8 + (lane & 7)) * KS + (lane >> 4) * 8 + L.kq;
    for (int t = 0; t < tiles; t++) {
        const int kn = e1 - e0 - t * GK;
        if (!bulk_wait((uint32_t)__cvta_generic_to_shared(&bars[warp][t % stages]), (uint32_t)(t / stages) & 1u) && lane == 0) atomicExch(err, ERR_BULK);
        __syncwarp();
        const bf *tile = mine + (size_t)(t % stages) * (L.tile / 2);
        float c0[4] = {0.0f, 0.0f, 0.0f, 0.0f}, c1[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 4
        for (int d = 0; d < L.kq; d += 16) {
            uint32_t qa[4], kb[4];
            ldsm4(qa, qp + d);
            ldsm4(kb, tile + koff + d);
            mma_bf16(c0, qa, kb[0], kb[1]);
            mma_bf16(c1, qa, kb[2], kb[3]);
        }
        const int e = 2 * (lane & 3);
        float s[4] = {c0[0] + c0[2], c0[1] + c0[3], c1[0] + c1[2], c1[1] + c1[3]};
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (e + (i & 1) + 8 * (i >> 1) >= kn) s[i] = -INFINITY;
        float mx = fmaxf(fmaxf(s[0], s[1]), fmaxf(s[2], s[3]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(m, mx), corr = exp2f(m - mn);   // (a tile has an entry: mn is finite)
        m = mn;
        float p[4];
        uint32_t pa[4];
#pragma unroll
        for (int i = 0; i < 4; i++) p[i] = exp2f(s[i] - mn);
        l = l * corr + ((p[0] + p[1]) + (p[2] + p[3]));
        pa[0] = bf16_pack(p[0], p[1]);
        pa[1] = bf16_pack(p[0] - bf16_lo(pa[0]), p[1] - bf16_hi(pa[0]));
        pa[2] = bf16_pack(p[2], p[3]);
        pa[3] = bf16_pack(p[2] - bf16_lo(pa[2]), p[3] - bf16_hi(pa[2]));
        if (__any_sync(0xffffffffu, corr != 1.0f)) {
#pragma unroll
            for (int i = 0; i < 2 * NT; i++) {
                acc[i][0] *= corr;
                acc[i][1] *= corr;
                acc[i][2] *= corr;
                acc[i][3] *= corr;
            }
        }
#pragma unroll
        for (int i = 0; i < NT; i++) {
            uint32_t vb[4];   // (channels past vq: what stands behind the row, in columns that nobody reads)
            ldsm4_t(vb, tile + voff + 16 * i);
            mma_bf16(acc[2 * i], pa, vb[0], vb[1]);
            mma_bf16(acc[2 * i + 1], pa, vb[2], vb[3]);
        }
        __syncwarp();   // the tile may be overwritten
        load_cells(t + stages, found);
        if (t + stages < tiles) {
            load_fresh(t + stages, found);
            found = look_up(t + stages + 1);
        }
    }
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    if ((lane & 3) == 0) {
        sm[warp * GH + (lane >> 2)] = m;
        sl[warp * GH + (lane >> 2)] = l;
    }
    __syncthreads();
    // the warps' sums, where the tiles were, each counted as its maximum asks for
    float *sacc = (float *)g_raw;
    {
        const int h = lane >> 2;
        float mw[DW], mb = -INFINITY, lb = 0.0f;
#pragma unroll
        for (int k = 0; k < DW; k++) {
            mw[k] = k < nw ? sm[k * GH + h] : -INFINITY;
            mb = fmaxf(mb, mw[k]);
        }
#pragma unroll
        for (int k = 0; k < DW; k++)
            if (mw[k] != -INFINITY) lb = fmaf(sl[k * GH + h], exp2f(mw[k] - mb), lb);
        const float w = m == -INFINITY ? 0.0f : exp2f(m - mb);
        float *o = sacc + ((size_t)warp * GH + h) * L.vq + 2 * (lane & 3);
#pragma unroll
        for (int i = 0; i < 2 * NT; i++)
            if (8 * i < L.vq) *reinterpret_cast<float2 *>(o + 8 * i) = make_float2((acc[i][0] + acc[i][2]) * w, (acc[i][1] + acc[i][3]) * w);
        cluster_wait();   // every block of the cluster has started
        for (int b = warp; b < blocks; b += nw)
            if ((lane & 3) == 0) cluster.map_shared_rank(recv_ml, b)[(int)blockIdx.x * GH + h] = make_float2(mb, lb);
    }
    __syncthreads();
    // block b owns elements b own .. of the heads' channels
    const int total = nh * L.vq, own = (total + blocks - 1) / blocks;
    for (int i = tid; i < total; i += (int)blockDim.x) {
        float v = 0.0f;
#pragma unroll
        for (int k = 0; k < DW; k++)
            if (k < nw) v += sacc[(size_t)k * GH * L.vq + i];
        const int b = i / own;
        cluster.map_shared_rank(recv, b)[(int)blockIdx.x * own + i - b * own] = v;
    }
    cluster_arrive();
    cluster_wait();
    if (warp == 0 && lane < GH) {   // what each block counts, the sink in the denominator
        const float sink = a.sink && lane < nh ? a.sink[g * rep + h0 + lane] * 1.4426950408889634f : -INFINITY;
        float2 ml[SPLITS_MAX];
        float mx = sink, w[SPLITS_MAX];
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++) {
            ml[b] = b < blocks ? recv_ml[b * GH + lane] : make_float2(-INFINITY, 0.0f);
            mx = fmaxf(mx, ml[b].x);
        }
        float den = exp2f(sink - mx);
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++) {
            w[b] = ml[b].x == -INFINITY ? 0.0f : exp2f(ml[b].x - mx);
            den = fmaf(ml[b].y, w[b], den);
        }
        den = 1.0f / den;
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++)
            if (b < blocks) sw[b * GH + lane] = w[b] * den;
    }
    __syncthreads();
    for (int j = tid; j < own; j += (int)blockDim.x) {
        const int i = (int)blockIdx.x * own + j, h = i / L.vq, c = i - h * L.vq;
        if (i >= total || c >= a.vdim) continue;
        float v = 0.0f;
#pragma unroll
        for (int b = 0; b < SPLITS_MAX; b++)
            if (b < blocks) v = fmaf(recv[b * own + j], sw[b * GH + h], v);
        const int64_t at = row * a.ldy + (int64_t)(g * rep + h0 + h) * a.vdim + c;
        if (a.y_type == B200_TYPE_F32) ((float *)a.y)[at] = v;
        else ((bf *)a.y)[at] = __float2bfloat16_rn(v);
    }
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

// warps and tiles per warp that fit, as many warps as possible; 0 warps: none do
DecodeSmem decode_plan(const GroupedArgs &a, int hw, int threads, int *warps, int *stages) {
    for (*warps = threads / 32; *warps >= 1; *warps /= 2)
        for (*stages = 2; *stages >= 1; --*stages) {
            const DecodeSmem L(a.dim, a.vdim, hw, *warps, *stages);
            if (L.bytes() <= SMEM_MAX) return L;
        }
    *warps = 0;
    return DecodeSmem(1, 1, hw, 1, 1);
}
template <int HW, int NP>
int run_decode(const GroupedArgs &a, int *err, cudaStream_t s) {
    int warps = 0, stages = 0;
    const DecodeSmem L = decode_plan(a, HW, decode_threads(HW, NP), &warps, &stages);
    B200_REQUIRE(warps > 0, "grouped decode: head size too large");
    const int rep = a.heads / a.kv_heads, hg = (rep + GH - 1) / GH;
    int rc = allow_smem(grouped_decode_kernel<HW, NP>, L.bytes());
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl_cluster(grouped_decode_kernel<HW, NP>, dim3((unsigned)a.splits, (unsigned)(a.kv_heads * hg), (unsigned)a.n), dim3((unsigned)(32 * warps)),
                              (unsigned)a.splits, L.bytes(), s, a, hg, stages, err);
}
template <int HW>
int run_decode_channels(const GroupedArgs &a, int *err, cudaStream_t s) {
    return a.vdim <= 64 ? run_decode<HW, 1>(a, err, s) : a.vdim <= 128 ? run_decode<HW, 2>(a, err, s) : run_decode<HW, 4>(a, err, s);
}
int run_decode_f32(const GroupedArgs &a, int *err, cudaStream_t s) {
    const int rep = a.heads / a.kv_heads;
    return rep > 4 ? run_decode_channels<8>(a, err, s) : rep > 2 ? run_decode_channels<4>(a, err, s) : rep > 1 ? run_decode_channels<2>(a, err, s)
                                                                                                              : run_decode_channels<1>(a, err, s);
}
bool decode_mma_plan(const GroupedArgs &a, int *warps, int *stages) {
    for (*warps = DW; *warps >= 1; *warps /= 2)
        for (*stages = 2; *stages >= 1; --*stages)
            if ((size_t)DecodeMmaSmem(a.dim, a.vdim, *warps, *stages).bytes <= SMEM_MAX) return true;
    return false;
}
template <int NT>
int run_decode_mma(const GroupedArgs &a, int warps, int stages, int *err, cudaStream_t s) {
    const int rep = a.heads / a.kv_heads, hg = (rep + GH - 1) / GH;
    const size_t smem = (size_t)DecodeMmaSmem(a.dim, a.vdim, warps, stages).bytes;
    int rc = allow_smem(grouped_decode_mma_kernel<NT>, smem);
    if (rc != B200_STATUS_SUCCESS) return rc;
    return launch_pdl_cluster(grouped_decode_mma_kernel<NT>, dim3((unsigned)a.splits, (unsigned)(a.kv_heads * hg), (unsigned)a.n), dim3((unsigned)(32 * warps)),
                              (unsigned)a.splits, smem, s, a, hg, stages, err);
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
    if (a.type == B200_TYPE_F32) decode_plan(a, GH, GT, &warps, &stages);
    else if (!decode_mma_plan(a, &warps, &stages)) warps = 0;
    if (a.vdim > 256 || warps == 0 || a.n_cells > 0x7fffffffLL) {   // heads a block cannot hold
        rc = launch_grouped_store(a, s);
        return rc != B200_STATUS_SUCCESS ? rc : launch_grouped_attn(a, s);
    }
    if (a.type == B200_TYPE_F32) return run_decode_f32(a, err, s);
    return a.vdim <= 64 ? run_decode_mma<4>(a, warps, stages, err, s) : a.vdim <= 128 ? run_decode_mma<8>(a, warps, stages, err, s) : run_decode_mma<16>(a, warps, stages, err, s);
}

}  // namespace b200
