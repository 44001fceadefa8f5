// Attention of single rows whose heads' weights are mixed in front of the values: a first launch leaves every head's scores (in the base of
// exp2) with maximum and sum per range of keys, a second one forms the weights of all heads for its keys, mixes them and meets the values
// of one key / value head.  Ranges of keys: the CTAs of a row form a cluster in the second launch and add up through distributed shared
// memory.  Behind prompt attention with joint values the mixing is a launch of its own (talk_heads), since it is linear in the weights.
//   float32    scores by eight keys of four lanes, sums by a lane per pair of value columns; f32 behind the loads
//   bfloat16   tensor-core tiles of sixteen heads by sixteen keys per warp, copied ahead into the warp's two buffers; weights enter their
//              products (with the mixing matrix, then with the values) as bf16 pairs
#include <cooperative_groups.h>

#include <algorithm>

#include "attn_rows.cuh"
#include "mma.cuh"

namespace forge {

namespace {

namespace cg = cooperative_groups;
using bf16 = __nv_bfloat16;

constexpr int kWarps = 8, kThreads = kWarps * 32, kHeads = 4, kTileKeys = 16, kTileHeads = 16, kMaxSplits = 8;
constexpr float kLog2e = 1.4426950408889634f;

// per row: scores [keys][heads_p], then {maximum, sum} [kMaxSplits][heads_p]
struct ScoreRow {
    int heads_p, keys;
    __host__ __device__ size_t floats() const { return size_t(heads_p) * (size_t(keys) + 2 * kMaxSplits); }
    __device__ float* scores(float* base, int r) const { return base + size_t(r) * floats(); }
    __device__ float2* stats(float* base, int r) const { return reinterpret_cast<float2*>(scores(base, r) + size_t(heads_p) * keys); }
};

// The range of keys of CTA `split`; what a row sees.
struct Range {
    int lo, front, n, begin, end;
    __device__ __forceinline__ Range(const AttnDims& d, int pos, int split, int splits) {
        lo = d.first_key(pos); front = d.front(pos); n = front + pos - lo + 1;
        const int per = ((n + splits - 1) / splits + 31) & ~31;
        begin = split * per; end = min(n, begin + per);
    }
};

// keys and values of one group of the block that a row completes
template <typename T>
__device__ __forceinline__ void pool_group(const AttnDims& d, T* cache, const int32_t* pt, int pos, int g) {
    pool_columns(d, cache, pt, pos, g * d.dim_p, d.dim_p / 8);
    pool_columns(d, cache, pt, pos, d.groups * d.dim_p + g * d.vdim_p, d.vdim_p / 8);
}

// ------------------------------------------------------------------------------------------------ float32
template <typename T>
__global__ void __launch_bounds__(kThreads) talk_scores_kernel(const AttnDims d, const T* q, T* cache, bool pools, float* scratch, const ScoreRow sr, const StepRows rows) {
    extern __shared__ float sm[];
    const int gq = d.heads / d.groups, blocks = (gq + kHeads - 1) / kHeads;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * kHeads, nh = min(kHeads, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* sq = sm;                                         // [kHeads][dim_p]
    float* sp = sq + kHeads * d.dim_p + warp * kHeads * 32; // [warp][kHeads][32]
    __shared__ float sml[kWarps][kHeads][2];
    pdl_trigger();
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const Range k(d, pos, split, splits);
    const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
    const size_t W = d.row();
    pdl_wait();
    for (int i = threadIdx.x; i < kHeads * d.dim_p; i += kThreads) {
        const int h = i / d.dim_p, c = i % d.dim_p;
        sq[i] = h < nh && c < d.dim ? to_f(q[(size_t(r) * d.heads + h0 + h) * d.dim_p + c]) : 0.f;
    }
    __syncthreads();
    float m[kHeads], l[kHeads];
#pragma unroll
    for (int h = 0; h < kHeads; ++h) { m[h] = -INFINITY; l[h] = 0.f; }
    const float inv_cap = d.softcap > 0.f ? 1.0f / d.softcap : 0.f;
    if (pools && split == splits - 1 && blockIdx.y % blocks == 0) pool_group(d, cache, pt, pos, g);
    const T* kbase = cache + size_t(g) * d.dim_p;
    float* out = sr.scores(scratch, r);
    for (int key0 = k.begin + warp * 32; key0 < k.end; key0 += kThreads) {
        const int nk = min(32, k.end - key0);
        const size_t my_row = d.key_row(pt, key0 + min(lane, nk - 1), k.front, k.lo);
        __syncwarp();
#pragma unroll
        for (int b = 0; b < 4; ++b) {   // eight keys by four lanes
            const int key = b * 8 + (lane >> 2), part = (lane & 3) * 8;
            const T* kr = kbase + __shfl_sync(0xffffffffu, my_row, key) * W;
            float s[kHeads];
#pragma unroll
            for (int h = 0; h < kHeads; ++h) s[h] = 0.f;
#pragma unroll 4
            for (int c = part; c < d.dim_p; c += 32) {
                float kv[8];
                load8(kv, kr + c);
#pragma unroll
                for (int h = 0; h < kHeads; ++h) {
                    float qv[8];
                    load8(qv, sq + h * d.dim_p + c);
#pragma unroll
                    for (int e = 0; e < 8; ++e) s[h] = fmaf(kv[e], qv[e], s[h]);
                }
            }
#pragma unroll
            for (int h = 0; h < kHeads; ++h) {
                s[h] += __shfl_xor_sync(0xffffffffu, s[h], 1);
                s[h] += __shfl_xor_sync(0xffffffffu, s[h], 2);
                float v = s[h] * d.scale;
                if (d.softcap > 0.f) v = d.softcap * tanhf(v * inv_cap);
                if ((lane & 3) == 0) sp[h * 32 + key] = key < nk ? v * kLog2e : -INFINITY;
            }
        }
        __syncwarp();
#pragma unroll
        for (int h = 0; h < kHeads; ++h) {
            const float s = sp[h * 32 + lane];
            if (lane < nk && h < nh) out[size_t(key0 + lane) * sr.heads_p + h0 + h] = s;
            float mx = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[h], mx);
            l[h] = l[h] * exp2f(m[h] - mn) + exp2f(s - mn);
            m[h] = mn;
        }
    }
#pragma unroll
    for (int h = 0; h < kHeads; ++h) {
        const float ls = warp_sum(l[h]);
        if (lane == 0) { sml[warp][h][0] = m[h]; sml[warp][h][1] = ls; }
    }
    __syncthreads();
    if (int(threadIdx.x) < nh) {
        const int h = threadIdx.x;
        float mt = -INFINITY, lt = 0.f;
        for (int w = 0; w < kWarps; ++w) mt = fmaxf(mt, sml[w][h][0]);
        for (int w = 0; w < kWarps; ++w) lt += mt == -INFINITY ? 0.f : sml[w][h][1] * exp2f(sml[w][h][0] - mt);
        sr.stats(scratch, r)[split * sr.heads_p + h0 + h] = make_float2(mt, lt);
    }
}

// {maximum, 1 / sum} of every head over all ranges
__device__ __forceinline__ void all_stats(float2* st, const ScoreRow& sr, float* scratch, int r, int heads, int splits) {
    for (int h = threadIdx.x; h < sr.heads_p; h += kThreads) {
        float m = -INFINITY, l = 0.f;
        if (h < heads) {
            const float2* in = sr.stats(scratch, r) + h;
            for (int s = 0; s < splits; ++s) m = fmaxf(m, in[s * sr.heads_p].x);
            for (int s = 0; s < splits; ++s) { const float2 v = in[s * sr.heads_p]; l += v.x == -INFINITY ? 0.f : v.y * exp2f(v.x - m); }
        }
        st[h] = make_float2(m, l > 0.f ? 1.0f / l : 0.f);
    }
}

// The warps' sums (so, `stride` values per warp, [head][vdim_p]) of a CTA become one, then those of the cluster's CTAs.
template <typename T>
__device__ __forceinline__ void add_rows(const AttnDims& d, float* so, int stride, int nh, int h0, int r, float factor, T* out, int out_ld) {
    const int split = blockIdx.x, splits = gridDim.x;
    __syncthreads();
    for (int i = threadIdx.x; i < nh * d.vdim_p; i += kThreads) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += so[w * stride + i];
        so[i] = v;
    }
    cg::cluster_group cl = cg::this_cluster();
    if (splits > 1) cl.sync();
    else __syncthreads();
    const int items = nh * d.vdim, share = (items + splits - 1) / splits;
    for (int i = split * share + threadIdx.x; i < min(items, (split + 1) * share); i += kThreads) {
        const int h = i / d.vdim, c = i % d.vdim;
        float v = 0.f;
        for (int s = 0; s < splits; ++s) v += (splits > 1 ? cl.map_shared_rank(so, s) : so)[h * d.vdim_p + c];
        out[size_t(r) * out_ld + (h0 + h) * d.vdim + c] = to_t<T>(v * factor);
    }
    if (splits > 1) cl.sync();   // nobody leaves while its shared memory is read
}

// VP: pairs of value columns per lane
template <typename T, int VP>
__global__ void __launch_bounds__(kThreads) talk_values_kernel(const AttnDims d, const T* cache, float* scratch, const ScoreRow sr, int score_splits, const float* __restrict__ talk, float factor, T* out,
                                                               int out_ld, const StepRows rows) {
    extern __shared__ float sm[];
    const int gq = d.heads / d.groups, blocks = (gq + kHeads - 1) / kHeads;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * kHeads, nh = min(kHeads, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float2* st = reinterpret_cast<float2*>(sm);                    // [heads_p]
    float* mix = sm + 2 * sr.heads_p;                              // [heads][kHeads]
    float* sp = mix + kHeads * d.heads + warp * kHeads * 32;       // [warp][kHeads][32]
    float* so = mix + kHeads * d.heads + kWarps * kHeads * 32;     // [warp][kHeads][vdim_p]
    pdl_trigger();
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const Range k(d, pos, split, splits);
    const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
    const size_t W = d.row();
    for (int i = threadIdx.x; i < kHeads * d.heads; i += kThreads) mix[i] = i % kHeads < nh ? talk[size_t(h0 + i % kHeads) * d.heads + i / kHeads] : 0.f;
    pdl_wait();
    all_stats(st, sr, scratch, r, d.heads, score_splits);
    __syncthreads();
    const float* in = sr.scores(scratch, r);
    const T* vbase = cache + size_t(d.groups) * d.dim_p + size_t(g) * d.vdim_p;
    float acc[kHeads][2 * VP];
#pragma unroll
    for (int h = 0; h < kHeads; ++h)
#pragma unroll
        for (int c = 0; c < 2 * VP; ++c) acc[h][c] = 0.f;
    for (int key0 = k.begin + warp * 32; key0 < k.end; key0 += kThreads) {
        const int nk = min(32, k.end - key0);
        const size_t my_row = d.key_row(pt, key0 + min(lane, nk - 1), k.front, k.lo);
        const float* s = in + size_t(key0 + min(lane, nk - 1)) * sr.heads_p;
        float w[kHeads];
#pragma unroll
        for (int h = 0; h < kHeads; ++h) w[h] = 0.f;
        for (int x = 0; x < d.heads; ++x) {
            const float p = exp2f(s[x] - st[x].x) * st[x].y;
#pragma unroll
            for (int h = 0; h < kHeads; ++h) w[h] = fmaf(mix[x * kHeads + h], p, w[h]);
        }
        __syncwarp();
#pragma unroll
        for (int h = 0; h < kHeads; ++h) sp[h * 32 + lane] = w[h];
        __syncwarp();
#pragma unroll 4
        for (int i = 0; i < nk; ++i) {
            const T* vr = vbase + __shfl_sync(0xffffffffu, my_row, i) * W;
#pragma unroll
            for (int c = 0; c < VP; ++c) {
                const int col = 2 * lane + 64 * c;
                if (col >= d.vdim_p) continue;
                const float v0 = to_f(vr[col]), v1 = to_f(vr[col + 1]);
#pragma unroll
                for (int h = 0; h < kHeads; ++h) { const float p = sp[h * 32 + i]; acc[h][2 * c] = fmaf(p, v0, acc[h][2 * c]); acc[h][2 * c + 1] = fmaf(p, v1, acc[h][2 * c + 1]); }
            }
        }
    }
#pragma unroll
    for (int h = 0; h < kHeads; ++h)
#pragma unroll
        for (int c = 0; c < VP; ++c)
            if (2 * lane + 64 * c < d.vdim_p) *reinterpret_cast<float2*>(so + (warp * kHeads + h) * d.vdim_p + 2 * lane + 64 * c) = make_float2(acc[h][2 * c], acc[h][2 * c + 1]);
    add_rows(d, so, kHeads * d.vdim_p, nh, h0, r, factor, out, out_ld);
}

// ------------------------------------------------------------------------------------------------ bfloat16
// sixteen rows of `cols` values (a multiple of 64) per tile, two tiles per warp
struct Tiles {
    int ld, stage;
    __host__ __device__ explicit Tiles(int cols) : ld(cols + 8), stage(kTileKeys * (cols + 8)) {}
};
size_t score_smem(const AttnDims& d) { const Tiles L(d.dim_p); return (size_t(kWarps) * 2 * L.stage + kTileHeads * L.ld) * 2; }
size_t value_smem(const AttnDims& d, const ScoreRow& sr) {
    const Tiles L(d.vdim_p);
    return std::max(size_t(kWarps) * 2 * L.stage * 2, size_t(kWarps) * kTileHeads * d.vdim_p * 4) + size_t(sr.heads_p) * 8;
}
__device__ __forceinline__ void copy_tile(uint32_t dst, int ld, const bf16* src, size_t W, int pieces, uint32_t row, int lane) {
#pragma unroll 4
    for (int p = lane; p < kTileKeys * pieces; p += 32) {   // a multiple of 32 pieces
        const int k = p / pieces, c = (p % pieces) * 8;
        cp_async16(dst + (k * ld + c) * 2, src + __shfl_sync(0xffffffffu, row, k) * W + c, true);
    }
}
// tiles of a warp: copies of two are in flight, those of earlier steps' keys from before the dependency wait
struct TileWalk {
    const AttnDims& d; const Range& k; const int32_t* pt; const bf16* base; uint32_t at; Tiles L; int pieces, warp, lane, written;
    __device__ __forceinline__ int first(int i) const { return k.begin + (warp + kWarps * i) * kTileKeys; }
    __device__ __forceinline__ void fetch(int i) const {
        const int key0 = first(i);
        if (key0 < k.end) copy_tile(at + (i & 1) * L.stage * 2, L.ld, base, d.row(), pieces, uint32_t(d.key_row(pt, min(key0 + (lane & (kTileKeys - 1)), k.end - 1), k.front, k.lo)), lane);
        cp_commit();
    }
    __device__ __forceinline__ bool old(int i) const { return min(k.end, first(i) + kTileKeys) <= written; }
};

__global__ void __launch_bounds__(kThreads) talk_scores_mma_kernel(const AttnDims d, const bf16* q, bf16* cache, bool pools, float* scratch, const ScoreRow sr, const StepRows rows) {
    extern __shared__ __align__(16) unsigned char sm_raw[];
    __shared__ float sml[kWarps][kTileHeads][2];
    const Tiles L(d.dim_p);
    bf16* tiles = reinterpret_cast<bf16*>(sm_raw);
    bf16* sq = tiles + size_t(kWarps) * 2 * L.stage;
    const int gq = d.heads / d.groups, blocks = (gq + kTileHeads - 1) / kTileHeads;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * kTileHeads, nh = min(kTileHeads, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    pdl_trigger();
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const Range k(d, pos, split, splits);
    const TileWalk walk{d, k, rows.page_table + size_t(seq) * rows.pages_per_seq, cache + size_t(g) * d.dim_p, uint32_t(__cvta_generic_to_shared(tiles + size_t(warp) * 2 * L.stage)), L, d.dim_p / 8, warp, lane,
                        d.pool > 0 && rows.fresh > d.window ? 0 : k.n - rows.fresh};
    int ahead = 0;
    while (ahead < 2 && walk.old(ahead)) walk.fetch(ahead++);
    pdl_wait();
    while (ahead < 2) walk.fetch(ahead++);
    for (int i = threadIdx.x; i < kTileHeads * (d.dim_p / 8); i += kThreads) {
        const int h = i / (d.dim_p / 8), c = i % (d.dim_p / 8) * 8;
        *reinterpret_cast<uint4*>(sq + h * L.ld + c) = h < nh ? *reinterpret_cast<const uint4*>(q + (size_t(r) * d.heads + h0 + h) * d.dim_p + c) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    if (pools && split == splits - 1 && blockIdx.y % blocks == 0) pool_group(d, cache, walk.pt, pos, g);
    const SmemMat mq{uint32_t(__cvta_generic_to_shared(sq)), L.ld};
    const int ksteps = (d.dim + 15) / 16;
    const float scale2 = d.scale * kLog2e, inv_cap = d.softcap > 0.f ? d.scale / d.softcap : 0.f;
    float* out = sr.scores(scratch, r) + h0;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    for (int i = 0;; ++i) {
        const int key0 = walk.first(i);
        if (key0 >= k.end) break;
        cp_wait<1>();
        __syncwarp();
        const SmemMat mk{walk.at + uint32_t((i & 1) * L.stage) * 2, L.ld};
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
        for (int c = 0; c < ksteps; ++c) {
            uint32_t fa[4], fb[4];
            mq.a(fa, 0, c * 16, lane);
            mk.b(fb, 0, c * 16, lane);
            mma(s[0], fa, fb[0], fb[1]);
            mma(s[1], fa, fb[2], fb[3]);
        }
        __syncwarp();   // the buffer is read
        walk.fetch(i + 2);
#pragma unroll
        for (int e = 0; e < 2; ++e) {   // heads lr, lr + 8
            float mx = m[e];
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    float& v = s[j][2 * e + b];
                    const int key = key0 + j * 8 + lc + b;
                    v = d.softcap > 0.f ? d.softcap * kLog2e * tanhf(v * inv_cap) : v * scale2;
                    if (key >= k.end) v = -INFINITY;
                    else if (lr + 8 * e < nh) out[size_t(key) * sr.heads_p + lr + 8 * e] = v;
                    mx = fmaxf(mx, v);
                }
            float add = 0.f;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int b = 0; b < 2; ++b) add += mx == -INFINITY ? 0.f : exp2f(s[j][2 * e + b] - mx);
            l[e] = (m[e] == -INFINITY ? 0.f : l[e] * exp2f(m[e] - mx)) + add;
            m[e] = mx;
        }
    }
    cp_wait<0>();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int o = 1; o <= 2; o <<= 1) {
            const float mo = __shfl_xor_sync(0xffffffffu, m[e], o), lo = __shfl_xor_sync(0xffffffffu, l[e], o), mx = fmaxf(m[e], mo);
            l[e] = (m[e] == -INFINITY ? 0.f : l[e] * exp2f(m[e] - mx)) + (mo == -INFINITY ? 0.f : lo * exp2f(mo - mx));
            m[e] = mx;
        }
        if ((lane & 3) == 0) { sml[warp][lr + 8 * e][0] = m[e]; sml[warp][lr + 8 * e][1] = l[e]; }
    }
    __syncthreads();
    if (int(threadIdx.x) < nh) {
        const int h = threadIdx.x;
        float mt = -INFINITY, lt = 0.f;
        for (int w = 0; w < kWarps; ++w) mt = fmaxf(mt, sml[w][h][0]);
        for (int w = 0; w < kWarps; ++w) lt += sml[w][h][0] == -INFINITY ? 0.f : sml[w][h][1] * exp2f(sml[w][h][0] - mt);
        sr.stats(scratch, r)[split * sr.heads_p + h0 + h] = make_float2(mt, lt);
    }
}

// VC: blocks of 64 value columns at most
template <int VC>
__global__ void __launch_bounds__(kThreads) talk_values_mma_kernel(const AttnDims d, const bf16* cache, float* scratch, const ScoreRow sr, int score_splits, const float* __restrict__ talk, float factor,
                                                                   bf16* out, int out_ld, const StepRows rows) {
    extern __shared__ __align__(16) unsigned char sm_raw[];
    const Tiles L(d.vdim_p);
    float2* st = reinterpret_cast<float2*>(sm_raw);                                     // [heads_p]
    bf16* tiles = reinterpret_cast<bf16*>(sm_raw + size_t(sr.heads_p) * 8);
    const int gq = d.heads / d.groups, blocks = (gq + kTileHeads - 1) / kTileHeads;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * kTileHeads, nh = min(kTileHeads, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    pdl_trigger();
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const Range k(d, pos, split, splits);
    const TileWalk walk{d, k, rows.page_table + size_t(seq) * rows.pages_per_seq, cache + size_t(d.groups) * d.dim_p + size_t(g) * d.vdim_p,
                        uint32_t(__cvta_generic_to_shared(tiles + size_t(warp) * 2 * L.stage)), L, d.vdim_p / 8, warp, lane, d.pool > 0 && rows.fresh > d.window ? 0 : k.n - rows.fresh};
    int ahead = 0;
    while (ahead < 2 && walk.old(ahead)) walk.fetch(ahead++);
    // rows h0 + lr, h0 + lr + 8 of the mixing matrix, sixteen columns at a time: the first block stays in registers
    auto mix_block = [&](uint32_t (&f)[4], int x0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int h = lr + (i & 1) * 8, x = x0 + lc + (i >> 1) * 8;
            const float a = h < nh && x < d.heads ? talk[size_t(h0 + h) * d.heads + x] : 0.f, b = h < nh && x + 1 < d.heads ? talk[size_t(h0 + h) * d.heads + x + 1] : 0.f;
            const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
            f[i] = *reinterpret_cast<const uint32_t*>(&v);
        }
    };
    uint32_t mix0[4];
    mix_block(mix0, 0);
    pdl_wait();
    while (ahead < 2) walk.fetch(ahead++);
    all_stats(st, sr, scratch, r, d.heads, score_splits);
    __syncthreads();
    const float* in = sr.scores(scratch, r);
    const int vsteps = (d.vdim + 15) / 16;
    float o[VC * 4][2][4];
#pragma unroll
    for (int v = 0; v < VC * 4; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[v][e >> 2][e & 3] = 0.f;
    for (int i = 0;; ++i) {
        const int key0 = walk.first(i);
        if (key0 >= k.end) break;
        float w[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        for (int x0 = 0; x0 < d.heads; x0 += 16) {
            uint32_t fa[4];
            if (x0 == 0) { fa[0] = mix0[0]; fa[1] = mix0[1]; fa[2] = mix0[2]; fa[3] = mix0[3]; }
            else mix_block(fa, x0);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int key = key0 + j * 8 + lr;
                uint32_t hi[2], lo[2];
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const int x = x0 + lc + 8 * b;
                    float p0 = 0.f, p1 = 0.f;
                    if (key < k.end && x < d.heads) {   // rows of scores are padded to sixteen heads
                        const float2 s = *reinterpret_cast<const float2*>(in + size_t(key) * sr.heads_p + x);
                        const float4 t = *reinterpret_cast<const float4*>(st + x);
                        p0 = exp2f(s.x - t.x) * t.y;
                        if (x + 1 < d.heads) p1 = exp2f(s.y - t.z) * t.w;
                    }
                    split_bf16x2(p0, p1, hi[b], lo[b]);
                }
                mma(w[j], fa, lo[0], lo[1]);
                mma(w[j], fa, hi[0], hi[1]);
            }
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) split_bf16x2(w[j][2 * e], w[j][2 * e + 1], ph[2 * j + e], pl[2 * j + e]);
        cp_wait<1>();
        __syncwarp();
        const SmemMat mv{walk.at + uint32_t((i & 1) * L.stage) * 2, L.ld};
#pragma unroll
        for (int v = 0; v < VC * 4; ++v) {
            if (v >= vsteps) break;
            uint32_t fb[4];
            mv.b_t(fb, 0, v * 16, lane);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                mma(o[v][j], pl, fb[2 * j], fb[2 * j + 1]);
                mma(o[v][j], ph, fb[2 * j], fb[2 * j + 1]);
            }
        }
        __syncwarp();   // the buffer is read
        walk.fetch(i + 2);
    }
    cp_wait<0>();
    __syncthreads();    // sums take the place of the tiles
    float* so = reinterpret_cast<float*>(tiles);                 // [warp][nh][vdim_p]
    const int stride = kTileHeads * d.vdim_p;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int h = lr + 8 * e;
        if (h >= nh) continue;
#pragma unroll
        for (int v = 0; v < VC * 4; ++v)
            if (v < vsteps)
#pragma unroll
                for (int j = 0; j < 2; ++j) *reinterpret_cast<float2*>(so + warp * stride + h * d.vdim_p + v * 16 + j * 8 + lc) = make_float2(o[v][j][2 * e], o[v][j][2 * e + 1]);
    }
    add_rows(d, so, stride, nh, h0, r, factor, out, out_ld);
}

// ------------------------------------------------------------------------------------------------ behind prompt attention
constexpr int kMixHeads = 4;     // heads of a group that a thread carries
constexpr int kMixThreads = 128, kAhead = 8;   // sources whose values are requested together
// A thread = eight columns of one group of one row.
__global__ void __launch_bounds__(kMixThreads) talk_heads_kernel(const AttnDims d, const bf16* __restrict__ o, const float* __restrict__ talk, float factor, bf16* __restrict__ out, int out_ld, int rows) {
    extern __shared__ __align__(16) float mix[];      // [source head][heads, padded]
    const int pieces = d.vdim_p / 8, per = d.groups * pieces, gq = d.heads / d.groups, gq_p = (gq + kMixHeads - 1) / kMixHeads * kMixHeads, ld = d.groups * gq_p;
    const size_t i = size_t(blockIdx.x) * kMixThreads + threadIdx.x;
    const int r = int(i / per), g = int(i % per) / pieces, c = int(i % pieces) * 8;
    const bool on = r < rows && c < d.vdim;
    const size_t W = size_t(d.groups) * d.vdim_p;
    const bf16* src = o + size_t(on ? r : 0) * d.heads * W + size_t(g) * d.vdim_p + c;
    uint4 held[kAhead];
    auto fetch = [&](int x0) {
#pragma unroll
        for (int j = 0; j < kAhead; ++j) held[j] = on && x0 + j < d.heads ? *reinterpret_cast<const uint4*>(src + size_t(x0 + j) * W) : make_uint4(0, 0, 0, 0);
    };
    fetch(0);
    for (int k = threadIdx.x; k < d.heads * ld; k += kMixThreads) {
        const int x = k / ld, h = k % ld / gq_p * gq + k % gq_p;
        mix[k] = k % gq_p < gq ? talk[size_t(h) * d.heads + x] * factor : 0.f;
    }
    __syncthreads();
    for (int h0 = 0; h0 < gq; h0 += kMixHeads) {
        float acc[kMixHeads][8];
#pragma unroll
        for (int h = 0; h < kMixHeads; ++h)
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[h][e] = 0.f;
        if (h0 > 0) fetch(0);
        for (int x0 = 0; x0 < d.heads; x0 += kAhead) {
            uint4 now[kAhead];
#pragma unroll
            for (int j = 0; j < kAhead; ++j) now[j] = held[j];
            if (x0 + kAhead < d.heads) fetch(x0 + kAhead);
#pragma unroll
            for (int j = 0; j < kAhead; ++j) {
                if (x0 + j >= d.heads) break;
                float v[8];
                load8(v, reinterpret_cast<const bf16*>(&now[j]));
                const float4 w4 = get4(mix + (x0 + j) * ld + g * gq_p + h0);
                const float w[kMixHeads] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                for (int h = 0; h < kMixHeads; ++h)
#pragma unroll
                    for (int e = 0; e < 8; ++e) acc[h][e] = fmaf(w[h], v[e], acc[h][e]);
            }
        }
        if (!on) continue;
#pragma unroll
        for (int h = 0; h < kMixHeads; ++h)
            if (h0 + h < gq) {
                bf16* dst = out + size_t(r) * out_ld + size_t(g * gq + h0 + h) * d.vdim + c;
                if (d.vdim % 8 == 0 && out_ld % 8 == 0) {
                    put4(dst, make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]));
                    put4(dst + 4, make_float4(acc[h][4], acc[h][5], acc[h][6], acc[h][7]));
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) if (c + e < d.vdim) dst[e] = __float2bfloat16_rn(acc[h][e]);
                }
            }
    }
}

ScoreRow score_row(const AttnDims& d, int max_keys) { return ScoreRow{pad_to(d.heads, 16), pad_to(std::max(1, max_keys), 32)}; }
bool mma_supported(const AttnDims& d) { return d.vdim_p <= 256 && score_smem(d) <= 220 * 1024 && value_smem(d, score_row(d, 1)) <= 220 * 1024; }
size_t plain_score_smem(const AttnDims& d) { return sizeof(float) * (size_t(kHeads) * d.dim_p + kWarps * kHeads * 32); }
size_t plain_value_smem(const AttnDims& d) { return sizeof(float) * (2 * size_t(pad_to(d.heads, 16)) + size_t(kHeads) * d.heads + kWarps * kHeads * 32 + size_t(kWarps) * kHeads * d.vdim_p); }

template <typename K>
int32_t allow_smem(K kern, size_t smem) {
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    return FORGE_OK;
}

template <typename T>
int32_t run_plain(const AttnDims& d, const void* q, void* cache, bool pools, const float* talk, float factor, float* scratch, const ScoreRow& sr, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st) {
    const int gq = d.heads / d.groups, y = d.groups * ((gq + kHeads - 1) / kHeads), vp = d.vdim_p / 64;
    int splits = 1;   // about two CTAs per SM, no split shorter than one round of its warps
    while (splits < kMaxSplits && rows.n * y * splits * 2 <= 296 && max_keys > splits * kThreads) splits *= 2;
    FORGE_TRY(allow_smem(talk_scores_kernel<T>, plain_score_smem(d)));
    FORGE_CUDA(launch_pdl(talk_scores_kernel<T>, dim3(splits, y, rows.n), dim3(kThreads), plain_score_smem(d), st, d, static_cast<const T*>(q), static_cast<T*>(cache), pools, scratch, sr, rows));
    FORGE_LAUNCH_CHECK();
    auto go = [&](auto kern) -> int32_t {
        FORGE_TRY(allow_smem(kern, plain_value_smem(d)));
        FORGE_CUDA(launch_pdl_cluster(kern, dim3(splits, y, rows.n), dim3(kThreads), splits, plain_value_smem(d), st, d, static_cast<const T*>(cache), scratch, sr, splits, talk, factor, static_cast<T*>(out), out_ld, rows));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    return vp <= 1 ? go(talk_values_kernel<T, 1>) : vp <= 2 ? go(talk_values_kernel<T, 2>) : go(talk_values_kernel<T, 8>);
}

int32_t run_mma(const AttnDims& d, const void* q, void* cache, bool pools, const float* talk, float factor, float* scratch, const ScoreRow& sr, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st) {
    const int gq = d.heads / d.groups, y = d.groups * ((gq + kTileHeads - 1) / kTileHeads);
    int splits = 1;
    while (splits < kMaxSplits && (long long)rows.n * y * splits * 2 <= 296 && max_keys > splits * kWarps * kTileKeys) splits *= 2;
    FORGE_TRY(allow_smem(talk_scores_mma_kernel, score_smem(d)));
    FORGE_CUDA(launch_pdl(talk_scores_mma_kernel, dim3(splits, y, rows.n), dim3(kThreads), score_smem(d), st, d, static_cast<const bf16*>(q), static_cast<bf16*>(cache), pools, scratch, sr, rows));
    FORGE_LAUNCH_CHECK();
    const size_t smem = value_smem(d, sr);
    auto go = [&](auto kern) -> int32_t {
        FORGE_TRY(allow_smem(kern, smem));
        FORGE_CUDA(launch_pdl_cluster(kern, dim3(splits, y, rows.n), dim3(kThreads), splits, smem, st, d, static_cast<const bf16*>(cache), scratch, sr, splits, talk, factor, static_cast<bf16*>(out), out_ld, rows));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    return d.vdim_p <= 64 ? go(talk_values_mma_kernel<1>) : d.vdim_p <= 128 ? go(talk_values_mma_kernel<2>) : go(talk_values_mma_kernel<4>);
}

}  // namespace

static size_t mix_smem(const AttnDims& d) { return size_t(d.heads) * d.groups * pad_to(d.heads / d.groups, kMixHeads) * 4; }
bool talk_rows_supported(const AttnDims& d) { return d.heads <= 128 && mix_smem(d) <= 200 * 1024 && d.vdim_p <= 512 && d.keep == 0 && d.bias_n == 0 && plain_score_smem(d) <= 200 * 1024 && plain_value_smem(d) <= 200 * 1024; }
size_t talk_rows_bytes(const AttnDims& d, int rows, int max_keys) { return size_t(rows) * score_row(d, max_keys).floats() * sizeof(float); }

int32_t talk_rows(const AttnDims& d, int dtype, const void* q, void* cache, bool pools, const float* talk, float factor, void* scratch, size_t max_bytes, void* out, int out_ld, const StepRows& rows, int max_keys,
                  cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    const ScoreRow sr = score_row(d, max_keys);
    const int per = int(std::min<size_t>({size_t(rows.n), size_t(65535), max_bytes / (sr.floats() * 4)}));
    if (!talk_rows_supported(d) || per < 1 || (per < rows.n && !rows.seq)) { set_error("mixed heads: %d heads of %d / %d, %d keys", d.heads, d.dim, d.vdim, max_keys); return FORGE_ERR_SHAPE; }
    const size_t es = dense_size(dtype);
    for (int r0 = 0; r0 < rows.n; r0 += per) {
        StepRows part = rows;
        part.n = std::min(per, rows.n - r0);
        part.pos += r0;
        if (rows.seq) part.seq += r0;
        const void* pq = static_cast<const char*>(q) + size_t(r0) * d.heads * d.dim_p * es;
        void* po = static_cast<char*>(out) + size_t(r0) * out_ld * es;
        float* sc = static_cast<float*>(scratch);
        if (dtype == FORGE_BF16 && mma_supported(d)) FORGE_TRY(run_mma(d, pq, cache, pools, talk, factor, sc, sr, po, out_ld, part, max_keys, st));
        else if (dtype == FORGE_BF16) FORGE_TRY(run_plain<bf16>(d, pq, cache, pools, talk, factor, sc, sr, po, out_ld, part, max_keys, st));
        else FORGE_TRY(run_plain<float>(d, pq, cache, pools, talk, factor, sc, sr, po, out_ld, part, max_keys, st));
    }
    return FORGE_OK;
}

int32_t talk_heads(const AttnDims& d, const void* o, const float* talk, float factor, void* out, int out_ld, int rows, cudaStream_t st) {
    if (rows <= 0) return FORGE_OK;
    const size_t smem = mix_smem(d), threads = size_t(rows) * d.groups * (d.vdim_p / 8);
    FORGE_TRY(allow_smem(talk_heads_kernel, smem));
    talk_heads_kernel<<<unsigned((threads + kMixThreads - 1) / kMixThreads), kMixThreads, smem, st>>>(d, static_cast<const bf16*>(o), talk, factor, static_cast<bf16*>(out), out_ld, rows);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace forge
