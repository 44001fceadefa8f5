// Dense linear layers of the layer-list models: out[token][row] = act[token][K] . W[row][K]^T.
//
// bfloat16 (gemm_dense_kernel): tcgen05 with both operands in shared memory.  A tile is 128 weight rows (MMA M) x NT
// tokens (MMA N = 16 .. 256); one kernel serves a decode step (NT = 16: a weight stream, 16 KB of weights per K step and
// SM in a ring of five stages) and a prompt (NT = 256).  Of T tiles over G CTAs the first G floor(T / G) are, for prompts,
// whole tiles dealt in turn (neighbouring CTAs then work on the same weight rows, which come from L2 once); the K steps of 64 of
// the remaining tiles are dealt evenly, CTA i of S taking the steps [i U / S, (i + 1) U / S) of their U, so every SM streams the
// same amount whatever the number of tiles.  A tile that several CTAs share is finished by the last of them to arrive
// (ticket): every share is left in scratch memory and added in K order, so the result does not depend on the order of
// arrival.  Nobody waits for another CTA.  Up to 32 tokens with at most one tile per SM, the CTAs of a tile form a cluster instead: each takes
// an equal part of its K steps and finishes some of its tokens, for which the others store their parts into its shared memory.  The ring of the sixteen-token form leaves room for a second CTA on the SM: the next product's weights are
// requested while this one ends.
// Warp roles: 0 = TMA producer, 1 = TMEM allocation and MMA issue, the rest = epilogue (TMEM lane = weight row): four warps, or for more than 32
// tokens eight, two per 32 rows, each with half of the columns.
// The weights lie in memory as the very images the ring holds (dense_tile_image), so a stage is one contiguous 16 KB bulk copy.
// Accumulators are double buffered in tensor memory: the epilogue of one tile runs under the products of the next.
// The weight stages of the ring are requested before the dependency wait of a programmatic launch, the activations after.
//
// Products in groups (GROUPED) take their tiles of tokens, each with the matrix it meets, from a table in memory; listed products
// (LISTED) take a fixed run of K steps and then those of the groups that the table names.  Both read the table behind the dependency wait.
//
// float32 (gemm_f32_kernel): a tiled product on the CUDA cores in plain f32 fused multiply-adds.
#include <algorithm>
#include <cstring>

#include "dense.cuh"
#include "tc5.cuh"

namespace forge {

namespace {

using namespace tc5;

constexpr int BK = 64;
template <int NT> constexpr int kEpilogueWarps = NT <= 32 ? 4 : 8;
template <int NT> constexpr int kThreads = 64 + 32 * kEpilogueWarps<NT>;

// activations: bfloat16 models take the fast exponential and quotient, whose errors are far inside the rounding of what is stored
template <typename T> __device__ __forceinline__ float act_sigmoid(float x, float v) {   // x * sigmoid(v)
    if constexpr (sizeof(T) == 2) return __fdividef(x, 1.0f + __expf(-v));
    else return x / (1.0f + expf(-v));
}
template <typename T> __device__ __forceinline__ float clamped_glu(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return act_sigmoid<T>(g, 1.702f * g) * (u + 1.0f);
}

// The fields of a segment this thread's row needs, in registers: a store through a pointer may not make the compiler fetch them
// again for every value.
template <typename T>
struct RowOut {
    int kind, seg;
    bool ok;                 // the row belongs to a segment
    bool fresh;
    size_t ld;
    float* f32; T* t;        // the row's place of token 0
    const int32_t* place;
    const T* blend; size_t blend_ld; float own, other;   // blend: the row's place of row 0
    float limit, mul, add, nw, nb, plus;
    // what is stored for v in row `to` of dst
    __device__ __forceinline__ float blended(float v, size_t to) const { return blend ? fmaf(other, to_f(blend[to * blend_ld]), own * v) : v; }
};
template <typename T>
__device__ __forceinline__ RowOut<T> row_out(const DenseOut& o, int row, int first_row) {
    RowOut<T> q{};
    int s = -1;
    for (int i = 0; i < o.nseg; ++i)
        if (first_row >= o.seg[i].row0 && first_row < o.seg[i].row0 + o.seg[i].rows) s = i;
    q.kind = -1;
    if (s < 0) return q;
    const OutSeg& g = o.seg[s];
    const int r = row - g.row0, group = g.group;
    q.kind = g.kind;
    q.seg = s;
    q.ok = r < g.rows;
    q.ld = size_t(g.ld);
    q.fresh = g.fresh;
    const int col = (q.kind == SEG_CLAMPED_GLU || q.kind == SEG_SILU_GLU) ? r >> 1 : (q.kind == SEG_CAST && group) ? (r / group) * g.group_ld + r % group : r;
    q.f32 = static_cast<float*>(g.dst) + col;
    q.t = static_cast<T*>(g.dst) + col;
    q.place = g.place;
    if (q.kind == SEG_CAST && g.blend && q.ok) { q.blend = static_cast<const T*>(g.blend) + col; q.blend_ld = size_t(g.blend_ld); q.own = g.own; q.other = g.other; }
    q.limit = g.limit;
    if (q.ok) {
        if (g.mul) q.mul = g.mul[r];
        if (g.add) q.add = g.add[r];
        if (q.kind == SEG_RESID) {
            if (g.after.w) q.nw = g.after.w[r];
            if (g.after.kind == AFTER_DYT) q.nb = g.after.b[r];
            if (g.after.w2) q.nb = g.after.w2[r];
            if (g.after.plus) q.plus = g.after.plus[r];
        }
    }
    return q;
}
// what a finished row of the stream leaves
template <typename T>
struct Leave {
    int kind;
    bool two;                // a second norm's input
    size_t ld, next_ld, parts;
    T *next, *next2;
    float alpha, nw, nb, plus;
    float* sums; float* keep; const float* again;
    __device__ __forceinline__ Leave(const OutSeg& g, const RowOut<T>& q, int row, int first_row)
        : kind(g.after.kind), two(g.after.w2 != nullptr), ld(q.ld), next_ld(size_t(g.after.ld)), parts(size_t(g.after.parts)), alpha(g.after.alpha), nw(q.nw), nb(q.nb), plus(q.plus) {
        const int r = row - g.row0;
        next = static_cast<T*>(g.after.dst) + r;
        next2 = next + g.after.col2;
        sums = kind == AFTER_RMS ? g.after.sums + (first_row - g.row0) / 32 : nullptr;
        keep = g.after.keep ? g.after.keep + r : nullptr;
        again = g.after.again ? g.after.again + r : nullptr;
    }
    __device__ __forceinline__ float next_value(float x) const { return kind == AFTER_DYT ? dynamic_tanh(x, alpha, nw, nb) : kind == AFTER_RMS ? x * nw : x; }
    // a finished value of the stream (token t): the entry of a pass of a loop
    __device__ __forceinline__ float enter(float x, size_t t) const {
        if (keep) keep[t * ld] = x;
        if (again) x += again[t * ld];
        return x + plus;
    }
};
// column of the activations the rows of the tile at `row` are multiplied with
__device__ __forceinline__ int act_col(const DenseOut& o, int row) {
    int c = 0;
    for (int i = 0; i < o.nseg; ++i) if (o.seg[i].row0 <= row) c = o.seg[i].act_col;
    return c;
}

// the epilogue of one value v; `up`: the value of the next row, used by the even rows of gated pairs, w: what those are multiplied with; `old`: what dst
// holds, if it is known; returns the stream's new value
template <typename T>
__device__ __forceinline__ float put_one(const RowOut<T>& g, const Leave<T>& n, float v, float up, float w, size_t t, float old, bool old_known, bool even_row) {
    float* f = g.f32 + t * g.ld;
    T* h = g.t + t * g.ld;
    switch (g.kind) {
        case SEG_CLAMPED_GLU: if (even_row) *h = to_t<T>(clamped_glu<T>(v, up, g.limit) * w); break;
        case SEG_SILU_GLU: if (even_row) *h = to_t<T>(act_sigmoid<T>(v, v) * up * w); break;
        case SEG_CAST: { const size_t to = g.place ? size_t(g.place[t]) : t; g.t[to * g.ld] = to_t<T>(g.blended(v, to)); break; }
        case SEG_SIGMOID: *h = to_t<T>(act_sigmoid<T>(1.f, v)); break;
        case SEG_SILU: *h = to_t<T>(act_sigmoid<T>(v, v)); break;
        case SEG_TANH: *h = to_t<T>(tanhf(v)); break;
        case SEG_SIGMOID_F32: *f = sigmoid(v); break;
        case SEG_DECAY: *f = -g.mul * softplus(v); break;
        case SEG_EXP_DECAY: *f = -expf(v); break;
        case SEG_RESID: {
            const float x = n.enter((g.fresh ? 0.f : old_known ? old : *f) + v, t);
            *f = x;
            if (n.kind) n.next[t * n.next_ld] = to_t<T>(n.next_value(x));
            if (n.two) n.next2[t * n.next_ld] = to_t<T>(x * n.nb);
            return x;
        }
        default: *f = v;
    }
    return 0.f;
}

// the sum of squares behind a token's scale
__device__ __forceinline__ float row_scale(const RowScale& s, float sum) { return s.mul / sqrtf(sum * s.inv_n + s.eps); }

// of few tokens, lane c: token tok0 + c (parts a multiple of four, or one)
template <int NT> __device__ __forceinline__ float lane_scale(const RowScale& s, int tok0, int cols, int lane) {
    constexpr int SHARE = 32 / NT;   // lanes per token
    const int c = lane % NT, i0 = lane / NT;
    const bool ok = c < cols;
    const float* src = s.sums + size_t(ok ? (s.row ? s.row[tok0 + c] : tok0 + c) : 0) * s.parts;
    float sum = 0.f;
    if (s.parts == 1) sum = ok ? *src : 0.f;
    else {
#pragma unroll 8
        for (int i = i0; i < s.parts / 4; i += SHARE) {
            const float4 v = ok ? reinterpret_cast<const float4*>(src)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
            sum += (v.x + v.y) + (v.z + v.w);
        }
        if (SHARE == 2) sum += __shfl_xor_sync(0xffffffffu, sum, 16);
    }
    return row_scale(s, sum);
}

enum Mode { PLAIN = 0, GROUPED, LISTED };

struct GemmParams {
    DenseOut out;
    const void* w;           // weight images
    int m, N, nk;            // tokens, rows, K steps per tile
    int tt_count;            // token tiles
    int waves;               // whole tiles per CTA
    uint32_t units;          // K steps of the tiles after them, dealt to the first `sharers` CTAs (at most one per step: no share is empty)
    int sharers;
    int cluster;             // > 0: CTA i takes part i % cluster of the K steps of tile i / cluster, and nothing is dealt out
    float* part; int* tickets;
    int* err;
    RowScale scale;
    int pitch, k_off;        // images per row tile, and in front of the first K step
    // GROUPED: row tiles per group, images from one group to the next, elements of the output from one group to the next
    GroupTable groups;
    int row_tiles; uint32_t group_images; long long group_dst;
    // LISTED: K steps in front of the groups', and of a group
    int k_fixed, k_group;
};

// (32-bit: the host checks that units * sharers fits; 64-bit divisions in front of the first load cost microseconds)
__device__ __forceinline__ uint32_t share_begin(uint32_t units, uint32_t g, uint32_t sharers) { return units * g / sharers; }
__device__ __forceinline__ int share_of(uint32_t units, uint32_t u, uint32_t sharers) { return int(((u + 1) * sharers - 1) / units); }

// the pieces of work of one CTA, in order: [k0, k0 + n) K steps of `tile`
template <int MODE> struct Work {
    int cta, grid, waves, nk, wave = 0;
    uint32_t u, u1;
    int tile, k0, n;
    // groups: how many the table names (of a listed product the host's bound, until it is read)
    __device__ __forceinline__ Work(const GemmParams& p, uint32_t u_begin, uint32_t u_end, int groups)
        : cta(blockIdx.x), grid(gridDim.x), waves(p.waves), nk(p.nk), u(u_begin), u1(u_end) {
        if (MODE == GROUPED) {   // whole tiles in turn, or one part of one tile
            const int tiles = groups * p.row_tiles;
            if (p.cluster > 0) { if (int(u / uint32_t(nk)) >= tiles) u1 = u; waves = 0; }
            else waves = tiles > cta ? (tiles - cta + grid - 1) / grid : 0;
        }
        if (MODE == LISTED) {
            const uint32_t end = u / uint32_t(nk) * uint32_t(nk) + uint32_t(p.k_fixed + groups * p.k_group);
            u1 = min(u1, end);
        }
    }
    __device__ __forceinline__ bool next() {
        if (wave < waves) { tile = wave++ * grid + cta; k0 = 0; n = nk; return true; }
        if (u >= u1) return false;
        const int t = int(u / uint32_t(nk));
        k0 = int(u) - t * nk;
        n = min(int(u1 - u), nk - k0);
        tile = waves * grid + t;
        u += uint32_t(n);
        return true;
    }
};
// where a tile's rows, tokens and weights lie
struct Tile { int row_tile, tok0, cols, group, w0; };
template <int NT, int MODE> __device__ __forceinline__ Tile tile_at(const GemmParams& p, int tile, int groups) {
    if constexpr (MODE == GROUPED) {
        const GroupTile g = p.groups.tiles[tile % groups];
        return Tile{tile / groups, g.row0, g.rows, g.group, g.w0};
    }
    const int tok0 = (tile % p.tt_count) * NT;
    return Tile{tile / p.tt_count, tok0, min(NT, p.m - tok0), 0, 0};
}
// K steps in order -> where they lie
template <int MODE> struct KMap {
    int end = 0, shift = 0;
    __device__ __forceinline__ int at(const GemmParams& p, int k) {
        if (MODE != LISTED) return k;
        if (k >= end) {
            if (k < p.k_fixed) end = p.k_fixed;
            else {
                const int a = (k - p.k_fixed) / p.k_group;
                end = p.k_fixed + (a + 1) * p.k_group;
                shift = (p.groups.tiles[a].group - a) * p.k_group;
            }
        }
        return k + shift;
    }
};

template <int NT> struct Ring {
    static constexpr int X_BYTES = NT * 128, STAGE = 16384 + X_BYTES;
    static constexpr int STAGES = NT <= 16 ? 5 : (200 * 1024) / STAGE;
    static constexpr int EXCHANGE = NT <= 16 ? 14336 : NT <= 32 ? 20480 : 0;   // parts that the other CTAs of a cluster store: four tokens take 2 KB
    static constexpr uint32_t COLS = NT <= 16 ? 32 : 2 * NT;   // two accumulators
};

template <int NT, int MODE>
__global__ void __launch_bounds__(kThreads<NT>, NT <= 16 ? 2 : 1) gemm_dense_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ GemmParams p) {
    constexpr int STAGE = Ring<NT>::STAGE, STAGES = Ring<NT>::STAGES;
    constexpr uint32_t kCols = Ring<NT>::COLS;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    __shared__ uint64_t full[STAGES], empty[STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_err, s_last;

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    uint32_t u0 = 0, u1 = 0;   // this CTA's share of the dealt-out K steps
    const int rank = p.cluster > 1 ? int(blockIdx.x) % p.cluster : 0;
    if (p.cluster > 0) {
        const uint32_t t = blockIdx.x / uint32_t(p.cluster) * uint32_t(p.nk);
        u0 = t + uint32_t(p.nk * rank / p.cluster); u1 = t + uint32_t(p.nk * (rank + 1) / p.cluster);
    } else if (int(blockIdx.x) < p.sharers) { u0 = share_begin(p.units, blockIdx.x, p.sharers); u1 = share_begin(p.units, blockIdx.x + 1, p.sharers); }
    if (tid == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(&acc_full[s], 1); mbar_init(&acc_empty[s], kEpilogueWarps<NT>); }
        s_err = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc<kCols>(&s_tmem);
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = s_tmem;
    pdl_trigger();
    if (p.cluster > 1) cluster_arrive();   // nobody stores into a CTA that has not begun

    if (warp == 0) {
        if (lane == 0) {
            // two walks over the same pieces: weight stages run up to a whole ring ahead of the dependency wait
            int groups = MODE == LISTED ? p.groups.max_tiles : 0;
            if constexpr (MODE == GROUPED) { pdl_wait(); groups = *p.groups.n; }
            Work<MODE> ww(p, u0, u1, groups), wx = ww;
            KMap<MODE> mw, mx;
            int kw = 0;
            size_t image = 0;
            bool more = ww.next();
            auto first_image = [&]() {
                const Tile t = tile_at<NT, MODE>(p, ww.tile, groups);
                image = size_t(t.row_tile) * p.pitch + size_t(t.group) * p.group_images + p.k_off;
            };
            if (more) first_image();
            const unsigned char* const weights = static_cast<const unsigned char*>(p.w);
            auto weight_stage = [&](int s) {   // one contiguous image of 128 rows x 64 columns, already swizzled
                mbar_expect_tx(&full[s], uint32_t(STAGE));
                bulk_load(ring + size_t(s) * STAGE, weights + (image + mw.at(p, ww.k0 + kw)) * 16384, 16384, &full[s]);
                if (++kw == ww.n) { kw = 0; more = ww.next(); if (more) first_image(); }
            };
            int ahead = 0;
            const int most = MODE == LISTED ? min(STAGES, p.k_fixed - ww.k0) : STAGES;
            for (; ahead < most && more; ++ahead) weight_stage(ahead);   // constant: may overlap the kernel in front
            if constexpr (MODE != GROUPED) pdl_wait();
            if constexpr (MODE == LISTED) {
                groups = *p.groups.n;
                wx = Work<MODE>(p, u0, u1, groups);
                if (more) { Work<MODE> w = wx; more = w.next() && kw < w.n; ww.n = w.n; }
            }
            int s = 0, i = 0;
            uint32_t phase = 1;   // parity of the round in front of the current one
            bool ok = true;
            while (ok && wx.next()) {
                const Tile t = tile_at<NT, MODE>(p, wx.tile, groups);
                const int tok0 = t.tok0, col0 = act_col(p.out, t.row_tile * 128);
                for (int k = 0; k < wx.n; ++k, ++i) {
                    if (i >= ahead) {
                        if (!mbar_wait(&empty[s], phase, &s_err)) { atomicExch(&s_err, 1); ok = false; break; }
                        weight_stage(s);
                    }
                    tma_2d(ring + size_t(s) * STAGE + 16384, &map_x, col0 + mx.at(p, wx.k0 + k) * BK, tok0, &full[s]);
                    if (++s == STAGES) { s = 0; phase ^= 1; }
                }
            }
        }
        if (p.cluster > 1) {
            __syncwarp();
            cluster_wait();
            cluster_sync();
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int s = 0;
            uint32_t phase = 0;
            bool ok = true;
            int seg = 0, groups = 0;
            if constexpr (MODE != PLAIN) { pdl_wait(); groups = *p.groups.n; }
            for (Work<MODE> w(p, u0, u1, groups); ok && w.next(); ++seg) {
                const int n = w.n, buf = seg & 1;
                if (seg >= 2 && !mbar_wait(&acc_empty[buf], ((seg >> 1) - 1) & 1, &s_err)) { ok = false; break; }
                fence_after();
                for (int k = 0; k < n; ++k) {
                    if (!mbar_wait(&full[s], phase, &s_err)) { ok = false; break; }
                    fence_after();
                    const uint32_t base = smem_u32(ring + size_t(s) * STAGE);
#pragma unroll
                    for (int k16 = 0; k16 < BK / 16; ++k16)
                        umma_ss(tmem + uint32_t(buf * NT), desc_kmajor(base + k16 * 32), desc_kmajor(base + 16384 + k16 * 32), idesc_bf16(NT),
                                (k > 0 || k16 > 0) ? 1u : 0u);
                    umma_commit(&empty[s]);
                    if (++s == STAGES) { s = 0; phase ^= 1; }
                }
                if (ok) umma_commit(&acc_full[buf]);
            }
            if (!ok) atomicExch(&s_err, 1);
        }
        if (p.cluster > 1) {
            __syncwarp();
            cluster_wait();
            cluster_sync();
        }
    } else {
        pdl_wait();
        const int quad = warp & 3;
        const uint32_t lane_addr = tmem + (uint32_t(quad * 32) << 16);
        constexpr int CH = NT == 32 ? 32 : 16;   // columns per read
        constexpr int EW = kEpilogueWarps<NT>, MINE = NT / (EW / 4);
        const int c_begin = (warp - 2) / 4 * MINE, c_end = c_begin + MINE;   // this warp's columns
        auto epilogue_sync = [&]() { asm volatile("bar.sync 1, %0;" ::"n"(EW * 32) : "memory"); };
        int seg_i = 0;
        float col_scale = 1.f;   // of the tokens, lane c: of column c (few tokens: all of the tile's)
        int scaled_tok0 = -1, scaled_cols = 0;
        const int groups = MODE != PLAIN ? *p.groups.n : 0;
        Work<MODE> w(p, u0, u1, groups);
        // a CTA of a cluster takes part in finishing its tile even if the list left it no steps
        bool none = false;
        auto next = [&]() {
            if (w.next()) return true;
            if (MODE != LISTED || p.cluster <= 1 || seg_i > 0) return false;
            none = true;
            w.tile = int(u0 / uint32_t(p.nk)); w.n = 0;
            return true;
        };
        for (; next(); ++seg_i) {
            const int tile = w.tile, n = w.n, buf = seg_i & 1;
            const uint32_t t_begin = uint32_t((tile - p.waves * int(gridDim.x)) * p.nk), t_end = t_begin + uint32_t(p.nk);   // among the dealt-out steps
            const Tile at_tile = tile_at<NT, MODE>(p, tile, groups);
            const int row0 = at_tile.row_tile * 128 + quad * 32, tok0 = at_tile.tok0, cols = at_tile.cols;
            const int row = row0 + lane;
            // every warp's rows lie in one segment (segments start at multiples of 32 rows)
            RowOut<__nv_bfloat16> g = row_out<__nv_bfloat16>(p.out, row, row0);
            if constexpr (MODE == GROUPED) { g.t += at_tile.group * p.group_dst; g.f32 += at_tile.group * p.group_dst; }
            if (NT <= 32 && p.scale.sums && (tok0 != scaled_tok0 || cols != scaled_cols)) {
                col_scale = lane_scale<NT <= 32 ? NT : 32>(p.scale, tok0, cols, lane);
                scaled_tok0 = tok0; scaled_cols = cols;
            }
            const float* pair_w = MODE == GROUPED && p.groups.weight ? p.groups.weight + at_tile.w0 : nullptr;
            // what dst holds is on its way while the product, or the chunk before, is finished
            float x_old[CH];
            const bool adds = g.kind == SEG_RESID && g.ok && !g.fresh;
            auto fetch_old = [&](int c0) {
#pragma unroll
                for (int c = 0; c < CH; ++c)
                    x_old[c] = adds && c < cols - c0 && (p.cluster <= 1 || (c >> 2) % p.cluster == rank) ? g.f32[size_t(tok0 + c0 + c) * g.ld] : 0.f;
            };
            if (g.kind == SEG_RESID) fetch_old(c_begin);
            // the four warps meet at the barriers of a shared tile: one whose wait gave up must not leave the loop alone
            if (!(MODE == LISTED && none) && !mbar_wait(&acc_full[buf], (seg_i >> 1) & 1, &s_err)) atomicExch(&s_err, 1);
            fence_after();
            auto finish = [&](int c0, float (&v)[CH]) {
                const int n_c = cols - c0;
                const size_t t0 = size_t(tok0 + c0);
                if (p.scale.sums) {
                    if (NT > 32) col_scale = lane < n_c ? row_scale(p.scale, p.scale.sums[p.scale.row ? p.scale.row[t0 + lane] : t0 + lane]) : 1.f;
#pragma unroll
                    for (int c = 0; c < CH; ++c) v[c] *= __shfl_sync(0xffffffffu, col_scale, c);
                }
#pragma unroll
                for (int c = 0; c < CH; ++c) v[c] += g.add;
                auto put_t = [&](auto f) {
                    __nv_bfloat16* dst = g.t + t0 * g.ld;
#pragma unroll
                    for (int c = 0; c < CH; ++c) if (c < n_c) dst[c * g.ld] = __float2bfloat16_rn(f(v[c]));
                };
                auto put_f = [&](auto f) {
                    float* dst = g.f32 + t0 * g.ld;
#pragma unroll
                    for (int c = 0; c < CH; ++c) if (c < n_c) dst[c * g.ld] = f(v[c]);
                };
                if (n_c == 1) {   // one token: little code
                    const float got = __shfl_xor_sync(0xffffffffu, v[0], 1);
                    float x = 0.f;
                    const Leave<__nv_bfloat16> n(p.out.seg[g.seg], g, row, row0);
                    if (g.ok) x = put_one(g, n, v[0], got, pair_w ? pair_w[c0] : 1.f, t0, x_old[0], true, !(lane & 1));
                    if (g.kind == SEG_RESID && n.sums) {
                        x = warp_sum(x * x);
                        if (lane == 0) n.sums[t0 * n.parts] = x;
                    }
                } else if (g.kind == SEG_CLAMPED_GLU || g.kind == SEG_SILU_GLU) {
                    // neighbouring lanes hold gate_j and up_j: the even lane takes the first half of the columns
                    const bool even = !(lane & 1), clamped = g.kind == SEG_CLAMPED_GLU;
                    const int mine = even ? 0 : CH / 2;
                    __nv_bfloat16* dst = g.t + (t0 + mine) * g.ld;
#pragma unroll
                    for (int c = 0; c < CH / 2; ++c) {
                        const float got = __shfl_xor_sync(0xffffffffu, even ? v[CH / 2 + c] : v[c], 1);
                        const float ga = even ? v[c] : got, up = even ? got : v[CH / 2 + c];
                        if (g.ok && mine + c < n_c) dst[c * g.ld] = __float2bfloat16_rn((clamped ? clamped_glu<__nv_bfloat16>(ga, up, g.limit) : act_sigmoid<__nv_bfloat16>(ga, ga) * up) * (pair_w ? pair_w[c0 + mine + c] : 1.f));
                    }
                } else if (g.kind == SEG_RESID) {
                    const Leave<__nv_bfloat16> n(p.out.seg[g.seg], g, row, row0);
                    float* dst = g.f32 + t0 * g.ld;
                    float x[CH];
#pragma unroll
                    for (int c = 0; c < CH; ++c) x[c] = x_old[c];
                    if (c0 + CH < c_end) fetch_old(c0 + CH);
                    if (n.keep || n.again) {
#pragma unroll
                        for (int c = 0; c < CH; ++c) { x[c] += v[c]; if (g.ok && c < n_c) x[c] = n.enter(x[c], t0 + c); }
                    } else {
#pragma unroll
                        for (int c = 0; c < CH; ++c) x[c] += v[c] + n.plus;
                    }
                    if (g.ok) {
#pragma unroll
                        for (int c = 0; c < CH; ++c) if (c < n_c) dst[c * g.ld] = x[c];
                        if (n.kind) {
                            __nv_bfloat16* nx = n.next + t0 * n.next_ld;
#pragma unroll
                            for (int c = 0; c < CH; ++c) if (c < n_c) nx[c * n.next_ld] = __float2bfloat16_rn(n.next_value(x[c]));
                        }
                        if (n.two) {
                            __nv_bfloat16* nx = n.next2 + t0 * n.next_ld;
#pragma unroll
                            for (int c = 0; c < CH; ++c) if (c < n_c) nx[c * n.next_ld] = __float2bfloat16_rn(x[c] * n.nb);
                        }
                    }
                    if (n.sums) {   // lane c ends with the sum over the warp's rows of column c's squares
#pragma unroll
                        for (int c = 0; c < CH; ++c) x[c] = g.ok ? x[c] * x[c] : 0.f;
                        if constexpr (CH == 16)
#pragma unroll
                            for (int c = 0; c < CH; ++c) x[c] += __shfl_xor_sync(0xffffffffu, x[c], 16);
#pragma unroll
                        for (int o = CH / 2; o > 0; o >>= 1)
#pragma unroll
                            for (int c = 0; c < o; ++c) {
                                const bool up = lane & o;
                                const float send = up ? x[c] : x[c + o], mine = up ? x[c + o] : x[c];
                                x[c] = mine + __shfl_xor_sync(0xffffffffu, send, o);
                            }
                        if (lane < CH && lane < n_c) n.sums[(t0 + lane) * n.parts] = x[0];
                    }
                } else if (g.ok) switch (g.kind) {
                    case SEG_CAST:
                        if (g.place || g.blend) {
                            int to[CH];
#pragma unroll
                            for (int c = 0; c < CH; ++c) to[c] = c >= n_c ? 0 : g.place ? g.place[t0 + c] : int(t0) + c;
                            if (g.blend) {
                                float other[CH];
#pragma unroll
                                for (int c = 0; c < CH; ++c) other[c] = c < n_c ? to_f(g.blend[size_t(to[c]) * g.blend_ld]) : 0.f;
#pragma unroll
                                for (int c = 0; c < CH; ++c) v[c] = fmaf(g.other, other[c], g.own * v[c]);
                            }
#pragma unroll
                            for (int c = 0; c < CH; ++c) if (c < n_c) g.t[size_t(to[c]) * g.ld] = __float2bfloat16_rn(v[c]);
                        } else put_t([](float x) { return x; });
                        break;
                    case SEG_SIGMOID: put_t([](float x) { return act_sigmoid<__nv_bfloat16>(1.f, x); }); break;
                    case SEG_SILU: put_t([](float x) { return act_sigmoid<__nv_bfloat16>(x, x); }); break;
                    case SEG_TANH: put_t([](float x) { return tanhf(x); }); break;
                    case SEG_SIGMOID_F32: put_f([](float x) { return sigmoid(x); }); break;
                    case SEG_DECAY: put_f([&](float x) { return -g.mul * softplus(x); }); break;
                    case SEG_EXP_DECAY: put_f([&](float x) { return -expf(x); }); break;
                    default: put_f([](float x) { return x; });
                }
            };
            auto load = [&](int c0, float (&v)[CH]) {
                uint32_t t[CH];
                if constexpr (CH == 16) tmem_ld16(lane_addr + uint32_t(buf * NT + c0), t);
                else tmem_ld32(lane_addr + uint32_t(buf * NT + c0), t);
                wait_ld();
#pragma unroll
                for (int c = 0; c < CH; ++c) v[c] = __uint_as_float(t[c]);
            };
            if (MODE == GROUPED || MODE == LISTED ? p.cluster <= 1 : n == p.nk) {
#pragma unroll 1
                for (int c0 = c_begin; c0 < c_end && c0 < cols; c0 += CH) {
                    float v[CH];
                    load(c0, v);
                    finish(c0, v);
                }
            } else if (NT <= 32 && p.cluster > 1) {
                // the tokens 4 c .. 4 c + 3 are finished by CTA c % cluster: box [c / cluster][sender][row][4]
                const Leave<__nv_bfloat16> nx(p.out.seg[g.seg], g, row, row0);
                const int at = (quad * 32 + lane) * 4, groups = (cols + 3) / 4, senders = p.cluster - 1;
                float* box = reinterpret_cast<float*>(ring + size_t(STAGES) * STAGE);
                float v[CH];
                if (MODE == LISTED && none) {
#pragma unroll
                    for (int c = 0; c < CH; ++c) v[c] = 0.f;
                } else load(0, v);
                cluster_wait();
#pragma unroll
                for (int c = 0; c < CH / 4; ++c) {
                    const int to = c % p.cluster;
                    if (c < groups && to != rank)
                        cluster_store4(cluster_addr(box + (c / p.cluster * senders + (rank < to ? rank : rank - 1)) * 512 + at, to), make_float4(v[4 * c], v[4 * c + 1], v[4 * c + 2], v[4 * c + 3]));
                }
                __syncwarp();
                cluster_sync();
#pragma unroll 1
                for (int k = 0; rank + k * p.cluster < groups; ++k) {
                    float t[4] = {0.f, 0.f, 0.f, 0.f}, old[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                    for (int c = 0; c < CH / 4; ++c)
                        if (c == rank + k * p.cluster)
#pragma unroll
                            for (int e = 0; e < 4; ++e) { t[e] = v[4 * c + e]; old[e] = x_old[4 * c + e]; }
                    for (int q = 0; q < senders; ++q) {
                        const float4 o = *reinterpret_cast<const float4*>(box + (k * senders + q) * 512 + at);
                        t[0] += o.x; t[1] += o.y; t[2] += o.z; t[3] += o.w;
                    }
                    const int c0 = (rank + k * p.cluster) * 4;
#pragma unroll 1
                    for (int e = 0; e < min(4, cols - c0); ++e) {
                        float val = t[0];
                        if (p.scale.sums) val *= __shfl_sync(0xffffffffu, col_scale, c0 + e);
                        val += g.add;
                        const float got = __shfl_xor_sync(0xffffffffu, val, 1);
                        float x = 0.f;
                        if (g.ok) x = put_one(g, nx, val, got, pair_w ? pair_w[c0 + e] : 1.f, size_t(tok0 + c0 + e), old[0], true, !(lane & 1));
                        if (g.kind == SEG_RESID && nx.sums) {
                            x = warp_sum(x * x);
                            if (lane == 0) nx.sums[size_t(tok0 + c0 + e) * nx.parts] = x;
                        }
                        t[0] = t[1]; t[1] = t[2]; t[2] = t[3];
                        old[0] = old[1]; old[1] = old[2]; old[2] = old[3];
                    }
                }
            } else if (MODE == PLAIN) {
                // a shared tile: this CTA's part goes to its slot (0: the part its share starts with, 1: the other one)
                float* mine = p.part + (size_t(blockIdx.x) * 2 + (u0 >= t_begin ? 0 : 1)) * (NT * 128);
#pragma unroll 1
                for (int c0 = c_begin; c0 < c_end && c0 < cols; c0 += CH) {
                    float v[CH];
                    load(c0, v);
#pragma unroll
                    for (int c = 0; c < CH; ++c) if (c < cols - c0) __stcg(mine + size_t(c0 + c) * 128 + quad * 32 + lane, v[c]);
                }
                const int first = share_of(p.units, t_begin, p.sharers), last = share_of(p.units, t_end - 1, p.sharers);
                __threadfence();
                epilogue_sync();
                if (tid == 64) {
                    const int old = atomicAdd(p.tickets + tile, 1);
                    s_last = old == last - first;
                    if (s_last) p.tickets[tile] = 0;
                }
                epilogue_sync();
                if (s_last) {
                    __threadfence();
                    if (g.kind == SEG_RESID) fetch_old(c_begin);
#pragma unroll 1
                    for (int c0 = c_begin; c0 < c_end && c0 < cols; c0 += CH) {
                        float v[CH];
#pragma unroll
                        for (int c = 0; c < CH; ++c) v[c] = 0.f;
                        // only the first share of the tile may be the second part of its CTA; loads of QB shares in flight together
                        constexpr int QB = NT <= 16 ? 4 : 2;
                        const int n_c = cols - c0;
                        const int first_slot = share_begin(p.units, first, p.sharers) >= t_begin ? 0 : 1;
                        for (int q = first; q <= last; q += QB) {
                            float t[QB][CH];
#pragma unroll
                            for (int b = 0; b < QB; ++b) {
                                const float* src = p.part + (size_t(q + b) * 2 + (q + b == first ? first_slot : 0)) * (NT * 128) + quad * 32 + lane + size_t(c0) * 128;
#pragma unroll
                                for (int c = 0; c < CH; ++c) t[b][c] = q + b <= last && c < n_c ? __ldcg(src + size_t(c) * 128) : 0.f;
                            }
#pragma unroll
                            for (int b = 0; b < QB; ++b)
#pragma unroll
                                for (int c = 0; c < CH; ++c) v[c] += t[b][c];
                        }
                        finish(c0, v);
                    }
                }
                epilogue_sync();   // s_last is read before it is written again
            }
            fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[buf]);
        }
        if (MODE == GROUPED && p.cluster > 1 && seg_i == 0) {   // a tile the table does not name
            __syncwarp();
            cluster_wait();
            cluster_sync();
        }
        fence_before();
    }
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free<kCols>(tmem);
    }
    if (tid == 0 && s_err && p.err) atomicExch(p.err, 1);
}

// most CTAs per tile, clusters of which all run at once (a cluster lies within one group of SMs, so large ones leave SMs idle); 0: too few tiles to fill the SMs
template <int NT, int MODE>
int32_t cluster_parts(long long tiles, int nk, size_t smem, int* parts) {
    static int fits[9] = {0};
    auto kern = gemm_dense_kernel<NT, MODE>;
    if (!fits[1])
        for (int c = 1; c <= 8; ++c) {
            cudaLaunchConfig_t cfg{};
            cudaLaunchAttribute at[1];
            cfg.gridDim = dim3(unsigned(c * 148)); cfg.blockDim = dim3(kThreads<NT>); cfg.dynamicSmemBytes = std::max(smem, size_t(120) * 1024);   // one CTA per SM
            at[0].id = cudaLaunchAttributeClusterDimension;
            at[0].val.clusterDim.x = unsigned(c); at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
            cfg.attrs = at; cfg.numAttrs = 1;
            FORGE_CUDA(cudaOccupancyMaxActiveClusters(&fits[c], kern, &cfg));
        }
    *parts = 0;
    for (int c = 1; c <= 8; ++c)
        if (tiles <= fits[c] && (c == 1 || (nk >= 2 * c && (c - 1) * ((NT / 4 + c - 1) / c) * 2048 <= Ring<NT>::EXCHANGE))) *parts = c;
    if (tiles * *parts < 90 && tiles > fits[8] && MODE == PLAIN) *parts = 0;
    return FORGE_OK;
}

constexpr int kShareSteps = 96;   // what sharing a tile of 256 tokens costs, in K steps (measured)
template <int NT, int MODE>
int32_t launch_dense(const DenseWeight& w, const void* act, int act_ld, int act_rows, GemmParams& p, int sms, cudaStream_t st) {
    CUtensorMap mx;
    int last_col = 0;
    for (int i = 0; i < p.out.nseg; ++i) last_col = std::max(last_col, p.out.seg[i].act_col);
    FORGE_TRY(make_map_2d(&mx, act, uint64_t(last_col + (MODE == LISTED ? w.K : p.nk * BK)), uint64_t(act_rows), uint64_t(act_ld) * 2, NT));
    p.tt_count = MODE == GROUPED ? 1 : (p.m + NT - 1) / NT;
    const long long tiles = MODE == GROUPED ? (long long)p.groups.max_tiles * p.row_tiles : (long long)((w.N + 127) / 128) * p.tt_count;   // at most
    auto kern = gemm_dense_kernel<NT, MODE>;
    const size_t smem = size_t(Ring<NT>::STAGES) * Ring<NT>::STAGE + Ring<NT>::EXCHANGE + 1024;
    FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(std::max(smem, size_t(120) * 1024))));
    if (NT <= 32 && tiles <= sms) {
        int parts = 0;
        FORGE_TRY((cluster_parts<NT, MODE>(tiles, p.nk, smem, &parts)));
        // a table stands in front of the first load: two CTAs per SM have twice as much on its way behind it
        if (MODE == GROUPED && NT <= 16 && parts == 1 && p.nk >= 8) parts = 2;
        if (parts > 0) {
            p.cluster = parts;
            FORGE_CUDA(launch_pdl_cluster(kern, dim3(unsigned(tiles * parts)), dim3(kThreads<NT>), parts, smem, st, mx, p));
            FORGE_LAUNCH_CHECK();
            return FORGE_OK;
        }
    }
    if constexpr (MODE == LISTED) { set_error("listed product: %lld tiles are too many", tiles); return FORGE_ERR_SHAPE; }
    if constexpr (MODE == GROUPED) {   // sixteen-token tiles: two CTAs fit an SM
        if (tiles * p.nk > INT32_MAX) { set_error("product in groups: %lld tiles of %d K steps are too many", tiles, p.nk); return FORGE_ERR_SHAPE; }
        FORGE_CUDA(launch_pdl(kern, dim3(unsigned(std::min((long long)sms * (NT <= 16 ? 2 : 1), tiles))), dim3(kThreads<NT>), smem, st, mx, p));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    }
    const int grid = int(std::max(1LL, std::min((long long)sms, std::max(NT >= 128 ? tiles : 1, tiles * p.nk / 4))));
    p.waves = NT >= 128 ? int(tiles / grid) : 0;   // a weight stream gains nothing from whole tiles in turn
    const long long units = (tiles - (long long)p.waves * grid) * p.nk;
    if (tiles * p.nk > INT32_MAX || (units + 1) * grid > INT32_MAX) { set_error("dense product: %lld tiles of %d K steps are too many", tiles, p.nk); return FORGE_ERR_SHAPE; }
    p.units = uint32_t(units);
    p.sharers = int(std::min((long long)grid, (units + 1) / 2));
    // leaving and adding shares costs about NT * kShareSteps / 256 K steps: where whole tiles are no dearer, every CTA takes at most one
    const long long rest = tiles - (long long)p.waves * grid;
    if (rest > 0 && rest <= grid && p.nk <= units / grid + NT * kShareSteps / 256) p.sharers = int(rest);
    FORGE_CUDA(launch_pdl(kern, dim3(grid), dim3(kThreads<NT>), smem, st, mx, p));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

// ------------------------------------------------------------------------------------------------ float32
// 64 rows x TM tokens per CTA, K in steps of 16, 256 threads.  Groups: blockIdx.y is a tile of the table, blockIdx.z its part of TM tokens.
struct F32Groups { GroupTable t; size_t group_w; size_t group_dst; };
template <int TM, bool GROUPS>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ w, int ldw, const float* __restrict__ x, int ldx, int K, int m, int N, const DenseOut out, const F32Groups gr) {
    constexpr int TN = 64, KS = 16, PT = TM / 16;   // tokens per thread
    __shared__ float sw[KS][TN + 4], sx[KS][TM + 4], s_scale[TM];
    const int tid = threadIdx.x, rr = (tid & 15) * 4, tt = (tid >> 4) * PT;
    const int row0 = blockIdx.x * TN;
    int tok0 = blockIdx.y * TM;
    const float* pair_w = nullptr;
    size_t dst_off = 0;
    if constexpr (GROUPS) {
        if (int(blockIdx.y) >= *gr.t.n) return;
        const GroupTile t = gr.t.tiles[blockIdx.y];
        if (int(blockIdx.z) * TM >= t.rows) return;
        tok0 = t.row0 + blockIdx.z * TM;
        m = t.row0 + t.rows;
        w += size_t(t.group) * gr.group_w;
        dst_off = size_t(t.group) * gr.group_dst;
        if (gr.t.weight) pair_w = gr.t.weight + t.w0 + blockIdx.z * TM;
    }
    for (int i = tid; i < TM; i += 256) {
        float sc = 1.f;
        if (out.scale.sums && tok0 + i < m) {
            const float* src = out.scale.sums + size_t(out.scale.row ? out.scale.row[tok0 + i] : tok0 + i) * out.scale.parts;
            float sum = 0.f;
            for (int j = 0; j < out.scale.parts; ++j) sum += src[j];
            sc = row_scale(out.scale, sum);
        }
        s_scale[i] = sc;
    }
    x += act_col(out, row0);
    float acc[4][PT];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < PT; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += KS) {
        for (int i = tid; i < TN * KS; i += 256) {
            const int r = i / KS, k = i % KS;
            sw[k][r] = row0 + r < N ? w[size_t(row0 + r) * ldw + k0 + k] : 0.f;
        }
        for (int i = tid; i < TM * KS; i += 256) {
            const int t = i / KS, k = i % KS;
            sx[k][t] = tok0 + t < m ? x[size_t(tok0 + t) * ldx + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            float a[4], b[PT];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = sw[k][rr + i];
#pragma unroll
            for (int j = 0; j < PT; ++j) b[j] = sx[k][tt + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < PT; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
    RowOut<float> g[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {   // four consecutive rows lie in one segment or past its end
        g[i] = row_out<float>(out, row0 + rr + i, (row0 + rr) & ~31);
        g[i].t += dst_off; g[i].f32 += dst_off;
    }
    const bool resid = g[0].kind == SEG_RESID;
#pragma unroll
    for (int j = 0; j < PT; ++j) {
        const size_t t = size_t(tok0 + tt + j);
        const bool live = int(t) < m;
        float v[4], sum = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = acc[i][j] * s_scale[tt + j] + g[i].add;
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (live && g[i].ok) {
                const Leave<float> n(out.seg[g[i].seg], g[i], row0 + rr + i, (row0 + rr) & ~31);
                const float xn = put_one(g[i], n, v[i], v[i | 1], pair_w ? pair_w[tt + j] : 1.f, t, 0.f, false, !(i & 1));
                sum = fmaf(xn, xn, sum);
            }
        if (__any_sync(0xffffffffu, resid)) {   // over the 32 rows of eight neighbouring lanes
            sum += __shfl_xor_sync(0xffffffffu, sum, 1);
            sum += __shfl_xor_sync(0xffffffffu, sum, 2);
            sum += __shfl_xor_sync(0xffffffffu, sum, 4);
            const After& a = out.seg[g[0].seg].after;
            if (live && resid && a.kind == AFTER_RMS && !(tid & 7)) a.sums[t * a.parts + (((row0 + rr) & ~31) - out.seg[g[0].seg].row0) / 32] = sum;
        }
    }
}

int32_t check_out(const DenseWeight& w, int rows, int act_ld, const DenseOut& out) {
    for (int i = 0; i < out.nseg; ++i) {
        const OutSeg& g = out.seg[i];
        const bool glu = g.kind == SEG_CLAMPED_GLU || g.kind == SEG_SILU_GLU, moved = g.act_col != (i ? out.seg[i - 1].act_col : 0);
        if (g.row0 % kSegAlign || g.row0 + g.rows > rows || (glu && (g.rows % 2 || g.add)) || (i && g.row0 < out.seg[i - 1].row0 + out.seg[i - 1].rows) ||
            g.act_col % kDensePad || g.act_col + w.K > act_ld || (i && moved && g.row0 % 128)) {
            set_error("dense product: bad output segment %d", i);
            return FORGE_ERR_SHAPE;
        }
    }
    return FORGE_OK;
}
int32_t check_weight(const DenseWeight& w, int act_ld) {
    if (w.K % kDensePad || act_ld < w.K || act_ld % kDensePad || w.pitch() % kDensePad || w.col0 % kDensePad || w.col0 + w.K > w.pitch()) { set_error("dense product: K=%d, activation rows of %d", w.K, act_ld); return FORGE_ERR_SHAPE; }
    return FORGE_OK;
}
int sm_count() {
    int dev = 0, sms = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    return std::min(sms, 148);
}

}  // namespace

// Load-time image of a bf16 matrix [N][K]: per 128 rows and 64 columns the 16 KB a stage of the ring holds, 128-byte rows with
// their 16-byte pieces at piece ^ (row & 7) (what a SWIZZLE_128B copy would write), K steps of a row tile one after another.
void dense_tile_image(void* dst, const void* rows, int N, int K) {
    const int nk = K / BK;
    const uint8_t* src = static_cast<const uint8_t*>(rows);
    uint8_t* out = static_cast<uint8_t*>(dst);
    memset(out, 0, dense_tile_bytes(N, K));
    for (int r = 0; r < N; ++r) {
        uint8_t* tile = out + size_t(r / 128) * nk * 16384 + size_t(r % 128) * 128;
        for (int kt = 0; kt < nk; ++kt)
            for (int c = 0; c < 8; ++c) memcpy(tile + size_t(kt) * 16384 + ((c ^ (r & 7)) << 4), src + (size_t(r) * K + kt * BK) * 2 + c * 16, 16);
    }
}

int32_t dense_gemm(const DenseWeight& w, const void* act, int act_ld, int m, const DenseOut& out, const DenseScratch& sc, int* err, cudaStream_t st) {
    if (m <= 0) return FORGE_OK;
    FORGE_TRY(check_weight(w, act_ld));
    FORGE_TRY(check_out(w, w.N, act_ld, out));
    if (w.dtype == FORGE_F32) {
        const float* wf = static_cast<const float*>(w.w) + w.col0;
        const float* xf = static_cast<const float*>(act);
        if (m <= 16) gemm_f32_kernel<16, false><<<dim3((w.N + 63) / 64, 1), 256, 0, st>>>(wf, w.pitch(), xf, act_ld, w.K, m, w.N, out, F32Groups{});
        else gemm_f32_kernel<64, false><<<dim3((w.N + 63) / 64, (m + 63) / 64), 256, 0, st>>>(wf, w.pitch(), xf, act_ld, w.K, m, w.N, out, F32Groups{});
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    }
    GemmParams p{};
    p.out = out; p.scale = out.scale; p.w = w.tiles; p.m = m; p.N = w.N; p.nk = w.K / BK; p.part = sc.part; p.tickets = sc.tickets; p.err = err;
    p.pitch = w.pitch() / BK; p.k_off = w.col0 / BK;
    const int sms = sm_count();
    int nt = group_tile_rows(m);
    const long long row_tiles = (w.N + 127) / 128;
    if (nt > 32 && row_tiles * ((m + nt - 1) / nt) * 2 <= sms) {   // wide tiles would leave SMs idle or share most of their steps: the width whose longest CTA moves least
        auto moved = [&](int n) {
            const long long tiles = row_tiles * ((m + n - 1) / n), steps = tiles > sms ? (tiles + sms - 1) / sms * p.nk : std::min<long long>(p.nk, tiles * p.nk / sms + n * kShareSteps / 256);
            return steps * (128 + n);
        };
        for (int n = nt / 2; n >= 32; n /= 2) if (moved(n) < moved(nt)) nt = n;
    }
    if (out.scale.sums && out.scale.parts > 1 && nt > kScaleRows) { set_error("dense product: %d tokens with scales in parts", m); return FORGE_ERR_SHAPE; }
    if (size_t((w.N + 127) / 128) * ((m + nt - 1) / nt) > sc.tickets_cap) { set_error("dense product: too many tiles for the ticket array"); return FORGE_ERR_SHAPE; }
    switch (nt) {
        case 16: return launch_dense<16, PLAIN>(w, act, act_ld, m, p, sms, st);
        case 32: return launch_dense<32, PLAIN>(w, act, act_ld, m, p, sms, st);
        case 64: return launch_dense<64, PLAIN>(w, act, act_ld, m, p, sms, st);
        case 128: return launch_dense<128, PLAIN>(w, act, act_ld, m, p, sms, st);
    }
    return launch_dense<256, PLAIN>(w, act, act_ld, m, p, sms, st);
}

int32_t dense_gemm_groups(const DenseWeight& w, const GroupShape& s, const GroupTable& t, const void* act, int act_ld, int act_rows, const DenseOut& out, int* err, cudaStream_t st) {
    if (act_rows <= 0 || t.max_tiles <= 0) return FORGE_OK;
    FORGE_TRY(check_weight(w, act_ld));
    FORGE_TRY(check_out(w, s.rows, act_ld, out));
    if (s.group_rows % 128 || s.group_cols % kDensePad) { set_error("product in groups: matrices %d rows and %d columns apart", s.group_rows, s.group_cols); return FORGE_ERR_SHAPE; }
    if (w.dtype == FORGE_F32) {
        const F32Groups g{t, size_t(s.group_rows) * w.pitch() + s.group_cols, s.group_dst};
        const float* wf = static_cast<const float*>(w.w) + w.col0;
        const float* xf = static_cast<const float*>(act);
        if (t.tile_rows <= 16) gemm_f32_kernel<16, true><<<dim3((s.rows + 63) / 64, t.max_tiles, 1), 256, 0, st>>>(wf, w.pitch(), xf, act_ld, w.K, 0, s.rows, out, g);
        else gemm_f32_kernel<64, true><<<dim3((s.rows + 63) / 64, t.max_tiles, (t.tile_rows + 63) / 64), 256, 0, st>>>(wf, w.pitch(), xf, act_ld, w.K, 0, s.rows, out, g);
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    }
    GemmParams p{};
    p.out = out; p.scale = out.scale; p.w = w.tiles; p.m = act_rows; p.N = s.rows; p.nk = w.K / BK; p.err = err;
    p.pitch = w.pitch() / BK; p.k_off = w.col0 / BK;
    p.groups = t; p.row_tiles = (s.rows + 127) / 128; p.group_dst = (long long)s.group_dst;
    p.group_images = uint32_t(s.group_rows / 128 * p.pitch + s.group_cols / BK);
    const int sms = sm_count();
    if (out.scale.sums && out.scale.parts > 1 && t.tile_rows > kScaleRows) { set_error("product in groups: tiles of %d tokens with scales in parts", t.tile_rows); return FORGE_ERR_SHAPE; }
    switch (t.tile_rows) {
        case 16: return launch_dense<16, GROUPED>(w, act, act_ld, act_rows, p, sms, st);
        case 32: return launch_dense<32, GROUPED>(w, act, act_ld, act_rows, p, sms, st);
        case 64: return launch_dense<64, GROUPED>(w, act, act_ld, act_rows, p, sms, st);
        case 128: return launch_dense<128, GROUPED>(w, act, act_ld, act_rows, p, sms, st);
        case 256: return launch_dense<256, GROUPED>(w, act, act_ld, act_rows, p, sms, st);
    }
    set_error("product in groups: tiles of %d rows", t.tile_rows);
    return FORGE_ERR_SHAPE;
}

bool dense_listed_supported(const DenseWeight& w, int m) { return w.dtype == FORGE_BF16 && m <= kScaleRows && (w.N + 127) / 128 <= 128; }

int32_t dense_gemm_listed(const DenseWeight& w, int k_fixed, int k_group, const GroupTable& t, const void* act, int act_ld, int m, const DenseOut& out, int* err, cudaStream_t st) {
    if (m <= 0) return FORGE_OK;
    FORGE_TRY(check_weight(w, act_ld));
    FORGE_TRY(check_out(w, w.N, act_ld, out));
    if (!dense_listed_supported(w, m) || k_fixed % BK || k_group % BK || k_fixed <= 0 || k_group <= 0 || w.ld || k_fixed + t.max_tiles * k_group > w.K) {
        set_error("listed product: %d rows, %d + %d * %d of %d columns", m, k_fixed, t.max_tiles, k_group, w.K);
        return FORGE_ERR_SHAPE;
    }
    GemmParams p{};
    p.out = out; p.scale = out.scale; p.w = w.tiles; p.m = m; p.N = w.N; p.err = err;
    p.pitch = w.K / BK; p.groups = t; p.k_fixed = k_fixed / BK; p.k_group = k_group / BK;
    p.nk = p.k_fixed + t.max_tiles * p.k_group;
    return m <= 16 ? launch_dense<16, LISTED>(w, act, act_ld, m, p, sm_count(), st) : launch_dense<32, LISTED>(w, act, act_ld, m, p, sm_count(), st);
}

}  // namespace forge
