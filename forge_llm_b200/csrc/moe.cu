// Routing of tokens to experts, in f32.  Everything is dealt out in a fixed order (no atomics): the same step gives the same bits.
#include <algorithm>

#include "moe.cuh"

namespace forge {

namespace {

__global__ void __launch_bounds__(1024) route_few_kernel(const RouterDims d, const float* logits, int rows, const RouteTables t) {
    extern __shared__ float s_w[];
    route_few_clear(d, s_w);
    pdl_trigger();
    pdl_wait();
    route_few_rows(d, logits, rows, t, s_w);
}

__global__ void __launch_bounds__(256) choose_kernel(const RouterDims d, const float* __restrict__ logits, int rows, const RouteTables t) {
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (r >= rows) return;
    choose(logits + size_t(r) * d.choices(), d, t.expert + size_t(r) * d.top, t.weight + size_t(r) * d.top);
    if (d.identity && (threadIdx.x & 31) == 0) {
        float passed = 0.f;
        for (int k = 0; k < d.top; ++k) if (t.expert[size_t(r) * d.top + k] >= d.experts) passed += t.weight[size_t(r) * d.top + k];
        t.passed[r] = passed;
    }
}

// One CTA.  Every warp owns a run of pairs; a pair's place among its expert's is what earlier warps, earlier pairs of the warp and
// earlier lanes hold.
__global__ void __launch_bounds__(1024) slots_kernel(const RouterDims d, int rows, int tile_rows, const RouteTables t) {
    extern __shared__ int s_cnt[];                                  // [32][experts]
    __shared__ int total[kMaxExperts], start[kMaxExperts], tile0[kMaxExperts];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = d.experts, pairs = rows * d.top;
    const int per = ((pairs + 31) / 32 + 31) & ~31, p0 = warp * per, p1 = min(pairs, p0 + per);
    int* cnt = s_cnt + warp * E;
    for (int i = threadIdx.x; i < 32 * E; i += 1024) s_cnt[i] = 0;
    __syncthreads();
    for (int p = p0; p < p1; p += 32) {
        int e = p + lane < p1 ? t.expert[p + lane] : -1;
        if (e >= E) e = -1;     // passed on: no slot
        const uint32_t same = __match_any_sync(0xffffffffu, e);
        if (e >= 0 && lane == __ffs(same) - 1) cnt[e] += __popc(same);
        __syncwarp();
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += 1024) {
        int sum = 0;
        for (int w = 0; w < 32; ++w) { const int c = s_cnt[w * E + e]; s_cnt[w * E + e] = sum; sum += c; }
        total[e] = sum;
    }
    __syncthreads();
    if (warp == 0) {   // where an expert's slots and tiles begin
        int slots = 0, tiles = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane, c = e < E ? total[e] : 0, n = (c + tile_rows - 1) / tile_rows;
            int sc = c, sn = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int a = __shfl_up_sync(0xffffffffu, sc, o), b = __shfl_up_sync(0xffffffffu, sn, o);
                if (lane >= o) { sc += a; sn += b; }
            }
            if (e < E) { start[e] = slots + sc - c; tile0[e] = tiles + sn - n; }
            slots += __shfl_sync(0xffffffffu, sc, 31);
            tiles += __shfl_sync(0xffffffffu, sn, 31);
        }
        if (lane == 0) *t.n_tiles = tiles;
        for (int i = slots + lane; i < pairs; i += 32) { t.row[i] = 0; t.slot_weight[i] = 0.f; }   // slots that nobody took are gathered, too
    }
    __syncthreads();
    for (int e = warp; e < E; e += 32)
        for (int i = lane; i * tile_rows < total[e]; i += 32) {
            const int at = start[e] + i * tile_rows;
            t.tiles[tile0[e] + i] = GroupTile{d.always + e, at, min(tile_rows, total[e] - i * tile_rows), at};
        }
    for (int p = p0; p < p1; p += 32) {
        const int i = p + lane;
        int e = i < p1 ? t.expert[i] : -1;
        if (e >= E) { e = -1; t.slot[i] = -1; }
        const uint32_t same = __match_any_sync(0xffffffffu, e);
        if (e >= 0) {
            const int slot = start[e] + cnt[e] + __popc(same & ((1u << lane) - 1));
            t.slot[i] = slot;
            t.row[slot] = i / d.top;
            t.slot_weight[slot] = t.weight[i];
        }
        __syncwarp();
        if (e >= 0 && lane == __ffs(same) - 1) cnt[e] += __popc(same);
        __syncwarp();
    }
}

template <typename T>
__global__ void __launch_bounds__(256) add_experts_kernel(float* __restrict__ x, const float* __restrict__ y, const int32_t* __restrict__ slot, int top, int width, const After after) {
    const int r = blockIdx.x;
    if (width % 4 == 0) {   // four columns per thread
        for (int c0 = blockIdx.y * 1024; c0 < width; c0 += gridDim.y * 1024) {
            const int c = c0 + threadIdx.x * 4;
            const bool ok = c < width;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (ok) {
                v = get4(x + size_t(r) * width + c);
#pragma unroll 2
                for (int k = 0; k < top; ++k) v = add4(v, get4(y + size_t(slot[size_t(r) * top + k]) * width + c));
            }
            v = leave_four<T>(after, v, size_t(r), size_t(width), c, ok);
            if (ok) put4(x + size_t(r) * width + c, v);
        }
        return;
    }
    for (int c0 = blockIdx.y * 256; c0 < width; c0 += gridDim.y * 256) {
        const int c = c0 + threadIdx.x;
        const bool ok = c < width;
        float v = ok ? x[size_t(r) * width + c] : 0.f;
        for (int k = 0; k < top; ++k) v += ok ? y[size_t(slot[size_t(r) * top + k]) * width + c] : 0.f;
        v = leave_value<T>(after, v, size_t(r), size_t(width), c, ok);
        if (ok) x[size_t(r) * width + c] = v;
    }
}

// A CTA per row.  NV: pieces of four columns per thread (rows of up to 1024 NV); 0: any width.
template <typename T, int NV, bool ROUTE>
__global__ void __launch_bounds__(256) add_normed_kernel(float* x, const float* y, int width, float eps, float gain, const MixtureSum mix, const After after, const RouteBehind route) {
    extern __shared__ __align__(16) float s_row[];     // routing: the row, its logits, then the tables
    __shared__ float red[8];
    __shared__ int s_last;
    const int r = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* xr = x + size_t(r) * width;
    const float* yr = y + size_t(r) * width;
    auto factor = [&](float ss) {
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) ss += red[w];
        return gain / sqrtf(ss / float(width) + eps);
    };
    pdl_trigger();
    // routing, a warp per choice: the first one's weights are on their way before the wait
    constexpr int KEEP = ROUTE ? NV * 4 : 1;     // pieces of eight columns per lane
    uint4 held[KEEP], held2[NV <= 2 ? KEEP : 1];
    __shared__ float s_corr[ROUTE ? 64 : 1];
    const T* own_w = static_cast<const T*>(route.w) + size_t(warp) * route.ld;
    if constexpr (ROUTE) {
        if (warp < route.d.choices())
#pragma unroll
            for (int i = 0; i < KEEP; ++i) { const int c = (lane + 32 * i) * 8; held[i] = c < width ? *reinterpret_cast<const uint4*>(own_w + c) : make_uint4(0, 0, 0, 0); }
        if constexpr (NV <= 2) {
            if (warp + 8 < route.d.choices())
#pragma unroll
                for (int i = 0; i < KEEP; ++i) { const int c = (lane + 32 * i) * 8; held2[i] = c < width ? *reinterpret_cast<const uint4*>(own_w + size_t(8) * route.ld + c) : make_uint4(0, 0, 0, 0); }
        }
        if (route.d.correction && int(threadIdx.x) < route.d.choices()) s_corr[threadIdx.x] = route.d.correction[threadIdx.x];
    }
    pdl_wait();
    const float passed = mix.passed ? mix.passed[r] : 0.f;
    if constexpr (NV > 0) {
        float4 vx[NV], vy[NV];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int c = 4 * (threadIdx.x + 256 * j);
            const bool ok = c < width;
            vx[j] = ok ? get4(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            vy[j] = ok ? get4(yr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (mix.e)
            for (int k = 0; k < mix.top; ++k) {
                const int s = mix.slot[size_t(r) * mix.top + k];
                if (s < 0) continue;
#pragma unroll
                for (int j = 0; j < NV; ++j) {
                    const int c = 4 * (threadIdx.x + 256 * j);
                    if (c < width) vy[j] = add4(vy[j], get4(mix.e + size_t(s) * width + c));
                }
            }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            float4& v = vy[j];
            v = make_float4(fmaf(passed, vx[j].x, v.x), fmaf(passed, vx[j].y, v.y), fmaf(passed, vx[j].z, v.z), fmaf(passed, vx[j].w, v.w));
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
        const float f = factor(ss);
#pragma unroll
        for (int j = 0; j < NV; ++j) {   // whole warps stay
            const int c = 4 * (threadIdx.x + 256 * j);
            const bool ok = c < width;
            float4 v = make_float4(fmaf(f, vy[j].x, vx[j].x), fmaf(f, vy[j].y, vx[j].y), fmaf(f, vy[j].z, vx[j].z), fmaf(f, vy[j].w, vx[j].w));
            v = leave_four<T>(after, v, size_t(r), size_t(width), c, ok);
            if (ok) put4(xr + c, v);
            if (ROUTE && ok) put4(s_row + c, v);
        }
        if constexpr (ROUTE) {
            const int C = route.d.choices(), rows = gridDim.x;
            float* s_z = s_row + 1024 * NV;
            for (int i = width + threadIdx.x; i < 1024 * NV; i += 256) s_row[i] = 0.f;
            __syncthreads();
            for (int e = warp; e < C; e += 8) {
                float z = 0.f;
#pragma unroll
                for (int i = 0; i < KEEP; ++i) {
                    const int c = (lane + 32 * i) * 8;
                    float w[8], v[8];
                    if (NV <= 2 && e == warp + 8) held[i] = held2[NV <= 2 ? i : 0];
                    else if (e != warp) held[i] = c < width ? *reinterpret_cast<const uint4*>(own_w + size_t(e - warp) * route.ld + c) : make_uint4(0, 0, 0, 0);
                    load8(w, reinterpret_cast<const T*>(&held[i]));
                    load8(v, s_row + c);
#pragma unroll
                    for (int k = 0; k < 8; ++k) z = fmaf(w[k], v[k], z);
                }
                z = warp_sum(z);
                if (lane == 0) s_z[e] = z;
            }
            float* s_w = s_z + ((C + 3) & ~3);
            int32_t* s_expert = reinterpret_cast<int32_t*>(s_w + route.d.groups() * (kScaleRows + 1));      // the row's choice, in the end of all rows
            const int top = route.d.top;
            float* s_weight = reinterpret_cast<float*>(s_expert + kScaleRows * top);
            for (int i = threadIdx.x; i < route.d.groups() * (kScaleRows + 1); i += 256) s_w[i] = 0.f;
            __syncthreads();
            if (warp == 0) {
                RouterDims rd = route.d;
                if (rd.correction) rd.correction = s_corr;
                if (C <= 32) choose<1>(s_z, rd, s_expert, s_weight);
                else choose<2>(s_z, rd, s_expert, s_weight);
            }
            if (rows > 1) {     // the last row makes the tables
                if (warp == 0) {
                    for (int k = lane; k < top; k += 32) { route.t.expert[r * top + k] = s_expert[k]; route.t.weight[r * top + k] = s_weight[k]; }
                    __threadfence();
                    __syncwarp();
                    if (lane == 0) {
                        s_last = atomicAdd(route.ticket, 1) == rows - 1;
                        if (s_last) *route.ticket = 0;
                        __threadfence();
                    }
                }
                __syncthreads();
                if (!s_last) return;
                for (int i = threadIdx.x; i < rows * top; i += 256) { s_expert[i] = __ldcg(route.t.expert + i); s_weight[i] = __ldcg(route.t.weight + i); }
            }
            __syncthreads();
            route_few_tables(route.d, rows, route.t, s_expert, s_weight, s_w);
        }
    } else {
        auto value = [&](int c) {
            float v = yr[c];
            if (mix.e)
                for (int k = 0; k < mix.top; ++k) {
                    const int s = mix.slot[size_t(r) * mix.top + k];
                    if (s >= 0) v += mix.e[size_t(s) * width + c];
                }
            return fmaf(passed, xr[c], v);
        };
        float ss = 0.f;
        for (int c = threadIdx.x; c < width; c += 256) { const float v = value(c); ss = fmaf(v, v, ss); }
        const float f = factor(ss);
        for (int c0 = 0; c0 < width; c0 += 256) {
            const int c = c0 + threadIdx.x;
            const bool ok = c < width;
            float v = ok ? fmaf(f, value(c), xr[c]) : 0.f;
            v = leave_value<T>(after, v, size_t(r), size_t(width), c, ok);
            if (ok) xr[c] = v;
        }
    }
}

size_t align16(size_t n) { return (n + 15) & ~size_t(15); }

}  // namespace

size_t route_bytes(const RouterDims& d, int rows) {
    const size_t pairs = size_t(rows) * d.top;
    return 5 * align16(pairs * 4) + align16(size_t(rows) * 4) + size_t(d.groups()) * kScaleRows * 4 + (pairs + d.groups() + d.experts) * sizeof(GroupTile) + 16;
}
GroupTable few_table(const RouterDims& d, int rows, const RouteTables& t) {
    return GroupTable{t.tiles, t.n_tiles, d.always + int(std::min<long long>(d.experts, (long long)rows * d.top)), rows <= 16 ? 16 : 32, t.row_weight};
}
GroupTable listed_table(const RouterDims& d, int rows, const RouteTables& t) {
    GroupTable l = few_table(d, rows, t);
    l.tiles = t.listed; l.n = t.n_listed; l.max_tiles -= d.always;
    return l;
}
RouteTables route_tables(void* p, const RouterDims& d, int rows) {
    const size_t pairs = align16(size_t(rows) * d.top * 4);
    char* b = static_cast<char*>(p);
    auto take = [&](size_t n) { char* at = b; b += n; return at; };
    RouteTables t;
    t.n_tiles = reinterpret_cast<int32_t*>(take(16));
    t.n_listed = t.n_tiles + 1;
    t.tiles = reinterpret_cast<GroupTile*>(take((size_t(rows) * d.top + d.groups()) * sizeof(GroupTile)));
    t.listed = reinterpret_cast<GroupTile*>(take(size_t(d.experts) * sizeof(GroupTile)));
    t.row_weight = reinterpret_cast<float*>(take(size_t(d.groups()) * kScaleRows * 4));
    t.expert = reinterpret_cast<int32_t*>(take(pairs)); t.weight = reinterpret_cast<float*>(take(pairs)); t.slot = reinterpret_cast<int32_t*>(take(pairs));
    t.row = reinterpret_cast<int32_t*>(take(pairs)); t.slot_weight = reinterpret_cast<float*>(take(pairs));
    t.passed = reinterpret_cast<float*>(take(align16(size_t(rows) * 4)));
    return t;
}

int32_t route_few(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st) {
    if (rows > kScaleRows || d.choices() > kMaxExperts) { set_error("routing: %d rows, %d experts", rows, d.experts); return FORGE_ERR_SHAPE; }
    *out = few_table(d, rows, t);
    const size_t smem = route_few_smem(d);
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(route_few_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    FORGE_CUDA(launch_pdl(route_few_kernel, dim3(1), dim3(1024), smem, st, d, logits, rows, t));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

int32_t route_slots(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st) {
    if (d.choices() > kMaxExperts || (long long)rows * d.top > (1 << 30)) { set_error("routing: %d rows, %d experts", rows, d.experts); return FORGE_ERR_SHAPE; }
    const int pairs = rows * d.top, tile_rows = group_tile_rows((pairs + d.experts - 1) / d.experts);
    *out = GroupTable{t.tiles, t.n_tiles, std::min(pairs, pairs / tile_rows + d.experts), tile_rows, t.slot_weight};
    choose_kernel<<<(rows + 7) / 8, 256, 0, st>>>(d, logits, rows, t);
    FORGE_LAUNCH_CHECK();
    FORGE_CUDA(cudaFuncSetAttribute(slots_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 32 * kMaxExperts * 4));
    slots_kernel<<<1, 1024, size_t(32) * d.experts * 4, st>>>(d, rows, tile_rows, t);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

int32_t add_experts(float* x, const float* y, const RouterDims& d, const RouteTables& t, int rows, int width, const After& after, int dtype, cudaStream_t st) {
    if (rows <= 0) return FORGE_OK;
    const dim3 grid(rows, rows < 64 ? (width + 255) / 256 : 1);
    if (dtype == FORGE_F32) add_experts_kernel<float><<<grid, 256, 0, st>>>(x, y, t.slot, d.top, width, after);
    else add_experts_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(x, y, t.slot, d.top, width, after);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

// (a CTA per row reads all of the router; what it holds on to lies in registers)
static int norm_pieces(int width) { return width <= 1024 ? 1 : width <= 2048 ? 2 : width <= 4096 ? 4 : 8; }
static size_t route_behind_smem(const RouterDims& d, int width) { return size_t(1024) * norm_pieces(width) * 4 + size_t((d.choices() + 3) & ~3) * 4 + route_few_smem(d) + size_t(kScaleRows) * d.top * 8; }
bool route_behind_supported(const RouterDims& d, int width, int rows) { return rows <= kScaleRows && width % 8 == 0 && width <= 4096 && d.choices() <= 64 && route_behind_smem(d, width) <= 200 * 1024; }

int32_t add_normed(float* x, const float* y, int rows, int width, float eps, float gain, const MixtureSum& mix, const After& after, const RouteBehind* route, int dtype, cudaStream_t st) {
    if (rows <= 0) return FORGE_OK;
    const bool wide = width % 4 != 0 || after.ld % 4 != 0 || after.col2 % 4 != 0 || width > 8192;
    if (route && (wide || dtype != FORGE_BF16 || route->ld % 8 || !route_behind_supported(route->d, width, rows))) { set_error("routing behind a norm: %d rows of %d", rows, width); return FORGE_ERR_SHAPE; }
    auto go = [&](auto type) -> int32_t {
        using T = decltype(type);
        const int nv = norm_pieces(width);
        auto kern = wide ? add_normed_kernel<T, 0, false> : nv == 1 ? add_normed_kernel<T, 1, false> : nv == 2 ? add_normed_kernel<T, 2, false> : nv == 4 ? add_normed_kernel<T, 4, false> : add_normed_kernel<T, 8, false>;
        if (route) kern = nv == 1 ? add_normed_kernel<__nv_bfloat16, 1, true> : nv == 2 ? add_normed_kernel<__nv_bfloat16, 2, true> : add_normed_kernel<__nv_bfloat16, 4, true>;
        const size_t smem = route ? route_behind_smem(route->d, width) : 0;
        if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        FORGE_CUDA(launch_pdl(kern, dim3(rows), dim3(256), smem, st, x, y, width, eps, gain, mix, after, route ? *route : RouteBehind{}));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace forge
