// Selective scan and the convolution in front of it.  T is the model's type (bfloat16 or float32); states, step sizes, decays, B, C and sums are f32 in
// either.
//
// A channel's states are dealt to a group of G neighbouring lanes (a power of two), two, four or eight each; a token's read-out is added over the
// group.  Over a segment a CTA carries its channels token by token, with the inputs of the next tile of tokens on their way while one is worked off;
// the read-outs of sixteen tokens are added together, each step of the sum halving how many a lane holds.  Step sizes of bfloat16
// models come from a small product (inner values by channel) that the CTA forms for its channels, a tile of tokens ahead.
#include <algorithm>
#include <type_traits>

#include "mma.cuh"
#include "selective.cuh"

namespace forge {

namespace {

template <typename T> __device__ __forceinline__ float decay(float x) {   // exp2 of a negative number
    if constexpr (sizeof(T) == 4) return exp2f(x);
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// log(1 + u) with u = exp(-|v|) by its series where u is small (the fast logarithm has no relative accuracy near one)
__device__ __forceinline__ float fast_softplus(float v) {
    const float u = __expf(-fabsf(v));
    const float series = u * fmaf(u, fmaf(u, fmaf(u, fmaf(u, fmaf(u, -1.f / 6.f, 0.2f), -0.25f), 1.f / 3.f), -0.5f), 1.f);
    return fmaxf(v, 0.f) + (u < 0.0625f ? series : __logf(1.f + u));
}

// ------------------------------------------------------------------------------------------------ convolution
template <typename T>
__global__ void __launch_bounds__(256) conv_one_kernel(const SelectiveDims d, const SelectiveArgs a, const StepRows rows) {
    conv_one<T>(d, a, rows, blockIdx.y, blockIdx.x * 256 + threadIdx.x);
}

// A thread = one channel over a run of tokens; the first run's thread alone reads what the ring keeps of its channel and then leaves there the segment's
// last inputs.
constexpr int kRun = 32, kMaxTaps = 16;
template <typename T>
__global__ void __launch_bounds__(128) conv_segments_kernel(const SelectiveDims d, const SelectiveArgs a, const ScanSeg* __restrict__ segs) {
    const ScanSeg s = segs[blockIdx.z];
    const int t0 = blockIdx.x * kRun, c = blockIdx.y * 128 + threadIdx.x;
    if (t0 >= s.n || c >= d.inner) return;
    const T* in = static_cast<const T*>(a.in) + size_t(s.row0) * a.in_ld + c;
    T* out = static_cast<T*>(a.x) + size_t(s.row0) * a.x_ld + c;
    T* ring = static_cast<T*>(a.ring) + size_t(s.slot) * d.ring_values() + c;
    auto input = [&](int t) { return t >= 0 ? to_f(in[size_t(t) * a.in_ld]) : s.pos0 + t >= 0 ? to_f(ring[size_t((s.pos0 + t) % d.taps) * d.inner]) : 0.f; };
    const float add = a.conv_add[c];
    if (d.taps <= 4) {
        float w[4], past[3];   // past[2]: the token before
#pragma unroll
        for (int j = 0; j < 4; ++j) w[j] = j >= 4 - d.taps ? a.conv[size_t(j - (4 - d.taps)) * d.inner + c] : 0.f;
#pragma unroll
        for (int j = 0; j < 3; ++j) past[j] = j >= 4 - d.taps ? input(t0 - 3 + j) : 0.f;
#pragma unroll 8
        for (int t = t0; t < min(s.n, t0 + kRun); ++t) {
            const float now = to_f(in[size_t(t) * a.in_ld]);
            out[size_t(t) * a.x_ld] = to_t<T>(conv_act<T>(fmaf(w[3], now, fmaf(w[2], past[2], fmaf(w[1], past[1], fmaf(w[0], past[0], add))))));
            past[0] = past[1]; past[1] = past[2]; past[2] = now;
        }
    } else {
        for (int t = t0; t < min(s.n, t0 + kRun); ++t) {
            float v = add;
            for (int j = 0; j < d.taps; ++j) v = fmaf(a.conv[size_t(j) * d.inner + c], input(t - (d.taps - 1 - j)), v);
            out[size_t(t) * a.x_ld] = to_t<T>(conv_act<T>(v));
        }
    }
    if (blockIdx.x == 0)
        for (int t = max(0, s.n - d.taps); t < s.n; ++t) ring[size_t((s.pos0 + t) % d.taps) * d.inner] = in[size_t(t) * a.in_ld];
}

// The same for bfloat16 channels in whole 16-byte pieces and at most four taps: a thread carries eight channels over eight tokens.
constexpr int kRun8 = 8;
__global__ void __launch_bounds__(128) conv_segments8_kernel(const SelectiveDims d, const SelectiveArgs a, const ScanSeg* __restrict__ segs) {
    using bf16 = __nv_bfloat16;
    const ScanSeg s = segs[blockIdx.z];
    const int t0 = blockIdx.x * kRun8, c = (blockIdx.y * 128 + threadIdx.x) * 8;
    if (t0 >= s.n || c >= d.inner) return;
    const bf16* in = static_cast<const bf16*>(a.in) + size_t(s.row0) * a.in_ld + c;
    bf16* out = static_cast<bf16*>(a.x) + size_t(s.row0) * a.x_ld + c;
    bf16* ring = static_cast<bf16*>(a.ring) + size_t(s.slot) * d.ring_values() + c;
    uint4 now[kRun8];
#pragma unroll
    for (int i = 0; i < kRun8; ++i) now[i] = t0 + i < s.n ? *reinterpret_cast<const uint4*>(in + size_t(t0 + i) * a.in_ld) : make_uint4(0, 0, 0, 0);
    float w[4][8], past[3][8], add[8];   // past[2]: the token before
    load8(add, a.conv_add + c);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int e = 0; e < 8; ++e) w[j][e] = 0.f;
        if (j >= 4 - d.taps) load8(w[j], a.conv + size_t(j - (4 - d.taps)) * d.inner + c);
    }
#pragma unroll
    for (int j = 0; j < 3; ++j) {
        const int q = t0 - 3 + j, p = s.pos0 + q;
#pragma unroll
        for (int e = 0; e < 8; ++e) past[j][e] = 0.f;
        if (j >= 4 - d.taps && p >= 0) load8(past[j], q >= 0 ? in + size_t(q) * a.in_ld : ring + size_t(p % d.taps) * d.inner);
    }
#pragma unroll
    for (int i = 0; i < kRun8; ++i) {
        float v[8], y[8];
        load8(v, reinterpret_cast<const bf16*>(&now[i]));
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            y[e] = conv_act<bf16>(fmaf(w[3][e], v[e], fmaf(w[2][e], past[2][e], fmaf(w[1][e], past[1][e], fmaf(w[0][e], past[0][e], add[e])))));
            past[0][e] = past[1][e]; past[1][e] = past[2][e]; past[2][e] = v[e];
        }
        if (t0 + i < s.n) {
            put4(out + size_t(t0 + i) * a.x_ld, make_float4(y[0], y[1], y[2], y[3]));
            put4(out + size_t(t0 + i) * a.x_ld + 4, make_float4(y[4], y[5], y[6], y[7]));
        }
    }
    if (blockIdx.x == 0)
        for (int t = max(0, s.n - d.taps); t < s.n; ++t) *reinterpret_cast<uint4*>(ring + size_t((s.pos0 + t) % d.taps) * d.inner) = *reinterpret_cast<const uint4*>(in + size_t(t) * a.in_ld);
}

// ------------------------------------------------------------------------------------------------ recurrence
// (by one instruction for both they are slower here: its latency counts, with few warps per SM)
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return make_float2(a.x * b.x, a.y * b.y); }
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return make_float2(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y)); }
template <int SP> struct States {   // states sub * SP .. of a channel, in pairs
    float2 v[SP / 2];
    __device__ __forceinline__ void load(const float* p, int n) {   // n: how many there are
#pragma unroll
        for (int i = 0; i < SP; i += 2) v[i / 2] = make_float2(i < n ? p[i] : 0.f, i + 1 < n ? p[i + 1] : 0.f);
    }
    __device__ __forceinline__ void load_pairs(const float* p) {    // all of them, aligned
#pragma unroll
        for (int i = 0; i < SP; i += SP >= 4 ? 4 : 2)
            if constexpr (SP >= 4) { const float4 t = get4(p + i); v[i / 2] = make_float2(t.x, t.y); v[i / 2 + 1] = make_float2(t.z, t.w); }
            else v[0] = *reinterpret_cast<const float2*>(p);
    }
    __device__ __forceinline__ void store(float* p, int n) const {
#pragma unroll
        for (int i = 0; i < SP; i += 2) { if (i < n) p[i] = v[i / 2].x; if (i + 1 < n) p[i + 1] = v[i / 2].y; }
    }
    __device__ __forceinline__ void store_pairs(float* p) const {
#pragma unroll
        for (int i = 0; i < SP; i += SP >= 4 ? 4 : 2)
            if constexpr (SP >= 4) put4(p + i, make_float4(v[i / 2].x, v[i / 2].y, v[i / 2 + 1].x, v[i / 2 + 1].y));
            else *reinterpret_cast<float2*>(p) = v[0];
    }
};

constexpr int kDecodeThreads = 128;

template <typename T, int G, int SP>
__global__ void __launch_bounds__(kDecodeThreads) selective_decode_kernel(const SelectiveDims d, const SelectiveArgs a, const StepRows rows) {
    constexpr int CB = kDecodeThreads / G;
    const int r = blockIdx.y, sub = threadIdx.x % G, c = blockIdx.x * CB + threadIdx.x / G;
    const bool ok = c < d.inner;
    const int cc = ok ? c : 0, n0 = sub * SP, n = max(0, d.state - n0);
    const bool whole = d.state % 4 == 0 && n >= SP;
    pdl_trigger();
    const int pos = rows.pos[r], slot = state_slot(rows, r);
    float* at = a.state + (size_t(slot) * d.inner + cc) * d.state + n0;
    States<SP> S, A;
    if (whole) { A.load_pairs(a.a2 + size_t(cc) * d.state + n0); S.load_pairs(at); }
    else { A.load(a.a2 + size_t(cc) * d.state + n0, n); S.load(at, n); }
    if (pos == 0)
#pragma unroll
        for (int i = 0; i < SP / 2; ++i) S.v[i] = make_float2(0.f, 0.f);
    const float skip = a.skip[cc], add = a.dt_w ? a.dt_add[cc] : 0.f;
    pdl_wait();
    float dt;
    if (a.dt_w) {
        const T* w = static_cast<const T*>(a.dt_w) + size_t(cc) * a.low_k;
        const T* low = static_cast<const T*>(a.low) + size_t(r) * a.low_ld;
        float z = 0.f;
        for (int k = sub * 8; k < a.low_k; k += G * 8) {
            float wv[8], lv[8];
            load8(wv, w + k);
            load8(lv, low + k);
#pragma unroll
            for (int e = 0; e < 8; ++e) z = fmaf(wv[e], lv[e], z);
        }
#pragma unroll
        for (int o = 1; o < G; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        dt = softplus(z + add);
    } else dt = a.dt[size_t(r) * a.dt_ld + cc];
    const float x = to_f(static_cast<const T*>(a.x)[size_t(r) * a.x_ld + cc]), gate = to_f(static_cast<const T*>(a.gate)[size_t(r) * a.gate_ld + cc]), dx = dt * x;
    const float* bc = a.bc + size_t(r) * a.bc_ld + n0;
    States<SP> B, C;
    if (whole && a.bc_ld % 4 == 0) { B.load_pairs(bc); C.load_pairs(bc + d.state); }
    else { B.load(bc, n); C.load(bc + d.state, n); }
    float2 sum = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < SP / 2; ++i) {
        const float2 e = mul2(make_float2(dt, dt), A.v[i]);
        S.v[i] = fma2(make_float2(decay<T>(e.x), decay<T>(e.y)), S.v[i], mul2(make_float2(dx, dx), B.v[i]));
        sum = fma2(S.v[i], C.v[i], sum);
    }
    float y = sum.x + sum.y;
#pragma unroll
    for (int o = 1; o < G; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!ok) return;
    if (whole) S.store_pairs(at);
    else S.store(at, n);
    if (sub == 0) static_cast<T*>(a.out)[size_t(r) * a.out_ld + c] = to_t<T>(fmaf(skip, x, y) * gate * a.factor);
}

constexpr int kTile = 32, kHalf = 16, kGroup = 4;     // tokens whose inputs are in shared memory, whose read-outs are in registers, whose factors are formed together
// What a CTA holds in shared memory: three tiles of B and C, step sizes, x and gates, and (KS > 0) the step sizes' inner values, one of read-outs.
template <typename T, int TH, int G, int SP, int KS> struct ScanSmem {
    static constexpr int CB = TH / G, NP = G * SP, BC = kTile * NP, XC = kTile * CB, LD = KS * 16 + 8;
    static constexpr size_t X = (6 * size_t(BC) + 4 * XC) * 4, LOW = X + 6 * size_t(XC) * sizeof(T), BYTES = LOW + (KS ? 3 * size_t(kTile) * LD * 2 : 0);
};
// KS > 0: step sizes are formed here, from inner values of 16 KS columns, on the tensor cores.  ASYNC: all rows are copied in 16-byte pieces (bfloat16, channels in
// eights, states in fours).
template <typename T, int TH, int G, int SP, int KS, bool ASYNC>
__global__ void __launch_bounds__(TH) selective_scan_kernel(const SelectiveDims d, const SelectiveArgs a, const ScanSeg* __restrict__ segs) {
    using L = ScanSmem<T, TH, G, SP, KS>;
    constexpr int CB = L::CB, NP = L::NP, BC = L::BC, XC = L::XC;   // channels per CTA, padded states
    extern __shared__ __align__(16) unsigned char sm[];
    float* const s_bc = reinterpret_cast<float*>(sm);     // [3][B | C][kTile][NP]
    float* const s_dt = s_bc + 6 * BC;                    // [3][kTile][CB]
    float* const s_y = s_dt + 3 * XC;                     // [kTile][CB]
    T* const s_x = reinterpret_cast<T*>(sm + L::X);       // [3][x | gate][kTile][CB]
    const uint32_t s_low = uint32_t(__cvta_generic_to_shared(sm + L::LOW));
    const ScanSeg s = segs[blockIdx.y];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, sub = tid % G, cl = tid / G, c0 = blockIdx.x * CB, c = c0 + cl;
    const bool ok = c < d.inner;
    const int cc = ok ? c : 0, n0 = sub * SP, n = max(0, d.state - n0);
    const bool whole = d.state % 4 == 0 && n >= SP;
    float* at = a.state + (size_t(s.slot) * d.inner + cc) * d.state + n0;
    States<SP> S, A;
    if (whole) { A.load_pairs(a.a2 + size_t(cc) * d.state + n0); S.load_pairs(at); }
    else { A.load(a.a2 + size_t(cc) * d.state + n0, n); S.load(at, n); }
    if (s.pos0 == 0)
#pragma unroll
        for (int i = 0; i < SP / 2; ++i) S.v[i] = make_float2(0.f, 0.f);
    const T* x = static_cast<const T*>(a.x) + size_t(s.row0) * a.x_ld + c0;
    const T* gate = static_cast<const T*>(a.gate) + size_t(s.row0) * a.gate_ld + c0;
    const float* dt = a.dt + size_t(s.row0) * a.dt_ld + c0;
    const float* bc = a.bc + size_t(s.row0) * a.bc_ld;
    const T* low = static_cast<const T*>(a.low) + size_t(s.row0) * a.low_ld;
    T* out = static_cast<T*>(a.out) + size_t(s.row0) * a.out_ld + c0;
    // a tile's inputs into buffer `buf`; rows behind the segment become zeros
    auto fetch = [&](int t0, int buf) {
        if (ASYNC) {
            const uint32_t x_at = uint32_t(__cvta_generic_to_shared(s_x + buf * 2 * XC)), bc_at = uint32_t(__cvta_generic_to_shared(s_bc + buf * 2 * BC));
            constexpr int XP = CB >= 8 ? CB / 8 : 1, BP = NP / 4;   // pieces per row
            for (int i = tid; i < 2 * kTile * XP; i += TH) {
                const int which = i / (kTile * XP), t = i / XP % kTile, k = i % XP * 8;
                const bool in = t0 + t < s.n && c0 + k < d.inner;
                const T* src = which ? gate + size_t(in ? t0 + t : 0) * a.gate_ld : x + size_t(in ? t0 + t : 0) * a.x_ld;
                cp_async16(x_at + uint32_t(which * XC + t * CB + k) * 2, src + (in ? k : 0), in);
            }
            for (int i = tid; i < 2 * kTile * BP; i += TH) {
                const int which = i / (kTile * BP), t = i / BP % kTile, k = i % BP * 4;
                const bool in = t0 + t < s.n && k < d.state;
                cp_async16(bc_at + uint32_t(which * BC + t * NP + k) * 4, bc + size_t(in ? t0 + t : 0) * a.bc_ld + (in ? which * d.state + k : 0), in);
            }
        } else {
            for (int i = tid; i < XC; i += TH) {
                const int t = i / CB, k = i % CB;
                const bool in = t0 + t < s.n && c0 + k < d.inner;
                s_x[buf * 2 * XC + i] = in ? x[size_t(t0 + t) * a.x_ld + k] : to_t<T>(0.f);
                s_x[buf * 2 * XC + XC + i] = in ? gate[size_t(t0 + t) * a.gate_ld + k] : to_t<T>(0.f);
            }
            for (int i = tid; i < 2 * BC; i += TH) {
                const int which = i / BC, t = i % BC / NP, k = i % NP;
                s_bc[buf * 2 * BC + i] = t0 + t < s.n && k < d.state ? bc[size_t(t0 + t) * a.bc_ld + which * d.state + k] : 0.f;
            }
        }
        if constexpr (KS > 0) {
            for (int i = tid; i < kTile * KS * 2; i += TH) {
                const int t = i / (KS * 2), k = i % (KS * 2) * 8;
                const bool in = t0 + t < s.n;
                cp_async16(s_low + uint32_t((buf * kTile + t) * L::LD + k) * 2, low + size_t(in ? t0 + t : 0) * a.low_ld + k, in);
            }
        } else {
            for (int i = tid; i < XC; i += TH) {
                const int t = i / CB, k = i % CB;
                s_dt[buf * XC + i] = t0 + t < s.n && c0 + k < d.inner ? dt[size_t(t0 + t) * a.dt_ld + k] : 0.f;
            }
        }
        cp_commit();
    };
    // step sizes on the tensor cores: 16 tokens by eight channels per tile; a warp keeps its channels' weights
    constexpr int WARPS = TH / 32, NTILES = (CB + 7) / 8, PER = (NTILES + WARPS - 1) / WARPS;
    uint32_t wf[KS ? PER : 1][KS ? KS : 1][2];
    float dt_add[PER][2];
    if constexpr (KS > 0)
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int ch = (warp + WARPS * p) * 8 + (lane >> 2), lc = (lane & 3) * 2;
            const bool in = warp + WARPS * p < NTILES && c0 + ch < d.inner && ch < CB;
            const T* w = static_cast<const T*>(a.dt_w) + size_t(in ? c0 + ch : 0) * a.low_k;
#pragma unroll
            for (int k = 0; k < KS; ++k)
#pragma unroll
                for (int h = 0; h < 2; ++h) wf[p][k][h] = in ? *reinterpret_cast<const uint32_t*>(w + k * 16 + h * 8 + lc) : 0u;
#pragma unroll
            for (int e = 0; e < 2; ++e) { const int own = c0 + (warp + WARPS * p) * 8 + lc + e; dt_add[p][e] = own < d.inner ? a.dt_add[own] : 0.f; }
        }
    auto step_sizes = [&](int t0, int buf) {
        if constexpr (KS > 0) {
            const SmemMat m{s_low + uint32_t(buf * kTile * L::LD) * 2, L::LD};
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                if (warp + WARPS * p >= NTILES) continue;
                float z[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
                for (int k = 0; k < KS; ++k)
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        uint32_t fa[4];
                        m.a(fa, h * 16, k * 16, lane);
                        mma(z[h], fa, wf[p][k][0], wf[p][k][1]);
                    }
#pragma unroll
                for (int h = 0; h < 2; ++h)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int t = h * 16 + (lane >> 2) + (e >> 1) * 8, k = (warp + WARPS * p) * 8 + (lane & 3) * 2 + (e & 1);
                        if (k < CB) s_dt[buf * XC + t * CB + k] = t0 + t < s.n ? fast_softplus(z[h][e] + dt_add[p][e & 1]) : 0.f;
                    }
            }
        }
    };
    fetch(0, 0);
    const int own = tid % CB;      // the channel of all elements that this thread finishes (CB divides the threads)
    const float skip = c0 + own < d.inner ? a.skip[c0 + own] : 0.f;
    if constexpr (KS > 0) {
        cp_wait<0>();
        __syncthreads();
        step_sizes(0, 0);
    }
    if (s.n > kTile) fetch(kTile, 1);
    for (int t0 = 0, buf = 0, next_buf = 1, free_buf = 2; t0 < s.n; t0 += kTile) {
        cp_wait<0>();      // the tile behind this one, requested a tile ago
        __syncthreads();
        if (t0 + 2 * kTile < s.n) fetch(t0 + 2 * kTile, free_buf);
        if (t0 + kTile < s.n) step_sizes(t0 + kTile, next_buf);
        // tokens behind the segment have a step size of zero: they change nothing
#pragma unroll 1
        for (int h = 0; h < kTile && t0 + h < s.n; h += kHalf) {
            float y[kHalf];
            const float* b_at = s_bc + buf * 2 * BC + h * NP + n0;
            const float* d_at = s_dt + buf * XC + h * CB + cl;
            const T* x_at = s_x + buf * 2 * XC + h * CB + cl;
            struct Group { States<SP> e[kGroup], u[kGroup], c[kGroup]; } now, next;
            auto factors = [&](Group& g, int q0) {
#pragma unroll
                for (int q = 0; q < kGroup; ++q) {
                    const float step = d_at[(q0 + q) * CB], dx = step * to_f(x_at[(q0 + q) * CB]);
                    g.u[q].load_pairs(b_at + (q0 + q) * NP);
                    g.c[q].load_pairs(b_at + BC + (q0 + q) * NP);
#pragma unroll
                    for (int i = 0; i < SP / 2; ++i) {
                        g.u[q].v[i] = mul2(make_float2(dx, dx), g.u[q].v[i]);
                        const float2 e = mul2(make_float2(step, step), A.v[i]);
                        g.e[q].v[i] = make_float2(decay<T>(e.x), decay<T>(e.y));
                    }
                }
            };
            factors(now, 0);
#pragma unroll
            for (int q0 = 0; q0 < kHalf; q0 += kGroup) {
                if (q0 + kGroup < kHalf) factors(next, q0 + kGroup);
#pragma unroll
                for (int q = 0; q < kGroup; ++q) {
#pragma unroll
                    for (int i = 0; i < SP / 2; ++i) S.v[i] = fma2(now.e[q].v[i], S.v[i], now.u[q].v[i]);
                    float2 r = mul2(S.v[0], now.c[q].v[0]);
#pragma unroll
                    for (int i = 1; i < SP / 2; ++i) r = fma2(S.v[i], now.c[q].v[i], r);
                    y[q0 + q] = r.x + r.y;
                }
                now = next;
            }
            // sums over the group of lanes: with every bit of the lane's number it goes on with half of the tokens, as far as they go
            int left = kHalf, first = 0;
#pragma unroll
            for (int o = 1; o < G; o <<= 1) {
                if (left > 1) {
                    left >>= 1;
                    const bool up = sub & o;
#pragma unroll
                    for (int q = 0; q < kHalf / 2; ++q)
                        if (q < left) {
                            const float got = __shfl_xor_sync(0xffffffffu, up ? y[q] : y[q + left], o);
                            y[q] = (up ? y[q + left] : y[q]) + got;
                        }
                    if (up) first += left;
                } else y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
            }
            if (G <= kHalf || sub < kHalf)
#pragma unroll
                for (int q = 0; q < kHalf; ++q) if (q < left) s_y[(h + first + q) * CB + cl] = y[q];
        }
        __syncthreads();
        if (c0 + own < d.inner)
#pragma unroll 4
            for (int i = tid; i < XC; i += TH) {
                const int t = i / CB;
                const T *xs = s_x + buf * 2 * XC + i;
                if (t0 + t < s.n) out[size_t(t0 + t) * a.out_ld + own] = to_t<T>(fmaf(skip, to_f(xs[0]), s_y[i]) * (to_f(xs[XC]) * a.factor));
            }
        const int done = buf;
        buf = next_buf; next_buf = free_buf; free_buf = done;
    }
    if (ok) {
        if (whole) S.store_pairs(at);
        else S.store(at, n);
    }
}

// go(lanes per channel, states per lane)
template <typename F>
int32_t with_group(int states, F go) {
    using std::integral_constant;
    const integral_constant<int, 2> two;
    if (states <= 2) return go(integral_constant<int, 1>{}, two);
    if (states <= 4) return go(integral_constant<int, 2>{}, two);
    if (states <= 8) return go(integral_constant<int, 4>{}, two);
    if (states <= 16) return go(integral_constant<int, 8>{}, two);
    if (states <= 32) return go(integral_constant<int, 8>{}, integral_constant<int, 4>{});
    if (states <= 64) return go(integral_constant<int, 16>{}, integral_constant<int, 4>{});
    if (states <= 128) return go(integral_constant<int, 32>{}, integral_constant<int, 4>{});
    return go(integral_constant<int, 32>{}, integral_constant<int, 8>{});
}

template <typename T, int TH, int G, int SP, int KS, bool ASYNC>
int32_t launch_scan(const SelectiveDims& d, const SelectiveArgs& a, const SegTable& t, cudaStream_t st) {
    constexpr int CB = TH / G;
    constexpr size_t smem = ScanSmem<T, TH, G, SP, KS>::BYTES;
    auto kern = selective_scan_kernel<T, TH, G, SP, KS, ASYNC>;
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    kern<<<dim3((d.inner + CB - 1) / CB, t.n), TH, smem, st>>>(d, a, t.segs);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}
template <int TH, int G, int SP, int KS>
int32_t scan_steps(const SelectiveDims& d, const SelectiveArgs& a, const SegTable& t, cudaStream_t st) {
    using bf16 = __nv_bfloat16;
    const bool pieces = d.inner % 8 == 0 && TH / G >= 8 && a.x_ld % 8 == 0 && a.gate_ld % 8 == 0 && d.state % 4 == 0;
    return pieces ? launch_scan<bf16, TH, G, SP, KS, true>(d, a, t, st) : launch_scan<bf16, TH, G, SP, KS, false>(d, a, t, st);
}
template <int TH, int G, int SP>
int32_t scan_segments(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const SegTable& t, cudaStream_t st) {
    if (dtype == FORGE_F32) return launch_scan<float, TH, G, SP, 0, false>(d, a, t, st);
    if (!a.dt_w) return scan_steps<TH, G, SP, 0>(d, a, t, st);
    return a.low_k == 64 ? scan_steps<TH, G, SP, 4>(d, a, t, st) : a.low_k == 128 ? scan_steps<TH, G, SP, 8>(d, a, t, st) : scan_steps<TH, G, SP, 16>(d, a, t, st);
}

}  // namespace

bool selective_steps_inside(int dtype, int low_k) { return dtype == FORGE_BF16 && (low_k == 64 || low_k == 128 || low_k == 256); }
bool selective_supported(const SelectiveDims& d) { return d.state >= 1 && d.state <= 256 && d.taps >= 1 && d.taps <= kMaxTaps; }

int32_t selective_conv(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const StepRows& ones, const SegTable& t, cudaStream_t st) {
    auto go = [&](auto type) -> int32_t {
        using T = decltype(type);
        if (ones.n > 0) {
            FORGE_CUDA(launch_pdl(conv_one_kernel<T>, dim3((d.inner + 255) / 256, ones.n), dim3(256), 0, st, d, a, ones));
            FORGE_LAUNCH_CHECK();
        }
        if (t.n > 0) {
            const bool eight = std::is_same<T, __nv_bfloat16>::value && d.inner % 8 == 0 && a.in_ld % 8 == 0 && a.x_ld % 8 == 0 && d.taps <= 4;
            if (eight) conv_segments8_kernel<<<dim3((t.max_n + kRun8 - 1) / kRun8, (d.inner + 1023) / 1024, t.n), 128, 0, st>>>(d, a, t.segs);
            else conv_segments_kernel<T><<<dim3((t.max_n + kRun - 1) / kRun, (d.inner + 127) / 128, t.n), 128, 0, st>>>(d, a, t.segs);
            FORGE_LAUNCH_CHECK();
        }
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int32_t selective_decode(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const StepRows& ones, cudaStream_t st) {
    if (ones.n <= 0) return FORGE_OK;
    return with_group(d.state, [&](auto g, auto sp) -> int32_t {
        constexpr int G = decltype(g)::value, SP = decltype(sp)::value, CB = kDecodeThreads / G;
        auto kern = dtype == FORGE_F32 ? selective_decode_kernel<float, G, SP> : selective_decode_kernel<__nv_bfloat16, G, SP>;
        FORGE_CUDA(launch_pdl(kern, dim3((d.inner + CB - 1) / CB, ones.n), dim3(kDecodeThreads), 0, st, d, a, ones));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    });
}

int32_t selective_segments(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const SegTable& t, cudaStream_t st) {
    if (t.n <= 0) return FORGE_OK;
    return with_group(d.state, [&](auto g, auto sp) -> int32_t { return scan_segments<(decltype(g)::value >= 8 ? 256 : 128), decltype(g)::value, decltype(sp)::value>(d, dtype, a, t, st); });
}

}  // namespace forge
