// Selective scan and the convolution in front of it.  T is the model's type (bfloat16 or float32); states, step sizes, decays, B, C and sums are f32 in
// either.
//
// A channel's states are dealt to a group of G neighbouring lanes (a power of two), four or eight each; a token's read-out is added over the
// group.  Over a segment a CTA carries its channels token by token, with the inputs of the next tile of tokens on their way while one is worked off;
// the read-outs of sixteen tokens are added together, each step of the sum halving how many a lane holds.
#include <algorithm>
#include <type_traits>

#include "selective.cuh"

namespace forge {

namespace {

template <typename T> __device__ __forceinline__ float decay(float x) {   // exp2 of a negative number
    if constexpr (sizeof(T) == 4) return exp2f(x);
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
template <typename T> __device__ __forceinline__ float conv_act(float v) {
    if constexpr (sizeof(T) == 4) return silu(v);
    return __fdividef(v, 1.0f + __expf(-v));   // far inside a bfloat16 rounding
}

// ------------------------------------------------------------------------------------------------ convolution
template <typename T>
__global__ void __launch_bounds__(256) conv_one_kernel(const SelectiveDims d, const SelectiveArgs a, const StepRows rows) {
    const int r = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    pdl_trigger();
    const int pos = rows.pos[r], slot = state_slot(rows, r);
    T* ring = static_cast<T*>(a.ring) + size_t(slot) * d.ring_values() + c;
    float v = 0.f, w = 0.f;
    if (c < d.inner) {   // what earlier steps have left
        v = a.conv_add[c];
        w = a.conv[size_t(d.taps - 1) * d.inner + c];
        for (int j = 0; j < d.taps - 1; ++j) {
            const int p = pos - (d.taps - 1 - j);
            if (p >= 0) v = fmaf(a.conv[size_t(j) * d.inner + c], to_f(ring[size_t(p % d.taps) * d.inner]), v);
        }
    }
    pdl_wait();
    if (c >= d.inner) return;
    const T in = static_cast<const T*>(a.in)[size_t(r) * a.in_ld + c];
    static_cast<T*>(a.x)[size_t(r) * a.x_ld + c] = to_t<T>(conv_act<T>(fmaf(w, to_f(in), v)));
    ring[size_t(pos % d.taps) * d.inner] = in;
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
template <int SP> struct States {   // states sub * SP .. of a channel
    float v[SP];
    __device__ __forceinline__ void load(const float* p, int n, bool whole) {   // n: how many there are
        if (whole) {
#pragma unroll
            for (int i = 0; i < SP; i += 4) { const float4 t = get4(p + i); v[i] = t.x; v[i + 1] = t.y; v[i + 2] = t.z; v[i + 3] = t.w; }
        } else
#pragma unroll
            for (int i = 0; i < SP; ++i) v[i] = i < n ? p[i] : 0.f;
    }
    __device__ __forceinline__ void store(float* p, int n, bool whole) const {
        if (whole) {
#pragma unroll
            for (int i = 0; i < SP; i += 4) put4(p + i, make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]));
        } else
#pragma unroll
            for (int i = 0; i < SP; ++i) if (i < n) p[i] = v[i];
    }
};

constexpr int kScanThreads = 128;

template <typename T, int G, int SP>
__global__ void __launch_bounds__(kScanThreads) selective_decode_kernel(const SelectiveDims d, const SelectiveArgs a, const StepRows rows) {
    constexpr int CB = kScanThreads / G;
    const int r = blockIdx.y, sub = threadIdx.x % G, c = blockIdx.x * CB + threadIdx.x / G;
    const bool ok = c < d.inner;
    const int cc = ok ? c : 0, n0 = sub * SP, n = max(0, d.state - n0);
    const bool whole = d.state % 4 == 0 && n >= SP;
    pdl_trigger();
    const int pos = rows.pos[r], slot = state_slot(rows, r);
    float* at = a.state + (size_t(slot) * d.inner + cc) * d.state + n0;
    States<SP> S, A;
    A.load(a.a2 + size_t(cc) * d.state + n0, n, whole);
    if (pos > 0) S.load(at, n, whole);
    else
#pragma unroll
        for (int i = 0; i < SP; ++i) S.v[i] = 0.f;
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
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < SP; ++i) {
        const float b = i < n ? bc[i] : 0.f, cv = i < n ? bc[d.state + i] : 0.f;
        S.v[i] = fmaf(decay<T>(dt * A.v[i]), S.v[i], dx * b);
        y = fmaf(S.v[i], cv, y);
    }
#pragma unroll
    for (int o = 1; o < G; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!ok) return;
    S.store(at, n, whole);
    if (sub == 0) static_cast<T*>(a.out)[size_t(r) * a.out_ld + c] = to_t<T>(fmaf(skip, x, y) * gate * a.factor);
}

constexpr int kTile = 32, kHalf = 16;     // tokens whose inputs are in shared memory, and whose read-outs are in registers
template <typename T, int G, int SP>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(const SelectiveDims d, const SelectiveArgs a, const ScanSeg* __restrict__ segs) {
    constexpr int CB = kScanThreads / G, NP = G * SP, BC = kTile * NP, XC = kTile * CB;   // channels per CTA, padded states
    constexpr int LB = (2 * BC + kScanThreads - 1) / kScanThreads, LX = (XC + kScanThreads - 1) / kScanThreads;
    extern __shared__ __align__(16) float sm[];
    float* s_bc = sm;                                             // [B | C][kTile][NP]
    float2* s_dx = reinterpret_cast<float2*>(s_bc + 2 * BC);      // [kTile][CB]: step size, times x
    float* s_y = reinterpret_cast<float*>(s_dx + XC);             // [kTile][CB]
    const ScanSeg s = segs[blockIdx.y];
    const int tid = threadIdx.x, sub = tid % G, cl = tid / G, c0 = blockIdx.x * CB, c = c0 + cl;
    const bool ok = c < d.inner;
    const int cc = ok ? c : 0, n0 = sub * SP, n = max(0, d.state - n0);
    const bool whole = d.state % 4 == 0 && n >= SP;
    float* at = a.state + (size_t(s.slot) * d.inner + cc) * d.state + n0;
    States<SP> S, A;
    A.load(a.a2 + size_t(cc) * d.state + n0, n, whole);
    if (s.pos0 > 0) S.load(at, n, whole);
    else
#pragma unroll
        for (int i = 0; i < SP; ++i) S.v[i] = 0.f;
    const T* x = static_cast<const T*>(a.x) + size_t(s.row0) * a.x_ld + c0;
    const T* gate = static_cast<const T*>(a.gate) + size_t(s.row0) * a.gate_ld + c0;
    const float* dt = a.dt + size_t(s.row0) * a.dt_ld + c0;
    const float* bc = a.bc + size_t(s.row0) * a.bc_ld;
    T* out = static_cast<T*>(a.out) + size_t(s.row0) * a.out_ld + c0;
    float rb[LB], rd[LX];
    T rg[LX], rx[LX];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int j = 0; j < LB; ++j) {
            const int i = tid + kScanThreads * j, which = i / BC, t = i % BC / NP, k = i % NP;
            rb[j] = i < 2 * BC && t0 + t < s.n && k < d.state ? bc[size_t(t0 + t) * a.bc_ld + which * d.state + k] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < LX; ++j) {
            const int i = tid + kScanThreads * j, t = i / CB, k = i % CB;
            const bool in = i < XC && t0 + t < s.n && c0 + k < d.inner;
            rd[j] = in ? dt[size_t(t0 + t) * a.dt_ld + k] : 0.f;
            rx[j] = in ? x[size_t(t0 + t) * a.x_ld + k] : to_t<T>(0.f);
            rg[j] = in ? gate[size_t(t0 + t) * a.gate_ld + k] : to_t<T>(0.f);
        }
    };
    fetch(0);
    const int own = tid % CB;      // the channel of all elements that this thread fetches and finishes (CB divides the threads)
    const float skip = c0 + own < d.inner ? a.skip[c0 + own] : 0.f;
    for (int t0 = 0; t0 < s.n; t0 += kTile) {
        float cx[LX], cg[LX];
#pragma unroll
        for (int j = 0; j < LB; ++j) { const int i = tid + kScanThreads * j; if (i < 2 * BC) s_bc[i] = rb[j]; }
#pragma unroll
        for (int j = 0; j < LX; ++j) {
            const int i = tid + kScanThreads * j;
            cx[j] = to_f(rx[j]); cg[j] = to_f(rg[j]) * a.factor;
            if (i < XC) s_dx[i] = make_float2(rd[j], rd[j] * cx[j]);
        }
        __syncthreads();
        if (t0 + kTile < s.n) fetch(t0 + kTile);
        // tokens behind the segment have a step size of zero: they change nothing
#pragma unroll 1
        for (int h = 0; h < kTile && t0 + h < s.n; h += kHalf) {
            float y[kHalf];
            const float* b_at = s_bc + h * NP + n0;
            const float2* d_at = s_dx + h * CB + cl;
#pragma unroll
            for (int q = 0; q < kHalf; ++q) {
                const float2 dx = d_at[q * CB];
                y[q] = 0.f;
#pragma unroll
                for (int i = 0; i < SP; i += 4) {
                    const float4 b = get4(b_at + q * NP + i), cv = get4(b_at + BC + q * NP + i);
                    S.v[i] = fmaf(decay<T>(dx.x * A.v[i]), S.v[i], dx.y * b.x);
                    S.v[i + 1] = fmaf(decay<T>(dx.x * A.v[i + 1]), S.v[i + 1], dx.y * b.y);
                    S.v[i + 2] = fmaf(decay<T>(dx.x * A.v[i + 2]), S.v[i + 2], dx.y * b.z);
                    S.v[i + 3] = fmaf(decay<T>(dx.x * A.v[i + 3]), S.v[i + 3], dx.y * b.w);
                    y[q] += fmaf(S.v[i], cv.x, S.v[i + 1] * cv.y) + fmaf(S.v[i + 2], cv.z, S.v[i + 3] * cv.w);
                }
            }
            // sums over the group: with every bit of the lane's number it goes on with half of the tokens, as far as they go
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
#pragma unroll
        for (int j = 0; j < LX; ++j) {
            const int i = tid + kScanThreads * j, t = i / CB;
            if (i < XC && t0 + t < s.n && c0 + own < d.inner) out[size_t(t0 + t) * a.out_ld + own] = to_t<T>(fmaf(skip, cx[j], s_y[i]) * cg[j]);
        }
    }
    if (ok) S.store(at, n, whole);
}

// go(lanes per channel, states per lane)
template <typename F>
int32_t with_group(int states, F go) {
    using std::integral_constant;
    const integral_constant<int, 4> four;
    if (states <= 4) return go(integral_constant<int, 1>{}, four);
    if (states <= 8) return go(integral_constant<int, 2>{}, four);
    if (states <= 16) return go(integral_constant<int, 4>{}, four);
    if (states <= 32) return go(integral_constant<int, 8>{}, four);
    if (states <= 64) return go(integral_constant<int, 16>{}, four);
    if (states <= 128) return go(integral_constant<int, 32>{}, four);
    return go(integral_constant<int, 32>{}, integral_constant<int, 8>{});
}

}  // namespace

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
        constexpr int G = decltype(g)::value, SP = decltype(sp)::value, CB = kScanThreads / G;
        auto kern = dtype == FORGE_F32 ? selective_decode_kernel<float, G, SP> : selective_decode_kernel<__nv_bfloat16, G, SP>;
        FORGE_CUDA(launch_pdl(kern, dim3((d.inner + CB - 1) / CB, ones.n), dim3(kScanThreads), 0, st, d, a, ones));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    });
}

int32_t selective_segments(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const SegTable& t, cudaStream_t st) {
    if (t.n <= 0) return FORGE_OK;
    return with_group(d.state, [&](auto g, auto sp) -> int32_t {
        constexpr int G = decltype(g)::value, SP = decltype(sp)::value, CB = kScanThreads / G;
        auto kern = dtype == FORGE_F32 ? selective_scan_kernel<float, G, SP> : selective_scan_kernel<__nv_bfloat16, G, SP>;
        const size_t smem = size_t(kTile) * (2 * G * SP + 3 * CB) * sizeof(float);
        if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        kern<<<dim3((d.inner + CB - 1) / CB, t.n), kScanThreads, smem, st>>>(d, a, t.segs);
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    });
}

}  // namespace forge
