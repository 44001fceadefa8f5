// Recurrent mixers in f32 arithmetic: single tokens (decode), segments token by token, and the row operators around them.
// T is the model's type (bfloat16 or float32); states, decays, step sizes, unit norms and sums are f32 in either.
#include <cooperative_groups.h>

#include <algorithm>
#include <type_traits>

#include "recurrent.cuh"

namespace forge {

namespace {

namespace cg = cooperative_groups;

constexpr int kConvTile = 32;     // tokens per warp; taps - 1 of them at most reach behind the segment

// ------------------------------------------------------------------------------------------------ decode
// Second step of a two-step projection inside a CTA of 256 threads: put(i, sum of w[i][k] in[k]) for i < n, k < K (a multiple of 64).  `held` keeps the
// first 16-byte pieces of a bfloat16 matrix: they are fetched in front of the dependency wait.
template <typename T, int H> struct LowRows {
    uint4 held[H];
    const T* w; int n, K, pieces, steps;   // pieces: of eight values per row
    bool narrow;                           // the pieces of a row lie in one warp
    __device__ __forceinline__ LowRows(const T* w_, int n_, int K_) : w(w_), n(n_), K(K_), pieces(K_ / 8), steps((n_ * (K_ / 8) + 255) / 256), narrow(K_ == 64 || K_ == 128 || K_ == 256) {
        if constexpr (std::is_same<T, __nv_bfloat16>::value)
            if (narrow)
#pragma unroll
                for (int j = 0; j < H; ++j) if (int(threadIdx.x) + 256 * j < n * pieces) held[j] = reinterpret_cast<const uint4*>(w)[threadIdx.x + 256 * j];
    }
    template <typename F> __device__ __forceinline__ void run(const float* in, F put) {
        const int lane = threadIdx.x & 31;
        if (narrow) {
            auto step = [&](int j, const T* src) {
                const int i = threadIdx.x + 256 * j, row = i / pieces, pc = i % pieces;
                float s = 0.f;
                if (row < n) {
                    float v[8], x[8];
                    load8(v, src);
                    load8(x, in + pc * 8);
#pragma unroll
                    for (int e = 0; e < 8; ++e) s = fmaf(v[e], x[e], s);
                }
                for (int m = pieces >> 1; m > 0; m >>= 1) s += __shfl_xor_sync(0xffffffffu, s, m);
                if (pc == 0 && row < n) put(row, s);
            };
            constexpr bool hold = std::is_same<T, __nv_bfloat16>::value;
            if constexpr (hold)
#pragma unroll
                for (int j = 0; j < H; ++j) if (j < steps) step(j, reinterpret_cast<const T*>(&held[j]));
            for (int j = hold ? H : 0; j < steps; ++j) step(j, w + (size_t(threadIdx.x) + 256 * j) * 8);
        } else {
            for (int row = threadIdx.x >> 5; row < n; row += 8) {
                float s = 0.f;
                for (int k = lane; k < K; k += 32) s = fmaf(to_f(w[size_t(row) * K + k]), in[k], s);
                s = warp_sum(s);
                if (lane == 0) put(row, s);
            }
        }
    }
};

// One CTA = 32 CPL value columns of one head of one row; the CTAs of a head form a cluster for the norm of its output.  A thread holds
// the state of CPL columns in the rows warp, warp + 8, ... of it; state, weights and what the convolution keeps are read before
// the dependency wait.
template <int N> __device__ __forceinline__ void load_cols(float (&v)[N], const float* p) {
    if constexpr (N == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else if constexpr (N == 2) { const float2 t = *reinterpret_cast<const float2*>(p); v[0] = t.x; v[1] = t.y; }
    else v[0] = *p;
}
template <int N> __device__ __forceinline__ void store_cols(float* p, const float (&v)[N]) {
    if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else if constexpr (N == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    else *p = v[0];
}
template <typename T, Rule RULE, bool CHANNEL, int RPT, int CPL>
__global__ void __launch_bounds__(256, CPL > 1 ? 2 : 1) recur_decode_kernel(const RecurDims d, const RecurArgs a, const StepRows rows) {
    constexpr bool DELTA = RULE == Rule::Delta;
    extern __shared__ float sm[];
    float* sq = sm;                 // [dim] queries, keys, decays
    float* sk = sq + d.dim;
    float* sg = sk + d.dim;
    float* sv = sg + d.dim;         // [NC]
    constexpr int NC = 32 * CPL;
    float* sgate = sv + NC;         // [NC]
    float* slow = sm + ((3 * d.dim + 2 * NC + 3) & ~3);   // [2][low_k] inner values of decay and gate
    __shared__ __align__(16) float red[8][NC], redo[8][NC];
    __shared__ float wsum[8][3], part;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, splits = gridDim.x, h = blockIdx.y, r = blockIdx.z;
    const int g = h / (d.heads / d.groups), c0 = split * NC, nc = min(NC, d.vdim - c0), cl = lane * CPL;
    const bool own = cl < nc;       // this lane's columns (vdim is a multiple of CPL)
    pdl_trigger();
    // positions are written in front of the step's first kernel, the state in the last step: both are complete
    const int pos = rows.pos[r], slot = state_slot(rows, r);
    float* S = a.state + (size_t(slot) * d.heads + h) * d.dim * d.vdim + c0 + cl;
    float st[RPT][CPL];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = warp + 8 * i;
#pragma unroll
        for (int c = 0; c < CPL; ++c) st[i][c] = 0.f;
        if (pos > 0 && row < d.dim && own) load_cols<CPL>(st[i], S + size_t(row) * d.vdim);
    }
    const int n_in = 2 * d.dim + nc;      // this CTA's channels: q, k, its values
    auto channel = [&](int i) { return i < d.dim ? g * d.dim + i : i < 2 * d.dim ? d.qk() + g * d.dim + i - d.dim : 2 * d.qk() + h * d.vdim + c0 + i - 2 * d.dim; };
    auto place = [&](int i) { return i < d.dim ? sq + i : i < 2 * d.dim ? sk + i - d.dim : sv + i - 2 * d.dim; };
    if constexpr (DELTA) {
        const T* ring = static_cast<const T*>(a.ring) + size_t(slot) * d.ring_values();
        for (int i = tid; i < n_in; i += 256) {
            const int ch = channel(i);
            float v = 0.f;
            for (int j = 0; j < d.taps - 1; ++j) {
                const int p = pos - (d.taps - 1 - j);
                if (p >= 0) v = fmaf(a.conv[size_t(j) * d.channels() + ch], to_f(ring[size_t(p % d.taps) * d.channels() + ch]), v);
            }
            *place(i) = v;
        }
    }
    const bool two_step = CHANNEL && a.decay_w, low_gate = two_step && a.gate_w;
    LowRows<T, 4> low_d(static_cast<const T*>(a.decay_w) + size_t(h) * d.dim * a.low_k, two_step ? d.dim : 0, a.low_k);
    LowRows<T, CPL> low_g(static_cast<const T*>(a.gate_w) + size_t(h * d.vdim + c0) * a.low_k, low_gate ? nc : 0, a.low_k);
    pdl_wait();
    if (two_step) {
        const T* in = static_cast<const T*>(a.low) + size_t(r) * a.low_ld;
        for (int i = tid; i < (low_gate ? 2 : 1) * a.low_k; i += 256) slow[i] = to_f(in[i < a.low_k ? i : a.gate_col + i - a.low_k]);
    }
    const T* x = static_cast<const T*>(a.x) + size_t(r) * a.x_ld;
    float gate[CPL];
#pragma unroll
    for (int c = 0; c < CPL; ++c) gate[c] = own && !low_gate ? to_f(static_cast<const T*>(a.gate)[size_t(r) * a.gate_ld + h * d.vdim + c0 + cl + c]) : 0.f;
    for (int i = tid; i < n_in; i += 256) {
        const int ch = channel(i);
        const T in = x[ch];
        if constexpr (DELTA) {
            const float v = fmaf(a.conv[size_t(d.taps - 1) * d.channels() + ch], to_f(in), *place(i));
            *place(i) = to_f(to_t<T>(silu(v)));
            // one CTA keeps each input
            if (i >= 2 * d.dim || (split == 0 && h % (d.heads / d.groups) == 0)) static_cast<T*>(a.ring)[size_t(slot) * d.ring_values() + size_t(pos % d.taps) * d.channels() + ch] = in;
        } else *place(i) = to_f(in);
    }
    if constexpr (CHANNEL) {
        if (!two_step) for (int i = tid; i < d.dim; i += 256) sg[i] = expf(a.decay[size_t(r) * a.decay_ld + h * d.dim + i]);
    }
    const float g1 = CHANNEL ? 0.f : expf(a.decay[size_t(r) * a.decay_ld + h]);
    const float beta = DELTA ? a.beta[size_t(r) * d.heads + h] : 0.f;
    __syncthreads();
    // sums over the head's channels: q q and k k, or q bonus k
    {
        float s0 = 0.f, s1 = 0.f;
        for (int i = tid; i < d.dim; i += 256) {
            if constexpr (DELTA) { s0 = fmaf(sq[i], sq[i], s0); s1 = fmaf(sk[i], sk[i], s1); }
            else if constexpr (RULE == Rule::TimeMix) s0 = fmaf(sq[i] * a.bonus[h * d.dim + i], sk[i], s0);
        }
        s0 = warp_sum(s0);
        if constexpr (DELTA) s1 = warp_sum(s1);
        if (lane == 0) { wsum[warp][0] = s0; wsum[warp][1] = s1; }
    }
    if (two_step) {
        low_d.run(slow, [&](int i, float z) {
            z += a.decay_add[h * d.dim + i];
            sg[i] = expf(RULE != Rule::TimeMix ? -a.decay_mul[h * d.dim + i] * softplus(z) : -expf(z));
        });
        if (low_gate) low_g.run(slow + a.low_k, [&](int i, float z) { sgate[i] = sigmoid(z); });
    }
    __syncthreads();
    if (low_gate && own)
#pragma unroll
        for (int c = 0; c < CPL; ++c) gate[c] = sgate[cl + c];
    float t0 = 0.f, t1 = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { t0 += wsum[w][0]; t1 += wsum[w][1]; }
    const float qs = DELTA ? d.q_scale / sqrtf(t0 + 1e-6f) : d.q_scale, ks = DELTA ? 1.0f / sqrtf(t1 + 1e-6f) : 1.f;
    float o[CPL], sum8[CPL];
    auto all_warps = [&](float (*buf)[NC], const float (&mine)[CPL]) {   // sum over the warps' rows
        store_cols<CPL>(&buf[warp][cl], mine);
        __syncthreads();
#pragma unroll
        for (int c = 0; c < CPL; ++c) sum8[c] = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            float t[CPL];
            load_cols<CPL>(t, &buf[w][cl]);
#pragma unroll
            for (int c = 0; c < CPL; ++c) sum8[c] += t[c];
        }
    };
#pragma unroll
    for (int c = 0; c < CPL; ++c) o[c] = 0.f;
    if constexpr (DELTA) {
        float dot[CPL], u[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) dot[c] = 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int row = warp + 8 * i;
            if (row < d.dim) {
                const float w = CHANNEL ? sg[row] : g1, k = sk[row] * ks;
#pragma unroll
                for (int c = 0; c < CPL; ++c) { st[i][c] *= w; dot[c] = fmaf(st[i][c], k, dot[c]); }
            }
        }
        all_warps(red, dot);
#pragma unroll
        for (int c = 0; c < CPL; ++c) u[c] = own ? beta * (sv[cl + c] - sum8[c]) : 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int row = warp + 8 * i;
            if (row < d.dim) {
                const float k = sk[row] * ks, q = sq[row] * qs;
#pragma unroll
                for (int c = 0; c < CPL; ++c) { st[i][c] = fmaf(k, u[c], st[i][c]); o[c] = fmaf(st[i][c], q, o[c]); }
                if (own) store_cols<CPL>(S + size_t(row) * d.vdim, st[i]);
            }
        }
    } else {
        float v[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) v[c] = own ? sv[cl + c] : 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int row = warp + 8 * i;
            if (row < d.dim) {
                const float w = CHANNEL ? sg[row] : g1, k = sk[row], q = sq[row] * qs;
#pragma unroll
                for (int c = 0; c < CPL; ++c) {
                    const float next = fmaf(k, v[c], st[i][c] * w);
                    o[c] = fmaf(RULE == Rule::Linear ? next : st[i][c], q, o[c]);
                    st[i][c] = next;
                }
                if (own) store_cols<CPL>(S + size_t(row) * d.vdim, st[i]);
            }
        }
    }
    all_warps(redo, o);
    if (warp == 0) {
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
            o[c] = sum8[c];
            if constexpr (RULE == Rule::TimeMix) o[c] = fmaf(t0, own ? sv[cl + c] : 0.f, o[c]);
            if (own) ss = fmaf(o[c], o[c], ss);
        }
        ss = warp_sum(ss);
        if (lane == 0) part = ss;
    }
    float total;
    if (splits > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        cluster.sync();
        total = 0.f;
        if (warp == 0)
            for (int s = 0; s < splits; ++s) total += *cluster.map_shared_rank(&part, s);
        cluster.sync();   // nobody leaves while its part is read
    } else {
        __syncthreads();
        total = part;
    }
    if (warp == 0 && own) {
        const float inv = 1.0f / sqrtf(total / float(d.vdim) + d.eps);
        T* out = static_cast<T*>(a.out) + size_t(r) * a.out_ld + h * d.vdim + c0 + cl;
#pragma unroll
        for (int c = 0; c < CPL; ++c) out[c] = to_t<T>(o[c] * inv * a.norm[size_t(h) * a.norm_head + c0 + cl + c] * gate[c]);
    }
}

// ------------------------------------------------------------------------------------------------ segments
// Convolution, silu and the factors that make q and k unit vectors.  A warp = a tile of tokens of one unit (a head of q or k, or
// up to 128 values).  The first tile's warp alone reads what the ring keeps of its channels and then leaves there the segment's
// last inputs.
template <typename T>
__global__ void __launch_bounds__(256) conv_rows_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs) {
    const ScanSeg s = segs[blockIdx.z];
    const int t0 = blockIdx.x * kConvTile, lane = threadIdx.x & 31;
    if (t0 >= s.n) return;
    const int vblocks = (d.heads * d.vdim + 127) / 128, unit = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (unit >= 2 * d.groups + vblocks) return;
    const bool is_v = unit >= 2 * d.groups;
    const int ch0 = is_v ? 2 * d.qk() + (unit - 2 * d.groups) * 128 : unit * d.dim;
    const int nch = is_v ? min(128, d.channels() - ch0) : d.dim;
    const T* x = static_cast<const T*>(a.x) + size_t(s.row0) * a.x_ld;
    T* y = static_cast<T*>(sc.conv) + size_t(s.row0) * d.channels();
    T* ring = static_cast<T*>(a.ring) + size_t(s.slot) * d.ring_values();
    for (int t = t0; t < min(s.n, t0 + kConvTile); ++t) {
        float sum = 0.f;
        for (int c = lane; c < nch; c += 32) {
            const int ch = ch0 + c;
            float v = 0.f;
            for (int j = 0; j < d.taps; ++j) {
                const int q = t - (d.taps - 1 - j), p = s.pos0 + q;
                float in = 0.f;
                if (q >= 0) in = to_f(x[size_t(q) * a.x_ld + ch]);
                else if (p >= 0) in = to_f(ring[size_t(p % d.taps) * d.channels() + ch]);
                v = fmaf(a.conv[size_t(j) * d.channels() + ch], in, v);
            }
            const T o = to_t<T>(silu(v));
            y[size_t(t) * d.channels() + ch] = o;
            sum = fmaf(to_f(o), to_f(o), sum);
        }
        if (!is_v) {
            sum = warp_sum(sum);
            if (lane == 0) sc.unit[size_t(s.row0 + t) * 2 * d.groups + unit] = (unit < d.groups ? d.q_scale : 1.f) / sqrtf(sum + 1e-6f);
        }
    }
    if (blockIdx.x == 0)
        for (int c = lane; c < nch; c += 32)
            for (int t = max(0, s.n - d.taps); t < s.n; ++t) ring[size_t((s.pos0 + t) % d.taps) * d.channels() + ch0 + c] = x[size_t(t) * a.x_ld + ch0 + c];
}

// The same for bfloat16 sizes in whole 16-byte pieces and at most four taps: a thread carries eight channels over eight tokens.
constexpr int kConvRun = 8;
__device__ __forceinline__ float fast_silu(float v) { return __fdividef(v, 1.0f + __expf(-v)); }   // far inside a bfloat16 rounding
__global__ void __launch_bounds__(128) conv_rows8_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs) {
    using bf16 = __nv_bfloat16;
    const ScanSeg s = segs[blockIdx.z];
    const int t0 = blockIdx.x * kConvRun, ch = (blockIdx.y * 128 + threadIdx.x) * 8, channels = d.channels();
    if (t0 >= s.n) return;
    const bool ok = ch < channels;
    const bf16* x = static_cast<const bf16*>(a.x) + size_t(s.row0) * a.x_ld + ch;
    bf16* y = static_cast<bf16*>(sc.conv) + size_t(s.row0) * channels + ch;
    bf16* ring = static_cast<bf16*>(a.ring) + size_t(s.slot) * d.ring_values() + ch;
    float w[4][8], past[3][8];   // past[2]: the token before
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int e = 0; e < 8; ++e) w[j][e] = 0.f;
        if (ok && j >= 4 - d.taps) load8(w[j], a.conv + size_t(j - (4 - d.taps)) * channels + ch);
    }
#pragma unroll
    for (int j = 0; j < 3; ++j) {
        const int q = t0 - 3 + j, p = s.pos0 + q;
#pragma unroll
        for (int e = 0; e < 8; ++e) past[j][e] = 0.f;
        if (ok && j >= 4 - d.taps && p >= 0) load8(past[j], q >= 0 ? x + size_t(q) * a.x_ld : ring + size_t(p % d.taps) * channels);
    }
    const int lanes = d.dim / 8, unit = ch / d.dim;   // threads of a head of q or k
    const bool is_qk = ok && unit < 2 * d.groups;
    uint4 in[kConvRun];
#pragma unroll
    for (int i = 0; i < kConvRun; ++i) in[i] = ok && t0 + i < s.n ? *reinterpret_cast<const uint4*>(x + size_t(t0 + i) * a.x_ld) : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < kConvRun; ++i) {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&in[i]);
        uint4 out;
        __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&out);
        float sum = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(h[e]);
            const float now[2] = {f.x, f.y};
            float v[2];
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                const int c = 2 * e + b;
                v[b] = fast_silu(fmaf(w[3][c], now[b], fmaf(w[2][c], past[2][c], fmaf(w[1][c], past[1][c], w[0][c] * past[0][c]))));
                past[0][c] = past[1][c]; past[1][c] = past[2][c]; past[2][c] = now[b];
            }
            o[e] = __floats2bfloat162_rn(v[0], v[1]);
            const float2 r = __bfloat1622float2(o[e]);
            sum = fmaf(r.x, r.x, fmaf(r.y, r.y, sum));
        }
        if (ok && t0 + i < s.n) *reinterpret_cast<uint4*>(y + size_t(t0 + i) * channels) = out;
        for (int m = lanes >> 1; m > 0; m >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, m);
        if (is_qk && t0 + i < s.n && (threadIdx.x & (lanes - 1)) == 0)
            sc.unit[size_t(s.row0 + t0 + i) * 2 * d.groups + unit] = (unit < d.groups ? d.q_scale : 1.f) / sqrtf(sum + 1e-6f);
    }
    if (ok && blockIdx.x == 0)
        for (int t = max(0, s.n - d.taps); t < s.n; ++t) *reinterpret_cast<uint4*>(ring + size_t((s.pos0 + t) % d.taps) * channels) = *reinterpret_cast<const uint4*>(x + size_t(t) * a.x_ld);
}
bool conv_rows8_supported(const RecurDims& d) {
    const int lanes = d.dim / 8;
    return d.taps <= 4 && d.dim % 8 == 0 && d.vdim % 8 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0;
}

// Token by token: a warp carries four value columns of one head, its lanes share the rows of the state.
template <typename T, Rule RULE, bool CHANNEL, int RPL>
__global__ void __launch_bounds__(128) scan_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs) {
    constexpr bool DELTA = RULE == Rule::Delta;
    const ScanSeg s = segs[blockIdx.z];
    const int lane = threadIdx.x & 31, h = blockIdx.y, c0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * 4;
    if (c0 >= d.vdim) return;
    const int nc = min(4, d.vdim - c0), g = h / (d.heads / d.groups);
    float* S = a.state + (size_t(s.slot) * d.heads + h) * d.dim * d.vdim + c0;
    const T* x = DELTA ? static_cast<const T*>(sc.conv) + size_t(s.row0) * d.channels() : static_cast<const T*>(a.x) + size_t(s.row0) * a.x_ld;
    const size_t ld = DELTA ? d.channels() : a.x_ld;
    float st[RPL][4], bonus[RPL];
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
        const int row = lane + 32 * i;
        bonus[i] = RULE == Rule::TimeMix && row < d.dim ? a.bonus[h * d.dim + row] : 0.f;
#pragma unroll
        for (int c = 0; c < 4; ++c) st[i][c] = s.pos0 > 0 && row < d.dim && c < nc ? S[size_t(row) * d.vdim + c] : 0.f;
    }
    struct In { T q[RPL], k[RPL], v[4]; float g[CHANNEL ? RPL : 1], beta, qs, ks; };
    auto load = [&](int t, In& in) {
        const T* xr = x + size_t(t) * ld;
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
            const int row = lane + 32 * i;
            const bool ok = row < d.dim;
            in.q[i] = ok ? xr[g * d.dim + row] : to_t<T>(0.f);
            in.k[i] = ok ? xr[d.qk() + g * d.dim + row] : to_t<T>(0.f);
            if (CHANNEL) in.g[i] = ok ? a.decay[size_t(s.row0 + t) * a.decay_ld + h * d.dim + row] : 0.f;
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) in.v[c] = c < nc ? xr[2 * d.qk() + h * d.vdim + c0 + c] : to_t<T>(0.f);
        if (!CHANNEL) in.g[0] = a.decay[size_t(s.row0 + t) * a.decay_ld + h];
        if (DELTA) {
            in.beta = a.beta[size_t(s.row0 + t) * d.heads + h];
            in.qs = sc.unit[size_t(s.row0 + t) * 2 * d.groups + g];
            in.ks = sc.unit[size_t(s.row0 + t) * 2 * d.groups + d.groups + g];
        }
    };
    In in, next;
    load(0, in);
    for (int t = 0; t < s.n; ++t) {
        load(min(t + 1, s.n - 1), next);
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if constexpr (DELTA) {
            float dot[4] = {0.f, 0.f, 0.f, 0.f};
            const float g1 = CHANNEL ? 0.f : expf(in.g[0]);
#pragma unroll
            for (int i = 0; i < RPL; ++i) {
                const float w = CHANNEL ? expf(in.g[CHANNEL ? i : 0]) : g1, k = to_f(in.k[i]) * in.ks;
#pragma unroll
                for (int c = 0; c < 4; ++c) { st[i][c] *= w; dot[c] = fmaf(st[i][c], k, dot[c]); }
            }
#pragma unroll
            for (int c = 0; c < 4; ++c) dot[c] = in.beta * (to_f(in.v[c]) - warp_sum(dot[c]));
#pragma unroll
            for (int i = 0; i < RPL; ++i) {
                const float k = to_f(in.k[i]) * in.ks, q = to_f(in.q[i]) * in.qs;
#pragma unroll
                for (int c = 0; c < 4; ++c) { st[i][c] = fmaf(k, dot[c], st[i][c]); o[c] = fmaf(st[i][c], q, o[c]); }
            }
        } else {
            float own = 0.f;
            const float g1 = CHANNEL ? 0.f : expf(in.g[0]);
#pragma unroll
            for (int i = 0; i < RPL; ++i) {
                const float w = CHANNEL ? expf(in.g[CHANNEL ? i : 0]) : g1, k = to_f(in.k[i]), q = to_f(in.q[i]) * d.q_scale;
                own = fmaf(q * bonus[i], k, own);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float next = fmaf(k, to_f(in.v[c]), st[i][c] * w);
                    o[c] = fmaf(RULE == Rule::Linear ? next : st[i][c], q, o[c]);
                    st[i][c] = next;
                }
            }
            if constexpr (RULE == Rule::TimeMix)
#pragma unroll
                for (int c = 0; c < 4; ++c) o[c] = fmaf(own, to_f(in.v[c]), o[c]);
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            o[c] = warp_sum(o[c]);
            if (lane == c && c < nc) sc.o[(size_t(s.row0 + t) * d.heads + h) * d.vdim + c0 + c] = o[c];
        }
        in = next;
    }
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
        const int row = lane + 32 * i;
#pragma unroll
        for (int c = 0; c < 4; ++c) if (row < d.dim && c < nc) S[size_t(row) * d.vdim + c] = st[i][c];
    }
}

// out = rms norm(o) * norm * gate per head; a warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) head_norm_kernel(const RecurDims d, const RecurArgs a, const float* __restrict__ o, int row0, int rows) {
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= rows * d.heads) return;
    const int r = row0 + i / d.heads, h = i % d.heads;
    const float* src = o + (size_t(r) * d.heads + h) * d.vdim;
    float ss = 0.f;
    for (int c = lane; c < d.vdim; c += 32) ss = fmaf(src[c], src[c], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / float(d.vdim) + d.eps);
    const T* gate = static_cast<const T*>(a.gate) + size_t(r) * a.gate_ld + h * d.vdim;
    T* out = static_cast<T*>(a.out) + size_t(r) * a.out_ld + h * d.vdim;
    for (int c = lane; c < d.vdim; c += 32) out[c] = to_t<T>(src[c] * inv * a.norm[size_t(h) * a.norm_head + c] * to_f(gate[c]));
}

// the same in 16-byte pieces for vdim = 4 * a power of two up to 128: vdim / 4 lanes per (row, head)
__global__ void __launch_bounds__(256) head_norm4_kernel(const RecurDims d, const RecurArgs a, const float* __restrict__ o, int row0, int rows) {
    const int lanes = d.vdim / 4, i = int((blockIdx.x * 256 + threadIdx.x) / lanes), c = int(threadIdx.x & (lanes - 1)) * 4;
    const bool ok = i < rows * d.heads;
    const int r = row0 + (ok ? i : 0) / d.heads, h = (ok ? i : 0) % d.heads;
    const float4 v = *reinterpret_cast<const float4*>(o + (size_t(r) * d.heads + h) * d.vdim + c);
    const uint2 g2 = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(a.gate) + size_t(r) * a.gate_ld + h * d.vdim + c);
    const float4 w = *reinterpret_cast<const float4*>(a.norm + size_t(h) * a.norm_head + c);
    float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
    for (int m = lanes >> 1; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    const float inv = 1.0f / sqrtf(ss / float(d.vdim) + d.eps);
    const float2 ga = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g2.x)), gb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g2.y));
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x * inv * w.x * ga.x, v.y * inv * w.y * ga.y), hi = __floats2bfloat162_rn(v.z * inv * w.z * gb.x, v.w * inv * w.w * gb.y);
    if (ok) *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(a.out) + size_t(r) * a.out_ld + h * d.vdim + c) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// ------------------------------------------------------------------------------------------------ token shift
// One CTA = 256 columns of one row (single rows) or of up to kShiftRows rows of a segment; the thread that reads what is kept of the row
// before a segment is the one that leaves the segment's last row there.
constexpr int kShiftRows = 16;
template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(T* dst, int ld, int width, int width_p, int n_mix, const float* __restrict__ mu, T* prev, const StepRows rows,
                                                          const ScanSeg* __restrict__ segs) {
    const int c = blockIdx.y * 256 + threadIdx.x;
    ScanSeg s;
    if (segs) s = segs[blockIdx.z];
    else s = ScanSeg{int(blockIdx.x), 1, state_slot(rows, blockIdx.x), rows.pos[blockIdx.x], 0, {}};
    const int t0 = segs ? blockIdx.x * kShiftRows : 0;
    pdl_trigger();
    pdl_wait();
    if (c >= width || t0 >= s.n) return;
    T* at = dst + size_t(s.row0) * ld + c;
    T* keep = prev + size_t(s.slot) * width + c;
    float before = t0 > 0 ? to_f(at[size_t(t0 - 1) * ld]) : s.pos0 > 0 ? to_f(*keep) : 0.f;
    if (t0 == 0) *keep = at[size_t(s.n - 1) * ld];
    float m[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) m[i] = i < n_mix ? mu[size_t(i) * width + c] : 0.f;
    for (int t = t0; t < min(s.n, t0 + kShiftRows); ++t) {
        const float h = to_f(at[size_t(t) * ld]);
#pragma unroll
        for (int i = 0; i < 8; ++i) if (i < n_mix) at[size_t(t) * ld + size_t(i + 1) * width_p] = to_t<T>(fmaf(before - h, m[i], h));
        before = h;
    }
}

// ------------------------------------------------------------------------------------------------ sum of two normed rows
// NV: four-value pieces per thread of rows of up to 1024 NV values (a multiple of four); 0: any width
template <typename T, int NV>
__global__ void __launch_bounds__(256) add_normed_pair_kernel(float* x, const float* ab, int width, float eps, const float* __restrict__ wa, const float* __restrict__ wb, const After after) {
    __shared__ float red[8][2];
    const int r = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* a = ab + size_t(r) * 2 * width;
    const float* b = a + width;
    float sa = 0.f, sb = 0.f;
    auto factors = [&]() {
        sa = warp_sum(sa); sb = warp_sum(sb);
        if (lane == 0) { red[warp][0] = sa; red[warp][1] = sb; }
        __syncthreads();
        sa = sb = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) { sa += red[w][0]; sb += red[w][1]; }
        sa = 0.5f / sqrtf(sa / float(width) + eps); sb = 0.5f / sqrtf(sb / float(width) + eps);
    };
    auto next = [&](float v, float w, float bias) { return after.kind == AFTER_DYT ? dynamic_tanh(v, after.alpha, w, bias) : v; };
    pdl_trigger();
    if constexpr (NV > 0) {
        float4 va[NV], vb[NV], vx[NV], ca[NV], cb[NV], cw[NV], cz[NV];
        const int n4 = width / 4;
        auto get = [&](const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; };
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i >= n4) continue;
            ca[j] = get(wa, i); cb[j] = get(wb, i);
            if (after.kind == AFTER_DYT) { cw[j] = get(after.w, i); cz[j] = get(after.b, i); }
        }
        pdl_wait();
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i >= n4) continue;
            va[j] = get(a, i); vb[j] = get(b, i); vx[j] = get(x + size_t(r) * width, i);
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            if (int(threadIdx.x) + 256 * j >= n4) continue;
            sa = fmaf(va[j].x, va[j].x, fmaf(va[j].y, va[j].y, fmaf(va[j].z, va[j].z, fmaf(va[j].w, va[j].w, sa))));
            sb = fmaf(vb[j].x, vb[j].x, fmaf(vb[j].y, vb[j].y, fmaf(vb[j].z, vb[j].z, fmaf(vb[j].w, vb[j].w, sb))));
        }
        factors();
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i >= n4) continue;
            float4 v = vx[j];
            v.x += va[j].x * sa * ca[j].x + vb[j].x * sb * cb[j].x; v.y += va[j].y * sa * ca[j].y + vb[j].y * sb * cb[j].y;
            v.z += va[j].z * sa * ca[j].z + vb[j].z * sb * cb[j].z; v.w += va[j].w * sa * ca[j].w + vb[j].w * sb * cb[j].w;
            reinterpret_cast<float4*>(x + size_t(r) * width)[i] = v;
            if (after.kind != AFTER_NONE) {
                T* dst = static_cast<T*>(after.dst) + size_t(r) * after.ld + 4 * i;
                dst[0] = to_t<T>(next(v.x, cw[j].x, cz[j].x)); dst[1] = to_t<T>(next(v.y, cw[j].y, cz[j].y));
                dst[2] = to_t<T>(next(v.z, cw[j].z, cz[j].z)); dst[3] = to_t<T>(next(v.w, cw[j].w, cz[j].w));
            }
        }
    } else {
        pdl_wait();
        for (int i = threadIdx.x; i < width; i += 256) { sa = fmaf(a[i], a[i], sa); sb = fmaf(b[i], b[i], sb); }
        factors();
        for (int i = threadIdx.x; i < width; i += 256) {
            const float v = x[size_t(r) * width + i] + a[i] * sa * wa[i] + b[i] * sb * wb[i];
            x[size_t(r) * width + i] = v;
            if (after.kind != AFTER_NONE)
                static_cast<T*>(after.dst)[size_t(r) * after.ld + i] = to_t<T>(next(v, after.kind == AFTER_DYT ? after.w[i] : 0.f, after.kind == AFTER_DYT ? after.b[i] : 0.f));
        }
    }
}

template <typename T, Rule RULE, bool CHANNEL, int RPT, int CPL>
int32_t launch_decode(const RecurDims& d, const RecurArgs& a, const StepRows& rows, cudaStream_t st) {
    const int splits = (d.vdim + 32 * CPL - 1) / (32 * CPL);
    const size_t smem = sizeof(float) * (3 * size_t(d.dim) + 64 * CPL + 4 + 2 * size_t(a.low_k));
    FORGE_CUDA(launch_pdl_cluster(recur_decode_kernel<T, RULE, CHANNEL, RPT, CPL>, dim3(splits, d.heads, rows.n), dim3(256), splits, smem, st, d, a, rows));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}
template <typename T, Rule RULE, bool CHANNEL>
int32_t decode_t(const RecurDims& d, const RecurArgs& a, const StepRows& rows, cudaStream_t st) {
    // enough rows to fill the SMs: whole heads (what all columns of a head share is formed once)
    const bool whole = (long long)rows.n * d.heads >= 148 && d.vdim > 32;
    if (whole && d.vdim <= 64 && d.vdim % 2 == 0 && d.dim <= 64) return launch_decode<T, RULE, CHANNEL, 8, 2>(d, a, rows, st);
    if (whole && d.vdim % 4 == 0 && d.dim <= 64) return launch_decode<T, RULE, CHANNEL, 8, 4>(d, a, rows, st);
    if (whole && d.vdim % 4 == 0 && d.dim <= 128) return launch_decode<T, RULE, CHANNEL, 16, 4>(d, a, rows, st);
    if (d.dim <= 64) return launch_decode<T, RULE, CHANNEL, 8, 1>(d, a, rows, st);
    if (d.dim <= 128) return launch_decode<T, RULE, CHANNEL, 16, 1>(d, a, rows, st);
    return launch_decode<T, RULE, CHANNEL, 32, 1>(d, a, rows, st);
}
template <typename T, Rule RULE, bool CHANNEL>
int32_t scan_t(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, cudaStream_t st) {
    const dim3 grid((d.vdim + 15) / 16, d.heads, n_segs);
    if (d.dim <= 32) scan_kernel<T, RULE, CHANNEL, 1><<<grid, 128, 0, st>>>(d, a, sc, segs);
    else if (d.dim <= 64) scan_kernel<T, RULE, CHANNEL, 2><<<grid, 128, 0, st>>>(d, a, sc, segs);
    else if (d.dim <= 128) scan_kernel<T, RULE, CHANNEL, 4><<<grid, 128, 0, st>>>(d, a, sc, segs);
    else scan_kernel<T, RULE, CHANNEL, 8><<<grid, 128, 0, st>>>(d, a, sc, segs);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}
template <typename T>
int32_t segments_t(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const SegTable& t, cudaStream_t st) {
    constexpr bool half = std::is_same<T, __nv_bfloat16>::value;
    if (d.rule == Rule::Delta) {
        const int tiles = (t.max_n + kConvTile - 1) / kConvTile, units = 2 * d.groups + (d.heads * d.vdim + 127) / 128;
        if (half && conv_rows8_supported(d)) conv_rows8_kernel<<<dim3((t.max_n + kConvRun - 1) / kConvRun, (d.channels() + 1023) / 1024, t.n), 128, 0, st>>>(d, a, sc, t.segs);
        else conv_rows_kernel<T><<<dim3(tiles, (units + 7) / 8, t.n), 256, 0, st>>>(d, a, sc, t.segs);
        FORGE_LAUNCH_CHECK();
    }
    const int walked = half && recur_chunked_supported(d) ? t.n_short : t.n;   // token by token
    if (walked > 0) {
        if (d.rule == Rule::TimeMix) FORGE_TRY((scan_t<T, Rule::TimeMix, true>(d, a, sc, t.segs, walked, st)));
        else if (d.rule == Rule::Linear) FORGE_TRY((scan_t<T, Rule::Linear, true>(d, a, sc, t.segs, walked, st)));
        else FORGE_TRY(d.channel ? (scan_t<T, Rule::Delta, true>(d, a, sc, t.segs, walked, st)) : (scan_t<T, Rule::Delta, false>(d, a, sc, t.segs, walked, st)));
    }
    FORGE_TRY(recur_chunked(d, a, sc, t.segs + walked, t.n - walked, t.n_chunks, st));
    const int lanes = d.vdim / 4;
    if (half && d.vdim % 4 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 && a.gate_ld % 4 == 0 && a.out_ld % 4 == 0)
        head_norm4_kernel<<<unsigned((size_t(t.rows) * d.heads * lanes + 255) / 256), 256, 0, st>>>(d, a, sc.o, t.row0, t.rows);
    else head_norm_kernel<T><<<(t.rows * d.heads + 7) / 8, 256, 0, st>>>(d, a, sc.o, t.row0, t.rows);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace

bool recur_supported(const RecurDims& d) { return d.dim <= 256 && d.vdim <= 256 && d.taps <= kConvTile && (d.rule == Rule::Delta ? d.taps >= 1 : d.channel && d.taps == 0); }

int32_t recur_decode(const RecurDims& d, int dtype, const RecurArgs& a, const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    auto go = [&](auto t) -> int32_t {
        using T = decltype(t);
        if (d.rule == Rule::TimeMix) return decode_t<T, Rule::TimeMix, true>(d, a, rows, st);
        if (d.rule == Rule::Linear) return decode_t<T, Rule::Linear, true>(d, a, rows, st);
        return d.channel ? decode_t<T, Rule::Delta, true>(d, a, rows, st) : decode_t<T, Rule::Delta, false>(d, a, rows, st);
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int32_t recur_segments(const RecurDims& d, int dtype, const RecurArgs& a, const RecurScratch& sc, const SegTable& t, cudaStream_t st) {
    if (t.n <= 0) return FORGE_OK;
    return dtype == FORGE_F32 ? segments_t<float>(d, a, sc, t, st) : segments_t<__nv_bfloat16>(d, a, sc, t, st);
}

int32_t token_shift(void* dst, int ld, int width, int width_p, int n_mix, const float* mu, void* prev, int dtype, const StepRows& rows, int n_single, const SegTable& t, cudaStream_t st) {
    if (n_mix > 8) { set_error("token shift: %d mixes", n_mix); return FORGE_ERR_SHAPE; }
    auto go = [&](auto type) -> int32_t {
        using T = decltype(type);
        const int cols = (width + 255) / 256;
        if (n_single > 0) {
            FORGE_CUDA(launch_pdl(token_shift_kernel<T>, dim3(n_single, cols), dim3(256), 0, st, static_cast<T*>(dst), ld, width, width_p, n_mix, mu, static_cast<T*>(prev), rows, static_cast<const ScanSeg*>(nullptr)));
            FORGE_LAUNCH_CHECK();
        }
        if (t.n > 0) {
            FORGE_CUDA(launch_pdl(token_shift_kernel<T>, dim3((t.max_n + kShiftRows - 1) / kShiftRows, cols, t.n), dim3(256), 0, st, static_cast<T*>(dst), ld, width, width_p, n_mix, mu, static_cast<T*>(prev), rows, t.segs));
            FORGE_LAUNCH_CHECK();
        }
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int32_t add_normed_pair(float* x, const float* ab, int rows, int width, float eps, const float* wa, const float* wb, const After& after, int dtype, cudaStream_t st) {
    if (rows <= 0) return FORGE_OK;
    auto go = [&](auto type) -> int32_t {
        using T = decltype(type);
        auto kern = width % 4 || width > 4096 ? add_normed_pair_kernel<T, 0> : width <= 2048 ? add_normed_pair_kernel<T, 2> : add_normed_pair_kernel<T, 4>;
        FORGE_CUDA(launch_pdl(kern, dim3(rows), dim3(256), 0, st, x, ab, width, eps, wa, wb, after));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace forge
