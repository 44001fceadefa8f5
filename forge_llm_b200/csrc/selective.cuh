// Selective scan: per channel c a state S [states] in f32 that every token decays by its own step size and extends,
//   S <- exp(dt_c A[c]) S + dt_c x_c B;  y_c = S . C + D_c x_c,  out = factor y gate,
// with x behind a short causal convolution per channel (bias, silu), whose last inputs are kept in a ring of `taps` rows, the input of
// position p in row p % taps.  A sequence's state counts as zero when its first row of a step is at position 0.
#pragma once

#include "recurrent.cuh"

namespace forge {

struct SelectiveDims {
    int inner = 0, state = 0, rank = 0, taps = 0;   // channels, states per channel, inner size of the step sizes' projection
    size_t state_values() const { return size_t(inner) * state; }
    __host__ __device__ size_t ring_values() const { return size_t(taps) * inner; }
};

struct SelectiveArgs {
    const void* in = nullptr; int in_ld = 0;               // T rows [inner]: in front of the convolution
    const float* conv = nullptr; const float* conv_add = nullptr; void* ring = nullptr;   // [taps][inner], [inner]; T [slot][taps][inner]
    void* x = nullptr; int x_ld = 0;                       // T rows [inner] behind it
    const float* bc = nullptr; int bc_ld = 0;              // f32 rows [B | C]
    const float* dt = nullptr; int dt_ld = 0;              // f32 rows [inner]: step sizes
    // or the projection that forms them (single tokens; segments if selective_steps_inside): T rows of low_k values per channel over low[row]; a step size is
    // softplus(z + dt_add)
    const void* dt_w = nullptr; const void* low = nullptr; int low_ld = 0, low_k = 0;
    const float* dt_add = nullptr;
    const float* a2 = nullptr;                             // [inner][state]: A in the base of exp2
    const float* skip = nullptr;                           // D
    float* state = nullptr;                                // [slot][inner][state]
    const void* gate = nullptr; int gate_ld = 0;           // T rows [inner]
    float factor = 1.f;
    void* out = nullptr; int out_ld = 0;                   // T rows [inner]
};

#ifdef __CUDACC__
// convolutions end in silu; bfloat16 models take the fast exponential and quotient (far inside a rounding)
template <typename T> __device__ __forceinline__ float conv_act(float v) {
    if constexpr (sizeof(T) == 4) return silu(v);
    else return __fdividef(v, 1.0f + __expf(-v));
}
// The convolution of channel c of row r, a single token.  What earlier steps have left is read in front of the dependency wait (rows of a loop: of the first).
template <typename T>
__device__ __forceinline__ void conv_one(const SelectiveDims& d, const SelectiveArgs& a, const StepRows& rows, int r, int c) {
    pdl_trigger();
    const int pos = rows.pos[r], slot = state_slot(rows, r);
    T* ring = static_cast<T*>(a.ring) + size_t(slot) * d.ring_values() + c;
    float v = 0.f, w = 0.f;
    if (c < d.inner) {
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
#endif

bool selective_supported(const SelectiveDims& d);
// the convolution of single tokens (rows) and of segments
int32_t selective_conv(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const StepRows& ones, const SegTable& t, cudaStream_t st);
bool selective_steps_inside(int dtype, int low_k);
// the recurrence of single tokens, and of segments of any length
int32_t selective_decode(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const StepRows& ones, cudaStream_t st);
int32_t selective_segments(const SelectiveDims& d, int dtype, const SelectiveArgs& a, const SegTable& t, cudaStream_t st);

}  // namespace forge
