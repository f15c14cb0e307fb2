// Device functions of the short causal convolutions (short_conv.cu has the layout and the
// rules), shared by the kernels that do something with the convolved rows in the same launch.
#pragma once

#include <cuda_runtime.h>

namespace rfx {
namespace conv {

constexpr int MAX_TAPS = 16;

// rows of this step that precede row r in its sequence, up to `cap`; the slots of
// the rows before are loaded side by side, not one after the other's answer
__device__ __forceinline__ int rows_before(const int* __restrict__ row_slot, int r, int cap) {
    const int slot = row_slot[r];
    int t = cap;  // the nearest row back that is not this sequence's ends the count (no early exit: no chain)
#pragma unroll
    for (int j = cap - 1; j >= 0; --j) {
        const bool same = r - j - 1 >= 0 && row_slot[r - j - 1] == slot;
        if (!same) t = j;
    }
    return t;
}

// the convolution of channel c (column col0 + c of proj) at row r
__device__ __forceinline__ float conv_at(const float* __restrict__ proj, int ld, int col0, int c,
                                         const float* __restrict__ bias, const float* __restrict__ w,
                                         int taps, const float* __restrict__ state_slot, int C, int r,
                                         int before) {
    const int T = taps - 1;
    const float b = bias ? bias[c] : 0.0f;
    float y = 0.0f;
    for (int j = 0; j < taps; ++j) {
        const int back = T - j;  // tap j meets the input `back` tokens ago
        float u;
        if (back <= before) u = proj[(size_t)(r - back) * ld + col0 + c] + b;
        else u = state_slot[(size_t)(T + before - back) * C + c];
        y = fmaf(w[(size_t)j * C + c], u, y);
    }
    return y;
}

// the same for channels c .. c + 3 (every offset a multiple of four floats)
__device__ __forceinline__ float4 conv4_at(const float* __restrict__ proj, int ld, int col0, int c,
                                           const float* __restrict__ bias, const float* __restrict__ w,
                                           int taps, const float* __restrict__ state_slot, int C, int r,
                                           int before) {
    const int T = taps - 1;
    const float4 b = bias ? *reinterpret_cast<const float4*>(bias + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int j = 0; j < taps; ++j) {
        const int back = T - j;
        const bool here = back <= before;  // one load from either place: no branch between the taps' loads
        float4 u = *reinterpret_cast<const float4*>(here ? proj + (size_t)(r - back) * ld + col0 + c
                                                         : state_slot + (size_t)(T + before - back) * C + c);
        if (here) { u.x += b.x; u.y += b.y; u.z += b.z; u.w += b.w; }
        const float4 f = *reinterpret_cast<const float4*>(w + (size_t)j * C + c);
        y.x = fmaf(f.x, u.x, y.x);
        y.y = fmaf(f.y, u.y, y.y);
        y.z = fmaf(f.z, u.z, y.z);
        y.w = fmaf(f.w, u.w, y.w);
    }
    return y;
}

// y / (1 + e^-y), 32-bit
__device__ __forceinline__ float silu_of(float y) { return y / (1.0f + expf(-y)); }

}  // namespace conv
}  // namespace rfx
