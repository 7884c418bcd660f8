// What the recurrences share: a head's state [value channel][key channel], LPC lanes to a value channel, lane l holding the
// float4 units l, l + LPC, ... (NV of them) of its key channels in registers as pairs.
#pragma once
#include "stack_dev.cuh"

namespace cq {

template <int LPC, int NV>
struct StateCol {
    f32x2 s[2 * NV];
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) s[i] = 0ull;
    }
    // col: the channel's dimp floats; places past them are zero
    __device__ __forceinline__ void load(const float* col, int l, int dimp) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int k = (i * LPC + l) * 4;
            ulonglong2 v = make_ulonglong2(0ull, 0ull);
            if (k < dimp) v = *reinterpret_cast<const ulonglong2*>(col + k);
            s[2 * i] = v.x; s[2 * i + 1] = v.y;
        }
    }
    __device__ __forceinline__ void store(float* col, int l, int dimp) const {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int k = (i * LPC + l) * 4;
            if (k < dimp) *reinterpret_cast<ulonglong2*>(col + k) = make_ulonglong2(s[2 * i], s[2 * i + 1]);
        }
    }
};
// This lane's units of a vector in shared memory.
template <int LPC, int NV>
__device__ __forceinline__ void lane_units(const float* p, int l, f32x2 (&v)[2 * NV]) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(p + (i * LPC + l) * 4);
        v[2 * i] = u.x; v[2 * i + 1] = u.y;
    }
}
// Sum over the LPC lanes of a value channel, in every one of them.
template <int LPC>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = LPC / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// CALL(LPC, NV) for the smallest layout that holds dimp key channels (at most kRecurMaxDim).
#define RECUR_DISPATCH(dimp, CALL)                                                                                  \
    ((dimp) <= 32 ? CALL(4, 2) : (dimp) <= 64 ? CALL(4, 4) : (dimp) <= 96 ? CALL(8, 3) : (dimp) <= 128 ? CALL(8, 4) : \
     (dimp) <= 192 ? CALL(16, 3) : (dimp) <= 256 ? CALL(16, 4) : CALL(32, 4))

}  // namespace cq
