// What the recurrences share: a head's state [value channel][key channel], LPC lanes to a value channel, lane l holding the
// float4 units l, l + LPC, ... (NV of them) of its key channels in registers as pairs.
#pragma once
#include "stack_dev.cuh"
#include "tma.cuh"

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

// A float32 tensor [n][heads][len] (row stride ld, head stride hs), brought by TMA as boxes of box_len places of one head x box_rows rows;
// places past a head's end and rows past the last arrive as zeros.  All lengths and strides are multiples of four.
inline int recur_map(CUtensorMap* m, const float* p, int len, int heads, int hs, int n, int ld, int box_len, int box_rows) {
    typedef CUresult (*Encode)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static Encode fn = [] {
        void* q = nullptr;
        cudaDriverEntryPointQueryResult r;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &q, cudaEnableDefault, &r) != cudaSuccess || r != cudaDriverEntryPointSuccess) q = nullptr;
        return (Encode)q;
    }();
    if (!fn) return (int)cudaErrorNotSupported;
    const cuuint64_t d[3] = {(cuuint64_t)len, (cuuint64_t)heads, (cuuint64_t)n}, st[2] = {(cuuint64_t)hs * 4, (cuuint64_t)ld * 4};
    const cuuint32_t b[3] = {(cuuint32_t)box_len, 1, (cuuint32_t)box_rows}, es[3] = {1, 1, 1};
    const CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 3, const_cast<float*>(p), d, st, b, es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : (int)cudaErrorInvalidValue;
}
constexpr int kRecurTile = 16;                          // tokens brought at a time
constexpr int recur_box(int d) { return d < 256 ? d : 256; }
// One head's `D` places of kRecurTile rows from row t on, [row][place] in pieces of 256 places.
template <int D>
__device__ __forceinline__ void recur_load(uint32_t dst, const CUtensorMap* m, int x, int head, int t, uint32_t bar) {
#pragma unroll
    for (int p = 0; p < D; p += 256) tma_load_3d(dst + p * kRecurTile * 4, m, x + p, head, t, bar);
}
// Address of a row's places for lane_units: with more than 256 places the pieces lie behind one another.
template <int D>
__device__ __forceinline__ const float* recur_unit(const float* base, int t, int place) {
    return D <= 256 ? base + t * D + place : base + (place >> 8) * (256 * kRecurTile) + t * 256 + (place & 255);
}
template <int LPC, int NV>
__device__ __forceinline__ void lane_row(const float* base, int t, int l, f32x2 (&v)[2 * NV]) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(recur_unit<LPC * NV * 4>(base, t, (i * LPC + l) * 4));
        v[2 * i] = u.x; v[2 * i + 1] = u.y;
    }
}
// CALL(LPC, NV) for the smallest layout that holds dimp key channels (at most kRecurMaxDim).
#define RECUR_DISPATCH(dimp, CALL)                                                                                  \
    ((dimp) <= 32 ? CALL(4, 2) : (dimp) <= 64 ? CALL(4, 4) : (dimp) <= 96 ? CALL(8, 3) : (dimp) <= 128 ? CALL(8, 4) : \
     (dimp) <= 192 ? CALL(16, 3) : (dimp) <= 256 ? CALL(16, 4) : CALL(32, 4))

}  // namespace cq
