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
// One token, one head to a cluster: CTA `rank` of the cluster has value channels [rank * cw, ...).  The cluster's CTAs exchange the sums of
// squares of their read-outs, so that each norms its own channels.
constexpr int kStepThreads = 256;
struct StepSplit { int ncl, cw; };
inline StepSplit step_split(int channels, int lpc) {
    const int ch = kStepThreads / lpc;                  // channels at a time
    int n = (channels + ch - 1) / ch;
    if (n > 8) n = 8;
    const int cw = ((channels + n - 1) / n + 7) / 8 * 8;
    return {(channels + cw - 1) / cw, cw};
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
// Sum over the cluster of every CTA's `v` (summed over its threads).  red: 8 warps' sums, slots: one word per CTA.  Every CTA has arrived at the
// cluster barrier once before.
__device__ __forceinline__ float cluster_sum(float v, int ncl, int rank, float* red, float* slots) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) s += red[i];
    if (ncl == 1) return s;
    cluster_wait();                                     // all CTAs of the cluster run
    if ((int)threadIdx.x < ncl) {
        uint32_t dst;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_u32(slots + rank)), "r"((int)threadIdx.x));
        asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(s) : "memory");
    }
    __syncwarp();
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    cluster_wait();
    s = 0.f;
    for (int i = 0; i < ncl; ++i) s += slots[i];        // the same order in every CTA
    return s;
}
// Launch with clusters of ncl CTAs along y.
template <typename... KArgs, typename... Args>
static int st_launch_cluster(void (*kern)(KArgs...), dim3 grid, int ncl, dim3 block, size_t smem, const LaunchCfg& cfg, Args... args) {
    cudaLaunchConfig_t lc = {};
    lc.gridDim = grid; lc.blockDim = block; lc.dynamicSmemBytes = smem; lc.stream = cfg.stream;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = 1; at[0].val.clusterDim.y = ncl; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at; lc.numAttrs = cfg.pdl ? 2 : 1;
    return (int)cudaLaunchKernelEx(&lc, kern, KArgs(args)...);
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
