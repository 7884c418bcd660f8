// One section (0 queries, 1 keys, 2 values) of a row of raw q / k / v projections, by the threads of one CTA.
#pragma once
#include "stack_dev.cuh"

namespace cq {

inline bool qkv_rows_ok(const QkvRowsArgs& a) {
    return a.heads >= 1 && a.kv_heads >= 1 && a.heads % a.kv_heads == 0 && a.rot_dims % 2 == 0 && a.rot_dims >= 0 && a.rot_dims <= a.dim && a.dim <= a.dimp && a.dimp % 8 == 0 && a.vdimp % 8 == 0 &&
           (a.rot_dims == 0 || a.rot) && a.ld % 4 == 0 && a.k_off % 4 == 0 && a.v_off % 4 == 0;
}
template <typename A>
__device__ __forceinline__ void qkv_section(const QkvRowsArgs& a, int t, int pos, int sec, int tid, int nt) {
    const int heads = sec == 0 ? a.heads : a.kv_heads, len = sec == 2 ? a.vdimp : a.dimp, crow = a.dimp + a.vdimp;
    const float* in = a.raw + (size_t)t * a.ld + (sec == 0 ? 0 : sec == 1 ? a.k_off : a.v_off);
    A* out = sec == 0 ? reinterpret_cast<A*>(a.q) + (size_t)t * a.ldq : reinterpret_cast<A*>(a.cache) + (size_t)pos * crow + (sec == 2 ? a.dimp : 0);
    const size_t hs = sec == 0 ? (size_t)a.dimp : (size_t)a.max_seq * crow;         // from head to head of the output
    const int rot = sec == 2 ? 0 : a.rot_dims, half = rot / 2;
    const int u0 = (rot + 3) / 4, units = len / 4 - u0;                             // whole float4 units behind the rotated part are copied
    for (int i = tid; i < heads * units; i += nt) {
        const int h = i / units, u = u0 + i % units;
        store4(out + (size_t)h * hs + 4 * u, *reinterpret_cast<const float4*>(in + (size_t)h * len + 4 * u));
    }
    if (rot == 0) return;
    for (int i = tid; i < heads * half; i += nt) {
        const int h = i / half, r = i % half;
        const float2 cs = a.rot[(size_t)pos * half + r];
        const float u = in[(size_t)h * len + r], v = in[(size_t)h * len + half + r];
        out[(size_t)h * hs + r] = to_act<A>(u * cs.x - v * cs.y);
        out[(size_t)h * hs + half + r] = to_act<A>(v * cs.x + u * cs.y);
    }
    if (rot % 4)                                                                    // the two places up to the next whole unit
        for (int h = tid; h < heads; h += nt)
            for (int r = rot; r < 4 * u0; ++r) out[(size_t)h * hs + r] = to_act<A>(in[(size_t)h * len + r]);
}

}  // namespace cq
