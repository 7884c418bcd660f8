// Row-wise kernels of the recurrent mixers' portions: norms with token-shift mixes, what a recurrence keeps of a portion's end,
// tanh, the clamped gated unit, head norms with an output gate.
#include "stack_dev.cuh"

namespace cq {

// One CTA per row: the row's norm and - again, from the stream - the row before's, so that no row waits for another.
template <typename A>
__global__ void __launch_bounds__(256) shift_rows_kernel(const ShiftRowsArgs a) {
    __shared__ float red[40];
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, n4 = (a.width + 3) / 4, o4 = a.ldo / 4;
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    const float4* x = reinterpret_cast<const float4*>(a.x + (size_t)t * a.ldx);
    const float4* xp = t > 0 ? reinterpret_cast<const float4*>(a.x + (size_t)(t - 1) * a.ldx) : nullptr;
    const float4* hp = t == 0 && pos > 0 ? reinterpret_cast<const float4*>(a.prev + (size_t)((pos - 1) & 1) * a.ldprev) : nullptr;
    const float4* w = reinterpret_cast<const float4*>(a.w);
    float ss = 0.f, sp = 0.f;
    for (int i = tid; i < n4; i += 256) { ss += dot4(x[i], x[i]); if (xp) sp += dot4(xp[i], xp[i]); }
    const float inv = inv_rms(cta_sum(ss, red), a.width, a.eps), invp = xp ? inv_rms(cta_sum(sp, red), a.width, a.eps) : 0.f;
    A* o = reinterpret_cast<A*>(a.out) + (size_t)t * a.ldo;
    const bool last = t + 1 == (int)gridDim.x;
    for (int i = tid; i < o4; i += 256) {
        float4 h = make_float4(0.f, 0.f, 0.f, 0.f), p = h;
        if (i < n4) {
            const float4 v = x[i], g = w[i];
            h = make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
            if (xp) { const float4 u = xp[i]; p = make_float4(u.x * invp * g.x, u.y * invp * g.y, u.z * invp * g.z, u.w * invp * g.w); }
            else if (hp) p = hp[i];
            if (last) reinterpret_cast<float4*>(a.tail)[i] = h;
        }
        store4(o + 4 * i, h);
        for (int m = 0; m < a.n_mix; ++m) {
            float4 r = h;
            if (i < n4) {
                const float4 mu = reinterpret_cast<const float4*>(a.mu + (size_t)m * a.ldmu)[i];
                r = make_float4(fmaf(p.x - h.x, mu.x, h.x), fmaf(p.y - h.y, mu.y, h.y), fmaf(p.z - h.z, mu.z, h.z), fmaf(p.w - h.w, mu.w, h.w));
            }
            store4(o + (size_t)(m + 1) * a.var_stride + 4 * i, r);
        }
    }
}
int launch_shift_rows(int act, const ShiftRowsArgs& a, int T, const LaunchCfg& cfg) {
    if (T < 1 || a.ldo % 8 || a.ldx % 4 || a.ldmu % 4 || a.ldprev % 4 || a.width > a.ldx || a.width > a.ldprev) return (int)cudaErrorInvalidValue;
    return act == ACT_F32 ? st_launch(shift_rows_kernel<float>, dim3(T), dim3(256), 0, cfg, a) : st_launch(shift_rows_kernel<bf16>, dim3(T), dim3(256), 0, cfg, a);
}

__global__ void __launch_bounds__(256) tail_rows_kernel(const TailRowsArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int t = a.T - 1 - blockIdx.y, pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    const float4* s = reinterpret_cast<const float4*>(a.src + (size_t)t * a.lds);
    float4* d = reinterpret_cast<float4*>(a.ring + (size_t)(pos % a.slots) * a.ldr);
    for (int i = blockIdx.x * 256 + threadIdx.x; i < a.n / 4; i += gridDim.x * 256) d[i] = s[i];
}
int launch_tail_rows(const TailRowsArgs& a, const LaunchCfg& cfg) {
    const int rows = a.T < a.keep ? a.T : a.keep;
    if (rows < 1) return 0;
    if (a.n % 4 || a.lds % 4 || a.ldr % 4 || a.n > a.ldr || a.keep > a.slots) return (int)cudaErrorInvalidValue;
    return st_launch(tail_rows_kernel, dim3((a.n / 4 + 255) / 256, rows), dim3(256), 0, cfg, a);
}

template <typename A>
__global__ void __launch_bounds__(128) tanh_rows_kernel(const float* __restrict__ raw, int ld, A* __restrict__ out, int ldo, size_t part_stride, int n) {
    pdl_launch_dependents(); pdl_wait();
    for (int i = threadIdx.x; i < ldo; i += 128) {
        const float v = i < n ? tanhf(raw[(size_t)blockIdx.x * ld + i]) : 0.f;
        A* o = out + (size_t)blockIdx.x * ldo + i;
        const A hi = to_act<A>(v);
        *o = hi;
        if (sizeof(A) == 2) o[part_stride] = to_act<A>(v - act_f(hi));
    }
}
int launch_tanh_rows(int act, const float* raw, int ld, void* out, int ldo, size_t part_stride, int n, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(tanh_rows_kernel<float>, dim3(T), dim3(128), 0, cfg, raw, ld, (float*)out, ldo, part_stride, n)
                          : st_launch(tanh_rows_kernel<bf16>, dim3(T), dim3(128), 0, cfg, raw, ld, (bf16*)out, ldo, part_stride, n);
}

template <typename A>
__global__ void __launch_bounds__(256) st_glu_rows_kernel(const float* __restrict__ raw, int ld, A* __restrict__ out, int ldo, int ff, float limit, float slope) {
    pdl_launch_dependents(); pdl_wait();
    const float* s = raw + (size_t)blockIdx.x * ld;
    for (int i = threadIdx.x; i < ldo; i += 256) {
        const int g = i / 8 * 16 + i % 8;
        out[(size_t)blockIdx.x * ldo + i] = to_act<A>(i < ff ? clamped_glu_f(s[g], s[g + 8], limit, slope) : 0.f);
    }
}
int launch_st_glu_rows(int act, const float* raw, int ld, void* out, int ldo, int ff, float limit, float slope, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(st_glu_rows_kernel<float>, dim3(T), dim3(256), 0, cfg, raw, ld, (float*)out, ldo, ff, limit, slope)
                          : st_launch(st_glu_rows_kernel<bf16>, dim3(T), dim3(256), 0, cfg, raw, ld, (bf16*)out, ldo, ff, limit, slope);
}

// Heads of 4 * LP places, LP a power of two: a thread per four places, the LP threads of a head side by side.
template <typename A, int LP>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const HeadNormArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, u = blockIdx.y * 256 + threadIdx.x, h = u / LP, i = u % LP * 4;
    const bool in = h < a.heads;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f), g = o, w = o;
    if (in) {
        o = *reinterpret_cast<const float4*>(a.o + (size_t)t * a.ldo + (size_t)u * 4); g = *reinterpret_cast<const float4*>(a.gate + (size_t)t * a.ldg + (size_t)u * 4);
        w = *reinterpret_cast<const float4*>(a.w + (size_t)h * a.w_hs + i);
    }
    float ss = dot4(o, o);                              // places past a head's length hold zeros
#pragma unroll
    for (int d = LP / 2; d > 0; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
    const float f = inv_rms(ss, a.n, a.eps) * a.scale;
    if (in) store4(reinterpret_cast<A*>(a.out) + (size_t)t * a.ldout + (size_t)u * 4, make_float4(o.x * f * w.x * silu_f(g.x), o.y * f * w.y * silu_f(g.y), o.z * f * w.z * silu_f(g.z), o.w * f * w.w * silu_f(g.w)));
}
// Any length: a warp per head, eight heads a CTA.
template <typename A>
__global__ void __launch_bounds__(256) head_norm_gate_any_kernel(const HeadNormArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, t = blockIdx.x;
    if (h >= a.heads) return;
    const float *o = a.o + (size_t)t * a.ldo + (size_t)h * a.np, *g = a.gate + (size_t)t * a.ldg + (size_t)h * a.np, *w = a.w + (size_t)h * a.w_hs;
    A* out = reinterpret_cast<A*>(a.out) + (size_t)t * a.ldout + (size_t)h * a.np;
    float ss = 0.f;
    for (int i = lane; i < a.n; i += 32) ss = fmaf(o[i], o[i], ss);
    const float inv = inv_rms(warp_sum(ss), a.n, a.eps) * a.scale;
    for (int i = lane; i < a.np; i += 32) out[i] = to_act<A>(i < a.n ? o[i] * inv * w[i] * silu_f(g[i]) : 0.f);
}
template <typename A>
static int go_head_norm(const HeadNormArgs& a, int T, const LaunchCfg& cfg) {
    const dim3 grid(T, (a.heads * (a.np / 4) + 255) / 256);
    switch (a.np) {
        case 32: return st_launch(head_norm_gate_kernel<A, 8>, grid, dim3(256), 0, cfg, a);
        case 64: return st_launch(head_norm_gate_kernel<A, 16>, grid, dim3(256), 0, cfg, a);
        case 128: return st_launch(head_norm_gate_kernel<A, 32>, grid, dim3(256), 0, cfg, a);
    }
    return st_launch(head_norm_gate_any_kernel<A>, dim3(T, (a.heads + 7) / 8), dim3(256), 0, cfg, a);
}
int launch_head_norm_gate(int act, const HeadNormArgs& a, int T, const LaunchCfg& cfg) {
    if (T < 1 || a.heads < 1 || a.np % 8 || a.ldo % 4 || a.ldg % 4 || a.ldout % 4) return (int)cudaErrorInvalidValue;
    return act == ACT_F32 ? go_head_norm<float>(a, T, cfg) : go_head_norm<bf16>(a, T, cfg);
}

}  // namespace cq
