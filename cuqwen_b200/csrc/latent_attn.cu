// Latent attention, any sizes, both activation types: one CTA per (head, query), an online softmax over tiles of 128 keys;
// and the two matrix steps that let a decoded token attend to the latents directly.  The 32-bit mode's only path.
#include "stack_dev.cuh"

namespace cq {

constexpr int kLaThreads = 128;

template <typename A>
__global__ void __launch_bounds__(kLaThreads) latent_attn_kernel(const LatentAttnArgs a) {
    extern __shared__ float la_smem[];                  // query [dn + dr], accumulators [dv], probabilities [128]
    __shared__ float red[40];
    float *q = la_smem, *acc = q + a.dn + a.dr, *pr = acc + a.dv;
    pdl_launch_dependents(); pdl_wait();
    const int h = blockIdx.x, hk = a.kv_group > 1 ? h / a.kv_group : h, t = blockIdx.y, tid = threadIdx.x;
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    const A* qn = reinterpret_cast<const A*>(a.qn) + (size_t)t * a.ldqn + (size_t)h * a.qn_hs;
    const A* qr = reinterpret_cast<const A*>(a.qr) + (size_t)t * a.ldqr + (size_t)h * a.qr_hs;
    for (int i = tid; i < a.dn; i += kLaThreads) q[i] = act_f(qn[i]);
    for (int i = tid; i < a.dr; i += kLaThreads) q[a.dn + i] = act_f(qr[i]);
    for (int i = tid; i < a.dv; i += kLaThreads) acc[i] = 0.f;
    const int lo = a.window > 0 && pos - a.window + 1 > 0 ? pos - a.window + 1 : 0;
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;       // the sink is a key without a value, unscaled
    for (int k0 = lo; k0 <= pos; k0 += kLaThreads) {
        __syncthreads();
        const int k = k0 + tid;
        float s = -INFINITY;
        if (k <= pos) {
            const A* kn = reinterpret_cast<const A*>(a.kn) + (size_t)(k - a.kbase) * a.ldkn + (size_t)hk * a.kn_hs;
            const A* kr = reinterpret_cast<const A*>(a.kr) + (size_t)k * a.ldkr;
            float d = 0.f;
            for (int i = 0; i < a.dn; ++i) d = fmaf(q[i], act_f(kn[i]), d);
            for (int i = 0; i < a.dr; ++i) d = fmaf(q[a.dn + i], act_f(kr[i]), d);
            s = d * a.scale;
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        if ((tid & 31) == 0) red[tid >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float mn = fmaxf(m, mx);                   // finite: key k0 is visible
        const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
        m = mn;
        const float p = k <= pos ? expf(s - mn) : 0.f;
        pr[tid] = p;
        l = l * alpha + cta_sum(p, red);                 // barriers inside: pr is complete
        const int n = pos - k0 + 1 < kLaThreads ? pos - k0 + 1 : kLaThreads;
        for (int c = tid; c < a.dv; c += kLaThreads) {
            const A* v = reinterpret_cast<const A*>(a.v) + (size_t)(k0 - a.kbase) * a.ldv + (size_t)hk * a.v_hs + c;
            float o = acc[c] * alpha;
            for (int j = 0; j < n; ++j) o = fmaf(pr[j], act_f(v[(size_t)j * a.ldv]), o);
            acc[c] = o;
        }
    }
    const float inv = a.out_scale / l;
    for (int c = tid; c < a.dv; c += kLaThreads) {
        float o = acc[c] * inv;
        if (a.gate) o *= sigmoid_f(a.gate[(size_t)t * a.ldg + (size_t)h * a.g_hs + c]);
        const size_t i = (size_t)t * a.ldo + (size_t)h * a.o_hs + c;
        if (a.out_f32) reinterpret_cast<float*>(a.out)[i] = o;
        else reinterpret_cast<A*>(a.out)[i] = to_act<A>(o);
    }
}
int launch_latent_attn(int act, const LatentAttnArgs& a, const LaunchCfg& cfg) {
    const size_t smem = (size_t)(a.dn + a.dr + a.dv + kLaThreads) * 4;
    if (a.T < 1 || a.heads < 1 || smem > 40 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(a.heads, a.T);
    return act == ACT_F32 ? st_launch(latent_attn_kernel<float>, grid, dim3(kLaThreads), smem, cfg, a) : st_launch(latent_attn_kernel<bf16>, grid, dim3(kLaThreads), smem, cfg, a);
}

// One head's query against the latents: its unrotated part carried through W_uk, its rotated part rotated, side by side as
// the cache rows are.  CTA = (head, 64 latent columns): eight lanes hold a row segment, thirty-two row groups walk the
// head's rows of W_uk; the first four segments of a thread are on their way before the dependency wait (the weights do not
// depend on the step).  The head's first CTA also rotates.
constexpr int kAqThreads = 256, kAqCols = 64, kAqPre = 4;
template <typename A>
__global__ void __launch_bounds__(kAqThreads) absorb_q_kernel(const AbsorbArgs a) {
    __shared__ float part[8][kAqCols];
    pdl_launch_dependents();
    const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, cl = (lane & 7) * 8, c0 = blockIdx.y * kAqCols + cl, grp = threadIdx.x >> 3;
    const bf16* w = a.wk + (size_t)h * a.dimp * a.pitch + c0;
    const bool live = c0 < a.kr_off;                     // kr_off = the padded latent length, a multiple of eight within the pitch
    uint4 pre[kAqPre];
#pragma unroll
    for (int i = 0; i < kAqPre; ++i) pre[i] = live && grp + 32 * i < a.dim ? ldg_stream(w + (size_t)(grp + 32 * i) * a.pitch) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    const float* q = a.q + (size_t)h * a.q_hs;
    A* out = reinterpret_cast<A*>(a.out) + (size_t)h * a.ldo;
    if (blockIdx.y == 0) {
        const int half = a.rot_dim / 2, pos = *a.pos_ptr;
        for (int i = threadIdx.x; i < half; i += kAqThreads) {
            const float2 cs = a.rot[(size_t)pos * half + i];
            const float u = __ldcg(q + a.rot_off + i), v = __ldcg(q + a.rot_off + half + i);
            out[a.kr_off + i] = to_act<A>(u * cs.x - v * cs.y);
            out[a.kr_off + half + i] = to_act<A>(v * cs.x + u * cs.y);
        }
    }
    float s[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    float qd[kAqPre];
#pragma unroll
    for (int i = 0; i < kAqPre; ++i) qd[i] = grp + 32 * i < a.dim ? __ldcg(q + grp + 32 * i) : 0.f;
#pragma unroll
    for (int i = 0; i < kAqPre; ++i) {
        float v[8];
        unpack8(pre[i], v);
#pragma unroll
        for (int k = 0; k < 8; ++k) s[k] = fmaf(qd[i], v[k], s[k]);
    }
    if (live)
        for (int d = grp + 32 * kAqPre; d < a.dim; d += 32) {
            float v[8];
            load8(w + (size_t)d * a.pitch, v);
            const float f = __ldcg(q + d);
#pragma unroll
            for (int k = 0; k < 8; ++k) s[k] = fmaf(f, v[k], s[k]);
        }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        s[k] += __shfl_xor_sync(0xffffffffu, s[k], 8);
        s[k] += __shfl_xor_sync(0xffffffffu, s[k], 16);
        if (lane < 8) part[warp][cl + k] = s[k];
    }
    __syncthreads();
    if (threadIdx.x < kAqCols && blockIdx.y * kAqCols + threadIdx.x < a.kr_off) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) v += part[k][threadIdx.x];
        out[blockIdx.y * kAqCols + threadIdx.x] = to_act<A>(v);
    }
}
int launch_absorb_q(int act, const AbsorbArgs& a, const LaunchCfg& cfg) {
    const dim3 grid(a.heads, (a.kr_off + kAqCols - 1) / kAqCols);
    return act == ACT_F32 ? st_launch(absorb_q_kernel<float>, grid, dim3(kAqThreads), 0, cfg, a) : st_launch(absorb_q_kernel<bf16>, grid, dim3(kAqThreads), 0, cfg, a);
}

// A warp per output value.
template <typename A>
__global__ void __launch_bounds__(256) uv_gate_kernel(const UvGateArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int h = blockIdx.x, v = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (v >= a.vdim) return;
    const float* o = a.o + (size_t)h * a.ldo;
    const bf16* w = a.wv + (size_t)(h * a.vdimp + v) * a.pitch;
    float s = 0.f;
    for (int r = lane; r < a.kv_rank; r += 32) s = fmaf(o[r], __bfloat162float(w[r]), s);
    s = warp_sum(s);
    if (lane == 0) {
        if (a.gate) s *= sigmoid_f(a.gate[(size_t)h * a.g_hs + v]);
        reinterpret_cast<A*>(a.out)[(size_t)h * a.o_hs + v] = to_act<A>(s);
    }
}
int launch_uv_gate(int act, const UvGateArgs& a, const LaunchCfg& cfg) {
    const dim3 grid(a.heads, (a.vdim + 7) / 8);
    return act == ACT_F32 ? st_launch(uv_gate_kernel<float>, grid, dim3(256), 0, cfg, a) : st_launch(uv_gate_kernel<bf16>, grid, dim3(256), 0, cfg, a);
}

}  // namespace cq
