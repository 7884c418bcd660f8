// Gated delta rule: state S of a head, S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, in float32.  Written with the
// state before the token,   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T,   so that both products read
// the same state and one round of sums serves them.
//
// Portions: the row kernel applies the convolutions, silu and unit norms and the heads' decays and step sizes; the scan walks
// the tokens as time_mix.cu's does.
#include "recur.cuh"

namespace cq {

constexpr float kUnitEps = 1e-6f;                       // added to the sum of squares of a unit vector

// One channel's convolution and silu at row t (position pos): earlier rows of the portion, before them the ring.
__device__ __forceinline__ float delta_conv(const DeltaArgs& a, int t, int pos, int ch) {
    float s = 0.f;
    for (int j = 0; j < a.taps && j <= pos; ++j) {      // j rows back
        const float x = t - j >= 0 ? __ldcg(a.raw + (size_t)(t - j) * a.ld + ch) : a.ring[(size_t)((pos - j) % a.taps) * a.g_off + ch];
        s = fmaf(a.conv[(size_t)(a.taps - 1 - j) * a.g_off + ch], x, s);
    }
    return silu_f(s);
}
__device__ __forceinline__ float delta_decay(const DeltaArgs& a, const float* raw, int h) { return expf(-a.a_exp[h] * softplus_f(__ldcg(raw + a.a_off + h) + a.dt[h])); }

// CTA = row; a warp per key head, query and key together.
__global__ void __launch_bounds__(256) delta_rows_kernel(const DeltaArgs a) {
    extern __shared__ float kq_smem[];                  // [kv_heads] k . q
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    for (int g = warp; g < a.kv_heads; g += 8) {
        float qq = 0.f, kk = 0.f, kq = 0.f;
        float* out = a.qk + ((size_t)t * a.kv_heads + g) * 2 * a.dimp;
        for (int i = lane; i < a.dimp; i += 32) {
            const float q = delta_conv(a, t, pos, g * a.dimp + i), k = delta_conv(a, t, pos, a.k_off + g * a.dimp + i);
            qq = fmaf(q, q, qq); kk = fmaf(k, k, kk); kq = fmaf(k, q, kq);
            out[i] = q; out[a.dimp + i] = k;            // the same lane scales them below
        }
        const float fq = 1.0f / (sqrtf((float)a.dim) * sqrtf(warp_sum(qq) + kUnitEps)), fk = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
        for (int i = lane; i < a.dimp; i += 32) { out[i] *= fq; out[a.dimp + i] *= fk; }
        kq = warp_sum(kq);
        if (lane == 0) kq_smem[g] = kq * fq * fk;
    }
    for (int c = threadIdx.x; c < a.heads * a.vdimp; c += 256) a.v[(size_t)t * a.heads * a.vdimp + c] = delta_conv(a, t, pos, a.v_off + c);
    __syncthreads();
    const float* raw = a.raw + (size_t)t * a.ld;
    for (int h = threadIdx.x; h < a.heads; h += 256)
        a.sc[(size_t)t * a.heads + h] = make_float4(delta_decay(a, raw, h), sigmoid_f(raw[a.b_off + h]), kq_smem[h / (a.heads / a.kv_heads)], 0.f);
}
int launch_delta_rows(const DeltaArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.taps < 1 || a.kv_heads > 8192) return (int)cudaErrorInvalidValue;
    return st_launch(delta_rows_kernel, dim3(a.T), dim3(256), (size_t)a.kv_heads * 4, cfg, a);
}

constexpr int kDrTile = 16;                             // tokens brought at a time
// CTA: head x CB value channels, NC of them to a thread.
template <int LPC, int NV, int NC, int CB>
__global__ void __launch_bounds__(CB / NC * LPC) delta_scan_kernel(const DeltaArgs a) {
    constexpr int D = LPC * NV * 4, NT = CB / NC * LPC, ROW = 2 * D + CB + 4;            // q | k | v | scalars
    extern __shared__ __align__(16) float dr_smem[];    // [2][kDrTile][ROW]
    pdl_launch_dependents(); pdl_wait();
    const int h = blockIdx.x, g = h / (a.heads / a.kv_heads), c0 = blockIdx.y * CB, tid = threadIdx.x, l = tid % LPC, cg = tid / LPC;
    const int first = a.pos_ptr ? *a.pos_ptr : a.pos0, nc = min(CB, a.vdimp - c0);
    for (int i = tid; i < 2 * kDrTile * ROW; i += NT) dr_smem[i] = 0.f;
    __syncthreads();
    auto bring = [&](int t0, int b) {
        const int n = min(kDrTile, a.T - t0), du = a.dimp / 4, cu = nc / 4, per = 2 * du + cu + 1;
        for (int i = tid; i < n * per; i += NT) {
            const int t = i / per, u = i - t * per, tt = t0 + t;
            float* dst = dr_smem + (b * kDrTile + t) * ROW;
            if (u < 2 * du) cp_async16(dst + (u < du ? 4 * u : D + 4 * (u - du)), a.qk + ((size_t)tt * a.kv_heads + g) * 2 * a.dimp + 4 * u);
            else if (u < 2 * du + cu) cp_async16(dst + 2 * D + 4 * (u - 2 * du), a.v + ((size_t)tt * a.heads + h) * a.vdimp + c0 + 4 * (u - 2 * du));
            else cp_async16(dst + 2 * D + CB, a.sc + (size_t)tt * a.heads + h);
        }
        cp_async_commit();
    };
    bring(0, 0);
    StateCol<LPC, NV> s[NC];
    float* st[NC];
#pragma unroll
    for (int j = 0; j < NC; ++j) {
        const int c = c0 + cg * NC + j;
        st[j] = a.state + ((size_t)h * a.vdimp + c) * a.dimp;
        if (c < a.vdimp && first > 0) s[j].load(st[j], l, a.dimp); else s[j].zero();
    }
    for (int t0 = 0, b = 0; t0 < a.T; t0 += kDrTile, b ^= 1) {
        if (t0 + kDrTile < a.T) { bring(t0 + kDrTile, b ^ 1); cp_async_wait<1>(); } else cp_async_wait<0>();
        __syncthreads();
        const int n = min(kDrTile, a.T - t0);
#pragma unroll 1
        for (int t = 0; t < n; ++t) {
            const float* row = dr_smem + (b * kDrTile + t) * ROW;
            f32x2 q[2 * NV], k[2 * NV];
            lane_units<LPC, NV>(row, l, q); lane_units<LPC, NV>(row + D, l, k);
            const float4 sc = *reinterpret_cast<const float4*>(row + 2 * D + CB);
            const f32x2 g2 = pack2(sc.x, sc.x);
            float sk[NC], sq[NC];
#pragma unroll
            for (int j = 0; j < NC; ++j) {
                f32x2 k0 = 0ull, k1 = 0ull, q0 = 0ull, q1 = 0ull;
#pragma unroll
                for (int i = 0; i < 2 * NV; i += 2) {
                    k0 = fma2(s[j].s[i], k[i], k0); k1 = fma2(s[j].s[i + 1], k[i + 1], k1);
                    q0 = fma2(s[j].s[i], q[i], q0); q1 = fma2(s[j].s[i + 1], q[i + 1], q1);
                }
                sk[j] = sum2(add2(k0, k1)); sq[j] = sum2(add2(q0, q1));
            }
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1)
#pragma unroll
                for (int j = 0; j < NC; ++j) { sk[j] += __shfl_xor_sync(0xffffffffu, sk[j], o); sq[j] += __shfl_xor_sync(0xffffffffu, sq[j], o); }
#pragma unroll
            for (int j = 0; j < NC; ++j) {
                const float u = sc.y * (row[2 * D + cg * NC + j] - sc.x * sk[j]), o = fmaf(sc.z, u, sc.x * sq[j]);
                const f32x2 u2 = pack2(u, u);
#pragma unroll
                for (int i = 0; i < 2 * NV; ++i) s[j].s[i] = fma2(s[j].s[i], g2, mul2(k[i], u2));
                const int c = c0 + cg * NC + j;
                if (l == 0 && c < a.vdimp) a.o[(size_t)(t0 + t) * a.ldo + (size_t)h * a.vdimp + c] = o;
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < NC; ++j) if (c0 + cg * NC + j < a.vdimp) s[j].store(st[j], l, a.dimp);
}
template <int LPC, int NV>
static int dr_go(const DeltaArgs& a, const LaunchCfg& cfg) {
    constexpr int NC = 2, CB = 32, D = LPC * NV * 4;
    const size_t smem = (size_t)2 * kDrTile * (2 * D + CB + 4) * 4;
    static bool once = false;
    if (!once) {
        const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<LPC, NV, NC, CB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    return st_launch(delta_scan_kernel<LPC, NV, NC, CB>, dim3(a.heads, (a.vdimp + CB - 1) / CB), dim3(CB / NC * LPC), smem, cfg, a);
}
int launch_delta_scan(const DeltaArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.dimp < 8 || a.dimp % 8 || a.dimp > kRecurMaxDim || a.vdimp % 8) return (int)cudaErrorInvalidValue;
#define GO(L, N) dr_go<L, N>(a, cfg)
    return RECUR_DISPATCH(a.dimp, GO);
#undef GO
}

// ---- one token --------------------------------------------------------------------------------------------------------
// CTA = value head.  The state of the first value channels is on its way before the dependency wait (it was written by an earlier
// step), and so are the ring's rows.  A key head's ring row is written by the first of the value heads that share it.
constexpr int kDsThreads = 512, kDsHold = 2;            // channels of a thread held at a time
template <int LPC, int NV>
__global__ void __launch_bounds__(kDsThreads) delta_step_kernel(const DeltaStepArgs sa) {
    constexpr int D = LPC * NV * 4, CH = kDsThreads / LPC;                               // value channels at a time
    extern __shared__ __align__(16) float ds_smem[];    // q [D], k [D], v [vdimp], o [vdimp]
    __shared__ float red[40];
    const DeltaArgs& a = sa.d;
    pdl_launch_dependents();
    const int h = blockIdx.x, per = a.heads / a.kv_heads, g = h / per, tid = threadIdx.x, l = tid % LPC, cg = tid / LPC, pos = *a.pos_ptr;
    float *q = ds_smem, *k = q + D, *v = k + D, *o = v + a.vdimp;
    StateCol<LPC, NV> s[kDsHold];
    auto fetch = [&](int c0) {
#pragma unroll
        for (int j = 0; j < kDsHold; ++j) {
            const int c = c0 + j * CH + cg;
            if (c < a.vdimp && pos > 0) s[j].load(a.state + ((size_t)h * a.vdimp + c) * a.dimp, l, a.dimp); else s[j].zero();
        }
    };
    fetch(0);
    pdl_wait();
    float* ring = a.ring + (size_t)(pos % a.taps) * a.g_off;
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int i = tid; i < D; i += kDsThreads) {
        float qv = 0.f, kv = 0.f;
        if (i < a.dimp) {
            const int cq = g * a.dimp + i, ck = a.k_off + cq;
            qv = delta_conv(a, 0, pos, cq); kv = delta_conv(a, 0, pos, ck);
        }
        q[i] = qv; k[i] = kv;
        qq = fmaf(qv, qv, qq); kk = fmaf(kv, kv, kk); kq = fmaf(kv, qv, kq);
    }
    for (int c = tid; c < a.vdimp; c += kDsThreads) {
        const int ch = a.v_off + h * a.vdimp + c;
        v[c] = delta_conv(a, 0, pos, ch);
        ring[ch] = __ldcg(a.raw + ch);                  // the ring's row of this position is read by no convolution of this step
    }
    if (h % per == 0)
        for (int i = tid; i < a.dimp; i += kDsThreads) { const int cq = g * a.dimp + i; ring[cq] = __ldcg(a.raw + cq); ring[a.k_off + cq] = __ldcg(a.raw + a.k_off + cq); }
    qq = cta_sum(qq, red); kk = cta_sum(kk, red); kq = cta_sum(kq, red);
    const float fq = 1.0f / (sqrtf((float)a.dim) * sqrtf(qq + kUnitEps)), fk = 1.0f / sqrtf(kk + kUnitEps);
    const float dec = delta_decay(a, a.raw, h), beta = sigmoid_f(__ldcg(a.raw + a.b_off + h));
    kq *= fq * fk;
    const f32x2 g2 = pack2(dec, dec), fq2 = pack2(fq, fq), fk2 = pack2(fk, fk);
    f32x2 qu[2 * NV], ku[2 * NV];
    lane_units<LPC, NV>(q, l, qu); lane_units<LPC, NV>(k, l, ku);
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) { qu[i] = mul2(qu[i], fq2); ku[i] = mul2(ku[i], fk2); }
    float ss = 0.f;
    for (int c0 = 0; c0 < a.vdimp; c0 += kDsHold * CH) {
        if (c0) fetch(c0);
#pragma unroll
        for (int j = 0; j < kDsHold; ++j) {
            const int c = c0 + j * CH + cg;
            f32x2 k0 = 0ull, k1 = 0ull, q0 = 0ull, q1 = 0ull;
#pragma unroll
            for (int i = 0; i < 2 * NV; i += 2) {
                k0 = fma2(s[j].s[i], ku[i], k0); k1 = fma2(s[j].s[i + 1], ku[i + 1], k1);
                q0 = fma2(s[j].s[i], qu[i], q0); q1 = fma2(s[j].s[i + 1], qu[i + 1], q1);
            }
            const float sk = lanes_sum<LPC>(sum2(add2(k0, k1))), sq = lanes_sum<LPC>(sum2(add2(q0, q1)));
            if (c < a.vdimp) {
                const float u = beta * (v[c] - dec * sk), x = fmaf(kq, u, dec * sq);
                const f32x2 u2 = pack2(u, u);
#pragma unroll
                for (int i = 0; i < 2 * NV; ++i) s[j].s[i] = fma2(s[j].s[i], g2, mul2(ku[i], u2));
                s[j].store(a.state + ((size_t)h * a.vdimp + c) * a.dimp, l, a.dimp);
                if (l == 0) { o[c] = x; ss = fmaf(x, x, ss); }
            }
        }
    }
    const float inv = inv_rms(cta_sum(ss, red), a.vdim, sa.eps) * sa.scale;
    const size_t ho = (size_t)h * a.vdimp;
    for (int c = tid; c < a.vdimp; c += kDsThreads) sa.out[ho + c] = __float2bfloat16_rn(c < a.vdim ? o[c] * inv * sa.norm[c] * silu_f(__ldcg(a.raw + a.g_off + ho + c)) : 0.f);
}
template <int LPC, int NV>
static int ds_go(const DeltaStepArgs& a, const LaunchCfg& cfg) {
    const size_t smem = (size_t)(2 * LPC * NV * 4 + 2 * a.d.vdimp) * 4;
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    return st_launch(delta_step_kernel<LPC, NV>, dim3(a.d.heads), dim3(kDsThreads), smem, cfg, a);
}
int launch_delta_step(const DeltaStepArgs& a, const LaunchCfg& cfg) {
    const DeltaArgs& d = a.d;
    if (d.heads < 1 || d.kv_heads < 1 || d.heads % d.kv_heads || d.taps < 1 || d.dimp < 8 || d.dimp % 8 || d.dimp > kRecurMaxDim || d.vdimp % 8) return (int)cudaErrorInvalidValue;
#define GO(L, N) ds_go<L, N>(a, cfg)
    return RECUR_DISPATCH(d.dimp, GO);
#undef GO
}

}  // namespace cq
