// Gated delta rule: state S of a head, S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, in float32.  Written with the
// state before the token,   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T,   so that both products read
// the same state and one round of sums serves them.
//
// Portions: the row kernel applies the convolutions, silu and unit norms and prepares the heads' decays, step sizes and the products of
// keys and queries among four tokens; the scan walks the tokens four at a time with the state in registers (recur.cuh).
#include "recur.cuh"

namespace cq {

constexpr float kUnitEps = 1e-6f;                       // added to the sum of squares of a unit vector

__device__ __forceinline__ float delta_decay(const DeltaArgs& a, const float* raw, int h) { return expf(-a.a_exp[h] * softplus_f(__ldcg(raw + a.a_off + h) + a.dt[h])); }

// CTA = (four tokens, key head): the head's queries and keys and the values of the heads that share it, then everything that the scan wants to
// know about the four tokens together.  Tokens past the portion's end are zeros that neither decay nor write.
constexpr int kDrThreads = 128;
// The 24 products: q_t = vector 2 t, k_t = vector 2 t + 1; (first vector) * 8 + second.
__constant__ unsigned char kDrPairs[24] = {0 * 9, 2 * 9, 4 * 9, 6 * 9, 1 * 9, 3 * 9, 5 * 9, 7 * 9, 8 + 3, 8 + 5, 24 + 5, 8 + 7, 24 + 7, 40 + 7, 8 + 0, 8 + 2, 24 + 2, 8 + 4, 24 + 4, 40 + 4, 8 + 6, 24 + 6, 40 + 6, 56 + 6};
template <int TAPS>                                     // 0: any number
__global__ void __launch_bounds__(kDrThreads) delta_rows_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float dq_smem[];    // [4][q dimp | k dimp]
    __shared__ float sums[24];                          // q . q [4], k . k [4], k_i . k_t (6), k_i . q_t (10)
    pdl_launch_dependents(); pdl_wait();
    const int blk = blockIdx.x, g = blockIdx.y, t0 = blk * 4, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, per = a.heads / a.kv_heads;
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t0, n = min(4, a.T - t0), d2 = 2 * a.dimp;
    const int uq = a.dimp / 4, units = 2 * uq + per * a.vdimp / 4;
    // the decays and step sizes of the group's heads, by the last warp while the others begin with the convolutions
    __shared__ float dec_s[4][32], step_s[4][32];
    auto scalars = [&](int j0) {
        for (int i = 127 - tid; i < 4 * 32; i += kDrThreads) {
            const int t = i >> 5, j = j0 + (i & 31);
            if (j < per) {
                const float* raw = a.raw + (size_t)(t0 + t) * a.ld;
                dec_s[t][i & 31] = t < n ? delta_decay(a, raw, g * per + j) : 1.f;
                step_s[t][i & 31] = t < n ? sigmoid_f(__ldcg(raw + a.b_off + g * per + j)) : 0.f;
            }
        }
    };
    scalars(0);
    for (int u = tid; u < units; u += kDrThreads) {
        const int ch = u < uq ? g * a.dimp + 4 * u : u < 2 * uq ? a.k_off + g * a.dimp + 4 * (u - uq) : a.v_off + g * per * a.vdimp + 4 * (u - 2 * uq);
        float4 y[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) y[t] = make_float4(0.f, 0.f, 0.f, 0.f);
        auto input = [&](int r) {                       // r: row of the four that the input belongs to
            if (r >= n || pos + r < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
            return t0 + r >= 0 ? __ldcg(reinterpret_cast<const float4*>(a.raw + (size_t)(t0 + r) * a.ld + ch)) : *reinterpret_cast<const float4*>(a.ring + (size_t)((pos + r) % a.taps) * a.g_off + ch);
        };
        auto tap = [&](int t, int j, float4 x) {        // input j rows before token t
            const float4 w = __ldg(reinterpret_cast<const float4*>(a.conv + (size_t)(a.taps - 1 - j) * a.g_off + ch));
            y[t] = make_float4(fmaf(w.x, x.x, y[t].x), fmaf(w.y, x.y, y[t].y), fmaf(w.z, x.z, y[t].z), fmaf(w.w, x.w, y[t].w));
        };
        if (TAPS > 0) {
            float4 x[TAPS + 3];
#pragma unroll
            for (int r = 0; r < TAPS + 3; ++r) x[r] = input(r - (TAPS - 1));
#pragma unroll
            for (int t = 0; t < 4; ++t)
#pragma unroll
                for (int j = TAPS - 1; j >= 0; --j) tap(t, j, x[t + TAPS - 1 - j]);
        } else
            for (int r = -(a.taps - 1); r < n; ++r) {
                const float4 x = input(r);
#pragma unroll
                for (int t = 0; t < 4; ++t) if (t >= r && t - r < a.taps) tap(t, t - r, x);
            }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const float4 z = t < n ? make_float4(silu_f(y[t].x), silu_f(y[t].y), silu_f(y[t].z), silu_f(y[t].w)) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (u < 2 * uq) reinterpret_cast<float4*>(dq_smem + t * d2)[u] = z;
            else if (t < n) reinterpret_cast<float4*>(a.v + (size_t)(t0 + t) * a.heads * a.vdimp + (size_t)g * per * a.vdimp)[u - 2 * uq] = z;
        }
    }
    __syncthreads();
    {
        float s[6];
        int p[6], q[6];                                 // this warp's six products of two of the eight vectors
#pragma unroll
        for (int j = 0; j < 6; ++j) {
            const int e = kDrPairs[warp + 4 * j], x = e >> 3, y = e & 7;
            p[j] = (x >> 1) * d2 + (x & 1) * a.dimp; q[j] = (y >> 1) * d2 + (y & 1) * a.dimp; s[j] = 0.f;
        }
        for (int c = lane; c < a.dimp; c += 32)
#pragma unroll
            for (int j = 0; j < 6; ++j) s[j] = fmaf(dq_smem[p[j] + c], dq_smem[q[j] + c], s[j]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int j = 0; j < 6; ++j) s[j] += __shfl_xor_sync(0xffffffffu, s[j], o);
        if (lane == 0)
#pragma unroll
            for (int j = 0; j < 6; ++j) sums[warp + 4 * j] = s[j];
    }
    __syncthreads();
    float fq[4], fk[4];
#pragma unroll
    for (int t = 0; t < 4; ++t) { fq[t] = 1.0f / (sqrtf((float)a.dim) * sqrtf(sums[t] + kUnitEps)); fk[t] = 1.0f / sqrtf(sums[4 + t] + kUnitEps); }
#pragma unroll
    for (int t = 0; t < 4; ++t)
        for (int c = tid; c < d2 / 4; c += kDrThreads) {
            if (t >= n) break;
            float4 z = reinterpret_cast<const float4*>(dq_smem + t * d2)[c];
            const float f = c < uq ? fq[t] : fk[t];
            z = make_float4(z.x * f, z.y * f, z.z * f, z.w * f);
            reinterpret_cast<float4*>(a.qk + ((size_t)(t0 + t) * a.kv_heads + g) * d2)[c] = z;
        }
    for (int j0 = 0; j0 < per; j0 += 32) {
        if (j0) { __syncthreads(); scalars(j0); __syncthreads(); }
        if (tid >= 32 || j0 + tid >= per) continue;
        const int h = g * per + j0 + tid;
        float dec[4], out[kDeltaBlock];
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            dec[t] = dec_s[t][tid];
            out[4 + t] = step_s[t][tid];
            out[t] = t ? out[t - 1] * dec[t] : dec[t];
        }
        int ia = 8, ib = 14;
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int i = 0; i <= t; ++i) {
                float f = 1.f;                          // decay from behind token i to token t
#pragma unroll
                for (int q = i + 1; q <= t; ++q) f *= dec[q];
                if (i < t) { out[ia] = f * sums[ia] * fk[i] * fk[t]; ++ia; }
                out[ib] = f * sums[ib] * fk[i] * fq[t]; ++ib;
                if (t == 3) out[24 + i] = f;
            }
        float4* dst = reinterpret_cast<float4*>(a.sc + ((size_t)blk * a.heads + h) * kDeltaBlock);
#pragma unroll
        for (int i = 0; i < 7; ++i) dst[i] = make_float4(out[4 * i], out[4 * i + 1], out[4 * i + 2], out[4 * i + 3]);
    }
}
int launch_delta_rows(const DeltaArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.taps < 1 || a.dimp % 8 || a.dimp > kRecurMaxDim || a.vdimp % 8 || a.ld % 4) return (int)cudaErrorInvalidValue;
    const dim3 grid((a.T + 3) / 4, a.kv_heads);
    const size_t smem = (size_t)8 * a.dimp * 4;
    return a.taps == 4 ? st_launch(delta_rows_kernel<4>, grid, dim3(kDrThreads), smem, cfg, a) : st_launch(delta_rows_kernel<0>, grid, dim3(kDrThreads), smem, cfg, a);
}

struct DeltaTmaps { CUtensorMap qk, v, sc; };
// CTA: head x CB value channels, NC of them to a thread; four tokens at a time: their products with the state before them are summed over the
// lanes together, the four corrections follow from the pair products of delta_rows, and the state takes one decay and four updates.
template <int LPC, int NV, int NC, int CB>
__global__ void __launch_bounds__(CB / NC * LPC) delta_scan_kernel(const DeltaArgs a, const __grid_constant__ DeltaTmaps m) {
    constexpr int D = LPC * NV * 4, SC = kRecurTile / 4 * kDeltaBlock, STAGE = kRecurTile * (2 * D + CB) + SC;       // q | k | v | block scalars
    static_assert(NC == 2, "a thread's channels are one 8-byte unit of a value row");
    extern __shared__ __align__(128) float dr_smem[];   // [2][STAGE]
    __shared__ __align__(8) unsigned long long bars[2];
    const uint32_t bar = smem_u32(bars), sm0 = smem_u32(dr_smem);
    const int h = blockIdx.x, g = h / (a.heads / a.kv_heads), c0 = blockIdx.y * CB, tid = threadIdx.x, l = tid % LPC, cg = tid / LPC, c = c0 + cg * NC;
    if (tid == 0) { mbar_init(bar, 1); mbar_init(bar + 8, 1); mbar_fence_init(); }
    pdl_launch_dependents(); pdl_wait();
    __syncthreads();
    const int first = a.pos_ptr ? *a.pos_ptr : a.pos0;
    auto bring = [&](int t, int b) {
        const uint32_t dst = sm0 + b * STAGE * 4, fb = bar + 8 * b;
        mbar_expect_tx(fb, STAGE * 4);
        recur_load<D>(dst, &m.qk, 0, 2 * g, t, fb); recur_load<D>(dst + kRecurTile * D * 4, &m.qk, 0, 2 * g + 1, t, fb);
        tma_load_3d(dst + 2 * kRecurTile * D * 4, &m.v, c0, h, t, fb);
        tma_load_3d(dst + kRecurTile * (2 * D + CB) * 4, &m.sc, 0, h, t / 4, fb);
    };
    if (tid == 0) { bring(0, 0); if (kRecurTile < a.T) bring(kRecurTile, 1); }
    StateCol<LPC, NV> s[NC];
    float* st = a.state + ((size_t)h * a.vdimp + c) * a.dimp;         // vdimp is a multiple of eight: both channels exist or none
#pragma unroll
    for (int j = 0; j < NC; ++j) if (c < a.vdimp && first > 0) s[j].load(st + j * a.dimp, l, a.dimp); else s[j].zero();
    float* out = a.o + (size_t)l * a.ldo + (size_t)h * a.vdimp + c;
    bool failed = false;
    for (int t0 = 0, i = 0; t0 < a.T; t0 += kRecurTile, ++i) {
        const int b = i & 1;
        if (!failed && !mbar_wait(bar + 8 * b, (uint32_t)(i >> 1) & 1u)) { failed = true; if (a.err) atomicExch(a.err, 22u); }
        const float *qb = dr_smem + b * STAGE, *kb = qb + kRecurTile * D, *vb = kb + kRecurTile * D, *cb = vb + kRecurTile * CB;
        const int n = min(kRecurTile, a.T - t0);
#pragma unroll 1
        for (int tb = 0; tb < n; tb += 4) {
            f32x2 k[4][2 * NV];
            float sk[4][NC], sq[4][NC];
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                f32x2 q[2 * NV];
                lane_row<LPC, NV>(kb, tb + t, l, k[t]); lane_row<LPC, NV>(qb, tb + t, l, q);
#pragma unroll
                for (int j = 0; j < NC; ++j) {
                    f32x2 ka = mul2(s[j].s[0], k[t][0]), qa = mul2(s[j].s[0], q[0]);
#pragma unroll
                    for (int x = 1; x < 2 * NV; ++x) { ka = fma2(s[j].s[x], k[t][x], ka); qa = fma2(s[j].s[x], q[x], qa); }
                    sk[t][j] = sum2(ka); sq[t][j] = sum2(qa);
                }
            }
#pragma unroll
            for (int o = LPC / 2; o > 0; o >>= 1)
#pragma unroll
                for (int t = 0; t < 4; ++t)
#pragma unroll
                    for (int j = 0; j < NC; ++j) { sk[t][j] += __shfl_xor_sync(0xffffffffu, sk[t][j], o); sq[t][j] += __shfl_xor_sync(0xffffffffu, sq[t][j], o); }
            float x[kDeltaBlock];
#pragma unroll
            for (int q = 0; q < 7; ++q) {
                const float4 v = reinterpret_cast<const float4*>(cb + (tb >> 2) * kDeltaBlock)[q];
                x[4 * q] = v.x; x[4 * q + 1] = v.y; x[4 * q + 2] = v.z; x[4 * q + 3] = v.w;
            }
            float u[4][NC], o[4][NC];
            {
                int ia = 8, ib = 14;
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const float2 v = *reinterpret_cast<const float2*>(vb + (tb + t) * CB + cg * NC);
#pragma unroll
                    for (int j = 0; j < NC; ++j) {
                        float e = (j ? v.y : v.x) - x[t] * sk[t][j];
#pragma unroll
                        for (int p = 0; p < t; ++p) e -= x[ia + p] * u[p][j];
                        u[t][j] = x[4 + t] * e;
                        float r = x[t] * sq[t][j];
#pragma unroll
                        for (int p = 0; p <= t; ++p) r = fmaf(x[ib + p], u[p][j], r);
                        o[t][j] = r;
                    }
                    ia += t; ib += t + 1;
                }
            }
            const f32x2 g2 = pack2(x[3], x[3]);
#pragma unroll
            for (int j = 0; j < NC; ++j) {
                f32x2 e[4];
#pragma unroll
                for (int t = 0; t < 4; ++t) { const float f = x[24 + t] * u[t][j]; e[t] = pack2(f, f); }
#pragma unroll
                for (int y = 0; y < 2 * NV; ++y) {
                    f32x2 z = mul2(s[j].s[y], g2);
#pragma unroll
                    for (int t = 0; t < 4; ++t) z = fma2(k[t][y], e[t], z);
                    s[j].s[y] = z;
                }
            }
            // lane t of a channel's first four stores token t
            float2 r = make_float2(o[0][0], o[0][1]);
#pragma unroll
            for (int t = 1; t < 4; ++t) { r.x = l == t ? o[t][0] : r.x; r.y = l == t ? o[t][1] : r.y; }
            if (tb + l < min(n, tb + 4) && c < a.vdimp) *reinterpret_cast<float2*>(out + (size_t)(t0 + tb) * a.ldo) = r;
        }
        __syncthreads();
        if (tid == 0 && t0 + 2 * kRecurTile < a.T) bring(t0 + 2 * kRecurTile, b);
    }
#pragma unroll
    for (int j = 0; j < NC; ++j) if (c < a.vdimp) s[j].store(st + j * a.dimp, l, a.dimp);
}
template <int LPC, int NV, int CB>
static int dr_launch(const DeltaArgs& a, const LaunchCfg& cfg) {
    constexpr int NC = 2, D = LPC * NV * 4;
    const size_t smem = (size_t)2 * (kRecurTile * (2 * D + CB) + kRecurTile / 4 * kDeltaBlock) * 4;
    static bool once = false;
    if (!once) {
        const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<LPC, NV, NC, CB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    DeltaTmaps m;
    if (int r = recur_map(&m.qk, a.qk, a.dimp, 2 * a.kv_heads, a.dimp, a.T, 2 * a.kv_heads * a.dimp, recur_box(D), kRecurTile)) return r;
    if (int r = recur_map(&m.v, a.v, a.vdimp, a.heads, a.vdimp, a.T, a.heads * a.vdimp, CB, kRecurTile)) return r;
    if (int r = recur_map(&m.sc, a.sc, kDeltaBlock, a.heads, kDeltaBlock, (a.T + 3) / 4, a.heads * kDeltaBlock, kDeltaBlock, kRecurTile / 4)) return r;
    return st_launch(delta_scan_kernel<LPC, NV, NC, CB>, dim3(a.heads, (a.vdimp + CB - 1) / CB), dim3(CB / NC * LPC), smem, cfg, a, m);
}
// The tokens' operands pass through an SM's shared memory once for every CTA there: few heads are cut finer, so that a CTA has an SM to itself.
template <int LPC, int NV>
static int dr_go(const DeltaArgs& a, const LaunchCfg& cfg) {
    if (a.heads * ((a.vdimp + 15) / 16) <= cfg.sm_count) return dr_launch<LPC, NV, 16>(a, cfg);
    return dr_launch<LPC, NV, 32>(a, cfg);
}
int launch_delta_scan(const DeltaArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.dimp < 8 || a.dimp % 8 || a.dimp > kRecurMaxDim || a.vdimp % 8 || a.ldo % 4) return (int)cudaErrorInvalidValue;
#define GO(L, N) dr_go<L, N>(a, cfg)
    return RECUR_DISPATCH(a.dimp, GO);
#undef GO
}

// ---- one token --------------------------------------------------------------------------------------------------------
// A cluster per value head.  On their way before the dependency wait, as earlier steps wrote them: the state of a CTA's first value channels,
// and the part of the convolutions that earlier tokens make.  A key head's ring row is written by the first of the value heads that share it.
constexpr int kDsHold = 2;                              // convolution channels of a thread that are begun before the wait
template <int LPC, int NV>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaStepArgs sa, const StepSplit sp) {
    constexpr int D = LPC * NV * 4, CH = kStepThreads / LPC;
    extern __shared__ __align__(16) float ds_smem[];    // q [D], k [D], v [cw], o [cw]
    __shared__ float red[8], slots[8], sc[8];
    const DeltaArgs& a = sa.d;
    pdl_launch_dependents();
    const int h = blockIdx.x, rank = blockIdx.y, per = a.heads / a.kv_heads, g = h / per, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = tid % LPC, cg = tid / LPC, pos = *a.pos_ptr;
    const int c0 = rank * sp.cw, cw = min(sp.cw, a.vdimp - c0);
    float *q = ds_smem, *k = q + D, *v = k + D, *o = v + sp.cw;
    if (sp.ncl > 1) cluster_arrive();
    StateCol<LPC, NV> s;
    auto fetch = [&](int c) { if (c < cw && pos > 0) s.load(a.state + ((size_t)h * a.vdimp + c0 + c) * a.dimp, l, a.dimp); else s.zero(); };
    fetch(cg);
    const int items = 2 * a.dimp + cw;                  // channels of the head's query, its key, and this CTA's values
    auto channel = [&](int i) { return i < a.dimp ? g * a.dimp + i : i < 2 * a.dimp ? a.k_off + g * a.dimp + i - a.dimp : a.v_off + h * a.vdimp + c0 + i - 2 * a.dimp; };
    auto before = [&](int ch) {
        float y = 0.f;
        for (int j = 1; j < a.taps && j <= pos; ++j) y = fmaf(a.conv[(size_t)(a.taps - 1 - j) * a.g_off + ch], a.ring[(size_t)((pos - j) % a.taps) * a.g_off + ch], y);
        return y;
    };
    float early[kDsHold], tap[kDsHold];
#pragma unroll
    for (int x = 0; x < kDsHold; ++x) {
        const int i = tid + x * kStepThreads;
        early[x] = tap[x] = 0.f;
        if (i < items) { const int ch = channel(i); early[x] = before(ch); tap[x] = a.conv[(size_t)(a.taps - 1) * a.g_off + ch]; }
    }
    for (int i = a.dimp + tid; i < D; i += kStepThreads) q[i] = k[i] = 0.f;
    pdl_wait();
    float* ring = a.ring + (size_t)(pos % a.taps) * a.g_off;        // no convolution of this step reads this row
    auto take = [&](int i, float y, float w) {
        const int ch = channel(i);
        const float x = __ldcg(a.raw + ch);
        (i < a.dimp ? q + i : i < 2 * a.dimp ? k + i - a.dimp : v + i - 2 * a.dimp)[0] = silu_f(fmaf(w, x, y));
        if (i >= 2 * a.dimp || (h % per == 0 && rank == 0)) ring[ch] = x;
    };
#pragma unroll
    for (int x = 0; x < kDsHold; ++x) if (tid + x * kStepThreads < items) take(tid + x * kStepThreads, early[x], tap[x]);
    for (int i = tid + kDsHold * kStepThreads; i < items; i += kStepThreads) { const int ch = channel(i); take(i, before(ch), a.conv[(size_t)(a.taps - 1) * a.g_off + ch]); }
    if (tid == kStepThreads - 1) { sc[3] = delta_decay(a, a.raw, h); sc[4] = sigmoid_f(__ldcg(a.raw + a.b_off + h)); }
    __syncthreads();
    if (warp < 3) {                                     // q . q, k . k, k . q
        const float *x = warp == 1 ? k : q, *y = warp == 0 ? q : k;
        float t = 0.f;
        for (int i = lane; i < a.dimp; i += 32) t = fmaf(x[i], y[i], t);
        t = warp_sum(t);
        if (lane == 0) sc[warp] = t;
    }
    __syncthreads();
    const float fq = 1.0f / (sqrtf((float)a.dim) * sqrtf(sc[0] + kUnitEps)), fk = 1.0f / sqrtf(sc[1] + kUnitEps), dec = sc[3], beta = sc[4], kq = sc[2] * fq * fk;
    const f32x2 g2 = pack2(dec, dec), fq2 = pack2(fq, fq), fk2 = pack2(fk, fk);
    f32x2 qu[2 * NV], ku[2 * NV];
    lane_units<LPC, NV>(q, l, qu); lane_units<LPC, NV>(k, l, ku);
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) { qu[i] = mul2(qu[i], fq2); ku[i] = mul2(ku[i], fk2); }
    float ss = 0.f;
    for (int cb = 0; cb < cw; cb += CH) {
        const int c = cb + cg;
        if (cb) fetch(c);
        f32x2 k0 = 0ull, k1 = 0ull, q0 = 0ull, q1 = 0ull;
#pragma unroll
        for (int i = 0; i < 2 * NV; i += 2) {
            k0 = fma2(s.s[i], ku[i], k0); k1 = fma2(s.s[i + 1], ku[i + 1], k1);
            q0 = fma2(s.s[i], qu[i], q0); q1 = fma2(s.s[i + 1], qu[i + 1], q1);
        }
        const float sk = lanes_sum<LPC>(sum2(add2(k0, k1))), sq = lanes_sum<LPC>(sum2(add2(q0, q1)));
        if (c < cw) {
            const float u = beta * (v[c] - dec * sk), x = fmaf(kq, u, dec * sq);
            const f32x2 u2 = pack2(u, u);
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i) s.s[i] = fma2(s.s[i], g2, mul2(ku[i], u2));
            s.store(a.state + ((size_t)h * a.vdimp + c0 + c) * a.dimp, l, a.dimp);
            if (l == 0) { o[c] = x; ss = fmaf(x, x, ss); }
        }
    }
    const float inv = inv_rms(cluster_sum(ss, sp.ncl, rank, red, slots), a.vdim, sa.eps) * sa.scale;
    for (int i = tid; i < cw; i += kStepThreads) {
        const int c = c0 + i;
        const size_t at = (size_t)h * a.vdimp + c;
        sa.out[at] = __float2bfloat16_rn(c < a.vdim ? o[i] * inv * sa.norm[c] * silu_f(__ldcg(a.raw + a.g_off + at)) : 0.f);
    }
}
template <int LPC, int NV>
static int ds_go(const DeltaStepArgs& a, const LaunchCfg& cfg) {
    const StepSplit sp = step_split(a.d.vdimp, LPC);
    const size_t smem = (size_t)(2 * LPC * NV * 4 + 2 * sp.cw) * 4;
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    return st_launch_cluster(delta_step_kernel<LPC, NV>, dim3(a.d.heads, sp.ncl), sp.ncl, dim3(kStepThreads), smem, cfg, a, sp);
}
int launch_delta_step(const DeltaStepArgs& a, const LaunchCfg& cfg) {
    const DeltaArgs& d = a.d;
    if (d.heads < 1 || d.kv_heads < 1 || d.heads % d.kv_heads || d.taps < 1 || d.dimp < 8 || d.dimp % 8 || d.dimp > kRecurMaxDim || d.vdimp % 8) return (int)cudaErrorInvalidValue;
#define GO(L, N) ds_go<L, N>(a, cfg)
    return RECUR_DISPATCH(d.dimp, GO);
#undef GO
}

}  // namespace cq
