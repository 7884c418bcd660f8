// Time mixing: state S of a head with a decay per key channel, S <- diag(w) S + k v^T, read out before the update with a bonus
// for the current token: o = S^T r + (sum_i r_i u_i k_i) v.  All of it in float32.
//
// Portions: the scan walks the tokens with the state in registers (recur.cuh); r, k, the decays (made in the epilogue of the low-rank
// product) and the values come a tile of tokens at a time by TMA, the bonus is summed beside the read-out.  Value channels are
// independent of one another, so a head is cut into CTAs of a few of them; and since a segment of the portion acts on the state it
// begins with by a factor per key channel and a sum, a long portion is also cut into segments.
#include "qkv_rows.cuh"
#include "recur.cuh"

namespace cq {

struct TimeMixTmaps { CUtensorMap r, k, w, v; };
// CTA: head x CB value channels x segment of the portion, NC channels to a thread.  A portion of several segments takes three passes:
// every segment's state from zero and its decay product (STATE_ONLY), the states the segments begin with (time_mix_join_kernel), and the
// segments' outputs.
template <int LPC, int NV, int NC, int CB, bool STATE_ONLY>
__global__ void __launch_bounds__(CB / NC * LPC) time_mix_scan_kernel(const TimeMixArgs a, const __grid_constant__ TimeMixTmaps m) {
    constexpr int D = LPC * NV * 4, NVEC = STATE_ONLY ? 2 : 3, STAGE = kRecurTile * (NVEC * D + CB);      // k | w | (r) | v
    static_assert(NC == 4, "a thread's channels are one 16-byte unit of a value row");
    extern __shared__ __align__(128) float tm_smem[];   // [2][STAGE]
    __shared__ __align__(8) unsigned long long bars[2];
    const uint32_t bar = smem_u32(bars), sm0 = smem_u32(tm_smem);
    const int h = blockIdx.x, c0 = blockIdx.y * CB, seg = blockIdx.z, tid = threadIdx.x, l = tid % LPC, cg = tid / LPC;
    if (tid == 0) { mbar_init(bar, 1); mbar_init(bar + 8, 1); mbar_fence_init(); }
    pdl_launch_dependents(); pdl_wait();
    __syncthreads();
    const int first = a.pos_ptr ? *a.pos_ptr : a.pos0;
    const int t_begin = seg * a.seg_len, t_end = min(t_begin + a.seg_len, a.T);
    const size_t ho = (size_t)h * a.dimp, states = (size_t)a.heads * a.dimp * a.dimp;
    auto bring = [&](int t, int b) {
        const uint32_t dst = sm0 + b * STAGE * 4, fb = bar + 8 * b;
        mbar_expect_tx(fb, STAGE * 4);
        recur_load<D>(dst, &m.k, 0, h, t, fb); recur_load<D>(dst + kRecurTile * D * 4, &m.w, 0, h, t, fb);
        if (!STATE_ONLY) recur_load<D>(dst + 2 * kRecurTile * D * 4, &m.r, 0, h, t, fb);
        tma_load_3d(dst + NVEC * kRecurTile * D * 4, &m.v, c0, h, t, fb);
    };
    if (tid == 0) { bring(t_begin, 0); if (t_begin + kRecurTile < t_end) bring(t_begin + kRecurTile, 1); }
    StateCol<LPC, NV> s[NC];
    f32x2 aux[2 * NV];                                  // STATE_ONLY: decay product; else the bonus of this lane's key channels
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int k = (i * LPC + l) * 4;
        ulonglong2 u = make_ulonglong2(0ull, 0ull);
        if (STATE_ONLY) u.x = u.y = pack2(1.f, 1.f);
        else if (k < a.dimp) u = *reinterpret_cast<const ulonglong2*>(a.u + ho + k);
        aux[2 * i] = u.x; aux[2 * i + 1] = u.y;
    }
    const bool joined = gridDim.z > 1;                  // every segment begins with its slot of seg_state (a.state itself is the last segment's to write)
    const float* from = joined ? a.seg_state + (size_t)seg * states : a.state;
    const int c = c0 + cg * NC;                         // this thread's channels; dimp is a multiple of eight: all of them exist or none
#pragma unroll
    for (int j = 0; j < NC; ++j) if (!STATE_ONLY && c < a.dimp && (joined || first > 0)) s[j].load(from + (ho + c + j) * a.dimp, l, a.dimp); else s[j].zero();
    bool failed = false;
    for (int t0 = t_begin, i = 0; t0 < t_end; t0 += kRecurTile, ++i) {
        const int b = i & 1;
        if (!failed && !mbar_wait(bar + 8 * b, (uint32_t)(i >> 1) & 1u)) { failed = true; if (a.err) atomicExch(a.err, 21u); }
        const float *kb = tm_smem + b * STAGE, *wb = kb + kRecurTile * D, *rb = wb + kRecurTile * D, *vb = kb + NVEC * kRecurTile * D;
        const int n = min(kRecurTile, t_end - t0);
#pragma unroll 2
        for (int t = 0; t < n; ++t) {
            f32x2 k[2 * NV], w[2 * NV];
            lane_row<LPC, NV>(kb, t, l, k); lane_row<LPC, NV>(wb, t, l, w);
            const float4 v4 = *reinterpret_cast<const float4*>(vb + t * CB + cg * NC);
            const float v[4] = {v4.x, v4.y, v4.z, v4.w};
            if (!STATE_ONLY) {
                f32x2 r[2 * NV], bon = 0ull;
                float o[NC];
                lane_row<LPC, NV>(rb, t, l, r);
#pragma unroll
                for (int q = 0; q < 2 * NV; ++q) bon = fma2(mul2(r[q], aux[q]), k[q], bon);
#pragma unroll
                for (int j = 0; j < NC; ++j) {
                    f32x2 acc = mul2(bon, pack2(v[j], v[j])), acc1 = 0ull;
#pragma unroll
                    for (int q = 0; q < 2 * NV; q += 2) { acc = fma2(s[j].s[q], r[q], acc); acc1 = fma2(s[j].s[q + 1], r[q + 1], acc1); }
                    o[j] = lanes_sum<LPC>(sum2(add2(acc, acc1)));
                }
                if (l == 0 && c < a.dimp) *reinterpret_cast<float4*>(a.o + (size_t)(t0 + t) * a.ldo + ho + c) = make_float4(o[0], o[1], o[2], o[3]);
            } else {
#pragma unroll
                for (int q = 0; q < 2 * NV; ++q) aux[q] = mul2(aux[q], w[q]);
            }
#pragma unroll
            for (int j = 0; j < NC; ++j) {
                const f32x2 v2 = pack2(v[j], v[j]);
#pragma unroll
                for (int q = 0; q < 2 * NV; ++q) s[j].s[q] = fma2(s[j].s[q], w[q], mul2(k[q], v2));
            }
        }
        __syncthreads();
        if (tid == 0 && t0 + 2 * kRecurTile < t_end) bring(t0 + 2 * kRecurTile, b);
    }
    if (!STATE_ONLY && t_end < a.T) return;
    float* to = STATE_ONLY ? a.seg_state + (size_t)(seg + 1) * states : a.state;
#pragma unroll
    for (int j = 0; j < NC; ++j) if (c < a.dimp) s[j].store(to + (ho + c + j) * a.dimp, l, a.dimp);
    if (STATE_ONLY && c0 == 0 && cg == 0) {
        StateCol<LPC, NV> p;
#pragma unroll
        for (int q = 0; q < 2 * NV; ++q) p.s[q] = aux[q];
        p.store(a.seg_decay + ((size_t)seg * a.heads + h) * a.dimp, l, a.dimp);
    }
}
// Slot g of seg_state: what segment g - 1 makes of a zero state becomes the state that segment g begins with, S <- decay product * (state
// before) + S; slot 0 the portion's.
__global__ void __launch_bounds__(256) time_mix_join_kernel(const TimeMixArgs a, int nseg) {
    pdl_launch_dependents(); pdl_wait();
    const size_t states = (size_t)a.heads * a.dimp * a.dimp, i = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= states) return;
    const int first = a.pos_ptr ? *a.pos_ptr : a.pos0;
    const size_t key = i % a.dimp, h = i / ((size_t)a.dimp * a.dimp);
    float4 s = first > 0 ? *reinterpret_cast<const float4*>(a.state + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    *reinterpret_cast<float4*>(a.seg_state + i) = s;
#pragma unroll 4
    for (int g = 1; g < nseg; ++g) {
        float4* p = reinterpret_cast<float4*>(a.seg_state + (size_t)g * states + i);
        const float4 x = *p, w = *reinterpret_cast<const float4*>(a.seg_decay + ((size_t)(g - 1) * a.heads + h) * a.dimp + key);
        s = make_float4(fmaf(w.x, s.x, x.x), fmaf(w.y, s.y, x.y), fmaf(w.z, s.z, x.z), fmaf(w.w, s.w, x.w));
        *p = s;
    }
}
template <int LPC, int NV>
static int tm_go(const TimeMixArgs& a, const LaunchCfg& cfg) {
    constexpr int NC = 4, CB = 32, D = LPC * NV * 4, NT = CB / NC * LPC;
    const size_t smem = (size_t)2 * kRecurTile * (3 * D + CB) * 4, smem2 = (size_t)2 * kRecurTile * (2 * D + CB) * 4;
    static bool once = false;
    if (!once) {
        cudaError_t e = cudaFuncSetAttribute(time_mix_scan_kernel<LPC, NV, NC, CB, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(time_mix_scan_kernel<LPC, NV, NC, CB, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    TimeMixTmaps m;
    auto map = [&](CUtensorMap* t, const float* p, int ld, int box) { return recur_map(t, p, a.dimp, a.heads, a.dimp, a.T, ld, box, kRecurTile); };
    if (int r = map(&m.r, a.r, a.ld, recur_box(D))) return r;
    if (int r = map(&m.k, a.k, a.ld, recur_box(D))) return r;
    if (int r = map(&m.w, a.w, a.ldw, recur_box(D))) return r;
    if (int r = map(&m.v, a.v, a.ld, CB)) return r;
    const int nseg = (a.T + a.seg_len - 1) / a.seg_len, cy = (a.dimp + CB - 1) / CB;
    if (nseg > 1) {
        if (int r = st_launch(time_mix_scan_kernel<LPC, NV, NC, CB, true>, dim3(a.heads, cy, nseg - 1), dim3(NT), smem2, cfg, a, m)) return r;
        if (int r = st_launch(time_mix_join_kernel, dim3((unsigned)(((size_t)a.heads * a.dimp * a.dimp / 4 + 255) / 256)), dim3(256), 0, cfg, a, nseg)) return r;
    }
    return st_launch(time_mix_scan_kernel<LPC, NV, NC, CB, false>, dim3(a.heads, cy, nseg), dim3(NT), smem, cfg, a, m);
}
// Segments of a portion: as many as fill the SMs with a few CTAs each, none shorter than 128 tokens.
int time_mix_segment(int heads, int dimp, int T, int sm_count) {
    const int ctas = heads * ((dimp + 31) / 32);
    int n = (8 * sm_count + ctas - 1) / ctas;
    if (n > T / 128) n = T / 128;
    if (n > kTmMaxSeg) n = kTmMaxSeg;
    return n < 2 ? T : (T + n - 1) / n;
}
int launch_time_mix_scan(const TimeMixArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.dimp < 8 || a.dimp % 8 || a.dimp > kRecurMaxDim || a.ld % 4 || a.ldw % 4 || a.ldo % 4 || a.seg_len < 1 || (a.seg_len < a.T && (!a.seg_state || !a.seg_decay))) return (int)cudaErrorInvalidValue;
#define GO(L, N) tm_go<L, N>(a, cfg)
    return RECUR_DISPATCH(a.dimp, GO);
#undef GO
}

// ---- one token --------------------------------------------------------------------------------------------------------
// A cluster per head; a CTA each for the token's q, k and v rows behind the heads (the first of their clusters).  On their way before the
// dependency wait: the state of a CTA's first value channels (an earlier step wrote it) and the first rows of w2.
constexpr int kTsRowLanes = 8;                          // lanes to a key channel's row of w2, eight values each at a time
template <int LPC, int NV>
__global__ void __launch_bounds__(kStepThreads) time_mix_step_kernel(const TimeMixStepArgs a, const StepSplit sp) {
    constexpr int D = LPC * NV * 4, CH = kStepThreads / LPC, ROWS = kStepThreads / kTsRowLanes, PRE = 2;
    extern __shared__ __align__(16) float ts_smem[];    // r [D], k [D], w [D], tanh [rank rounded up to eight], o [cw]
    __shared__ float red[8], slots[8], bonus_s;
    pdl_launch_dependents();
    const int h = blockIdx.x, rank = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = tid % LPC, cg = tid / LPC, pos = *a.pos_ptr;      // written before the step's first kernel released its dependents
    if (h >= a.heads) {
        pdl_wait();
        if (rank == 0) qkv_section<bf16>(a.qkv, 0, pos, h - a.heads, tid, kStepThreads);
        return;
    }
    const int c0 = rank * sp.cw, cw = min(sp.cw, a.dimp - c0), rankp = (a.rank + 7) / 8 * 8;
    float *r = ts_smem, *k = r + D, *w = k + D, *th = w + D, *o = th + rankp;
    const size_t ho = (size_t)h * a.dimp;
    if (sp.ncl > 1) cluster_arrive();
    StateCol<LPC, NV> s;
    auto fetch = [&](int c) { if (c < cw && pos > 0) s.load(a.state + (ho + c0 + c) * a.dimp, l, a.dimp); else s.zero(); };
    fetch(cg);
    const int row = tid / kTsRowLanes, part = tid % kTsRowLanes * 8;
    uint4 pre[PRE];                                     // the pitch covers whole units of eight, zeros behind the rank
#pragma unroll
    for (int j = 0; j < PRE; ++j) pre[j] = row + j * ROWS < a.dimp && part < rankp ? ldg_stream(a.w2 + (ho + row + j * ROWS) * a.w2_pitch + part) : make_uint4(0u, 0u, 0u, 0u);
    for (int i = a.dimp + tid; i < D; i += kStepThreads) r[i] = k[i] = w[i] = 0.f;
    pdl_wait();
    for (int i = tid; i < 2 * a.dimp; i += kStepThreads) { if (i < a.dimp) r[i] = __ldcg(a.r + ho + i); else k[i - a.dimp] = __ldcg(a.k + ho + i - a.dimp); }
    for (int i = tid; i < rankp; i += kStepThreads) th[i] = i < a.rank ? tanhf(__ldcg(a.w1 + i)) : 0.f;
    __syncthreads();
    for (int j = 0; row + j * ROWS < a.dimp; ++j) {     // the lanes of a row leave together; rows of a warp may differ by one round
        const int key = row + j * ROWS;
        float z = 0.f;
        for (int p = part; p < rankp; p += kTsRowLanes * 8) {
            float x[8];
            if (j < PRE && p == part) unpack8(j == 0 ? pre[0] : pre[1], x); else load8(a.w2 + (ho + key) * a.w2_pitch + p, x);
#pragma unroll
            for (int q = 0; q < 8; ++q) z = fmaf(th[p + q], x[q], z);
        }
        const unsigned mask = 0xffu << (lane & 24);
#pragma unroll
        for (int d = kTsRowLanes / 2; d > 0; d >>= 1) z += __shfl_xor_sync(mask, z, d);
        if (part == 0) w[key] = expf(-expf(z + a.w0[ho + key]));
    }
    if (warp == kStepThreads / 32 - 1) {
        __syncwarp();
        float b = 0.f;
        for (int i = lane; i < a.dimp; i += 32) b = fmaf(r[i] * a.u[ho + i], k[i], b);
        b = warp_sum(b);
        if (lane == 0) bonus_s = b;
    }
    __syncthreads();
    const float bonus = bonus_s;
    f32x2 rr[2 * NV], kk[2 * NV], ww[2 * NV];
    lane_units<LPC, NV>(r, l, rr); lane_units<LPC, NV>(k, l, kk); lane_units<LPC, NV>(w, l, ww);
    float ss = 0.f;
    for (int cb = 0; cb < cw; cb += CH) {
        const int c = cb + cg;
        if (cb) fetch(c);
        const float v = c < cw ? __ldcg(a.v + ho + c0 + c) : 0.f;
        const f32x2 v2 = pack2(v, v);
        f32x2 acc = 0ull, acc1 = 0ull;
#pragma unroll
        for (int i = 0; i < 2 * NV; i += 2) {
            acc = fma2(s.s[i], rr[i], acc); acc1 = fma2(s.s[i + 1], rr[i + 1], acc1);
            s.s[i] = fma2(s.s[i], ww[i], mul2(kk[i], v2)); s.s[i + 1] = fma2(s.s[i + 1], ww[i + 1], mul2(kk[i + 1], v2));
        }
        const float x = lanes_sum<LPC>(sum2(add2(acc, acc1))) + bonus * v;
        if (c < cw) {
            s.store(a.state + (ho + c0 + c) * a.dimp, l, a.dimp);
            if (l == 0) { o[c] = x; ss = fmaf(x, x, ss); }
        }
    }
    const float inv = inv_rms(cluster_sum(ss, sp.ncl, rank, red, slots), a.dim, a.eps) * a.scale;
    for (int i = tid; i < cw; i += kStepThreads) {
        const int c = c0 + i;
        a.out[ho + c] = __float2bfloat16_rn(c < a.dim ? o[i] * inv * a.norm[ho + c] * silu_f(__ldcg(a.g + ho + c)) : 0.f);
    }
}
template <int LPC, int NV>
static int ts_go(const TimeMixStepArgs& a, const LaunchCfg& cfg) {
    const StepSplit sp = step_split(a.dimp, LPC);
    const size_t smem = (size_t)(3 * LPC * NV * 4 + sp.cw + (a.rank + 7) / 8 * 8) * 4;
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    return st_launch_cluster(time_mix_step_kernel<LPC, NV>, dim3(a.heads + (a.qkv.raw ? 3 : 0), sp.ncl), sp.ncl, dim3(kStepThreads), smem, cfg, a, sp);
}
int launch_time_mix_step(const TimeMixStepArgs& a, const LaunchCfg& cfg) {
    if (a.heads < 1 || a.dimp < 8 || a.dimp % 8 || a.dimp > kRecurMaxDim || a.rank < 1 || a.w2_pitch % 8 || a.w2_pitch < a.rank || (a.qkv.raw && !qkv_rows_ok(a.qkv))) return (int)cudaErrorInvalidValue;
#define GO(L, N) ts_go<L, N>(a, cfg)
    return RECUR_DISPATCH(a.dimp, GO);
#undef GO
}

}  // namespace cq
