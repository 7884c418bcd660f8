// Decode attention of one token over the latent cache in bfloat16, all heads sharing one stream of cache rows (a latent is
// key and value at once, so a row is read once per sixteen heads).
//
// latent_partial_kernel: grid (key ranges, groups of sixteen heads).  A CTA brings 64 rows at a time into shared memory
// (cp.async, two buffers; rows of earlier steps are requested before the dependency wait), scores on mma.sync m16n8k16 with
// the sixteen heads as the M rows - warp w takes keys 8 w .. 8 w + 7 of the tile - an online softmax in float32 over the
// tile, then P V with the columns of the latent dealt over the warps.  Un-normalised partials and (max, sum) per head go out.
// latent_fold_kernel: grid (heads, slices of 32 value rows): merges the ranges and the sink - up to eight slices of a head
// form a cluster whose CTAs merge a share of the columns each and exchange them through distributed shared memory -
// multiplies the head's latent output with W_uv, applies the gate.
//
// Grouped attention runs the same partial kernel over a cache per key / value head whose rows are [key | value]: the groups of
// sixteen are cut from the query heads of one key / value head, the score stops at the key's end, P V starts there.
// grouped_fold_kernel merges the ranges.
#include "stack_dev.cuh"
#include "tma.cuh"

namespace cq {

constexpr int kLdTile = 64, kLdThreads = 256, kLdHeads = 16;
constexpr int kLdMaxSplit = 148;
__host__ __device__ inline int ld_pitch(int crow) { return (crow + 15) / 16 * 16 + 8; }          // elements; an odd number of 16-byte units
__host__ __device__ inline int ld_smem(int crow) {
    return (2 * kLdTile + kLdHeads) * ld_pitch(crow) * 2 + kLdHeads * (kLdTile + 2) * 4 + kLdHeads * (kLdTile + 8) * 2 + 3 * kLdHeads * 4;
}

__device__ __forceinline__ void ld_cp16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void ld_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void ld_waitg() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ld_sm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_sm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_sm2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Keys [lo, hi) of a range: the visible keys dealt over the ranges in whole tiles.
__device__ __forceinline__ void ld_range(const LatentDecodeArgs& a, int pos, int split, int& lo, int& hi) {
    const int first = a.window > 0 && pos - a.window + 1 > 0 ? pos - a.window + 1 : 0, n = pos + 1 - first;
    const int tiles = (n + kLdTile - 1) / kLdTile, per = (tiles + a.nsplit - 1) / a.nsplit * kLdTile;
    lo = first + split * per;
    hi = lo + per < pos + 1 ? lo + per : pos + 1;
}

template <int MAXP>      // pairs of eight latent columns per warp: kvrp <= 128 * MAXP
__global__ void __launch_bounds__(kLdThreads) latent_partial_kernel(const LatentDecodeArgs a) {
    extern __shared__ __align__(16) unsigned char ld_raw[];
    const int pitch = ld_pitch(a.crow), pb = pitch * 2;
    const uint32_t sk = smem_u32(ld_raw), sq = sk + 2 * kLdTile * pb;
    float* S = reinterpret_cast<float*>(ld_raw + (2 * kLdTile + kLdHeads) * pb);                 // [16][66]
    bf16* P = reinterpret_cast<bf16*>(S + kLdHeads * (kLdTile + 2));                             // [16][72]
    float* rowf = reinterpret_cast<float*>(P + kLdHeads * (kLdTile + 8));                        // rescale factor, max, sum per head
    const uint32_t sp = smem_u32(P);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int tiles16 = (a.group + kLdHeads - 1) / kLdHeads, kvh = a.group ? blockIdx.y / tiles16 : 0, sub = a.group ? blockIdx.y % tiles16 * kLdHeads : 0;
    const int h0 = a.group ? kvh * a.group + sub : blockIdx.y * kLdHeads;
    const int nh = min(kLdHeads, a.group ? a.group - sub : a.heads - h0);
    const bf16* cache = a.cache + (size_t)kvh * a.kv_stride;
    const int qrow = a.group ? a.kdim : a.crow, qunits = qrow / 8;
    pdl_launch_dependents();
    const int pos = *a.pos_ptr;                 // written before the step's first kernel released its dependents
    int lo, hi;
    ld_range(a, pos, blockIdx.x, lo, hi);
    const int units = a.crow / 8, ksteps = (qrow + 15) / 16;
    if (lo >= hi) {                             // an empty range: the fold skips it
        pdl_wait();
        if (tid < nh) { float* ml = a.part_ml + ((size_t)blockIdx.x * a.heads + h0 + tid) * 2; ml[0] = -INFINITY; ml[1] = 0.f; }
        return;
    }
    // the last K step may run past a row whose length is no multiple of sixteen: its places stay zero
    for (int i = tid; i < 2 * kLdTile + kLdHeads; i += kLdThreads) *reinterpret_cast<uint4*>(ld_raw + (size_t)i * pb + (pitch - 8) * 2) = make_uint4(0u, 0u, 0u, 0u);
    if (a.crow & 8) for (int i = tid; i < 2 * kLdTile + kLdHeads; i += kLdThreads) *reinterpret_cast<uint4*>(ld_raw + (size_t)i * pb + a.crow * 2) = make_uint4(0u, 0u, 0u, 0u);
    // rows k0 .. of the cache into buffer b; only = 1: all but the row of this step's token, 2: that row alone, 0: all
    auto load = [&](int k0, int b, int only) {
        for (int i = tid; i < kLdTile * units; i += kLdThreads) {
            const int r = i / units, u = i - r * units, k = k0 + r;
            const uint32_t dst = sk + (b * kLdTile + r) * pb + u * 16;
            if (k >= hi) { if (only != 2) *reinterpret_cast<uint4*>(ld_raw + (dst - sk)) = make_uint4(0u, 0u, 0u, 0u); }
            else if (only == 0 || (only == 2) == (k == pos)) ld_cp16(dst, cache + (size_t)k * a.crow + u * 8);
        }
    };
    load(lo, 0, 1);
    ld_commit();
    pdl_wait();
    if (lo + kLdTile > pos) load(lo, 0, 2);
    for (int i = tid; i < kLdHeads * units; i += kLdThreads) {
        const int r = i / units, u = i - r * units;
        unsigned char* dst = ld_raw + (size_t)(2 * kLdTile + r) * pb + u * 16;
        if (r < nh && u < qunits) ld_cp16(smem_u32(dst), a.q + (size_t)(h0 + r) * qrow + u * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
    }
    ld_commit();
    if (tid < kLdHeads) { rowf[kLdHeads + tid] = -INFINITY; rowf[2 * kLdHeads + tid] = 0.f; }
    const int npair = (a.kvrp + 15) / 16;
    float o[MAXP][2][4];
#pragma unroll
    for (int p = 0; p < MAXP; ++p)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[p][j][i] = 0.f;
    const int g = lane >> 2, t = lane & 3;
    int b = 0;
    for (int k0 = lo; k0 < hi; k0 += kLdTile, b ^= 1) {
        if (k0 + kLdTile < hi) { load(k0 + kLdTile, b ^ 1, 0); ld_commit(); ld_waitg<1>(); }
        else ld_waitg<0>();
        __syncthreads();
        // scores: this warp's eight keys
        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
        const uint32_t qa = sq + (lane & 15) * pb + (lane >> 4) * 16;
        const uint32_t ka = sk + (b * kLdTile + warp * 8 + (lane & 7)) * pb + ((lane >> 3) & 1) * 16;
#pragma unroll 4
        for (int ks = 0; ks < ksteps; ++ks) {
            uint32_t qf[4], b0, b1;
            ld_sm4(qa + ks * 32, qf);
            ld_sm2(ka + ks * 32, b0, b1);
            if (ks & 1) ld_mma(s1, qf, b0, b1); else ld_mma(s0, qf, b0, b1);
        }
        {
            const int c = warp * 8 + 2 * t;
            const bool v0 = k0 + c < hi, v1 = k0 + c + 1 < hi;
            S[g * (kLdTile + 2) + c] = v0 ? (s0[0] + s1[0]) * a.scale : -INFINITY;
            S[g * (kLdTile + 2) + c + 1] = v1 ? (s0[1] + s1[1]) * a.scale : -INFINITY;
            S[(g + 8) * (kLdTile + 2) + c] = v0 ? (s0[2] + s1[2]) * a.scale : -INFINITY;
            S[(g + 8) * (kLdTile + 2) + c + 1] = v1 ? (s0[3] + s1[3]) * a.scale : -INFINITY;
        }
        __syncthreads();
        // softmax of the tile: sixteen lanes a head (warp w: heads 2 w, 2 w + 1), four keys a lane
        {
            const int h = warp * 2 + (lane >> 4), l16 = lane & 15;
            const float* row = S + h * (kLdTile + 2) + l16 * 4;
            float x[4], mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < 4; ++i) { x[i] = row[i]; mx = fmaxf(mx, x[i]); }
#pragma unroll
            for (int d = 8; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float m = rowf[kLdHeads + h], mn = fmaxf(m, mx);        // finite: the tile's first key is visible
            float sum = 0.f;
            uint32_t pk[2];
#pragma unroll
            for (int i = 0; i < 4; ++i) { x[i] = expf(x[i] - mn); sum += x[i]; }
            pk[0] = pack_bf(x[0], x[1]); pk[1] = pack_bf(x[2], x[3]);
#pragma unroll
            for (int d = 8; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
            *reinterpret_cast<uint2*>(P + h * (kLdTile + 8) + l16 * 4) = make_uint2(pk[0], pk[1]);
            __syncwarp();
            if (l16 == 0) {
                const float al = m == -INFINITY ? 0.f : expf(m - mn);
                rowf[h] = al; rowf[kLdHeads + h] = mn; rowf[2 * kLdHeads + h] = rowf[2 * kLdHeads + h] * al + sum;
            }
        }
        __syncthreads();
        const float al0 = rowf[g], al1 = rowf[g + 8];
#pragma unroll
        for (int p = 0; p < MAXP; ++p)
#pragma unroll
            for (int j = 0; j < 2; ++j) { o[p][j][0] *= al0; o[p][j][1] *= al0; o[p][j][2] *= al1; o[p][j][3] *= al1; }
#pragma unroll
        for (int ks = 0; ks < kLdTile / 16; ++ks) {
            uint32_t pf[4];
            ld_sm4(sp + (lane & 15) * (kLdTile + 8) * 2 + (ks * 16 + (lane >> 4) * 8) * 2, pf);
            const uint32_t va = sk + (b * kLdTile + ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pb + (lane >> 4) * 16 + (a.group ? a.kdim * 2 : 0);
#pragma unroll
            for (int p = 0; p < MAXP; ++p) {
                const int pair = warp + p * 8;
                if (pair < npair) {
                    uint32_t v[4];
                    ld_sm4t(va + pair * 32, v);
                    ld_mma(o[p][0], pf, v[0], v[1]);
                    ld_mma(o[p][1], pf, v[2], v[3]);
                }
            }
        }
        __syncthreads();                        // the buffer and P may be overwritten
    }
    float* po = a.part_o + ((size_t)blockIdx.x * a.heads + h0) * a.kvrp;
#pragma unroll
    for (int p = 0; p < MAXP; ++p) {
        const int pair = warp + p * 8;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int c = pair * 16 + j * 8 + 2 * t;
            if (c < a.kvrp) {
                if (g < nh) *reinterpret_cast<float2*>(po + (size_t)g * a.kvrp + c) = make_float2(o[p][j][0], o[p][j][1]);
                if (g + 8 < nh) *reinterpret_cast<float2*>(po + (size_t)(g + 8) * a.kvrp + c) = make_float2(o[p][j][2], o[p][j][3]);
            }
        }
    }
    if (tid < nh) { float* ml = a.part_ml + ((size_t)blockIdx.x * a.heads + h0 + tid) * 2; ml[0] = rowf[kLdHeads + tid]; ml[1] = rowf[2 * kLdHeads + tid]; }
}

constexpr int kLfRows = 32;
__global__ void __launch_bounds__(256) latent_fold_kernel(const LatentDecodeArgs a) {
    extern __shared__ float lf_smem[];          // [kvrp] the head's latent output
    __shared__ float wgt[kLdMaxSplit];
    __shared__ float red[16];
    __shared__ __align__(16) float mrg[8][128];
    const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_launch_dependents();
    const int ncl = gridDim.y == a.ncl ? a.ncl : 1, rank = ncl > 1 ? (int)blockIdx.y : 0;
    if (ncl > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // waited for before the first store to another CTA: by then all have started
    // the weights do not depend on the step: on their way before the wait (four rows a warp, two 16-byte units a lane)
    uint4 w[4][2];
    const int v0 = blockIdx.y * kLfRows + warp * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
            w[i][j] = v0 + i < a.vdim && lane + 32 * j < a.kvrp / 8 ? ldg_stream(a.wv + (size_t)(h * a.vdimp + v0 + i) * a.pitch + (lane + 32 * j) * 8) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    // This CTA's columns of the merged output, 128 at a time: a lane four columns, a warp every eighth key range; every CTA of
    // the cluster receives them.  The partials are requested together with the ranges' (max, sum); those of an empty range are
    // whatever an earlier step left (finite) and get the weight zero.
    const int cw = ((a.kvrp + ncl - 1) / ncl + 127) / 128 * 128;
    const float* po = a.part_o + (size_t)h * a.kvrp;
    const size_t ps = (size_t)a.heads * a.kvrp;
    float4 pre[8];
    {
        const int c = rank * cw + lane * 4;
#pragma unroll
        for (int k = 0; k < 8; ++k) pre[k] = c < a.kvrp && warp + 8 * k < a.nsplit ? __ldcg(reinterpret_cast<const float4*>(po + (warp + 8 * k) * ps + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float m = -INFINITY, l = 0.f;
    if (tid < a.nsplit) {
        const float2 v = __ldcg(reinterpret_cast<const float2*>(a.part_ml) + (size_t)tid * a.heads + h);
        m = v.x; l = v.y;
    }
    float mx = m;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    const float sink = a.sink ? a.sink[h] : -INFINITY;
    mx = sink;
#pragma unroll
    for (int i = 0; i < 8; ++i) mx = fmaxf(mx, red[i]);
    const float e = m == -INFINITY ? 0.f : expf(m - mx);
    const float s = warp_sum(e * l);
    if (lane == 0) red[8 + warp] = s;
    if (tid < a.nsplit) wgt[tid] = e;
    __syncthreads();
    float den = a.sink ? expf(sink - mx) : 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) den += red[8 + i];
    const float inv = 1.0f / den;
    if (ncl > 1) asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    for (int cb = rank * cw; cb < (rank + 1) * cw && cb < a.kvrp; cb += 128) {
        const int c = cb + lane * 4;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (cb != rank * cw) {
#pragma unroll
            for (int k = 0; k < 8; ++k) pre[k] = c < a.kvrp && warp + 8 * k < a.nsplit ? __ldcg(reinterpret_cast<const float4*>(po + (warp + 8 * k) * ps + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        auto acc = [&](float f, float4 v) { o.x = fmaf(f, v.x, o.x); o.y = fmaf(f, v.y, o.y); o.z = fmaf(f, v.z, o.z); o.w = fmaf(f, v.w, o.w); };
#pragma unroll
        for (int k = 0; k < 8; ++k) if (warp + 8 * k < a.nsplit) acc(wgt[warp + 8 * k], pre[k]);
        if (c < a.kvrp)
            for (int k = warp + 64; k < a.nsplit; k += 8) acc(wgt[k], __ldcg(reinterpret_cast<const float4*>(po + k * ps + c)));
        reinterpret_cast<float4*>(mrg[warp])[lane] = o;
        __syncthreads();
        if (tid < 128 && cb + tid < a.kvrp) {
            float v = 0.f;
#pragma unroll
            for (int k = 0; k < 8; ++k) v += mrg[k][tid];
            v *= inv;
            if (ncl == 1) lf_smem[cb + tid] = v;
            else
                for (int r = 0; r < ncl; ++r) {
                    uint32_t dst;
                    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dst) : "r"(smem_u32(lf_smem + cb + tid)), "r"(r));
                    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dst), "f"(v) : "memory");
                }
        }
        __syncthreads();
    }
    if (ncl > 1) asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int v = v0 + i;
        if (v >= a.vdim) break;
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int u = lane + 32 * j;
            if (u < a.kvrp / 8) {
                float x[8];
                unpack8(w[i][j], x);
#pragma unroll
                for (int k = 0; k < 8; ++k) acc = fmaf(lf_smem[u * 8 + k], x[k], acc);
            }
        }
        for (int u = lane + 64; u < a.kvrp / 8; u += 32) {                // latents of more than 512
            float x[8];
            load8(a.wv + (size_t)(h * a.vdimp + v) * a.pitch + u * 8, x);
#pragma unroll
            for (int k = 0; k < 8; ++k) acc = fmaf(lf_smem[u * 8 + k], x[k], acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) {
            if (a.gate) acc *= sigmoid_f(__ldcg(a.gate + (size_t)h * a.g_hs + v));
            a.out[(size_t)h * a.o_hs + v] = __float2bfloat16_rn(acc);
        }
    }
}

// CTA = (head, 128 value columns): a warp takes every eighth key range, a lane four columns.
__global__ void __launch_bounds__(256) grouped_fold_kernel(const LatentDecodeArgs a) {
    __shared__ float wgt[kLdMaxSplit];
    __shared__ float red[16];
    __shared__ __align__(16) float mrg[8][128];
    const int h = blockIdx.x, cb = blockIdx.y * 128, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c = cb + lane * 4;
    pdl_launch_dependents(); pdl_wait();
    const float* po = a.part_o + (size_t)h * a.kvrp;
    const size_t ps = (size_t)a.heads * a.kvrp;
    float4 pre[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) pre[k] = c < a.kvrp && warp + 8 * k < a.nsplit ? __ldcg(reinterpret_cast<const float4*>(po + (warp + 8 * k) * ps + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
    float m = -INFINITY, l = 0.f;
    if (tid < a.nsplit) {
        const float2 v = __ldcg(reinterpret_cast<const float2*>(a.part_ml) + (size_t)tid * a.heads + h);
        m = v.x; l = v.y;
    }
    float mx = m;
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    mx = red[0];
#pragma unroll
    for (int i = 1; i < 8; ++i) mx = fmaxf(mx, red[i]);
    const float e = m == -INFINITY ? 0.f : expf(m - mx);                // a range without keys weighs nothing (its partials are an earlier step's, finite)
    const float s = warp_sum(e * l);
    if (lane == 0) red[8 + warp] = s;
    if (tid < a.nsplit) wgt[tid] = e;
    __syncthreads();
    float den = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) den += red[8 + i];
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    auto acc = [&](float f, float4 v) { o.x = fmaf(f, v.x, o.x); o.y = fmaf(f, v.y, o.y); o.z = fmaf(f, v.z, o.z); o.w = fmaf(f, v.w, o.w); };
#pragma unroll
    for (int k = 0; k < 8; ++k) if (warp + 8 * k < a.nsplit) acc(wgt[warp + 8 * k], pre[k]);
    if (c < a.kvrp)
        for (int k = warp + 64; k < a.nsplit; k += 8) acc(wgt[k], __ldcg(reinterpret_cast<const float4*>(po + k * ps + c)));
    reinterpret_cast<float4*>(mrg[warp])[lane] = o;
    __syncthreads();
    if (tid < 128 && cb + tid < a.kvrp) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) v += mrg[k][tid];
        a.out[(size_t)h * a.o_hs + cb + tid] = __float2bfloat16_rn(v * (a.out_scale / den));
    }
}

int latent_decode_splits(int heads, int crow, int kvrp, int window, int max_seq, int sm_count) {
    if (ld_smem(crow) > 225 * 1024 || kvrp > 1024) return 0;
    const int groups = (heads + kLdHeads - 1) / kLdHeads;
    const int keys = window > 0 && window < max_seq ? window : max_seq, tiles = (keys + kLdTile - 1) / kLdTile;
    int n = sm_count / groups;
    if (n > kLdMaxSplit) n = kLdMaxSplit;
    if (n > tiles) n = tiles;
    return n < 1 ? 1 : n;
}
int grouped_decode_splits(int heads, int kv_heads, int kdim, int vdimp, int max_seq, int sm_count) {
    if (ld_smem(kdim + vdimp) > 225 * 1024 || vdimp > 1024) return 0;
    const int groups = kv_heads * ((heads / kv_heads + kLdHeads - 1) / kLdHeads), tiles = (max_seq + kLdTile - 1) / kLdTile;
    int n = sm_count / groups;
    if (n > kLdMaxSplit) n = kLdMaxSplit;
    if (n > tiles) n = tiles;
    return n < 1 ? 1 : n;
}
template <int MAXP>
static int ld_go(const LatentDecodeArgs& a, const LaunchCfg& cfg) {
    static bool once = false;
    if (!once) {
        cudaError_t e = cudaFuncSetAttribute(latent_partial_kernel<MAXP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_partial_kernel<MAXP>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    return st_launch(latent_partial_kernel<MAXP>, dim3(a.nsplit, a.group ? a.heads / a.group * ((a.group + kLdHeads - 1) / kLdHeads) : (a.heads + kLdHeads - 1) / kLdHeads), dim3(kLdThreads), (size_t)ld_smem(a.crow), cfg, a);
}
static int ld_partial(const LatentDecodeArgs& a, const LaunchCfg& cfg) { return a.kvrp <= 128 ? ld_go<1>(a, cfg) : a.kvrp <= 512 ? ld_go<4>(a, cfg) : ld_go<8>(a, cfg); }
int launch_grouped_decode(const LatentDecodeArgs& a, const LaunchCfg& cfg, const std::function<int(int, const char*)>& done) {
    if (a.group < 1 || a.heads % a.group || a.kdim % 8 || a.kvrp % 8 || a.crow != a.kdim + a.kvrp || a.kvrp > 1024 || a.nsplit < 1 || a.nsplit > kLdMaxSplit) return done((int)cudaErrorInvalidValue, "grouped_decode");
    if (int r = done(ld_partial(a, cfg), "grouped_partial")) return r;
    return done(st_launch(grouped_fold_kernel, dim3(a.heads, (a.kvrp + 127) / 128), dim3(256), 0, cfg, a), "grouped_fold");
}
int launch_latent_decode(const LatentDecodeArgs& a, const LaunchCfg& cfg, const std::function<int(int, const char*)>& done) {
    if (a.group || a.crow % 8 || a.kvrp % 8 || a.kvrp > 1024 || a.nsplit < 1 || a.nsplit > kLdMaxSplit || a.heads < 1) return done((int)cudaErrorInvalidValue, "latent_decode");
    if (int r = done(ld_partial(a, cfg), "latent_partial")) return r;
    const int slices = (a.vdim + kLfRows - 1) / kLfRows;
    LatentDecodeArgs f = a;
    f.ncl = slices <= 8 ? slices : 1;
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(a.heads, slices); lc.blockDim = dim3(256); lc.dynamicSmemBytes = (size_t)a.kvrp * 4; lc.stream = cfg.stream;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = 1; at[0].val.clusterDim.y = f.ncl; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at; lc.numAttrs = cfg.pdl ? 2 : 1;
    return done((int)cudaLaunchKernelEx(&lc, latent_fold_kernel, f), "latent_fold");
}

}  // namespace cq
