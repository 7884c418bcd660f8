// Windowed attention of a portion's queries over per-head keys and values with a shared rotated key part, a sink and an
// output gate, in bfloat16 on the tcgen05 tensor cores: prefill_attn_tc.cu's scheme with query / key rows in two parts
// (unrotated, per head; rotated, one for all heads), any lengths, and the first visible key as the first tile's start.
//
// One CTA = 128 queries of one head.  Per tile of 64 keys:
//   warp 0      TMA: the two key parts and the values in 64-column swizzled boxes (columns past a part's end arrive as
//               zeros), rings of one or two slots, keys and values apart - as deep as lets two CTAs share an SM
//   warp 1      one lane issues S = Q K^T (128 x 64 x 16 steps over both parts) into one of two TMEM buffers, and O += P V once
//               the softmax warps have written P
//   warps 2-9   two threads per query row, 32 of the tile's keys each: scale, mask, P = 2^(s - m), row sums in float32; m
//               starts at the sink, whose term is the first in the row sum, and moves - O being rescaled in TMEM - only when
//               a row's maximum outgrows it by 2^8
// Every mbarrier wait is bounded; a wait that runs out sets *err and the CTA drains.
#include "stack_dev.cuh"
#include "tcgen05.cuh"

namespace cq {

constexpr int kLpBM = 128, kLpBN = 64, kLpThreads = 320;
constexpr int kLpQBlk = kLpBM * 128, kLpKBlk = kLpBN * 128, kLpPTile = kLpBM * kLpBN * 2;

struct LatentPrefillArgs {
    CUtensorMap tqn, tqr, tkn, tkr, tv;
    bf16* out; int ldo, o_hs;
    const float* gate; int ldg, g_hs;
    const float* sink;
    int T, pos0, kbase, window, vdim, vcols;        // vcols: value columns written (vdim rounded up to eight)
    int nbn, nbr, nbv, kn_steps, kr_steps;          // 64-column blocks of each part, 16-column steps of the key parts
    int nks, nvs;                                   // ring slots
    float scale_log2, out_scale;
    int kv_group;                                   // query heads to a key / value head
    uint32_t tmem_cols;
    unsigned* err;
};

__device__ __forceinline__ float lp_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

__global__ void __launch_bounds__(kLpThreads, 2) latent_prefill_attn_kernel(const __grid_constant__ LatentPrefillArgs a) {
    extern __shared__ __align__(1024) unsigned char lp_smem[];
    const uint32_t base = smem_u32(lp_smem);
    const int nbk = a.nbn + a.nbr, kslot = nbk * kLpKBlk, vslot = a.nbv * kLpKBlk;
    const uint32_t sQ = base, sK = sQ + nbk * kLpQBlk, sV = sK + a.nks * kslot, sP = sV + a.nvs * vslot, bars = sP + kLpPTile;
    const uint32_t b_q = bars, b_kfull = bars + 8, b_kfree = bars + 24, b_vfull = bars + 40, b_vfree = bars + 56, b_sfull = bars + 72, b_p = bars + 88, b_pv = bars + 96,
                   tmem_slot = bars + 104;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y, hkv = head / a.kv_group;
    const int q0 = (gridDim.x - 1 - blockIdx.x) * kLpBM;                 // the longest rows first
    const int p_first = a.pos0 + q0, p_last = a.pos0 + min(q0 + kLpBM, a.T) - 1;
    const int k_first = a.window > 0 && p_first - a.window + 1 > 0 ? p_first - a.window + 1 : 0;
    const int nj = (p_last + 1 - k_first + kLpBN - 1) / kLpBN;
    bool failed = false;

    if (threadIdx.x == 0) {
        mbar_init(b_q, 1);
        for (int s = 0; s < 2; ++s) { mbar_init(b_kfull + 8 * s, 1); mbar_init(b_kfree + 8 * s, 1); mbar_init(b_vfull + 8 * s, 1); mbar_init(b_vfree + 8 * s, 1); mbar_init(b_sfull + 8 * s, 1); }
        mbar_init(b_p, 8); mbar_init(b_pv, 1);
        mbar_fence_init();
    }
    if (warp == 1) { tmem_alloc(tmem_slot, a.tmem_cols); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = lds32(tmem_slot);
    const uint32_t tS = tmem, tO = tmem + 2u * kLpBN;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(b_q, (uint32_t)(nbk * kLpQBlk));
            for (int b = 0; b < a.nbn; ++b) tma_load_3d(sQ + b * kLpQBlk, &a.tqn, 64 * b, head, q0, b_q);
            for (int b = 0; b < a.nbr; ++b) tma_load_3d(sQ + (a.nbn + b) * kLpQBlk, &a.tqr, 64 * b, head, q0, b_q);
            for (int j = 0; j < nj; ++j) {
                const int key = k_first + j * kLpBN;
                const int ks = j % a.nks, vs = j % a.nvs; const uint32_t kp = (uint32_t)(j / a.nks) & 1u, vp = (uint32_t)(j / a.nvs) & 1u;
                if (!mbar_wait(b_kfree + 8 * ks, kp ^ 1u)) { failed = true; break; }
                mbar_expect_tx(b_kfull + 8 * ks, (uint32_t)kslot);
                for (int b = 0; b < a.nbn; ++b) tma_load_3d(sK + ks * kslot + b * kLpKBlk, &a.tkn, 64 * b, hkv, key - a.kbase, b_kfull + 8 * ks);
                for (int b = 0; b < a.nbr; ++b) tma_load_2d(sK + ks * kslot + (a.nbn + b) * kLpKBlk, &a.tkr, 64 * b, key, b_kfull + 8 * ks);
                if (!mbar_wait(b_vfree + 8 * vs, vp ^ 1u)) { failed = true; break; }
                mbar_expect_tx(b_vfull + 8 * vs, (uint32_t)vslot);
                for (int b = 0; b < a.nbv; ++b) tma_load_3d(sV + vs * vslot + b * kLpKBlk, &a.tv, 64 * b, hkv, key - a.kbase, b_vfull + 8 * vs);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idS = umma_idesc_bf16(kLpBM, kLpBN, 0), idPV = umma_idesc_bf16(kLpBM, (a.vdim + 15) / 16 * 16, 1);
            auto issue_s = [&](int j) -> bool {
                const int ks = j % a.nks;
                if (!mbar_wait(b_kfull + 8 * ks, (uint32_t)(j / a.nks) & 1u)) return false;
                tc_fence_after();
                const uint32_t kt = sK + ks * kslot;
                for (int part = 0, blk0 = 0, acc = 0; part < 2; ++part, blk0 = a.nbn)
                    for (int st = 0; st < (part ? a.kr_steps : a.kn_steps); ++st, acc = 1) {
                        const uint32_t off = (uint32_t)((st & 3) * 32), blk = (uint32_t)(blk0 + (st >> 2));
                        umma_f16(tS + (uint32_t)((j & 1) * kLpBN), umma_desc_sw128(sQ + blk * kLpQBlk + off, 16, 1024), umma_desc_sw128(kt + blk * kLpKBlk + off, 16, 1024), idS, (uint32_t)acc);
                    }
                umma_commit(b_sfull + 8 * (j & 1));
                umma_commit(b_kfree + 8 * ks);
                return true;
            };
            if (!mbar_wait(b_q, 0u)) failed = true;
            if (!failed && !issue_s(0)) failed = true;
            for (int j = 0; j < nj && !failed; ++j) {
                const int vs = j % a.nvs;
                if (j + 1 < nj && !issue_s(j + 1)) { failed = true; break; }
                if (!mbar_wait(b_vfull + 8 * vs, (uint32_t)(j / a.nvs) & 1u) || !mbar_wait(b_p, (uint32_t)j & 1u)) { failed = true; break; }
                tc_fence_after();
#pragma unroll
                for (int st = 0; st < kLpBN / 16; ++st)
                    umma_f16(tO, umma_desc_sw128(sP + (uint32_t)(st * 32), 16, 1024), umma_desc_sw128(sV + vs * vslot + st * 2048, kLpKBlk, 1024), idPV, (uint32_t)((j | st) != 0));
                umma_commit(b_pv);
                umma_commit(b_vfree + 8 * vs);
            }
        }
    } else {
        // As in prefill_attn_tc.cu: warp w reaches the TMEM lanes 32 (w mod 4) ..; the two threads of a row agree on m through
        // shared memory; nothing leaves the loop early, after a failed wait a warp goes on without waiting.
        const int q = warp & 3, hsel = (warp - 2) >> 2, r = q * 32 + lane, qpos = p_first + r;
        const uint32_t lane_off = (uint32_t)(q * 32) << 16;
        float* mxbuf = reinterpret_cast<float*>(lp_smem + (bars - base) + 128);          // [2 halves][128 rows]
        const int nch = (a.vdim + 31) / 32;                                              // 32-column pieces of O, dealt to the two halves in turn
        const bool has_sink = a.sink != nullptr;
        float m = has_sink ? a.sink[head] * 1.4426950408889634f : -1e30f, l = has_sink && hsel == 0 ? 1.f : 0.f;
        for (int j = 0; j < nj; ++j) {
            if (!failed && !mbar_wait(b_sfull + 8 * (j & 1), ((uint32_t)j >> 1) & 1u)) failed = true;
            tc_fence_after();
            const int key0 = k_first + j * kLpBN + hsel * 32;
            const bool edge = key0 - hsel * 32 + kLpBN - 1 > p_first || (a.window > 0 && key0 - hsel * 32 <= p_last - a.window);      // some key is hidden from some query
            float x[32];
            tmem_ld32(tS + (uint32_t)((j & 1) * kLpBN + hsel * 32) + lane_off, x);
            float mxl = -INFINITY;
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                x[i] *= a.scale_log2;
                if (edge && (key0 + i > qpos || (a.window > 0 && key0 + i <= qpos - a.window))) x[i] = -INFINITY;
                mxl = fmaxf(mxl, x[i]);
            }
            mxbuf[hsel * 128 + r] = mxl;
            asm volatile("bar.sync 1, 256;" ::: "memory");
            const float mx = fmaxf(mxl, mxbuf[(hsel ^ 1) * 128 + r]);
            asm volatile("bar.sync 1, 256;" ::: "memory");
            float alpha = 1.f;
            const bool mine = mx > m + 8.0f;
            const bool moved = __any_sync(0xffffffffu, mine);
            if (mine) { alpha = lp_ex2(m - mx); m = mx; }
            float rs = 0.f;
            uint32_t pk[16];
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
                const float e0 = lp_ex2(x[i] - m), e1 = lp_ex2(x[i + 1] - m);
                rs += e0 + e1;
                pk[i >> 1] = pack_bf(e0, e1);
            }
            if (j > 0) {
                if (!failed && !mbar_wait(b_pv, (uint32_t)(j - 1) & 1u)) failed = true;
                tc_fence_after();
                if (moved) {
#pragma unroll 1
                    for (int c = hsel; c < nch; c += 2) {
                        float v[32];
                        tmem_ld32(tO + lane_off + (uint32_t)(c * 32), v);
#pragma unroll
                        for (int i = 0; i < 32; ++i) v[i] *= alpha;
                        tmem_st32(tO + lane_off + (uint32_t)(c * 32), v);
                    }
                    tmem_wait_st();
                }
            }
            const uint32_t prow = sP + (uint32_t)(r * 128);
#pragma unroll
            for (int i = 0; i < 4; ++i)
                sts128(prow + ((uint32_t)((hsel * 4 + i) ^ (r & 7)) << 4), make_uint4(pk[4 * i], pk[4 * i + 1], pk[4 * i + 2], pk[4 * i + 3]));
            l = l * alpha + rs;
            fence_async_smem();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_p);
        }
        if (hsel == 1) mxbuf[r] = l;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (hsel == 0) { l += mxbuf[r]; mxbuf[128 + r] = l; }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (hsel == 1) l = mxbuf[128 + r];
        if (!failed && !mbar_wait(b_pv, (uint32_t)(nj - 1) & 1u)) failed = true;
        tc_fence_after();
        const float inv = a.out_scale / l;
        const int t = q0 + r;
#pragma unroll 1
        for (int c = hsel; c < nch; c += 2) {
            float v[32];
            tmem_ld32(tO + lane_off + (uint32_t)(c * 32), v);
            if (t < a.T && !failed) {
                bf16* dst = a.out + (size_t)t * a.ldo + (size_t)head * a.o_hs + c * 32;
                const float* gp = a.gate ? a.gate + (size_t)t * a.ldg + (size_t)head * a.g_hs + c * 32 : nullptr;
#pragma unroll
                for (int i = 0; i < 32; i += 8) {
                    if (c * 32 + i >= a.vcols) break;
                    float o[8];
#pragma unroll
                    for (int k = 0; k < 8; ++k) o[k] = v[i + k] * inv;
                    if (gp) {
                        float gv[8];
                        load8(gp + i, gv);
#pragma unroll
                        for (int k = 0; k < 8; ++k) o[k] *= __fdividef(1.0f, 1.0f + __expf(-gv[k]));
                    }
                    *reinterpret_cast<uint4*>(dst + i) = make_uint4(pack_bf(o[0], o[1]), pack_bf(o[2], o[3]), pack_bf(o[4], o[5]), pack_bf(o[6], o[7]));
                }
            }
            __syncwarp();
        }
    }
    if (failed && a.err) atomicExch(a.err, 12u);
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, a.tmem_cols);
}

typedef CUresult (*LpEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static LpEncodeFn lp_encode() {
    static LpEncodeFn fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) p = nullptr;
        return (LpEncodeFn)p;
    }();
    return fn;
}
// [n][heads][len] with row stride ld and head stride hs (elements); heads 0: [n][len].  Box: 64 columns (x one head) x rows.
static int lp_map(CUtensorMap* m, const void* p, int len, int heads, int hs, size_t n, int ld, int box_rows) {
    LpEncodeFn fn = lp_encode();
    if (!fn) return (int)cudaErrorNotSupported;
    const cuuint64_t d3[3] = {(cuuint64_t)len, (cuuint64_t)heads, (cuuint64_t)n}, s3[2] = {(cuuint64_t)hs * 2, (cuuint64_t)ld * 2};
    const cuuint64_t d2[2] = {(cuuint64_t)len, (cuuint64_t)n}, s2[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t b3[3] = {64, 1, (cuuint32_t)box_rows}, b2[2] = {64, (cuuint32_t)box_rows}, es[3] = {1, 1, 1};
    const CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, heads ? 3 : 2, const_cast<void*>(p), heads ? d3 : d2, heads ? s3 : s2, heads ? b3 : b2, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : (int)cudaErrorInvalidValue;
}

static int lp_smem_bytes(int nbk, int nbv, int nks, int nvs) { return nbk * kLpQBlk + nks * nbk * kLpKBlk + nvs * nbv * kLpKBlk + kLpPTile + 128 + 1024; }

bool latent_prefill_fits(int dn, int dr, int dv) {
    return dv <= 256 && lp_smem_bytes((dn + 63) / 64 + (dr + 63) / 64, (dv + 63) / 64, 1, 1) <= 225 * 1024;
}
int launch_latent_prefill_attn(const LatentAttnArgs& t, int n_keys, size_t cache_rows, unsigned* err, const LaunchCfg& cfg) {
    if (t.T < 1 || t.heads < 1 || t.pos_ptr || t.out_f32 || n_keys < 1 || (t.kv_group > 1 && t.heads % t.kv_group) || !latent_prefill_fits(t.dn, t.dr, t.dv) || ((t.ldqn | t.qn_hs | t.ldqr | t.qr_hs | t.ldkn | t.kn_hs | t.ldkr | t.ldv | t.v_hs | t.ldo | t.o_hs) & 7))
        return (int)cudaErrorInvalidValue;
    LatentPrefillArgs a{};
    if (int r = lp_map(&a.tqn, t.qn, t.dn, t.heads, t.qn_hs, (size_t)t.T, t.ldqn, kLpBM)) return r;
    if (t.dr > 0) if (int r = lp_map(&a.tqr, t.qr, t.dr, t.heads, t.qr_hs, (size_t)t.T, t.ldqr, kLpBM)) return r;
    const int grp = t.kv_group > 1 ? t.kv_group : 1, kvh = t.heads / grp;
    if (int r = lp_map(&a.tkn, t.kn, t.dn, kvh, t.kn_hs, (size_t)n_keys, t.ldkn, kLpBN)) return r;
    if (t.dr > 0) if (int r = lp_map(&a.tkr, t.kr, t.dr, 0, 0, cache_rows, t.ldkr, kLpBN)) return r;
    if (int r = lp_map(&a.tv, t.v, t.dv, kvh, t.v_hs, (size_t)n_keys, t.ldv, kLpBN)) return r;
    a.out = (bf16*)t.out; a.ldo = t.ldo; a.o_hs = t.o_hs; a.gate = t.gate; a.ldg = t.ldg; a.g_hs = t.g_hs; a.sink = t.sink;
    a.T = t.T; a.pos0 = t.pos0; a.kbase = t.kbase; a.window = t.window; a.vdim = t.dv; a.vcols = (t.dv + 7) / 8 * 8;
    a.nbn = (t.dn + 63) / 64; a.nbr = (t.dr + 63) / 64; a.nbv = (t.dv + 63) / 64; a.kn_steps = (t.dn + 15) / 16; a.kr_steps = (t.dr + 15) / 16;
    a.scale_log2 = t.scale * 1.4426950408889634f; a.out_scale = t.out_scale; a.kv_group = grp; a.err = err;
    a.tmem_cols = t.dv <= 128 ? 256u : 512u;
    // two slots each if two CTAs still fit an SM (and its TMEM), else one each if that lets them; a CTA that has the SM to itself takes two
    const int nbk = a.nbn + a.nbr, half = 113 * 1024;
    a.nks = a.nvs = 2;
    if (a.tmem_cols == 256u && lp_smem_bytes(nbk, a.nbv, 2, 2) > half) {
        if (lp_smem_bytes(nbk, a.nbv, 1, 2) <= half) a.nks = 1;
        else if (lp_smem_bytes(nbk, a.nbv, 1, 1) <= half) a.nks = a.nvs = 1;
    }
    if (lp_smem_bytes(nbk, a.nbv, a.nks, a.nvs) > 225 * 1024) a.nks = a.nvs = 1;
    static bool once = false;
    if (!once) {
        const cudaError_t e = cudaFuncSetAttribute(latent_prefill_attn_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    return st_launch(latent_prefill_attn_kernel, dim3((t.T + kLpBM - 1) / kLpBM, t.heads), dim3(kLpThreads), (size_t)lp_smem_bytes(nbk, a.nbv, a.nks, a.nvs), cfg, a);
}

}  // namespace cq
