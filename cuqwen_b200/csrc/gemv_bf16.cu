// The bfloat16 GEMV kernel (see gemv_seg.cuh) and its launcher.
#include "gemv_seg.cuh"
#include "gemv_stage.cuh"
#include "stack_dev.cuh"

namespace cq {

constexpr int kSgWarps = 8, kSgThreads = (kSgWarps + 1) * 32, kSgNC = kSgWarps * 32;
constexpr int kSgPiece = 256;                       // bytes of a row per ring step and K-part: 128 columns
struct SegLayout { int off_x, off_f, off_red, off_ring, box_stride, stage_bytes, off_bars, total; };
__host__ __device__ inline SegLayout seg_layout(int K, int nvar, bool f32, bool pending, int brows, int kw, int nst) {
    SegLayout L;
    int o = 0;
    L.off_x = o; o += nvar * K * 2;
    L.off_f = o; o += f32 ? (pending ? 8 : 4) * K : 0;
    L.off_red = o; o += (kSgWarps * 16 + 40) * 4;
    o = (o + 127) / 128 * 128;
    L.off_ring = o;
    L.box_stride = brows * kSgPiece;                // a multiple of 128
    L.stage_bytes = kw * L.box_stride;
    o += nst * L.stage_bytes;
    o += 1024;                                      // a block of fewer than 16 rows per row-warp lets fragment loads run up to 15 rows past the last box
    L.off_bars = o; o += 2 * nst * 8;
    L.total = o;
    return L;
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// 1 / sqrt(sum / n + eps) over the consumer threads
__device__ __forceinline__ float seg_inv_rms(float ss, int n, float eps, float* red) {
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    consumer_sync(kSgNC);
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < kSgWarps; ++i) v += red[i];
    consumer_sync(kSgNC);                           // red is free again
    return inv_rms(v, n, eps);
}

// The input vector as bfloat16 in shared memory.  A thread owns the float4 units tid, tid + 256, ... of the vector from the
// first load to the last store, so only the sums need barriers.
__device__ __forceinline__ void seg_stage(const SegGemvArgs& a, unsigned char* sm, const SegLayout& L, bool first, unsigned vars) {
    const int tid = threadIdx.x;
    if (a.stage == SEG_PLAIN) {
        uint4* xs = reinterpret_cast<uint4*>(sm + L.off_x);
        for (int p = 0; p < 2; ++p) {
            const uint4* src = reinterpret_cast<const uint4*>(a.xb[p]);
#pragma unroll 4
            for (int i = tid; i < a.kp[p] / 8; i += kSgNC) xs[i] = i < a.klen[p] / 8 ? __ldcg(src + i) : make_uint4(0u, 0u, 0u, 0u);
            xs += a.kp[p] / 8;
        }
        consumer_sync(kSgNC);
        return;
    }
    float4* xf = reinterpret_cast<float4*>(sm + L.off_f);
    float* red = reinterpret_cast<float*>(sm + L.off_red);
    const int n4 = (a.width + 3) / 4, k4 = a.K / 4;         // the source vectors are padded with zeros to a multiple of eight
    const float4* x = reinterpret_cast<const float4*>(a.x);
    float ss = 0.f;
    if (a.y) {
        float4* yf = xf + k4;
        const float4 *y = reinterpret_cast<const float4*>(a.y), *yw = reinterpret_cast<const float4*>(a.y_w);
        float sy = 0.f;
#pragma unroll 4
        for (int i = tid; i < n4; i += kSgNC) {
            const float4 v = __ldcg(y + i);
            xf[i] = __ldcg(x + i); yf[i] = v;
            sy += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        const float inv = seg_inv_rms(sy, a.width, a.eps, red);
#pragma unroll 4
        for (int i = tid; i < n4; i += kSgNC) {
            float4 v = xf[i];
            const float4 u = yf[i], w = __ldg(yw + i);
            v.x += u.x * inv * w.x; v.y += u.y * inv * w.y; v.z += u.z * inv * w.z; v.w += u.w * inv * w.w;
            xf[i] = v;
            if (first && a.x_next) reinterpret_cast<float4*>(a.x_next)[i] = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
#pragma unroll 4
        for (int i = tid; i < n4; i += kSgNC) {
            const float4 v = __ldcg(x + i);
            xf[i] = v;
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    }
    const bool norm = a.stage == SEG_NORM || a.stage == SEG_MIX;
    const float inv = norm ? seg_inv_rms(ss, a.width, a.eps, red) : 1.f;
    if (a.stage == SEG_MIX) {
        const int pos = *a.pos_ptr;
        const float4 *w = reinterpret_cast<const float4*>(a.nw[0]), *prev = reinterpret_cast<const float4*>(a.prev + (size_t)((pos + 1) & 1) * a.ldprev);
        float4* keep = reinterpret_cast<float4*>(a.prev + (size_t)(pos & 1) * a.ldprev);
#pragma unroll 2
        for (int i = tid; i < k4; i += kSgNC) {
            float4 h = make_float4(0.f, 0.f, 0.f, 0.f), p = h;
            if (i < n4) {
                h = xf[i];
                const float4 g = __ldg(w + i);
                if (pos > 0) p = __ldcg(prev + i);
                h.x *= inv * g.x; h.y *= inv * g.y; h.z *= inv * g.z; h.w *= inv * g.w;
                if (first) keep[i] = h;
            }
            for (int k = 0; k < a.nvar; ++k) {
                if (!(vars >> k & 1u)) continue;
                float4 v = h;
                if (k > 0 && i < n4) {
                    const float4 m = __ldg(reinterpret_cast<const float4*>(a.mu + (size_t)(k - 1) * a.ldmu) + i);
                    v = make_float4(fmaf(p.x - h.x, m.x, h.x), fmaf(p.y - h.y, m.y, h.y), fmaf(p.z - h.z, m.z, h.z), fmaf(p.w - h.w, m.w, h.w));
                }
                reinterpret_cast<uint2*>(sm + L.off_x + k * a.K * 2)[i] = make_uint2(pack_bf(v.x, v.y), pack_bf(v.z, v.w));
            }
        }
        consumer_sync(kSgNC);
        return;
    }
    for (int k = 0; k < a.nvar; ++k) {
        uint2* o = reinterpret_cast<uint2*>(sm + L.off_x + k * a.K * 2);
        const float4* w = reinterpret_cast<const float4*>(a.nw[k]);
#pragma unroll 4
        for (int i = tid; i < k4; i += kSgNC) {
            uint2 r = make_uint2(0u, 0u);
            if (i < n4) {
                float4 v = xf[i];
                if (norm) { const float4 g = __ldg(w + i); v.x *= inv * g.x; v.y *= inv * g.y; v.z *= inv * g.z; v.w *= inv * g.w; }
                r = make_uint2(pack_bf(v.x, v.y), pack_bf(v.z, v.w));
            }
            o[i] = r;
        }
    }
    consumer_sync(kSgNC);
}

__device__ __forceinline__ void seg_finish(const SegGemvArgs& a, int seg, int row, float v, float pre) {
    switch (a.epi[seg]) {
        case LIN_F32: reinterpret_cast<float*>(a.out[seg])[row] = v; break;
        case LIN_ACT: reinterpret_cast<bf16*>(a.out[seg])[row] = __float2bfloat16_rn(v); break;
        case LIN_RELU2: { const float p = fmaxf(v, 0.f); reinterpret_cast<bf16*>(a.out[seg])[row] = __float2bfloat16_rn(p * p); break; }
        case LIN_ADD: reinterpret_cast<float*>(a.out[seg])[row] = pre + a.c0 * v; break;
        case LIN_CAP: reinterpret_cast<float*>(a.out[seg])[row] = a.c0 * tanhf(v / a.c0); break;
        case LIN_GELU_SIDE: reinterpret_cast<bf16*>(a.out[seg])[row] = __float2bfloat16_rn(gelu_tanh_f(v) * pre); break;
    }
}
// Row `row` of the gate and row + 8 of the up matrix (LIN_GLU: eight rows of each in turn).
__device__ __forceinline__ void seg_finish_glu(const SegGemvArgs& a, int seg, int row, float gate, float up) {
    reinterpret_cast<bf16*>(a.out[seg])[(row >> 4) * 8 + (row & 7)] = __float2bfloat16_rn(clamped_glu_f(gate, up, a.c0, a.c1));
}
// The epilogue's operand from global memory, fetched before the block's arithmetic.
__device__ __forceinline__ float seg_fetch(const SegGemvArgs& a, int seg, int row, int row_end) {
    if (row >= row_end) return 0.f;
    if (a.epi[seg] == LIN_ADD) return __ldcg(reinterpret_cast<const float*>(a.out[seg]) + row);
    if (a.epi[seg] == LIN_GELU_SIDE) return row < a.side_dim ? __bfloat162float(a.side[(size_t)(*a.tokens) * a.side_pitch + row]) : 0.f;
    return 0.f;
}

// The cache row of the step's token: the normed latent and the rotated key part (LatentRowsArgs' dkv half), consumer threads.
__device__ __forceinline__ void seg_cache_row(const LatentRowsArgs& a, float* red) {
    const int pos = *a.pos_ptr, tid = threadIdx.x;
    float ss = 0.f;
    for (int i = tid; i < a.kv_rank; i += kSgNC) { const float v = __ldcg(a.dkv + i); ss += v * v; }
    const float inv = seg_inv_rms(ss, a.kv_rank, a.eps, red);
    bf16* o = reinterpret_cast<bf16*>(a.cache) + (size_t)pos * a.ldc;
    for (int i = tid; i < a.kv_rank; i += kSgNC) o[i] = __float2bfloat16_rn(__ldcg(a.dkv + i) * inv * a.dkv_w[i]);
    const int half = a.rot_dim / 2;
    for (int i = tid; i < half; i += kSgNC) {
        const float2 cs = a.rot[(size_t)pos * half + i];
        const float u = __ldcg(a.dkv + a.kr_off + i), v = __ldcg(a.dkv + a.kr_off + half + i);
        o[a.kr_off + i] = __float2bfloat16_rn(u * cs.x - v * cs.y);
        o[a.kr_off + half + i] = __float2bfloat16_rn(v * cs.x + u * cs.y);
    }
}

__global__ void __launch_bounds__(kSgThreads, 1) gemv_seg_kernel(const __grid_constant__ SegGemvArgs a) {
    extern __shared__ __align__(128) unsigned char sg_smem[];
    pdl_launch_dependents();
    const SegLayout L = seg_layout(a.K, a.stage == SEG_PLAIN ? 1 : a.nvar, a.stage != SEG_PLAIN, a.y != nullptr, a.brows, a.kw, a.nst);
    const uint32_t sm0 = smem_u32(sg_smem), bar_full = sm0 + L.off_bars, bar_empty = bar_full + 8 * a.nst;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ncta = gridDim.x - a.has_kv;
    if ((int)blockIdx.x == ncta) {                              // the extra CTA
        if (warp < kSgWarps) { pdl_wait(); seg_cache_row(a.kv, reinterpret_cast<float*>(sg_smem + L.off_red)); }
        return;
    }
    if (threadIdx.x == 0) {
        for (int s = 0; s < a.nst; ++s) { mbar_init(bar_full + 8 * s, 1); mbar_init(bar_empty + 8 * s, kSgWarps); }
        mbar_fence_init();
    }
    __syncthreads();
    const int PT = a.K / 128, kw = a.kw, S = (PT + kw - 1) / kw, PT0 = a.stage == SEG_PLAIN ? a.kp[0] / 128 : PT;
    bool failed = false;
    int slot = 0; uint32_t par = 0;
    if (warp == kSgWarps) {
        for (int blk = blockIdx.x; blk < a.nblk; blk += ncta) {
            int seg = 0;
            while (seg + 1 < a.nseg && blk >= a.seg_blk0[seg + 1]) ++seg;
            const int row = (blk - a.seg_blk0[seg]) * a.brows;
            for (int p = 0; p < S; ++p) {
                if (!failed && !mbar_wait(bar_empty + 8 * slot, par ^ 1u)) { failed = true; if (a.err) atomicExch(a.err, 4u); }
                int parts = PT - p * kw; if (parts > kw) parts = kw;
                if (lane == 0) mbar_expect_tx(bar_full + 8 * slot, (uint32_t)(parts * L.box_stride));
                __syncwarp();
                if (lane < parts) {
                    const int c = p * kw + lane;
                    const int map = c < PT0 ? seg : 1, cc = c < PT0 ? c : c - PT0;
                    tma_load_3d(sm0 + L.off_ring + slot * L.stage_bytes + lane * L.box_stride, &a.tmap[map], 0, row, cc * (kSgPiece / kChunkBytes), bar_full + 8 * slot);
                }
                if (++slot == a.nst) { slot = 0; par ^= 1u; }
            }
        }
        return;
    }
    pdl_wait();
    unsigned vars = 0;                                          // copies of the input that this CTA's segments read
    if (a.stage == SEG_MIX)
        for (int blk = blockIdx.x; blk < a.nblk; blk += ncta) {
            int seg = 0;
            while (seg + 1 < a.nseg && blk >= a.seg_blk0[seg + 1]) ++seg;
            vars |= 1u << a.seg_var[seg];
        }
    seg_stage(a, sg_smem, L, blockIdx.x == 0, vars);
    float* red = reinterpret_cast<float*>(sg_smem + L.off_red);
    const int g = lane >> 2, t = lane & 3, rwi = warp % a.rw, kwi = warp / a.rw;
    const int cstride = a.brows * kChunkBytes;
    for (int blk = blockIdx.x; blk < a.nblk; blk += ncta) {
        int seg = 0;
        while (seg + 1 < a.nseg && blk >= a.seg_blk0[seg + 1]) ++seg;
        const int b0 = (blk - a.seg_blk0[seg]) * a.brows, row0 = b0 + rwi * 16;
        const int row_end = min(b0 + a.brows, a.seg_rows[seg]);
        const bool live = row0 < row_end && kwi < kw;
        const uint4* xs = reinterpret_cast<const uint4*>(sg_smem + L.off_x + (a.stage == SEG_PLAIN ? 0 : a.seg_var[seg] * a.K * 2));
        float preA = 0.f, preB = 0.f;
        if (kw > 1) { if (kwi == 0 && lane < 16) preA = seg_fetch(a, seg, row0 + lane, row_end); }
        else if (t == 0) { preA = seg_fetch(a, seg, row0 + g, row_end); preB = seg_fetch(a, seg, row0 + g + 8, row_end); }
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
        for (int p = 0; p < S; ++p) {
            if (!failed && !mbar_wait(bar_full + 8 * slot, par)) { failed = true; if (a.err) atomicExch(a.err, 1u); }
            const int c = p * kw + kwi;
            if (live && c < PT) {
                const uint32_t wrow = sm0 + L.off_ring + slot * L.stage_bytes + kwi * L.box_stride + (rwi * 16 + g) * kChunkBytes + t * 16;
                uint4 wa[4], wb[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) { wa[i] = lds128(wrow + i * cstride); wb[i] = lds128(wrow + 8 * kChunkBytes + i * cstride); }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const uint4 xv = xs[c * 16 + i * 4 + t];
                    mma_bf16(c0, wa[i].x, wb[i].x, wa[i].y, wb[i].y, xv.x, xv.y);
                    mma_bf16(c1, wa[i].z, wb[i].z, wa[i].w, wb[i].w, xv.z, xv.w);
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_empty + 8 * slot);
            if (++slot == a.nst) { slot = 0; par ^= 1u; }
        }
        const float vA = c0[0] + c1[0], vB = c0[2] + c1[2];
        if (kw > 1) {
            if (t == 0) { red[warp * 16 + g] = vA; red[warp * 16 + g + 8] = vB; }
            consumer_sync(kSgNC);
            if (a.epi[seg] == LIN_GLU) {
                if (kwi == 0 && lane < 8 && row0 + lane < row_end) {
                    float v = 0.f, u = 0.f;
                    for (int k = 0; k < kw; ++k) { v += red[(k * a.rw + rwi) * 16 + lane]; u += red[(k * a.rw + rwi) * 16 + lane + 8]; }
                    seg_finish_glu(a, seg, row0 + lane, v, u);
                }
            } else if (kwi == 0 && lane < 16 && row0 + lane < row_end) {
                float v = 0.f;
                for (int k = 0; k < kw; ++k) v += red[(k * a.rw + rwi) * 16 + lane];
                seg_finish(a, seg, row0 + lane, v, preA);
            }
            consumer_sync(kSgNC);
        } else if (t == 0 && live) {
            if (a.epi[seg] == LIN_GLU) { if (row0 + g < row_end) seg_finish_glu(a, seg, row0 + g, vA, vB); }
            else {
                if (row0 + g < row_end) seg_finish(a, seg, row0 + g, vA, preA);
                if (row0 + g + 8 < row_end) seg_finish(a, seg, row0 + g + 8, vB, preB);
            }
        }
    }
}

int launch_gemv_seg(SegGemvArgs& a, const SegMat* mats, int nmat, const LaunchCfg& cfg) {
    const bool two = a.stage == SEG_PLAIN && a.kp[1] > 0;
    if (nmat < 1 || nmat > kSegMax || (two && nmat != 2) || a.K < 128 || a.K % 128 || (a.stage == SEG_PLAIN && a.K != a.kp[0] + a.kp[1])) return (int)cudaErrorInvalidValue;
    a.nseg = two ? 1 : nmat;
    int total = 0;
    for (int s = 0; s < a.nseg; ++s) { a.seg_rows[s] = mats[s].rows; total += mats[s].rows; }
    // Block height: the rows spread evenly over the SMs in as few rounds of at most 128 rows as it takes.
    const int sms = cfg.sm_count;
    const int rounds = (total + 128 * sms - 1) / (128 * sms);
    int brows = (total + rounds * sms - 1) / (rounds * sms);
    if (brows < 8) brows = 8;
    bool glu = false;                                // its pairs of rows lie in one 16-row tile
    for (int s = 0; s < a.nseg; ++s) if (a.epi[s] == LIN_GLU) { glu = true; if (mats[s].rows % 16) return (int)cudaErrorInvalidValue; }
    const int step = glu ? 16 : 1;
    brows = (brows + step - 1) / step * step;
    auto blocks = [&](int br) { int n = 0; for (int s = 0; s < a.nseg; ++s) n += (mats[s].rows + br - 1) / br; return n; };
    while (brows < 128 && blocks(brows) > rounds * sms) brows += step;
    a.brows = brows;
    a.nblk = 0;
    for (int s = 0; s < a.nseg; ++s) { a.seg_blk0[s] = a.nblk; a.nblk += (mats[s].rows + brows - 1) / brows; }
    int rw = 1;
    while (16 * rw < brows) rw *= 2;
    int kw = kSgWarps / rw;
    while (kw > 1 && kw > a.K / 128) kw /= 2;
    a.rw = rw; a.kw = kw;
    const int nvar = a.stage == SEG_PLAIN ? 1 : a.nvar;
    int nst = 8;
    auto total_smem = [&](int n) { return seg_layout(a.K, nvar, a.stage != SEG_PLAIN, a.y != nullptr, brows, kw, n).total; };
    while (nst > 1 && total_smem(nst) > 222 * 1024) --nst;
    if (total_smem(nst) > 222 * 1024) return (int)cudaErrorInvalidValue;
    a.nst = nst;
    for (int m = 0; m < nmat; ++m)
        if (int r = make_weight_map(&a.tmap[m], mats[m].w, (size_t)mats[m].pitch * 2, (size_t)mats[m].rows, kSgPiece, brows)) return r;
    static bool once = false;
    if (!once) {
        cudaError_t e = cudaFuncSetAttribute(gemv_seg_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(gemv_seg_kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
        if (e != cudaSuccess) return (int)e;
        once = true;
    }
    const int grid = (a.nblk < sms ? a.nblk : sms) + a.has_kv;
    return st_launch(gemv_seg_kernel, dim3(grid), dim3(kSgThreads), (size_t)total_smem(nst), cfg, a);
}

}  // namespace cq
