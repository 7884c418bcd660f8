// bfloat16 member of the GEMV family, for designs whose layers feed one vector to several matrices: up to six matrices
// ("segments") side by side in one launch, or two matrices summed into the same rows.  The data path is gemv.cuh's - a
// producer warp streams boxes of the row-major weights into a ring of shared-memory stages, eight consumer warps run the
// tensor-core inner product (mma.sync m16n8k16, fp32 accumulation) - with float32 input vectors that the prologue
// normalises and narrows, and an epilogue per segment.
//
//   SEG_NORM    x' = x + y / rms(y) * y_w (y may be null; CTA 0 stores x'), then one or two copies x' / rms(x') * nw[i]
//               narrowed to bfloat16; every segment names the copy it multiplies
//   SEG_MIX     h = x / rms(x) * nw[0] (CTA 0 leaves it in the ring of previous rows), copy 0 = h, copy i = h + (previous
//               token's h - h) * mu[i - 1]; a CTA makes the copies that its segments read
//   SEG_NARROW  x itself, narrowed
//   SEG_PLAIN   one or two bfloat16 vectors end to end; with two, columns [0, kp[0]) come from matrix 0 and the rest from
//               matrix 1, and both add into the one segment's rows
#pragma once
#include <cuda.h>

#include "stack.h"

namespace cq {

enum SegStage : int { SEG_PLAIN = 0, SEG_NORM = 1, SEG_NARROW = 2, SEG_MIX = 3 };
constexpr int kSegMax = 6;

struct alignas(64) SegGemvArgs {
    CUtensorMap tmap[kSegMax];
    int stage;
    const bf16* xb[2]; int klen[2], kp[2];          // SEG_PLAIN: vectors, their lengths (a multiple of 8) and the padded lengths (multiples of 128)
    const float *x, *y, *y_w; float* x_next;        // SEG_NORM / SEG_NARROW
    const float* nw[2]; int nvar; float eps; int width;
    const float* mu; int ldmu; float* prev; int ldprev; const int* pos_ptr;    // SEG_MIX: prev = two rows by position parity
    float c0, c1;                                   // constants of the epilogues
    int K;                                          // staged columns, a multiple of 128
    int nseg, seg_rows[kSegMax], seg_blk0[kSegMax], seg_var[kSegMax], epi[kSegMax]; void* out[kSegMax];      // epi: LinEpi
    const bf16* side; int side_pitch, side_dim; const int* tokens;             // LIN_GELU_SIDE
    int brows, nblk, rw, kw, nst;                   // rows of a CTA block, blocks, row-warps x K-parts, ring stages
    unsigned* err;
    int has_kv; LatentRowsArgs kv;                  // one CTA more than the blocks need: the token's cache row (its dkv half)
};

struct SegMat { const bf16* w; int rows, pitch; };   // rows as stored, pitch = columns as stored (a multiple of 128)
// Fills the maps and the work split and launches.  SEG_PLAIN with kp[1] > 0: mats[0] and mats[1] are the two summed matrices.
int launch_gemv_seg(SegGemvArgs& a, const SegMat* mats, int nmat, const LaunchCfg& cfg);

}  // namespace cq
