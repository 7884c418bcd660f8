// Designs described layer by layer (model_dir.h): argument blocks and launchers of their kernels, and the host object that
// holds their weights, cache and workspace.  The engine's entry points (engine.cu) drive it: the same control block,
// mailbox, CUDA graph, sampler and prefill calls as the models of the table.
//
// Activations are bfloat16 or float32 (Act); weights are bfloat16 as stored, norm weights and sinks are widened to float32.
// The residual stream, norms, angles, scores, softmax and every accumulation are float32 in both.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <functional>

#include "common.cuh"
#include "launch.h"

namespace cq {

typedef __nv_bfloat16 bf16;
enum Act : int { ACT_BF16 = 0, ACT_F32 = 1 };

// ---- row kernels (stack_rows.cu) ---------------------------------------------------------------------------------------
// x[t] = scale * embed[tokens[t]]
int launch_st_embed(const bf16* table, int pitch, const int* tokens, float* x, int ldx, int width, float scale, int T, const LaunchCfg& cfg);
// The first launch of a decode step: takes over the mailbox, then the same for ctl->token.
int launch_st_embed_step(const bf16* table, int pitch, StepCtl* ctl, float* x, int width, float scale, const LaunchCfg& cfg);

// Per row: x += y / rms(y) * y_w (y may be null), then n_out copies x / rms(x) * w[i] -> out[i].
struct NormRowsArgs {
    float* x; int ldx;
    const float* y; int ldy; const float* y_w;
    const float* w[2]; void* out[2]; int ldo; int n_out;
    int width; float eps;
    const int* rows;      // row t of the output comes from row rows[t] of x (null: t); y must be null then
};
int launch_st_norms(int act, const NormRowsArgs& a, int T, const LaunchCfg& cfg);

// out[t] = x[t] in the activation type
int launch_st_narrow(int act, const float* x, int ldx, void* out, int ldo, int T, const LaunchCfg& cfg);

// Per row: the query latent and the cache row of a token from the raw projections.
//   cq[t] = dq / rms(dq) * dq_w;  cache row pos = [ckv / rms(ckv) * dkv_w | rotated key part]
struct LatentRowsArgs {
    const float* dq; int ld; const float* dq_w; void* cq; int ldcq; int q_rank;      // dq null: only the cache row
    const float* dkv;                                   // null: the layer has no latent projection of its own
    const float* dkv_w; void* cache; int ldc, kv_rank, kr_off, rot_dim;      // kr_off: where the rotated part starts, in dkv rows and in cache rows
    const float2* rot;                                  // (cos, sin) [position][rot_dim / 2]
    float eps;
    const int* pos_ptr; int pos0;                       // position of row t: (pos_ptr ? *pos_ptr : pos0) + t
};
int launch_st_latent_rows(int act, const LatentRowsArgs& a, int T, const LaunchCfg& cfg);

// q[t][h] = [unrotated dim | rotated rot_dim], heads head_pitch apart, rot part at rot_off: rotated and narrowed.
struct RopeQArgs { const float* in; void* out; int ld, heads, head_pitch, rot_off, rot_dim; const float2* rot; const int* pos_ptr; int pos0; };
int launch_st_rope_q(int act, const RopeQArgs& a, int T, const LaunchCfg& cfg);

// ---- matrix products of both activation types on the CUDA cores (stack_linear.cu) -----------------------------------
enum LinEpi : int {
    LIN_F32 = 0,          // out (float) = acc
    LIN_ACT = 1,          // out (activation type) = acc
    LIN_RELU2 = 2,        // out (activation type) = max(acc, 0)^2
    LIN_ADD = 3,          // out (float) += c0 * acc
    LIN_GELU_SIDE = 4,    // out (activation type) = gelu_tanh(acc) * side[tokens[t]][r]
    LIN_CAP = 5,          // out (float) = c0 * tanh(acc / c0)
    LIN_GLU = 6,          // out (activation type) = clamped_glu(gate, up, limit c0, slope c1); rows come as eight of the gate, eight of the up matrix in turn
    LIN_DECAY = 7         // out (float) = exp(-exp(acc + bias[r]))
};
struct LinArgs {
    const void* x; int ldx; const bf16* w; int pitch, K;
    const void* x2; int ldx2; const bf16* w2; int pitch2, K2;      // a second product summed into the same rows (w2 null: none)
    int T, R, epi;
    void* out; int ldo;
    const bf16* side; int side_pitch, side_dim; const int* tokens; // LIN_GELU_SIDE
    float c0, c1;                                                  // constants of the epilogue
    const float* bias;                                             // LIN_DECAY
};
// LIN_GLU is not among its epilogues: LIN_F32, then launch_st_glu_rows.
int launch_st_linear(int act, const LinArgs& a, const LaunchCfg& cfg);

// ---- latent attention (latent_attn.cu) -------------------------------------------------------------------------------
// Softmax attention over [unrotated | rotated] keys with a window, a sink and an output gate.  Keys and values either
// per head (prefill: k = W_uk c, v = W_uv c of every key in reach) or the latents themselves (decode: queries carried
// into the latent space by absorb_q, values left there for uv_gate).  Grouped attention is the same with one key part (dr 0)
// and several query heads to a key / value head (kv_group).
struct LatentAttnArgs {
    const void *qn, *qr; int ldqn, qn_hs, dn, ldqr, qr_hs, dr;      // unrotated and rotated query parts: row stride, head stride, length
    const void* kn; int ldkn, kn_hs;                                // unrotated keys; row 0 is key `kbase`
    const void* kr; int ldkr;                                       // rotated keys, shared by the heads; row 0 is key 0
    const void* v; int ldv, v_hs, dv;                               // values; row 0 is key `kbase`
    int kbase;
    const float* sink;                                              // [heads] or null
    const float* gate; int ldg, g_hs;                               // out *= sigmoid(gate), or null
    void* out; int ldo, o_hs;                                       // activation type, or float when out_f32
    int out_f32;
    int T, heads, window;                                           // window 0: all earlier keys
    float scale;
    const int* pos_ptr; int pos0;
    int kv_group;                                                   // query heads that share a key / value head (0 and 1: none)
    float out_scale;                                                // factor of the output
};
int launch_latent_attn(int act, const LatentAttnArgs& a, const LaunchCfg& cfg);
// The same for bfloat16 portions on the tensor cores (latent_prefill_attn.cu), where the sizes fit: keys and values hold n_keys
// rows from kbase on, kr the cache's cache_rows.
bool latent_prefill_fits(int dn, int dr, int dv);
int launch_latent_prefill_attn(const LatentAttnArgs& a, int n_keys, size_t cache_rows, unsigned* err, const LaunchCfg& cfg);
// One token's queries as the cache rows are laid out: out[h] = [W_uk[h]^T q[h] (kv_rank) | rotated q[h] (rot_dim, from
// kr_off)], so that a score is one dot product with a cache row.  q float [heads][q_hs], its rotated part from rot_off.
struct AbsorbArgs {
    const float* q; int q_hs, rot_off, rot_dim; const float2* rot; const int* pos_ptr;
    const bf16* wk; int pitch, heads, dim, dimp; void* out; int ldo, kr_off;
};
int launch_absorb_q(int act, const AbsorbArgs& a, const LaunchCfg& cfg);
// bfloat16 decode attention over cache rows, split over the keys (latent_decode.cu): partials, then one kernel that merges
// them, multiplies with W_uv and applies the gate.
struct LatentDecodeArgs {
    const bf16* q; int crow;                             // [heads][crow], crow = kv_rank (padded) + rot_dim (padded)
    const bf16* cache; int kvrp;                         // rows [crow]; the values are their first kvrp places
    const float* sink; int heads, window; float scale; const int* pos_ptr;
    int nsplit; float* part_o; float* part_ml;           // [nsplit][heads][kvrp], [nsplit][heads][2]
    int ncl;                                             // set by the launcher: CTAs of a head that share the merge
    const bf16* wv; int pitch, vdim, vdimp, kv_rank; const float* gate; int g_hs; bf16* out; int o_hs;
    // Grouped attention: a cache of rows [key kdim | value kvrp] per key / value head, group query heads to each, kv_stride
    // elements from head to head; group 0: one cache for all heads whose rows are key and value at once.
    int group, kdim; size_t kv_stride; float out_scale;
};
// Splits that launch_latent_decode wants for a cache of max_seq rows; 0 = sizes it does not cover.
int latent_decode_splits(int heads, int crow, int kvrp, int window, int max_seq, int sm_count);
int launch_latent_decode(const LatentDecodeArgs& a, const LaunchCfg& cfg, const std::function<int(int, const char*)>& done);
// The grouped form; the fold writes the merged heads times out_scale.
int grouped_decode_splits(int heads, int kv_heads, int kdim, int vdimp, int max_seq, int sm_count);
int launch_grouped_decode(const LatentDecodeArgs& a, const LaunchCfg& cfg, const std::function<int(int, const char*)>& done);
// att[h][v] = sigmoid(g[h][v]) * sum_r W_uv[h][v][r] o[h][r].  o float [heads][ldo].
struct UvGateArgs { const float* o; int ldo; const bf16* wv; int pitch, heads, vdim, vdimp, kv_rank; const float* gate; int g_hs; void* out; int o_hs; };
int launch_uv_gate(int act, const UvGateArgs& a, const LaunchCfg& cfg);

// ---- grouped attention (grouped_attn.cu) -------------------------------------------------------------------------------
// Rows of raw projections [q heads x dimp | k kv_heads x dimp | v kv_heads x vdimp]: rotated queries to q, [rotated key | value]
// to the cache [kv_heads][max_seq][dimp + vdimp] at the rows' positions.
struct QkvRowsArgs {
    const float* raw; int ld, k_off, v_off;
    int heads, kv_heads, dim, dimp, vdimp;
    void* q; int ldq; void* cache; int max_seq;
    const float2* rot; int rot_dims;                                // rot_dims 0: no rotation
    const int* pos_ptr; int pos0;
};
int launch_qkv_rows(int act, const QkvRowsArgs& a, int T, const LaunchCfg& cfg);

// ---- recurrent mixers ---------------------------------------------------------------------------------------------------
// States live from token to token: float32, zero at position 0.  Everything that enters a recurrence is float32 as well.
//
// h = norm(x); out variant 0 = h, variant i = h + (previous token's h - h) * mu[i - 1].  prev: ring of two rows by position
// parity; the last row's h goes to `tail` (launch_tail_rows puts it into the ring once every row has been read).
struct ShiftRowsArgs {
    const float* x; int ldx; const float* w; int width; float eps;
    void* out; int ldo; size_t var_stride; const float* mu; int ldmu, n_mix;
    const float* prev; int ldprev; float* tail;
    const int* pos_ptr; int pos0;
};
int launch_shift_rows(int act, const ShiftRowsArgs& a, int T, const LaunchCfg& cfg);
// The last min(T, keep) rows of src (row t at position pos0 + t) into ring rows by position (mod slots).
struct TailRowsArgs { const float* src; int lds, T; float* ring; int ldr, n, slots, keep; const int* pos_ptr; int pos0; };
int launch_tail_rows(const TailRowsArgs& a, const LaunchCfg& cfg);
// out = tanh(raw) in the activation type; bfloat16: as two parts whose sum carries it to 16 bits (the second part_stride elements on).
int launch_tanh_rows(int act, const float* raw, int ld, void* out, int ldo, size_t part_stride, int n, int T, const LaunchCfg& cfg);
// out[t][i] = clamped_glu of the pair (gate, up) i of a row laid out as LIN_GLU's.
int launch_st_glu_rows(int act, const float* raw, int ld, void* out, int ldo, int ff, float limit, float slope, int T, const LaunchCfg& cfg);
// out[t][h] = o[t][h] / rms(o[t][h]) * w[h] * silu(gate[t][h]) * scale, heads of n values np apart.
struct HeadNormArgs { const float* o; int ldo, heads, n, np; const float* w; int w_hs; const float* gate; int ldg; float eps, scale; void* out; int ldout; };
int launch_head_norm_gate(int act, const HeadNormArgs& a, int T, const LaunchCfg& cfg);

constexpr int kRecurMaxDim = 512;                                   // key channels of a head

// Time mixing (time_mix.cu).  State [heads][dimp (value channel)][dimp (key channel)].
struct TimeMixArgs {
    const float *r, *k, *v; int ld;                                 // heads dimp apart
    const float* w; int ldw;                                        // decays
    const float* u;
    int heads, dimp, T;
    float* state; float* o; int ldo;
    const int* pos_ptr; int pos0;
    int seg_len; float *seg_state, *seg_decay;                      // tokens of a segment (T: one segment, no scratch); scratch [kTmMaxSeg][state], [kTmMaxSeg][heads][dimp]
    unsigned* err;
};
constexpr int kTmMaxSeg = 16;
int time_mix_segment(int heads, int dimp, int T, int sm_count);    // a good seg_len
int launch_time_mix_scan(const TimeMixArgs& a, const LaunchCfg& cfg);
// One token in bfloat16: low-rank decay, recurrence, head norm, gate - and, in the same launch, the token's qkv rows (qkv.raw null: none).
struct TimeMixStepArgs {
    const float *r, *k, *v, *g, *w1;                                // raw projections
    const bf16* w2; int w2_pitch, rank; const float *w0, *u, *norm;
    int heads, dim, dimp; float* state; float eps, scale; bf16* out;
    const int* pos_ptr;
    QkvRowsArgs qkv;
};
int launch_time_mix_step(const TimeMixStepArgs& a, const LaunchCfg& cfg);

// Gated delta rule (delta_rule.cu).  State [heads][vdimp][dimp]; ring [taps][channels]: raw projections by position.
// delta_rows: convolution, silu, unit vectors; per value head and block of four tokens (kDeltaBlock floats) decays up to each token [4], step
// sizes [4], decayed k_i . k_t of i < t [6] and k_i . q_t of i <= t [10], decays from each token to the last [4].
constexpr int kDeltaBlock = 32;
struct DeltaArgs {
    const float* raw; int ld, k_off, v_off, g_off, a_off, b_off;    // raw rows [q | k | v | g | a | b]
    const float* conv; int taps; float* ring;                       // conv [taps][channels], channels = g_off
    const float *a_exp, *dt;                                        // exp(A_log), dt_bias [heads]
    int heads, kv_heads, dim, dimp, vdim, vdimp, T;
    float *qk, *v, *sc;                                             // [T][kv_heads][q dimp | k dimp], [T][heads * vdimp], [blocks][heads][kDeltaBlock]
    float* state; float* o; int ldo;
    const int* pos_ptr; int pos0;
    unsigned* err;
};
int launch_delta_rows(const DeltaArgs& a, const LaunchCfg& cfg);
int launch_delta_scan(const DeltaArgs& a, const LaunchCfg& cfg);
// One token in bfloat16: all of it, head norm and gate included.
struct DeltaStepArgs { DeltaArgs d; const float* norm; float eps, scale; bf16* out; };
int launch_delta_step(const DeltaStepArgs& a, const LaunchCfg& cfg);

// (cos, sin) of pos * freq for every position; freq in double.
int launch_rot_table(float2* table, int n_pos, int dims, double base, const LaunchCfg& cfg);

}  // namespace cq
