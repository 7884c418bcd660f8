// The host object of a layer-list design and one pass over its layers; shared by stack.cu (weights, caches, the latent
// attention layers) and stack_mixers.cu (the sequential layers with recurrent mixers).
#pragma once
#include "stack.h"

#include <cstring>
#include <string>

#include "gemv_seg.cuh"
#include "prefill_gemm.cuh"
#include "stack_host.h"

namespace cq {

inline int pad8(int v) { return (v + 7) / 8 * 8; }
constexpr int kChunk = 2048;                // tokens of a portion that go through the layers together
constexpr int kLogitRows = 64;              // rows of logits computed at a time

struct StMat { bf16* w = nullptr; int rows = 0, cols = 0, pitch = 0; };     // rows with padding, cols with padding of groups

struct StLayer {
    LayerSpec spec;
    LatentAttnSpec a;
    int ff = 0;
    // latent attention
    int dimp = 0, rotp = 0, vdimp = 0, kvrp = 0, qrp = 0, crow = 0, head_q = 0;
    int cache = -1, rot = -1, nsplit = 0;      // nsplit: key ranges of the bfloat16 decode attention (0: sizes it does not cover)
    StMat dq, uq, dkv, uk, uv, g, o, up, down, side_gate, side_proj;
    float *norm1 = nullptr, *norm2 = nullptr, *dq_norm = nullptr, *dkv_norm = nullptr, *sink = nullptr, *side_norm = nullptr;
    // sequential layers (o, up, down, rot, nsplit, dimp, vdimp, crow as above): the first launch's matrices, matrix i reading input
    // copy i, and where their parts start in a raw row
    //   delta      in[0] = [q | k | v | g | a | b]
    //   parallel   in[0] = left [q | k | v], in[1..5] = right r, k, v, g, w1
    // up: rows of the gate and the up matrix in turn, eight at a time
    StMat in[kSegMax], w2, o2;                 // o2: output projection of the recurrence beside an attention
    int nin = 0, ldraw = 0, in_off[kSegMax] = {}, k_off = 0, v_off = 0, g_off = 0, a_off = 0, b_off = 0;
    int rdimp = 0, rankp = 0;                  // time mixing: padded head length and rank
    float *mu = nullptr, *w0 = nullptr, *u = nullptr, *head_norm = nullptr, *conv = nullptr, *a_exp = nullptr, *dt = nullptr;
    size_t kv_off = 0, state_off = 0, ring_off = 0;      // bytes into the cache: keys and values, state, previous inputs by position
};

struct Arena2 {
    uint8_t* base = nullptr; size_t used = 0; bool dry = true;
    void* get(size_t bytes) { const size_t o = used; used += (bytes + 255) / 256 * 256; return dry ? nullptr : base + o; }
};

struct Stack {
    StackSpec spec;
    int act = ACT_BF16, esz = 2, max_seq = 0, vocab_p = 0, wp = 0, sidep = 0;
    std::vector<StLayer> layers;
    StMat embed, side_embed, head;
    float* final_norm = nullptr;
    uint8_t* arena = nullptr;
    uint64_t weight_bytes = 0;
    // cache and rotation tables
    uint8_t* cache = nullptr; size_t cache_bytes = 0; std::vector<size_t> cache_off;
    std::vector<RotarySpec> rots; std::vector<float2*> rot_tables;
    // workspace: a decode step's (one row), and a portion's (kChunk rows; allocated at first use)
    struct Ws {
        int rows = 0, kv_rows = 0;
        float *x = nullptr, *x2 = nullptr, *raw = nullptr, *qf = nullptr, *y = nullptr, *o_lat = nullptr, *part_o = nullptr, *part_ml = nullptr;
        float *z = nullptr, *qk = nullptr, *vv = nullptr, *ro = nullptr, *tail = nullptr; float *seg_state = nullptr, *seg_decay = nullptr, *sc = nullptr;      // recurrences: segments of a portion, decays, convolution outputs, read-outs, head scalars
        void *zin = nullptr, *att2 = nullptr;
        void *xn1 = nullptr, *xn2 = nullptr, *cq = nullptr, *q = nullptr, *att = nullptr, *h = nullptr, *sg = nullptr, *kv = nullptr;
        uint8_t* arena = nullptr;
    } dec, pf;
    float* dec_x = nullptr;             // where a decode step leaves the residual stream (every layer's part added)
    float* logits = nullptr;            // decode step
    float* logits_rows = nullptr; void* xn_rows = nullptr; int* want_rows = nullptr;
    int max_raw = 0, max_q = 0, max_att = 0, max_ff = 0, max_qr = 0, max_kv = 0, max_kvr = 0, max_heads = 0, max_split = 1;
    int max_var = 1, max_z = 0, max_rank = 0, max_qk = 0, max_vv = 0, max_sc = 0, max_ro = 0, max_tm_state = 0;
    int next_pos = 0;                   // designs with a recurrence: the position that the states have reached (-1: none)
};



#define SK(call) do { cudaError_t e_ = (cudaError_t)(call); if (e_ != cudaSuccess) return report_error(e_ == cudaErrorInvalidValue ? CUQWEN_ERR_ARG : CUQWEN_ERR_CUDA, "%s: %s (%s:%d)", #call, cudaGetErrorString(e_), __FILE__, __LINE__); } while (0)

// One pass over the layers for T rows.  decode: T = 1, token and position from the control block, attention over latents.
struct Pass {
    cuqwen_engine* e; Stack* s; Stack::Ws* w; LaunchCfg cfg;
    int T; bool decode; const int* tokens; const int* pos_ptr; int pos0;
    const std::function<int()>* after;

    int done(int err, const char* what) {
        if (err) return report_error(err == (int)cudaErrorInvalidValue ? CUQWEN_ERR_ARG : CUQWEN_ERR_CUDA, "%s: %s", what, cudaGetErrorString((cudaError_t)err));
        return after ? (*after)() : CUQWEN_OK;
    }
#define GO(call) do { if (int r_ = done(call, #call)) return r_; } while (0)
    LinArgs lin(const void* x, int ldx, const StMat& m, int epi, void* out, int ldo) {
        LinArgs a{};
        a.x = x; a.ldx = ldx; a.w = m.w; a.pitch = m.pitch; a.K = m.cols; a.T = T; a.R = m.rows; a.epi = epi; a.out = out; a.ldo = ldo;
        return a;
    }
    int norms(const float* y, const float* y_w, const float* w1, const float* w2) {
        NormRowsArgs n{};
        n.x = w->x; n.ldx = s->wp; n.y = y; n.ldy = s->wp; n.y_w = y_w; n.width = s->spec.width; n.eps = (float)s->spec.norm_eps; n.ldo = s->wp;
        if (w1) { n.w[n.n_out] = w1; n.out[n.n_out++] = w->xn1; }
        if (w2) { n.w[n.n_out] = w2; n.out[n.n_out++] = w->xn2; }
        GO(launch_st_norms(s->act, n, T, cfg));
        return CUQWEN_OK;
    }
    uint8_t* cache_of(const StLayer& l) { return s->cache + s->cache_off[l.cache]; }

    unsigned* err_word() { return reinterpret_cast<unsigned*>(&e->ctl->pad[0]); }

    // What a product may have besides its rows and matrices: a second product (m2 x2) summed into the one matrix's rows, a table row per
    // token, the epilogue's constants, an input of its own for every matrix (matrix i reads the rows from i * var_rows on).
    struct With {
        const void* x2 = nullptr; int ldx2 = 0; const StMat* m2 = nullptr;
        const LinArgs* side = nullptr;
        float c0 = 1.f, c1 = 0.f;
        const float* bias = nullptr;
        int var_rows = 0;
    };
    // out[t] = epilogue(W x[t]) for n rows of x; several matrices (one epilogue) write their rows side by side.  The tensor-core GEMM in
    // bfloat16, the CUDA-core kernels in float32.
    int product(int epi, const void* x, int ldx, const StMat* const* m, int nm, void* out, int ldo, int n) { return product(epi, x, ldx, m, nm, out, ldo, n, With{}); }
    int product(int epi, const void* x, int ldx, const StMat* const* m, int nm, void* out, int ldo, int n, const With& o) {
        if (s->act == ACT_BF16 && (n > 1 || epi == LIN_GLU)) {
            static const int modes[] = {PF_OUT_F32, PF_BF16, PF_BF16_RELU2, PF_ADD_F32, PF_BF16_GELU_SIDE, PF_CAP_F32, PF_BF16_GLU, PF_DECAY_F32};
            PfGemmArgs g; memset(&g, 0, sizeof g);
            PfBf16Mat pm[kPfMaxMat], pm2{};
            for (int i = 0; i < nm; ++i) pm[i] = PfBf16Mat{m[i]->w, m[i]->rows, m[i]->pitch, i * o.var_rows};
            g.T = n; g.K = pad8(m[0]->cols); g.ldo = ldo; g.out_f = (float*)out; g.out_b = (bf16*)out; g.err = err_word(); g.mode = modes[epi]; g.c0 = o.c0; g.c1 = o.c1; g.bias_f = o.bias;
            if (o.m2) { pm2 = PfBf16Mat{o.m2->w, o.m2->rows, o.m2->pitch}; g.K2 = o.m2->cols; }
            if (o.side) { g.side = o.side->side; g.side_pitch = o.side->side_pitch; g.side_dim = o.side->side_dim; g.tokens = o.side->tokens; }
            GO(launch_prefill_gemm_bf16(g, x, ldx, pm, nm, o.m2 ? o.x2 : nullptr, o.ldx2, o.m2 ? &pm2 : nullptr, cfg.stream));
            return CUQWEN_OK;
        }
        size_t off = 0;
        for (int i = 0; i < nm; ++i) {
            LinArgs a = lin((const uint8_t*)x + (size_t)i * o.var_rows * ldx * s->esz, ldx, *m[i], epi, (uint8_t*)out + off * (epi == LIN_F32 || epi == LIN_ADD || epi == LIN_CAP || epi == LIN_DECAY ? 4 : s->esz), ldo);
            a.T = n; a.c0 = o.c0; a.c1 = o.c1; a.bias = o.bias;
            if (o.m2) { a.x2 = o.x2; a.ldx2 = o.ldx2; a.w2 = o.m2->w; a.pitch2 = o.m2->pitch; a.K2 = o.m2->cols; }
            if (o.side) { a.side = o.side->side; a.side_pitch = o.side->side_pitch; a.side_dim = o.side->side_dim; a.tokens = o.side->tokens; }
            GO(launch_st_linear(s->act, a, cfg));
            off += m[i]->rows;
        }
        return CUQWEN_OK;
    }
    int head(const void* x, float* out, int n) {
        const StMat* m[1] = {&s->head};
        With o;
        o.c0 = (float)s->spec.logit_softcap;
        return product(o.c0 > 0.f ? LIN_CAP : LIN_F32, x, s->wp, m, 1, out, s->vocab_p, n, o);
    }

    LinArgs side_args(size_t layer) {
        LinArgs g{};
        g.side = s->side_embed.w + layer * s->spec.side_dim; g.side_pitch = s->side_embed.pitch; g.side_dim = s->spec.side_dim; g.tokens = tokens;
        return g;
    }

    SegGemvArgs seg(int stage, int K) {
        SegGemvArgs g; memset(&g, 0, sizeof g);
        g.stage = stage; g.K = K; g.eps = (float)s->spec.norm_eps; g.width = s->spec.width; g.nvar = 1; g.c0 = 1.f; g.tokens = tokens; g.pos_ptr = pos_ptr; g.err = err_word();
        return g;
    }
    static SegMat sm(const StMat& m) { return SegMat{m.w, m.rows, m.pitch}; }
    int narrow_x() { GO(launch_st_narrow(s->act, w->x, s->wp, w->xn1, s->wp, T, cfg)); return CUQWEN_OK; }
    // latent attention layers (stack.cu)
    int attention(const StLayer& l, const float* gate, int ldraw);
    int layers(bool cache_only);
    LatentRowsArgs latent_rows(const StLayer& l, int ldraw);
    int fused_layers();
    // sequential layers (stack_mixers.cu)
    int seq_layers(bool cache_only);
    int seq_fused_layers();
    int parallel_mixer(const StLayer& l, bool stop);
    int delta_mixer(const StLayer& l, bool stop);
    int clamped_glu(const StLayer& l);
    int grouped_attention(const StLayer& l);
    TimeMixArgs time_mix(const StLayer& l);
    DeltaArgs delta(const StLayer& l);
    QkvRowsArgs qkv(const StLayer& l);
    uint8_t* at(size_t off) { return s->cache + off; }
    const float* last_y() const { return s->spec.side_dim ? w->y : nullptr; }
    const float* last_y_w() const { return s->spec.side_dim ? s->layers.back().side_norm : nullptr; }
};

}  // namespace cq
