// Sequential layers (x += m * mixer(norm1 x), then x += m * ff(norm2 x)) whose mixers are recurrent: grouped attention beside time
// mixing, or the gated delta rule.  Launch sequences of a portion and of a decode step.
//
//   raw of a parallel layer   left [q | k | v], right r, k, v, g, and the thin w1 product: six matrices, each over a copy of the input of its own
//   raw of a delta layer      [q | k | v | g | a | b]
#include "stack_pass.h"

namespace cq {

QkvRowsArgs Pass::qkv(const StLayer& l) {
    const GroupedAttnSpec& g = l.spec.left;
    QkvRowsArgs a{};
    a.raw = w->raw; a.ld = l.ldraw; a.k_off = l.k_off; a.v_off = l.v_off; a.heads = g.heads; a.kv_heads = g.kv_heads; a.dim = g.dim; a.dimp = l.dimp; a.vdimp = l.vdimp;
    a.q = w->q; a.ldq = g.heads * l.dimp; a.cache = at(l.kv_off); a.max_seq = s->max_seq;
    a.rot_dims = g.rot.dims; a.rot = l.rot >= 0 ? s->rot_tables[l.rot] : nullptr;
    a.pos_ptr = pos_ptr; a.pos0 = pos0;
    return a;
}
TimeMixArgs Pass::time_mix(const StLayer& l) {
    const TimeMixSpec& t = l.spec.right;
    TimeMixArgs a{};
    a.r = w->raw + l.in_off[1]; a.k = w->raw + l.in_off[2]; a.v = w->raw + l.in_off[3]; a.ld = l.ldraw;
    a.w = w->z; a.ldw = t.heads * l.rdimp; a.u = l.u; a.err = err_word();
    a.heads = t.heads; a.dimp = l.rdimp; a.T = T;
    a.state = (float*)at(l.state_off); a.o = w->ro; a.ldo = t.heads * l.rdimp; a.pos_ptr = pos_ptr; a.pos0 = pos0;
    a.seg_len = T > 1 ? time_mix_segment(t.heads, l.rdimp, T, cfg.sm_count) : 1; a.seg_state = w->seg_state; a.seg_decay = w->seg_decay;
    return a;
}
DeltaArgs Pass::delta(const StLayer& l) {
    const DeltaSpec& d = l.spec.delta;
    DeltaArgs a{};
    a.raw = w->raw; a.ld = l.ldraw; a.k_off = l.k_off; a.v_off = l.v_off; a.g_off = l.g_off; a.a_off = l.a_off; a.b_off = l.b_off;
    a.conv = l.conv; a.taps = d.conv; a.ring = (float*)at(l.ring_off); a.a_exp = l.a_exp; a.dt = l.dt;
    a.heads = d.heads; a.kv_heads = d.kv_heads; a.dim = d.dim; a.dimp = l.dimp; a.vdim = d.vdim; a.vdimp = l.vdimp; a.T = T;
    a.qk = w->qk; a.v = w->vv; a.sc = w->sc; a.state = (float*)at(l.state_off); a.o = w->ro; a.ldo = d.heads * l.vdimp; a.err = err_word(); a.pos_ptr = pos_ptr; a.pos0 = pos0;
    return a;
}

// Softmax attention of the queries in w->q over the cache -> w->att, times the layer's left_scale.
int Pass::grouped_attention(const StLayer& l) {
    const GroupedAttnSpec& g = l.spec.left;
    uint8_t* c = at(l.kv_off);
    if (decode && l.nsplit > 0) {
        LatentDecodeArgs d{};
        d.q = (const bf16*)w->q; d.crow = l.crow; d.cache = (const bf16*)c; d.kvrp = l.vdimp; d.heads = g.heads; d.scale = (float)g.scale; d.pos_ptr = pos_ptr;
        d.nsplit = l.nsplit; d.part_o = w->part_o; d.part_ml = w->part_ml; d.out = (bf16*)w->att; d.o_hs = l.vdimp;
        d.group = g.heads / g.kv_heads; d.kdim = l.dimp; d.kv_stride = (size_t)s->max_seq * l.crow; d.out_scale = (float)l.spec.left_scale;
        return launch_grouped_decode(d, cfg, [this](int err, const char* what) { return done(err, what); });
    }
    LatentAttnArgs t{};
    t.qn = w->q; t.ldqn = g.heads * l.dimp; t.qn_hs = l.dimp; t.dn = g.dim; t.qr = w->q;
    t.kn = c; t.ldkn = l.crow; t.kn_hs = s->max_seq * l.crow; t.kr = c;
    t.v = c + (size_t)l.dimp * s->esz; t.ldv = l.crow; t.v_hs = t.kn_hs; t.dv = g.vdim;
    t.out = w->att; t.ldo = g.heads * l.vdimp; t.o_hs = l.vdimp; t.T = T; t.heads = g.heads; t.scale = (float)g.scale; t.pos_ptr = pos_ptr; t.pos0 = pos0;
    t.kv_group = g.heads / g.kv_heads; t.out_scale = (float)l.spec.left_scale;
    if (s->act == ACT_BF16 && !decode && latent_prefill_fits(g.dim, 0, g.vdim)) GO(launch_latent_prefill_attn(t, pos0 + T, (size_t)s->max_seq, err_word(), cfg));
    else GO(launch_latent_attn(s->act, t, cfg));
    return CUQWEN_OK;
}

// ---- portions, and every step of the 32-bit mode: one launch per operation ------------------------------------------------
// stop: only what the sequence leaves behind (cache rows, states) is wanted.
int Pass::parallel_mixer(const StLayer& l, bool stop) {
    const StackSpec& sp = s->spec;
    const TimeMixSpec& t = l.spec.right;
    const GroupedAttnSpec& g = l.spec.left;
    ShiftRowsArgs h{};
    h.x = w->x; h.ldx = s->wp; h.w = l.norm1; h.width = sp.width; h.eps = (float)sp.norm_eps; h.out = w->xn1; h.ldo = s->wp; h.var_stride = (size_t)w->rows * s->wp;
    h.mu = l.mu; h.ldmu = s->wp; h.n_mix = 5; h.prev = (const float*)at(l.ring_off); h.ldprev = s->wp; h.tail = w->tail; h.pos_ptr = pos_ptr; h.pos0 = pos0;
    GO(launch_shift_rows(s->act, h, T, cfg));
    TailRowsArgs tail{w->tail, 0, 1, (float*)at(l.ring_off), s->wp, s->wp, 2, 1, pos_ptr, pos0 + T - 1};
    GO(launch_tail_rows(tail, cfg));
    const StMat* in[kSegMax];
    for (int i = 0; i < l.nin; ++i) in[i] = &l.in[i];
    With own;
    own.var_rows = w->rows;
    if (int r = product(LIN_F32, w->xn1, s->wp, in, l.nin, w->raw, l.ldraw, T, own)) return r;
    GO(launch_qkv_rows(s->act, qkv(l), T, cfg));
    // decays: the thin product's tanh goes through w2 as two parts in bfloat16
    const size_t part = (size_t)w->rows * l.rankp;
    GO(launch_tanh_rows(s->act, w->raw + l.in_off[5], l.ldraw, w->zin, l.rankp, part, t.rank, T, cfg));
    const StMat* w2[1] = {&l.w2};
    With low;
    low.bias = l.w0;
    if (s->act == ACT_BF16) { low.x2 = (const uint8_t*)w->zin + part * s->esz; low.ldx2 = l.rankp; low.m2 = &l.w2; }
    if (int r = product(LIN_DECAY, w->zin, l.rankp, w2, 1, w->z, t.heads * l.rdimp, T, low)) return r;
    const TimeMixArgs tm = time_mix(l);
    GO(launch_time_mix_scan(tm, cfg));
    if (stop) return CUQWEN_OK;
    HeadNormArgs n{w->ro, tm.ldo, t.heads, t.dim, l.rdimp, l.head_norm, l.rdimp, w->raw + l.in_off[4], l.ldraw, (float)sp.norm_eps, (float)l.spec.right_scale, w->att2, tm.ldo};
    GO(launch_head_norm_gate(s->act, n, T, cfg));
    if (int r = grouped_attention(l)) return r;
    const StMat* o[1] = {&l.o};
    With both;
    both.x2 = w->att2; both.ldx2 = tm.ldo; both.m2 = &l.o2; both.c0 = (float)sp.residual_mult;
    return product(LIN_ADD, w->att, g.heads * l.vdimp, o, 1, w->x, s->wp, T, both);
}
int Pass::delta_mixer(const StLayer& l, bool stop) {
    const StackSpec& sp = s->spec;
    if (int r = norms(nullptr, nullptr, l.norm1, nullptr)) return r;
    const StMat* in[1] = {&l.in[0]};
    if (int r = product(LIN_F32, w->xn1, s->wp, in, 1, w->raw, l.ldraw, T)) return r;
    const DeltaArgs d = delta(l);
    GO(launch_delta_rows(d, cfg));
    TailRowsArgs tail{w->raw, l.ldraw, T, d.ring, l.g_off, l.g_off, d.taps, d.taps - 1, pos_ptr, pos0};
    if (d.taps > 1) GO(launch_tail_rows(tail, cfg));
    GO(launch_delta_scan(d, cfg));
    if (stop) return CUQWEN_OK;
    HeadNormArgs n{w->ro, d.ldo, d.heads, d.vdim, l.vdimp, l.head_norm, 0, w->raw + l.g_off, l.ldraw, (float)sp.norm_eps, 1.f, w->att, d.ldo};
    GO(launch_head_norm_gate(s->act, n, T, cfg));
    const StMat* o[1] = {&l.o};
    With m;
    m.c0 = (float)sp.residual_mult;
    return product(LIN_ADD, w->att, d.ldo, o, 1, w->x, s->wp, T, m);
}
int Pass::clamped_glu(const StLayer& l) {
    const DenseMlpSpec& f = l.spec.mlp;
    const int ffp = l.up.rows / 2;
    if (int r = norms(nullptr, nullptr, l.norm2, nullptr)) return r;
    const StMat *up[1] = {&l.up}, *down[1] = {&l.down};
    With c, m;
    c.c0 = (float)f.limit; c.c1 = (float)f.slope; m.c0 = (float)s->spec.residual_mult;
    if (s->act == ACT_BF16) { if (int r = product(LIN_GLU, w->xn1, s->wp, up, 1, w->h, ffp, T, c)) return r; }
    else {
        if (int r = product(LIN_F32, w->xn1, s->wp, up, 1, w->raw, l.up.rows, T)) return r;
        GO(launch_st_glu_rows(s->act, w->raw, l.up.rows, w->h, ffp, l.ff, c.c0, c.c1, T, cfg));
    }
    return product(LIN_ADD, w->h, ffp, down, 1, w->x, s->wp, T, m);
}
int Pass::seq_layers(bool cache_only) {
    for (size_t i = 0; i < s->layers.size(); ++i) {
        const StLayer& l = s->layers[i];
        const bool stop = cache_only && i + 1 == s->layers.size();
        if (int r = l.spec.kind == MIX_PARALLEL ? parallel_mixer(l, stop) : delta_mixer(l, stop)) return r;
        if (l.ff && !stop) if (int r = clamped_glu(l)) return r;
    }
    return CUQWEN_OK;
}

// ---- a decode step's layers in bfloat16, fused ----------------------------------------------------------------------------
// delta: [q | k | v | g | a | b] with the norm in the prologue; convolutions, recurrence, head norm and gate; o onto the stream.
// parallel: the six matrices with the norm and the mixes in the prologue; the recurrence of every right head beside the token's
// rotations and cache row; the split attention and its fold; [left o + right o] onto the stream.
// Feed-forward: [gate, up] with the norm in the prologue and the gated unit in the epilogue; down onto the stream.
int Pass::seq_fused_layers() {
    const StackSpec& sp = s->spec;
    const float m = (float)sp.residual_mult;
    auto add_to_stream = [&](const bf16* a, const StMat& wa, const bf16* b, const StMat* wb) {
        SegGemvArgs g = seg(SEG_PLAIN, wa.pitch + (wb ? wb->pitch : 0));
        g.xb[0] = a; g.klen[0] = wa.cols; g.kp[0] = wa.pitch;
        if (wb) { g.xb[1] = b; g.klen[1] = wb->cols; g.kp[1] = wb->pitch; }
        g.epi[0] = LIN_ADD; g.out[0] = w->x; g.c0 = m;
        const SegMat mats[2] = {sm(wa), wb ? sm(*wb) : SegMat{}};
        return done(launch_gemv_seg(g, mats, wb ? 2 : 1, cfg), "output projection");
    };
    for (const StLayer& l : s->layers) {
        SegGemvArgs g = seg(l.spec.kind == MIX_PARALLEL ? SEG_MIX : SEG_NORM, l.in[0].pitch);
        g.x = w->x; g.nw[0] = l.norm1;
        SegMat in[kSegMax];
        for (int i = 0; i < l.nin; ++i) { in[i] = sm(l.in[i]); g.seg_var[i] = i; g.epi[i] = LIN_F32; g.out[i] = w->raw + l.in_off[i]; }
        if (l.spec.kind == MIX_PARALLEL) { g.nvar = l.nin; g.mu = l.mu; g.ldmu = s->wp; g.prev = (float*)at(l.ring_off); g.ldprev = s->wp; }
        GO(launch_gemv_seg(g, in, l.nin, cfg));
        if (l.spec.kind == MIX_PARALLEL) {
            const TimeMixSpec& t = l.spec.right;
            TimeMixStepArgs a{};
            a.r = w->raw + l.in_off[1]; a.k = w->raw + l.in_off[2]; a.v = w->raw + l.in_off[3]; a.g = w->raw + l.in_off[4]; a.w1 = w->raw + l.in_off[5];
            a.w2 = l.w2.w; a.w2_pitch = l.w2.pitch; a.rank = t.rank; a.w0 = l.w0; a.u = l.u; a.norm = l.head_norm;
            a.heads = t.heads; a.dim = t.dim; a.dimp = l.rdimp; a.state = (float*)at(l.state_off); a.eps = (float)sp.norm_eps; a.scale = (float)l.spec.right_scale; a.out = (bf16*)w->att2;
            a.pos_ptr = pos_ptr; a.qkv = qkv(l);
            GO(launch_time_mix_step(a, cfg));
            if (int r = grouped_attention(l)) return r;
            if (int r = add_to_stream((const bf16*)w->att, l.o, (const bf16*)w->att2, &l.o2)) return r;
        } else {
            DeltaStepArgs a{delta(l), l.head_norm, (float)sp.norm_eps, 1.f, (bf16*)w->att};
            GO(launch_delta_step(a, cfg));
            if (int r = add_to_stream((const bf16*)w->att, l.o, nullptr, nullptr)) return r;
        }
        if (l.ff) {
            SegGemvArgs u = seg(SEG_NORM, l.up.pitch);
            u.x = w->x; u.nw[0] = l.norm2; u.epi[0] = LIN_GLU; u.out[0] = w->h; u.c0 = (float)l.spec.mlp.limit; u.c1 = (float)l.spec.mlp.slope;
            const SegMat up[1] = {sm(l.up)};
            GO(launch_gemv_seg(u, up, 1, cfg));
            if (int r = add_to_stream((const bf16*)w->h, l.down, nullptr, nullptr)) return r;
        }
    }
    SegGemvArgs g = seg(SEG_NORM, s->head.pitch);
    g.x = w->x; g.nw[0] = s->final_norm; g.c0 = (float)sp.logit_softcap; g.epi[0] = g.c0 > 0.f ? LIN_CAP : LIN_F32; g.out[0] = s->logits;
    const SegMat head[1] = {sm(s->head)};
    GO(launch_gemv_seg(g, head, 1, cfg));
    s->dec_x = w->x;
    return CUQWEN_OK;
}

}  // namespace cq
