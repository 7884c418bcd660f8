// Host side of the layer-list designs: weights from a model directory, caches and states, and the launch sequences of a decode
// step and of a prompt portion (latent attention layers; stack_mixers.cu has those of sequential layers).  Kernels: stack.h.
//
// Layout.  Every per-head or per-part length is padded to a multiple of eight with zero weight rows / columns when the
// weights are loaded, so that rows start on 16-byte boundaries and padded places hold zeros; weight rows are padded to a
// multiple of 128 columns.  For the usual sizes nothing is added.
//   q            [heads][dim | rot_dim]
//   cache row    [latent kv_rank | rotated key part rot_dim], one array [max_seq_len][row] per layer with a projection of its own
// Sequential layers: keys and values [kv_heads][max_seq_len][key dim | value vdim]; recurrent states float32 [heads][value channel]
// [key channel]; the inputs that a later token still needs in rings by position.
//   raw          [query latent q_rank | cache row | gate heads * vdim], float32 sums of the first launch of a layer
#include "stack_pass.h"

#include <cmath>

namespace cq {

const StackSpec& stack_spec(const Stack* s) { return s->spec; }
int stack_act(const Stack* s) { return s->act; }
float* stack_logits(const Stack* s) { return s->logits; }
size_t stack_cache_bytes(const Stack* s, void** ptr) { *ptr = s->cache; return s->cache_bytes; }
void stack_residual(const Stack* s, void** ptr, size_t* bytes) { *ptr = s->dec_x ? s->dec_x : s->dec.x; *bytes = (size_t)s->spec.width * 4; }
int stack_chunk() { return kChunk; }
int stack_begin(Stack* s, int pos0) {
    if (!s->spec.recurrent()) return CUQWEN_OK;
    if (pos0 != 0 && pos0 != s->next_pos)
        return s->next_pos < 0 ? report_error(CUQWEN_ERR_STATE, "the recurrent states are lost after an error: start over at position 0")
                               : report_error(CUQWEN_ERR_STATE, "the recurrent states stand at position %d: a sequence goes on there, or starts over at 0 (asked for %d)", s->next_pos, pos0);
    s->next_pos = -1;
    return CUQWEN_OK;
}
void stack_end(Stack* s, int pos) { s->next_pos = pos; }

static int alloc_ws(Stack* s, Stack::Ws* w, int rows, bool decode) {
    Arena2 dry, real;
    for (int pass = 0; pass < 2; ++pass) {
        Arena2& a = pass ? real : dry;
        const size_t R = (size_t)rows, E = (size_t)s->esz;
        w->x = (float*)a.get(R * s->wp * 4);
        w->raw = (float*)a.get(R * s->max_raw * 4);
        w->qf = (float*)a.get(R * s->max_q * 4);
        w->y = (float*)a.get(R * s->wp * 4);
        w->xn1 = a.get(R * s->wp * E * s->max_var); w->xn2 = a.get(R * s->wp * E);
        w->cq = a.get(R * s->max_qr * E); w->q = a.get(R * s->max_q * E);
        w->att = a.get(R * s->max_att * E); w->h = a.get(R * (s->max_ff ? s->max_ff : 8) * E);
        w->sg = a.get(R * (s->sidep ? s->sidep : 8) * E);
        if (s->spec.recurrent()) {
            w->z = (float*)a.get(R * s->max_z * 4); w->zin = a.get(2 * R * s->max_rank * E); w->qk = (float*)a.get(R * s->max_qk * 4); w->vv = (float*)a.get(R * s->max_vv * 4);
            w->ro = (float*)a.get(R * s->max_ro * 4); w->att2 = a.get(R * s->max_ro * E); w->sc = (float*)a.get((R + 3) / 4 * s->max_sc * kDeltaBlock * 4); w->tail = (float*)a.get((size_t)s->wp * 4);
            if (!decode) { w->seg_state = (float*)a.get((size_t)kTmMaxSeg * s->max_tm_state * 4); w->seg_decay = (float*)a.get((size_t)kTmMaxSeg * s->max_z * 4); }
        }
        if (decode) {
            w->x2 = (float*)a.get(R * s->wp * 4);
            w->o_lat = (float*)a.get((size_t)s->max_kvr * 4);
            w->part_o = (float*)a.get((size_t)s->max_split * s->max_kvr * 4);
            w->part_ml = (float*)a.get((size_t)s->max_split * s->max_heads * 8);
        } else if (s->max_kv > 0) {
            // keys and values of everything a portion's queries can reach: the portion and the widest window before it
            int reach = 0;
            for (const StLayer& l : s->layers) { const int r = l.a.window > 0 && l.a.window < s->max_seq ? l.a.window - 1 : s->max_seq; reach = r > reach ? r : reach; }
            w->kv_rows = rows + reach < s->max_seq ? rows + reach : s->max_seq;
            w->kv = a.get((size_t)w->kv_rows * s->max_kv * E);
        }
        if (!pass) {
            SK(cudaMalloc((void**)&w->arena, dry.used + 256));
            SK(cudaMemset(w->arena, 0, dry.used + 256));
            real.base = w->arena; real.dry = false;
        }
    }
    w->rows = rows;
    return CUQWEN_OK;
}

int stack_create(cuqwen_engine* e, const StackSpec& spec, int act, int max_seq_len) {
    Stack* s = e->stack = new Stack();
    s->spec = spec; s->act = act; s->esz = act == ACT_F32 ? 4 : 2; s->max_seq = max_seq_len;
    s->wp = pad8(spec.width); s->sidep = pad8(spec.side_dim); s->vocab_p = pad8(spec.vocab);
    if (!spec.side_dim) s->sidep = 0;
    size_t coff = 0;
    auto up = [](int& m, int v) { if (v > m) m = v; };
    auto rotation = [&](const RotarySpec& r) {
        for (size_t i = 0; i < s->rots.size(); ++i) if (s->rots[i].dims == r.dims && s->rots[i].base == r.base) return (int)i;
        s->rots.push_back(r);
        return (int)s->rots.size() - 1;
    };
    auto room = [&](size_t bytes) { const size_t o = coff; coff += (bytes + 255) / 256 * 256; return o; };
    for (const LayerSpec& L : spec.layers) {
        StLayer l;
        l.spec = L; l.a = L.attn; l.ff = L.mlp.ff;
        up(s->max_ff, pad8(l.ff));
        if (L.kind == MIX_LATENT) {
            l.dimp = pad8(l.a.dim); l.rotp = pad8(l.a.rot_dim); l.vdimp = pad8(l.a.vdim); l.kvrp = pad8(l.a.kv_rank); l.qrp = pad8(l.a.q_rank);
            l.crow = l.kvrp + l.rotp; l.head_q = l.dimp + l.rotp;
            l.rot = rotation(l.a.rot);
            if (l.a.kv_from < 0) {
                l.cache = (int)s->cache_off.size();
                s->cache_off.push_back(room((size_t)max_seq_len * l.crow * s->esz));
            } else l.cache = s->layers[l.a.kv_from].cache;
            up(s->max_raw, l.qrp + (l.a.kv_from < 0 ? l.crow : 0) + l.a.heads * l.vdimp); up(s->max_q, l.a.heads * l.head_q); up(s->max_att, l.a.heads * l.vdimp);
            up(s->max_qr, l.qrp); up(s->max_kv, l.a.heads * (l.dimp + l.vdimp)); up(s->max_kvr, l.a.heads * l.kvrp); up(s->max_heads, l.a.heads);
            up(s->max_q, l.a.heads * l.crow);
            if (act == ACT_BF16) l.nsplit = latent_decode_splits(l.a.heads, l.crow, l.kvrp, l.a.window, max_seq_len, e->sms);
        } else if (L.kind == MIX_PARALLEL) {
            const GroupedAttnSpec& g = L.left;
            const TimeMixSpec& t = L.right;
            l.dimp = pad8(g.dim); l.vdimp = pad8(g.vdim); l.crow = l.dimp + l.vdimp;
            if (g.rot.dims > 0) l.rot = rotation(g.rot);
            l.k_off = g.heads * l.dimp; l.v_off = l.k_off + g.kv_heads * l.dimp;
            l.rdimp = pad8(t.dim); l.rankp = pad8(t.rank);
            const int rw = t.heads * l.rdimp;
            if (l.rdimp > kRecurMaxDim) return report_error(CUQWEN_ERR_DIMS, "a recurrence's head has at most %d key channels", kRecurMaxDim);
            l.nin = 6;
            l.in_off[1] = l.v_off + g.kv_heads * l.vdimp;
            for (int i = 2; i < 6; ++i) l.in_off[i] = l.in_off[i - 1] + rw;
            l.ldraw = l.in_off[5] + l.rankp;
            l.kv_off = room((size_t)g.kv_heads * max_seq_len * l.crow * s->esz); l.state_off = room((size_t)rw * l.rdimp * 4); l.ring_off = room((size_t)2 * s->wp * 4);
            up(s->max_q, g.heads * l.dimp); up(s->max_att, g.heads * l.vdimp); up(s->max_var, 6); up(s->max_z, rw); up(s->max_rank, l.rankp); up(s->max_ro, rw); up(s->max_tm_state, rw * l.rdimp);
            up(s->max_kvr, g.heads * l.vdimp); up(s->max_heads, g.heads);
            if (act == ACT_BF16) l.nsplit = grouped_decode_splits(g.heads, g.kv_heads, l.dimp, l.vdimp, max_seq_len, e->sms);
        } else {
            const DeltaSpec& d = L.delta;
            l.dimp = pad8(d.dim); l.vdimp = pad8(d.vdim);
            if (l.dimp > kRecurMaxDim) return report_error(CUQWEN_ERR_DIMS, "a recurrence's head has at most %d key channels", kRecurMaxDim);
            l.nin = 1;
            l.k_off = d.kv_heads * l.dimp; l.v_off = 2 * l.k_off; l.g_off = l.v_off + d.heads * l.vdimp; l.a_off = l.g_off + d.heads * l.vdimp; l.b_off = l.a_off + pad8(d.heads);
            l.ldraw = l.b_off + pad8(d.heads);
            l.state_off = room((size_t)d.heads * l.vdimp * l.dimp * 4); l.ring_off = room((size_t)d.conv * l.g_off * 4);
            up(s->max_att, d.heads * l.vdimp); up(s->max_qk, l.v_off); up(s->max_vv, d.heads * l.vdimp); up(s->max_ro, d.heads * l.vdimp); up(s->max_sc, d.heads);
        }
        up(s->max_raw, l.ldraw); up(s->max_split, l.nsplit);
        if (L.mlp.kind == MLP_CLAMPED_GLU && act == ACT_F32) up(s->max_raw, 2 * pad8(l.ff));
        s->layers.push_back(l);
    }
    s->cache_bytes = coff;
    SK(cudaMalloc((void**)&s->cache, coff + 256));
    SK(cudaMemset(s->cache, 0, coff + 256));
    for (const RotarySpec& r : s->rots) {
        float2* t = nullptr;
        SK(cudaMalloc((void**)&t, (size_t)max_seq_len * (r.dims / 2) * sizeof(float2)));
        s->rot_tables.push_back(t);
        SK(launch_rot_table(t, max_seq_len, r.dims, r.base, LaunchCfg{e->stream, e->sms, false}));
    }
    if (int r = alloc_ws(s, &s->dec, 1, true)) return r;
    SK(cudaMalloc((void**)&s->logits, (size_t)s->vocab_p * 4)); SK(cudaMemset(s->logits, 0, (size_t)s->vocab_p * 4));
    e->p.model_id = CUQWEN_MODEL_CUSTOM; e->p.vocab_size = spec.vocab; e->p.dim = spec.width; e->p.n_layers = (int)spec.layers.size();
    const LayerSpec& first = spec.layers[0];
    switch (first.kind) {
        case MIX_LATENT: e->p.n_heads = first.attn.heads; e->p.n_kv_heads = 1; e->p.head_dim = first.attn.dim + first.attn.rot_dim; e->p.rope_theta = (float)first.attn.rot.base; break;
        case MIX_PARALLEL: e->p.n_heads = first.left.heads; e->p.n_kv_heads = first.left.kv_heads; e->p.head_dim = first.left.dim; e->p.rope_theta = (float)first.left.rot.base; break;
        case MIX_DELTA: e->p.n_heads = first.delta.heads; e->p.n_kv_heads = first.delta.kv_heads; e->p.head_dim = first.delta.dim; break;
    }
    e->p.intermediate_size = first.mlp.ff; e->p.norm_eps = (float)spec.norm_eps;
    e->vocab_l = spec.vocab;
    SK(cudaStreamSynchronize(e->stream));
    return CUQWEN_OK;
}

void stack_destroy(cuqwen_engine* e) {
    Stack* s = e->stack;
    if (!s) return;
    void* bufs[] = {s->arena, s->cache, s->dec.arena, s->pf.arena, s->logits, s->logits_rows, s->xn_rows, s->want_rows};
    for (void* b : bufs) if (b) cudaFree(b);
    for (float2* t : s->rot_tables) cudaFree(t);
    delete s;
    e->stack = nullptr;
}

// ---- weights --------------------------------------------------------------------------------------------------------
// Lengths of consecutive groups of rows (or columns) and the places they take: group i of `len` elements starts at `at`.
struct Groups {
    std::vector<std::pair<int, int>> g;       // (length, start of its padded place)
    int total = 0, padded = 0;
    Groups& add(int len) { g.emplace_back(len, padded); total += len; padded += pad8(len); return *this; }
    static Groups one(int len) { return Groups().add(len); }
    static Groups heads(int n, int a, int b = 0) { Groups r; for (int i = 0; i < n; ++i) { r.add(a); if (b) r.add(b); } return r; }
};

// A matrix out of the rows of one tensor or of several, every row at its place among n_rows.
struct Part { std::string name; Groups rows; };
static int put_rows(const Safetensors& st, Stack* s, Arena2& ar, const std::vector<Part>& parts, int n_rows, const Groups& cols, StMat* m, bool counted = true) {
    m->rows = n_rows; m->cols = cols.padded; m->pitch = (cols.padded + 127) / 128 * 128;
    const size_t bytes = (size_t)m->rows * m->pitch * 2;
    m->w = (bf16*)ar.get(bytes);
    std::vector<uint16_t> host;
    for (const Part& p : parts) {
        const Safetensors::Tensor* t = st.expect(p.name, p.rows.total, cols.total);
        if (!t) return CUQWEN_ERR_DIMS;
        if (counted && ar.dry) s->weight_bytes += (uint64_t)p.rows.total * cols.total * 2;
        if (ar.dry) continue;
        if (parts.size() == 1 && n_rows == p.rows.total && m->pitch == cols.total) { SK(cudaMemcpy(m->w, t->data, bytes, cudaMemcpyHostToDevice)); return CUQWEN_OK; }
        if (host.empty()) host.assign((size_t)m->rows * m->pitch, 0);
        size_t src_row = 0;
        for (const auto& rg : p.rows.g)
            for (int r = 0; r < rg.first; ++r, ++src_row) {
                const uint8_t* src = t->data + src_row * cols.total * 2;
                uint16_t* dst = host.data() + (size_t)(rg.second + r) * m->pitch;
                for (const auto& cg : cols.g) { memcpy(dst + cg.second, src, (size_t)cg.first * 2); src += (size_t)cg.first * 2; }
            }
    }
    if (!ar.dry) SK(cudaMemcpy(m->w, host.data(), bytes, cudaMemcpyHostToDevice));
    return CUQWEN_OK;
}
static int put_matrix(const Safetensors& st, Stack* s, Arena2& ar, const std::string& name, const Groups& rows, const Groups& cols, StMat* m, bool counted = true) {
    return put_rows(st, s, ar, {Part{name, rows}}, rows.padded, cols, m, counted);
}
// Values of a tensor [rows, cols] (cols 0: a vector of `rows`) widened to float32: value (r, c) goes to dst[at(r, c)].
template <typename At>
static int take_floats(const Safetensors& st, Stack* s, const Arena2& ar, const std::string& name, int rows, int cols, std::vector<float>& dst, At at) {
    const Safetensors::Tensor* t = st.expect(name, rows, cols);
    if (!t) return CUQWEN_ERR_DIMS;
    const int nc = cols ? cols : 1;
    if (ar.dry) { s->weight_bytes += (uint64_t)rows * nc * 2; return CUQWEN_OK; }
    for (int r = 0; r < rows; ++r)
        for (int c = 0; c < nc; ++c) {
            uint16_t h; memcpy(&h, t->data + 2 * ((size_t)r * nc + c), 2);
            const uint32_t u = (uint32_t)h << 16;
            memcpy(&dst[at(r, c)], &u, 4);
        }
    return CUQWEN_OK;
}
static int put_floats(Arena2& ar, const std::vector<float>& host, float** v) {
    *v = (float*)ar.get(host.size() * 4);
    if (!ar.dry) SK(cudaMemcpy(*v, host.data(), host.size() * 4, cudaMemcpyHostToDevice));
    return CUQWEN_OK;
}
static int put_vector(const Safetensors& st, Stack* s, Arena2& ar, const std::string& name, int n, float** v, float offset = 0.f) {
    std::vector<float> host(pad8(n), 0.f);
    if (int r = take_floats(st, s, ar, name, n, 0, host, [](int i, int) { return (size_t)i; })) return r;
    for (int i = 0; i < n; ++i) host[i] += offset;
    return put_floats(ar, host, v);
}
// One value per place of `heads` heads of dim values, padded head by head; the tensor is a vector, or a matrix [heads, dim].
static int put_heads(const Safetensors& st, Stack* s, Arena2& ar, const std::string& name, int heads, int dim, bool matrix, float** v) {
    const size_t dimp = pad8(dim);
    std::vector<float> host(heads * dimp, 0.f);
    if (int r = take_floats(st, s, ar, name, matrix ? heads : heads * dim, matrix ? dim : 0, host,
                            [=](int i, int c) { return matrix ? i * dimp + c : (size_t)(i / dim) * dimp + i % dim; })) return r;
    return put_floats(ar, host, v);
}

#define TRY(x) do { if (int r_ = (x)) return r_; } while (0)
// Softmax attention beside time mixing: tensors under MIX.left and MIX.right.
static int walk_parallel(const Safetensors& st, Stack* s, Arena2& ar, const std::string& mix, StLayer& l) {
    const int W = s->spec.width;
    const Groups cols = Groups::one(W);
    const GroupedAttnSpec& g = l.spec.left;
    const TimeMixSpec& t = l.spec.right;
    const std::string a = mix + "left.", b = mix + "right.";
    auto placed = [](Groups r, int at) { for (auto& x : r.g) x.second += at; return r; };
    TRY(put_rows(st, s, ar, {Part{a + "q", Groups::heads(g.heads, g.dim)}, Part{a + "k", placed(Groups::heads(g.kv_heads, g.dim), l.k_off)}, Part{a + "v", placed(Groups::heads(g.kv_heads, g.vdim), l.v_off)}},
                 l.in_off[1], cols, &l.in[0]));
    TRY(put_matrix(st, s, ar, a + "o", cols, Groups::heads(g.heads, g.vdim), &l.o));
    const char* names[] = {"r", "k", "v", "g", "w"};
    std::vector<float> mu((size_t)5 * s->wp, 0.f);
    for (int i = 0; i < 5; ++i) TRY(take_floats(st, s, ar, b + "mu." + names[i], W, 0, mu, [=](int c, int) { return (size_t)i * s->wp + c; }));
    TRY(put_floats(ar, mu, &l.mu));
    for (int i = 0; i < 4; ++i) TRY(put_matrix(st, s, ar, b + names[i], Groups::heads(t.heads, t.dim), cols, &l.in[1 + i]));
    TRY(put_matrix(st, s, ar, b + "w1", Groups::one(t.rank), cols, &l.in[5]));
    TRY(put_matrix(st, s, ar, b + "w2", Groups::heads(t.heads, t.dim), Groups::one(t.rank), &l.w2));
    TRY(put_heads(st, s, ar, b + "w0", t.heads, t.dim, false, &l.w0));
    TRY(put_heads(st, s, ar, b + "u", t.heads, t.dim, true, &l.u));
    TRY(put_heads(st, s, ar, b + "norm", t.heads, t.dim, false, &l.head_norm));
    TRY(put_matrix(st, s, ar, b + "o", cols, Groups::heads(t.heads, t.dim), &l.o2));
    return CUQWEN_OK;
}
static int walk_delta(const Safetensors& st, Stack* s, Arena2& ar, const std::string& mix, StLayer& l) {
    const Groups cols = Groups::one(s->spec.width);
    const DeltaSpec& d = l.spec.delta;
    auto placed = [](Groups r, int at) { for (auto& x : r.g) x.second += at; return r; };
    const Groups k = Groups::heads(d.kv_heads, d.dim), v = Groups::heads(d.heads, d.vdim);
    TRY(put_rows(st, s, ar, {Part{mix + "q", k}, Part{mix + "k", placed(k, l.k_off)}, Part{mix + "v", placed(v, l.v_off)}, Part{mix + "g", placed(v, l.g_off)},
                             Part{mix + "a", placed(Groups::one(d.heads), l.a_off)}, Part{mix + "b", placed(Groups::one(d.heads), l.b_off)}}, l.ldraw, cols, &l.in[0]));
    std::vector<float> conv((size_t)d.conv * l.g_off, 0.f);
    const char* names[] = {"q", "k", "v"};
    for (int i = 0; i < 3; ++i) {
        const int n = i < 2 ? d.kv_heads : d.heads, len = i < 2 ? d.dim : d.vdim, lenp = i < 2 ? l.dimp : l.vdimp, at = i == 0 ? 0 : i == 1 ? l.k_off : l.v_off;
        TRY(take_floats(st, s, ar, mix + names[i] + ".conv", n * len, d.conv, conv, [=](int r, int c) { return (size_t)c * l.g_off + at + r / len * lenp + r % len; }));
    }
    TRY(put_floats(ar, conv, &l.conv));
    std::vector<float> al(pad8(d.heads), 0.f);
    TRY(take_floats(st, s, ar, mix + "A_log", d.heads, 0, al, [](int i, int) { return (size_t)i; }));
    for (int i = 0; i < d.heads; ++i) al[i] = expf(al[i]);
    TRY(put_floats(ar, al, &l.a_exp));
    TRY(put_vector(st, s, ar, mix + "dt_bias", d.heads, &l.dt));
    TRY(put_vector(st, s, ar, mix + "norm", d.vdim, &l.head_norm));
    TRY(put_matrix(st, s, ar, mix + "o", cols, v, &l.o));
    return CUQWEN_OK;
}
static int walk_tensors(const Safetensors& st, Stack* s, Arena2& ar) {
    const StackSpec& sp = s->spec;
    const Groups W = Groups::one(sp.width);
    TRY(put_matrix(st, s, ar, "embed", Groups::one(sp.vocab), W, &s->embed, false));
    if (sp.side_dim) TRY(put_matrix(st, s, ar, "side.embed", Groups::one(sp.vocab), Groups::one(sp.side_dim * (int)sp.layers.size()), &s->side_embed, false));
    for (size_t i = 0; i < s->layers.size(); ++i) {
        StLayer& l = s->layers[i];
        const LatentAttnSpec& a = l.a;
        const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.";
        TRY(put_vector(st, s, ar, p + "norm1", sp.width, &l.norm1, (float)sp.norm_offset));
        if (sp.sequential) {
            TRY(l.spec.kind == MIX_PARALLEL ? walk_parallel(st, s, ar, mix, l) : walk_delta(st, s, ar, mix, l));
            if (l.ff) {
                TRY(put_vector(st, s, ar, p + "norm2", sp.width, &l.norm2, (float)sp.norm_offset));
                Groups gate, upr;                       // rows i .. i + 7 of the gate, then those of the up matrix
                for (int r = 0; r < l.ff; r += 8) { const int n = l.ff - r < 8 ? l.ff - r : 8; gate.g.emplace_back(n, 2 * r); upr.g.emplace_back(n, 2 * r + 8); }
                gate.total = upr.total = l.ff;
                TRY(put_rows(st, s, ar, {Part{p + "mlp.gate", gate}, Part{p + "mlp.up", upr}}, 2 * pad8(l.ff), W, &l.up));
                TRY(put_matrix(st, s, ar, p + "mlp.down", W, Groups::one(l.ff), &l.down));
            }
            continue;
        }
        TRY(put_matrix(st, s, ar, mix + "dq", Groups::one(a.q_rank), W, &l.dq));
        TRY(put_vector(st, s, ar, mix + "dq.norm", a.q_rank, &l.dq_norm));
        TRY(put_matrix(st, s, ar, mix + "uq", Groups::heads(a.heads, a.dim, a.rot_dim), Groups::one(a.q_rank), &l.uq));
        if (a.kv_from < 0) {
            TRY(put_matrix(st, s, ar, mix + "dkv", Groups::heads(1, a.kv_rank, a.rot_dim), W, &l.dkv));
            TRY(put_vector(st, s, ar, mix + "dkv.norm", a.kv_rank, &l.dkv_norm));
        }
        TRY(put_matrix(st, s, ar, mix + "uk", Groups::heads(a.heads, a.dim), Groups::one(a.kv_rank), &l.uk));
        TRY(put_matrix(st, s, ar, mix + "uv", Groups::heads(a.heads, a.vdim), Groups::one(a.kv_rank), &l.uv));
        if (a.sink) TRY(put_vector(st, s, ar, mix + "sink", a.heads, &l.sink));
        if (a.gate) TRY(put_matrix(st, s, ar, mix + "g", Groups::heads(a.heads, a.vdim), W, &l.g));
        TRY(put_matrix(st, s, ar, mix + "o", W, Groups::heads(a.heads, a.vdim), &l.o));
        if (l.ff) {
            TRY(put_vector(st, s, ar, p + "norm2", sp.width, &l.norm2));
            TRY(put_matrix(st, s, ar, p + "mlp.up", Groups::one(l.ff), W, &l.up));
            TRY(put_matrix(st, s, ar, p + "mlp.down", W, Groups::one(l.ff), &l.down));
        }
        if (sp.side_dim) {
            TRY(put_matrix(st, s, ar, p + "side.gate", Groups::one(sp.side_dim), W, &l.side_gate));
            TRY(put_matrix(st, s, ar, p + "side.proj", W, Groups::one(sp.side_dim), &l.side_proj));
            TRY(put_vector(st, s, ar, p + "side.norm", sp.width, &l.side_norm));
        }
    }
    TRY(put_vector(st, s, ar, "final.norm", sp.width, &s->final_norm, (float)sp.norm_offset));
    TRY(put_matrix(st, s, ar, "head", Groups::one(sp.vocab), W, &s->head));
#undef TRY
    return CUQWEN_OK;
}

int stack_load(cuqwen_engine* e, const char* dir) {
    Stack* s = e->stack;
    Safetensors st;
    if (int r = st.open((std::string(dir) + "/model.safetensors").c_str())) return r;
    Arena2 dry, real;
    s->weight_bytes = (uint64_t)(s->spec.width + s->spec.side_dim * (int)s->layers.size()) * 2;      // a token's embedding rows
    if (int r = walk_tensors(st, s, dry)) return r;
    SK(cudaMalloc((void**)&s->arena, dry.used + 256));
    real.base = s->arena; real.dry = false;
    if (int r = walk_tensors(st, s, real)) return r;
    SK(cudaDeviceSynchronize());
    return CUQWEN_OK;
}

uint64_t stack_step_bytes(const Stack* s, int ctx) {
    uint64_t b = s->weight_bytes;
    for (const StLayer& l : s->layers) {
        if (l.spec.kind == MIX_PARALLEL) {             // keys and values; the state is read and written
            b += (uint64_t)ctx * l.spec.left.kv_heads * (l.spec.left.dim + l.spec.left.vdim) * s->esz + (uint64_t)8 * l.spec.right.heads * l.spec.right.dim * l.spec.right.dim;
            continue;
        }
        if (l.spec.kind == MIX_DELTA) { b += (uint64_t)8 * l.spec.delta.heads * l.spec.delta.dim * l.spec.delta.vdim; continue; }
        const int n = l.a.window > 0 && l.a.window < ctx ? l.a.window : ctx;
        b += (uint64_t)n * (l.a.kv_rank + l.a.rot_dim) * s->esz;
    }
    return b;
}

// ---- launch sequences -------------------------------------------------------------------------------------------------
// Attention of the queries in w->qf (float32, not yet rotated) -> w->att, gated.
int Pass::attention(const StLayer& l, const float* gate, int ldraw) {
    const LatentAttnSpec& a = l.a;
    uint8_t* c = cache_of(l);
    const float2* rot = s->rot_tables[l.rot];
    LatentAttnArgs t{};
    t.out_scale = 1.f;
    t.kr = c + (size_t)l.kvrp * s->esz; t.ldkr = l.crow; t.dr = a.rot_dim;
    t.sink = l.sink; t.T = T; t.heads = a.heads; t.window = a.window; t.scale = (float)a.scale; t.pos_ptr = pos_ptr; t.pos0 = pos0;
    if (decode) {
        AbsorbArgs b{w->qf, l.head_q, l.dimp, a.rot_dim, rot, pos_ptr, l.uk.w, l.uk.pitch, a.heads, a.dim, l.dimp, w->q, l.crow, l.kvrp};
        GO(launch_absorb_q(s->act, b, cfg));
        if (l.nsplit > 0) {
            LatentDecodeArgs d{};
            d.q = (const bf16*)w->q; d.crow = l.crow; d.cache = (const bf16*)c; d.kvrp = l.kvrp; d.sink = l.sink; d.heads = a.heads; d.window = a.window; d.scale = (float)a.scale;
            d.pos_ptr = pos_ptr; d.nsplit = l.nsplit; d.part_o = w->part_o; d.part_ml = w->part_ml;
            d.wv = l.uv.w; d.pitch = l.uv.pitch; d.vdim = a.vdim; d.vdimp = l.vdimp; d.kv_rank = a.kv_rank; d.gate = gate; d.g_hs = l.vdimp; d.out = (bf16*)w->att; d.o_hs = l.vdimp;
            return launch_latent_decode(d, cfg, [this](int err, const char* what) { return done(err, what); });
        }
        t.qn = w->q; t.ldqn = a.heads * l.crow; t.qn_hs = l.crow; t.dn = a.kv_rank;
        t.qr = (uint8_t*)w->q + (size_t)l.kvrp * s->esz; t.ldqr = a.heads * l.crow; t.qr_hs = l.crow;
        t.kn = c; t.ldkn = l.crow; t.kn_hs = 0; t.v = c; t.ldv = l.crow; t.v_hs = 0; t.dv = a.kv_rank;
        t.out = w->o_lat; t.out_f32 = 1; t.ldo = a.heads * l.kvrp; t.o_hs = l.kvrp;
        GO(launch_latent_attn(s->act, t, cfg));
        UvGateArgs u{};
        u.o = w->o_lat; u.ldo = l.kvrp; u.wv = l.uv.w; u.pitch = l.uv.pitch; u.heads = a.heads; u.vdim = a.vdim; u.vdimp = l.vdimp; u.kv_rank = a.kv_rank;
        u.gate = gate; u.g_hs = l.vdimp; u.out = w->att; u.o_hs = l.vdimp;
        GO(launch_uv_gate(s->act, u, cfg));
        return CUQWEN_OK;
    }
    RopeQArgs rq{w->qf, w->q, l.uq.rows, a.heads, l.head_q, l.dimp, a.rot_dim, rot, pos_ptr, pos0};
    GO(launch_st_rope_q(s->act, rq, T, cfg));
    // keys and values of every token the portion's queries reach, side by side in a row
    const int k0 = a.window > 0 && pos0 - a.window + 1 > 0 ? pos0 - a.window + 1 : 0, n = pos0 + T - k0;
    const int kcols = a.heads * l.dimp, ldkv = kcols + a.heads * l.vdimp;
    const StMat* kv[2] = {&l.uk, &l.uv};
    if (int r = product(LIN_ACT, c + (size_t)k0 * l.crow * s->esz, l.crow, kv, 2, w->kv, ldkv, n)) return r;
    t.qr = (uint8_t*)w->q + (size_t)l.dimp * s->esz; t.ldqr = a.heads * l.head_q; t.qr_hs = l.head_q;
    t.qn = w->q; t.ldqn = a.heads * l.head_q; t.qn_hs = l.head_q; t.dn = a.dim;
    t.kn = w->kv; t.ldkn = ldkv; t.kn_hs = l.dimp; t.v = (uint8_t*)w->kv + (size_t)kcols * s->esz; t.ldv = ldkv; t.v_hs = l.vdimp; t.dv = a.vdim; t.kbase = k0;
    t.gate = gate; t.ldg = ldraw; t.g_hs = l.vdimp; t.out = w->att; t.ldo = a.heads * l.vdimp; t.o_hs = l.vdimp;
    if (s->act == ACT_BF16 && latent_prefill_fits(a.dim, a.rot_dim, a.vdim)) GO(launch_latent_prefill_attn(t, n, (size_t)s->max_seq, err_word(), cfg));
    else GO(launch_latent_attn(s->act, t, cfg));
    return CUQWEN_OK;
}

// All layers, one launch per operation.  cache_only: nothing after the last layer's cache rows is needed.  Leaves the
// residual stream in w->x with the last layer's token input still to be added (last_y).
int Pass::layers(bool cache_only) {
    const StackSpec& sp = s->spec;
    const float* y = nullptr; const float* y_w = nullptr;
    for (size_t i = 0; i < s->layers.size(); ++i) {
        const StLayer& l = s->layers[i];
        const LatentAttnSpec& a = l.a;
        const bool own = a.kv_from < 0, stop = cache_only && i + 1 == s->layers.size();
        if (stop && !own) return CUQWEN_OK;
        if (int r = norms(y, y_w, l.norm1, l.ff && !stop ? l.norm2 : nullptr)) return r;
        const int c_off = l.qrp, g_off = c_off + (own ? l.crow : 0), ldraw = g_off + (a.gate ? a.heads * l.vdimp : 0);
        if (stop) {
            const StMat* kv[1] = {&l.dkv};
            if (int r = product(LIN_F32, w->xn1, s->wp, kv, 1, w->raw + c_off, ldraw, T)) return r;
            LatentRowsArgs lr = latent_rows(l, ldraw);
            lr.dq = nullptr;
            GO(launch_st_latent_rows(s->act, lr, T, cfg));
            return CUQWEN_OK;
        }
        const StMat* first[3]; int nf = 0;
        first[nf++] = &l.dq;
        if (own) first[nf++] = &l.dkv;
        if (a.gate) first[nf++] = &l.g;
        if (int r = product(LIN_F32, w->xn1, s->wp, first, nf, w->raw, ldraw, T)) return r;
        const StMat *up[1] = {&l.up}, *uq[1] = {&l.uq}, *o[1] = {&l.o}, *sg[1] = {&l.side_gate}, *sp1[1] = {&l.side_proj};
        if (l.ff) if (int r = product(LIN_RELU2, w->xn2, s->wp, up, 1, w->h, l.up.rows, T)) return r;
        LatentRowsArgs lr = latent_rows(l, ldraw);
        GO(launch_st_latent_rows(s->act, lr, T, cfg));
        if (int r = product(LIN_F32, w->cq, l.qrp, uq, 1, w->qf, l.uq.rows, T)) return r;
        if (int r = attention(l, a.gate ? w->raw + g_off : nullptr, ldraw)) return r;
        With ff;
        if (l.ff) { ff.x2 = w->h; ff.ldx2 = l.up.rows; ff.m2 = &l.down; }
        if (int r = product(LIN_ADD, w->att, a.heads * l.vdimp, o, 1, w->x, s->wp, T, ff)) return r;
        if (sp.side_dim) {
            // the token input reads the stream itself, narrowed like every activation
            if (int r = narrow_x()) return r;
            const LinArgs e1 = side_args(i);
            With row;
            row.side = &e1;
            if (int r = product(LIN_GELU_SIDE, w->xn1, s->wp, sg, 1, w->sg, s->sidep, T, row)) return r;
            if (int r = product(LIN_F32, w->sg, s->sidep, sp1, 1, w->y, s->wp, T)) return r;
            y = w->y; y_w = l.side_norm;
        }
    }
    return CUQWEN_OK;
}

LatentRowsArgs Pass::latent_rows(const StLayer& l, int ldraw) {
    const LatentAttnSpec& a = l.a;
    LatentRowsArgs lr{};
    lr.dq = w->raw; lr.ld = ldraw; lr.dq_w = l.dq_norm; lr.cq = w->cq; lr.ldcq = l.qrp; lr.q_rank = a.q_rank;
    if (a.kv_from < 0) { lr.dkv = w->raw + l.qrp; lr.dkv_w = l.dkv_norm; lr.cache = cache_of(l); lr.ldc = l.crow; lr.kv_rank = a.kv_rank; lr.kr_off = l.kvrp; lr.rot_dim = a.rot_dim; lr.rot = s->rot_tables[l.rot]; }
    lr.eps = (float)s->spec.norm_eps; lr.pos_ptr = pos_ptr; lr.pos0 = pos0;
    return lr;
}

// A decode step's layers in bfloat16, fused: per layer eight launches - [dq | dkv | g | up] with the previous layer's token
// input and both norms in the prologue; uq with the latent's norm, and the cache row; the queries into latent space; the
// split attention and its fold with W_uv and the gate; [o + down]; the token input's two matrices (its norm is left to the
// next prologue).  The stream alternates between two buffers: a prologue reads one and CTA 0 writes the other.
int Pass::fused_layers() {
    const StackSpec& sp = s->spec;
    float *x = w->x, *other = w->x2;
    const float* y_w = nullptr;
    auto take_x = [&](SegGemvArgs& g) {              // the stream, with the token input that is still to be added
        g.x = x;
        if (y_w) { g.y = w->y; g.y_w = y_w; g.x_next = other; float* t = x; x = other; other = t; y_w = nullptr; }
    };
    for (size_t i = 0; i < s->layers.size(); ++i) {
        const StLayer& l = s->layers[i];
        const LatentAttnSpec& a = l.a;
        const bool own = a.kv_from < 0;
        const int c_off = l.qrp, g_off = c_off + (own ? l.crow : 0), ldraw = g_off + (a.gate ? a.heads * l.vdimp : 0);
        {
            SegGemvArgs g = seg(SEG_NORM, l.dq.pitch);
            SegMat m[4]; int n = 0;
            take_x(g);
            auto add = [&](const StMat& mat, int var, int epi, void* out) { g.seg_var[n] = var; g.epi[n] = epi; g.out[n] = out; m[n++] = sm(mat); };
            g.nw[0] = l.norm1;
            add(l.dq, 0, LIN_F32, w->raw);
            if (own) add(l.dkv, 0, LIN_F32, w->raw + c_off);
            if (a.gate) add(l.g, 0, LIN_F32, w->raw + g_off);
            if (l.ff) { g.nw[1] = l.norm2; g.nvar = 2; add(l.up, 1, LIN_RELU2, w->h); }
            GO(launch_gemv_seg(g, m, n, cfg));
        }
        {
            SegGemvArgs g = seg(SEG_NORM, l.uq.pitch);
            g.x = w->raw; g.width = a.q_rank; g.nw[0] = l.dq_norm; g.epi[0] = LIN_F32; g.out[0] = w->qf;
            if (own) { g.has_kv = 1; g.kv = latent_rows(l, ldraw); }
            const SegMat m[1] = {sm(l.uq)};
            GO(launch_gemv_seg(g, m, 1, cfg));
        }
        if (int r = attention(l, a.gate ? w->raw + g_off : nullptr, ldraw)) return r;
        {
            SegGemvArgs g = seg(SEG_PLAIN, l.o.pitch + (l.ff ? l.down.pitch : 0));
            g.xb[0] = (const bf16*)w->att; g.klen[0] = a.heads * l.vdimp; g.kp[0] = l.o.pitch;
            if (l.ff) { g.xb[1] = (const bf16*)w->h; g.klen[1] = l.up.rows; g.kp[1] = l.down.pitch; }
            g.epi[0] = LIN_ADD; g.out[0] = x;
            const SegMat m[2] = {sm(l.o), sm(l.down)};
            GO(launch_gemv_seg(g, m, l.ff ? 2 : 1, cfg));
        }
        if (sp.side_dim) {
            SegGemvArgs g = seg(SEG_NARROW, l.side_gate.pitch);
            const LinArgs e1 = side_args(i);
            g.x = x; g.side = e1.side; g.side_pitch = e1.side_pitch; g.side_dim = e1.side_dim; g.epi[0] = LIN_GELU_SIDE; g.out[0] = w->sg;
            const SegMat m[1] = {sm(l.side_gate)};
            GO(launch_gemv_seg(g, m, 1, cfg));
            SegGemvArgs p = seg(SEG_PLAIN, l.side_proj.pitch);
            p.xb[0] = (const bf16*)w->sg; p.klen[0] = s->sidep; p.kp[0] = l.side_proj.pitch; p.epi[0] = LIN_F32; p.out[0] = w->y;
            const SegMat m2[1] = {sm(l.side_proj)};
            GO(launch_gemv_seg(p, m2, 1, cfg));
            y_w = l.side_norm;
        }
    }
    SegGemvArgs g = seg(SEG_NORM, s->head.pitch);
    take_x(g);
    g.nw[0] = s->final_norm; g.epi[0] = LIN_F32; g.out[0] = s->logits;
    const SegMat m[1] = {sm(s->head)};
    GO(launch_gemv_seg(g, m, 1, cfg));
    s->dec_x = x;
    return CUQWEN_OK;
}

int stack_record_step(cuqwen_engine* e, const LaunchCfg& cfg, const std::function<int()>& after) {
    Stack* s = e->stack;
    Pass p{e, s, &s->dec, cfg, 1, true, &e->ctl->token, &e->ctl->pos, 0, &after};
    LaunchCfg plain = cfg; plain.pdl = false;
    if (int r = p.done(launch_st_embed_step(s->embed.w, s->embed.pitch, e->ctl, s->dec.x, s->spec.width, (float)s->spec.embed_scale, plain), "embedding")) return r;
    if (s->act == ACT_BF16) return s->spec.sequential ? p.seq_fused_layers() : p.fused_layers();
    if (int r = s->spec.sequential ? p.seq_layers(false) : p.layers(false)) return r;
    if (int r = p.norms(p.last_y(), p.last_y_w(), s->final_norm, nullptr)) return r;
    return p.head(s->dec.xn1, s->logits, 1);
}

int stack_run_chunk(cuqwen_engine* e, int T, int pos0, const int* want, int n_want, float* logits_host) {
    Stack* s = e->stack;
    if (T < 1 || T > kChunk) return report_error(CUQWEN_ERR_ARG, "a portion has 1 to %d tokens", kChunk);
    if (!s->pf.arena) {
        if (int r = alloc_ws(s, &s->pf, kChunk < s->max_seq ? kChunk : s->max_seq, false)) return r;
        SK(cudaMalloc((void**)&s->logits_rows, (size_t)kLogitRows * s->vocab_p * 4));
        SK(cudaMalloc((void**)&s->xn_rows, (size_t)kLogitRows * s->wp * s->esz));
        SK(cudaMalloc((void**)&s->want_rows, (size_t)kChunk * 4));
    }
    const LaunchCfg cfg{e->stream, e->sms, false};
    Pass p{e, s, &s->pf, cfg, T, false, e->pf_tok, nullptr, pos0, nullptr};
    if (int r = p.done(launch_st_embed(s->embed.w, s->embed.pitch, e->pf_tok, s->pf.x, s->wp, s->spec.width, (float)s->spec.embed_scale, T, cfg), "embedding")) return r;
    if (int r = s->spec.sequential ? p.seq_layers(n_want == 0) : p.layers(n_want == 0)) return r;
    if (n_want == 0) return CUQWEN_OK;
    if (p.last_y()) if (int r = p.norms(p.last_y(), p.last_y_w(), nullptr, nullptr)) return r;
    SK(cudaMemcpyAsync(s->want_rows, want, (size_t)n_want * 4, cudaMemcpyHostToDevice, e->stream));
    for (int i = 0; i < n_want; i += kLogitRows) {
        const int n = n_want - i < kLogitRows ? n_want - i : kLogitRows;
        NormRowsArgs a{};
        a.x = s->pf.x; a.ldx = s->wp; a.w[0] = s->final_norm; a.out[0] = s->xn_rows; a.ldo = s->wp; a.n_out = 1; a.width = s->spec.width; a.eps = (float)s->spec.norm_eps; a.rows = s->want_rows + i;
        if (int r = p.done(launch_st_norms(s->act, a, n, cfg), "final norm")) return r;
        if (int r = p.head(s->xn_rows, s->logits_rows, n)) return r;
        SK(cudaMemcpy2DAsync(logits_host + (size_t)i * s->spec.vocab, (size_t)s->spec.vocab * 4, s->logits_rows, (size_t)s->vocab_p * 4, (size_t)s->spec.vocab * 4, n, cudaMemcpyDeviceToHost, e->stream));
        SK(cudaStreamSynchronize(e->stream));
    }
    return CUQWEN_OK;
}

}  // namespace cq
