// Reader of model directories (see model_dir.h): the design registry and the safetensors index.  Host only.
#include "model_dir.h"

#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstring>

#include "../../include/cuqwen_b200.h"
#include "errors.h"
#include "json.h"

namespace cq {

namespace {

// Fields of a configuration object; the first one that is missing or out of range is remembered.
struct Fields {
    const Json* o;
    std::string where, bad;
    Fields(const Json* obj, std::string w) : o(obj), where(std::move(w)) { if (!o || o->kind != Json::Obj) bad = where + " is not an object"; }
    const Json* get(const char* k) const { return o ? o->get(k) : nullptr; }
    int integer(const char* k, int lo = 1) {
        const Json* v = get(k);
        if (!v || v->kind != Json::Num || v->num != std::floor(v->num) || v->num < lo || v->num > 1e9) { if (bad.empty()) bad = where + "." + k + " must be an integer of at least " + std::to_string(lo); return lo; }
        return (int)v->num;
    }
    double number(const char* k) {
        const Json* v = get(k);
        if (!v || v->kind != Json::Num || !std::isfinite(v->num)) { if (bad.empty()) bad = where + "." + k + " must be a number"; return 0; }
        return v->num;
    }
    bool absent(const char* k) const { const Json* v = get(k); return !v || v->is_null(); }
};

int config_error(const std::string& what) { return report_error(CUQWEN_ERR_DIMS, "config.json: %s", what.c_str()); }

int parse_latent_attention(const Json* mixer, const std::string& where, LatentAttnSpec* a, int layer, const std::vector<LayerSpec>& before) {
    Fields f(mixer, where);
    a->heads = f.integer("heads"); a->dim = f.integer("dim"); a->rot_dim = f.integer("rot_dim"); a->vdim = f.integer("vdim");
    a->q_rank = f.integer("q_rank"); a->kv_rank = f.integer("kv_rank"); a->scale = f.number("scale");
    if (!f.bad.empty()) return config_error(f.bad);
    if (a->rot_dim % 2) return config_error(where + ".rot_dim must be even");
    Fields rot(f.get("rot"), where + ".rot");
    a->rot.base = rot.number("base");
    a->rot.dims = rot.absent("dims") ? a->rot_dim : rot.integer("dims");
    if (!rot.bad.empty()) return config_error(rot.bad);
    if (a->rot.dims != a->rot_dim || !(a->rot.base > 0)) return config_error(where + ".rot must cover rot_dim with a positive base");
    if (!f.absent("mask")) {
        Fields m(f.get("mask"), where + ".mask");
        a->window = m.absent("size") ? 0 : m.integer("size");
        if (!m.bad.empty()) return config_error(m.bad);
    }
    if (!f.absent("kv_from")) {
        a->kv_from = f.integer("kv_from", 0);
        if (!f.bad.empty()) return config_error(f.bad);
        if (a->kv_from >= layer || before[a->kv_from].attn.kv_from >= 0) return config_error(where + ".kv_from must name an earlier layer with a latent projection of its own");
        const LatentAttnSpec& s = before[a->kv_from].attn;
        if (s.kv_rank != a->kv_rank || s.rot_dim != a->rot_dim || s.rot.base != a->rot.base)
            return config_error(where + ": kv_rank, rot_dim and rotation must equal those of layer " + std::to_string(a->kv_from));
    }
    return CUQWEN_OK;
}

// Falivik: parallel layers (two norms of the same stream), windowed latent attention with a sink per head and an output
// gate, latents optionally shared between layers, squared-relu feed-forward, a per-layer token input.
int parse_falivik(const Json& cfg, StackSpec* s) {
    Fields top(&cfg, "model");
    s->vocab = top.integer("vocab"); s->width = top.integer("width");
    if (!top.bad.empty()) return config_error(top.bad);
    Fields norm(top.get("norm"), "norm");
    s->norm_eps = norm.number("eps");
    if (!norm.bad.empty()) return config_error(norm.bad);
    if (!top.absent("token_side")) {
        Fields side(top.get("token_side"), "token_side");
        s->side_dim = side.integer("dim");
        if (!side.bad.empty()) return config_error(side.bad);
    }
    const Json* layers = top.get("layers");
    if (!layers || layers->kind != Json::Arr || layers->arr.empty()) return config_error("layers must be a list");
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const Json& l = layers->arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]";
        Fields f(&l, where);
        if (!f.bad.empty()) return config_error(f.bad);
        const Json* type = f.get("type");
        if (!type || type->kind != Json::Str || type->str != "latent_attention") return config_error(where + ".type: this design has the mixer latent_attention only");
        LayerSpec L;
        L.attn.sink = L.attn.gate = true;
        if (int r = parse_latent_attention(f.get("mixer"), where + ".mixer", &L.attn, (int)i, s->layers)) return r;
        if (!f.absent("mlp")) {
            Fields m(f.get("mlp"), where + ".mlp");
            const Json* kind = m.get("kind");
            if (!kind || kind->kind != Json::Str || kind->str != "dense") return config_error(where + ".mlp.kind: this design has dense feed-forwards only");
            L.mlp.ff = m.integer("ff");
            if (!m.bad.empty()) return config_error(m.bad);
        }
        s->layers.push_back(L);
    }
    return CUQWEN_OK;
}

int parse_rotary(const Fields& f, const std::string& where, int dim, RotarySpec* r) {
    if (f.absent("rot")) return CUQWEN_OK;
    Fields rot(f.get("rot"), where + ".rot");
    r->base = rot.number("base"); r->dims = rot.integer("dims", 0);
    if (!rot.bad.empty()) return config_error(rot.bad);
    if (r->dims % 2 || r->dims > dim || !(r->base > 0)) return config_error(where + ".rot: an even number of dims, at most the head's, and a positive base");
    return CUQWEN_OK;
}
int parse_clamped_glu(const Json* mlp, const std::string& where, double slope, DenseMlpSpec* m) {
    Fields f(mlp, where);
    const Json* kind = f.get("kind");
    if (!kind || kind->kind != Json::Str || kind->str != "dense") return config_error(where + ".kind: this design has dense feed-forwards only");
    m->kind = MLP_CLAMPED_GLU; m->ff = f.integer("ff"); m->limit = f.number("limit"); m->slope = slope;
    if (!f.bad.empty()) return config_error(f.bad);
    if (!(m->limit > 0)) return config_error(where + ".limit must be positive");
    return CUQWEN_OK;
}
int parse_parallel(const Json* mixer, const std::string& where, LayerSpec* L) {
    Fields f(mixer, where);
    L->kind = MIX_PARALLEL;
    L->left_scale = f.number("left_scale"); L->right_scale = f.number("right_scale");
    if (!f.bad.empty()) return config_error(f.bad);
    Fields l(f.get("left"), where + ".left"), r(f.get("right"), where + ".right");
    GroupedAttnSpec& a = L->left;
    a.heads = l.integer("heads"); a.kv_heads = l.integer("kv_heads"); a.dim = l.integer("dim"); a.vdim = l.integer("vdim"); a.scale = l.number("scale");
    if (!l.bad.empty()) return config_error(l.bad);
    if (a.heads % a.kv_heads) return config_error(where + ".left.heads must be a multiple of kv_heads");
    if (int e = parse_rotary(l, where + ".left", a.dim, &a.rot)) return e;
    L->right.heads = r.integer("heads"); L->right.dim = r.integer("dim");
    return r.bad.empty() ? (int)CUQWEN_OK : config_error(r.bad);
}
int parse_delta(const Json* mixer, const std::string& where, LayerSpec* L) {
    Fields f(mixer, where);
    L->kind = MIX_DELTA;
    DeltaSpec& d = L->delta;
    d.heads = f.integer("heads"); d.kv_heads = f.integer("kv_heads"); d.dim = f.integer("dim"); d.vdim = f.integer("vdim"); d.conv = f.integer("conv");
    if (!f.bad.empty()) return config_error(f.bad);
    if (d.heads % d.kv_heads) return config_error(where + ".heads must be a multiple of kv_heads");
    return CUQWEN_OK;
}

// Gipotar: sequential pre-norm layers (norm weights stored about zero) whose mixer is either softmax attention beside time
// mixing or a gated delta rule; clamped gated feed-forward or none; scaled embedding, soft-capped logits.
int parse_gipotar(const Json& cfg, StackSpec* s) {
    constexpr double kSlope = 1.702;
    Fields top(&cfg, "model");
    s->sequential = true; s->norm_offset = 1;
    s->vocab = top.integer("vocab"); s->width = top.integer("width");
    if (!top.absent("residual_mult")) s->residual_mult = top.number("residual_mult");
    if (!top.absent("logit_softcap")) s->logit_softcap = top.number("logit_softcap");
    if (!top.bad.empty()) return config_error(top.bad);
    if (s->logit_softcap < 0) return config_error("logit_softcap must not be negative");
    Fields norm(top.get("norm"), "norm");
    s->norm_eps = norm.number("eps");
    if (!norm.bad.empty()) return config_error(norm.bad);
    if (!top.absent("embedding")) {
        Fields e(top.get("embedding"), "embedding");
        if (!e.absent("scale")) s->embed_scale = e.number("scale");
        if (!e.bad.empty()) return config_error(e.bad);
    }
    const Json* layers = top.get("layers");
    if (!layers || layers->kind != Json::Arr || layers->arr.empty()) return config_error("layers must be a list");
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const std::string where = "layers[" + std::to_string(i) + "]";
        Fields f(&layers->arr[i], where);
        if (!f.bad.empty()) return config_error(f.bad);
        const Json* type = f.get("type");
        const std::string t = type && type->kind == Json::Str ? type->str : "";
        LayerSpec L;
        if (t == "parallel") { if (int r = parse_parallel(f.get("mixer"), where + ".mixer", &L)) return r; }
        else if (t == "delta") { if (int r = parse_delta(f.get("mixer"), where + ".mixer", &L)) return r; }
        else return config_error(where + ".type: this design has the mixers parallel and delta");
        if (!f.absent("mlp")) if (int r = parse_clamped_glu(f.get("mlp"), where + ".mlp", kSlope, &L.mlp)) return r;
        s->layers.push_back(L);
    }
    return CUQWEN_OK;
}

struct Design { const char* name; int (*parse)(const Json&, StackSpec*); };
const Design kDesigns[] = {
    {"Falivik", parse_falivik},
    {"Gipotar", parse_gipotar},
};

bool read_file(const std::string& path, std::string* out) {
    FILE* f = fopen(path.c_str(), "rb");
    if (!f) return false;
    char buf[65536];
    size_t n;
    while ((n = fread(buf, 1, sizeof buf, f)) > 0) out->append(buf, n);
    const bool ok = !ferror(f);
    fclose(f);
    return ok;
}

}  // namespace

int read_model_config(const char* dir, StackSpec* out) {
    const std::string path = std::string(dir) + "/config.json";
    std::string text;
    if (!read_file(path, &text)) return report_error(CUQWEN_ERR_IO, "cannot read %s", path.c_str());
    Json cfg;
    if (!JsonReader::parse(text.data(), text.size(), &cfg)) return report_error(CUQWEN_ERR_IO, "%s is not valid JSON", path.c_str());
    const Json* a = cfg.get("architecture");
    if (!a || a->kind != Json::Str) return config_error("no \"architecture\" name");
    for (const Design& d : kDesigns)
        if (a->str == d.name) { *out = StackSpec(); out->design = d.name; return d.parse(cfg, out); }
    return config_error("unknown architecture \"" + a->str + "\"");
}

int read_model_shapes(const char* dir, StackSpec* spec) {
    Safetensors st;
    bool opened = false;
    for (size_t i = 0; i < spec->layers.size(); ++i) {
        LayerSpec& L = spec->layers[i];
        if (L.kind != MIX_PARALLEL) continue;
        if (!opened) { if (int r = st.open((std::string(dir) + "/model.safetensors").c_str())) return r; opened = true; }
        const std::string name = "l" + std::to_string(i) + ".mix.right.w1";
        const Safetensors::Tensor* t = st.find(name);
        if (!t) return report_error(CUQWEN_ERR_DIMS, "tensor %s is missing", name.c_str());
        if (t->shape.size() != 2 || t->shape[0] < 1 || t->shape[0] > (1 << 20)) return report_error(CUQWEN_ERR_DIMS, "tensor %s is no matrix", name.c_str());
        L.right.rank = (int)t->shape[0];
    }
    return CUQWEN_OK;
}

std::string describe_spec(const StackSpec& s) {
    char b[640];
    snprintf(b, sizeof b, "design %s\nvocab %d\nwidth %d\nlayers %zu\nnorm_eps %.9g\nside_dim %d\n", s.design.c_str(), s.vocab, s.width, s.layers.size(), s.norm_eps, s.side_dim);
    std::string t = b;
    if (s.sequential) {
        snprintf(b, sizeof b, "residual_mult %.9g\nembed_scale %.9g\nlogit_softcap %.9g\n", s.residual_mult, s.embed_scale, s.logit_softcap);
        t += b;
    }
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const LayerSpec& L = s.layers[i];
        if (L.kind == MIX_LATENT) {
            const LatentAttnSpec& a = L.attn;
            snprintf(b, sizeof b, "layer %zu latent_attention heads %d dim %d rot_dim %d vdim %d q_rank %d kv_rank %d window %d kv_from %d scale %.9g rot_base %.9g sink %d gate %d ff %d\n",
                     i, a.heads, a.dim, a.rot_dim, a.vdim, a.q_rank, a.kv_rank, a.window, a.kv_from, a.scale, a.rot.base, a.sink, a.gate, L.mlp.ff);
        } else if (L.kind == MIX_PARALLEL)
            snprintf(b, sizeof b, "layer %zu parallel left_heads %d left_kv_heads %d left_dim %d left_vdim %d score_scale %.9g rot_dims %d rot_base %.9g right_heads %d right_dim %d left_scale %.9g right_scale %.9g ff %d limit %.9g\n",
                     i, L.left.heads, L.left.kv_heads, L.left.dim, L.left.vdim, L.left.scale, L.left.rot.dims, L.left.rot.base, L.right.heads, L.right.dim, L.left_scale, L.right_scale, L.mlp.ff, L.mlp.limit);
        else
            snprintf(b, sizeof b, "layer %zu delta heads %d kv_heads %d dim %d vdim %d conv %d ff %d limit %.9g\n", i, L.delta.heads, L.delta.kv_heads, L.delta.dim, L.delta.vdim, L.delta.conv, L.mlp.ff, L.mlp.limit);
        t += b;
    }
    return t;
}

// ---- safetensors: 8-byte little-endian header length, the JSON header, then the data ----------------------------------
Safetensors::~Safetensors() { if (map_) munmap(map_, size_); }

int Safetensors::open(const char* path) {
    const int fd = ::open(path, O_RDONLY);
    if (fd < 0) return report_error(CUQWEN_ERR_IO, "cannot open %s", path);
    struct stat st;
    if (fstat(fd, &st) || st.st_size < 8) { close(fd); return report_error(CUQWEN_ERR_IO, "%s is too short", path); }
    size_ = (size_t)st.st_size;
    map_ = mmap(nullptr, size_, PROT_READ, MAP_PRIVATE, fd, 0);
    close(fd);
    if (map_ == MAP_FAILED) { map_ = nullptr; return report_error(CUQWEN_ERR_IO, "mmap failed for %s", path); }
    const uint8_t* p = (const uint8_t*)map_;
    uint64_t n = 0;
    for (int i = 7; i >= 0; --i) n = n << 8 | p[i];
    if (n > size_ - 8) return report_error(CUQWEN_ERR_IO, "%s: header longer than the file", path);
    Json h;
    if (!JsonReader::parse((const char*)p + 8, (size_t)n, &h) || h.kind != Json::Obj) return report_error(CUQWEN_ERR_IO, "%s: header is not a JSON object", path);
    const uint8_t* data = p + 8 + n;
    const size_t room = size_ - 8 - (size_t)n;
    for (const auto& kv : h.obj) {
        if (kv.first == "__metadata__") continue;
        const Json *dt = kv.second.get("dtype"), *sh = kv.second.get("shape"), *off = kv.second.get("data_offsets");
        if (!dt || dt->kind != Json::Str || !sh || sh->kind != Json::Arr || !off || off->kind != Json::Arr || off->arr.size() != 2)
            return report_error(CUQWEN_ERR_IO, "%s: bad entry for tensor %s", path, kv.first.c_str());
        Tensor t;
        t.name = kv.first; t.dtype = dt->str;
        double count = 1;
        for (const Json& d : sh->arr) { t.shape.push_back((int64_t)d.num); count *= d.num; }
        const double a = off->arr[0].num, b = off->arr[1].num;
        const int es = t.dtype == "BF16" || t.dtype == "F16" || t.dtype == "I16" ? 2 : t.dtype == "F32" || t.dtype == "I32" ? 4 : t.dtype == "I64" || t.dtype == "F64" ? 8 : 1;
        if (!(a >= 0) || !(b >= a) || b > (double)room || count * es != b - a) return report_error(CUQWEN_ERR_IO, "%s: tensor %s lies outside the file or does not fit its shape", path, kv.first.c_str());
        t.data = data + (size_t)a; t.bytes = (size_t)(b - a);
        tensors_.push_back(std::move(t));
    }
    std::sort(tensors_.begin(), tensors_.end(), [](const Tensor& x, const Tensor& y) { return x.name < y.name; });
    return CUQWEN_OK;
}

const Safetensors::Tensor* Safetensors::find(const std::string& name) const {
    auto it = std::lower_bound(tensors_.begin(), tensors_.end(), name, [](const Tensor& t, const std::string& n) { return t.name < n; });
    return it != tensors_.end() && it->name == name ? &*it : nullptr;
}

const Safetensors::Tensor* Safetensors::expect(const std::string& name, int64_t rows, int64_t cols) const {
    const Tensor* t = find(name);
    if (!t) { report_error(CUQWEN_ERR_IO, "tensor %s is missing", name.c_str()); return nullptr; }
    const bool fits = cols ? t->shape.size() == 2 && t->shape[0] == rows && t->shape[1] == cols : t->shape.size() == 1 && t->shape[0] == rows;
    if (t->dtype != "BF16" || !fits) {
        std::string sh;
        for (int64_t d : t->shape) sh += (sh.empty() ? "" : ", ") + std::to_string(d);
        report_error(CUQWEN_ERR_DIMS, "tensor %s is %s [%s], expected BF16 [%lld%s]", name.c_str(), t->dtype.c_str(), sh.c_str(), (long long)rows,
                     cols ? (", " + std::to_string(cols)).c_str() : "");
        return nullptr;
    }
    return t;
}

}  // namespace cq
