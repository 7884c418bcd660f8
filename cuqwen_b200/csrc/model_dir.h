// Model directories: config.json + model.safetensors.  The configuration names its design; the registry in model_dir.cu
// turns it into a StackSpec - a list of layers, each with its own mixer, feed-forward and sizes - which is all that the
// rest of the library knows about a model.  A further design adds a registry row and, where it brings a mechanism that is
// not here yet, a member beside the existing ones.
#pragma once
#include <stddef.h>
#include <stdint.h>

#include <string>
#include <vector>

namespace cq {

// Rotation of the first `dims` entries of a vector, entry i paired with entry i + dims / 2, angle pos * base^(-2 i / dims).
struct RotarySpec { int dims = 0; double base = 0; };

// Softmax attention over a low-rank latent per token (queries through a latent of their own).  The cache row of a token is
// [normed latent (kv_rank) | rotated key part shared by all heads (rot_dim)].
struct LatentAttnSpec {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    int window = 0;          // length of the stretch of positions, ending with its own, that a query sees; 0 = all up to its own
    int kv_from = -1;        // >= 0: attends to the rows that layer's latent projection cached; no projection of its own
    double scale = 0;
    RotarySpec rot;
    bool sink = false;       // the softmax denominator has one more learned term per head
    bool gate = false;       // heads times sigmoid(W_g h) before the output projection
};

// Causal softmax attention; query head h uses key / value head h / (heads / kv_heads); rot.dims 0 = no rotation.
struct GroupedAttnSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    double scale = 0;
    RotarySpec rot;
};

// Recurrence with a decay per key channel that depends on the token through a product of two thin matrices (rank: their
// common length, known from the weights), and a bonus for the current token.  Its inputs are mixes of the token's and the
// previous token's mixer input.
struct TimeMixSpec { int heads = 0, dim = 0, rank = 0; };

// Recurrence that corrects what the state holds for a key (gated delta rule), its q / k / v through a causal convolution of
// `conv` taps; value head h uses key head h / (heads / kv_heads).
struct DeltaSpec { int heads = 0, kv_heads = 0, dim = 0, vdim = 0, conv = 0; };

enum MixerKind : int {
    MIX_LATENT = 0,          // attn
    MIX_PARALLEL = 1,        // left_scale * grouped attention + right_scale * time mixing, of the same input
    MIX_DELTA = 2
};

enum MlpKind : int {
    MLP_RELU2 = 0,           // W_down relu(W_up h)^2
    MLP_CLAMPED_GLU = 1      // g = min(W_gate h, limit), u = clamp(W_up h, +-limit): W_down (g sigmoid(slope g) (u + 1))
};
struct DenseMlpSpec { int ff = 0; MlpKind kind = MLP_RELU2; double limit = 0, slope = 0; };      // ff 0 = no feed-forward

struct LayerSpec {
    MixerKind kind = MIX_LATENT;
    LatentAttnSpec attn;
    GroupedAttnSpec left; TimeMixSpec right; double left_scale = 1, right_scale = 1;
    DeltaSpec delta;
    DenseMlpSpec mlp;
};

// Layers with one residual sum: x += mixer(norm1 x) + mlp(norm2 x), then (side_dim > 0) x += rmsnorm(W_proj (gelu(W_gate x) * e))
// with e the layer's slice of a second embedding table's row.  Sequential layers: x += m * mixer(norm1 x), then
// x += m * mlp(norm2 x), m = residual_mult.
struct StackSpec {
    std::string design;
    int vocab = 0, width = 0, side_dim = 0;
    double norm_eps = 0;
    bool sequential = false;
    double residual_mult = 1, embed_scale = 1, logit_softcap = 0;      // logits = cap * tanh(logits / cap); 0 = as they are
    double norm_offset = 0;                                            // added to the stored weights of the layers' and the model's norms
    std::vector<LayerSpec> layers;
    bool recurrent() const { for (const LayerSpec& l : layers) if (l.kind != MIX_LATENT) return true; return false; }
};

// Reads DIR/config.json; returns a CUQWEN_* code (message through report_error).
int read_model_config(const char* dir, StackSpec* out);
// Fills the sizes that only the tensors' shapes tell, from DIR/model.safetensors.
int read_model_shapes(const char* dir, StackSpec* spec);
// One line per fact, for logs and tests.
std::string describe_spec(const StackSpec& s);

// The tensors of a memory-mapped safetensors file.
class Safetensors {
public:
    struct Tensor { std::string name, dtype; std::vector<int64_t> shape; const uint8_t* data = nullptr; size_t bytes = 0; };
    ~Safetensors();
    int open(const char* path);                          // CUQWEN_* code
    const Tensor* find(const std::string& name) const;
    // The tensor, checked: dtype "BF16" and this shape (cols 0: a vector of `rows`).  Null after report_error otherwise.
    const Tensor* expect(const std::string& name, int64_t rows, int64_t cols) const;

private:
    void* map_ = nullptr;
    size_t size_ = 0;
    std::vector<Tensor> tensors_;
};

}  // namespace cq
