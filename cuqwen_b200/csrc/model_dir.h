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

struct DenseMlpSpec { int ff = 0; };      // W_down relu(W_up h)^2; ff 0 = no feed-forward

struct LayerSpec { LatentAttnSpec attn; DenseMlpSpec mlp; };

// All layers: x += mixer(norm1 x) + mlp(norm2 x), then (side_dim > 0) x += rmsnorm(W_proj (gelu(W_gate x) * e)) with e the
// layer's slice of a second embedding table's row.
struct StackSpec {
    std::string design;
    int vocab = 0, width = 0, side_dim = 0;
    double norm_eps = 0;
    std::vector<LayerSpec> layers;
};

// Reads DIR/config.json; returns a CUQWEN_* code (message through report_error).
int read_model_config(const char* dir, StackSpec* out);
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
