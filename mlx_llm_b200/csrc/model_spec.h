// What a decoder consists of when config.json lists its layers one by one: every layer names a token mixer and a
// feed-forward, each with its own sizes and constants.  The engine walks this description (engine_layers.cu); a model
// family only supplies the reader of its config.json and its tensor names (model_registry.cu).
#pragma once
#include <cstdint>
#include <string>
#include <vector>

enum class MixerKind { LatentAttention, Mamba2 };
enum class MlpKind { None, DenseGated, Routed };
// act(gate, up) of a gated feed-forward:
//   GeluTanh      gelu(gate) * up with the tanh form of gelu
//   ClippedSwish  g = min(gate, limit), u = clamp(up, -limit, limit):  g * sigmoid(alpha * g) * (u + 1)
enum class GateAct { GeluTanh, ClippedSwish };
struct GateSpec {
    GateAct act = GateAct::GeluTanh;
    float limit = 0.f, alpha = 0.f;
};

// Rotation of consecutive pairs (2i, 2i+1), i < dims/2, by position * base^(-2i/dims); the rest passes unchanged.
struct PairRotSpec {
    double base = 10000.0;
    int dims = 0;
};
// Attention over a shared low-rank latent: per token one vector of kv_rank values and one rotated key part of rot_dim
// values are cached; every head's keys and values are linear images of the latent.
struct LatentAttnSpec {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0;
    float scale = 0.f;
    PairRotSpec rot;
    constexpr int row() const { return kv_rank + rot_dim; }               // values cached per token
    // ... padded for 16-wide tensor-core steps, and to one 64-wide load box at least
    constexpr int row_pad() const { return row() < 64 ? 64 : (row() + 15) / 16 * 16; }
};
// Selective state space with a scalar decay per head: inputs pass a short causal convolution, the state is
// [heads][vdim][state] in f32, the output is gated and normed in groups.
struct Mamba2Spec {
    int heads = 0, vdim = 0, state = 0, groups = 0, norm_groups = 0, conv = 0;
    constexpr int inner() const { return heads * vdim; }
    constexpr int channels() const { return inner() + 2 * groups * state; }  // x | B | C, the convolved inputs
    constexpr int in_rows() const { return inner() + channels() + heads; }   // z | x | B | C | dt
};
// Routed experts: sigmoid scores, the best `top` experts, the score multiplies the expert's input.
struct RoutedSpec {
    int experts = 0, top = 0, ff = 0;
    GateSpec gate;
};
struct LayerSpec {
    MixerKind mixer = MixerKind::LatentAttention;
    LatentAttnSpec attn;
    Mamba2Spec ssm;
    MlpKind mlp = MlpKind::None;
    int ff = 0;  // dense
    GateSpec gate;
    RoutedSpec moe;
};
// Tensor names of a family: the `i`-th layer's prefix and the few names outside the layers.
struct TensorNames {
    std::string embed = "embed", final_norm = "final.norm", layer = "l", norm1 = "norm1", norm2 = "norm2", mixer = "mix", mlp = "mlp";
    std::string layer_key(int i, const std::string& s) const { return layer + std::to_string(i) + "." + s; }
};
struct ModelSpec {
    std::string family;
    int vocab = 0, width = 0;
    float eps = 1e-5f, logit_scale = 1.f;
    std::vector<LayerSpec> layers;
    TensorNames names;
};
