// What a decoder consists of when config.json lists its layers one by one: every layer names a token mixer and a
// feed-forward, each with its own sizes and constants.  The engine walks this description (engine_layers.cu); a model
// family only supplies the reader of its config.json and its tensor names (model_registry.cu).
#pragma once
#include <cstdint>
#include <string>
#include <vector>

enum class MixerKind { LatentAttention, Mamba2, GroupedAttention, Memory, SideBySide, GatedAverage };
enum class MlpKind { None, DenseGated, DensePlain, Routed };
// act(gate, up) of a gated feed-forward:
//   GeluTanh      gelu(gate) * up with the tanh form of gelu
//   ClippedSwish  g = min(gate, limit), u = clamp(up, -limit, limit):  g * sigmoid(alpha * g) * (u + 1)
//   Swish         gate * sigmoid(gate) * up
// A row weight multiplies the pre-activations (the expert's input), or with scale_out the result (its output).
enum class GateAct { GeluTanh, ClippedSwish, Swish };
struct GateSpec {
    GateAct act = GateAct::GeluTanh;
    float limit = 0.f, alpha = 0.f;
    bool scale_out = false;
};

// Which earlier positions a query may see.  None: all of them; Window: itself and the size - 1 before it; Chunk: those of its own
// stretch of `size` positions, counted from the sequence's start.  first() never falls as the position rises.  The sequence's first
// `keep` positions stay visible behind first() as well (grouped attention).
struct MaskSpec {
    enum Kind { None, Window, Chunk } kind = None;
    int size = 0, keep = 0;
    constexpr int first(int pos) const { return kind == Window ? (pos >= size ? pos - size + 1 : 0) : kind == Chunk ? pos / size * size : 0; }
    // the keys ahead of first(pos) that are visible, and the tiles of `t` keys that hold them ahead of first(pos)'s own tile
    constexpr int kept(int pos) const { return keep < first(pos) ? keep : first(pos); }
    constexpr int kept_tiles(int pos, int t) const { return (keep + t - 1) / t < first(pos) / t ? (keep + t - 1) / t : first(pos) / t; }
    constexpr bool operator==(const MaskSpec& o) const { return kind == o.kind && size == o.size && keep == o.keep; }
};

// Rotation of dims/2 pairs by position * base^(-2i/dims); the rest passes unchanged.  Which coordinates form pair i is the
// mixer's: (2i, 2i+1) in latent attention, (i, i + dims/2) in memories and, unless it says otherwise, in grouped attention.
// With a scaling factor (YaRN) the pairs that turn slowly within `original` positions turn `factor` times slower still, those that turn
// fast stay, with a ramp between the pairs of `fast` and `slow` turns; cosines and sines grow by 0.1 ln(factor) + 1.
struct RotSpec {
    double base = 10000.0;
    int dims = 0;
    double factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;  // factor 0: no scaling
    bool operator==(const RotSpec& o) const {
        return base == o.base && dims == o.dims && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
    }
};
// Attention over a shared low-rank latent: per token one vector of kv_rank values and one rotated key part of rot_dim
// values (0: none) are cached; every head's keys and values are linear images of the latent.
struct LatentAttnSpec {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0;
    float scale = 0.f;
    RotSpec rot;
    MaskSpec mask;
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
// Attention with kv_heads <= heads key / value heads, cached per token.  Keys and values may differ in size.
// maps 2 (differential): every head has two queries and every key / value head two keys, [map 1 | map 2]; each map is an attention of its
// own over the same values, and the head's output is norm(a1 - lambda a2) (1 - diff), the RMS norm over vdim without a weight.
struct GroupedAttnSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 0.f;
    float softcap = 0.f;  // score <- softcap * tanh(score / softcap); 0: no cap
    bool sink = false;    // exp(0) is added to the softmax's denominator
    bool bias = false;    // biases of the query, key and value projections
    bool qk_norm = false; // RMS norm of queries and keys before the rotation, per head ...
    bool norm_all = false; // ... or over all heads at once
    int maps = 1;
    float diff = 0.f;
    bool head_gate = false; // a head's output is multiplied by the sigmoid of a projection of the layer's input, one number per head
    bool neighbours = false; // the rotation's pairs are (2i, 2i+1)
    RotSpec rot;
    MaskSpec mask;
    constexpr int group() const { return heads / kv_heads; }
    constexpr int q_heads() const { return heads * maps; }
    constexpr int k_heads() const { return kv_heads * maps; }
    // values per cached head row, zero-padded for 16-wide steps and to one 64-wide load box at least
    constexpr int k_row() const { return dim < 64 ? 64 : (dim + 15) / 16 * 16; }
    constexpr int v_row() const { return vdim < 64 ? 64 : (vdim + 15) / 16 * 16; }
};
// Linear memory: a state S [dim][vdim] per head in f32, read with the query after the token's own write,
//     S <- decay * S;   S <- S + k u^T;   o = S^T q;   out = norm(o) * gate
// u = v (delta off) or u = beta (v - S^T k) with the decayed S (delta on).  With a bonus b the read-out comes first and sees the
// token's own write only through b:
//     o = S^T q + (q . (b k)) v;   S <- decay * S + k v^T
enum class MemDecay { Fixed, PerHead, PerChannel };  // Fixed: constants; the others from a projection z:
enum class DecayMap { Softplus, Exp };               // exp(-exp(A_log) softplus(z + dt_bias)), or exp(-exp(z + dt_bias))
enum class MemGate { Silu, Sigmoid };
struct MemorySpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;  // kv_heads: heads of q and k
    int conv = 0;          // taps of the causal convolution (then silu) on q, k and v; 0: none
    bool unit = false;     // q and k are unit vectors per head, q times dim^-1/2 (off: k times dim^-1/2)
    float unit_eps = 1e-6f; // x / sqrt(sum x^2 + unit_eps)
    bool delta = false;
    bool norm = false;     // the output norm has a weight [vdim]
    bool norm_heads = false; // ... [heads * vdim]
    bool low_rank = false; // decay and gate come from two-factor projections
    bool bonus = false;
    // > 0: width of the layer's normed input h.  q, k, v, gate and decay then each read a mixture of their own, h + (h' - h) mu, with
    // h' the previous token's h (kept in the record); the decay's projection has two factors with a tanh between them.
    int shift = 0;
    MemDecay decay = MemDecay::Fixed;
    DecayMap decay_map = DecayMap::Softplus;
    MemGate gate = MemGate::Silu;
    RotSpec rot;           // dims 0: no rotation
    constexpr int q_cols() const { return kv_heads * dim; }
    constexpr int channels() const { return 2 * kv_heads * dim + heads * vdim; }  // q | k | v
    constexpr int state_floats() const { return heads * dim * vdim; }
    constexpr int keep() const { return conv > 1 ? conv - 1 : 0; }                 // inputs of the convolution kept between steps
    constexpr int decays() const { return decay == MemDecay::PerChannel ? heads * dim : decay == MemDecay::PerHead ? heads : 0; }
};
// Gated recurrence whose gates read only the current token (minimal GRU), element by element, the state in f32:
//     S <- (1 - z) S + z c,   z = sigmoid(Z + b_z),   c = u + 1/2 for u >= 0 and sigmoid(u) below,   u = U + b_x;   out = S silu(G)
struct GatedAverageSpec {
    int width = 0;
};
// Routed experts: the best `top` of them run for a token.
//   Sigmoid  scores sigmoid(z); a chosen expert's weight is its score
//   Softmax  scores softmax(z); the choice goes by score + correction, the chosen scores are normalised to a sum of `scale`
// The last `identity` router outputs are experts that return their input.  shared_ff > 0: one more expert that every token takes,
// weighted by the sigmoid of a number of its own.
enum class RouteScore { Sigmoid, Softmax };
struct RoutedSpec {
    int experts = 0, top = 0, ff = 0;
    int identity = 0, shared_ff = 0;
    RouteScore score = RouteScore::Sigmoid;
    float scale = 1.f;
    GateSpec gate;
    constexpr int outputs() const { return experts + identity; }
    constexpr int sources() const { return top + (shared_ff > 0 ? 1 : 0); }  // rows that are summed per token
};
struct LayerSpec {
    MixerKind mixer = MixerKind::LatentAttention;
    LatentAttnSpec attn;
    Mamba2Spec ssm;
    GroupedAttnSpec gqa;              // GroupedAttention, SideBySide
    MemorySpec mem;                   // Memory, SideBySide
    GatedAverageSpec avg;             // GatedAverage
    std::vector<double> decay;        // MemDecay::Fixed: per head
    int kv_from = -1;                 // grouped attention: the layer whose cached keys and values this one reads; -1: its own
    float gqa_scale = 1.f, mem_scale = 1.f;
    std::string gqa_key, mem_key;     // what their tensors' names have behind the mixer's prefix
    // one norm: mixer and feed-forward both read it, and their sum is added to the stream (plain feed-forwards only)
    bool parallel = false;
    MlpKind mlp = MlpKind::None;
    int ff = 0;  // dense; DensePlain: down(gelu(up)), the exact gelu
    GateSpec gate;
    RoutedSpec moe;
    bool has_gqa() const { return mixer == MixerKind::GroupedAttention || mixer == MixerKind::SideBySide; }
    bool has_mem() const { return mixer == MixerKind::Memory || mixer == MixerKind::SideBySide; }
};
// Layers start .. stop-1 run `times` times in a row with the same weights, each pass with a cache and a state of its own.
// Ahead of each pass a vector of its own is added to the stream, and, from the second on, the embedding output.
struct LoopSpec {
    int start = 0, stop = 0, times = 0;
};
struct LayerRun {
    int layer, pass;   // pass -1 outside the loop
    bool opens_pass;   // the first layer of its pass
};
// Tensor names of a family: the `i`-th layer's prefix and the few names outside the layers.
struct TensorNames {
    std::string embed = "embed", final_norm = "final.norm", layer = "l", norm1 = "norm1", norm2 = "norm2", mixer = "mix", mlp = "mlp",
                head = "head", loop_step = "loop.step", pairs = "bigram", side = "side", depth = "dwa";
    std::string layer_key(int i, const std::string& s) const { return layer + std::to_string(i) + "." + s; }
};
// A second embedding table, indexed by the previous and the current token: row (previous * mul_prev + current * mul_cur) mod buckets,
// for a sequence's first token row `buckets`.  buckets 0: none.
struct PairSpec {
    int buckets = 0;
    int64_t mul_prev = 0, mul_cur = 0;
};
struct ModelSpec {
    std::string family;
    int vocab = 0, width = 0;
    float embed_scale = 1.f;
    PairSpec pairs;
    float eps = 1e-5f, logit_scale = 1.f;
    float norm_offset = 0.f;  // added to the stored weights of the layers' norms and the final norm
    bool own_head = false;    // an output projection beside the embedding table
    // > 0: this many residual streams.  A sub-layer reads sum_s in[s] x_s; afterwards x_t = sum_s mix[s][t] x_s + out[t] y; the model
    // ends with their sum.  0: one stream, x + y.
    int streams = 0;
    // The norms lie behind the sub-layers, which read the stream itself:  x <- x + residual_mult * norm(sublayer(x)), in norm_groups
    // equal parts that are normed by themselves.
    bool post_norm = false;
    float residual_mult = 1.f;
    int norm_groups = 1;
    // > 0: behind the feed-forward a layer adds residual_mult * norm(proj(gelu(gate x) * e)), with e the layer's side_dim columns of the
    // current token's row in a table of its own
    int side_dim = 0;
    // a layer passes on the weighted sum of the embedding output and of what it and every layer before it computed
    bool depth_average = false;
    std::vector<LayerSpec> layers;
    LoopSpec loop;
    TensorNames names;
    std::vector<LayerRun> runs() const {
        std::vector<LayerRun> r;
        const int n = (int)layers.size();
        for (int i = 0; i < loop.start; i++) r.push_back({i, -1, false});
        for (int t = 0; t < loop.times; t++)
            for (int i = loop.start; i < loop.stop; i++) r.push_back({i, t, i == loop.start});
        for (int i = loop.stop; i < n; i++) r.push_back({i, -1, false});
        return r;
    }
};
