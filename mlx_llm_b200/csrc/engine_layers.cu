// Models described layer by layer (model_spec.h): weights, workspace and the forward over one ragged batch.
//
// The forward is called by the engine's step (b2_engine_forward) with the packer's metadata, like the flat decoders'
// layers; pages, block tables, recurrent slots, scheduling and sampling are the engine's.  The residual stream is f32.
// Every sub-layer leaves what it adds in `y` (f32); the next norm adds it to the stream on its way (b2_add_norm_launch; with several
// streams b2_stream_norm_launch).  Where the norms lie behind the sub-layers, one kernel norms y, adds it and leaves the next sub-layer's
// input (b2_post_norm_launch).
#include <algorithm>
#include <cmath>
#include <cstring>

#include "engine.h"
#include "layer_kernels.h"

namespace {

int up(int n, int to) { return (n + to - 1) / to * to; }
// Padded dimensions of a projection: features in whole 128-row tiles, inputs in whole 64-wide slabs (256-wide where that
// costs little), so that every projection kernel is eligible whatever the model's sizes are.  The padding is zero.
int pad_n(int n) { return up(n, 128); }
int pad_k(int k) { return k >= 768 ? up(k, 256) : up(k, 64); }

constexpr int kSideSplit = 256;

struct GroupW {  // one matrix per group (expert or head), [G][N][K], N and K padded to 64
    int G = 0, N = 0, K = 0;
    void* w = nullptr;
};
struct LayerP {
    float *norm1 = nullptr, *norm2 = nullptr;
    // several streams: what the mixer (0) and the feed-forward (1) read, leave behind and add
    struct {
        float *from = nullptr, *mix = nullptr, *to = nullptr;
    } hc[2];
    // latent attention
    Proj qkv, attn_o;  // rows: q | latent | rotated key part
    float* c_norm = nullptr;
    GroupW k_up_t, v_up;  // [head][kv_rank][dim] and [head][vdim][kv_rank]
    Proj kv_up;           // the same matrices for whole contexts (bf16): plain keys, then values, heads padded to 64-row blocks
    int rope = -1, gather = 0;
    // mamba2
    Proj ssm_in, ssm_o;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *A_log = nullptr, *D = nullptr, *ssm_norm = nullptr;
    // feed-forward
    Proj gu, down, router;  // router: experts | identity experts | the shared expert's number
    GroupW e_gu, e_down;
    Proj s_gu, s_down;      // the shared expert; its first matrix lies behind the router's,
    Proj both;              // which makes one product of the two for few tokens
    float* correction = nullptr;
    // Layers of grouped attention and memories: one product for everything that reads the normed stream, one for everything
    // that is added to it (columns: attention heads | memory heads | feed-forward).
    Proj in, lr, out;  // lr: the second factors of a memory's decay and gate, block-diagonal
    // token shift: `in` holds four matrices that read a mixture each (r, k, v, gate; part_n rows apart) and, behind them, the decay's
    // first factor (a fifth mixture; w1 is that part); lr its second one
    Proj w1;
    int part_n = 0, rank = 0;
    float *mu = nullptr, *bonus = nullptr;
    struct {
        int q = 0, k = 0, v = 0, c = 0, gate = 0, beta = 0, decay = 0, up = 0;  // columns of `in`
        int head_gate = 0, z = 0, u = 0;                                       // ... (z, u, gate: of a gated average)
        int lr_gate = 0;                                                       // columns of `lr`: decay from 0, gate
        int m = 0, f = 0;                                                      // columns of the row `out` reads
    } at;
    float *q_bias = nullptr, *k_bias = nullptr, *v_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *mem_norm = nullptr;
    float *decay = nullptr, *log_decay = nullptr;
    int mem_rope = -1;
    float lambda = 0.f;  // weight of the second map
    float *z_bias = nullptr, *u_bias = nullptr;
    Proj side_gate, side_proj;
    GroupW side_split;  // side_gate by stretches of the stream's columns, for few tokens
    float *side_norm = nullptr, *avg = nullptr;
};
struct RopeTab {
    RotSpec spec;
    float *cos = nullptr, *sin = nullptr;
};

}  // namespace

struct LayeredModel {
    ModelSpec spec;
    std::vector<LayerP> layers;
    std::vector<LayerRun> runs;
    std::vector<int64_t> run_state;  // floats into the slot's record, per run of a layer
    void* embed = nullptr;  // [pad_n(vocab), pad_k(width)]: embedding table, and output projection unless the model has one
    void* head = nullptr;
    float* loop_step = nullptr;  // [times][width]
    Proj pairs, side;            // tables of the token pairs and of the layers' token inputs
    int64_t pair_state = 0;      // where the slot's record keeps the last token
    float* final_norm = nullptr;
    std::vector<RopeTab> ropes;
    int rope_positions = 0;
    std::vector<MaskSpec> gathers;  // distinct masks of the latent layers, whose contexts a step gathers
    int64_t state_floats = 0;
    int* route_counters = nullptr;
    // prefill attention: gathered latents, rotated key parts and expanded keys / values of the contexts in a step
    uint16_t *kv_lat = nullptr, *kv_rot = nullptr, *kv_exp = nullptr;
    int kv_cap = 0, kv_ld_lat = 0, kv_ld_rot = 0, kv_ld_exp = 0;  // rows; widest rows over the layers
    // decode attention: partial results per work item
    float* dec_part = nullptr;
    size_t dec_part_floats = 0, dec_part_row = 0;  // capacity; heads * (values + 2) of the largest layer
    // factors of the memories' chunks, one layer at a time
    uint8_t* chunks = nullptr;
    size_t chunk_bytes = 0;
    uint8_t* arena = nullptr;
    int t_cap = 0, l_cap = 0;
    float* capture = nullptr;
    int64_t capture_cap = 0;
};

namespace {

size_t esz(const b2_model* m) { return m->f32 ? 4 : 2; }

__device__ inline uint64_t mix64d(uint64_t z) {
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return z ^ (z >> 31);
}
// Random block: mean + sd * (sum of four uniforms, unit variance), a function of (seed, element) only
__global__ void random_fill_kernel(void* dst, bool f32, int64_t ld, int64_t cols, int64_t n, uint64_t seed, float mean, float sd) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const uint64_t u = mix64d(seed + (uint64_t)(i + 1) * 0x9E3779B97F4A7C15ull);
    const float s = (float)((u & 0xffff) + ((u >> 16) & 0xffff) + ((u >> 32) & 0xffff) + (u >> 48));
    const float v = mean + sd * (s - 131070.f) * (1.0f / 37837.2f);
    const int64_t at = (i / cols) * ld + i % cols;
    if (f32)
        reinterpret_cast<float*>(dst)[at] = v;
    else
        reinterpret_cast<uint16_t*>(dst)[at] = f2bf(v);
}

// Fills device tensors from a weights container, or with random values when there is none.
struct Filler {
    b2_model* m;
    const b2_weights* w;
    std::string prefix;
    uint64_t seed;
    int64_t bytes = 0;
    std::vector<float> host;
    std::vector<uint16_t> half;

    int32_t alloc(size_t n, void** out) {
        B2_CUDA(cudaMalloc(out, n ? n : 16));
        m->allocs.push_back(*out);
        m->weight_bytes += (int64_t)n;
        B2_CUDA(cudaMemsetAsync(*out, 0, n ? n : 16, m->ctx->stream));
        return B2_OK;
    }
    int32_t fetch(const std::string& name, std::vector<int64_t> shape) {
        const std::string key = prefix.empty() ? name : prefix + "." + name;
        auto it = w->t.find(key);
        B2_REQUIRE(it != w->t.end(), B2_ERR_MISSING_TENSOR, "missing tensor `" + key + "`");
        B2_REQUIRE(it->second.shape == shape, B2_ERR_CONFIG, "tensor `" + key + "` does not have the shape config.json implies");
        B2_REQUIRE(b2_tensor_to_f32(it->second, host), B2_ERR_CONFIG, "tensor `" + key + "` is not a floating-point tensor");
        return B2_OK;
    }
    // rows x cols of `src` (row-major, tight) to dst (row stride ld), in the model's storage format
    int32_t put(const float* src, int rows, int cols, void* dst, int ld) {
        const size_t es = esz(m);
        const void* from = src;
        if (!m->f32) {
            half.resize((size_t)rows * cols);
            for (size_t i = 0; i < half.size(); i++) {
                uint32_t u;
                memcpy(&u, &src[i], 4);
                half[i] = (u & 0x7fffffffu) > 0x7f800000u ? (uint16_t)((u >> 16) | 0x40u) : (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
            }
            from = half.data();
        }
        B2_CUDA(cudaMemcpy2DAsync(dst, (size_t)ld * es, from, (size_t)cols * es, (size_t)cols * es, (size_t)rows, cudaMemcpyHostToDevice, m->ctx->stream));
        B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
        return B2_OK;
    }
    int32_t random(void* dst, bool f32, int rows, int cols, int ld, float mean, float sd) {
        const int64_t n = (int64_t)rows * cols;
        random_fill_kernel<<<(unsigned)((n + 255) / 256), 256, 0, m->ctx->stream>>>(dst, f32, ld, cols, n, ++seed * 0x9E3779B97F4A7C15ull, mean, sd);
        B2_CUDA(cudaGetLastError());
        return B2_OK;
    }
    void* at(void* base, int64_t elems) const { return (uint8_t*)base + elems * (int64_t)esz(m); }

    int32_t proj(Proj& p, int N, int K) {
        p.bits = 0;
        p.N = pad_n(N);
        p.K = pad_k(K);
        return alloc((size_t)p.N * p.K * esz(m), &p.w);
    }
    // tensor [rows, cols] to rows row0.. of p
    int32_t rows(Proj& p, int row0, const std::string& key, int rows, int cols) {
        void* dst = at(p.w, (int64_t)row0 * p.K);
        if (!w) return random(dst, m->f32, rows, cols, p.K, 0.f, 1.0f / sqrtf((float)cols));
        B2_CHECK(fetch(key, {rows, cols}));
        return put(host.data(), rows, cols, dst, p.K);
    }
    // tensor [parts * part_rows, cols]: part i to rows row0 + i * stride of p
    int32_t rows_split(Proj& p, int row0, int stride, const std::string& key, int parts, int part_rows, int cols) {
        if (w) B2_CHECK(fetch(key, {(int64_t)parts * part_rows, cols}));
        for (int i = 0; i < parts; i++) {
            void* dst = at(p.w, (int64_t)(row0 + i * stride) * p.K);
            if (w)
                B2_CHECK(put(host.data() + (size_t)i * part_rows * cols, part_rows, cols, dst, p.K));
            else
                B2_CHECK(random(dst, m->f32, part_rows, cols, p.K, 0.f, 1.0f / sqrtf((float)cols)));
        }
        return B2_OK;
    }
    // a small tensor kept in f32, as stored or (two dimensions) transposed
    int32_t vec(float*& dst, const std::string& key, std::vector<int64_t> shape, float mean, float sd, bool transpose = false, float offset = 0.f) {
        int64_t n = 1;
        for (auto d : shape) n *= d;
        B2_CHECK(alloc((size_t)n * 4, (void**)&dst));
        if (!w) return random(dst, true, 1, (int)n, (int)n, mean, sd);
        B2_CHECK(fetch(key, shape));
        if (offset != 0.f)
            for (float& v : host) v += offset;
        if (transpose) {
            const std::vector<float> a = host;
            for (int64_t r = 0; r < shape[0]; r++)
                for (int64_t c = 0; c < shape[1]; c++) host[(size_t)(c * shape[0] + r)] = a[(size_t)(r * shape[1] + c)];
        }
        B2_CUDA(cudaMemcpyAsync(dst, host.data(), (size_t)n * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
        return B2_OK;
    }
    int32_t upload(float*& dst, const std::vector<float>& v) {
        B2_CHECK(alloc(v.size() * 4, (void**)&dst));
        B2_CUDA(cudaMemcpyAsync(dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
        return B2_OK;
    }
    // first dimension of a two-dimensional tensor whose size only its shape tells; `fallback` for random weights
    int32_t rows_of(const std::string& name, int fallback, int* out) {
        *out = fallback;
        if (!w) return B2_OK;
        const std::string key = prefix.empty() ? name : prefix + "." + name;
        auto it = w->t.find(key);
        B2_REQUIRE(it != w->t.end(), B2_ERR_MISSING_TENSOR, "missing tensor `" + key + "`");
        B2_REQUIRE(it->second.shape.size() == 2 && it->second.shape[0] > 0, B2_ERR_CONFIG, "tensor `" + key + "` is not a matrix");
        *out = (int)it->second.shape[0];
        return B2_OK;
    }
    // tensor [rows, cols] to the block of p at (row0, col0)
    int32_t block(Proj& p, int row0, int col0, const std::string& key, int rows, int cols) {
        void* dst = at(p.w, (int64_t)row0 * p.K + col0);
        if (!w) return random(dst, m->f32, rows, cols, p.K, 0.f, 1.0f / sqrtf((float)cols));
        B2_CHECK(fetch(key, {rows, cols}));
        return put(host.data(), rows, cols, dst, p.K);
    }
    int32_t group(GroupW& g, int G, int N, int K) {
        g.G = G;
        g.N = up(N, 64);
        g.K = up(K, 64);
        return alloc((size_t)G * g.N * g.K * esz(m), &g.w);
    }
    int32_t group_rows(GroupW& g, int i, int row0, const std::string& key, int rows, int cols) {
        void* dst = at(g.w, ((int64_t)i * g.N + row0) * g.K);
        if (!w) return random(dst, m->f32, rows, cols, g.K, 0.f, 1.0f / sqrtf((float)cols));
        B2_CHECK(fetch(key, {rows, cols}));
        return put(host.data(), rows, cols, dst, g.K);
    }
    // tensor [G * rows, cols] split by rows over the groups, each part transposed when asked
    int32_t group_split(GroupW& g, const std::string& key, int rows, int cols, bool transpose) {
        if (!w) {
            for (int i = 0; i < g.G; i++)
                B2_CHECK(random(at(g.w, (int64_t)i * g.N * g.K), m->f32, transpose ? cols : rows, transpose ? rows : cols, g.K, 0.f, 1.0f / sqrtf((float)cols)));
            return B2_OK;
        }
        B2_CHECK(fetch(key, {(int64_t)g.G * rows, cols}));
        std::vector<float> part((size_t)rows * cols);
        for (int i = 0; i < g.G; i++) {
            const float* s = host.data() + (size_t)i * rows * cols;
            if (transpose)
                for (int r = 0; r < rows; r++)
                    for (int c = 0; c < cols; c++) part[(size_t)c * rows + r] = s[(size_t)r * cols + c];
            B2_CHECK(put(transpose ? part.data() : s, transpose ? cols : rows, transpose ? rows : cols, at(g.w, (int64_t)i * g.N * g.K), g.K));
        }
        return B2_OK;
    }
};

int rope_table(LayeredModel& lm, const RotSpec& rot) {
    for (size_t r = 0; r < lm.ropes.size(); r++)
        if (lm.ropes[r].spec == rot) return (int)r;
    lm.ropes.push_back(RopeTab{rot});
    return (int)lm.ropes.size() - 1;
}

// Grouped attention, memories, and in parallel layers the feed-forward: one matrix in, one matrix out.
int32_t load_branches(Filler& f, LayeredModel& lm, int i) {
    const LayerSpec& L = lm.spec.layers[i];
    const TensorNames& tn = lm.spec.names;
    LayerP& P = lm.layers[i];
    const int W = lm.spec.width;
    const GroupedAttnSpec& a = L.gqa;
    const MemorySpec& s = L.mem;
    auto aq = [&](const std::string& n) { return tn.layer_key(i, tn.mixer + "." + L.gqa_key + n); };
    auto am = [&](const std::string& n) { return tn.layer_key(i, tn.mixer + "." + L.mem_key + n); };
    const bool ff = L.parallel && L.mlp == MlpKind::DensePlain, own_kv = L.kv_from < 0;
    B2_REQUIRE(L.mlp == MlpKind::None || L.parallel == (L.mlp == MlpKind::DensePlain), B2_ERR_UNSUPPORTED,
               "plain feed-forwards belong to parallel layers, gated and routed ones to sequential layers");
    int n = 0, ra = 0, rg = 0, ra8 = 0, need = 0;
    auto take = [&](int& at, int cols) {
        at = n;
        n += up(cols, 8);
    };
    if (L.has_gqa()) {
        B2_REQUIRE(a.dim <= 256 && a.vdim <= 256, B2_ERR_UNSUPPORTED, "grouped attention: head sizes up to 256");
        take(P.at.q, a.q_heads() * a.dim);
        if (own_kv) take(P.at.k, a.k_heads() * a.dim);
        if (own_kv) take(P.at.v, a.kv_heads * a.vdim);
        if (a.head_gate) take(P.at.head_gate, a.heads);
    }
    if (L.has_mem()) {
        B2_REQUIRE(s.dim <= 256, B2_ERR_UNSUPPORTED, "memory: key sizes up to 256");
        take(P.at.c, s.channels());
        if (s.low_rank) {
            const int r = std::max(8, std::min(s.dim, s.vdim));  // for random weights
            B2_CHECK(f.rows_of(am("a1"), r, &ra));
            B2_CHECK(f.rows_of(am("g1"), r, &rg));
            ra8 = up(ra, 8);
            take(P.at.gate, ra8 + rg);
            need = P.at.gate + pad_k(ra8 + rg);  // the second factors' product reads whole slabs
        } else {
            take(P.at.gate, s.heads * s.vdim);
            if (s.decay == MemDecay::PerHead) take(P.at.decay, s.heads);
        }
        if (s.delta) take(P.at.beta, s.heads);
    }
    if (ff) take(P.at.up, L.ff);
    B2_CHECK(f.proj(P.in, std::max(n, need), W));
    if (L.has_gqa()) {
        B2_CHECK(f.rows(P.in, P.at.q, aq("q"), a.q_heads() * a.dim, W));
        if (own_kv) {
            B2_CHECK(f.rows(P.in, P.at.k, aq("k"), a.k_heads() * a.dim, W));
            B2_CHECK(f.rows(P.in, P.at.v, aq("v"), a.kv_heads * a.vdim, W));
        }
        if (a.head_gate) B2_CHECK(f.rows(P.in, P.at.head_gate, aq("g"), a.heads, W));
        P.lambda = a.diff;
        if (a.maps == 2 && f.w) {
            double dot[2] = {0, 0};
            for (int i = 0; i < 2; i++) {
                const std::string n = std::to_string(i + 1);
                B2_CHECK(f.fetch(aq("lq" + n), {a.dim}));
                const std::vector<float> q = f.host;
                B2_CHECK(f.fetch(aq("lk" + n), {a.dim}));
                for (int d = 0; d < a.dim; d++) dot[i] += (double)q[d] * f.host[d];
            }
            P.lambda = (float)(std::exp(dot[0]) - std::exp(dot[1]) + (double)a.diff);
        }
        if (a.bias) {
            B2_CHECK(f.vec(P.q_bias, aq("q.b"), {a.heads * a.dim}, 0.f, 0.1f));
            B2_CHECK(f.vec(P.k_bias, aq("k.b"), {a.kv_heads * a.dim}, 0.f, 0.1f));
            B2_CHECK(f.vec(P.v_bias, aq("v.b"), {a.kv_heads * a.vdim}, 0.f, 0.1f));
        }
        if (a.qk_norm) {
            B2_CHECK(f.vec(P.q_norm, aq("q.norm"), {a.dim}, 1.f, 0.f));
            if (own_kv) B2_CHECK(f.vec(P.k_norm, aq("k.norm"), {a.dim}, 1.f, 0.f));
        }
        if (a.norm_all) {
            B2_CHECK(f.vec(P.q_norm, aq("q.norm"), {a.heads * a.dim}, 1.f, 0.f));
            if (own_kv) B2_CHECK(f.vec(P.k_norm, aq("k.norm"), {a.kv_heads * a.dim}, 1.f, 0.f));
        }
        P.rope = rope_table(lm, a.rot);
        lm.dec_part_row = std::max(lm.dec_part_row, (size_t)a.q_heads() * (a.v_row() + 2));
    }
    if (L.has_mem()) {
        const int Q = s.q_cols(), V = s.heads * s.vdim;
        B2_CHECK(f.rows(P.in, P.at.c, am("q"), Q, W));
        B2_CHECK(f.rows(P.in, P.at.c + Q, am("k"), Q, W));
        B2_CHECK(f.rows(P.in, P.at.c + 2 * Q, am("v"), V, W));
        if (s.conv > 0) {  // [taps][channels], the channels of q, k and v side by side
            std::vector<float> all((size_t)s.conv * s.channels());
            int c0 = 0;
            for (auto& part : {std::pair<const char*, int>{"q.conv", Q}, {"k.conv", Q}, {"v.conv", V}}) {
                if (f.w) {
                    B2_CHECK(f.fetch(am(part.first), {part.second, s.conv}));
                    for (int c = 0; c < part.second; c++)
                        for (int j = 0; j < s.conv; j++) all[(size_t)j * s.channels() + c0 + c] = f.host[(size_t)c * s.conv + j];
                }
                c0 += part.second;
            }
            if (f.w)
                B2_CHECK(f.upload(P.conv_w, all));
            else
                B2_CHECK(f.vec(P.conv_w, "", {s.conv, s.channels()}, 0.f, 0.5f));
        }
        if (s.low_rank) {
            B2_CHECK(f.rows(P.in, P.at.gate, am("a1"), ra, W));
            B2_CHECK(f.rows(P.in, P.at.gate + ra8, am("g1"), rg, W));
            P.at.lr_gate = up(s.decays(), 8);
            B2_CHECK(f.proj(P.lr, P.at.lr_gate + V, ra8 + rg));
            B2_CHECK(f.block(P.lr, 0, 0, am("a2"), s.decays(), ra));
            B2_CHECK(f.block(P.lr, P.at.lr_gate, ra8, am("g2"), V, rg));
        } else {
            B2_CHECK(f.rows(P.in, P.at.gate, am("g"), V, W));
            if (s.decay == MemDecay::PerHead) B2_CHECK(f.rows(P.in, P.at.decay, am("a"), s.heads, W));
        }
        if (s.delta) B2_CHECK(f.rows(P.in, P.at.beta, am("b"), s.heads, W));
        if (s.decay == MemDecay::Fixed) {
            std::vector<float> d, lg;
            for (double x : L.decay) {
                d.push_back((float)x);
                lg.push_back((float)std::log(x));
            }
            B2_CHECK(f.upload(P.decay, d));
            B2_CHECK(f.upload(P.log_decay, lg));
        } else {
            B2_CHECK(f.vec(P.dt_bias, am("dt_bias"), {s.decays()}, -3.f, 1.f));
            B2_CHECK(f.vec(P.A_log, am("A_log"), {s.heads}, 1.f, 0.7f));
        }
        if (s.norm) B2_CHECK(f.vec(P.mem_norm, am("norm"), {s.vdim}, 1.f, 0.f));
        P.mem_rope = s.conv > 0 ? -1 : rope_table(lm, s.rot);
    }
    // what is added to the stream
    const int att = L.has_gqa() ? a.heads * a.vdim : 0, mem = L.has_mem() ? s.heads * s.vdim : 0;
    P.at.m = up(att, 8);
    P.at.f = P.at.m + up(mem, 8);
    B2_CHECK(f.proj(P.out, W, P.at.f + (ff ? L.ff : 0)));
    if (att) B2_CHECK(f.block(P.out, 0, 0, aq("o"), W, att));
    if (mem) B2_CHECK(f.block(P.out, 0, P.at.m, am("o"), W, mem));
    if (ff) {
        B2_CHECK(f.rows(P.in, P.at.up, tn.layer_key(i, tn.mlp + ".up"), L.ff, W));
        B2_CHECK(f.block(P.out, 0, P.at.f, tn.layer_key(i, tn.mlp + ".down"), W, L.ff));
    }
    return B2_OK;
}

// A memory behind a token shift: r, k, v and gate read a mixture of their own each, the decay comes from two factors.
int32_t load_shifted(Filler& f, LayeredModel& lm, int i) {
    const LayerSpec& L = lm.spec.layers[i];
    const TensorNames& tn = lm.spec.names;
    LayerP& P = lm.layers[i];
    const int W = lm.spec.width;
    const MemorySpec& s = L.mem;
    auto key = [&](const std::string& n) { return tn.layer_key(i, tn.mixer + "." + L.mem_key + n); };
    B2_REQUIRE(s.dim <= 256 && s.shift == W, B2_ERR_UNSUPPORTED, "memory: key sizes up to 256");
    const int Q = s.q_cols(), V = s.heads * s.vdim;
    B2_REQUIRE(Q == V, B2_ERR_UNSUPPORTED, "token shift: keys and values of one size");
    P.part_n = pad_n(Q);
    B2_CHECK(f.rows_of(key("w1"), std::max(8, s.dim), &P.rank));
    B2_CHECK(f.proj(P.in, 4 * P.part_n + P.rank, W));
    P.w1 = P.in;
    P.w1.N = pad_n(P.rank);
    P.w1.w = f.at(P.in.w, (int64_t)4 * P.part_n * P.in.K);
    std::vector<float> mu;
    const char* parts[5] = {"r", "k", "v", "g", "w"};
    for (int j = 0; j < 5; j++) {
        if (j < 4) B2_CHECK(f.rows(P.in, j * P.part_n, key(parts[j]), Q, W));
        if (f.w) {
            B2_CHECK(f.fetch(key(std::string("mu.") + parts[j]), {W}));
            mu.insert(mu.end(), f.host.begin(), f.host.end());
        }
    }
    if (f.w)
        B2_CHECK(f.upload(P.mu, mu));
    else
        B2_CHECK(f.vec(P.mu, "", {5, W}, 0.4f, 0.2f));
    B2_CHECK(f.rows(P.w1, 0, key("w1"), P.rank, W));
    B2_CHECK(f.proj(P.lr, Q, P.rank));
    B2_CHECK(f.rows(P.lr, 0, key("w2"), Q, P.rank));
    B2_CHECK(f.vec(P.dt_bias, key("w0"), {Q}, -3.f, 1.5f));
    B2_CHECK(f.vec(P.bonus, key("u"), {s.heads, s.dim}, 0.5f, 0.3f));
    B2_CHECK(f.vec(P.mem_norm, key("norm"), {V}, 1.f, 0.f));
    P.at.gate = 3 * Q;
    B2_CHECK(f.proj(P.out, W, V));
    return f.rows(P.out, 0, key("o"), W, V);
}

// A gated average: one product for everything that reads the stream, one back.
int32_t load_average(Filler& f, LayeredModel& lm, int i) {
    const TensorNames& tn = lm.spec.names;
    LayerP& P = lm.layers[i];
    const int W = lm.spec.width, n = lm.spec.layers[i].avg.width, n8 = up(n, 8);
    auto key = [&](const std::string& s) { return tn.layer_key(i, tn.mixer + "." + s); };
    P.at.z = 0;
    P.at.u = n8;
    P.at.gate = 2 * n8;
    B2_CHECK(f.proj(P.in, 3 * n8, W));
    B2_CHECK(f.rows(P.in, P.at.z, key("z"), n, W));
    B2_CHECK(f.rows(P.in, P.at.u, key("x"), n, W));
    B2_CHECK(f.rows(P.in, P.at.gate, key("g"), n, W));
    for (auto& b : {std::pair<const char*, float**>{"z.b", &P.z_bias}, {"x.b", &P.u_bias}}) {  // zero behind the width
        std::vector<float> v((size_t)n8, 0.f);
        if (f.w) {
            B2_CHECK(f.fetch(key(b.first), {n}));
            std::copy(f.host.begin(), f.host.end(), v.begin());
        } else if (b.second == &P.z_bias) {
            for (int j = 0; j < n; j++) v[j] = -1.f - 5.f * j / n;
        }
        B2_CHECK(f.upload(*b.second, v));
    }
    B2_CHECK(f.proj(P.out, W, n));
    return f.rows(P.out, 0, key("o"), W, n);
}

// What a layer has besides mixer and feed-forward: its token input, its weights of the average over the depth.
int32_t load_extras(Filler& f, LayeredModel& lm, int i) {
    const TensorNames& tn = lm.spec.names;
    LayerP& P = lm.layers[i];
    const int W = lm.spec.width, n = lm.spec.side_dim;
    auto side = [&](const std::string& s) { return tn.layer_key(i, tn.side + "." + s); };
    if (n > 0) {
        B2_CHECK(f.proj(P.side_gate, n, W));
        B2_CHECK(f.rows(P.side_gate, 0, side("gate"), n, W));
        if (!f.m->f32 && W % kSideSplit == 0 && W > kSideSplit) {
            B2_CHECK(f.group(P.side_split, W / kSideSplit, n, kSideSplit));
            for (int g = 0; g < P.side_split.G; g++)
                B2_CUDA(cudaMemcpy2DAsync(f.at(P.side_split.w, (int64_t)g * P.side_split.N * kSideSplit), (size_t)kSideSplit * 2, f.at(P.side_gate.w, (int64_t)g * kSideSplit),
                                          (size_t)P.side_gate.K * 2, (size_t)kSideSplit * 2, (size_t)n, cudaMemcpyDeviceToDevice, f.m->ctx->stream));
        }
        B2_CHECK(f.proj(P.side_proj, W, n));
        B2_CHECK(f.rows(P.side_proj, 0, side("proj"), W, n));
        B2_CHECK(f.vec(P.side_norm, side("norm"), {W}, 1.f, 0.f));
    }
    if (lm.spec.depth_average) B2_CHECK(f.vec(P.avg, tn.layer_key(i, tn.depth), {i + 2}, 1.f / (i + 2), 0.f));
    return B2_OK;
}

int32_t load_layer(Filler& f, LayeredModel& lm, int i) {
    const LayerSpec& L = lm.spec.layers[i];
    const TensorNames& tn = lm.spec.names;
    LayerP& P = lm.layers[i];
    const int W = lm.spec.width;
    auto key = [&](const std::string& s) { return tn.layer_key(i, s); };
    auto mix = [&](const std::string& s) { return tn.layer_key(i, tn.mixer + "." + s); };
    auto mlp = [&](const std::string& s) { return tn.layer_key(i, tn.mlp + "." + s); };
    B2_CHECK(f.vec(P.norm1, key(tn.norm1), {W}, 1.f, 0.f, false, lm.spec.norm_offset));
    for (int q = 0; q < (lm.spec.streams > 0 ? L.mlp == MlpKind::None ? 1 : 2 : 0); q++) {
        const int n = lm.spec.streams;
        const std::string hc = "hc" + std::to_string(q + 1) + ".";
        B2_CHECK(f.vec(P.hc[q].from, key(hc + "in"), {n}, 1.f / n, 0.1f / n));
        B2_CHECK(f.vec(P.hc[q].mix, key(hc + "mix"), {n, n}, 1.f / n, 0.1f / n));
        B2_CHECK(f.vec(P.hc[q].to, key(hc + "out"), {n}, 1.f, 0.2f));
    }
    B2_CHECK(load_extras(f, lm, i));
    if (L.mixer == MixerKind::GatedAverage) {
        B2_CHECK(load_average(f, lm, i));
    } else if (L.mixer == MixerKind::Memory && L.mem.shift > 0) {
        B2_REQUIRE(!L.parallel, B2_ERR_UNSUPPORTED, "a token shift in a parallel layer");
        B2_CHECK(load_shifted(f, lm, i));
    } else if (L.has_gqa() || L.has_mem()) {
        B2_CHECK(load_branches(f, lm, i));
        if (L.parallel) return B2_OK;
    } else if (L.parallel) {
        return b2_fail(B2_ERR_UNSUPPORTED, "parallel layers are available for grouped attention and memories");
    } else if (L.mixer == MixerKind::LatentAttention) {
        const LatentAttnSpec& a = L.attn;
        const int q = a.heads * (a.dim + a.rot_dim);
        B2_CHECK(f.proj(P.qkv, q + a.row(), W));
        B2_CHECK(f.rows(P.qkv, 0, mix("q"), q, W));
        B2_CHECK(f.rows(P.qkv, q, mix("dkv"), a.row(), W));
        B2_CHECK(f.vec(P.c_norm, mix("dkv.norm"), {a.kv_rank}, 1.f, 0.f));
        B2_CHECK(f.group(P.k_up_t, a.heads, a.kv_rank, a.dim));
        B2_CHECK(f.group_split(P.k_up_t, mix("uk"), a.dim, a.kv_rank, true));
        B2_CHECK(f.group(P.v_up, a.heads, a.vdim, a.kv_rank));
        B2_CHECK(f.group_split(P.v_up, mix("uv"), a.vdim, a.kv_rank, false));
        if (!f.m->f32 && b2_latent_prefill_eligible(a)) {
            const int kb = up(a.dim, 64), vb = up(a.vdim, 64), v0 = a.heads * kb;
            B2_CHECK(f.proj(P.kv_up, v0 + a.heads * vb, a.kv_rank));
            B2_CHECK(f.rows_split(P.kv_up, 0, kb, mix("uk"), a.heads, a.dim, a.kv_rank));
            B2_CHECK(f.rows_split(P.kv_up, v0, vb, mix("uv"), a.heads, a.vdim, a.kv_rank));
            lm.kv_ld_lat = std::max(lm.kv_ld_lat, P.kv_up.K);
            lm.kv_ld_rot = std::max(lm.kv_ld_rot, up(a.rot_dim, 64));
            lm.kv_ld_exp = std::max(lm.kv_ld_exp, P.kv_up.N);
        }
        lm.dec_part_row = std::max(lm.dec_part_row, (size_t)a.heads * (a.kv_rank + 2));
        B2_CHECK(f.proj(P.attn_o, W, a.heads * a.vdim));
        B2_CHECK(f.rows(P.attn_o, 0, mix("o"), W, a.heads * a.vdim));
        while (P.gather < (int)lm.gathers.size() && !(lm.gathers[P.gather] == a.mask)) P.gather++;
        if (P.gather == (int)lm.gathers.size()) lm.gathers.push_back(a.mask);
        if (a.rot_dim > 0) P.rope = rope_table(lm, a.rot);
    } else {
        const Mamba2Spec& s = L.ssm;
        B2_CHECK(f.proj(P.ssm_in, s.in_rows(), W));
        B2_CHECK(f.rows(P.ssm_in, 0, mix("in"), s.in_rows(), W));
        B2_CHECK(f.vec(P.conv_w, mix("conv"), {s.channels(), s.conv}, 0.f, 0.5f, true));
        B2_CHECK(f.vec(P.conv_b, mix("conv.b"), {s.channels()}, 0.f, 0.1f));
        B2_CHECK(f.vec(P.dt_bias, mix("dt_bias"), {s.heads}, -3.f, 1.f));
        B2_CHECK(f.vec(P.A_log, mix("A_log"), {s.heads}, 1.f, 0.7f));
        B2_CHECK(f.vec(P.D, mix("D"), {s.heads}, 1.f, 0.f));
        B2_CHECK(f.vec(P.ssm_norm, mix("norm"), {s.inner()}, 1.f, 0.f));
        B2_CHECK(f.proj(P.ssm_o, W, s.inner()));
        B2_CHECK(f.rows(P.ssm_o, 0, mix("o"), W, s.inner()));
    }
    if (L.mlp == MlpKind::None) return B2_OK;
    B2_CHECK(f.vec(P.norm2, key(tn.norm2), {W}, 1.f, 0.f, false, lm.spec.norm_offset));
    if (L.mlp == MlpKind::DenseGated) {
        const int ffp = up(L.ff, 64);
        B2_CHECK(f.proj(P.gu, 2 * ffp, W));
        B2_CHECK(f.rows(P.gu, 0, mlp("gate"), L.ff, W));
        B2_CHECK(f.rows(P.gu, ffp, mlp("up"), L.ff, W));
        B2_CHECK(f.proj(P.down, W, L.ff));
        B2_CHECK(f.rows(P.down, 0, mlp("down"), W, L.ff));
    } else {
        const RoutedSpec& r = L.moe;
        const int ffp = up(r.ff, 64);
        const int rn = pad_n(r.outputs() + (r.shared_ff > 0 ? 1 : 0));
        B2_CHECK(f.proj(P.router, rn + (r.shared_ff > 0 ? 2 * up(r.shared_ff, 64) : 0), W));
        P.router.N = rn;
        B2_CHECK(f.rows(P.router, 0, mlp("router"), r.outputs(), W));
        if (r.score == RouteScore::Softmax) B2_CHECK(f.vec(P.correction, mlp("correction"), {r.outputs()}, 0.f, 0.01f));
        if (r.shared_ff > 0) {
            const int sp = up(r.shared_ff, 64);
            B2_CHECK(f.rows(P.router, r.outputs(), mlp("shared.sg"), 1, W));
            P.s_gu = P.router;
            P.s_gu.N = pad_n(2 * sp);
            P.s_gu.w = f.at(P.router.w, (int64_t)P.router.N * P.router.K);
            P.both = P.router;
            P.both.N = P.router.N + P.s_gu.N;
            B2_CHECK(f.rows(P.s_gu, 0, mlp("shared.gate"), r.shared_ff, W));
            B2_CHECK(f.rows(P.s_gu, sp, mlp("shared.up"), r.shared_ff, W));
            B2_CHECK(f.proj(P.s_down, W, r.shared_ff));
            B2_CHECK(f.rows(P.s_down, 0, mlp("shared.down"), W, r.shared_ff));
        }
        B2_CHECK(f.group(P.e_gu, r.experts, 2 * ffp, W));
        B2_CHECK(f.group(P.e_down, r.experts, W, r.ff));
        for (int e = 0; e < r.experts; e++) {
            const std::string ek = "e" + std::to_string(e) + ".";
            B2_CHECK(f.group_rows(P.e_gu, e, 0, mlp(ek + "gate"), r.ff, W));
            B2_CHECK(f.group_rows(P.e_gu, e, ffp, mlp(ek + "up"), r.ff, W));
            B2_CHECK(f.group_rows(P.e_down, e, 0, mlp(ek + "down"), W, r.ff));
        }
    }
    return B2_OK;
}

// floats of a layer's recurrent record
int64_t record_floats(const LayerSpec& L) {
    if (L.mixer == MixerKind::Mamba2) return up(L.ssm.inner() * L.ssm.state, 4) + up(L.ssm.channels() * (L.ssm.conv - 1), 4);
    if (L.mixer == MixerKind::GatedAverage) return up(L.avg.width, 4);
    return L.has_mem() ? up(L.mem.state_floats() + L.mem.channels() * L.mem.keep() + L.mem.shift, 4) : 0;
}

// ---- workspace ------------------------------------------------------------------------------------------------------
// One allocation, carved for a capacity of `t` tokens and `l` logits rows; the parts a layer needs only while it runs
// share one region.  With base == null the carving only measures.
struct Carver {
    uint8_t* base;
    size_t off = 0;
    template <typename T = void>
    T* take(size_t bytes) {
        off = (off + 255) / 256 * 256;
        T* p = reinterpret_cast<T*>(base ? base + off : nullptr);
        off += bytes;
        return p;
    }
};
constexpr int kFewTokens = 64;  // up to here the weights' bytes decide: products that read the same rows are merged
struct Common {
    float *x, *y, *logits;
    float* past;  // [layers][t][ldx] embedding output and the layers' results, for averages over the depth
    void *xn, *last;
    int ldx, ldn, ldl;
};
struct LatentBufs {
    void *qkv, *q, *q_lat, *o_lat, *att;
    int plain_pad, rot_pad, o_pad, ld_att;
};
struct SsmBufs {
    void *zx, *xbc, *gn;
    float* y;
    int ld_xbc, ld_gn;
};
struct BranchBufs {
    void *in, *lr, *q, *v, *row, *mix, *low;
    float *low_f;
    float *mq, *mk, *lg, *beta, *o;
    int ld_v;
};
struct AverageBufs {
    void *in, *row;
};
struct SideBufs {
    float* z;
    void* act;
};
struct DenseBufs {
    void *gu, *act;
    int ld_act;
};
struct MoeBufs {
    float *both;  // few tokens: logits | the shared expert's pre-activations
    float *logits, *weight, *row_w, *pass, *shared_w;
    int32_t *expert, *offsets, *pos, *src;
    void *xs, *gu, *act, *s_gu, *s_act;
    int ld_act;
};
Common carve_common(Carver& c, const LayeredModel& lm, size_t es, size_t t, size_t l) {
    Common o;
    int top = 1;  // rows of y per token
    for (auto& L : lm.spec.layers)
        if (L.mlp == MlpKind::Routed) top = std::max(top, L.moe.sources());
    o.ldx = pad_n(lm.spec.width);
    o.ldn = pad_k(lm.spec.width);
    o.ldl = pad_n(lm.spec.vocab);
    o.x = c.take<float>(t * o.ldx * std::max(lm.spec.streams, 1) * 4);
    o.past = c.take<float>(lm.spec.depth_average ? lm.layers.size() * t * o.ldx * 4 : 0);
    o.y = c.take<float>(t * top * o.ldx * 4);
    o.xn = c.take(t * o.ldn * es);
    o.last = c.take(l * o.ldn * es);
    o.logits = c.take<float>(l * o.ldl * 4);
    return o;
}
LatentBufs carve_latent(Carver c, const LatentAttnSpec& a, const LayerP& P, size_t es, size_t t, size_t* end) {
    LatentBufs o;
    o.plain_pad = P.k_up_t.K;
    o.rot_pad = up(a.rot_dim, 64);
    o.o_pad = P.v_up.K;
    o.ld_att = P.attn_o.K;
    o.qkv = c.take(t * P.qkv.N * es);
    o.q = c.take(t * a.heads * (o.plain_pad + o.rot_pad) * es);
    o.q_lat = c.take(t * a.heads * a.row_pad() * es);
    o.o_lat = c.take(t * a.heads * o.o_pad * es);
    o.att = c.take(t * o.ld_att * es);
    *end = std::max(*end, c.off);
    return o;
}
SsmBufs carve_ssm(Carver c, const Mamba2Spec& s, const LayerP& P, size_t es, size_t t, size_t* end) {
    SsmBufs o;
    o.ld_xbc = up(s.channels(), 8);
    o.ld_gn = P.ssm_o.K;
    o.zx = c.take(t * P.ssm_in.N * es);
    o.xbc = c.take(t * o.ld_xbc * es);
    o.y = c.take<float>(t * s.inner() * 4);
    o.gn = c.take(t * o.ld_gn * es);
    *end = std::max(*end, c.off);
    return o;
}
BranchBufs carve_branches(Carver c, const LayerSpec& L, const LayerP& P, size_t es, size_t t, size_t* end) {
    BranchBufs o{};
    const MemorySpec& s = L.mem;
    o.in = c.take(t * P.in.N * es);
    o.row = c.take(t * P.out.K * es);
    if (L.has_gqa()) o.q = c.take(t * L.gqa.q_heads() * L.gqa.k_row() * es);
    if (L.has_mem()) {
        o.lr = c.take(s.shift > 0 && es == 2 ? 0 : t * P.lr.N * es);
        if (s.shift > 0) {
            o.mix = c.take(t * 5 * pad_k(s.shift) * es);
            o.low_f = c.take<float>(t * P.w1.N * 4);
            o.low = c.take(es == 4 ? t * P.lr.K * es : 0);
        }
        o.ld_v = up(s.heads * s.vdim, 8);
        o.v = s.conv > 0 ? c.take(t * o.ld_v * es) : nullptr;
        o.mq = c.take<float>(s.bonus ? 0 : t * s.q_cols() * 4);
        o.mk = c.take<float>(s.bonus ? 0 : t * s.q_cols() * 4);
        o.lg = c.take<float>(t * s.decays() * 4);
        o.beta = c.take<float>(t * s.heads * 4);
        o.o = c.take<float>(t * s.heads * s.vdim * 4);
    }
    *end = std::max(*end, c.off);
    return o;
}
AverageBufs carve_average(Carver c, const LayerP& P, size_t es, size_t t, size_t* end) {
    AverageBufs o;
    o.in = c.take(t * P.in.N * es);
    o.row = c.take(t * P.out.K * es);
    *end = std::max(*end, c.off);
    return o;
}
SideBufs carve_side(Carver c, const LayerP& P, size_t es, size_t t, size_t* end) {
    SideBufs o;
    o.z = c.take<float>(std::max(t * P.side_gate.N, (size_t)kFewTokens * P.side_split.G * P.side_split.N) * 4);
    o.act = c.take(t * P.side_proj.K * es);
    *end = std::max(*end, c.off);
    return o;
}
DenseBufs carve_dense(Carver c, const LayerP& P, size_t es, size_t t, size_t* end) {
    DenseBufs o;
    o.ld_act = P.down.K;
    o.gu = c.take(t * P.gu.N * es);
    o.act = c.take(t * o.ld_act * es);
    *end = std::max(*end, c.off);
    return o;
}
MoeBufs carve_moe(Carver c, const RoutedSpec& r, const LayerP& P, int ldn, size_t es, size_t t, size_t* end) {
    MoeBufs o;
    const size_t n = t * r.top;
    o.ld_act = P.e_down.K;
    o.logits = c.take<float>(t * P.router.N * 4);
    o.weight = c.take<float>(n * 4);
    o.row_w = c.take<float>(n * 4);
    o.pass = c.take<float>(t * 4);
    o.shared_w = c.take<float>(t * 4);
    o.expert = c.take<int32_t>(n * 4);
    o.pos = c.take<int32_t>(t * r.sources() * 4);
    o.src = c.take<int32_t>(n * 4);
    o.offsets = c.take<int32_t>((size_t)(r.experts + 1) * 4);
    o.xs = c.take(es == 2 ? n * ldn * es : 0);
    o.gu = c.take(n * P.e_gu.N * es);
    o.act = c.take(n * o.ld_act * es);
    o.both = c.take<float>((size_t)kFewTokens * P.both.N * 4);
    o.s_gu = c.take(t * P.s_gu.N * es);
    o.s_act = c.take(t * P.s_down.K * es);
    *end = std::max(*end, c.off);
    return o;
}
size_t arena_bytes(const LayeredModel& lm, size_t es, size_t t, size_t l) {
    Carver c{nullptr};
    carve_common(c, lm, es, t, l);
    size_t end = c.off;
    for (size_t i = 0; i < lm.layers.size(); i++) {
        const LayerSpec& L = lm.spec.layers[i];
        const LayerP& P = lm.layers[i];
        if (L.mixer == MixerKind::LatentAttention)
            carve_latent(c, L.attn, P, es, t, &end);
        else if (L.mixer == MixerKind::Mamba2)
            carve_ssm(c, L.ssm, P, es, t, &end);
        else if (L.mixer == MixerKind::GatedAverage)
            carve_average(c, P, es, t, &end);
        else
            carve_branches(c, L, P, es, t, &end);
        if (lm.spec.side_dim > 0) carve_side(c, P, es, t, &end);
        if (L.mlp == MlpKind::DenseGated) carve_dense(c, P, es, t, &end);
        if (L.mlp == MlpKind::Routed) carve_moe(c, L.moe, P, pad_k(lm.spec.width), es, t, &end);
    }
    return end + 256;
}
int32_t ensure_arena(b2_model* m, int T, int n_logits) {
    LayeredModel& lm = *m->layered;
    if (T <= lm.t_cap && n_logits <= lm.l_cap && lm.arena) return B2_OK;
    B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    if (T > lm.t_cap) lm.t_cap = up(std::max(T, 128) * 9 / 8, 128);  // at least one box of the projections' row loads
    if (n_logits > lm.l_cap) lm.l_cap = up(std::max(n_logits, 128) * 9 / 8, 128);
    if (lm.arena) B2_CUDA(cudaFree(lm.arena));
    lm.arena = nullptr;
    const size_t bytes = arena_bytes(lm, esz(m), (size_t)lm.t_cap, (size_t)std::max(lm.l_cap, 128));
    if (lm.l_cap == 0) lm.l_cap = 128;
    B2_CUDA(cudaMalloc((void**)&lm.arena, bytes));
    B2_CUDA(cudaMemsetAsync(lm.arena, 0, bytes, m->ctx->stream));
    return B2_OK;
}

constexpr size_t kMaxExpandBytes = 8ull << 30;  // expanded keys and values of one layer; longer contexts stay latent

template <typename T>
int32_t regrow_zero(b2_ctx* ctx, T*& p, size_t elems) {
    if (p) B2_CUDA(cudaFree(p));
    p = nullptr;
    B2_CUDA(cudaMalloc((void**)&p, elems * sizeof(T)));
    B2_CUDA(cudaMemsetAsync(p, 0, elems * sizeof(T), ctx->stream));
    return B2_OK;
}
// Buffers of their own, not parts of the arena: rows past the contexts in use are read with weight zero, so they must
// never hold anything but bf16 numbers.
int32_t ensure_expand(b2_model* m, int rows) {
    LayeredModel& lm = *m->layered;
    if (rows <= lm.kv_cap) return B2_OK;
    B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    lm.kv_cap = up(std::max(rows + rows / 8, 1024), 128);
    B2_CHECK(regrow_zero(m->ctx, lm.kv_lat, (size_t)lm.kv_cap * lm.kv_ld_lat));
    B2_CHECK(regrow_zero(m->ctx, lm.kv_rot, std::max<size_t>((size_t)lm.kv_cap * lm.kv_ld_rot, 8)));
    return regrow_zero(m->ctx, lm.kv_exp, (size_t)lm.kv_cap * lm.kv_ld_exp);
}
int32_t ensure_decode(b2_model* m, int items) {
    LayeredModel& lm = *m->layered;
    const size_t need = (size_t)items * lm.dec_part_row;
    if (need <= lm.dec_part_floats) return B2_OK;
    B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    lm.dec_part_floats = need * 5 / 4;
    return regrow_zero(m->ctx, lm.dec_part, lm.dec_part_floats);
}

int32_t ensure_chunks(b2_model* m, size_t bytes) {
    LayeredModel& lm = *m->layered;
    if (bytes <= lm.chunk_bytes) return B2_OK;
    B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    lm.chunk_bytes = bytes * 5 / 4;
    return regrow_zero(m->ctx, lm.chunks, lm.chunk_bytes);
}

// ---- forward --------------------------------------------------------------------------------------------------------
int32_t linear(b2_model* m, const Proj& p, const void* x, int ldx, int M, int rows_cap, void* out, int ldo, bool out_f32) {
    b2_prof_mark(m->ctx, B2_CLS_GEMM);
    if (m->f32) return b2_linear_f32_launch(m->ctx, (const float*)x, ldx, (const float*)p.w, M, p.N, p.K, (float*)out, ldo);
    GemmParams g{};
    g.x = (const uint16_t*)x;
    g.w = p.w;
    g.group = 64;
    g.M = M;
    g.N = p.N;
    g.K = p.K;
    g.ldx = ldx;
    g.ldo = ldo;
    g.ldres = ldo;
    g.x_rows_cap = rows_cap;
    g.epilogue = out_f32 ? EPI_F32 : EPI_BF16;
    if (out_f32)
        g.out_f32 = (float*)out;
    else
        g.out = (uint16_t*)out;
    return b2_gemm_launch(m->ctx, g);
}

// Keys that the single tokens of a step see under a mask: in all, and the most 16-key tiles of one token.
struct DecodeKeys {
    long sum = 0;
    int tiles = 1;
};
DecodeKeys decode_keys(const std::vector<SeqStep>& seqs, const MaskSpec& mask) {
    DecodeKeys k;
    for (auto& s : seqs)
        if (s.n == 1) {
            const int pos = s.cache->len, lo = mask.first(pos);
            k.sum += pos + 1 - lo + mask.kept(pos);
            k.tiles = std::max(k.tiles, pos / 16 - lo / 16 + 1 + mask.kept_tiles(pos, 16));
        }
    return k;
}
double masked_pairs(const LayeredStep& s, const MaskSpec& mask) {  // (query, visible key) pairs of the prefilling sequences
    if (mask.kind == MaskSpec::None) return s.pf_pairs;
    double n = 0;
    for (auto& q : *s.seqs)
        for (int i = 0, pos = q.cache->len; q.n > 1 && i < q.n; i++, pos++) n += pos + 1 - mask.first(pos) + mask.kept(pos);
    return n;
}
// Latent decode attention: one CTA fills an SM, so the work items (times the head groups) should fill whole rounds of the
// machine: the smallest chunk, in whole tiles from 128 keys on, that does not open another round.
struct DecodeSplit {
    int chunk_tiles, row_chunks;  // 16-key boxes per chunk; most chunks of a row
};
DecodeSplit latent_split(const b2_ctx* ctx, int groups, const MaskSpec& mask, const std::vector<SeqStep>& seqs) {
    const int tile = b2_latent_decode_tile();
    int rows = 0, longest = 1;
    auto keys_of = [&](const SeqStep& s) { return s.cache->len + 1 - mask.first(s.cache->len) / 16 * 16; };
    for (auto& s : seqs)
        if (s.n == 1) {
            rows++;
            longest = std::max(longest, keys_of(s));
        }
    const int sms = ctx->sm_count, budget = std::max(1, (rows * groups + sms - 1) / sms) * sms / groups;
    auto items = [&](int keys) {
        int n = 0;
        for (auto& s : seqs)
            if (s.n == 1) n += (keys_of(s) + keys - 1) / keys;
        return n;
    };
    int lo = (128 + tile - 1) / tile, hi = std::max(lo, (longest + tile - 1) / tile);  // in tiles; the longest context in one chunk is one item per row
    while (lo < hi) {
        const int mid = (lo + hi) / 2;
        if (items(mid * tile) <= budget)
            hi = mid;
        else
            lo = mid + 1;
    }
    return {lo * tile / 16, (longest + lo * tile - 1) / (lo * tile)};
}
int latent_head_groups(const LatentAttnSpec& a) { return a.heads > 16 ? (a.heads + 31) / 32 : 1; }

struct Fwd {  // one step
    b2_model* m;
    LayeredModel& lm;
    b2_pool* pool;
    const LayeredStep& s;
    Common c;
    Carver scratch;
    size_t es, end = 0;

    // `run`: number of the layer's run, whose cache and state are used
    int32_t latent(const LayerSpec& L, const LayerP& P, int run);
    int32_t ssm(const LayerSpec& L, const LayerP& P, int run);
    int32_t branches(const LayerSpec& L, const LayerP& P, int run);
    int32_t attend(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run);
    int32_t remember(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run);
    int32_t shift(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run);
    int32_t average(const LayerSpec& L, const LayerP& P, int run);
    int32_t mix(const LayerSpec& L, const LayerP& P, int run);
    int32_t token_input(const LayerP& P, int layer);
    int32_t post_norm_layers(float* capture);
    int32_t dense(const LayerSpec& L, const LayerP& P);
    int32_t moe(const LayerSpec& L, const LayerP& P, const int32_t** rows, const float** pass);
};

int32_t Fwd::latent(const LayerSpec& L, const LayerP& P, int run) {
    b2_ctx* ctx = m->ctx;
    const LatentAttnSpec& a = L.attn;
    const LatentBufs b = carve_latent(scratch, a, P, es, (size_t)lm.t_cap, &end);
    const int T = s.T, W = a.row_pad(), q_row = b.plain_pad + b.rot_pad;
    const float scale_log2 = a.scale * 1.4426950408889634f;
    void* cache = pool->planes[pool->layer_plane[run]].base;
    B2_CHECK(linear(m, P.qkv, c.xn, c.ldn, T, lm.t_cap, b.qkv, P.qkv.N, false));
    LatentPrepParams pp{};
    pp.qkv = b.qkv;
    pp.ld = P.qkv.N;
    pp.T = T;
    pp.positions = s.mo->positions;
    pp.slot_mapping = s.mo->slot_mapping;
    if (P.rope >= 0) {
        pp.cos_t = lm.ropes[P.rope].cos;
        pp.sin_t = lm.ropes[P.rope].sin;
    }
    pp.c_norm = P.c_norm;
    pp.eps = lm.spec.eps;
    pp.cache = cache;
    pp.q = b.q;
    pp.plain_pad = b.plain_pad;
    pp.rot_pad = b.rot_pad;
    pp.q_lat = b.q_lat;
    b2_prof_mark(ctx, B2_CLS_ROPE_KV);
    B2_CHECK(b2_latent_prep_launch(ctx, m->f32, a, pp));

    // Portions of more than a token: keys and values of their contexts expanded per head.  Otherwise (single tokens, f32,
    // head sizes or contexts outside that kernel's reach) attention in latent coordinates.
    const LayeredStep::Gather& ga = s.gather[P.gather];
    const bool expand = s.pf_work > 0 && P.kv_up.w && (size_t)ga.rows * P.kv_up.N * 2 <= kMaxExpandBytes;
    if (expand) {
        B2_CHECK(ensure_expand(m, ga.rows));
        LatentGatherParams gp{};
        gp.cache = cache;
        gp.block_tables = pool->block_tables;
        gp.max_blocks = pool->max_blocks;
        gp.page_size = pool->block_size;
        gp.B = s.B;
        gp.rows = ga.rows;
        gp.seq_slot = s.in->seq_slot;
        gp.context_lens = s.mo->context_lens;
        gp.kv_off = ga.kv_off;
        gp.cu_seqlens = s.mo->cu_seqlens;
        gp.lat = lm.kv_lat;
        gp.ld_lat = P.kv_up.K;
        gp.rot = lm.kv_rot;
        gp.rot_pad = b.rot_pad;
        B2_CHECK(b2_latent_gather_launch(ctx, a, gp));
        B2_CHECK(linear(m, P.kv_up, lm.kv_lat, P.kv_up.K, ga.rows, lm.kv_cap, lm.kv_exp, P.kv_up.N, false));
        LatentPrefillParams fp{};
        fp.q = b.q;
        fp.q_rows = lm.t_cap;
        fp.kv = lm.kv_exp;
        fp.rot = lm.kv_rot;
        fp.kv_rows = lm.kv_cap;
        fp.ld_kv = P.kv_up.N;
        fp.v_col0 = a.heads * b.plain_pad;
        fp.plain_blocks = b.plain_pad / 64;
        fp.pf_seq = s.mo->pf_seq;
        fp.pf_qstart = s.mo->pf_qstart;
        fp.n_work = s.mo->counts + 3;
        fp.cu_seqlens = s.mo->cu_seqlens;
        fp.context_lens = s.mo->context_lens;
        fp.kv_off = ga.kv_off;
        fp.scale_log2 = scale_log2;
        fp.out = b.att;
        fp.ldo = b.ld_att;
        fp.vdim = a.vdim;
        b2_prof_mark(ctx, B2_CLS_ATTN_PREFILL);
        B2_CHECK(b2_latent_prefill_launch(ctx, a, fp, s.pf_work));
        ctx->attn_prefill_flops += 2.0 * (a.dim + a.rot_dim + a.vdim) * a.heads * masked_pairs(s, a.mask);
    }
    // rows that attend in latent coordinates: the single tokens, or every token
    const int rows = expand ? s.n_dec : T;
    const bool listed = rows == s.n_dec;  // the packer's decode list describes them
    const int32_t* row_idx = rows < T ? s.mo->dec_qrow : nullptr;
    if (rows > 0) {
        GroupedGemmParams g{};
        g.x = b.q;
        g.x_gstride = q_row;
        g.ldx = a.heads * q_row;
        g.row_idx = row_idx;
        g.map_out = row_idx != nullptr;
        g.w = P.k_up_t.w;
        g.N = P.k_up_t.N;
        g.K = P.k_up_t.K;
        g.G = a.heads;
        g.out = b.q_lat;
        g.out_gstride = W;
        g.ldo = a.heads * W;
        g.n_out = a.kv_rank;
        g.M = rows;
        g.x_rows = lm.t_cap;
        b2_prof_mark(ctx, B2_CLS_GEMM);
        B2_CHECK(b2_grouped_gemm_launch(ctx, m->f32, g));
        if (!m->f32 && b2_latent_decode_eligible(a)) {
            LatentDecodeParams dp{};
            dp.q_lat = b.q_lat;
            dp.cache = cache;
            dp.block_tables = pool->block_tables;
            dp.max_blocks = pool->max_blocks;
            dp.page_size = pool->block_size;
            dp.cache_rows = pool->max_pages * pool->block_size;
            int items = rows;
            if (listed) {
                dp.ctx = s.mo->dec_ctx;
                dp.qrow = s.mo->dec_qrow;
                dp.slot = s.mo->dec_slot;
                dp.work_seq = s.mo->dec_work_seq;
                dp.work_chunk = s.mo->dec_work_chunk;
                dp.work_off = s.mo->dec_work_off;
                dp.n_work = s.mo->counts + 2;
                dp.chunk_tiles = s.chunk_tiles;
                items = s.dec_work;
                if (a.mask.kind != MaskSpec::None) {  // not the packer's items: the same number for every row
                    const DecodeSplit d = latent_split(m->ctx, latent_head_groups(a), a.mask, *s.seqs);
                    dp.chunk_tiles = d.chunk_tiles;
                    dp.row_chunks = d.row_chunks;
                    items = rows * d.row_chunks;
                }
                B2_CHECK(ensure_decode(m, items));
                dp.part_o = lm.dec_part;
                dp.part_ml = lm.dec_part + (size_t)items * a.heads * a.kv_rank;
                ctx->attn_decode_bytes += (double)decode_keys(*s.seqs, a.mask).sum * W * 2;
            } else {  // one work item per token: nothing is split, no partial results
                dp.positions = s.mo->positions;
                dp.token_seq = s.mo->token_seq;
                dp.seq_slot = s.in->seq_slot;
                dp.chunk_tiles = up(s.max_ctx, b2_latent_decode_tile()) / 16;
            }
            dp.scale_log2 = scale_log2;
            dp.o_lat = b.o_lat;
            dp.o_pad = b.o_pad;
            b2_prof_mark(ctx, B2_CLS_ATTN_DECODE);
            B2_CHECK(b2_latent_decode_launch(ctx, a, dp, items, rows));
        } else {
            LatentAttnParams ap{};
            ap.q_lat = b.q_lat;
            ap.cache = cache;
            ap.block_tables = pool->block_tables;
            ap.max_blocks = pool->max_blocks;
            ap.page_size = pool->block_size;
            ap.seq_slot = s.in->seq_slot;
            ap.token_seq = s.mo->token_seq;
            ap.positions = s.mo->positions;
            ap.row_idx = row_idx;
            ap.o_lat = b.o_lat;
            ap.o_pad = b.o_pad;
            ap.T = rows;
            b2_prof_mark(ctx, B2_CLS_ATTN_DECODE);
            B2_CHECK(b2_latent_attn_simple_launch(ctx, m->f32, a, ap));
        }
        GroupedGemmParams v{};
        v.x = b.o_lat;
        v.x_gstride = b.o_pad;
        v.ldx = a.heads * b.o_pad;
        v.row_idx = row_idx;
        v.map_out = row_idx != nullptr;
        v.w = P.v_up.w;
        v.N = P.v_up.N;
        v.K = P.v_up.K;
        v.G = a.heads;
        v.out = b.att;
        v.out_gstride = a.vdim;
        v.ldo = b.ld_att;
        v.n_out = a.vdim;
        v.M = rows;
        v.x_rows = lm.t_cap;
        b2_prof_mark(ctx, B2_CLS_GEMM);
        B2_CHECK(b2_grouped_gemm_launch(ctx, m->f32, v));
    }
    B2_CHECK(b2_zero_cols_launch(ctx, m->f32, b.att, b.ld_att, a.heads * a.vdim, b.ld_att, T));
    return linear(m, P.attn_o, b.att, b.ld_att, T, lm.t_cap, c.y, c.ldx, true);
}

int32_t Fwd::ssm(const LayerSpec& L, const LayerP& P, int run) {
    const SsmBufs b = carve_ssm(scratch, L.ssm, P, es, (size_t)lm.t_cap, &end);
    B2_CHECK(linear(m, P.ssm_in, c.xn, c.ldn, s.T, lm.t_cap, b.zx, P.ssm_in.N, false));
    SsmParams p{};
    p.zx = b.zx;
    p.ld = P.ssm_in.N;
    p.T = s.T;
    p.B = s.B;
    p.cu_seqlens = s.mo->cu_seqlens;
    p.context_lens = s.mo->context_lens;
    p.token_seq = s.mo->token_seq;
    p.seq_slot = s.in->seq_slot;
    p.state = pool->state + lm.run_state[run];
    p.slot_stride = pool->state_floats;
    p.conv_w = P.conv_w;
    p.conv_b = P.conv_b;
    p.dt_bias = P.dt_bias;
    p.A_log = P.A_log;
    p.D = P.D;
    p.norm = P.ssm_norm;
    p.eps = lm.spec.eps;
    p.xbc = b.xbc;
    p.ld_xbc = b.ld_xbc;
    p.y = b.y;
    p.out = b.gn;
    p.ldo = b.ld_gn;
    b2_prof_mark(m->ctx, B2_CLS_RECURRENT);
    B2_CHECK(b2_ssm_launch(m->ctx, m->f32, L.ssm, p));
    return linear(m, P.ssm_o, b.gn, b.ld_gn, s.T, lm.t_cap, c.y, c.ldx, true);
}

int32_t Fwd::attend(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run) {
    b2_ctx* ctx = m->ctx;
    const GroupedAttnSpec& a = L.gqa;
    int kv_run = run;  // whose cache: this run's, or that of the last run of another layer
    while (L.kv_from >= 0 && lm.runs[kv_run].layer != L.kv_from) kv_run--;
    const KvPlane* planes = &pool->planes[pool->layer_plane[kv_run]];
    GqaPrepParams pp{};
    pp.in = b.in;
    pp.ld = P.in.N;
    pp.q_off = P.at.q;
    pp.k_off = P.at.k;
    pp.v_off = P.at.v;
    pp.T = s.T;
    pp.q_bias = P.q_bias;
    pp.k_bias = P.k_bias;
    pp.v_bias = P.v_bias;
    pp.q_norm = P.q_norm;
    pp.k_norm = P.k_norm;
    pp.own_kv = L.kv_from < 0;
    pp.eps = lm.spec.eps;
    pp.positions = s.mo->positions;
    pp.slot_mapping = s.mo->slot_mapping;
    pp.cos_t = lm.ropes[P.rope].cos;
    pp.sin_t = lm.ropes[P.rope].sin;
    pp.q = b.q;
    pp.k_cache = planes[0].base;
    pp.v_cache = planes[1].base;
    pp.page_size = pool->block_size;
    b2_prof_mark(ctx, B2_CLS_ROPE_KV);
    B2_CHECK(b2_gqa_prep_launch(ctx, m->f32, a, pp));
    GqaAttnParams p{};
    p.q = b.q;
    p.k_cache = pp.k_cache;
    p.v_cache = pp.v_cache;
    p.block_tables = pool->block_tables;
    p.max_blocks = pool->max_blocks;
    p.page_size = pool->block_size;
    p.max_pages = pool->max_pages;
    p.T = s.T;
    p.positions = s.mo->positions;
    p.token_seq = s.mo->token_seq;
    p.seq_slot = s.in->seq_slot;
    p.dec_ctx = s.mo->dec_ctx;
    p.dec_qrow = s.mo->dec_qrow;
    p.dec_slot = s.mo->dec_slot;
    p.work_seq = s.mo->dec_work_seq;
    p.work_chunk = s.mo->dec_work_chunk;
    p.work_off = s.mo->dec_work_off;
    p.n_dec_work = s.mo->counts + 2;
    p.chunk_tiles = s.chunk_tiles;
    p.pf_seq = s.mo->pf_seq;
    p.pf_qstart = s.mo->pf_qstart;
    p.n_pf_work = s.mo->counts + 3;
    p.cu_seqlens = s.mo->cu_seqlens;
    p.context_lens = s.mo->context_lens;
    p.q_rows = lm.t_cap;
    p.out_scale = L.gqa_scale;
    p.lambda = P.lambda;
    p.eps = lm.spec.eps;
    p.gate = (const uint8_t*)b.in + P.at.head_gate * es;
    p.ld_gate = P.in.N;
    p.out = b.row;
    p.ldo = P.out.K;
    // f32, and head sizes outside the kernels' reach: the plain form.  Otherwise portions of more than a token on their own
    // kernel where it takes them, everything else one row per token.
    const bool rows = !m->f32 && b2_gqa_decode_eligible(a), tiles = rows && b2_gqa_prefill_eligible(a);
    if (!rows || (s.pf_work > 0 && !tiles)) {
        b2_prof_mark(ctx, s.pf_work > 0 ? B2_CLS_ATTN_PREFILL : B2_CLS_ATTN_DECODE);
        return rows ? b2_gqa_decode_launch(ctx, a, p, 0) : b2_gqa_simple_launch(ctx, m->f32, a, p);
    }
    if (s.n_dec > 0) {
        const DecodeKeys keys = decode_keys(*s.seqs, a.mask);
        int items = s.dec_work;
        if (a.mask.kind != MaskSpec::None) {  // not the packer's items: the same number for every row
            p.chunk_tiles = b2_small_cta_chunk_tiles(keys.sum, b2_gqa_head_blocks(a), ctx->sm_count);
            p.row_chunks = (keys.tiles + p.chunk_tiles - 1) / p.chunk_tiles;
            items = s.n_dec * p.row_chunks;
        }
        B2_CHECK(ensure_decode(m, items));
        p.part_o = lm.dec_part;
        p.part_ml = lm.dec_part + (size_t)items * a.q_heads() * a.v_row();
        B2_CHECK(b2_decode_attn_counters(ctx, s.n_dec, b2_gqa_head_blocks(a), &p.counters));
        b2_prof_mark(ctx, B2_CLS_ATTN_DECODE);
        B2_CHECK(b2_gqa_decode_launch(ctx, a, p, items));
        ctx->attn_decode_bytes += (double)keys.sum * a.kv_heads * (a.dim * a.maps + a.vdim) * 2;
    }
    if (s.pf_work > 0) {
        b2_prof_mark(ctx, B2_CLS_ATTN_PREFILL);
        B2_CHECK(b2_gqa_prefill_launch(ctx, a, p, s.pf_work));
        ctx->attn_prefill_flops += 2.0 * (a.dim + a.vdim) * a.q_heads() * masked_pairs(s, a.mask);
    }
    return B2_OK;
}

// What a memory behind a token shift reads: five mixtures, r | k | v | gate side by side in b.in, the first factor's result of the
// decay in b.low_f, and in f32 the whole projection in b.lr.
int32_t Fwd::shift(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run) {
    b2_ctx* ctx = m->ctx;
    const MemorySpec& sp = L.mem;
    const int ldm = 5 * c.ldn, Q = sp.q_cols();
    ShiftParams h{};
    h.h = c.xn;
    h.ld_h = c.ldn;
    h.T = s.T;
    h.width = sp.shift;
    h.ldo = c.ldn;
    h.mu = P.mu;
    h.out = b.mix;
    h.cu_seqlens = s.mo->cu_seqlens;
    h.context_lens = s.mo->context_lens;
    h.token_seq = s.mo->token_seq;
    h.seq_slot = s.in->seq_slot;
    h.kept = pool->state + lm.run_state[run] + sp.state_floats();
    h.slot_stride = pool->state_floats;
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    B2_CHECK(b2_token_shift_launch(ctx, m->f32, h));
    GroupedGemmParams g{};
    g.x = b.mix;
    g.x_gstride = c.ldn;
    g.ldx = ldm;
    g.w = P.in.w;
    g.N = P.part_n;
    g.K = P.in.K;
    g.G = 4;
    g.out = b.in;
    g.out_gstride = Q;
    g.ldo = P.in.N;
    g.n_out = Q;
    g.M = s.T;
    g.x_rows = lm.t_cap;
    const void* mix_w = (const uint8_t*)b.mix + (size_t)4 * c.ldn * es;
    if (!m->f32 && s.T <= kFewTokens && P.w1.N <= P.part_n) {  // everything in one launch
        g.stream = true;
        g.G = 5;
        g.tail_n = P.w1.N;
        g.tail_out = b.low_f;
        b2_prof_mark(ctx, B2_CLS_GEMM);
        return b2_grouped_gemm_launch(ctx, false, g);
    }
    if (!m->f32 && s.T > 32 && P.part_n == Q) {  // whole tiles: four plain products
        for (int j = 0; j < 4; j++) {
            Proj part = P.in;
            part.N = P.part_n;
            part.w = (uint8_t*)P.in.w + (size_t)j * P.part_n * P.in.K * es;
            B2_CHECK(linear(m, part, (const uint8_t*)b.mix + (size_t)j * c.ldn * es, ldm, s.T, lm.t_cap, (uint8_t*)b.in + (size_t)j * Q * es, P.in.N, false));
        }
    } else {
        b2_prof_mark(ctx, B2_CLS_GEMM);
        B2_CHECK(b2_grouped_gemm_launch(ctx, m->f32, g));
    }
    B2_CHECK(linear(m, P.w1, mix_w, ldm, s.T, lm.t_cap, b.low_f, P.w1.N, true));
    if (!m->f32) return B2_OK;  // (the rest belongs to the recurrence's preparation)
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    B2_CHECK(b2_tanh_launch(ctx, b.low_f, P.w1.N, s.T, P.rank, (float*)b.low, P.lr.K));
    return linear(m, P.lr, b.low, P.lr.K, s.T, lm.t_cap, b.lr, P.lr.N, true);
}

int32_t Fwd::remember(const LayerSpec& L, const LayerP& P, const BranchBufs& b, int run) {
    const MemorySpec& sp = L.mem;
    MemoryParams p{};
    p.in = b.in;
    p.ld = P.in.N;
    p.c_off = P.at.c;
    p.b_off = P.at.beta;
    if (sp.shift > 0) {
        p.dec = b.lr;
        p.ld_dec = P.lr.N;
        if (!m->f32) {
            p.low = b.low_f;
            p.ld_low = P.w1.N;
            p.rank = P.rank;
            p.low_w = P.lr.w;
            p.low_k = P.lr.K;
        }
        p.bonus = P.bonus;
        p.h = c.xn;
        p.ld_h = c.ldn;
    } else if (sp.low_rank) {
        B2_CHECK(linear(m, P.lr, (const uint8_t*)b.in + P.at.gate * es, P.in.N, s.T, lm.t_cap, b.lr, P.lr.N, false));
        p.dec = b.lr;
        p.ld_dec = P.lr.N;
    } else if (sp.decay == MemDecay::PerHead) {
        p.dec = (const uint8_t*)b.in + P.at.decay * es;
        p.ld_dec = P.in.N;
    }
    p.T = s.T;
    p.B = s.B;
    p.cu_seqlens = s.mo->cu_seqlens;
    p.context_lens = s.mo->context_lens;
    p.token_seq = s.mo->token_seq;
    p.seq_slot = s.in->seq_slot;
    p.positions = s.mo->positions;
    p.state = pool->state + lm.run_state[run];
    p.slot_stride = pool->state_floats;
    p.conv_w = P.conv_w;
    p.dt_bias = P.dt_bias;
    p.A_log = P.A_log;
    p.decay = P.decay;
    p.log_decay = P.log_decay;
    if (P.mem_rope >= 0) {
        p.cos_t = lm.ropes[P.mem_rope].cos;
        p.sin_t = lm.ropes[P.mem_rope].sin;
    }
    p.q = b.mq;
    p.k = b.mk;
    p.v = sp.conv > 0 ? b.v : (const void*)((const uint8_t*)b.in + (P.at.c + 2 * sp.q_cols()) * es);
    p.ld_v = sp.conv > 0 ? b.ld_v : P.in.N;
    p.lg = b.lg;
    p.beta = b.beta;
    p.o = b.o;
    if (!m->f32 && s.n_chunks > 0 && b2_memory_chunk_eligible(sp)) {
        B2_CHECK(ensure_chunks(m, (size_t)s.n_chunks * b2_memory_chunk_bytes(sp)));
        p.n_chunks = s.n_chunks;
        p.chunk_off = s.chunk_off;
        p.chunk = lm.chunks;
    }
    b2_prof_mark(m->ctx, B2_CLS_RECURRENT);
    return b2_memory_launch(m->ctx, m->f32, sp, p);
}

int32_t Fwd::branches(const LayerSpec& L, const LayerP& P, int run) {
    const BranchBufs b = carve_branches(scratch, L, P, es, (size_t)lm.t_cap, &end);
    if (L.has_mem() && L.mem.shift > 0)
        B2_CHECK(shift(L, P, b, run));
    else
        B2_CHECK(linear(m, P.in, c.xn, c.ldn, s.T, lm.t_cap, b.in, P.in.N, false));
    if (L.has_gqa()) B2_CHECK(attend(L, P, b, run));
    if (L.has_mem()) B2_CHECK(remember(L, P, b, run));
    BranchOutParams p{};
    p.out = b.row;
    p.ldo = P.out.K;
    p.T = s.T;
    p.att_cols = L.has_gqa() ? L.gqa.heads * L.gqa.vdim : 0;
    if (L.has_mem()) {
        p.o = b.o;
        p.heads = L.mem.heads;
        p.vdim = L.mem.vdim;
        p.m_off = P.at.m;
        p.gate = L.mem.low_rank ? (const uint8_t*)b.lr + P.at.lr_gate * es : (const uint8_t*)b.in + P.at.gate * es;
        p.ld_gate = L.mem.low_rank ? P.lr.N : P.in.N;
        p.act = L.mem.gate;
        p.norm = P.mem_norm;
        p.norm_heads = L.mem.norm_heads;
        p.eps = lm.spec.eps;
        p.scale = L.mem_scale;
    }
    if (L.parallel && L.mlp == MlpKind::DensePlain) {
        p.up = (const uint8_t*)b.in + P.at.up * es;
        p.ld_up = P.in.N;
        p.ff = L.ff;
        p.f_off = P.at.f;
    }
    if (p.o || p.up || p.att_cols < p.ldo) {
        b2_prof_mark(m->ctx, B2_CLS_ELEMENTWISE);
        B2_CHECK(b2_branch_out_launch(m->ctx, m->f32, p));
    }
    return linear(m, P.out, b.row, P.out.K, s.T, lm.t_cap, c.y, c.ldx, true);
}

int32_t Fwd::average(const LayerSpec& L, const LayerP& P, int run) {
    const AverageBufs b = carve_average(scratch, P, es, (size_t)lm.t_cap, &end);
    B2_CHECK(linear(m, P.in, c.xn, c.ldn, s.T, lm.t_cap, b.in, P.in.N, false));
    GatedAverageParams p{};
    p.in = b.in;
    p.ld = P.in.N;
    p.z_off = P.at.z;
    p.u_off = P.at.u;
    p.g_off = P.at.gate;
    p.width = L.avg.width;
    p.z_bias = P.z_bias;
    p.u_bias = P.u_bias;
    p.T = s.T;
    p.B = s.B;
    p.cu_seqlens = s.mo->cu_seqlens;
    p.context_lens = s.mo->context_lens;
    p.seq_slot = s.in->seq_slot;
    p.state = pool->state + lm.run_state[run];
    p.slot_stride = pool->state_floats;
    p.out = b.row;
    p.ldo = P.out.K;
    for (auto& q : *s.seqs) {
        p.n_short += q.n < kMemoryChunkMin;
        p.n_long += q.n > kMemoryChunk;
    }
    if (s.n_chunks > 0) {
        B2_CHECK(ensure_chunks(m, (size_t)s.n_chunks * b2_gated_average_chunk_floats(p.width) * 4));
        p.n_chunks = s.n_chunks;
        p.chunk_off = s.chunk_off;
        p.chunk = reinterpret_cast<float*>(lm.chunks);
    }
    b2_prof_mark(m->ctx, B2_CLS_RECURRENT);
    B2_CHECK(b2_gated_average_launch(m->ctx, m->f32, p));
    return linear(m, P.out, b.row, P.out.K, s.T, lm.t_cap, c.y, c.ldx, true);
}

int32_t Fwd::mix(const LayerSpec& L, const LayerP& P, int run) {
    switch (L.mixer) {
        case MixerKind::LatentAttention: return latent(L, P, run);
        case MixerKind::Mamba2: return ssm(L, P, run);
        case MixerKind::GatedAverage: return average(L, P, run);
        default: return branches(L, P, run);
    }
}

int32_t Fwd::token_input(const LayerP& P, int layer) {
    const SideBufs b = carve_side(scratch, P, es, (size_t)lm.t_cap, &end);
    const bool few = !m->f32 && s.T <= kFewTokens;
    TokenGateParams p{};
    p.z = b.z;
    p.parts = 1;
    if (few && P.side_split.G > 0) {  // a group per stretch of the columns, summed by the gate
        GroupedGemmParams g{};
        g.x = c.xn;
        g.x_gstride = kSideSplit;
        g.ldx = c.ldn;
        g.w = P.side_split.w;
        g.N = P.side_split.N;
        g.K = P.side_split.K;
        g.G = P.side_split.G;
        g.out = b.z;
        g.out_gstride = (int64_t)s.T * g.N;
        g.ldo = g.n_out = g.N;
        g.out_f32 = g.stream = true;
        g.M = s.T;
        g.x_rows = lm.t_cap;
        b2_prof_mark(m->ctx, B2_CLS_GEMM);
        B2_CHECK(b2_grouped_gemm_launch(m->ctx, false, g));
        p.ldz = g.N;
        p.parts = g.G;
        p.part_stride = g.out_gstride;
    } else {
        B2_CHECK(linear(m, P.side_gate, c.xn, c.ldn, s.T, lm.t_cap, b.z, P.side_gate.N, true));
        p.ldz = P.side_gate.N;
    }
    p.table = lm.side.w;
    p.ld_table = lm.side.K;
    p.col0 = layer * lm.spec.side_dim;
    p.vocab = lm.spec.vocab;
    p.ids = s.ids_dev;
    p.T = s.T;
    p.n = lm.spec.side_dim;
    p.out = b.act;
    p.ldo = P.side_proj.K;
    b2_prof_mark(m->ctx, B2_CLS_ELEMENTWISE);
    B2_CHECK(b2_token_gate_launch(m->ctx, m->f32, p));
    if (few && P.side_proj.K <= kSideSplit) {
        GroupedGemmParams g{};
        g.x = b.act;
        g.ldx = P.side_proj.K;
        g.w = P.side_proj.w;
        g.N = P.side_proj.N;
        g.K = P.side_proj.K;
        g.G = 1;
        g.out = c.y;
        g.ldo = c.ldx;
        g.n_out = P.side_proj.N;
        g.out_f32 = g.stream = true;
        g.M = s.T;
        g.x_rows = lm.t_cap;
        b2_prof_mark(m->ctx, B2_CLS_GEMM);
        return b2_grouped_gemm_launch(m->ctx, false, g);
    }
    return linear(m, P.side_proj, b.act, P.side_proj.K, s.T, lm.t_cap, c.y, c.ldx, true);
}

// Layers whose norms lie behind their sub-layers.  c.xn always holds the stream in storage format; with an average over the depth the
// embedding output and every layer's result stay in c.past.
int32_t Fwd::post_norm_layers(float* capture) {
    b2_ctx* ctx = m->ctx;
    const ModelSpec& spec = lm.spec;
    EmbedPairsParams e{};
    e.table = lm.embed;
    e.ld_table = c.ldn;
    e.T = s.T;
    e.width = spec.width;
    e.vocab = spec.vocab;
    e.ids = s.ids_dev;
    e.scale = spec.embed_scale;
    e.pairs = spec.pairs;
    e.pair_table = lm.pairs.w;
    e.ld_pairs = lm.pairs.K;
    e.cu_seqlens = s.mo->cu_seqlens;
    e.context_lens = s.mo->context_lens;
    e.token_seq = s.mo->token_seq;
    e.seq_slot = s.in->seq_slot;
    e.kept = spec.pairs.buckets > 0 ? pool->state + lm.pair_state : nullptr;
    e.slot_stride = pool->state_floats;
    e.x = spec.depth_average ? c.past : c.x;
    e.ldx = c.ldx;
    e.out = c.xn;
    e.ldo = c.ldn;
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    B2_CHECK(b2_embed_pairs_launch(ctx, m->f32, e));
    PostNormParams p{};
    p.x = e.x;
    p.x_out = c.x;
    p.y = c.y;
    p.eps = spec.eps;
    p.mult = spec.residual_mult;
    p.past = c.past;
    p.past_stride = (int64_t)lm.t_cap * c.ldx;
    p.out = c.xn;
    p.ldx = p.ldy = c.ldx;
    p.ldo = c.ldn;
    p.rows = s.T;
    p.width = spec.width;
    for (size_t i = 0; i < lm.layers.size(); i++) {
        const LayerSpec& L = spec.layers[i];
        const LayerP& P = lm.layers[i];
        auto norm = [&](const float* w, int groups, bool last) {  // last: of the layer
            p.w = w;
            p.groups = groups;
            const bool avg = last && spec.depth_average;
            p.avg = avg ? P.avg : nullptr;
            p.depth = (int)i + 1;
            p.keep = avg && i + 1 < lm.layers.size() ? c.past + (i + 1) * p.past_stride : nullptr;
            b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
            B2_CHECK(b2_post_norm_launch(ctx, m->f32, p));
            p.x = c.x;
            return (int32_t)B2_OK;
        };
        const bool ff = L.mlp == MlpKind::DenseGated, side = spec.side_dim > 0;
        B2_CHECK(mix(L, P, (int)i));
        B2_CHECK(norm(P.norm1, spec.norm_groups, !ff && !side));
        if (ff) {
            B2_CHECK(dense(L, P));
            B2_CHECK(norm(P.norm2, spec.norm_groups, !side));
        }
        if (side) {
            B2_CHECK(token_input(P, (int)i));
            B2_CHECK(norm(P.side_norm, 1, true));
        }
        if (capture)
            B2_CUDA(cudaMemcpy2DAsync(capture + (int64_t)i * s.T * spec.width, (size_t)spec.width * 4, c.x, (size_t)c.ldx * 4, (size_t)spec.width * 4, (size_t)s.T,
                                      cudaMemcpyDeviceToHost, ctx->stream));
    }
    return B2_OK;
}

int32_t Fwd::dense(const LayerSpec& L, const LayerP& P) {
    const DenseBufs b = carve_dense(scratch, P, es, (size_t)lm.t_cap, &end);
    B2_CHECK(linear(m, P.gu, c.xn, c.ldn, s.T, lm.t_cap, b.gu, P.gu.N, false));
    b2_prof_mark(m->ctx, B2_CLS_ELEMENTWISE);
    GateRows g;
    g.gu = b.gu;
    g.ldg = P.gu.N;
    g.up_off = up(L.ff, 64);
    g.rows = s.T;
    g.ff = L.ff;
    g.out = b.act;
    g.ldo = b.ld_act;
    B2_CHECK(b2_gate_launch(m->ctx, m->f32, L.gate, g));
    return linear(m, P.down, b.act, b.ld_act, s.T, lm.t_cap, c.y, c.ldx, true);
}

int32_t Fwd::moe(const LayerSpec& L, const LayerP& P, const int32_t** rows, const float** pass) {
    b2_ctx* ctx = m->ctx;
    const RoutedSpec& r = L.moe;
    const MoeBufs b = carve_moe(scratch, r, P, c.ldn, es, (size_t)lm.t_cap, &end);
    const bool shared = r.shared_ff > 0, both = shared && s.T <= kFewTokens;
    if (both)
        B2_CHECK(linear(m, P.both, c.xn, c.ldn, s.T, lm.t_cap, b.both, P.both.N, true));
    else
        B2_CHECK(linear(m, P.router, c.xn, c.ldn, s.T, lm.t_cap, b.logits, P.router.N, true));
    RouteParams rp{};
    rp.logits = both ? b.both : b.logits;
    rp.ld = both ? P.both.N : P.router.N;
    rp.T = s.T;
    rp.experts = r.experts;
    rp.top = r.top;
    rp.score = r.score;
    rp.identity = r.identity;
    rp.shared = r.shared_ff > 0;
    rp.correction = P.correction;
    rp.scale = r.scale;
    rp.pass = b.pass;
    rp.shared_w = b.shared_w;
    rp.expert = b.expert;
    rp.weight = b.weight;
    rp.offsets = b.offsets;
    rp.pos = b.pos;
    rp.src = b.src;
    rp.row_w = b.row_w;
    rp.counters = lm.route_counters;
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    B2_CHECK(b2_route_launch(ctx, rp));
    GroupedGemmParams g{};
    g.x = c.xn;
    g.ldx = c.ldn;
    g.row_idx = b.src;
    if (!m->f32 && b2_grouped_gemm_wants_rows(ctx, s.T * r.top, true, r.experts, P.e_gu.N)) {
        B2_CHECK(b2_gather_rows_launch(ctx, (const uint16_t*)c.xn, b.src, s.T * r.top, c.ldn, c.ldn, (uint16_t*)b.xs));
        g.x = b.xs;
        g.row_idx = nullptr;
        g.x_rows = lm.t_cap * r.top;
    }
    g.w = P.e_gu.w;
    g.N = P.e_gu.N;
    g.K = P.e_gu.K;
    g.G = r.experts;
    g.out = b.gu;
    g.ldo = g.n_out = P.e_gu.N;
    g.offsets = b.offsets;
    g.M = s.T * r.top;
    b2_prof_mark(ctx, B2_CLS_GEMM);
    B2_CHECK(b2_grouped_gemm_launch(ctx, m->f32, g));
    GateRows ge, gs;
    ge.gu = b.gu;
    ge.ldg = P.e_gu.N;
    ge.up_off = up(r.ff, 64);
    ge.row_w = b.row_w;
    ge.rows = g.M;
    ge.ff = r.ff;
    ge.out = b.act;
    ge.ldo = b.ld_act;
    if (shared) {
        if (!both) B2_CHECK(linear(m, P.s_gu, c.xn, c.ldn, s.T, lm.t_cap, b.s_gu, P.s_gu.N, false));
        gs.gu = both ? (const void*)(b.both + P.router.N) : b.s_gu;
        gs.gu_f32 = both;
        gs.ldg = both ? P.both.N : P.s_gu.N;
        gs.up_off = up(r.shared_ff, 64);
        gs.row_w = b.shared_w;
        gs.rows = s.T;
        gs.ff = r.shared_ff;
        gs.out = b.s_act;
        gs.ldo = P.s_down.K;
    }
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    if (both) {
        B2_CHECK(b2_gate_launch(ctx, m->f32, r.gate, ge, gs));
    } else {
        B2_CHECK(b2_gate_launch(ctx, m->f32, r.gate, ge));
        if (shared) B2_CHECK(b2_gate_launch(ctx, m->f32, r.gate, gs));
    }
    GroupedGemmParams d{};
    d.x = b.act;
    d.ldx = b.ld_act;
    d.w = P.e_down.w;
    d.N = P.e_down.N;
    d.K = P.e_down.K;
    d.G = r.experts;
    d.out = c.y;
    d.ldo = c.ldx;
    d.n_out = lm.spec.width;
    d.out_f32 = true;
    d.offsets = b.offsets;
    d.M = g.M;
    d.x_rows = lm.t_cap * r.top;
    b2_prof_mark(ctx, B2_CLS_GEMM);
    B2_CHECK(b2_grouped_gemm_launch(ctx, m->f32, d));
    // the shared expert's result: the rows of y behind the routed ones
    if (shared) B2_CHECK(linear(m, P.s_down, b.s_act, P.s_down.K, s.T, lm.t_cap, c.y + (size_t)s.T * r.top * c.ldx, c.ldx, true));
    *rows = b.pos;
    if (r.identity > 0) *pass = b.pass;
    return B2_OK;
}

}  // namespace

int b2_layered_q_tile(const b2_model*) { return 128; }
// Work items of the layers without a mask (the packer's list).
int b2_layered_chunk_tiles(const b2_model* m, const std::vector<SeqStep>& seqs) {
    int groups = 1, blocks = 0;
    bool latent = false;
    for (auto& L : m->layered->spec.layers) {
        if (L.mixer == MixerKind::LatentAttention && L.attn.mask.kind == MaskSpec::None) {
            latent = true;
            groups = std::max(groups, latent_head_groups(L.attn));
        }
        if (L.has_gqa()) blocks = std::max(blocks, b2_gqa_head_blocks(L.gqa));
    }
    if (latent) return latent_split(m->ctx, groups, MaskSpec{}, seqs).chunk_tiles;
    return b2_small_cta_chunk_tiles(decode_keys(seqs, MaskSpec{}).sum, std::max(blocks, 1), m->ctx->sm_count);  // several small CTAs per SM
}
const std::vector<MaskSpec>& b2_layered_gathers(const b2_model* m) { return m->layered->gathers; }

void b2_layered_cache_layout(const b2_model* m, int block_size, std::vector<std::vector<size_t>>& page_bytes, int64_t& state_floats) {
    for (const LayerRun& r : m->layered->runs) {
        const LayerSpec& L = m->layered->spec.layers[r.layer];
        page_bytes.emplace_back();
        if (L.has_gqa() && L.kv_from < 0) {
            page_bytes.back().push_back((size_t)block_size * L.gqa.k_heads() * L.gqa.k_row() * esz(m));
            page_bytes.back().push_back((size_t)block_size * L.gqa.kv_heads * L.gqa.v_row() * esz(m));
        }
        if (L.mixer == MixerKind::LatentAttention) page_bytes.back().push_back((size_t)block_size * L.attn.row_pad() * esz(m));
    }
    state_floats = m->layered->state_floats;
}

int32_t b2_layered_ensure_rope(b2_model* m, int positions) {
    LayeredModel& lm = *m->layered;
    if (positions <= lm.rope_positions || lm.ropes.empty()) return B2_OK;
    int n = std::max(4096, lm.rope_positions);
    while (n < positions) n *= 2;
    B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    for (RopeTab& r : lm.ropes) {
        const int half = r.spec.dims / 2;
        std::vector<float> c((size_t)n * half), s((size_t)n * half);
        const RotSpec& t = r.spec;
        const double turned = 2.0 * std::log(t.base), mult = t.factor > 0 ? 0.1 * std::log(t.factor) + 1.0 : 1.0;
        // the pair (not rounded) that makes this many turns within `original` positions
        auto pair_of = [&](double turns) { return t.dims * std::log(t.original / (2.0 * M_PI * turns)) / turned; };
        const double lo = t.factor > 0 ? std::max(std::floor(pair_of(t.fast)), 0.0) : 0.0;
        const double hi = t.factor > 0 ? std::min(std::ceil(pair_of(t.slow)), t.dims - 1.0) : 0.0;
        for (int i = 0; i < half; i++) {
            double f = std::pow(t.base, -2.0 * i / t.dims);
            if (t.factor > 0) {
                const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
                f = f / t.factor * ramp + f * (1.0 - ramp);
            }
            for (int p = 0; p < n; p++) {  // rounded once, to f32
                c[(size_t)p * half + i] = (float)(std::cos(p * f) * mult);
                s[(size_t)p * half + i] = (float)(std::sin(p * f) * mult);
            }
        }
        if (r.cos) cudaFree(r.cos);
        if (r.sin) cudaFree(r.sin);
        B2_CUDA(cudaMalloc((void**)&r.cos, std::max<size_t>(c.size(), 1) * 4));
        B2_CUDA(cudaMalloc((void**)&r.sin, std::max<size_t>(s.size(), 1) * 4));
        B2_CUDA(cudaMemcpyAsync(r.cos, c.data(), c.size() * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        B2_CUDA(cudaMemcpyAsync(r.sin, s.data(), s.size() * 4, cudaMemcpyHostToDevice, m->ctx->stream));
        B2_CUDA(cudaStreamSynchronize(m->ctx->stream));
    }
    lm.rope_positions = n;
    return B2_OK;
}

int32_t b2_model_build_layered(b2_ctx* ctx, const ModelSpec& spec, const b2_weights* w, const std::string& prefix, uint64_t seed, bool f32,
                               b2_model** out) {
    B2_CUDA(cudaSetDevice(ctx->device));
    b2_model* m = new b2_model();
    m->ctx = ctx;
    m->f32 = f32;
    m->layered = new LayeredModel();
    LayeredModel& lm = *m->layered;
    lm.spec = spec;
    lm.layers.resize(spec.layers.size());
    lm.runs = spec.runs();
    for (auto& L : spec.layers) {
        const RoutedSpec& r = L.moe;
        B2_REQUIRE(spec.streams > 0 || L.mlp != MlpKind::Routed || (r.identity == 0 && r.score == RouteScore::Sigmoid), B2_ERR_UNSUPPORTED,
                   "identity experts are available for models with several streams");
    }
    B2_REQUIRE(spec.streams <= kMaxStreams && (spec.streams == 0 || spec.loop.times == 0), B2_ERR_UNSUPPORTED,
               "residual streams: up to 16, without repeated layers");
    bool plain = spec.streams == 0 && spec.loop.times == 0;
    for (auto& L : spec.layers) plain = plain && !L.parallel && (L.mlp == MlpKind::None || L.mlp == MlpKind::DenseGated);
    B2_REQUIRE(plain || (!spec.post_norm && !spec.depth_average && spec.side_dim == 0 && spec.pairs.buckets == 0), B2_ERR_UNSUPPORTED,
               "norms behind the sub-layers: for sequential layers with dense feed-forwards");
    for (const LayerRun& r : lm.runs) {
        lm.run_state.push_back(lm.state_floats);
        lm.state_floats += record_floats(spec.layers[r.layer]);
    }
    if (spec.pairs.buckets > 0) {
        lm.pair_state = lm.state_floats;
        lm.state_floats += 4;
    }
    m->cfg.num_layers = (int32_t)spec.layers.size();
    m->cfg.hidden_size = spec.width;
    m->cfg.vocab_size = spec.vocab;
    m->cfg.rms_norm_eps = spec.eps;
    m->cfg.tie_word_embeddings = spec.own_head ? 0 : 1;
    m->cfg.compute_f32 = f32 ? 1 : 0;
    m->hkv_l = 1;  // the latent is one key/value head
    Filler f{m, w, prefix, seed};
    auto build = [&]() -> int32_t {
        Proj head;
        B2_CHECK(f.proj(head, spec.vocab, spec.width));
        B2_CHECK(f.rows(head, 0, spec.names.embed, spec.vocab, spec.width));
        lm.embed = lm.head = head.w;
        if (spec.own_head) {
            B2_CHECK(f.proj(head, spec.vocab, spec.width));
            B2_CHECK(f.rows(head, 0, spec.names.head, spec.vocab, spec.width));
            lm.head = head.w;
        }
        if (spec.pairs.buckets > 0) {
            B2_CHECK(f.proj(lm.pairs, spec.pairs.buckets + 1, spec.width));
            B2_CHECK(f.rows(lm.pairs, 0, spec.names.pairs, spec.pairs.buckets + 1, spec.width));
        }
        if (spec.side_dim > 0) {
            const int cols = spec.side_dim * (int)spec.layers.size();
            B2_CHECK(f.proj(lm.side, spec.vocab, cols));
            B2_CHECK(f.rows(lm.side, 0, spec.names.side + ".embed", spec.vocab, cols));
        }
        if (spec.loop.times > 0) B2_CHECK(f.vec(lm.loop_step, spec.names.loop_step, {spec.loop.times, spec.width}, 0.f, 0.1f));
        for (size_t i = 0; i < spec.layers.size(); i++) B2_CHECK(load_layer(f, lm, (int)i));
        B2_CHECK(f.vec(lm.final_norm, spec.names.final_norm, {spec.width}, 1.f, 0.f, false, spec.norm_offset));
        B2_CUDA(cudaMalloc((void**)&lm.route_counters, 1025 * sizeof(int)));
        B2_CUDA(cudaMemsetAsync(lm.route_counters, 0, 1025 * sizeof(int), ctx->stream));
        B2_CUDA(cudaEventCreate(&m->ev0));
        B2_CUDA(cudaEventCreate(&m->ev1));
        B2_CUDA(cudaStreamSynchronize(ctx->stream));
        return B2_OK;
    };
    const int32_t rc = build();
    if (rc != B2_OK) {
        b2_model_free(m);
        return rc;
    }
    *out = m;
    return B2_OK;
}

void b2_layered_release(b2_model* m) {
    if (!m->layered) return;
    LayeredModel& lm = *m->layered;
    for (RopeTab& r : lm.ropes) {
        if (r.cos) cudaFree(r.cos);
        if (r.sin) cudaFree(r.sin);
    }
    if (lm.route_counters) cudaFree(lm.route_counters);
    for (void* p : {(void*)lm.arena, (void*)lm.kv_lat, (void*)lm.kv_rot, (void*)lm.kv_exp, (void*)lm.dec_part, (void*)lm.chunks})
        if (p) cudaFree(p);
    delete m->layered;
    m->layered = nullptr;
}

int32_t b2_forward_layered(b2_model* m, b2_pool* pool, const LayeredStep& s, float** logits_dev, int* logits_ld) {
    b2_ctx* ctx = m->ctx;
    LayeredModel& lm = *m->layered;
    const ModelSpec& spec = lm.spec;
    B2_REQUIRE(pool->model == m, B2_ERR_MSG, "forward: the caches belong to another model's pool");
    B2_REQUIRE(s.T <= 65535, B2_ERR_UNSUPPORTED, "forward: at most 65535 tokens in one step of a layered model");
    B2_CHECK(ensure_arena(m, s.T, s.n_logits));
    Carver carver{lm.arena};
    const Common c = carve_common(carver, lm, esz(m), (size_t)lm.t_cap, (size_t)lm.l_cap);
    Fwd f{m, lm, pool, s, c, carver, esz(m)};
    const int64_t per_layer = (int64_t)s.T * spec.width;
    const bool capture = lm.capture && lm.capture_cap >= per_layer * (int64_t)lm.runs.size();
    b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
    if (!spec.post_norm) B2_CHECK(b2_embed_residual_launch(ctx, m->f32, lm.embed, c.ldn, s.ids_dev, s.T, spec.width, spec.vocab, c.x, c.ldx, std::max(spec.streams, 1)));
    AddNormParams an{};
    an.x = c.x;
    an.y = c.y;
    an.ldx = an.ldy = c.ldx;
    an.width = spec.width;
    an.eps = spec.eps;
    an.n_src = 0;  // nothing is pending behind the embedding
    StreamNormParams sn{};
    sn.x = c.x;
    sn.streams = spec.streams;
    sn.y = c.y;
    sn.h = c.xn;
    sn.ldx = sn.ldy = c.ldx;
    sn.ldh = c.ldn;
    sn.width = spec.width;
    sn.eps = spec.eps;
    // takes up what is pending, then norms (w null: only the addition); `from`: weights of the streams, null for their sum
    auto norm = [&](const float* w, const float* from, int rows, const int32_t* row_idx, void* out, float scale, bool write, float* sum = nullptr) {
        b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
        if (spec.streams > 0) {
            sn.from = from;
            sn.w = w;
            sn.rows = rows;
            sn.row_idx = row_idx;
            sn.out = out;
            sn.ldo = c.ldn;
            sn.out_scale = scale;
            sn.sum = sum;
            sn.write_x = write && sn.mix;
            return b2_stream_norm_launch(ctx, m->f32, sn);
        }
        an.w = w;
        an.rows = rows;
        an.row_idx = row_idx;
        an.out = out;
        an.ldo = c.ldn;
        an.out_scale = scale;
        an.write_x = write && (an.n_src > 0 || an.vec || an.table);
        return b2_add_norm_launch(ctx, m->f32, an);
    };
    auto pending = [&](const LayerP* P, int q, const int32_t* rows, int n, const float* pass = nullptr) {
        an.y_rows = sn.y_rows = rows;
        an.n_src = sn.n_src = n;
        sn.mix = P ? P->hc[q].mix : nullptr;
        sn.to = P ? P->hc[q].to : nullptr;
        sn.pass = pass;
    };
    float* sums = nullptr;  // of the streams
    if (capture && spec.streams > 0) B2_CUDA(cudaMallocAsync((void**)&sums, (size_t)s.T * c.ldx * 4, ctx->stream));
    if (spec.post_norm) B2_CHECK(f.post_norm_layers(capture ? lm.capture : nullptr));
    for (size_t r = 0; r < lm.runs.size() && !spec.post_norm; r++) {
        const LayerRun& run = lm.runs[r];
        const LayerSpec& L = spec.layers[run.layer];
        const LayerP& P = lm.layers[run.layer];
        if (run.opens_pass) {  // what a pass adds to the stream
            an.vec = lm.loop_step + (size_t)run.pass * spec.width;
            if (run.pass > 0) {
                an.table = lm.embed;
                an.ids = s.ids_dev;
                an.ld_table = c.ldn;
                an.vocab = spec.vocab;
            }
        }
        B2_CHECK(norm(P.norm1, P.hc[0].from, s.T, nullptr, c.xn, 1.f, true));
        an.vec = nullptr;
        an.table = nullptr;
        B2_CHECK(f.mix(L, P, (int)r));
        pending(&P, 0, nullptr, 1);
        if (L.mlp != MlpKind::None && !L.parallel) {
            B2_CHECK(norm(P.norm2, P.hc[1].from, s.T, nullptr, c.xn, 1.f, true));
            const int32_t* rows = nullptr;
            const float* pass = nullptr;
            if (L.mlp == MlpKind::DenseGated) {
                B2_CHECK(f.dense(L, P));
                pending(&P, 1, nullptr, 1);
            } else {
                B2_CHECK(f.moe(L, P, &rows, &pass));
                pending(&P, 1, rows, L.moe.sources(), pass);
            }
        }
        if (capture) {
            B2_CHECK(norm(nullptr, nullptr, s.T, nullptr, nullptr, 1.f, true, sums));  // the addition alone
            pending(nullptr, 0, nullptr, 0);
            B2_CUDA(cudaMemcpy2DAsync(lm.capture + (int64_t)r * per_layer, (size_t)spec.width * 4, sums ? sums : c.x, (size_t)c.ldx * 4, (size_t)spec.width * 4, (size_t)s.T,
                                      cudaMemcpyDeviceToHost, ctx->stream));
        }
    }
    if (sums) B2_CUDA(cudaFreeAsync(sums, ctx->stream));
    if (s.n_logits > 0) {
        if (spec.post_norm) {
            PostNormParams p{};
            p.y = c.x;
            p.y_rows = s.logit_rows;
            p.w = lm.final_norm;
            p.groups = spec.norm_groups;
            p.eps = spec.eps;
            p.mult = spec.logit_scale;
            p.out = c.last;
            p.ldx = p.ldy = c.ldx;
            p.ldo = c.ldn;
            p.rows = s.n_logits;
            p.width = spec.width;
            b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
            B2_CHECK(b2_post_norm_launch(ctx, m->f32, p));
        } else {
            B2_CHECK(norm(lm.final_norm, nullptr, s.n_logits, s.logit_rows, c.last, spec.logit_scale, false));
        }
        Proj head;
        head.N = pad_n(spec.vocab);
        head.K = c.ldn;
        head.w = lm.head;
        B2_CHECK(linear(m, head, c.last, c.ldn, s.n_logits, lm.l_cap, c.logits, c.ldl, true));
        b2_prof_mark(ctx, B2_CLS_ELEMENTWISE);
        B2_CHECK(b2_argmax_f32_launch(ctx, c.logits, c.ldl, s.n_logits, spec.vocab, m->ws.argmax));
    }
    B2_CUDA(cudaGetLastError());
    *logits_dev = c.logits;
    *logits_ld = c.ldl;
    return B2_OK;
}

extern "C" {

int64_t b2_model_state_bytes(const b2_model* m) { return m && m->layered ? m->layered->state_floats * 4 : 0; }

int32_t b2_model_capture_residual(b2_model* m, float* out_host, int64_t capacity_floats) {
    B2_REQUIRE(m && m->layered, B2_ERR_UNSUPPORTED, "b2_model_capture_residual: not a layered model");
    m->layered->capture = out_host;
    m->layered->capture_cap = out_host ? capacity_floats : 0;
    return B2_OK;
}

}  // extern "C"
