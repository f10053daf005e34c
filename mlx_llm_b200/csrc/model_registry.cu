// Model families: which one a config.json names, and how a model of it is built.
//
// The Llama / Qwen3 families (src/config.rs:64-113 decides by `architectures` / `model_type`) are flat configurations
// (b2_model_config); a layered family names itself in `architecture` and lists its layers, each with a mixer and a
// feed-forward, which become a ModelSpec.  A new layered design whose mechanisms exist already is one more reader here.
#include <cstring>
#include <fstream>
#include <sstream>

#include "engine.h"
#include "json_mini.h"

namespace {

using b2json::Value;

struct Reader {  // typed access to one JSON object; remembers the first thing that was missing or malformed
    std::string err;
    const Value* obj(const Value* v, const char* key, const std::string& where) {
        const Value* f = v ? v->get(key) : nullptr;
        if (!f || f->kind != Value::Object) return fail("object", key, where), nullptr;
        return f;
    }
    int num(const Value* v, const char* key, const std::string& where, int lo = 1) {
        long long x = 0;
        const Value* f = v ? v->get(key) : nullptr;
        if (!f || !f->as_i64(x)) return fail("integer", key, where), 0;
        if (x < lo || x > (1 << 30)) return fail("in-range integer", key, where), 0;
        return (int)x;
    }
    int64_t factor(const Value* v, const char* key, const std::string& where) {  // of a token id: their product fits 64 bits
        long long x = 0;
        const Value* f = v ? v->get(key) : nullptr;
        if (!f || !f->as_i64(x)) return fail("integer", key, where), 0;
        if (x < 0 || x > (1ll << 32)) return fail("in-range integer", key, where), 0;
        return x;
    }
    double real(const Value* v, const char* key, const std::string& where) {
        double x = 0;
        const Value* f = v ? v->get(key) : nullptr;
        if (!f || !f->as_f64(x)) fail("number", key, where);
        return x;
    }
    std::string str(const Value* v, const char* key, const std::string& where) {
        const Value* f = v ? v->get(key) : nullptr;
        if (!f || f->kind != Value::String) return fail("string", key, where), std::string();
        return f->str;
    }
    void require(bool ok, const std::string& what) {
        if (!ok && err.empty()) err = "config.json: " + what;
    }
    void fail(const char* type, const char* key, const std::string& where) {
        if (err.empty()) err = std::string("config.json: missing ") + type + " `" + key + "` in " + where;
    }
};

// ---- mixers and feed-forwards by the name a layered config.json gives them ------------------------------------
void read_latent_attention(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    LatentAttnSpec& a = L.attn;
    L.mixer = MixerKind::LatentAttention;
    a.heads = r.num(m, "heads", at);
    a.dim = r.num(m, "dim", at);
    a.rot_dim = r.num(m, "rot_dim", at);
    a.vdim = r.num(m, "vdim", at);
    a.kv_rank = r.num(m, "kv_rank", at);
    a.scale = (float)r.real(m, "scale", at);
    const Value* rot = r.obj(m, "rot", at);
    a.rot.base = r.real(rot, "base", at + ".rot");
    a.rot.dims = r.num(rot, "dims", at + ".rot");
    r.require(a.rot.dims % 2 == 0 && a.rot.dims <= a.rot_dim, at + ": rot.dims must be even and at most rot_dim");
    r.require(a.rot.base > 0, at + ": rot.base must be positive");
}
void read_mamba2(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    Mamba2Spec& s = L.ssm;
    L.mixer = MixerKind::Mamba2;
    s.heads = r.num(m, "heads", at);
    s.vdim = r.num(m, "vdim", at);
    s.state = r.num(m, "state", at);
    s.groups = r.num(m, "groups", at);
    s.norm_groups = r.num(m, "norm_groups", at);
    s.conv = r.num(m, "conv", at);
    if (!r.err.empty()) return;
    r.require(s.heads % s.groups == 0, at + ": groups must divide heads");
    r.require(s.inner() % s.norm_groups == 0, at + ": norm_groups must divide heads * vdim");
}
void read_rot(Reader& r, const Value* m, const std::string& at, int dim, RotSpec& rot) {
    const Value* v = r.obj(m, "rot", at);
    rot.base = r.real(v, "base", at + ".rot");
    rot.dims = r.num(v, "dims", at + ".rot", 0);
    r.require(rot.dims % 2 == 0 && rot.dims <= dim, at + ": rot.dims must be even and at most dim");
    r.require(rot.base > 0, at + ": rot.base must be positive");
}
void read_retention(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    MemorySpec& s = L.mem;
    L.mixer = MixerKind::Memory;
    s.heads = s.kv_heads = r.num(m, "heads", at);
    s.dim = r.num(m, "dim", at);
    s.vdim = r.num(m, "vdim", at);
    read_rot(r, m, at, s.dim, s.rot);
    const Value* d = m ? m->get("decay") : nullptr;
    r.require(d && d->kind == Value::Array && (int)d->arr.size() == s.heads, at + ": `decay` must list one number per head");
    if (!r.err.empty()) return;
    for (auto& v : d->arr) {
        double x = 0;
        r.require(v->as_f64(x) && x > 0 && x <= 1, at + ": a decay must be in (0, 1]");
        L.decay.push_back(x);
    }
}
void read_delta_sizes(Reader& r, const Value* m, const std::string& at, MemorySpec& s) {
    s.heads = r.num(m, "heads", at);
    s.kv_heads = r.num(m, "kv_heads", at);
    s.dim = r.num(m, "dim", at);
    s.vdim = r.num(m, "vdim", at);
    s.conv = r.num(m, "conv", at);
    if (r.err.empty()) r.require(s.heads % s.kv_heads == 0, at + ": kv_heads must divide heads");
    s.unit = s.delta = s.norm = true;
}
void read_delta(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    L.mixer = MixerKind::Memory;
    read_delta_sizes(r, m, at, L.mem);
    L.mem.decay = MemDecay::PerHead;
}
// capped sink attention on the left, a delta memory with a decay per key channel on the right
void read_side_by_side(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    L.mixer = MixerKind::SideBySide;
    L.gqa_key = "left.";
    L.mem_key = "right.";
    GroupedAttnSpec& a = L.gqa;
    const Value* l = r.obj(m, "left", at);
    const std::string la = at + ".left";
    a.heads = r.num(l, "heads", la);
    a.kv_heads = r.num(l, "kv_heads", la);
    a.dim = r.num(l, "dim", la);
    a.vdim = r.num(l, "vdim", la);
    a.scale = (float)r.real(l, "scale", la);
    a.softcap = (float)r.real(l, "softcap", la);
    read_rot(r, l, la, a.dim, a.rot);
    a.sink = a.bias = a.qk_norm = true;
    if (r.err.empty()) r.require(a.heads % a.kv_heads == 0, la + ": kv_heads must divide heads");
    if (r.err.empty()) r.require(a.softcap > 0, la + ": softcap must be positive");
    read_delta_sizes(r, r.obj(m, "right", at), at + ".right", L.mem);
    L.mem.decay = MemDecay::PerChannel;
    L.mem.gate = MemGate::Sigmoid;
    L.mem.low_rank = true;
    L.gqa_scale = (float)r.real(m, "left_scale", at);
    L.mem_scale = (float)r.real(m, "right_scale", at);
}
void read_mask(Reader& r, const Value* m, const std::string& at, MaskSpec::Kind kind, MaskSpec& mask) {
    mask.kind = kind;
    mask.size = r.num(r.obj(m, "mask", at), "size", at + ".mask");
}
// latent attention without a rotated part, over a sliding window
void read_window_latent(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    LatentAttnSpec& a = L.attn;
    L.mixer = MixerKind::LatentAttention;
    a.heads = r.num(m, "heads", at);
    a.dim = r.num(m, "dim", at);
    a.vdim = r.num(m, "vdim", at);
    a.kv_rank = r.num(m, "kv_rank", at);
    a.scale = (float)r.real(m, "scale", at);
    read_mask(r, m, at, MaskSpec::Window, a.mask);
}
// grouped attention inside chunks, queries and keys normed over all heads at once, on its own keys or another layer's
void read_chunk_attention(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    GroupedAttnSpec& a = L.gqa;
    L.mixer = MixerKind::GroupedAttention;
    a.heads = r.num(m, "heads", at);
    a.kv_heads = r.num(m, "kv_heads", at);
    a.dim = r.num(m, "dim", at);
    a.vdim = r.num(m, "vdim", at);
    a.scale = (float)r.real(m, "scale", at);
    a.norm_all = true;
    read_rot(r, m, at, a.dim, a.rot);
    read_mask(r, m, at, MaskSpec::Chunk, a.mask);
    const Value* from = m ? m->get("kv_from") : nullptr;
    if (from && from->kind != Value::Null) L.kv_from = r.num(m, "kv_from", at, 0);
    if (r.err.empty()) r.require(a.heads % a.kv_heads == 0, at + ": kv_heads must divide heads");
}
// Optional sub-object: null when it is missing or null.
const Value* optional(const Value* v, const char* key) {
    const Value* f = v ? v->get(key) : nullptr;
    return f && f->kind != Value::Null ? f : nullptr;
}
// differential attention under a window that keeps the first tokens, gated per head, neighbouring coordinates rotated with scaled
// frequencies, on its own keys or another layer's
void read_differential(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    GroupedAttnSpec& a = L.gqa;
    L.mixer = MixerKind::GroupedAttention;
    a.heads = r.num(m, "heads", at);
    a.kv_heads = r.num(m, "kv_heads", at);
    a.dim = r.num(m, "dim", at);
    a.vdim = r.num(m, "vdim", at);
    a.scale = (float)r.real(m, "scale", at);
    a.diff = (float)r.real(m, "diff", at);
    a.maps = 2;
    a.qk_norm = a.head_gate = a.neighbours = true;
    if (optional(m, "rot")) read_rot(r, m, at, a.dim, a.rot);
    if (const Value* s = optional(optional(m, "rot"), "scaling")) {
        const std::string sa = at + ".rot.scaling";
        a.rot.factor = r.real(s, "factor", sa);
        a.rot.original = r.real(s, "original", sa);
        a.rot.fast = r.real(s, "fast", sa);
        a.rot.slow = r.real(s, "slow", sa);
        if (r.err.empty()) r.require(a.rot.factor > 0 && a.rot.original > 0 && a.rot.fast > 0 && a.rot.slow > 0 && a.rot.base != 1, sa + ": its numbers must be positive");
    }
    if (const Value* mask = optional(m, "mask")) {
        a.mask.kind = MaskSpec::Window;
        a.mask.size = r.num(mask, "size", at + ".mask");
        if (optional(mask, "keep_first")) a.mask.keep = r.num(mask, "keep_first", at + ".mask", 0);
    }
    if (optional(m, "kv_from")) L.kv_from = r.num(m, "kv_from", at, 0);
    if (r.err.empty()) r.require(a.heads % a.kv_heads == 0, at + ": kv_heads must divide heads");
}
void read_min_gru(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    L.mixer = MixerKind::GatedAverage;
    L.avg.width = r.num(m, "width", at);
}
// kv_from names an earlier layer of the list whose keys and values this one can read
void check_shared_keys(Reader& r, const std::string& at, const std::vector<LayerSpec>& before, const LayerSpec& L) {
    if (!r.err.empty() || L.kv_from < 0) return;
    const bool ok = L.kv_from < (int)before.size() && before[L.kv_from].mixer == MixerKind::GroupedAttention && before[L.kv_from].kv_from < 0;
    r.require(ok, at + ": kv_from must name an earlier attention layer with keys and values of its own");
    if (!ok) return;
    const GroupedAttnSpec &a = L.gqa, &b = before[L.kv_from].gqa;
    r.require(a.kv_heads == b.kv_heads && a.dim == b.dim && a.vdim == b.vdim, at + ": kv_from names a layer with other key / value heads");
}
// time mixing: token shift, a decay per key channel, a bonus for the current token
void read_time_mix(Reader& r, const Value* m, const std::string& at, LayerSpec& L) {
    MemorySpec& s = L.mem;
    L.mixer = MixerKind::Memory;
    s.heads = s.kv_heads = r.num(m, "heads", at);
    s.dim = s.vdim = r.num(m, "dim", at);
    s.bonus = s.norm = s.norm_heads = true;
    s.decay = MemDecay::PerChannel;
    s.decay_map = DecayMap::Exp;
}
struct MixerReader {
    const char* name;
    void (*read)(Reader&, const Value*, const std::string&, LayerSpec&);
};
using MixerTable = std::vector<MixerReader>;
void read_mixer(Reader& r, const MixerTable& known, const Value* layer, const std::string& at, LayerSpec& L) {
    const std::string type = r.str(layer, "type", at);
    for (auto& mr : known)
        if (type == mr.name) return mr.read(r, r.obj(layer, "mixer", at), at + ".mixer", L);
    r.require(false, at + ": unknown mixer `" + type + "`");
}

void read_mlp(Reader& r, const Value* mlp, const std::string& at, const GateSpec& dense, float expert_alpha, LayerSpec& L) {
    if (!mlp || mlp->kind == Value::Null) {
        L.mlp = MlpKind::None;
        return;
    }
    const std::string kind = r.str(mlp, "kind", at);
    if (kind == "dense") {
        L.mlp = MlpKind::DenseGated;
        L.ff = r.num(mlp, "ff", at);
        L.gate = dense;
    } else if (kind == "moe") {
        L.mlp = MlpKind::Routed;
        const Value* ro = r.obj(mlp, "router", at);
        L.moe.experts = r.num(ro, "experts", at + ".router");
        L.moe.top = r.num(ro, "top", at + ".router");
        const Value* ex = r.obj(mlp, "expert", at);
        L.moe.ff = r.num(ex, "ff", at + ".expert");
        L.moe.gate.act = GateAct::ClippedSwish;
        L.moe.gate.limit = (float)r.real(ex, "limit", at + ".expert");
        L.moe.gate.alpha = expert_alpha;
        r.require(L.moe.top <= L.moe.experts, at + ": more chosen experts than experts");
    } else {
        r.require(false, at + ": unknown feed-forward kind `" + kind + "`");
    }
}

// ---- Zukitar: latent attention and Mamba-2 layers, dense GELU and clipped-swish routed feed-forwards, tied head -----
constexpr float kZukitarExpertAlpha = 1.702f;
bool names_architecture(const Value& v, const char* name) {
    const Value* a = v.get("architecture");
    return a && a->kind == Value::String && a->str == name;
}
bool claims_zukitar(const Value& v) { return names_architecture(v, "Zukitar"); }
int32_t read_zukitar(const Value& v, ModelSpec& spec) {
    Reader r;
    spec.family = "Zukitar";
    spec.vocab = r.num(&v, "vocab", "the model");
    spec.width = r.num(&v, "width", "the model");
    spec.eps = (float)r.real(r.obj(&v, "norm", "the model"), "eps", "norm");
    spec.logit_scale = (float)r.real(&v, "logit_scale", "the model");
    const Value* ls = v.get("layers");
    r.require(ls && ls->kind == Value::Array && !ls->arr.empty(), "`layers` must be a non-empty list");
    if (r.err.empty())
        for (size_t i = 0; i < ls->arr.size(); i++) {
            const Value* lv = ls->arr[i].get();
            const std::string at = "layers[" + std::to_string(i) + "]";
            LayerSpec L;
            read_mixer(r, {{"latent_attention", read_latent_attention}, {"mamba2", read_mamba2}}, lv, at, L);
            read_mlp(r, lv->get("mlp"), at + ".mlp", GateSpec{GateAct::GeluTanh, 0.f, 0.f}, kZukitarExpertAlpha, L);
            spec.layers.push_back(L);
        }
    B2_REQUIRE(r.err.empty(), B2_ERR_CONFIG, r.err);
    return B2_OK;
}

// ---- Tirezen: retention, delta memories, capped sink attention beside a delta memory; parallel layers with plain GELU
// feed-forwards, norm weights around zero, a repeated stretch of layers, an output projection of its own -----------------
bool claims_tirezen(const Value& v) { return names_architecture(v, "Tirezen"); }
int32_t read_tirezen(const Value& v, ModelSpec& spec) {
    Reader r;
    spec.family = "Tirezen";
    spec.vocab = r.num(&v, "vocab", "the model");
    spec.width = r.num(&v, "width", "the model");
    spec.eps = (float)r.real(r.obj(&v, "norm", "the model"), "eps", "norm");
    spec.norm_offset = 1.f;
    spec.own_head = true;
    const Value* ls = v.get("layers");
    r.require(ls && ls->kind == Value::Array && !ls->arr.empty(), "`layers` must be a non-empty list");
    if (r.err.empty())
        for (size_t i = 0; i < ls->arr.size(); i++) {
            const Value* lv = ls->arr[i].get();
            const std::string at = "layers[" + std::to_string(i) + "]";
            LayerSpec L;
            read_mixer(r, {{"retention", read_retention}, {"delta", read_delta}, {"parallel", read_side_by_side}}, lv, at, L);
            L.parallel = true;
            const Value* mlp = lv->get("mlp");
            if (mlp && mlp->kind != Value::Null) {
                const std::string kind = r.str(mlp, "kind", at + ".mlp");
                r.require(kind == "dense", at + ".mlp: unknown feed-forward kind `" + kind + "`");
                L.mlp = MlpKind::DensePlain;
                L.ff = r.num(mlp, "ff", at + ".mlp");
            }
            spec.layers.push_back(L);
        }
    const Value* loop = v.get("loop");
    if (loop && loop->kind != Value::Null) {
        spec.loop.start = r.num(loop, "start", "loop", 0);
        spec.loop.stop = r.num(loop, "stop", "loop", 0);
        spec.loop.times = r.num(loop, "times", "loop", 1);
        r.require(spec.loop.start < spec.loop.stop && spec.loop.stop <= (int)spec.layers.size(), "loop: start and stop must bound a stretch of the layers");
    }
    B2_REQUIRE(r.err.empty(), B2_ERR_CONFIG, r.err);
    return B2_OK;
}

// ---- Zokuzen: time mixing, windowed latent attention, chunked attention that may read another layer's keys; several residual
// streams; softmax-routed experts with identity experts and a shared one; norm weights around zero, tied head ---------------
bool claims_zokuzen(const Value& v) { return names_architecture(v, "Zokuzen"); }
void read_mixture(Reader& r, const Value* mlp, const std::string& at, LayerSpec& L) {
    const std::string kind = r.str(mlp, "kind", at);
    r.require(kind == "moe", at + ": unknown feed-forward kind `" + kind + "`");
    if (!r.err.empty()) return;
    L.mlp = MlpKind::Routed;
    RoutedSpec& m = L.moe;
    const Value* ro = r.obj(mlp, "router", at);
    const std::string ra = at + ".router";
    m.score = RouteScore::Softmax;
    m.experts = r.num(ro, "experts", ra);
    m.top = r.num(ro, "top", ra);
    if (ro && ro->get("identity")) m.identity = r.num(ro, "identity", ra, 0);
    m.scale = (float)r.real(ro, "scale", ra);
    m.ff = r.num(r.obj(mlp, "expert", at), "ff", at + ".expert");
    m.gate.act = GateAct::Swish;
    m.gate.scale_out = true;
    const Value* sh = mlp->get("shared");
    if (sh && sh->kind != Value::Null) m.shared_ff = r.num(sh, "ff", at + ".shared");
    r.require(m.top <= m.outputs(), at + ": more chosen experts than experts");
}
int32_t read_zokuzen(const Value& v, ModelSpec& spec) {
    Reader r;
    spec.family = "Zokuzen";
    spec.vocab = r.num(&v, "vocab", "the model");
    spec.width = r.num(&v, "width", "the model");
    spec.streams = r.num(&v, "streams", "the model");
    spec.eps = (float)r.real(r.obj(&v, "norm", "the model"), "eps", "norm");
    spec.norm_offset = 1.f;
    const Value* ls = v.get("layers");
    r.require(ls && ls->kind == Value::Array && !ls->arr.empty(), "`layers` must be a non-empty list");
    if (r.err.empty())
        for (size_t i = 0; i < ls->arr.size(); i++) {
            const Value* lv = ls->arr[i].get();
            const std::string at = "layers[" + std::to_string(i) + "]";
            LayerSpec L;
            read_mixer(r, {{"wkv", read_time_mix}, {"latent_attention", read_window_latent}, {"attention", read_chunk_attention}}, lv, at, L);
            if (L.mixer == MixerKind::Memory) L.mem.shift = spec.width;
            const Value* mlp = lv->get("mlp");
            if (mlp && mlp->kind != Value::Null) read_mixture(r, mlp, at + ".mlp", L);
            check_shared_keys(r, at, spec.layers, L);
            spec.layers.push_back(L);
        }
    B2_REQUIRE(r.err.empty(), B2_ERR_CONFIG, r.err);
    return B2_OK;
}

// ---- Pokadra: differential attention, minimal gated recurrences, clipped-swish feed-forwards; norms in groups behind the sub-layers,
// embeddings of token pairs, token inputs per layer, averages over the depth, an output projection of its own --------------
constexpr float kPokadraAlpha = 1.702f;
bool claims_pokadra(const Value& v) { return names_architecture(v, "Pokadra"); }
int32_t read_pokadra(const Value& v, ModelSpec& spec) {
    Reader r;
    spec.family = "Pokadra";
    spec.vocab = r.num(&v, "vocab", "the model");
    spec.width = r.num(&v, "width", "the model");
    const Value* norm = r.obj(&v, "norm", "the model");
    spec.eps = (float)r.real(norm, "eps", "norm");
    spec.norm_groups = r.num(norm, "groups", "norm");
    if (r.err.empty()) r.require(spec.width % spec.norm_groups == 0, "norm: groups must divide the width");
    spec.residual_mult = (float)r.real(&v, "residual_mult", "the model");
    const Value* emb = r.obj(&v, "embedding", "the model");
    spec.embed_scale = (float)r.real(emb, "scale", "embedding");
    if (const Value* p = optional(emb, "bigram")) {
        spec.pairs.buckets = r.num(p, "buckets", "embedding.bigram");
        spec.pairs.mul_prev = r.factor(p, "mul_prev", "embedding.bigram");
        spec.pairs.mul_cur = r.factor(p, "mul_cur", "embedding.bigram");
    }
    if (optional(&v, "token_side")) spec.side_dim = r.num(optional(&v, "token_side"), "dim", "token_side");
    spec.own_head = spec.post_norm = spec.depth_average = true;
    const Value* ls = v.get("layers");
    r.require(ls && ls->kind == Value::Array && !ls->arr.empty(), "`layers` must be a non-empty list");
    if (r.err.empty())
        for (size_t i = 0; i < ls->arr.size(); i++) {
            const Value* lv = ls->arr[i].get();
            const std::string at = "layers[" + std::to_string(i) + "]";
            LayerSpec L;
            read_mixer(r, {{"attention", read_differential}, {"mingru", read_min_gru}}, lv, at, L);
            if (const Value* mlp = optional(lv, "mlp")) {
                const std::string kind = r.str(mlp, "kind", at + ".mlp");
                r.require(kind == "dense", at + ".mlp: unknown feed-forward kind `" + kind + "`");
                L.mlp = MlpKind::DenseGated;
                L.ff = r.num(mlp, "ff", at + ".mlp");
                L.gate = GateSpec{GateAct::ClippedSwish, (float)r.real(mlp, "limit", at + ".mlp"), kPokadraAlpha};
            }
            check_shared_keys(r, at, spec.layers, L);
            spec.layers.push_back(L);
        }
    B2_REQUIRE(r.err.empty(), B2_ERR_CONFIG, r.err);
    return B2_OK;
}

// ---- the table ------------------------------------------------------------------------------------------------
struct ModelFamily {
    const char* name;
    bool (*claims)(const Value& root);
    int32_t (*read_layers)(const Value& root, ModelSpec& spec);  // null: a flat b2_model_config family
};
bool claims_flat(const Value&) { return true; }  // b2_model_config_from_json decides (and refuses what it does not know)
const ModelFamily kFamilies[] = {{"Zukitar", claims_zukitar, read_zukitar}, {"Tirezen", claims_tirezen, read_tirezen}, {"Zokuzen", claims_zokuzen, read_zokuzen},
                                 {"Pokadra", claims_pokadra, read_pokadra},
                                 {"llama", claims_flat, nullptr}};

int32_t find_family(const char* json, b2json::ValuePtr& root, const ModelFamily** out) {
    std::string err;
    root = b2json::parse(json, err);
    B2_REQUIRE(root && root->kind == Value::Object, B2_ERR_CONFIG, "config.json: " + (err.empty() ? std::string("not an object") : err));
    const Value* a = root->get("architecture");
    for (auto& f : kFamilies)
        if (f.claims(*root)) {
            B2_REQUIRE(f.read_layers || !(a && a->kind == Value::String), B2_ERR_UNSUPPORTED,
                       "config.json: unknown architecture `" + (a ? a->str : std::string()) + "`");
            *out = &f;
            return B2_OK;
        }
    return b2_fail(B2_ERR_UNSUPPORTED, "config.json: no model family claims this configuration");
}

int32_t read_spec(const char* json, ModelSpec& spec, bool* layered) {
    b2json::ValuePtr root;
    const ModelFamily* f = nullptr;
    B2_CHECK(find_family(json, root, &f));
    *layered = f->read_layers != nullptr;
    return *layered ? f->read_layers(*root, spec) : B2_OK;
}

}  // namespace

extern "C" {

int32_t b2_model_family_from_json(const char* json, char* out, int32_t cap) {
    B2_REQUIRE(json && out && cap > 0, B2_ERR_MSG, "b2_model_family_from_json: null argument");
    b2json::ValuePtr root;
    const ModelFamily* f = nullptr;
    B2_CHECK(find_family(json, root, &f));
    ModelSpec spec;
    b2_model_config c;
    B2_CHECK(f->read_layers ? f->read_layers(*root, spec) : b2_model_config_from_json(json, &c));  // a malformed one is refused here too
    strncpy(out, f->name, (size_t)cap - 1);
    out[cap - 1] = 0;
    return B2_OK;
}

int32_t b2_model_from_json(b2_ctx* ctx, const b2_weights* w, const char* prefix, const char* json, const b2_quant_spec* quant,
                           int32_t compute_f32, b2_model** out) {
    B2_REQUIRE(ctx && w && json && out, B2_ERR_MSG, "b2_model_from_json: null argument");
    ModelSpec spec;
    bool layered = false;
    B2_CHECK(read_spec(json, spec, &layered));
    if (layered) {
        B2_REQUIRE(!quant, B2_ERR_UNSUPPORTED, spec.family + ": quantize-on-load is available for the flat families only");
        return b2_model_build_layered(ctx, spec, w, prefix ? prefix : "", 0, compute_f32 != 0, out);
    }
    b2_model_config c;
    B2_CHECK(b2_model_config_from_json(json, &c));
    c.compute_f32 = compute_f32 ? 1 : 0;
    return b2_model_from_weights(ctx, w, prefix, &c, quant, out);
}

int32_t b2_model_synthetic_json(b2_ctx* ctx, const char* json, uint64_t seed, b2_model** out) {
    B2_REQUIRE(ctx && json && out, B2_ERR_MSG, "b2_model_synthetic_json: null argument");
    ModelSpec spec;
    bool layered = false;
    B2_CHECK(read_spec(json, spec, &layered));
    if (layered) return b2_model_build_layered(ctx, spec, nullptr, "", seed, false, out);
    b2_model_config c;
    B2_CHECK(b2_model_config_from_json(json, &c));
    return b2_model_synthetic(ctx, &c, seed, out);
}

int32_t b2_model_open(b2_ctx* ctx, const char* dir, const b2_quant_spec* quant, int32_t compute_f32, b2_model** out) {
    B2_REQUIRE(ctx && dir && out, B2_ERR_MSG, "b2_model_open: null argument");
    const std::string path = std::string(dir) + "/config.json";
    std::ifstream f(path);
    B2_REQUIRE(f.good(), B2_ERR_IO, "cannot open " + path);
    std::stringstream ss;
    ss << f.rdbuf();
    b2_weights* w = nullptr;
    B2_CHECK(b2_weights_from_dir(dir, &w));
    const int32_t rc = b2_model_from_json(ctx, w, "", ss.str().c_str(), quant, compute_f32, out);
    b2_weights_free(w);
    return rc;
}

}  // extern "C"
