// stark_b200_load for the layered family: config.json and model.safetensors of a layered decoder walked and checked in
// full, then created, filled and finalized -- the same reading artifact.py does for Python hosts.  Host code only.
#include <algorithm>
#include <cmath>

#include "artifact_reader.cuh"
#include "model.cuh"

namespace sb {

namespace {

constexpr uint64_t kDefaultContext = 8192;  // the configuration sets no limit on positions

bool number(const Json *v, double &out) {
    if (!v || v->kind != Json::Number || !std::isfinite(v->num)) return false;
    out = v->num;
    return true;
}
bool number(const Json *v, float &out) {
    double d;
    if (!number(v, d)) return false;
    out = (float)d;
    return true;
}
bool count(const Json *v, uint32_t &out) { return as_u32(v, out) && out != 0; }
bool count(const Json *v, uint64_t &out) {
    uint32_t n;
    if (!as_u32(v, n)) return false;
    out = n;
    return true;
}

// What an architecture fixes for all of its models.
struct Architecture {
    const char *name;
    uint32_t mixer;
    const char *mixer_type;  // a layer entry's type, or its beginning
    bool any_suffix;
    uint32_t feed_forward, arrangement, flags;
};
const Architecture kArchitectures[] = {
    {"Guvulorn", STARK_B200_MIXER_LATENT, "latent_attention", true, STARK_B200_FF_CLAMPED_GATE, STARK_B200_ARRANGE_POST_NORM,
     STARK_B200_LAYERED_NORM_AROUND_ZERO | STARK_B200_LAYERED_HAS_EMBED_NORM},
    {"Pomelix", STARK_B200_MIXER_GROUPED, "attention", false, STARK_B200_FF_SILU_GATE, STARK_B200_ARRANGE_PARALLEL,
     STARK_B200_LAYERED_TIED_HEAD},
};
const Architecture *architecture_of(const Json &root) {
    for (const Architecture &a : kArchitectures)
        if (is_str(root.get("architecture"), a.name)) return &a;
    return nullptr;
}

bool read_latent(const Json &m, stark_b200_layer_desc &d) {
    const Json *rot = m.get("rot");
    if (!as_u32(m.get("rot_dim"), d.rot_dim) || !count(m.get("kv_rank"), d.kv_rank) || !rot || !number(rot->get("base"), d.rot_base))
        return false;
    d.rot_dims = d.rot_dim;
    if (!is_none(rot->get("dims")) && !as_u32(rot->get("dims"), d.rot_dims)) return false;
    if (const Json *s = rot->get("scaling"); !is_none(s)) {
        d.rot_scaling = STARK_B200_ROT_YARN;
        return number(s->get("factor"), d.rot_factor) && number(s->get("original"), d.rot_original) &&
               number(s->get("fast"), d.rot_fast) && number(s->get("slow"), d.rot_slow);
    }
    return true;
}

bool read_grouped(const Json &m, stark_b200_layer_desc &d) {
    d.q_temp_every = 1;
    if (!count(m.get("kv_heads"), d.kv_heads) || d.heads % d.kv_heads) return false;
    if (!is_none(m.get("conv")) && !as_u32(m.get("conv"), d.conv_taps)) return false;
    if (const Json *t = m.get("q_temp"); !is_none(t))
        if (!number(t->get("coef"), d.q_temp_coef) || !count(t->get("every"), d.q_temp_every)) return false;
    d.v_mix = is_true(m.get("v_mix")) ? 1u : 0u;
    return is_none(m.get("v_mix")) || d.v_mix || is_false(m.get("v_mix"));
}

stark_b200_status read_layer(const Architecture &arch, const Json &entry, stark_b200_layer_desc &d) {
    d.struct_size = sizeof(d);
    d.weights_of = UINT32_MAX;
    const Json *type = entry.get("type"), *m = entry.get("mixer"), *mlp = entry.get("mlp");
    if (!type || type->kind != Json::String || !m) return STARK_B200_INVALID_ARGUMENT;
    if (arch.any_suffix ? type->str.rfind(arch.mixer_type, 0) != 0 : type->str != arch.mixer_type) return STARK_B200_UNSUPPORTED;
    d.mixer = arch.mixer;
    if (!count(m->get("heads"), d.heads) || !count(m->get("dim"), d.dim) || !count(m->get("vdim"), d.vdim) ||
        !number(m->get("scale"), d.scale) || !(arch.mixer == STARK_B200_MIXER_LATENT ? read_latent(*m, d) : read_grouped(*m, d)))
        return STARK_B200_INVALID_ARGUMENT;
    if (!is_none(mlp)) {
        if (!is_str(mlp->get("kind"), "dense")) return STARK_B200_UNSUPPORTED;
        d.feed_forward = arch.feed_forward;
        if (!count(mlp->get("ff"), d.ff_width)) return STARK_B200_INVALID_ARGUMENT;
        if (d.feed_forward == STARK_B200_FF_CLAMPED_GATE && !number(mlp->get("limit"), d.ff_limit)) return STARK_B200_INVALID_ARGUMENT;
    }
    if (!is_none(entry.get("weights_of")) && !as_u32(entry.get("weights_of"), d.weights_of)) return STARK_B200_INVALID_ARGUMENT;
    return STARK_B200_OK;
}

}  // namespace

bool layered_claims(const Json &root) { return architecture_of(root) != nullptr; }

stark_b200_status load_layered(const std::string &dir, const Json &root, uint64_t context_tokens, stark_b200_model **out_model) {
    const Architecture *arch = architecture_of(root);
    if (!arch) return STARK_B200_UNSUPPORTED;
    stark_b200_layered_config c{};
    c.struct_size = sizeof(c);
    c.abi_version = STARK_B200_ABI_VERSION;
    c.compute = STARK_B200_BF16;
    const uint64_t context = context_tokens ? context_tokens : kDefaultContext;
    if (context > (1u << 20)) return STARK_B200_CONTEXT_LIMIT;
    c.context_tokens = (uint32_t)context;
    const Json *emb = root.get("embedding"), *norm = root.get("norm"), *layers = root.get("layers");
    if (!norm || !layers || layers->kind != Json::Array || layers->items.empty() || !count(root.get("vocab"), c.vocab) ||
        !count(root.get("width"), c.width) || !number(norm->get("eps"), c.eps))
        return STARK_B200_INVALID_ARGUMENT;
    c.arrangement = arch->arrangement;
    c.flags = arch->flags;
    c.residual_mult = 1.0f;
    if (c.arrangement == STARK_B200_ARRANGE_PARALLEL && !number(root.get("residual_mult"), c.residual_mult))
        return STARK_B200_INVALID_ARGUMENT;
    c.embed_scale = 1.0f;
    if (!is_none(emb) && !is_none(emb->get("scale")) && !number(emb->get("scale"), c.embed_scale)) return STARK_B200_INVALID_ARGUMENT;
    if (const Json *b = is_none(emb) ? nullptr : emb->get("bigram"); !is_none(b)) {
        if (!count(b->get("buckets"), c.bigram_buckets) || !count(b->get("mul_prev"), c.bigram_mul_prev) ||
            !count(b->get("mul_cur"), c.bigram_mul_cur))
            return STARK_B200_INVALID_ARGUMENT;
    }
    std::vector<stark_b200_layer_desc> descs(layers->items.size());
    c.layers = (uint32_t)descs.size();
    stark_b200_status st;
    for (uint32_t i = 0; i < c.layers; ++i)
        if ((st = read_layer(*arch, layers->items[i], descs[i])) != STARK_B200_OK) return st;
    for (uint32_t i = 0; i < c.layers; ++i)  // a layer that points to one without tensors of its own means that one's source
        for (uint32_t hops = 0; descs[i].weights_of != UINT32_MAX; ++hops) {
            if (descs[i].weights_of >= c.layers || hops > c.layers) return STARK_B200_INVALID_ARGUMENT;
            if (descs[descs[i].weights_of].weights_of == UINT32_MAX) break;
            descs[i].weights_of = descs[descs[i].weights_of].weights_of;
        }
    TensorFile file;
    if ((st = read_safetensors(dir + "/model.safetensors", file)) != STARK_B200_OK) return st;
    // Every tensor the decoder reads, in one place: walked once without a model (all checks), then again to upload.
    auto walk = [&](stark_b200_model *model) -> stark_b200_status {
        auto put = [&](const std::string &name, uint32_t layer, uint32_t which, uint64_t rows, uint64_t columns) -> stark_b200_status {
            // a scalar has no dimensions, a vector one
            std::vector<uint64_t> shape = columns ? std::vector<uint64_t>{rows, columns}
                                                  : (rows ? std::vector<uint64_t>{rows} : std::vector<uint64_t>{});
            const uint8_t *data = tensor_bytes(file, name, "BF16", shape, 2);
            if (!data) return STARK_B200_INVALID_ARGUMENT;
            if (!model) return STARK_B200_OK;
            return stark_b200_layered_set_tensor(model, layer, which, data, columns ? (uint32_t)rows : 1u,
                                                 (uint32_t)(columns ? columns : std::max<uint64_t>(rows, 1u)));
        };
        const uint64_t D = c.width;
        const bool parallel = c.arrangement == STARK_B200_ARRANGE_PARALLEL;
        stark_b200_status s;
#define SB_PUT(...)                                            \
    do {                                                       \
        if ((s = put(__VA_ARGS__)) != STARK_B200_OK) return s; \
    } while (0)
        SB_PUT("embed", 0, STARK_B200_LAYERED_EMBED, c.vocab, D);
        if (c.bigram_buckets) SB_PUT("bigram", 0, STARK_B200_LAYERED_BIGRAM, (uint64_t)c.bigram_buckets + 1u, D);
        if (c.flags & STARK_B200_LAYERED_HAS_EMBED_NORM) SB_PUT("embed.norm", 0, STARK_B200_LAYERED_EMBED_NORM, D, 0);
        SB_PUT("final.norm", 0, STARK_B200_LAYERED_FINAL_NORM, D, 0);
        if (!(c.flags & STARK_B200_LAYERED_TIED_HEAD)) SB_PUT("head", 0, STARK_B200_LAYERED_HEAD, c.vocab, D);
        for (uint32_t i = 0; i < c.layers; ++i) {
            const stark_b200_layer_desc &d = descs[i];
            if (d.weights_of != UINT32_MAX) continue;
            const std::string p = "l" + std::to_string(i), mix = p + ".mix.", mlp = p + ".mlp.";
            const uint64_t H = d.heads, G = d.kv_heads;
            SB_PUT(p + ".norm1", i, STARK_B200_LAYERED_NORM1, D, 0);
            SB_PUT(mix + "q", i, STARK_B200_LAYERED_Q, H * ((uint64_t)d.dim + d.rot_dim), D);
            SB_PUT(mix + "o", i, STARK_B200_LAYERED_O, D, H * d.vdim);
            if (d.mixer == STARK_B200_MIXER_LATENT) {
                SB_PUT(mix + "dkv", i, STARK_B200_LAYERED_DKV, (uint64_t)d.kv_rank + d.rot_dim, D);
                SB_PUT(mix + "dkv.norm", i, STARK_B200_LAYERED_DKV_NORM, d.kv_rank, 0);
                SB_PUT(mix + "uk", i, STARK_B200_LAYERED_UK, H * d.dim, d.kv_rank);
                SB_PUT(mix + "uv", i, STARK_B200_LAYERED_UV, H * d.vdim, d.kv_rank);
            } else {
                SB_PUT(mix + "k", i, STARK_B200_LAYERED_K, G * d.dim, D);
                SB_PUT(mix + "v", i, STARK_B200_LAYERED_V, G * d.vdim, D);
                if (d.conv_taps) {
                    SB_PUT(mix + "q.conv", i, STARK_B200_LAYERED_Q_CONV, H * d.dim, d.conv_taps);
                    SB_PUT(mix + "k.conv", i, STARK_B200_LAYERED_K_CONV, G * d.dim, d.conv_taps);
                    SB_PUT(mix + "v.conv", i, STARK_B200_LAYERED_V_CONV, G * d.vdim, d.conv_taps);
                }
                if (d.v_mix) SB_PUT(mix + "vmix", i, STARK_B200_LAYERED_V_SHARE, 0, 0);
                else file.used.insert(mix + "vmix");  // a share in a layer that does not mix is unused
            }
            if (parallel) SB_PUT(p + ".ls1", i, STARK_B200_LAYERED_SCALE1, D, 0);
            if (d.feed_forward == STARK_B200_FF_NONE) continue;
            if (parallel) SB_PUT(p + ".ls2", i, STARK_B200_LAYERED_SCALE2, D, 0);
            else SB_PUT(p + ".norm2", i, STARK_B200_LAYERED_NORM2, D, 0);
            SB_PUT(mlp + "gate", i, STARK_B200_LAYERED_GATE, d.ff_width, D);
            SB_PUT(mlp + "up", i, STARK_B200_LAYERED_UP, d.ff_width, D);
            SB_PUT(mlp + "down", i, STARK_B200_LAYERED_DOWN, D, d.ff_width);
            if (d.feed_forward != STARK_B200_FF_CLAMPED_GATE) continue;
            SB_PUT(mlp + "gate.b", i, STARK_B200_LAYERED_GATE_BIAS, d.ff_width, 0);
            SB_PUT(mlp + "up.b", i, STARK_B200_LAYERED_UP_BIAS, d.ff_width, 0);
            SB_PUT(mlp + "down.b", i, STARK_B200_LAYERED_DOWN_BIAS, D, 0);
        }
#undef SB_PUT
        return STARK_B200_OK;
    };
    if ((st = walk(nullptr)) != STARK_B200_OK) return st;
    for (const auto &t : file.tensors)
        if (!file.used.count(t.first)) return STARK_B200_INVALID_ARGUMENT;  // every tensor must be consumed
    stark_b200_model *model = nullptr;
    if ((st = stark_b200_layered_create(&c, descs.data(), &model)) != STARK_B200_OK) return st;
    auto fail = [&](stark_b200_status s) {
        stark_b200_destroy(&model);
        return s;
    };
    if ((st = walk(model)) != STARK_B200_OK) return fail(st);
    if ((st = stark_b200_model_finalize(model)) != STARK_B200_OK) return fail(st);
    *out_model = model;
    return STARK_B200_OK;
}

}  // namespace sb
