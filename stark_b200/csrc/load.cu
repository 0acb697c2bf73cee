// stark_b200_load: a converted-model directory (config.json + model.safetensors in the reference's own layout)
// straight into a dense decoder, for callers that are not Python.  The counterpart of the reference's
// `stark_glm_load(path_utf8, path_len, options, &model)` (vendor/glm-exl3-bridge/include/stark_glm.h:85-87) and of
// its artifact loader: config.json as `LanguageModelConfig` (crates/stark-engine/src/config/model/language_model.rs:5-11),
// model.safetensors through the bounded header reader (parameters/safetensors_metadata.rs:117-132, header <= 100 MB),
// per-matrix specs in `__metadata__` under `<name>.spec` (parameters/loader.rs:399-408), fused [q; k; v] and
// [up; gate] rows, planes either [rows, groups] or [groups, round_up4(rows)] (weight_matrix.rs:150-154), and the
// rule that every tensor of the file must be consumed (language_model/mod.rs:125).  config.json decides the family:
// layered decoders go to load_layered.cu.  Anything outside the dense
// decode path this engine implements is refused, never approximated.  Host code only: no kernel lives here.
#include <cmath>
#include <cstring>
#include <memory>
#include <string>
#include <vector>

#include "artifact_reader.cuh"
#include "model.cuh"

namespace sb {

namespace {

bool same(const Json &a, const Json &b) {
    if (a.kind != b.kind) return false;
    switch (a.kind) {
        case Json::Null: return true;
        case Json::Bool: return a.b == b.b;
        case Json::Number: return a.num == b.num;
        case Json::String: return a.str == b.str;
        case Json::Array:
            if (a.items.size() != b.items.size()) return false;
            for (size_t i = 0; i < a.items.size(); ++i)
                if (!same(a.items[i], b.items[i])) return false;
            return true;
        case Json::Object:
            if (a.fields.size() != b.fields.size()) return false;
            for (auto &f : a.fields) {
                const Json *o = b.get(f.first.c_str());
                if (!o || !same(f.second, *o)) return false;
            }
            return true;
    }
    return false;
}

// The norm form the dense path implements: scale only, no offset, no mean subtraction (read_artifact's checks).
bool plain_norm(const Json *n, const Json &reference) {
    return n && same(*n, reference) && is_none(n->get("scale_offset")) && is_false(n->get("subtract_mean")) &&
           is_true(n->get("has_scale")) && is_false(n->get("has_biases"));
}

struct Artifact : TensorFile {
    stark_b200_dense_config cfg{};
    uint32_t max_sequence = 32768;
};

stark_b200_status read_config(const Json &root, Artifact &a) {
    if (!is_str(root.get("type"), "LanguageModelConfig")) return STARK_B200_UNSUPPORTED;
    const Json *dec = root.get("decoder_config");
    const Json *tr = dec ? dec->get("transformer_config") : nullptr;
    const Json *layers = tr ? tr->get("layer_configs") : nullptr;
    const Json *emb = dec ? dec->get("embedding_config") : nullptr;
    if (!layers || layers->kind != Json::Array || layers->items.empty() || !emb) return STARK_B200_UNSUPPORTED;
    const Json &first = layers->items[0];
    const Json *mixer = first.get("mixer_config"), *rope = first.get("rope_config"), *norm = first.get("pre_mixer_norm_config");
    if (!mixer || !rope || !norm) return STARK_B200_UNSUPPORTED;
    if (is_str(emb->get("type"), "TiedEmbeddingConfig")) a.cfg.tied = 1;
    else if (is_str(emb->get("type"), "UntiedEmbeddingConfig")) a.cfg.tied = 0;
    else return STARK_B200_UNSUPPORTED;
    for (const char *key : {"input_scale", "logit_soft_cap", "logit_scale"})
        if (!is_none(emb->get(key))) return STARK_B200_UNSUPPORTED;
    if (!is_none(dec->get("ple_model_config")) || !is_none(dec->get("embedding_norm_config"))) return STARK_B200_UNSUPPORTED;
    for (const Json &lc : layers->items) {
        if (!same(lc, first)) return STARK_B200_UNSUPPORTED;  // layers that differ from one another
        const Json *m = lc.get("mixer_config");
        if (!m || !is_str(m->get("type"), "AttentionConfig") || !is_true(m->get("is_causal")) || !is_none(m->get("scale")))
            return STARK_B200_UNSUPPORTED;
        if (!is_none(m->get("sliding_window_size")) || !is_none(m->get("logit_soft_cap")) || !is_false(m->get("has_sinks")))
            return STARK_B200_UNSUPPORTED;
        for (const char *key : {"has_qkvg_biases", "has_out_biases", "has_gate", "normalize_values", "is_kv_sharing"})
            if (!is_false(m->get(key))) return STARK_B200_UNSUPPORTED;
        const Json *mlp = lc.get("mlp_config");
        const Json *act = mlp ? mlp->get("activation") : nullptr;
        if (!mlp || !is_str(mlp->get("type"), "DenseMLPConfig") || !act || !is_str(act->get("type"), "SiLU"))
            return STARK_B200_UNSUPPORTED;
        const Json *rc = lc.get("rope_config");
        if (!rc || !is_str(rc->get("type"), "UnscaledRoPEConfig")) return STARK_B200_UNSUPPORTED;
        for (const char *key : {"mixer_conv_config", "post_mixer_norm_config", "mlp_conv_config", "post_mlp_norm_config",
                                "ple_config", "kv_source_layer_index"})
            if (!is_none(lc.get(key))) return STARK_B200_UNSUPPORTED;
        for (const Json *n : {lc.get("pre_mixer_norm_config"), lc.get("pre_mlp_norm_config"), m->get("query_norm_config"),
                              m->get("key_norm_config")})
            if (!plain_norm(n, *norm)) return STARK_B200_UNSUPPORTED;
    }
    const Json *out_norm = tr->get("output_norm_config");
    if (!out_norm || !same(*out_norm, *norm)) return STARK_B200_UNSUPPORTED;
    a.cfg.layers = (uint32_t)layers->items.size();
    const Json *eps = norm->get("epsilon"), *base = rope->get("base");
    if (!as_u32(tr->get("model_dim"), a.cfg.hidden) || !as_u32(mixer->get("num_heads"), a.cfg.q_heads) ||
        !as_u32(mixer->get("num_groups"), a.cfg.kv_heads) || !as_u32(mixer->get("head_dim"), a.cfg.head_dim) ||
        !as_u32(tr->get("hidden_dim"), a.cfg.inter) || !as_u32(dec->get("vocab_size"), a.cfg.vocab) || !eps ||
        eps->kind != Json::Number || !base || base->kind != Json::Number)
        return STARK_B200_INVALID_ARGUMENT;
    a.cfg.eps = (float)eps->num;
    a.cfg.rope_theta = (float)base->num;
    if (a.cfg.head_dim != kHeadDim) return STARK_B200_UNSUPPORTED;
    uint32_t seq = 0;
    if (as_u32(rope->get("max_sequence_length"), seq) && seq) a.max_sequence = seq;
    return STARK_B200_OK;
}

stark_b200_status load_matrix(Artifact &a, stark_b200_model *model, uint32_t layer, uint32_t which, const std::string &name,
                              uint32_t rows, uint32_t columns) {
    auto spec_text = a.metadata.find(name + ".spec");
    Json spec;
    if (spec_text == a.metadata.end() || !parse_json(spec_text->second.data(), spec_text->second.size(), spec))
        return STARK_B200_UNSUPPORTED;
    uint32_t group = 0, bits = 0;
    if (!is_str(spec.get("type"), "MLXSpec") || !as_u32(spec.get("group_size"), group) || group != 64 ||
        !as_u32(spec.get("bits"), bits) || bits != 4)
        return STARK_B200_UNSUPPORTED;  // the decoder's matvec kernels are written for 4-bit group-64 matrices
    const uint32_t groups = columns / 64u;
    stark_b200_affine_desc d{};
    d.struct_size = sizeof(d);
    d.abi_version = STARK_B200_ABI_VERSION;
    d.rows = rows;
    d.columns = columns;
    d.bits = bits;
    d.group = 64;
    d.plane_kind = STARK_B200_PLANE_BF16;
    d.location = STARK_B200_HOST;
    std::vector<uint64_t> plane_shape;
    const Json *layout = spec.get("layout");
    if (is_str(layout, "input_output")) {
        plane_shape = {rows, groups};
    } else if (is_str(layout, "output_input")) {
        d.scale_layout = 1;
        d.plane_pitch = rows + ((4u - rows % 4u) % 4u);
        plane_shape = {groups, d.plane_pitch};
    } else {
        return STARK_B200_UNSUPPORTED;
    }
    const uint8_t *codes = tensor_bytes(a, name + ".weights", "U8", {rows, (uint64_t)columns * bits / 8u}, 1);
    const uint8_t *scales = tensor_bytes(a, name + ".scales", "BF16", plane_shape, 2);
    const uint8_t *biases = tensor_bytes(a, name + ".biases", "BF16", plane_shape, 2);
    if (!codes || !scales || !biases) return STARK_B200_INVALID_ARGUMENT;
    if (!model) return STARK_B200_OK;  // validation pass
    return stark_b200_model_set_affine(model, layer, which, codes, scales, biases, &d);
}

stark_b200_status load_vector(Artifact &a, stark_b200_model *model, uint32_t layer, uint32_t which, const std::string &name,
                              uint32_t width) {
    const uint8_t *data = tensor_bytes(a, name + ".scales", "F32", {width}, 4);
    if (!data) return STARK_B200_INVALID_ARGUMENT;
    if (!model) return STARK_B200_OK;  // validation pass
    return stark_b200_model_set_vector(model, layer, which, reinterpret_cast<const float *>(data), width);
}

}  // namespace

}  // namespace sb

using namespace sb;

extern "C" stark_b200_status stark_b200_load(const uint8_t *path_utf8, size_t path_len, const stark_b200_load_options *options,
                                             stark_b200_model **out_model) {
    if (!path_utf8 || !path_len || !options || !out_model) return STARK_B200_INVALID_ARGUMENT;
    if (options->struct_size != sizeof(stark_b200_load_options) || options->abi_version != STARK_B200_ABI_VERSION)
        return STARK_B200_ABI_MISMATCH;
    *out_model = nullptr;
    const std::string dir(reinterpret_cast<const char *>(path_utf8), path_len);
    std::string text;
    if (!read_file(dir + "/config.json", text, 64u << 20)) return STARK_B200_IO_FAILURE;
    Json root;
    if (!parse_json(text.data(), text.size(), root)) return STARK_B200_INVALID_ARGUMENT;
    if (layered_claims(root)) return load_layered(dir, root, options->context_tokens, out_model);
    auto artifact = std::make_unique<Artifact>();
    Artifact &a = *artifact;
    stark_b200_status st = read_config(root, a);
    if (st != STARK_B200_OK) return st;
    if ((st = read_safetensors(dir + "/model.safetensors", a)) != STARK_B200_OK) return st;
    uint64_t context = options->context_tokens ? options->context_tokens : a.max_sequence;
    if (context > a.max_sequence) return STARK_B200_CONTEXT_LIMIT;
    a.cfg.struct_size = sizeof(a.cfg);
    a.cfg.abi_version = STARK_B200_ABI_VERSION;
    a.cfg.context_tokens = (uint32_t)context;
    const auto &c = a.cfg;
    const uint32_t qw = c.q_heads * c.head_dim, kw = c.kv_heads * c.head_dim;
    // Every tensor the decoder reads, in one place: walked once without a model (names, specs, types, shapes and
    // offsets are checked and the all-consumed rule applied before any device memory is touched), then again to
    // upload.
    auto walk = [&](stark_b200_model *model) -> stark_b200_status {
        stark_b200_status s;
        if (c.tied) {
            if ((s = load_matrix(a, model, 0, STARK_B200_MAT_EMBED, "decoder.embedding.embedding", c.vocab, c.hidden)) != STARK_B200_OK) return s;
        } else {
            if ((s = load_matrix(a, model, 0, STARK_B200_MAT_EMBED, "decoder.embedding.input_embedding", c.vocab, c.hidden)) != STARK_B200_OK) return s;
            if ((s = load_matrix(a, model, 0, STARK_B200_MAT_LM_HEAD, "decoder.embedding.output_embedding", c.vocab, c.hidden)) != STARK_B200_OK) return s;
        }
        for (uint32_t i = 0; i < c.layers; ++i) {
            const std::string p = "decoder.transformer.layers." + std::to_string(i);
            if ((s = load_vector(a, model, i, STARK_B200_VEC_ATTN_NORM, p + ".pre_mixer_norm", c.hidden)) != STARK_B200_OK) return s;
            if ((s = load_vector(a, model, i, STARK_B200_VEC_MLP_NORM, p + ".pre_mlp_norm", c.hidden)) != STARK_B200_OK) return s;
            if ((s = load_vector(a, model, i, STARK_B200_VEC_Q_NORM, p + ".mixer.query_norm", c.head_dim)) != STARK_B200_OK) return s;
            if ((s = load_vector(a, model, i, STARK_B200_VEC_K_NORM, p + ".mixer.key_norm", c.head_dim)) != STARK_B200_OK) return s;
            if ((s = load_matrix(a, model, i, STARK_B200_MAT_QKV, p + ".mixer.qkvg_projection.weights", qw + 2u * kw, c.hidden)) != STARK_B200_OK) return s;
            if ((s = load_matrix(a, model, i, STARK_B200_MAT_O, p + ".mixer.out_projection.weights", c.hidden, qw)) != STARK_B200_OK) return s;
            if ((s = load_matrix(a, model, i, STARK_B200_MAT_UPGATE, p + ".mlp.up_projection.weights", 2u * c.inter, c.hidden)) != STARK_B200_OK) return s;
            if ((s = load_matrix(a, model, i, STARK_B200_MAT_DOWN, p + ".mlp.down_projection.weights", c.hidden, c.inter)) != STARK_B200_OK) return s;
        }
        return load_vector(a, model, 0, STARK_B200_VEC_FINAL_NORM, "decoder.transformer.output_norm", c.hidden);
    };
    if ((st = walk(nullptr)) != STARK_B200_OK) return st;
    if (a.used.size() != a.tensors.size()) return STARK_B200_INVALID_ARGUMENT;  // every tensor must be consumed
    stark_b200_model *model = nullptr;
    if ((st = stark_b200_model_create(&a.cfg, &model)) != STARK_B200_OK) return st;
    auto fail = [&](stark_b200_status s) {
        stark_b200_destroy(&model);
        return s;
    };
    if ((st = walk(model)) != STARK_B200_OK) return fail(st);
    if ((st = stark_b200_model_finalize(model)) != STARK_B200_OK) return fail(st);
    *out_model = model;
    return STARK_B200_OK;
}
