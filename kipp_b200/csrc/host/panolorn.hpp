// Panolorn: a decoder whose layers are listed one by one in its config.json.  Every layer is attention
// and a feed-forward (dense, a mixture of experts, or none), each with a norm on either side of it
// (sandwich_norm_block): x <- x + norm1b(mixer(norm1(x))), x <- x + norm2b(ff(norm2(x))).
//
//   attention   grouped-query attention with value heads of their own size; q and k divided by their root
//               mean square per head (no weights); no rotation, instead head h of H takes
//               2^(-8 (h + 1) / H) off a capped score per position of distance; blocks of positions as the
//               mask; a sink of score 0 in the softmax's denominator; a sigmoid gate per element of the
//               concatenated heads, read from the mixer's input
//
// Feed-forwards: dense, W_down (gelu(W_gate h) * (W_up h)) with gelu in its tanh form; or experts
// W_down (silu(W_gate h) * (W_up h)) chosen by sigmoid scores, whose weight (the score as it is) multiplies
// the expert's INPUT, with a shared expert that runs for every token.  The embedding is scaled, the
// logits come from the embedding table as it is.
//
// config.json keys: architecture, vocab, width, norm.eps, embedding.scale, layers[i].{type, mixer, mlp}.
// Tensor names: embed, l<i>.{norm1, norm1b, norm2, norm2b}, l<i>.mix.*, l<i>.mlp.*, final.norm.
#pragma once
#include "zunilorn.hpp"

namespace kipp {
namespace panolorn {

using venizen::need;
using venizen::need_int;
using venizen::need_number;
using zasudra::optional_number;
using zunilorn::present;

inline Json feed_forward_sizes(const Json& o, const std::string& where) {
    Json f = Json::object();
    f.set("ff", need_int(o, "ff", where));
    return f;
}

// The keys after checks; every size and constant a model of this design can choose is kept.
inline Json normalize(const Json& c) {
    if (!c.is_object()) fail(KIPP_E_CONFIG, "config.json must hold a JSON object");
    Json out = Json::object();
    out.set("architecture", architecture_of(c));
    out.set("vocab", need_int(c, "vocab", ""));
    out.set("width", need_int(c, "width", ""));
    const double eps = need_number(need(c, "norm", ""), "eps", "norm.");
    if (!(eps > 0)) fail(KIPP_E_CONFIG, "norm.eps must be positive");
    Json norm = Json::object();
    norm.set("eps", eps);
    out.set("norm", std::move(norm));
    Json embedding = Json::object();
    embedding.set("scale", present(c, "embedding") ? optional_number(c.get("embedding"), "scale", "embedding.", 1.0) : 1.0);
    out.set("embedding", std::move(embedding));

    const Json& layers = need(c, "layers", "");
    if (!layers.is_array() || layers.size() == 0) fail(KIPP_E_CONFIG, "config key 'layers' must be a list of layers");
    Json ls = Json::array();
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& l = layers.at(i);
        const std::string where = format("layers[%zu].", i), wm = where + "mixer.";
        const Json& type = need(l, "type", where);
        if (!type.is_string()) fail(KIPP_E_CONFIG, "config key '" + where + "type' must be a string");
        if (type.as_string() != "attention") fail(KIPP_E_CONFIG, "unknown layer type '" + type.as_string() + "' (attention)");
        const Json& mx = need(l, "mixer", where);
        Json layer = Json::object(), mixer = Json::object(), mask = Json::object();
        layer.set("type", type.as_string());
        const long long heads = need_int(mx, "heads", wm);
        const long long kv = present(mx, "kv_heads") ? need_int(mx, "kv_heads", wm) : heads;
        const long long dim = need_int(mx, "dim", wm);
        if (heads % kv) fail(KIPP_E_CONFIG, "config key '" + wm + "heads' must be a multiple of kv_heads");
        mixer.set("heads", heads);
        mixer.set("kv_heads", kv);
        mixer.set("dim", dim);
        mixer.set("vdim", present(mx, "vdim") ? need_int(mx, "vdim", wm) : dim);
        mixer.set("scale", need_number(mx, "scale", wm));
        const double softcap = optional_number(mx, "softcap", wm, 0.0);
        if (softcap < 0) fail(KIPP_E_CONFIG, "config key '" + wm + "softcap' must not be negative");
        mixer.set("softcap", softcap);
        mask.set("size", present(mx, "mask") ? need_int(mx.get("mask"), "size", wm + "mask.") : 0LL);   // 0: every earlier token
        mixer.set("mask", std::move(mask));
        layer.set("mixer", std::move(mixer));
        if (present(l, "mlp")) {
            const Json& mlp = l.get("mlp");
            const std::string wf = where + "mlp.";
            const Json& kind = need(mlp, "kind", wf);
            const std::string fk = kind.is_string() ? kind.as_string() : "";
            Json f = Json::object();
            f.set("kind", fk);
            if (fk == "dense") {
                f.set("ff", need_int(mlp, "ff", wf));
            } else if (fk == "moe") {
                const Json& router = need(mlp, "router", wf);
                const std::string wr = wf + "router.";
                const long long experts = need_int(router, "experts", wr), top = need_int(router, "top", wr);
                if (top > experts) fail(KIPP_E_CONFIG, "config key '" + wr + "top' must not exceed the number of experts");
                Json r = Json::object();
                r.set("experts", experts);
                r.set("top", top);
                f.set("router", std::move(r));
                f.set("expert", feed_forward_sizes(need(mlp, "expert", wf), wf + "expert."));
                if (present(mlp, "shared")) f.set("shared", feed_forward_sizes(mlp.get("shared"), wf + "shared."));
                else f.set("shared", nullptr);
            } else {
                fail(KIPP_E_CONFIG, "config key '" + wf + "kind' must be dense or moe");
            }
            layer.set("mlp", std::move(f));
        } else {
            layer.set("mlp", nullptr);
        }
        ls.push(std::move(layer));
    }
    out.set("layers", std::move(ls));
    return out;
}

// What head h of H takes off a score per position of distance between query and key.
inline Json slopes(long long heads) {
    Json s = Json::array();
    for (long long h = 0; h < heads; ++h) s.push(std::exp2(-8.0 * (double)(h + 1) / (double)heads));
    return s;
}

inline Json gated_part(long long width, long long ff, const char* activation) {
    Json f = Json::object();
    f.set("kind", "gated_mlp");
    f.set("hidden_size", width);
    f.set("intermediate_size", ff);
    f.set("activation", activation);
    f.set("up_add", 0.0);
    return f;
}

inline Json plan(const Json& c) {
    const long long width = c.get("width").as_int(), vocab = c.get("vocab").as_int();
    const double eps = c.get("norm").get("eps").as_double();
    Json p = Json::object();
    p.set("hidden_size", width);
    p.set("vocab_size", vocab);
    p.set("max_positions", 0LL);
    p.set("config", c);
    Json stages = Json::array();
    {
        Json emb = Json::object();
        emb.set("kind", "token_embedding");
        emb.set("vocab_size", vocab);
        emb.set("hidden_size", width);
        emb.set("weight_name", "embed");
        emb.set("scale", c.get("embedding").get("scale").as_double());
        Json stage = Json::object();
        stage.set("prefix", "");
        stage.set("part", std::move(emb));
        stages.push(std::move(stage));
    }
    p.set("embedding", std::move(stages));

    Json blocks = Json::array(), order = Json::array();
    const Json& layers = c.get("layers");
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& l = layers.at(i);
        const Json& mx = l.get("mixer");
        const long long chunk = mx.get("mask").get("size").as_int();
        Json mixer = Json::object(), position = Json::object();
        position.set("kind", "no_position");
        mixer.set("kind", "attention");
        mixer.set("hidden_size", width);
        mixer.set("num_heads", mx.get("heads").as_int());
        mixer.set("num_kv_heads", mx.get("kv_heads").as_int());
        mixer.set("head_dim", mx.get("dim").as_int());
        mixer.set("value_dim", mx.get("vdim").as_int());
        mixer.set("position", std::move(position));
        mixer.set("qk_norm_eps", eps);
        mixer.set("unit_norm", true);
        mixer.set("scale", mx.get("scale").as_double());
        mixer.set("softcap", mx.get("softcap").as_double());
        mixer.set("distance_slopes", slopes(mx.get("heads").as_int()));
        mixer.set("chunk", chunk);
        mixer.set("forget_blocks", chunk > 0);
        mixer.set("sink", "unit");
        mixer.set("element_gate", true);
        mixer.set("names", venizen::names_of({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}, {"gate", "g"}}));
        Json block = Json::object();
        block.set("kind", "sandwich_norm_block");
        Json names = Json::array();
        for (const char* n : {"", "mix.", "", "", "mlp.", ""}) names.push(n);
        block.set("names", std::move(names));
        block.set("input_norm", venizen::rmsnorm_part(width, eps, "norm1"));
        block.set("mixer", std::move(mixer));
        block.set("mixer_out_norm", venizen::rmsnorm_part(width, eps, "norm1b"));
        const Json& f = l.get("mlp");
        if (!f.is_null()) {
            Json ffn;
            if (f.get("kind").as_string() == "dense") {
                ffn = gated_part(width, f.get("ff").as_int(), "gelu_tanh");
            } else {
                ffn = Json::object();
                ffn.set("kind", "expert_mixture");
                ffn.set("hidden_size", width);
                ffn.set("intermediate_size", f.get("expert").get("ff").as_int());
                ffn.set("experts", f.get("router").get("experts").as_int());
                ffn.set("top", f.get("router").get("top").as_int());
                ffn.set("routing", "sigmoid_scores");
                ffn.set("renormalize", false);
                ffn.set("weight_on_input", true);
                ffn.set("gated", true);
                ffn.set("up_add", 0.0);
                if (!f.get("shared").is_null()) {
                    ffn.set("shared", gated_part(width, f.get("shared").get("ff").as_int(), "swish"));
                    ffn.set("shared_prefix", "shared.");
                }
            }
            block.set("post_norm", venizen::rmsnorm_part(width, eps, "norm2"));
            block.set("ffn", std::move(ffn));
            block.set("ffn_out_norm", venizen::rmsnorm_part(width, eps, "norm2b"));
        } else {
            for (const char* key : {"post_norm", "ffn", "ffn_out_norm"}) block.set(key, nullptr);
        }
        Json layer = Json::object();
        layer.set("prefix", format("l%zu.", i));
        layer.set("part", std::move(block));
        blocks.push(std::move(layer));
        Json run = Json::object();
        run.set("layer", (long long)i);
        run.set("cache", (long long)i);
        run.set("writes_cache", true);
        order.push(std::move(run));
    }
    p.set("layers", std::move(blocks));
    p.set("order", std::move(order));

    Json fn = Json::object();
    fn.set("prefix", "");
    fn.set("part", venizen::rmsnorm_part(width, eps, "final.norm"));
    p.set("final_norm", std::move(fn));
    Json head = Json::object();
    head.set("kind", "output_head");
    head.set("vocab_size", vocab);
    head.set("hidden_size", width);
    head.set("tied_to", "embed");
    head.set("weight_name", "head");
    Json hd = Json::object();
    hd.set("prefix", "");
    hd.set("part", std::move(head));
    p.set("head", std::move(hd));
    return p;
}

}  // namespace panolorn

inline void register_panolorn() {
    Registry::get().add_architecture("Panolorn", Architecture{panolorn::normalize, panolorn::plan});
}

}  // namespace kipp
