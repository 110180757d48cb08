// Nogavik: a decoder whose layers are listed one by one in its config.json, each with one of three
// mixers:
//
//   mamba2             the selective state space layer in its matrix-state form (state_space,
//                      recurrent_parts.hpp)
//   latent_attention   attention over a cached latent with a shared part rotated by neighbouring pairs
//                      and a gate per element of the heads (latent_parts.hpp); a layer may read the
//                      latent another one cached (kv_from)
//   parallel           grouped-query attention without positions (biases, then a norm of q and k per
//                      head, value heads of their own size) beside the gated delta rule (gated_delta);
//                      each one's output is normed over the width, and half their sum joins the stream
//
// A layer is x <- x + mixer(norm1(x)) + ff(norm2(x)), both norms of the same x (parallel_block with a
// second norm), then what the layer's own embedding of the token adds (token_side).  The feed-forward is
// dense with the square of relu, or absent.  The norms' weights are stored as their distance from one; the
// norms inside the mixers and the token side have plain weights.  The logits come from the embedding table.
//
// config.json keys: architecture, vocab, width, norm.eps, token_side.dim, layers[i].{type, mixer, mlp}.
// Tensor names: embed, side.embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.{up,down},
// l<i>.side.{gate,proj,norm}, final.norm.
#pragma once
#include "panolorn.hpp"

namespace kipp {
namespace nogavik {

using varunex::optional_int;
using venizen::need;
using venizen::need_int;
using venizen::need_number;
using zunilorn::present;

constexpr double BRANCH_SCALE = 0.5;      // what the sum of the two normed outputs is multiplied by

// heads, kv_heads (absent: as heads), dim, vdim (absent: as dim)
inline Json head_sizes(const Json& mx, const std::string& where) {
    Json m = Json::object();
    const long long heads = need_int(mx, "heads", where), kv = optional_int(mx, "kv_heads", where, heads, 1);
    const long long dim = need_int(mx, "dim", where);
    if (heads % kv) fail(KIPP_E_CONFIG, "config key '" + where + "heads' must be a multiple of kv_heads");
    m.set("heads", heads);
    m.set("kv_heads", kv);
    m.set("dim", dim);
    m.set("vdim", optional_int(mx, "vdim", where, dim, 1));
    return m;
}

inline Json mixer_keys(const Json& mx, const std::string& kind, const std::string& wm, size_t layer) {
    Json m = Json::object();
    if (kind == "mamba2") {
        const long long heads = need_int(mx, "heads", wm), groups = optional_int(mx, "groups", wm, 1, 1);
        const long long vdim = need_int(mx, "vdim", wm), parts = optional_int(mx, "norm_groups", wm, 1, 1);
        if (heads % groups) fail(KIPP_E_CONFIG, "config key '" + wm + "heads' must be a multiple of groups");
        if ((heads * vdim) % parts) fail(KIPP_E_CONFIG, "config key '" + wm + "norm_groups' must divide heads * vdim");
        m.set("heads", heads);
        m.set("groups", groups);
        m.set("vdim", vdim);
        m.set("state", need_int(mx, "state", wm));
        m.set("conv", need_int(mx, "conv", wm));
        m.set("norm_groups", parts);
    } else if (kind == "latent_attention") {
        const long long dim = need_int(mx, "dim", wm), rot_dim = need_int(mx, "rot_dim", wm, 0);
        m.set("heads", need_int(mx, "heads", wm));
        m.set("dim", dim);
        m.set("rot_dim", rot_dim);
        m.set("vdim", optional_int(mx, "vdim", wm, dim, 1));
        m.set("kv_rank", need_int(mx, "kv_rank", wm));
        m.set("q_rank", need_int(mx, "q_rank", wm));
        m.set("scale", need_number(mx, "scale", wm));
        Json rot = venizen::rotation(mx, rot_dim, wm);
        if (rot.get("dims").as_int() != rot_dim)
            fail(KIPP_E_CONFIG, "config key '" + wm + "rot.dims' must equal rot_dim: the whole rotated part turns");
        m.set("rot", std::move(rot));
        m.set("kv_from", nullptr);
        if (present(mx, "kv_from")) {
            const long long from = need_int(mx, "kv_from", wm, 0);
            if (from >= (long long)layer) fail(KIPP_E_CONFIG, "config key '" + wm + "kv_from' must name an earlier layer");
            m.set("kv_from", from);
        }
    } else if (kind == "parallel") {
        const Json &left = need(mx, "left", wm), &right = need(mx, "right", wm);
        Json l = head_sizes(left, wm + "left."), r = head_sizes(right, wm + "right.");
        l.set("scale", need_number(left, "scale", wm + "left."));
        r.set("conv", need_int(right, "conv", wm + "right."));
        // the widths of the bottlenecks are the shapes of their tensors unless keys give them (the
        // random-weights writer needs them)
        for (const char* key : {"decay_rank", "gate_rank"})
            if (present(right, key)) r.set(key, need_int(right, key, wm + "right."));
        m.set("left", std::move(l));
        m.set("right", std::move(r));
    } else {
        fail(KIPP_E_CONFIG, "unknown layer type '" + kind + "' (mamba2, latent_attention, parallel)");
    }
    return m;
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
    out.set("token_side", nullptr);
    if (present(c, "token_side")) {
        Json side = Json::object();
        side.set("dim", need_int(c.get("token_side"), "dim", "token_side."));
        out.set("token_side", std::move(side));
    }
    const Json& layers = need(c, "layers", "");
    if (!layers.is_array() || layers.size() == 0) fail(KIPP_E_CONFIG, "config key 'layers' must be a list of layers");
    Json ls = Json::array();
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& l = layers.at(i);
        const std::string where = format("layers[%zu].", i);
        const Json& type = need(l, "type", where);
        if (!type.is_string()) fail(KIPP_E_CONFIG, "config key '" + where + "type' must be a string");
        Json layer = Json::object();
        layer.set("type", type.as_string());
        layer.set("mixer", mixer_keys(need(l, "mixer", where), type.as_string(), where + "mixer.", i));
        layer.set("mlp", nullptr);
        if (present(l, "mlp")) {
            const Json& mlp = l.get("mlp");
            const std::string fk = mlp.get_string("kind", "dense");
            if (fk != "dense") fail(KIPP_E_CONFIG, "feed-forward kind '" + fk + "' is not supported (dense)");
            Json f = Json::object();
            f.set("kind", fk);
            f.set("ff", need_int(mlp, "ff", where + "mlp."));
            layer.set("mlp", std::move(f));
        }
        ls.push(std::move(layer));
    }
    // a layer that reads another one's latent: the lender caches one of its own, of the same form
    for (size_t i = 0; i < ls.size(); ++i) {
        if (ls.at(i).get("type").as_string() != "latent_attention") continue;
        const Json& mx = ls.at(i).get("mixer");
        if (mx.get("kv_from").is_null()) continue;
        const Json& other = ls.at((size_t)mx.get("kv_from").as_int());
        const std::string where = format("layers[%zu].mixer.kv_from", i);
        if (other.get("type").as_string() != "latent_attention")
            fail(KIPP_E_CONFIG, "config key '" + where + "' must name a latent attention layer");
        const Json& om = other.get("mixer");
        if (!om.get("kv_from").is_null()) fail(KIPP_E_CONFIG, "config key '" + where + "' must name a layer with a latent of its own");
        for (const char* key : {"kv_rank", "rot_dim"})
            if (om.get(key).as_int() != mx.get(key).as_int())
                fail(KIPP_E_CONFIG, "config key '" + where + "': the two layers differ in '" + key + "'");
        if (mx.get("rot_dim").as_int() > 0 && om.get("rot").get("base").as_double() != mx.get("rot").get("base").as_double())
            fail(KIPP_E_CONFIG, "config key '" + where + "': the two layers differ in their rotation");
    }
    out.set("layers", std::move(ls));
    return out;
}

// the model's norm: the weight is stored as its distance from one
inline Json norm_part(long long width, double eps, const char* name) {
    Json j = venizen::rmsnorm_part(width, eps, name);
    j.set("weight_offset", 1.0);
    return j;
}

inline Json mixer_part(const std::string& kind, const Json& mx, long long width, double eps) {
    Json mixer = Json::object();
    mixer.set("hidden_size", width);
    mixer.set("eps", eps);
    if (kind == "mamba2") {
        mixer.set("kind", "state_space");
        mixer.set("num_heads", mx.get("heads").as_int());
        mixer.set("value_dim", mx.get("vdim").as_int());
        mixer.set("state_dim", mx.get("state").as_int());
        mixer.set("groups", mx.get("groups").as_int());
        mixer.set("conv", mx.get("conv").as_int());
        mixer.set("norm_groups", mx.get("norm_groups").as_int());
        return mixer;
    }
    if (kind == "latent_attention") {
        mixer.set("kind", "latent_attention");
        mixer.set("num_heads", mx.get("heads").as_int());
        mixer.set("head_dim", mx.get("dim").as_int());
        mixer.set("value_dim", mx.get("vdim").as_int());
        mixer.set("rot_dim", mx.get("rot_dim").as_int());
        mixer.set("kv_rank", mx.get("kv_rank").as_int());
        mixer.set("q_rank", mx.get("q_rank").as_int());
        mixer.set("scale", mx.get("scale").as_double());
        mixer.set("element_gate", true);
        mixer.set("interleaved", true);
        mixer.set("shared_kv", !mx.get("kv_from").is_null());
        mixer.set("position", venizen::rotary_part(mx.get("rot"), mx.get("rot_dim").as_int()));
        return mixer;
    }
    const Json &l = mx.get("left"), &r = mx.get("right");
    Json none = Json::object();
    none.set("kind", "no_position");
    Json attn = Json::object();
    attn.set("kind", "attention");
    attn.set("hidden_size", width);
    attn.set("num_heads", l.get("heads").as_int());
    attn.set("num_kv_heads", l.get("kv_heads").as_int());
    attn.set("head_dim", l.get("dim").as_int());
    attn.set("value_dim", l.get("vdim").as_int());
    attn.set("position", std::move(none));
    attn.set("qk_norm_eps", eps);
    attn.set("bias", true);
    attn.set("scale", l.get("scale").as_double());
    attn.set("names", venizen::names_of({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}, {"q_norm", "q.norm"}, {"k_norm", "k.norm"},
                                         {"q_bias", "q.b"}, {"k_bias", "k.b"}, {"v_bias", "v.b"}}));
    Json delta = Json::object();
    delta.set("kind", "gated_delta");
    delta.set("hidden_size", width);
    delta.set("num_heads", r.get("heads").as_int());
    delta.set("num_kv_heads", r.get("kv_heads").as_int());
    delta.set("head_dim", r.get("dim").as_int());
    delta.set("value_dim", r.get("vdim").as_int());
    delta.set("conv", r.get("conv").as_int());
    delta.set("eps", eps);
    delta.set("gate", "sigmoid");
    for (const char* key : {"decay_rank", "gate_rank"})
        if (present(r, key)) delta.set(key, r.get(key).as_int());
    Json bl = Json::object(), br = Json::object(), branches = Json::array(), out_norm = Json::object();
    bl.set("prefix", "left.");
    bl.set("part", std::move(attn));
    bl.set("norm", "left.out");
    br.set("prefix", "right.");
    br.set("part", std::move(delta));
    br.set("norm", "right.out");
    branches.push(std::move(bl));
    branches.push(std::move(br));
    out_norm.set("size", width);
    out_norm.set("eps", eps);
    mixer.set("kind", "parallel");
    mixer.set("branches", std::move(branches));
    mixer.set("out_norm", std::move(out_norm));
    mixer.set("out_scale", BRANCH_SCALE);
    return mixer;
}

inline Json plan(const Json& c) {
    const long long width = c.get("width").as_int(), vocab = c.get("vocab").as_int();
    const double eps = c.get("norm").get("eps").as_double();
    const Json& layers = c.get("layers");
    const long long side_dim = c.get("token_side").is_null() ? 0 : c.get("token_side").get("dim").as_int();
    const long long side_cols = side_dim * (long long)layers.size();
    Json p = Json::object();
    p.set("hidden_size", width);
    p.set("vocab_size", vocab);
    p.set("max_positions", 0LL);
    p.set("config", c);
    Json stages = Json::array();
    auto stage = [&](Json part) {
        Json s = Json::object();
        s.set("prefix", "");
        s.set("part", std::move(part));
        stages.push(std::move(s));
    };
    Json emb = Json::object();
    emb.set("kind", "token_embedding");
    emb.set("vocab_size", vocab);
    emb.set("hidden_size", width);
    emb.set("weight_name", "embed");
    stage(std::move(emb));
    if (side_dim > 0) {
        Json table = Json::object();
        table.set("kind", "token_side_table");
        table.set("vocab_size", vocab);
        table.set("cols", side_cols);
        table.set("weight_name", "side.embed");
        stage(std::move(table));
    }
    p.set("embedding", std::move(stages));

    Json blocks = Json::array(), order = Json::array();
    for (size_t i = 0; i < layers.size(); ++i) {
        const Json& l = layers.at(i);
        const Json& mx = l.get("mixer");
        const std::string type = l.get("type").as_string();
        Json block = Json::object(), names = Json::array();
        block.set("kind", "parallel_block");
        for (const char* n : {"", "mix.", "mlp.", "", "side."}) names.push(n);
        block.set("names", std::move(names));
        block.set("norm", norm_part(width, eps, "norm1"));
        block.set("mixer", mixer_part(type, mx, width, eps));
        block.set("ffn", nullptr);
        block.set("ffn_norm", nullptr);
        if (!l.get("mlp").is_null()) {
            Json ffn = Json::object();
            ffn.set("kind", "dense_mlp");
            ffn.set("hidden_size", width);
            ffn.set("intermediate_size", l.get("mlp").get("ff").as_int());
            ffn.set("activation", "relu_squared");
            block.set("ffn", std::move(ffn));
            block.set("ffn_norm", norm_part(width, eps, "norm2"));
        }
        block.set("side", nullptr);
        if (side_dim > 0) {
            Json side = Json::object();
            side.set("kind", "token_side");
            side.set("hidden_size", width);
            side.set("vocab_size", vocab);
            side.set("dim", side_dim);
            side.set("table", "side.embed");
            side.set("table_cols", side_cols);
            side.set("offset", side_dim * (long long)i);
            side.set("eps", eps);
            block.set("side", std::move(side));
        } else if (l.get("mlp").is_null()) {
            Json three = Json::array();
            for (const char* n : {"", "mix.", "mlp."}) three.push(n);
            block.set("names", std::move(three));
        }
        Json layer = Json::object();
        layer.set("prefix", format("l%zu.", i));
        layer.set("part", std::move(block));
        blocks.push(std::move(layer));
        const bool borrows = type == "latent_attention" && !mx.get("kv_from").is_null();
        Json run = Json::object();
        run.set("layer", (long long)i);
        run.set("cache", borrows ? mx.get("kv_from").as_int() : (long long)i);
        run.set("writes_cache", !borrows);
        order.push(std::move(run));
    }
    p.set("layers", std::move(blocks));
    p.set("order", std::move(order));

    Json fn = Json::object();
    fn.set("prefix", "");
    fn.set("part", norm_part(width, eps, "final.norm"));
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

}  // namespace nogavik

inline void register_nogavik() {
    Registry::get().add_architecture("Nogavik", Architecture{nogavik::normalize, nogavik::plan});
}

}  // namespace kipp
