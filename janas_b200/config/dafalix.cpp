// Typed configuration of the Dafalix decoder, read from its config.json.
//
// The file names the design ("architecture": "Dafalix"), the sizes (vocab, width, streams), the
// constants (norm.eps, residual_mult), optionally a loop {start, stop, times} (a span of
// layers that is passed through `times` times; each pass keeps keys, values and states apart) and a
// list of layers, each with its mixer's type, the mixer's sizes and its feed-forward, or null:
//
//   type "parallel": mixer {left {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims,
//       scaling {factor}}}, right {width, blocks, conv}, left_scale, right_scale}
//   type "mlstm":    mixer {heads, dim, vdim, gate_cap}
//   mlp {kind "moe", expert {ff}, router {experts, top}}
//
// What the design fixes is written here.  The residual stream is `streams` streams per row that each
// sublayer reads as a weighted sum through a layer norm with a bias, and that are mixed as its
// result, multiplied value by value by a vector of the layer's, joins.  "parallel": windowed softmax
// attention with a weighted RMS norm per head on q and k before the rotation (value i turns with
// value i + dims / 2), beside a real-gated linear recurrent unit behind a short convolution; both
// read the same input and are added with two factors.  "mlstm": a matrix memory with exponential
// gates, a norm per head and a sigmoid gate.  Experts are SwiGLU without biases; the router's scores
// are sigmoids, used as they are, and weigh what the experts read.  The head is the embedding table.
//
// Tensor names: embed, final.norm, final.norm.b; layer i below "l<i>": norm1, norm1.b, norm2, norm2.b,
// ls1, ls2, hc1.{in, out, mix}, hc2.{in, out, mix}, mix.left.{q, k, v, o, q.norm, k.norm},
// mix.right.{y, x, conv, ra, ri (each with .b), lam, o} or mix.{q, k, v, g, i, i.b, f, f.b, o, norm},
// mlp.{e<j>.gate, e<j>.up, e<j>.down, router}.
#include "dafalix.h"

namespace jb {

namespace {

long long need_int(const Json &d, const char *key, const std::string &where) {
    const Json &v = d.get(key);
    if (v.is_bool() || !v.is_number() || !v.whole())
        config_error("config.json: " + where + key + " must be a whole number, got " + v.dump());
    return v.as_int();
}

double need_num(const Json &d, const char *key, const std::string &where) {
    const Json &v = d.get(key);
    if (v.is_bool() || !v.is_number())
        config_error("config.json: " + where + key + " must be a number, got " + v.dump());
    return v.as_double();
}

long long opt_int(const Json &d, const char *key, const std::string &where, long long dflt) {
    return d.get(key).is_null() ? dflt : need_int(d, key, where);
}

double opt_num(const Json &d, const char *key, const std::string &where, double dflt) {
    return d.get(key).is_null() ? dflt : need_num(d, key, where);
}

const Json &need_obj(const Json &d, const char *key, const std::string &where) {
    if (!d.get(key).is_object()) config_error("config.json: " + where + key + " must be an object");
    return d.get(key);
}

Json names(std::initializer_list<std::pair<const char *, const char *>> list) {
    Json j = Json::object();
    for (auto &kv : list) j.set(kv.first, kv.second);
    return j;
}

}  // namespace

DafalixConfig DafalixConfig::from_json(const Json &d) {
    DafalixConfig c;
    c.vocab = need_int(d, "vocab", "");
    c.width = need_int(d, "width", "");
    c.streams = opt_int(d, "streams", "", 1);
    c.residual_mult = opt_num(d, "residual_mult", "", 1.0);
    c.norm_eps = need_num(need_obj(d, "norm", ""), "eps", "norm.");
    if (!d.get("loop").is_null()) {
        const Json &lp = need_obj(d, "loop", "");
        c.has_loop = true;
        c.loop_start = need_int(lp, "start", "loop.");
        c.loop_stop = need_int(lp, "stop", "loop.");
        c.loop_times = need_int(lp, "times", "loop.");
    }
    const Json &ls = d.get("layers");
    if (!ls.is_array() || ls.size() == 0) config_error("config.json: layers must be a list of layers");
    for (size_t i = 0; i < ls.size(); i++) {
        const Json &l = ls[i];
        std::string where = fmt("layers[%zu].", i);
        if (!l.is_object() || !l.get("type").is_string() || !l.get("mixer").is_object())
            config_error("config.json: " + where + " needs a type and a mixer");
        Layer y;
        y.type = l.get("type").as_string();
        const Json &m = l.get("mixer");
        std::string mw = where + "mixer.";
        if (y.type == "mlstm") {
            y.heads = need_int(m, "heads", mw);
            y.dim = need_int(m, "dim", mw);
            y.vdim = opt_int(m, "vdim", mw, y.dim);
            y.gate_cap = need_num(m, "gate_cap", mw);
        } else if (y.type == "parallel") {
            const Json &a = need_obj(m, "left", mw), &r = need_obj(m, "right", mw);
            std::string aw = mw + "left.", rw = mw + "right.";
            y.heads = need_int(a, "heads", aw);
            y.kv_heads = opt_int(a, "kv_heads", aw, y.heads);
            y.dim = need_int(a, "dim", aw);
            y.vdim = opt_int(a, "vdim", aw, y.dim);
            y.scale = need_num(a, "scale", aw);
            if (!a.get("mask").is_null()) {
                y.window = need_int(need_obj(a, "mask", aw), "size", aw + "mask.");
                if (y.window <= 0) config_error("config.json: " + aw + "mask.size must be positive");
            }
            if (!a.get("rot").is_null()) {
                const Json &ro = need_obj(a, "rot", aw);
                y.rot_dims = need_int(ro, "dims", aw + "rot.");
                y.rot_base = need_num(ro, "base", aw + "rot.");
                if (!ro.get("scaling").is_null()) {
                    y.rot_scaled = true;
                    y.rot_factor = need_num(need_obj(ro, "scaling", aw + "rot."), "factor", aw + "rot.scaling.");
                }
            }
            y.rec_width = need_int(r, "width", rw);
            y.rec_blocks = opt_int(r, "blocks", rw, 1);
            y.rec_conv = opt_int(r, "conv", rw, 1);
            y.left_scale = opt_num(m, "left_scale", mw, 1.0);
            y.right_scale = opt_num(m, "right_scale", mw, 1.0);
        } else {
            config_error("config.json: " + where + "type '" + y.type + "': this design's mixers are 'parallel' and 'mlstm'");
        }
        const Json &f = l.get("mlp");
        if (!f.is_null()) {
            std::string fw = where + "mlp.";
            if (!f.is_object() || !f.get("kind").is_string())
                config_error("config.json: " + where + "mlp must be null or an object with a kind");
            if (f.get("kind").as_string() != "moe")
                config_error("config.json: " + fw + "kind '" + f.get("kind").as_string() + "': this design's is 'moe'");
            y.has_mlp = true;
            const Json &ro = need_obj(f, "router", fw);
            y.experts = need_int(ro, "experts", fw + "router.");
            y.top = need_int(ro, "top", fw + "router.");
            y.expert_ff = need_int(need_obj(f, "expert", fw), "ff", fw + "expert.");
        }
        c.layers.push_back(y);
    }
    c.validate();
    return c;
}

void DafalixConfig::validate() const {
    if (vocab <= 0 || width <= 0) config_error("config.json: vocab and width must be positive");
    if (streams <= 0 || streams > 32) config_error("config.json: streams must be between 1 and 32");
    if (layers.empty() || layers.size() > 100000) config_error("config.json: layers must not be empty");
    if (has_loop && (loop_start < 0 || loop_stop <= loop_start || loop_stop > (long long)layers.size() ||
                     loop_times < 1 || loop_times > 100000))
        config_error("config.json: loop needs 0 <= start < stop <= the number of layers and times of at least 1");
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        std::string where = fmt("config.json: layers[%zu]: ", i);
        if (y.heads <= 0 || y.dim <= 0 || y.vdim <= 0) config_error(where + "heads, dim and vdim must be positive");
        if (y.type == "mlstm") {
            if (y.dim > 1024) config_error(where + "the memory's kernel takes heads of up to 1024 query values");
            if (!(y.gate_cap > 0)) config_error(where + "gate_cap must be positive");
        } else {
            if (y.kv_heads <= 0 || y.heads % y.kv_heads) config_error(where + "left.heads must be a multiple of left.kv_heads");
            if (y.dim > 512 || y.vdim > 512) config_error(where + "the attention kernels take head sizes up to 512");
            if (y.rot_dims < 0 || y.rot_dims % 2 || y.rot_dims > y.dim)
                config_error(where + "left.rot.dims must be even and at most dim");
            if (y.rot_dims > 0 && (y.rot_base <= 0 || y.rot_factor <= 0))
                config_error(where + "left.rot.base and left.rot.scaling.factor must be positive");
            if (y.rec_width <= 0 || y.rec_blocks <= 0 || y.rec_width % y.rec_blocks)
                config_error(where + "right.blocks must divide right.width");
            if (y.rec_conv <= 0) config_error(where + "right.conv must be positive");
        }
        if (y.has_mlp) {
            if (y.experts <= 0 || y.expert_ff <= 0) config_error(where + "the router needs experts");
            if (y.top <= 0 || y.top > y.experts) config_error(where + "router.top must be between 1 and experts");
        }
    }
}

std::vector<int> DafalixConfig::order() const {
    std::vector<int> out;
    int n = (int)layers.size(), start = has_loop ? (int)loop_start : 0, stop = has_loop ? (int)loop_stop : 0;
    for (int i = 0; i < start; i++) out.push_back(i);
    for (long long pass = 0; has_loop && pass < loop_times; pass++)
        for (int i = start; i < stop; i++) out.push_back(i);
    for (int i = stop; i < n; i++) out.push_back(i);
    return out;
}

Json DafalixConfig::to_json() const {
    Json d = Json::object();
    d.set("architecture", "Dafalix");
    Json ls = Json::array();
    for (auto &y : layers) {
        Json l = Json::object(), m = Json::object();
        if (y.type == "mlstm") {
            m.set("dim", y.dim);
            m.set("gate_cap", y.gate_cap);
            m.set("heads", y.heads);
            m.set("vdim", y.vdim);
        } else {
            Json a = Json::object(), r = Json::object();
            a.set("dim", y.dim);
            a.set("heads", y.heads);
            a.set("kv_heads", y.kv_heads);
            if (y.window > 0) {
                Json w = Json::object();
                w.set("size", y.window);
                a.set("mask", w);
            }
            if (y.rot_dims > 0) {
                Json ro = Json::object();
                ro.set("base", y.rot_base);
                ro.set("dims", y.rot_dims);
                if (y.rot_scaled) {
                    Json sc = Json::object();
                    sc.set("factor", y.rot_factor);
                    ro.set("scaling", sc);
                }
                a.set("rot", ro);
            }
            a.set("scale", y.scale);
            a.set("vdim", y.vdim);
            r.set("blocks", y.rec_blocks);
            r.set("conv", y.rec_conv);
            r.set("width", y.rec_width);
            m.set("left", a);
            m.set("left_scale", y.left_scale);
            m.set("right", r);
            m.set("right_scale", y.right_scale);
        }
        l.set("mixer", m);
        if (y.has_mlp) {
            Json f = Json::object(), e = Json::object(), ro = Json::object();
            e.set("ff", y.expert_ff);
            f.set("expert", e);
            f.set("kind", "moe");
            ro.set("experts", y.experts);
            ro.set("top", y.top);
            f.set("router", ro);
            l.set("mlp", f);
        } else {
            l.set("mlp", Json());
        }
        l.set("type", y.type);
        ls.push(l);
    }
    d.set("layers", ls);
    Json lp;
    if (has_loop) {
        lp = Json::object();
        lp.set("start", loop_start);
        lp.set("stop", loop_stop);
        lp.set("times", loop_times);
    }
    d.set("loop", lp);
    Json n = Json::object();
    n.set("eps", norm_eps);
    d.set("norm", n);
    d.set("residual_mult", residual_mult);
    d.set("streams", streams);
    d.set("vocab", vocab);
    d.set("width", width);
    return d;
}

ModelSpec DafalixConfig::to_model_spec() const {
    // every norm of the residual stream: a layer norm over the width; the weight's tensor is
    // named as the norm, the bias has a suffix
    PartSpec norm{"layernorm", Json::object()};
    norm.params.set("size", width);
    norm.params.set("eps", norm_eps);
    norm.params.set("names", names({{"weight", ""}, {"bias", "b"}}));
    // the design gives no limit on positions: the cache's size is the limit
    const long long positions = 1ll << 30;
    ModelSpec s;
    s.architecture = "Dafalix";
    s.hidden_size = width;
    s.vocab_size = vocab;
    s.max_positions = positions;
    s.streams = streams;
    s.embedding_name = "embed";
    s.head_name = "head";
    s.tie_embeddings = true;
    s.final_norm_name = "final.norm";
    s.final_norm = norm;
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        PartSpec mixer;
        if (y.type == "mlstm") {
            mixer.kind = "mlstm";
            mixer.params.set("hidden_size", width);
            mixer.params.set("heads", y.heads);
            mixer.params.set("head_dim", y.dim);
            mixer.params.set("v_head_dim", y.vdim);
            mixer.params.set("gate_cap", y.gate_cap);
            mixer.params.set("eps", norm_eps);
            mixer.params.set("floor", 1e-6);
            mixer.params.set("names", names({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"g", "g"}, {"i", "i"}, {"f", "f"},
                                             {"bias", ".b"}, {"o", "o"}, {"norm", "norm"}}));
        } else {
            PartSpec left{"sink_attention", Json::object()}, right{"rglru", Json::object()};
            left.params.set("hidden_size", width);
            left.params.set("num_heads", y.heads);
            left.params.set("num_kv_heads", y.kv_heads);
            left.params.set("head_dim", y.dim);
            left.params.set("v_head_dim", y.vdim);
            left.params.set("scale", y.scale);
            left.params.set("window", y.window);
            left.params.set("bias", false);
            left.params.set("qk_norm_eps", norm_eps);
            if (y.rot_dims > 0) {
                PartSpec pos{"rope_neox", Json::object()};
                pos.params.set("rotary_dim", y.rot_dims);
                pos.params.set("theta", y.rot_base);
                pos.params.set("max_positions", positions);
                pos.params.set("linear_factor", y.rot_factor);
                left.params.set("position", pos.to_json());
            }
            left.params.set("names", names({{"q", "q"}, {"k", "k"}, {"v", "v"}, {"o", "o"}, {"q_norm", "q.norm"},
                                            {"k_norm", "k.norm"}}));
            right.params.set("hidden_size", width);
            right.params.set("width", y.rec_width);
            right.params.set("blocks", y.rec_blocks);
            right.params.set("conv_taps", y.rec_conv);
            right.params.set("names", names({{"y", "y"}, {"x", "x"}, {"conv", "conv"}, {"r", "ra"}, {"i", "ri"},
                                             {"bias", ".b"}, {"lambda", "lam"}, {"o", "o"}}));
            mixer.kind = "pair";
            mixer.params.set("hidden_size", width);
            mixer.params.set("left", left.to_json());
            mixer.params.set("right", right.to_json());
            mixer.params.set("join", "sum");
            mixer.params.set("left_scale", y.left_scale);
            mixer.params.set("right_scale", y.right_scale);
            mixer.params.set("names", names({{"left", "left"}, {"right", "right"}}));
        }
        LayerSpec l;
        l.block = "streams";
        l.prefix = fmt("l%zu", i);
        l.mixer = mixer;
        l.mixer_name = "mix";
        l.mixer_norm = norm;
        l.mixer_norm_name = "norm1";
        l.block_params.set("hidden_size", width);
        l.block_params.set("streams", streams);
        l.block_params.set("residual_mult", residual_mult);
        l.block_params.set("mixer_streams", "hc1");
        l.block_params.set("ffn_streams", "hc2");
        l.block_params.set("mixer_scale", "ls1");
        l.block_params.set("ffn_scale", "ls2");
        if (y.has_mlp) {
            PartSpec ffn{"routed", Json::object()};
            ffn.params.set("hidden_size", width);
            ffn.params.set("experts", y.experts);
            ffn.params.set("expert_ff", y.expert_ff);
            ffn.params.set("top", y.top);
            ffn.params.set("score", "sigmoid");
            ffn.params.set("gated", true);
            ffn.params.set("activation", "silu");
            ffn.params.set("weight_on_input", true);
            ffn.params.set("names", names({{"expert", "e"}, {"gate", "gate"}, {"up", "up"}, {"down", "down"},
                                           {"router", "router"}}));
            l.feed_forward = ffn;
            l.ffn_name = "mlp";
            l.ffn_norm = norm;
            l.ffn_norm_name = "norm2";
        } else {
            // what surrounds an absent feed-forward may still stand in the file
            Json unused = Json::array();
            auto add = [&](const char *name, std::initializer_list<long long> shape) {
                Json o = Json::object(), sh = Json::array();
                for (long long v : shape) sh.push(Json(v));
                o.set("name", name);
                o.set("shape", sh);
                unused.push(o);
            };
            add("norm2", {width});
            add("norm2.b", {width});
            add("ls2", {width});
            add("hc2.in", {streams});
            add("hc2.out", {streams});
            add("hc2.mix", {streams, streams});
            l.block_params.set("unused", unused);
        }
        s.layers.push_back(l);
    }
    for (int layer : order()) {
        RunEntry r;
        r.layer = layer;
        s.run_order.push_back(r);
    }
    s.validate();
    return s;
}

void register_dafalix() {
    register_architecture("Dafalix", "dafalix", [](const Json &d) {
        return std::unique_ptr<ArchConfig>(new DafalixConfig(DafalixConfig::from_json(d)));
    });
}

}  // namespace jb
