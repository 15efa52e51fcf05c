// Typed configuration of the Salivik decoder, read from its config.json.
//
// The file names the design ("architecture": "Salivik"), the sizes (vocab, width), the
// constant norm.eps, a list of layers and a loop.  Each layer gives its mixer's type and
// sizes and its feed-forward, or null for none:
//
//   type "attention":         mixer {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims}}
//   type "retention":         mixer {heads, dim, vdim, decay [one number per head], rot {base, dims}}
//   type "latent_attention":  mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mask {size},
//       rot {base, dims, scaling {factor, original, fast, slow}}}
//   mlp {kind "dense", ff, limit} or {kind "moe", expert {ff, limit}, router {experts, top},
//       shared {ff, limit} or null}
//
// loop {start, stop, times}: layers start .. stop-1 run `times` times in a row with the same
// weights, every pass as run-order entries of its own (its own places in the cache); every
// pass, the first one too, begins with one matrix over the residual stream and the embedding
// output side by side, whose result is the residual stream from there on.
//
// What the design fixes is written here: the embedding rows go through an RMS norm; a layer
// has an RMS norm in front of each sublayer and none on its result; the rotation turns value
// i with value i + dims / 2; the attention's values are its keys before the rotation, its
// softmax has a one added to the denominator (a sink of score 0 for every head), and a
// sigmoid gate multiplies the joined heads; the retention's keys are scaled by
// dim^(-1/2), each head's result is divided by its root mean square and the joined heads are
// gated by a silu; the latent attention has a learned sink per head and no gate; the
// feed-forwards are gated units with both sides cut off at `limit` (g sigmoid(1.702 g) (u + 1));
// the router adds a bias to its logits and weighs the chosen experts by a softmax over
// their logits alone.
//
// Tensor names: embed, embed.norm, loop.in, final.norm, head; layer i below "l<i>": norm1, norm2,
// mix.{q, k, g, o}, mix.{q, k, v, g, o} or mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, o},
// mlp.{gate, up, down} or mlp.{e<j>.gate, e<j>.up, e<j>.down, router, router.b, shared.gate,
// shared.up, shared.down}.
#include "salivik.h"

#include <cmath>

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

const Json &need_obj(const Json &d, const char *key, const std::string &where) {
    if (!d.get(key).is_object()) config_error("config.json: " + where + key + " must be an object");
    return d.get(key);
}

SalivikConfig::Rotation read_rotation(const Json &m, const std::string &w) {
    SalivikConfig::Rotation r;
    if (m.get("rot").is_null()) return r;
    const Json &d = need_obj(m, "rot", w);
    std::string rw = w + "rot.";
    r.dims = need_int(d, "dims", rw);
    r.base = need_num(d, "base", rw);
    if (!d.get("scaling").is_null()) {
        const Json &s = need_obj(d, "scaling", rw);
        r.scaled = true;
        r.factor = need_num(s, "factor", rw + "scaling.");
        r.original = need_num(s, "original", rw + "scaling.");
        r.fast = need_num(s, "fast", rw + "scaling.");
        r.slow = need_num(s, "slow", rw + "scaling.");
    }
    return r;
}

Json rotation_json(const SalivikConfig::Rotation &r) {
    Json o = Json::object();
    o.set("base", r.base);
    o.set("dims", r.dims);
    if (r.scaled) {
        Json s = Json::object();
        s.set("factor", r.factor);
        s.set("fast", r.fast);
        s.set("original", r.original);
        s.set("slow", r.slow);
        o.set("scaling", s);
    }
    return o;
}

PartSpec position_part(const SalivikConfig::Rotation &r, long long positions) {
    if (r.dims <= 0) return PartSpec{"none", Json::object()};
    PartSpec pos{"rope_neox", Json::object()};
    pos.params.set("rotary_dim", r.dims);
    pos.params.set("theta", r.base);
    pos.params.set("max_positions", positions);
    if (r.scaled) {
        Json s = Json::object();
        s.set("factor", r.factor);
        s.set("original", r.original);
        s.set("fast", r.fast);
        s.set("slow", r.slow);
        pos.params.set("yarn", s);
    }
    return pos;
}

// the experts', the shared expert's and the dense feed-forward's gated unit
Json unit_json(double limit) {
    Json u = Json::object();
    u.set("alpha", 1.702);
    u.set("limit", limit);
    u.set("shift", 1.0);
    return u;
}

}  // namespace

SalivikConfig SalivikConfig::from_json(const Json &d) {
    SalivikConfig c;
    c.vocab = need_int(d, "vocab", "");
    c.width = need_int(d, "width", "");
    c.norm_eps = need_num(need_obj(d, "norm", ""), "eps", "norm.");
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
        if (y.type != "attention" && y.type != "retention" && y.type != "latent_attention")
            config_error("config.json: " + where + "type '" + y.type +
                         "': this design's mixers are 'attention', 'retention' and 'latent_attention'");
        y.heads = need_int(m, "heads", mw);
        y.dim = need_int(m, "dim", mw);
        y.vdim = opt_int(m, "vdim", mw, y.dim);
        y.rot = read_rotation(m, mw);
        if (y.type == "retention") {
            const Json &dc = m.get("decay");
            if (!dc.is_array()) config_error("config.json: " + mw + "decay must list one number per head");
            for (size_t k = 0; k < dc.size(); k++) {
                if (dc[k].is_bool() || !dc[k].is_number())
                    config_error("config.json: " + mw + "decay must list numbers");
                y.decay.push_back(dc[k].as_double());
            }
        } else {
            y.scale = need_num(m, "scale", mw);
            if (!m.get("mask").is_null()) {
                y.window = need_int(need_obj(m, "mask", mw), "size", mw + "mask.");
                if (y.window <= 0) config_error("config.json: " + mw + "mask.size must be positive");
            }
            if (y.type == "attention") {
                y.kv_heads = opt_int(m, "kv_heads", mw, y.heads);
            } else {
                y.rot_dim = need_int(m, "rot_dim", mw);
                y.kv_rank = need_int(m, "kv_rank", mw);
                y.q_rank = need_int(m, "q_rank", mw);
            }
        }
        const Json &f = l.get("mlp");
        if (!f.is_null()) {
            std::string fw = where + "mlp.";
            if (!f.is_object() || !f.get("kind").is_string())
                config_error("config.json: " + where + "mlp must be null or an object with a kind");
            y.has_mlp = true;
            y.mlp_kind = f.get("kind").as_string();
            if (y.mlp_kind == "dense") {
                y.ff = need_int(f, "ff", fw);
                y.limit = need_num(f, "limit", fw);
            } else if (y.mlp_kind == "moe") {
                const Json &ro = need_obj(f, "router", fw);
                y.experts = need_int(ro, "experts", fw + "router.");
                y.top = need_int(ro, "top", fw + "router.");
                const Json &e = need_obj(f, "expert", fw);
                y.expert_ff = need_int(e, "ff", fw + "expert.");
                y.expert_limit = need_num(e, "limit", fw + "expert.");
                if (!f.get("shared").is_null()) {
                    const Json &s = need_obj(f, "shared", fw);
                    y.shared_ff = need_int(s, "ff", fw + "shared.");
                    y.shared_limit = need_num(s, "limit", fw + "shared.");
                    if (y.shared_ff <= 0) config_error("config.json: " + fw + "shared.ff must be positive");
                }
            } else {
                config_error("config.json: " + fw + "kind '" + y.mlp_kind + "': this design's are 'dense' and 'moe'");
            }
        }
        c.layers.push_back(y);
    }
    const Json &lp = d.get("loop");
    if (!lp.is_null()) {
        if (!lp.is_object()) config_error("config.json: loop must be null or an object with start, stop and times");
        c.has_loop = true;
        c.loop_start = need_int(lp, "start", "loop.");
        c.loop_stop = need_int(lp, "stop", "loop.");
        c.loop_times = need_int(lp, "times", "loop.");
    }
    c.validate();
    return c;
}

void SalivikConfig::validate() const {
    if (vocab <= 0 || width <= 0) config_error("config.json: vocab and width must be positive");
    if (layers.empty() || layers.size() > 100000) config_error("config.json: layers must not be empty");
    long long n = (long long)layers.size();
    if (has_loop && (loop_start < 0 || loop_stop <= loop_start || loop_stop > n || loop_times < 1 || loop_times > 100000))
        config_error("config.json: loop needs 0 <= start < stop <= the number of layers and times >= 1");
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        std::string where = fmt("config.json: layers[%zu]: ", i);
        if (y.heads <= 0 || y.dim <= 0 || y.vdim <= 0) config_error(where + "heads, dim and vdim must be positive");
        long long turned = y.type == "latent_attention" ? y.rot_dim : y.dim;
        if (y.rot.dims < 0 || y.rot.dims % 2 || y.rot.dims > turned)
            config_error(where + "rot.dims must be even and at most " +
                         (y.type == "latent_attention" ? "rot_dim" : "dim"));
        if (y.rot.dims > 0 && !(y.rot.base > 0)) config_error(where + "rot.base must be positive");
        if (y.rot.scaled && (!(y.rot.factor > 0) || !(y.rot.original > 0) || !(y.rot.fast > 0) || !(y.rot.slow > 0) ||
                             y.rot.base == 1.0))
            config_error(where + "rot.scaling needs factor, original, fast and slow above 0 and a base other than 1");
        if (y.type == "attention") {
            if (y.kv_heads <= 0 || y.heads % y.kv_heads) config_error(where + "heads must be a multiple of kv_heads");
            if (y.vdim != y.dim) config_error(where + "the values are the keys: vdim must be dim");
            if (y.dim > 512) config_error(where + "the attention kernels take head sizes up to 512");
        } else if (y.type == "retention") {
            if ((long long)y.decay.size() != y.heads) config_error(where + "decay must list one number per head");
            if (y.dim > 1024) config_error(where + "the recurrence's kernel takes heads of up to 1024 values");
        } else {
            if (y.kv_rank <= 0 || y.q_rank <= 0 || y.rot_dim < 0)
                config_error(where + "kv_rank and q_rank must be positive, rot_dim not negative");
            if (y.kv_rank + y.rot_dim > 512)
                config_error(where + "kv_rank + rot_dim is above 512, the longest row the attention kernels take");
        }
        if (y.has_mlp && y.mlp_kind == "dense" && (y.ff <= 0 || !(y.limit > 0)))
            config_error(where + "mlp.ff and mlp.limit must be positive");
        if (y.has_mlp && y.mlp_kind == "moe") {
            if (y.experts <= 0 || y.expert_ff <= 0) config_error(where + "the router needs experts");
            if (y.top <= 0 || y.top > y.experts) config_error(where + "router.top must be between 1 and experts");
            if (!(y.expert_limit > 0) || (y.shared_ff > 0 && !(y.shared_limit > 0)))
                config_error(where + "an expert's limit must be positive");
        }
    }
}

std::vector<std::pair<int, bool>> SalivikConfig::order() const {
    std::vector<std::pair<int, bool>> out;
    int n = (int)layers.size(), start = has_loop ? (int)loop_start : 0, stop = has_loop ? (int)loop_stop : 0;
    for (int i = 0; i < start; i++) out.push_back({i, false});
    for (long long pass = 0; has_loop && pass < loop_times; pass++)
        for (int i = start; i < stop; i++) out.push_back({i, i == start});
    for (int i = stop; i < n; i++) out.push_back({i, false});
    return out;
}

Json SalivikConfig::to_json() const {
    Json d = Json::object();
    d.set("architecture", "Salivik");
    Json ls = Json::array();
    for (auto &y : layers) {
        Json l = Json::object(), m = Json::object();
        if (y.type == "retention") {
            Json dc = Json::array();
            for (double v : y.decay) dc.push(Json(v));
            m.set("decay", dc);
        }
        m.set("dim", y.dim);
        m.set("heads", y.heads);
        if (y.type == "attention") m.set("kv_heads", y.kv_heads);
        if (y.type == "latent_attention") m.set("kv_rank", y.kv_rank);
        if (y.window > 0) {
            Json w = Json::object();
            w.set("size", y.window);
            m.set("mask", w);
        }
        if (y.type == "latent_attention") m.set("q_rank", y.q_rank);
        if (y.rot.dims > 0) m.set("rot", rotation_json(y.rot));
        if (y.type == "latent_attention") m.set("rot_dim", y.rot_dim);
        if (y.type != "retention") m.set("scale", y.scale);
        m.set("vdim", y.vdim);
        l.set("mixer", m);
        if (y.has_mlp && y.mlp_kind == "dense") {
            Json f = Json::object();
            f.set("ff", y.ff);
            f.set("kind", y.mlp_kind);
            f.set("limit", y.limit);
            l.set("mlp", f);
        } else if (y.has_mlp) {
            Json f = Json::object(), e = Json::object(), ro = Json::object();
            e.set("ff", y.expert_ff);
            e.set("limit", y.expert_limit);
            f.set("expert", e);
            f.set("kind", y.mlp_kind);
            ro.set("experts", y.experts);
            ro.set("top", y.top);
            f.set("router", ro);
            Json s;
            if (y.shared_ff > 0) {
                s = Json::object();
                s.set("ff", y.shared_ff);
                s.set("limit", y.shared_limit);
            }
            f.set("shared", s);
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
    d.set("vocab", vocab);
    d.set("width", width);
    return d;
}

ModelSpec SalivikConfig::to_model_spec() const {
    // every norm of the residual stream: an RMS norm over the width whose weight is the
    // tensor named as the norm
    PartSpec norm{"rmsnorm", Json::object()};
    norm.params.set("size", width);
    norm.params.set("eps", norm_eps);
    {
        Json nm = Json::object();
        nm.set("weight", "");
        norm.params.set("names", nm);
    }
    // the design gives no limit on positions: the cache's size is the limit
    const long long positions = 1ll << 30;
    ModelSpec s;
    s.architecture = "Salivik";
    s.hidden_size = width;
    s.vocab_size = vocab;
    s.max_positions = positions;
    s.embedding_name = "embed";
    s.embedding_norm = norm;
    s.embedding_norm_name = "embed.norm";
    s.head_name = "head";
    s.tie_embeddings = false;
    s.final_norm_name = "final.norm";
    s.final_norm = norm;
    if (has_loop) s.join_name = "loop.in";
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        PartSpec mixer;
        Json nm = Json::object();
        mixer.params.set("hidden_size", width);
        mixer.params.set("position", position_part(y.rot, positions).to_json());
        if (y.type == "attention") {
            mixer.kind = "sink_attention";
            mixer.params.set("num_heads", y.heads);
            mixer.params.set("num_kv_heads", y.kv_heads);
            mixer.params.set("head_dim", y.dim);
            mixer.params.set("scale", y.scale);
            mixer.params.set("window", y.window);
            mixer.params.set("bias", false);
            mixer.params.set("values_are_keys", true);
            mixer.params.set("sink_score", 0.0);
            mixer.params.set("gate", true);
            for (const char *k : {"q", "k", "o"}) nm.set(k, k);
            nm.set("gate", "g");
        } else if (y.type == "retention") {
            mixer.kind = "decay_attention";
            mixer.params.set("heads", y.heads);
            mixer.params.set("head_dim", y.dim);
            mixer.params.set("v_head_dim", y.vdim);
            Json dc = Json::array();
            for (double v : y.decay) dc.push(Json(v));
            mixer.params.set("decay", dc);
            mixer.params.set("eps", norm_eps);
            mixer.params.set("activation", "none");
            mixer.params.set("key_scale", 1.0 / std::sqrt((double)y.dim));
            mixer.params.set("head_norm", true);
            mixer.params.set("gate", "silu");
            for (const char *k : {"q", "k", "v", "g", "o"}) nm.set(k, k);
        } else {
            mixer.kind = "latent_attention";
            mixer.params.set("num_heads", y.heads);
            mixer.params.set("head_dim", y.dim);
            mixer.params.set("rot_dim", y.rot_dim);
            mixer.params.set("v_head_dim", y.vdim);
            mixer.params.set("kv_rank", y.kv_rank);
            mixer.params.set("q_rank", y.q_rank);
            mixer.params.set("scale", y.scale);
            mixer.params.set("eps", norm_eps);
            mixer.params.set("gate", false);
            mixer.params.set("window", y.window);
            mixer.params.set("sink", true);
            for (const char *k : {"dq", "uq", "dkv", "uk", "uv", "o", "sink"}) nm.set(k, k);
            nm.set("dq_norm", "dq.norm");
            nm.set("dkv_norm", "dkv.norm");
        }
        mixer.params.set("names", nm);
        LayerSpec l;
        l.block = "prenorm";
        l.prefix = fmt("l%zu", i);
        l.mixer = mixer;
        l.mixer_name = "mix";
        l.mixer_norm = norm;
        l.mixer_norm_name = "norm1";
        if (y.has_mlp) {
            PartSpec ffn;
            Json fn = Json::object();
            for (const char *k : {"gate", "up", "down"}) fn.set(k, k);
            ffn.params.set("hidden_size", width);
            if (y.mlp_kind == "dense") {
                ffn.kind = "swiglu";
                ffn.params.set("intermediate_size", y.ff);
                ffn.params.set("unit", unit_json(y.limit));
            } else {
                ffn.kind = "routed";
                ffn.params.set("experts", y.experts);
                ffn.params.set("expert_ff", y.expert_ff);
                ffn.params.set("top", y.top);
                ffn.params.set("score", "chosen_softmax");
                ffn.params.set("router_bias", true);
                ffn.params.set("gated", true);
                ffn.params.set("activation", "silu");
                ffn.params.set("unit", unit_json(y.expert_limit));
                if (y.shared_ff > 0) {
                    ffn.params.set("shared_ff", y.shared_ff);
                    ffn.params.set("shared_unit", unit_json(y.shared_limit));
                }
                fn.set("expert", "e");
                fn.set("router", "router");
                fn.set("router_bias", "router.b");
                fn.set("shared", "shared");
            }
            ffn.params.set("names", fn);
            l.feed_forward = ffn;
            l.ffn_name = "mlp";
            l.ffn_norm = norm;
            l.ffn_norm_name = "norm2";
        }
        s.layers.push_back(l);
    }
    for (auto &e : order()) {
        RunEntry r;
        r.layer = e.first;
        r.join_embedding = e.second;
        s.run_order.push_back(r);
    }
    s.validate();
    return s;
}

void register_salivik() {
    register_architecture("Salivik", "salivik", [](const Json &d) {
        return std::unique_ptr<ArchConfig>(new SalivikConfig(SalivikConfig::from_json(d)));
    });
}

}  // namespace jb
