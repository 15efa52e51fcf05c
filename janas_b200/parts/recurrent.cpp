// Mixers whose memory of the sequence is a state of fixed size (no keys and values):
// mingru, mamba2, decay_attention, mlstm and rglru (the last four are described at their classes).
//
// mingru: a gated running value whose gates read the current token alone,
//
//   z = sigmoid(Wz h + bz);  u = Wx h + bx;  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//   S_t = (1 - z_t) S_{t-1} + z_t c_t   (element by element, S before the first token = 0)
//   out = Wo (S_t * silu(Wg h))
//
// z, x and g are one product over h ([z | x | g], W columns each); gates, candidate,
// the recurrence and the state are float32 in both compute types; what goes into Wo is
// rounded to the compute type.  The state [W] lives in the cache per slot and is carried
// from step to step, so prompts in portions, decoding and batches of unequal rows all
// run the same kernels (csrc/recurrent.cu).
#include <algorithm>
#include <cmath>

#include "part.h"

namespace jb {

namespace {

// params: hidden_size, width, bias (default true: z and x have one), names (optional):
// z, x, g, o, bias (a suffix)
class MinGRU : public Mixer {
public:
    MinGRU(const PartSpec &s, DType dt, Device *d) : Mixer(s, dt, d) {
        hidden_ = s.get_int("hidden_size");
        width_ = s.get_int("width");
        bias_ = s.has("bias") ? s.params.get("bias").as_bool() : true;
        if (hidden_ <= 0 || width_ <= 0) config_error("mingru: sizes must be positive");
        const Json &nm = s.params.get("names");
        auto leaf = [&](const char *key, const char *dflt) {
            return nm.is_object() && nm.get(key).is_string() ? nm.get(key).as_string() : std::string(dflt);
        };
        n_z_ = leaf("z", "z_proj.weight");
        n_x_ = leaf("x", "x_proj.weight");
        n_g_ = leaf("g", "g_proj.weight");
        n_o_ = leaf("o", "o_proj.weight");
        n_bias_ = leaf("bias", ".bias");
    }

    void tensors(const std::string &p, TensorList &out) const override {
        out.emplace_back(name(p, n_z_), TensorSpec{{width_, hidden_}, MATRIX, false});
        if (bias_) out.emplace_back(name(p, n_z_ + n_bias_), TensorSpec{{width_}, PARAM, false, 0.0f, 0.5f});
        out.emplace_back(name(p, n_x_), TensorSpec{{width_, hidden_}, MATRIX, false});
        if (bias_) out.emplace_back(name(p, n_x_ + n_bias_), TensorSpec{{width_}, PARAM, false, 0.0f, 0.5f});
        out.emplace_back(name(p, n_g_), TensorSpec{{width_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_o_), TensorSpec{{hidden_, width_}, MATRIX, false});
    }

    void load(const std::string &p, TensorMap &t) override {
        std::vector<DevTensor> in = {take(t, name(p, n_z_)), take(t, name(p, n_x_)), take(t, name(p, n_g_))};
        w_in_ = fuse_rows(*dev, in);
        if (bias_) {
            // one vector over the product's columns; g has no bias
            std::vector<DevTensor> bs = {take(t, name(p, n_z_ + n_bias_)), take(t, name(p, n_x_ + n_bias_)),
                                         dev->tensor(F32, {width_}, true)};
            for (auto &b : bs) b.shape = {b.numel(), 1};
            b_in_ = fuse_rows(*dev, bs);
        }
        w_o_ = take(t, name(p, n_o_));
    }

    size_t weight_bytes() const override { return w_in_.bytes() + w_o_.bytes() + b_in_.bytes(); }

    StateSpec state_spec() const override { return StateSpec{{width_}, F32}; }
    bool supports(StepKind) const override { return true; }
    bool graph_safe() const override { return true; }

    Stack forward(StepContext &ctx, const void *h, LayerCache &cache) override {
        Device &d = *ctx.dev;
        if (!cache.state || cache.state_spec.shape.size() != 1 || cache.state_spec.shape[0] != width_)
            fail(JB_LLM_EINVAL, "mingru: the cache holds no state of this mixer's width for the layer");
        long long n = ctx.n_rows;
        Stack P = ops::linear(d, h, ctx.dtype, n, hidden_, w_in_);
        Buf a = ops::mingru(d, P, 0, width_, bias_ ? (const float *)b_in_.ptr : nullptr, (float *)cache.state,
                            ctx.row_seq, ctx.seq_slot, ctx.n_seqs, ctx.kind == DECODE, ctx.dtype);
        P = Stack();
        return ops::linear(d, a.ptr, ctx.dtype, n, width_, w_o_);
    }

    Json info() const override {
        Json o = Json::object();
        o.set("width", width_);
        return o;
    }

private:
    long long hidden_, width_;
    bool bias_;
    std::string n_z_, n_x_, n_g_, n_o_, n_bias_;
    DevTensor w_in_, b_in_, w_o_;
};

// the most rows one sequence brings to the step (0 where the host does not know: a captured step)
long long longest(const StepContext &ctx) {
    long long m = 0;
    for (long long v : ctx.seq_len) m = std::max(m, v);
    return m;
}

// A selective state space mixer in Mamba-2's form (state-space duality): H heads of P values,
// a state of N x P values per head, G groups of heads that share B and C.
//
//   [z | x | B | C | dt] = Win h        (H P, H P, G N, G N and H columns)
//   [x | B | C] <- silu(conv([x | B | C]) + b)      a causal convolution over time per column
//   dt <- softplus(dt + dt_bias)                    no clamp
//   S_t = exp(-exp(A_log_h) dt_t) S_{t-1} + dt_t B_t x_t^T;   y_t = S_t^T C_t + D_h x_t
//   out = Wo (rms in norm_groups equal parts of (y * silu(z)), times w)
//
// The state per sequence: the convolution's last taps - 1 inputs, then S, both float32.
// The steps, decays, exponentials, the recurrence and the norm are float32 in both compute
// types; what goes into Wo is rounded to the compute type.
//
// params: hidden_size, heads, head_dim (P), state (N), groups, conv_taps, norm_groups, eps,
// names (optional): in, conv, conv_bias, dt_bias, a_log, d, norm, o
class Mamba2 : public Mixer {
public:
    Mamba2(const PartSpec &s, DType dt, Device *d) : Mixer(s, dt, d) {
        hidden_ = s.get_int("hidden_size");
        H_ = s.get_int("heads");
        P_ = s.get_int("head_dim");
        N_ = s.get_int("state");
        G_ = s.get_int("groups", 1);
        taps_ = (int)s.get_int("conv_taps", 1);
        parts_ = s.get_int("norm_groups", 1);
        eps_ = (float)s.get_double("eps");
        if (hidden_ <= 0 || H_ <= 0 || P_ <= 0 || N_ <= 0 || G_ <= 0) config_error("mamba2: sizes must be positive");
        if (H_ % G_) config_error("mamba2: heads must be a multiple of groups");
        if (N_ > 1024) config_error("mamba2: the recurrence's kernel takes states of up to 1024 rows");
        if (taps_ < 1) config_error("mamba2: conv_taps must be positive");
        inner_ = H_ * P_;
        if (parts_ <= 0 || inner_ % parts_) config_error("mamba2: norm_groups must divide heads * head_dim");
        conv_ = inner_ + 2 * G_ * N_;
        const Json &nm = s.params.get("names");
        auto leaf = [&](const char *key, const char *dflt) {
            return nm.is_object() && nm.get(key).is_string() ? nm.get(key).as_string() : std::string(dflt);
        };
        n_in_ = leaf("in", "in_proj.weight");
        n_conv_ = leaf("conv", "conv1d.weight");
        n_conv_b_ = leaf("conv_bias", "conv1d.bias");
        n_dtb_ = leaf("dt_bias", "dt_bias");
        n_alog_ = leaf("a_log", "A_log");
        n_d_ = leaf("d", "D");
        n_norm_ = leaf("norm", "norm.weight");
        n_o_ = leaf("o", "out_proj.weight");
    }

    void tensors(const std::string &p, TensorList &out) const override {
        out.emplace_back(name(p, n_in_), TensorSpec{{2 * inner_ + 2 * G_ * N_ + H_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_conv_), TensorSpec{{conv_, taps_}, PARAM, false, 0.25f, 0.25f});
        out.emplace_back(name(p, n_conv_b_), TensorSpec{{conv_}, PARAM, false, 0.0f, 0.1f});
        out.emplace_back(name(p, n_dtb_), TensorSpec{{H_}, PARAM, false, -1.0f, 0.5f});
        out.emplace_back(name(p, n_alog_), TensorSpec{{H_}, PARAM, false, 0.0f, 0.5f});
        out.emplace_back(name(p, n_d_), TensorSpec{{H_}, PARAM, false, 1.0f, 0.1f});
        out.emplace_back(name(p, n_norm_), TensorSpec{{inner_}, PARAM, false, 1.0f, 0.1f});
        out.emplace_back(name(p, n_o_), TensorSpec{{hidden_, inner_}, MATRIX, false});
    }

    void load(const std::string &p, TensorMap &t) override {
        w_in_ = take(t, name(p, n_in_));
        conv_w_ = take(t, name(p, n_conv_));
        conv_b_ = take(t, name(p, n_conv_b_));
        dt_bias_ = take(t, name(p, n_dtb_));
        a_log_ = take(t, name(p, n_alog_));
        d_ = take(t, name(p, n_d_));
        norm_ = take(t, name(p, n_norm_));
        w_o_ = take(t, name(p, n_o_));
    }

    size_t weight_bytes() const override {
        return w_in_.bytes() + w_o_.bytes() + conv_w_.bytes() + conv_b_.bytes() + dt_bias_.bytes() + a_log_.bytes() +
               d_.bytes() + norm_.bytes();
    }

    DevTensor *first_matrix() override { return w_in_ ? &w_in_ : nullptr; }
    void share_first_product(long long col0) override {
        shared_ = true;
        col0_ = col0;
    }

    long long conv_state() const { return (long long)(taps_ - 1) * conv_; }
    StateSpec state_spec() const override { return StateSpec{{conv_state() + H_ * N_ * P_}, F32}; }
    bool strided_state() const override { return true; }
    bool graph_safe() const override { return true; }

    Stack forward(StepContext &ctx, const void *h, LayerCache &cache) override {
        Device &d = *ctx.dev;
        if (!cache.state || cache.state_spec.bytes() < state_spec().bytes())
            fail(JB_LLM_EINVAL, "mamba2: the cache holds no state of this mixer's size for the layer");
        long long n = ctx.n_rows;
        long long stride = cache.state_stride > 0 ? cache.state_stride : state_spec().shape[0];
        float *st = (float *)cache.state;
        Stack own;
        if (!shared_) own = ops::linear(d, h, ctx.dtype, n, hidden_, w_in_);
        else if (!ctx.shared) fail(JB_LLM_EFAIL, "mamba2: the shared first product is missing");
        const Stack &P = shared_ ? *ctx.shared : own;
        const long long c0 = shared_ ? col0_ : 0;
        // [x | B | C] through the convolution and silu, float32
        Stack xbc;
        xbc.S = 1;
        xbc.n = n;
        xbc.m = conv_;
        bool two = ctx.kind == EXTEND && taps_ > 1;
        xbc.buf = ops::causal_conv(d, P, c0 + inner_, conv_, (const float *)conv_w_.ptr, (const float *)conv_b_.ptr, taps_,
                                   st, stride, ctx.row_pos, ctx.row_seq, ctx.seq_slot, true, F32, true, !two);
        if (two)
            ops::causal_conv(d, P, c0 + inner_, conv_, (const float *)conv_w_.ptr, (const float *)conv_b_.ptr, taps_, st,
                             stride, ctx.row_pos, ctx.row_seq, ctx.seq_slot, true, F32, false, true);
        ops::MatrixScan m;
        m.H = (int)H_;
        m.G = (int)G_;
        m.N = (int)N_;
        m.P = (int)P_;
        m.val_col0 = 0;
        m.key_col0 = inner_;
        m.qry_col0 = inner_ + G_ * N_;
        m.dt = &P;
        m.dt_col0 = c0 + inner_ + conv_;
        m.dt_bias = (const float *)dt_bias_.ptr;
        m.a_log = (const float *)a_log_.ptr;
        m.skip = (const float *)d_.ptr;
        Buf y = ops::matrix_state_scan(d, xbc, m, st + conv_state(), stride, ctx.row_seq, ctx.seq_slot, ctx.n_seqs,
                                       ctx.kind == DECODE, longest(ctx));
        xbc = Stack();
        Buf a = ops::gated_part_norm(d, y.as<float>(), n, inner_, (int)parts_, &P, c0, nullptr, 0,
                                     (const float *)norm_.ptr, eps_, ctx.dtype, ctx.kind == DECODE && ctx.dtype == BF16);
        own = Stack();
        return ops::linear(d, a.ptr, ctx.dtype, n, inner_, w_o_);
    }

    Json info() const override {
        Json o = Json::object();
        o.set("inner", inner_);
        o.set("state_floats", state_spec().shape[0]);
        return o;
    }

private:
    long long hidden_, H_, P_, N_, G_, parts_, inner_ = 0, conv_ = 0;
    int taps_;
    float eps_;
    std::string n_in_, n_conv_, n_conv_b_, n_dtb_, n_alog_, n_d_, n_norm_, n_o_;
    DevTensor w_in_, w_o_, conv_w_, conv_b_, dt_bias_, a_log_, d_, norm_;
    bool shared_ = false;        // the in-product's rows went into a pair's shared first product
    long long col0_ = 0;
};

// Linear attention with a fixed decay per head (lightning attention's recurrence): H heads,
// D query/key values and Dv values a head, a state of D x Dv values per head.
//
//   q = silu(Wq h), k = silu(Wk h), v = silu(Wv h)       laid out head by head
//   S_t = decay_a S_{t-1} + k_t v_t^T;   o_t = S_t^T q_t          no other scale
//   out = Wo (rms(all heads of o) w * sigmoid(Wg h))
//
// q, k, v and the gate are one product over h; the recurrence, the state and the norm are
// float32 in both compute types.
//
// Retention's form of it ("Retentive Network: A Successor to Transformer for Large Language
// Models"), by the parameters activation, position, key_scale, head_norm and gate:
//   q = turn(Wq h), k = turn(Wk h) key_scale, v = Wv h
//   out = Wo (rms(each head of o) * silu(Wg h))           no weight in the norm
//
// params: hidden_size, heads, head_dim (D), v_head_dim (Dv, default D), decay (a list of one
// number per head), eps, activation ("silu", the default, or "none": of q, k and v), position (a
// part, rope_neox or none; absent: none; goes with activation none), key_scale (default 1; on k
// after the rotation; goes with activation none), head_norm (default false: one norm with a weight
// over all heads; true: each head by its own root mean square, no weight), gate ("sigmoid", the
// default, or "silu"), names (optional): q, k, v, g, o, norm
class DecayAttention : public Mixer {
public:
    DecayAttention(const PartSpec &s, DType dt, Device *d) : Mixer(s, dt, d) {
        hidden_ = s.get_int("hidden_size");
        H_ = s.get_int("heads");
        D_ = s.get_int("head_dim");
        Dv_ = s.get_int("v_head_dim", D_);
        eps_ = (float)s.get_double("eps");
        if (hidden_ <= 0 || H_ <= 0 || D_ <= 0 || Dv_ <= 0) config_error("decay_attention: sizes must be positive");
        if (D_ > 1024) config_error("decay_attention: the recurrence's kernel takes heads of up to 1024 values");
        const Json &dc = s.params.get("decay");
        if (!dc.is_array() || (long long)dc.size() != H_)
            config_error("decay_attention: decay must list one number per head");
        for (size_t i = 0; i < dc.size(); i++) {
            if (!dc[i].is_number()) config_error("decay_attention: decay must list numbers");
            decay_host_.push_back((float)dc[i].as_double());
        }
        auto word = [&](const char *key, const char *dflt) {
            return s.params.get(key).is_string() ? s.params.get(key).as_string() : std::string(dflt);
        };
        std::string act = word("activation", "silu"), gate = word("gate", "sigmoid");
        if (act != "silu" && act != "none") config_error("decay_attention: activation is silu or none");
        if (gate != "sigmoid" && gate != "silu") config_error("decay_attention: gate is sigmoid or silu");
        silu_ = act == "silu";
        gate_silu_ = gate == "silu";
        head_norm_ = s.has("head_norm") && s.params.get("head_norm").as_bool();
        key_scale_ = s.has("key_scale") ? (float)s.get_double("key_scale") : 1.0f;
        if (s.has("position")) position_ = build_position(s.get_part("position"), dt, d);
        bool turned = position_ && position_->rotary_dim() > 0;
        if (silu_ && (turned || key_scale_ != 1.0f))
            config_error("decay_attention: a rotation or a factor on the keys goes with activation none");
        if (turned && (position_->rotary_dim() > D_ || position_->pairs()))
            config_error("decay_attention: the rotation turns value i with value i + dims / 2, within a head");
        const Json &nm = s.params.get("names");
        auto leaf = [&](const char *key, const char *dflt) {
            return nm.is_object() && nm.get(key).is_string() ? nm.get(key).as_string() : std::string(dflt);
        };
        n_q_ = leaf("q", "q_proj.weight");
        n_k_ = leaf("k", "k_proj.weight");
        n_v_ = leaf("v", "v_proj.weight");
        n_g_ = leaf("g", "g_proj.weight");
        n_o_ = leaf("o", "o_proj.weight");
        n_norm_ = leaf("norm", "norm.weight");
    }

    void tensors(const std::string &p, TensorList &out) const override {
        out.emplace_back(name(p, n_q_), TensorSpec{{H_ * D_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_k_), TensorSpec{{H_ * D_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_v_), TensorSpec{{H_ * Dv_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_g_), TensorSpec{{H_ * Dv_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_o_), TensorSpec{{hidden_, H_ * Dv_}, MATRIX, false});
        if (!head_norm_) out.emplace_back(name(p, n_norm_), TensorSpec{{H_ * Dv_}, PARAM, false, 1.0f, 0.1f});
        if (position_) position_->tensors(name(p, "position"), out);
    }

    void load(const std::string &p, TensorMap &t) override {
        std::vector<DevTensor> in = {take(t, name(p, n_q_)), take(t, name(p, n_k_)), take(t, name(p, n_v_)),
                                     take(t, name(p, n_g_))};
        w_in_ = fuse_rows(*dev, in);
        w_o_ = take(t, name(p, n_o_));
        if (!head_norm_) norm_ = take(t, name(p, n_norm_));
        if (position_) position_->load(name(p, "position"), t);
        decay_ = dev->tensor(F32, {H_});
        cuda_check(cudaMemcpy(decay_.ptr, decay_host_.data(), decay_host_.size() * 4, cudaMemcpyHostToDevice),
                   "copying the heads' decays");
    }

    size_t weight_bytes() const override { return w_in_.bytes() + w_o_.bytes() + norm_.bytes() + decay_.bytes(); }

    DevTensor *first_matrix() override { return w_in_ ? &w_in_ : nullptr; }
    void share_first_product(long long col0) override {
        shared_ = true;
        col0_ = col0;
    }

    void prepare(long long n_positions) override {
        if (position_) position_->prepare(n_positions);
    }
    StateSpec state_spec() const override { return StateSpec{{H_ * D_ * Dv_}, F32}; }
    bool strided_state() const override { return true; }
    bool graph_safe() const override { return true; }

    Stack forward(StepContext &ctx, const void *h, LayerCache &cache) override {
        Device &d = *ctx.dev;
        if (!cache.state || cache.state_spec.bytes() < state_spec().bytes())
            fail(JB_LLM_EINVAL, "decay_attention: the cache holds no state of this mixer's size for the layer");
        long long n = ctx.n_rows;
        long long stride = cache.state_stride > 0 ? cache.state_stride : state_spec().shape[0];
        Stack own;
        if (!shared_) own = ops::linear(d, h, ctx.dtype, n, hidden_, w_in_);
        else if (!ctx.shared) fail(JB_LLM_EFAIL, "decay_attention: the shared first product is missing");
        const Stack &P = shared_ ? *ctx.shared : own;
        const long long c0 = shared_ ? col0_ : 0;
        int rot = position_ ? position_->rotary_dim() : 0;
        if (rot > 0 && ctx.max_pos >= position_->n_positions())
            fail(JB_LLM_EINVAL, fmt("position %lld is beyond the %lld positions the encoding was prepared "
                                    "for", ctx.max_pos, position_->n_positions()));
        ops::MatrixScan m;
        m.H = (int)H_;
        m.G = (int)H_;
        m.N = (int)D_;
        m.P = (int)Dv_;
        m.qry_col0 = c0;
        m.key_col0 = c0 + H_ * D_;
        m.val_col0 = c0 + 2 * H_ * D_;
        m.silu = silu_;
        m.decay = (const float *)decay_.ptr;
        // Many rows: q, k and v are activated once, ahead of the recurrence, whose blocks would
        // otherwise each activate the rows they read (several blocks read the same k and q).
        Stack act;
        if (rot > 0 || key_scale_ != 1.0f) {
            // the turned and scaled q and k (and v) in float32
            act = ops::turn_heads(d, P, c0, (int)H_, D_, Dv_, rot ? position_->cos() : nullptr,
                                  rot ? position_->sin() : nullptr, rot / 2, ctx.row_pos, key_scale_);
        } else if (silu_ && ctx.kind != DECODE && n >= 64) {
            act.buf = ops::activation(d, P, 2 * H_ * D_ + H_ * Dv_, ops::activation_kind("silu"), F32, c0);
            act.S = 1;
            act.n = n;
            act.m = 2 * H_ * D_ + H_ * Dv_;
            m.silu = false;
        }
        if (act) {
            m.qry_col0 = 0;
            m.key_col0 = H_ * D_;
            m.val_col0 = 2 * H_ * D_;
        }
        Buf y = ops::matrix_state_scan(d, act ? act : P, m, (float *)cache.state, stride, ctx.row_seq, ctx.seq_slot,
                                       ctx.n_seqs, ctx.kind == DECODE, longest(ctx));
        act = Stack();
        Buf a = ops::gated_part_norm(d, y.as<float>(), n, H_ * Dv_, head_norm_ ? (int)H_ : 1, nullptr, 0, &P,
                                     c0 + 2 * H_ * D_ + H_ * Dv_, head_norm_ ? nullptr : (const float *)norm_.ptr, eps_,
                                     ctx.dtype, ctx.kind == DECODE && ctx.dtype == BF16, gate_silu_);
        own = Stack();
        return ops::linear(d, a.ptr, ctx.dtype, n, H_ * Dv_, w_o_);
    }

    Json info() const override {
        Json o = Json::object();
        o.set("state_floats", state_spec().shape[0]);
        return o;
    }

private:
    long long hidden_, H_, D_, Dv_;
    float eps_;
    std::vector<float> decay_host_;
    std::string n_q_, n_k_, n_v_, n_g_, n_o_, n_norm_;
    DevTensor w_in_, w_o_, norm_, decay_;
    bool silu_ = true, gate_silu_ = false, head_norm_ = false;
    float key_scale_ = 1.0f;
    std::unique_ptr<PositionEncoding> position_;
    bool shared_ = false;        // the [q | k | v | g] rows went into a pair's shared first product
    long long col0_ = 0;
};

// Matrix memory with exponential gates, mLSTM ("xLSTM: Extended Long Short-Term Memory"): H heads, D query/key
// values and Dv values a head, with c(z) = cap tanh(z / cap):
//
//   q = Wq h D^(-1/2), k = Wk h, v = Wv h;   i = c(Wi h + bi), f = log sigmoid(c(Wf h + bf))   one each per head
//   m_t = max(f + m_{t-1}, i), from 0;   a = e^(f + m_{t-1} - m_t), b = e^(i - m_t)
//   S_t = a S_{t-1} + b k_t v_t^T;   n_t = a n_{t-1} + b k_t
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + floor)
//   out = Wo (concat_heads(rms(o)) w * sigmoid(Wg h))
//
// q, k, v, the output gate and the two log gates are one product over h; the gates, the state
// [per head S | n, then all heads' m], the division and the norm are float32 in both compute types.
//
// params: hidden_size, heads, head_dim (D), v_head_dim (Dv, default D), gate_cap, eps, floor (default 1e-6),
// names (optional): q, k, v, g, i, f, bias (a suffix of i and f), o, norm
class MatrixLSTM : public Mixer {
public:
    MatrixLSTM(const PartSpec &s, DType dt, Device *d) : Mixer(s, dt, d) {
        hidden_ = s.get_int("hidden_size");
        H_ = s.get_int("heads");
        D_ = s.get_int("head_dim");
        Dv_ = s.get_int("v_head_dim", D_);
        eps_ = (float)s.get_double("eps");
        cap_ = (float)s.get_double("gate_cap");
        floor_ = s.has("floor") ? (float)s.get_double("floor") : 1e-6f;
        if (hidden_ <= 0 || H_ <= 0 || D_ <= 0 || Dv_ <= 0) config_error("mlstm: sizes must be positive");
        if (D_ > 1024) config_error("mlstm: the recurrence's kernel takes heads of up to 1024 query values");
        if (!(cap_ > 0.0f)) config_error("mlstm: gate_cap must be positive");
        const Json &nm = s.params.get("names");
        auto leaf = [&](const char *key, const char *dflt) {
            return nm.is_object() && nm.get(key).is_string() ? nm.get(key).as_string() : std::string(dflt);
        };
        n_q_ = leaf("q", "q_proj.weight");
        n_k_ = leaf("k", "k_proj.weight");
        n_v_ = leaf("v", "v_proj.weight");
        n_g_ = leaf("g", "g_proj.weight");
        n_i_ = leaf("i", "i_proj");
        n_f_ = leaf("f", "f_proj");
        n_bias_ = leaf("bias", ".bias");
        n_o_ = leaf("o", "o_proj.weight");
        n_norm_ = leaf("norm", "norm.weight");
        i_col_ = 2 * H_ * D_ + 2 * H_ * Dv_;
    }

    void tensors(const std::string &p, TensorList &out) const override {
        out.emplace_back(name(p, n_q_), TensorSpec{{H_ * D_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_k_), TensorSpec{{H_ * D_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_v_), TensorSpec{{H_ * Dv_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_g_), TensorSpec{{H_ * Dv_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_i_), TensorSpec{{H_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_f_), TensorSpec{{H_, hidden_}, MATRIX, false});
        out.emplace_back(name(p, n_i_ + n_bias_), TensorSpec{{H_}, PARAM, false, 0.0f, 0.5f});
        out.emplace_back(name(p, n_f_ + n_bias_), TensorSpec{{H_}, PARAM, false, 3.0f, 1.0f});
        out.emplace_back(name(p, n_o_), TensorSpec{{hidden_, H_ * Dv_}, MATRIX, false});
        out.emplace_back(name(p, n_norm_), TensorSpec{{H_ * Dv_}, PARAM, false, 1.0f, 0.1f});
    }

    void load(const std::string &p, TensorMap &t) override {
        std::vector<DevTensor> in;
        for (const std::string *nm : {&n_q_, &n_k_, &n_v_, &n_g_, &n_i_, &n_f_}) in.push_back(take(t, name(p, *nm)));
        // rows of sums four to a load
        long long rows = i_col_ + 2 * H_;
        if (rows % 8) in.push_back(dev->tensor(in[0].dt, {8 - rows % 8, hidden_}, true));
        w_in_ = fuse_rows(*dev, in);
        i_bias_ = take(t, name(p, n_i_ + n_bias_));
        f_bias_ = take(t, name(p, n_f_ + n_bias_));
        w_o_ = take(t, name(p, n_o_));
        norm_ = take(t, name(p, n_norm_));
    }

    size_t weight_bytes() const override {
        return w_in_.bytes() + w_o_.bytes() + norm_.bytes() + i_bias_.bytes() + f_bias_.bytes();
    }

    DevTensor *first_matrix() override { return w_in_ ? &w_in_ : nullptr; }
    void share_first_product(long long col0) override {
        shared_ = true;
        col0_ = col0;
    }

    StateSpec state_spec() const override { return StateSpec{{H_ * (D_ * Dv_ + D_ + 1)}, F32}; }
    bool strided_state() const override { return true; }
    bool graph_safe() const override { return true; }

    Stack forward(StepContext &ctx, const void *h, LayerCache &cache) override {
        Device &d = *ctx.dev;
        if (!cache.state || cache.state_spec.bytes() < state_spec().bytes())
            fail(JB_LLM_EINVAL, "mlstm: the cache holds no state of this mixer's size for the layer");
        long long n = ctx.n_rows;
        long long stride = cache.state_stride > 0 ? cache.state_stride : state_spec().shape[0];
        Stack own;
        if (!shared_) own = ops::linear(d, h, ctx.dtype, n, hidden_, w_in_);
        else if (!ctx.shared) fail(JB_LLM_EFAIL, "mlstm: the shared first product is missing");
        const Stack &P = shared_ ? *ctx.shared : own;
        const long long c0 = shared_ ? col0_ : 0;
        ops::GatedMemory m;
        m.H = (int)H_;
        m.N = (int)D_;
        m.P = (int)Dv_;
        m.qry_col0 = c0;
        m.key_col0 = c0 + H_ * D_;
        m.val_col0 = c0 + 2 * H_ * D_;
        m.gate_col0 = m.val_col0 + H_ * Dv_;
        m.i_col0 = c0 + i_col_;
        m.f_col0 = m.i_col0 + H_;
        m.i_bias = (const float *)i_bias_.ptr;
        m.f_bias = (const float *)f_bias_.ptr;
        m.w = (const float *)norm_.ptr;
        m.cap = cap_;
        m.q_scale = (float)(1.0 / std::sqrt((double)D_));
        m.floor = floor_;
        m.eps = eps_;
        Buf a = ops::gated_memory(d, P, m, (float *)cache.state, stride, ctx.row_seq, ctx.seq_slot, ctx.n_seqs,
                                  ctx.kind == DECODE, longest(ctx), ctx.dtype);
        own = Stack();
        return ops::linear(d, a.ptr, ctx.dtype, n, H_ * Dv_, w_o_);
    }

    Json info() const override {
        Json o = Json::object();
        o.set("state_floats", state_spec().shape[0]);
        return o;
    }

private:
    long long hidden_, H_, D_, Dv_, i_col_ = 0;
    float eps_, cap_, floor_;
    std::string n_q_, n_k_, n_v_, n_g_, n_i_, n_f_, n_bias_, n_o_, n_norm_;
    DevTensor w_in_, w_o_, norm_, i_bias_, f_bias_;
    bool shared_ = false;        // the first product's rows went into a pair's shared one
    long long col0_ = 0;
};

// A recurrent block around a real-gated linear recurrent unit ("Griffin: Mixing Gated Linear Recurrences with
// Local Attention for Efficient Language Models"), W channels in `blocks` equal parts:
//
//   y = gelu_tanh(Wy h + by);   u = conv(Wx h + bx) + bc        a causal convolution over time per channel
//   in each part b:  r = sigmoid(Ra_b u_b + ra_b),  i = sigmoid(Ri_b u_b + ri_b)
//   log a = -8 r softplus(lam);   S_t = a S_{t-1} + sqrt(1 - a^2) i u;   out = Wo (S * y)
//
// The state per sequence: the convolution's last taps - 1 inputs (Wx h + bx), then S, both float32.  The two
// branches are one product over h, the gates one product per part over u in the compute type; u itself, the
// gates, decays and the recurrence are float32 in both compute types.
//
// params: hidden_size, width (W), blocks (default 1), conv_taps, names (optional): y, x, conv, r, i (the parts'
// matrices [blocks, W / blocks, W / blocks]), bias (a suffix of all five), lambda, o
class RealGatedLRU : public Mixer {
public:
    RealGatedLRU(const PartSpec &s, DType dt, Device *d) : Mixer(s, dt, d) {
        hidden_ = s.get_int("hidden_size");
        W_ = s.get_int("width");
        blocks_ = s.get_int("blocks", 1);
        taps_ = (int)s.get_int("conv_taps", 1);
        if (hidden_ <= 0 || W_ <= 0 || blocks_ <= 0) config_error("rglru: sizes must be positive");
        if (W_ % blocks_) config_error("rglru: blocks must divide width");
        if (taps_ < 1) config_error("rglru: conv_taps must be positive");
        part_ = W_ / blocks_;
        const Json &nm = s.params.get("names");
        auto leaf = [&](const char *key, const char *dflt) {
            return nm.is_object() && nm.get(key).is_string() ? nm.get(key).as_string() : std::string(dflt);
        };
        n_y_ = leaf("y", "y_proj");
        n_x_ = leaf("x", "x_proj");
        n_conv_ = leaf("conv", "conv1d");
        n_r_ = leaf("r", "r_gate");
        n_i_ = leaf("i", "i_gate");
        n_bias_ = leaf("bias", ".bias");
        n_lam_ = leaf("lambda", "lambda");
        n_o_ = leaf("o", "o_proj");
    }

    void tensors(const std::string &p, TensorList &out) const override {
        for (const std::string *nm : {&n_y_, &n_x_}) {
            out.emplace_back(name(p, *nm), TensorSpec{{W_, hidden_}, MATRIX, false});
            out.emplace_back(name(p, *nm + n_bias_), TensorSpec{{W_}, PARAM, false, 0.0f, 0.02f});
        }
        out.emplace_back(name(p, n_conv_), TensorSpec{{W_, taps_}, PARAM, false, 0.25f, 0.25f});
        out.emplace_back(name(p, n_conv_ + n_bias_), TensorSpec{{W_}, PARAM, false, 0.0f, 0.1f});
        for (const std::string *nm : {&n_r_, &n_i_}) {
            out.emplace_back(name(p, *nm), TensorSpec{{blocks_, part_, part_}, MATRIX, false});
            out.emplace_back(name(p, *nm + n_bias_), TensorSpec{{blocks_, part_}, PARAM, false, 0.0f, 0.5f});
        }
        out.emplace_back(name(p, n_lam_), TensorSpec{{W_}, PARAM, false, -4.0f, 1.5f});
        out.emplace_back(name(p, n_o_), TensorSpec{{hidden_, W_}, MATRIX, false});
    }

    void load(const std::string &p, TensorMap &t) override {
        std::vector<DevTensor> in = {take(t, name(p, n_y_)), take(t, name(p, n_x_))};
        w_in_ = fuse_rows(*dev, in);
        y_b_ = take(t, name(p, n_y_ + n_bias_));
        x_b_ = take(t, name(p, n_x_ + n_bias_));
        conv_w_ = take(t, name(p, n_conv_));
        conv_b_ = take(t, name(p, n_conv_ + n_bias_));
        // per part [r's rows | i's rows], all parts one after the other
        DevTensor r = take(t, name(p, n_r_)), i = take(t, name(p, n_i_));
        r.shape = i.shape = {blocks_, part_ * part_};
        std::vector<DevTensor> both = {r, i};
        r = i = DevTensor();
        w_gates_ = fuse_cols(*dev, both);
        w_gates_.shape = {blocks_ * 2 * part_, part_};
        r_b_ = take(t, name(p, n_r_ + n_bias_));
        i_b_ = take(t, name(p, n_i_ + n_bias_));
        lam_ = take(t, name(p, n_lam_));
        w_o_ = take(t, name(p, n_o_));
    }

    size_t weight_bytes() const override {
        return w_in_.bytes() + w_o_.bytes() + w_gates_.bytes() + conv_w_.bytes() + conv_b_.bytes() + y_b_.bytes() +
               x_b_.bytes() + r_b_.bytes() + i_b_.bytes() + lam_.bytes();
    }

    DevTensor *first_matrix() override { return w_in_ ? &w_in_ : nullptr; }
    void share_first_product(long long col0) override {
        shared_ = true;
        col0_ = col0;
    }

    long long conv_state() const { return (long long)(taps_ - 1) * W_; }
    StateSpec state_spec() const override { return StateSpec{{conv_state() + W_}, F32}; }
    bool strided_state() const override { return true; }
    bool graph_safe() const override { return true; }

    Stack forward(StepContext &ctx, const void *h, LayerCache &cache) override {
        Device &d = *ctx.dev;
        if (!cache.state || cache.state_spec.bytes() < state_spec().bytes())
            fail(JB_LLM_EINVAL, "rglru: the cache holds no state of this mixer's size for the layer");
        long long n = ctx.n_rows;
        long long stride = cache.state_stride > 0 ? cache.state_stride : state_spec().shape[0];
        float *st = (float *)cache.state;
        Stack own;
        if (!shared_) own = ops::linear(d, h, ctx.dtype, n, hidden_, w_in_);
        else if (!ctx.shared) fail(JB_LLM_EFAIL, "rglru: the shared first product is missing");
        const Stack &P = shared_ ? *ctx.shared : own;
        const long long c0 = shared_ ? col0_ : 0;
        // u in float32 for the recurrence, and part by part in the compute type for the gates
        Buf parts;
        bool two = ctx.kind == EXTEND && taps_ > 1;
        const float *cw = (const float *)conv_w_.ptr, *cb = (const float *)conv_b_.ptr, *xb = (const float *)x_b_.ptr;
        Buf u = ops::causal_conv(d, P, c0 + W_, W_, cw, cb, taps_, st, stride, ctx.row_pos, ctx.row_seq, ctx.seq_slot,
                                 false, F32, true, !two, xb, &parts, ctx.dtype, part_);
        if (two)
            ops::causal_conv(d, P, c0 + W_, W_, cw, cb, taps_, st, stride, ctx.row_pos, ctx.row_seq, ctx.seq_slot, false,
                             F32, false, true, xb);
        ops::HeadStack G = ops::linear_heads(d, parts.ptr, ctx.dtype, (int)blocks_, n, part_, w_gates_);
        parts = Buf();
        ops::LruParams lp;
        lp.rb = (const float *)r_b_.ptr;
        lp.ib = (const float *)i_b_.ptr;
        lp.lam = (const float *)lam_.ptr;
        lp.yb = (const float *)y_b_.ptr;
        Buf a = ops::lru(d, G, lp, u.as<float>(), W_, P, c0, st + conv_state(), stride, ctx.row_seq, ctx.seq_slot,
                         ctx.n_seqs, ctx.kind == DECODE, longest(ctx), ctx.dtype);
        own = Stack();
        return ops::linear(d, a.ptr, ctx.dtype, n, W_, w_o_);
    }

    Json info() const override {
        Json o = Json::object();
        o.set("state_floats", state_spec().shape[0]);
        return o;
    }

private:
    long long hidden_, W_, blocks_, part_ = 0;
    int taps_;
    std::string n_y_, n_x_, n_conv_, n_r_, n_i_, n_bias_, n_lam_, n_o_;
    DevTensor w_in_, w_o_, w_gates_, conv_w_, conv_b_, y_b_, x_b_, r_b_, i_b_, lam_;
    bool shared_ = false;        // the first product's rows went into a pair's shared one
    long long col0_ = 0;
};

}  // namespace

void register_recurrent_mixers() {
    register_part("mixer", "mlstm", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new MatrixLSTM(s, dt, d));
    });
    register_part("mixer", "rglru", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new RealGatedLRU(s, dt, d));
    });
    register_part("mixer", "mamba2", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new Mamba2(s, dt, d));
    });
    register_part("mixer", "decay_attention", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new DecayAttention(s, dt, d));
    });
    register_part("mixer", "mingru", [](const PartSpec &s, DType dt, Device *d) {
        return std::unique_ptr<Part>(new MinGRU(s, dt, d));
    });
}

}  // namespace jb
