// Part kinds for decoders that mix windowed softmax attention with linear recurrences, one mixer a layer.
//
//   mixer   "windowed_attention"       grouped-query softmax attention with any of: biases on q, k and v, rotary positions
//                                      on the first entries of each head (pairs of neighbours, or halves), a sliding
//                                      window that keeps the sequence's first tokens in sight, a one in the softmax's
//                                      denominator, a gate on every element of the heads' output; its keys and values
//                                      may be another layer's
//           "gated_linear_attention"   a matrix state per head that fades by one factor per key channel and token (GLA)
//           "matrix_memory"            the matrix memory of xLSTM (mLSTM) as a mixer of its own
//
// Every size and constant is a parameter of the part.  Positions and angles, scores and softmax, gates of the recurrences,
// decays and their exponentials, the recurrent state, the heads' norms and the residual sum are 32-bit in both compute
// types; the matrix products run in the compute type.
#include <cmath>

#include "part_helpers.h"
#include "parts.h"

namespace sandy {
namespace {
using namespace part_helpers;

ops::StepSeqs seqs_of(const StepContext& ctx) { return ops::StepSeqs{ctx.n_tokens, ctx.n_seqs, ctx.token_seq, ctx.q_start, ctx.seq_slots}; }

HostTensor zeros(int64_t n) { return host_f32(alloc_f32((size_t)n), {n}); }

// ---- windowed attention ------------------------------------------------------------------------------------------
// Parameters: width, n_heads, n_kv_heads, qk_dim, v_dim, scale, bias (q, k and v), rot_dims, rot_base, rot_interleaved,
//   window (null: none), keep_first, unit_sink, out_gate, own_kv (false: no key/value projections; the layer call names
//   the cache entry of the layer whose keys and values are read, with write_cache off).
// Tensors: q, k, v, o ([out, in]); with bias q_bias, k_bias, v_bias; with out_gate gate [H * v_dim, width].
//
// Per token: q, k, v = W h + b; the first rot_dims entries of each query and key head turn by position * rot_base^(-2i / rot_dims);
//   query i sees key j <= i when i - j < window or j < keep_first; p = exp(s) / (1 + sum exp(s)) with unit_sink, softmax without;
//   x += W_o (heads * sigmoid(W_gate h)), the gate element by element.
// Keys (turned) and values live in pages whose head size is the larger of qk_dim and v_dim rounded up to 16, zeros beyond
// each one's own size.  q, k, v and the gate are one product; the gate's sigmoid and product run in the attention kernels'
// write-back.
class WindowedAttention : public Mixer {
public:
    explicit WindowedAttention(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), H_((int)s.get_int("n_heads")), G_((int)s.get_int("n_kv_heads", s.get_int("n_heads"))),
          d_((int)s.get_int("qk_dim")), e_((int)s.get_int("v_dim")), scale_((float)s.get_double("scale")), bias_(s.get_bool("bias", false)),
          rot_dims_((int)s.get_int("rot_dims", 0)), interleaved_(s.get_bool("rot_interleaved", false)),
          window_((int)s.get_optional_int("window").value_or(0)), keep_((int)s.get_int("keep_first", 0)),
          unit_sink_(s.get_bool("unit_sink", false)), out_gate_(s.get_bool("out_gate", false)), own_kv_(s.get_bool("own_kv", true)),
          pad_((int)round_up(std::max(d_, e_), 16)), kv_cols_(own_kv_ ? (int64_t)G_ * (d_ + e_) : 0),
          n_wide_((int64_t)H_ * d_ + kv_cols_ + (out_gate_ ? (int64_t)H_ * e_ : 0)),
          wide_(width_, n_wide_, bias_, "out_in", "wide"), out_((int64_t)H_ * pad_, width_, false, "out_in", "out") {
        if (G_ <= 0 || H_ <= 0 || H_ % G_)
            throw ConfigError("windowed_attention: " + std::to_string(H_) + " heads do not divide into " + std::to_string(G_) + " key/value heads");
        if (d_ <= 0 || e_ <= 0 || pad_ > ops::kMaxHeadDim)
            throw ConfigError("windowed_attention: head sizes must be 1 .. " + std::to_string(ops::kMaxHeadDim));
        if (rot_dims_ < 0 || rot_dims_ > d_ || rot_dims_ % 2) throw ConfigError("windowed_attention: rot_dims must be even and at most qk_dim");
        if (window_ < 0 || keep_ < 0) throw ConfigError("windowed_attention: window and keep_first must not be negative");
        if (rot_dims_) freq_host_ = rotary_frequencies(rot_dims_, s.get_double("rot_base"), nullptr);
    }
    TensorRequests requests() const override {
        TensorRequests r;
        r["q"] = want({(int64_t)H_ * d_, width_});
        if (bias_) r["q_bias"] = want({(int64_t)H_ * d_}, "bias");
        if (own_kv_) {
            r["k"] = want({(int64_t)G_ * d_, width_});
            r["v"] = want({(int64_t)G_ * e_, width_});
            if (bias_) {
                r["k_bias"] = want({(int64_t)G_ * d_}, "bias");
                r["v_bias"] = want({(int64_t)G_ * e_}, "bias");
            }
        }
        if (out_gate_) r["gate"] = want({(int64_t)H_ * e_, width_});
        r["o"] = want({width_, (int64_t)H_ * e_});
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        std::vector<const HostTensor*> rows{&t.at("q")}, offsets;
        const HostTensor none = zeros((int64_t)H_ * e_);
        if (bias_) offsets.push_back(&t.at("q_bias"));
        if (own_kv_) {
            rows.push_back(&t.at("k"));
            rows.push_back(&t.at("v"));
            if (bias_) {
                offsets.push_back(&t.at("k_bias"));
                offsets.push_back(&t.at("v_bias"));
            }
        }
        if (out_gate_) {
            rows.push_back(&t.at("gate"));
            if (bias_) offsets.push_back(&none);
        }
        TensorMap m;
        m["wide.weight"] = stack_rows(rows, width_);
        if (bias_) {
            HostTensor b = stack_rows(offsets, 1);
            b.shape = {n_wide_};
            m["wide.bias"] = b;
        }
        m["out.weight"] = join_columns({{&t.at("o"), (int64_t)H_ * e_, e_, pad_}}, width_, (int64_t)H_ * pad_);
        wide_.bind(m, dtype);
        out_.bind(m, dtype);
        if (rot_dims_) freq_ = floats_to_device(freq_host_);
        if (unit_sink_) sink_ = floats_to_device(std::vector<float>((size_t)H_, 0.0f));      // exp(0) joins the denominator
    }
    size_t weight_bytes() const override { return wide_.weight_bytes() + out_.weight_bytes(); }
    CacheSpec cache_spec() const override { return CacheSpec::paged(G_, pad_, window_, keep_); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        if (call.write_cache != own_kv_) throw ConfigError("windowed_attention: a layer writes its cache entry when it has keys and values of its own");
        const int64_t T = h.rows();
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        Tensor wide = ws.get("mix_wide", T, n_wide_, ctx.compute_dtype);
        wide_.run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        const KVView cache = ctx.caches->kv(call.cache);
        const int* table = ctx.block_tables.at((size_t)cache.group);
        Tensor q = ws.get("mix_q", T, (int64_t)H_ * pad_, ctx.compute_dtype);
        ops::AttentionPrepare p;
        p.n_heads = H_; p.n_kv_heads = G_; p.qk_dim = d_; p.v_dim = e_;
        p.q_off = 0; p.k_off = H_ * d_; p.v_off = (H_ + G_) * d_;
        p.freq = rot_dims_ ? (const float*)freq_.view.data : nullptr;
        p.rot_dims = rot_dims_;
        p.interleaved = interleaved_;
        p.write_cache = call.write_cache;
        ops::attention_prepare(l, p, wide, cache, table, ctx.max_blocks, ctx.token_seq, ctx.positions, q);
        Tensor heads = ws.get("mix_heads", T, (int64_t)H_ * pad_, ctx.compute_dtype);
        ops::AttentionExtras extras;
        extras.sink = unit_sink_ ? (const float*)sink_.view.data : nullptr;
        extras.keep_first = keep_;
        Tensor gate;
        if (out_gate_) {
            gate = wide.col_range(n_wide_ - (int64_t)H_ * e_, n_wide_);
            extras.elem_gate = &gate;
        }
        ops::attention(l, ctx.attention_step(cache.group, window_, keep_), q, cache, heads, H_, scale_, window_, ws, &extras);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    int64_t width_;
    int H_, G_, d_, e_;
    float scale_;
    bool bias_;
    int rot_dims_;
    bool interleaved_;
    int window_, keep_;
    bool unit_sink_, out_gate_, own_kv_;
    int pad_;
    int64_t kv_cols_, n_wide_;
    Linear wide_, out_;
    std::vector<float> freq_host_;
    DeviceWeight freq_, sink_;
};

// ---- gated linear attention ----------------------------------------------------------------------------------------
// Parameters: width, eps, n_heads, qk_dim, v_dim, tau, rank (0 or absent: as the tensors have).
// Tensors: q, k [H * qk_dim, width], v, gate [H * v_dim, width], o [width, H * v_dim], norm [v_dim] (shared by the heads),
//   decay_in [rank, width], decay_out [H * qk_dim, rank], decay_bias [H * qk_dim].
//
// Per token: q = W_q h * qk_dim^(-1/2), k = W_k h, v = W_v h; alpha = sigmoid(W_out (W_in h) + bias)^(1 / tau), one per key
//   channel; per head S <- diag(alpha) S + k v^T, o = S^T q (csrc/gated_linear.cu); o over its root mean square, times the
//   gain, times silu(W_gate h); x += W_o [heads].
// W_in h is a product of its own, written in float32; the second, small one runs in 32-bit inside the recurrence's kernels.
// A request's state: S [H][v_dim][qk_dim].
class GatedLinearAttention : public Mixer {
public:
    explicit GatedLinearAttention(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), eps_((float)s.get_double("eps")), H_((int)s.get_int("n_heads")), d_((int)s.get_int("qk_dim")),
          e_((int)s.get_int("v_dim")), tau_(s.get_double("tau")), rank_(s.get_int("rank", 0)),
          n_wide_(2 * (int64_t)H_ * d_ + 2 * (int64_t)H_ * e_), wide_(width_, n_wide_, false, "out_in", "wide"),
          out_((int64_t)H_ * e_, width_, false, "out_in", "out") {
        if (H_ <= 0 || d_ <= 0 || e_ <= 0 || d_ > 256) throw ConfigError("gated_linear_attention: heads and head sizes must be positive, qk_dim at most 256");
        if (!(tau_ > 0)) throw ConfigError("gated_linear_attention: tau must be positive");
        if (rank_ < 0 || rank_ > 512) throw ConfigError("gated_linear_attention: the decay's rank is at most 512");
    }
    TensorRequests requests() const override {
        TensorRequests r;
        const int64_t rank = rank_ > 0 ? rank_ : -1;                   // as long as the file has it
        r["q"] = want({(int64_t)H_ * d_, width_});
        r["k"] = want({(int64_t)H_ * d_, width_});
        r["v"] = want({(int64_t)H_ * e_, width_});
        r["gate"] = want({(int64_t)H_ * e_, width_});
        r["o"] = want({width_, (int64_t)H_ * e_});
        r["norm"] = want({(int64_t)e_}, "gamma");
        r["decay_in"] = want({rank, width_});
        r["decay_out"] = want({(int64_t)H_ * d_, rank});
        r["decay_bias"] = want({(int64_t)H_ * d_}, "bias");
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        const int64_t rank = t.at("decay_in").shape.at(0), HD = (int64_t)H_ * d_;
        if (rank < 1 || rank > 512 || t.at("decay_out").shape.at(1) != rank)
            throw ConfigError("gated_linear_attention: the decay's two matrices must share a rank of 1 .. 512, got " + std::to_string(rank) + " and " +
                              std::to_string(t.at("decay_out").shape.at(1)));
        TensorMap m;
        m["wide.weight"] = stack_rows({&t.at("q"), &t.at("k"), &t.at("v"), &t.at("gate")}, width_);
        m["out.weight"] = t.at("o");
        m["low.weight"] = t.at("decay_in");
        wide_.bind(m, dtype);
        out_.bind(m, dtype);
        low_.reset(new Linear(width_, rank, false, "out_in", "low"));
        low_->bind(m, dtype);
        const std::vector<float> a2 = to_f32(t.at("decay_out"));
        auto turned = alloc_f32((size_t)(rank * HD));                  // [rank, H * qk_dim]: neighbouring channels side by side
        for (int64_t c = 0; c < HD; c++)
            for (int64_t r = 0; r < rank; r++) turned.get()[r * HD + c] = a2[(size_t)(c * rank + r)];
        w2t_ = to_device(host_f32(turned, {rank, HD}), DType::F32);
        bias_ = to_device(t.at("decay_bias"), DType::F32);
        gain_ = to_device(t.at("norm"), DType::F32);
    }
    size_t weight_bytes() const override {
        return wide_.weight_bytes() + out_.weight_bytes() + (low_ ? low_->weight_bytes() : 0) + w2t_.bytes() + bias_.bytes();
    }
    CacheSpec cache_spec() const override { return CacheSpec::state({ops::gla_state_floats(shape())}); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        const int64_t T = h.rows();
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        Tensor wide = ws.get("mix_wide", T, n_wide_, ctx.compute_dtype);
        wide_.run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        Tensor low = ws.get("mix_gates", T, w2t_.view.rows, DType::F32);
        low_->run(ctx, &h, nullptr, low, ops::Act::None, nullptr);
        Tensor read = ws.get("mix_read", T, (int64_t)H_ * e_, DType::F32);
        ops::gla_scan(l, seqs_of(ctx), shape(), wide, low, w2t_.view, bias_.view, ctx.caches->state(call.cache), read, ctx.max_q_len, ws);
        Tensor heads = ws.get("mix_heads", T, (int64_t)H_ * e_, ctx.compute_dtype);
        Tensor gate = wide.col_range(n_wide_ - (int64_t)H_ * e_, n_wide_);
        ops::head_norm_gate(l, read, &gain_.view, &gate, ops::GateAct::Silu, 1.0f, eps_, H_, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    ops::GlaShape shape() const {
        ops::GlaShape m;
        m.n_heads = H_; m.qk_dim = d_; m.v_dim = e_;
        m.q_off = 0; m.k_off = H_ * d_; m.v_off = 2 * H_ * d_;
        m.inv_tau = (float)(1.0 / tau_);
        m.q_scale = 1.0f / std::sqrt((float)d_);
        return m;
    }
    int64_t width_;
    float eps_;
    int H_, d_, e_;
    double tau_;
    int64_t rank_, n_wide_;
    Linear wide_, out_;
    std::unique_ptr<Linear> low_;
    DeviceWeight w2t_, bias_, gain_;
};

// ---- matrix memory -----------------------------------------------------------------------------------------------------
// Parameters: width, eps, n_heads, qk_dim, v_dim, gate_cap.
// Tensors: q, k [H * qk_dim, width], v, gate [H * v_dim, width], o [width, H * v_dim], norm [H * v_dim], i, f [H, width],
//   i_bias, f_bias [H].
//
// Per token and head: log i = cap tanh((w_i . h + b_i) / cap), log f = logsigmoid(cap tanh((w_f . h + b_f) / cap)); the
//   matrix memory's recurrence (csrc/matrix_state.cu) on q / sqrt(qk_dim), k, v; the read-out over its root mean square, times
//   the gain, times sigmoid(W_gate h); x += W_o [heads].  The gates' pre-activations are a product of their own, in float32.
class MatrixMemory : public Mixer {
public:
    explicit MatrixMemory(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), eps_((float)s.get_double("eps")), H_((int)s.get_int("n_heads")), d_((int)s.get_int("qk_dim")),
          e_((int)s.get_int("v_dim")), cap_((float)s.get_double("gate_cap")), n_wide_(2 * (int64_t)H_ * d_ + 2 * (int64_t)H_ * e_),
          wide_(width_, n_wide_, false, "out_in", "wide"), gates_(width_, 2 * (int64_t)H_, false, "out_in", "gates"),
          out_((int64_t)H_ * e_, width_, false, "out_in", "out") {
        if (H_ <= 0 || d_ <= 0 || e_ <= 0 || d_ > 256) throw ConfigError("matrix_memory: heads and head sizes must be positive, qk_dim at most 256");
        if (!(cap_ > 0)) throw ConfigError("matrix_memory: gate_cap must be positive");
    }
    TensorRequests requests() const override {
        TensorRequests r;
        r["q"] = want({(int64_t)H_ * d_, width_});
        r["k"] = want({(int64_t)H_ * d_, width_});
        r["v"] = want({(int64_t)H_ * e_, width_});
        r["gate"] = want({(int64_t)H_ * e_, width_});
        r["o"] = want({width_, (int64_t)H_ * e_});
        r["norm"] = want({(int64_t)H_ * e_}, "gamma");
        r["i"] = want({(int64_t)H_, width_});
        r["i_bias"] = want({(int64_t)H_}, "bias");
        r["f"] = want({(int64_t)H_, width_});
        r["f_bias"] = want({(int64_t)H_}, "bias");
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        TensorMap m;
        m["wide.weight"] = stack_rows({&t.at("q"), &t.at("k"), &t.at("v"), &t.at("gate")}, width_);
        m["gates.weight"] = stack_rows({&t.at("i"), &t.at("f")}, width_);
        m["out.weight"] = t.at("o");
        wide_.bind(m, dtype);
        gates_.bind(m, dtype);
        out_.bind(m, dtype);
        gate_bias_ = to_device(stack_rows({&t.at("i_bias"), &t.at("f_bias")}, 1), DType::F32);
        gain_ = to_device(t.at("norm"), DType::F32);
    }
    size_t weight_bytes() const override { return wide_.weight_bytes() + gates_.weight_bytes() + out_.weight_bytes(); }
    CacheSpec cache_spec() const override { return CacheSpec::state({ops::mlstm_state_floats(H_, d_, e_)}); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        const int64_t T = h.rows();
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        Tensor wide = ws.get("mix_wide", T, n_wide_, ctx.compute_dtype);
        wide_.run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        Tensor gates = ws.get("mix_gates", T, 2 * (int64_t)H_, DType::F32);
        gates_.run(ctx, &h, nullptr, gates, ops::Act::None, nullptr);
        ops::MlstmShape ms;
        ms.n_heads = H_; ms.qk_dim = d_; ms.v_dim = e_;
        ms.q_off = 0; ms.k_off = H_ * d_; ms.v_off = 2 * H_ * d_;
        ms.cap = cap_;
        ms.q_scale = 1.0f / std::sqrt((float)d_);
        Tensor read = ws.get("mix_read", T, (int64_t)H_ * e_, DType::F32);
        ops::mlstm_scan(l, seqs_of(ctx), ms, wide, gates, (const float*)gate_bias_.view.data, ctx.caches->state(call.cache), read, ctx.max_q_len);
        Tensor heads = ws.get("mix_heads", T, (int64_t)H_ * e_, ctx.compute_dtype);
        Tensor gate = wide.col_range(n_wide_ - (int64_t)H_ * e_, n_wide_);
        ops::head_norm_gate(l, read, &gain_.view, &gate, ops::GateAct::Sigmoid, 1.0f, eps_, H_, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    int64_t width_;
    float eps_;
    int H_, d_, e_;
    float cap_;
    int64_t n_wide_;
    Linear wide_, gates_, out_;
    DeviceWeight gate_bias_, gain_;
};

template <typename T>
PartFactory simple() {
    PartFactory f;
    f.make = [](const PartSpec& s) { return std::unique_ptr<Part>(new T(s)); };
    return f;
}

}  // namespace

void register_linear_parts() {
    register_part("mixer", "windowed_attention", simple<WindowedAttention>());
    register_part("mixer", "gated_linear_attention", simple<GatedLinearAttention>());
    register_part("mixer", "matrix_memory", simple<MatrixMemory>());
}

}  // namespace sandy
