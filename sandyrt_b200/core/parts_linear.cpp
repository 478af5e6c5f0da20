// Part kinds for decoders that mix windowed softmax attention with linear recurrences, one mixer a layer or two side by side.
//
//   mixer   "windowed_attention"       grouped-query softmax attention with any of: biases on q, k and v, rotary positions
//                                      on the first entries of each head (pairs of neighbours, or halves; YaRN's rescaling), a
//                                      sliding window that keeps the sequence's first tokens in sight, capped scores, a sink in
//                                      the softmax's denominator (a learned number per head, or a one), a gate on every element
//                                      of the heads' output; its keys and values may be another layer's, and its values its keys
//           "gated_linear_attention"   a matrix state per head that fades by one factor per key channel and token (GLA)
//           "matrix_memory"            the matrix memory of xLSTM (mLSTM) as a mixer of its own
//           "channel_delta"            the delta rule with a decay per key channel, behind short convolutions
//           "attention_beside_channel_delta"
//                                      the first and the one before on one input; result = left_scale * left + right_scale * right
//           "time_mixing"              a token shift with a mix of its own for every projection, a decay per key channel that
//                                      depends on the input, and a bonus for the current token (RWKV)
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

// The offsets of a product put together from several, one behind the other.
HostTensor join_offsets(const std::vector<HostTensor>& parts, int64_t n) {
    std::vector<const HostTensor*> p;
    for (const HostTensor& t : parts) p.push_back(&t);
    HostTensor b = stack_rows(p, 1);
    b.shape = {n};
    return b;
}

// [channels, rank] -> [rank, channels], float32: neighbouring channels side by side, as the recurrence's kernels read it.
DeviceWeight turned_to_device(const HostTensor& t) {
    const int64_t n = t.shape.at(0), rank = t.shape.at(1);
    const std::vector<float> v = to_f32(t);
    auto turned = alloc_f32((size_t)(rank * n));
    for (int64_t c = 0; c < n; c++)
        for (int64_t r = 0; r < rank; r++) turned.get()[r * n + c] = v[(size_t)(c * rank + r)];
    return to_device(host_f32(turned, {rank, n}), DType::F32);
}

// The rank two matrices of a low-rank product share, as the weight file has it.
int64_t shared_rank(const TensorMap& t, const std::string& in, const std::string& out, const std::string& who) {
    const int64_t rank = t.at(in).shape.at(0);
    if (rank < 1 || rank > 512 || t.at(out).shape.at(1) != rank)
        throw ConfigError(who + ": " + in + " and " + out + " must share a rank of 1 .. 512, got " + std::to_string(rank) + " and " +
                          std::to_string(t.at(out).shape.at(1)));
    return rank;
}

// ---- windowed attention ------------------------------------------------------------------------------------------
// Parameters: width, n_heads, n_kv_heads, qk_dim, v_dim, scale, bias (q, k and v), rot_dims, rot_base, rot_interleaved,
//   rot_yarn (null, or {factor, original, fast, slow}), window (null: none), keep_first, softcap (0: none), sink, unit_sink,
//   out_gate, own_kv (false: no key/value projections; the layer call names the cache entry of the layer whose keys and values
//   are read, with write_cache off), values_are_keys (no value projection: a value is its key as projected, before it turns).
// Tensors: q, k, v, o ([out, in]); with bias q_bias, k_bias, v_bias; with sink sink [H]; with out_gate gate [H * v_dim, width].
//
// Per token: q, k, v = W h + b; the first rot_dims entries of each query and key head turn by position * rot_base^(-2i / rot_dims),
//   under YaRN by rescaled frequencies and with cosine and sine times its magnitude;
//   score = (q . k) scale, then softcap * tanh(score / softcap); query i sees key j <= i when i - j < window or j < keep_first;
//   p = exp(s) / (exp(sink_h) + sum exp(s)), a one in place of exp(sink_h) with unit_sink, plain softmax without either;
//   x += W_o (heads * sigmoid(W_gate h)), the gate element by element.
// Keys (turned) and values live in pages whose head size is the larger of qk_dim and v_dim rounded up to 16, zeros beyond
// each one's own size.  q, k, v and the gate are one product; the gate's sigmoid and product run in the attention kernels'
// write-back.
//
// AttentionPath is everything of it but the two products, so that a mixer which runs something beside it can share them: its
// columns of the wide product (q | k | v | gate) and its columns of the output product's input.  `pre` goes in front of the
// names of its parameters and tensors; `head_scale` is a factor on every head's output.
class AttentionPath {
public:
    AttentionPath(const PartSpec& s, const std::string& pre, const std::string& who, float head_scale = 1.0f)
        : pre_(pre), who_(who), width_(s.get_int("width")), H_((int)s.get_int(pre + "n_heads")),
          G_((int)s.get_int(pre + "n_kv_heads", s.get_int(pre + "n_heads"))), d_((int)s.get_int(pre + "qk_dim")),
          e_((int)s.get_int(pre + "v_dim")), scale_((float)s.get_double(pre + "scale")), bias_(s.get_bool(pre + "bias", false)),
          rot_dims_((int)s.get_int(pre + "rot_dims", 0)), interleaved_(s.get_bool(pre + "rot_interleaved", false)),
          window_((int)s.get_optional_int(pre + "window").value_or(0)), keep_((int)s.get_int(pre + "keep_first", 0)),
          softcap_((float)s.get_double(pre + "softcap", 0.0)), has_sink_(s.get_bool(pre + "sink", false)),
          unit_sink_(s.get_bool(pre + "unit_sink", false)), out_gate_(s.get_bool(pre + "out_gate", false)),
          own_kv_(s.get_bool(pre + "own_kv", true)), v_is_k_(s.get_bool(pre + "values_are_keys", false)), head_scale_(head_scale),
          pad_((int)round_up(std::max(d_, e_), 16)) {
        if (G_ <= 0 || H_ <= 0 || H_ % G_)
            throw ConfigError(who_ + ": " + std::to_string(H_) + " heads do not divide into " + std::to_string(G_) + " key/value heads");
        if (d_ <= 0 || e_ <= 0 || pad_ > ops::kMaxHeadDim)
            throw ConfigError(who_ + ": head sizes must be 1 .. " + std::to_string(ops::kMaxHeadDim));
        if (rot_dims_ < 0 || rot_dims_ > d_ || rot_dims_ % 2) throw ConfigError(who_ + ": rot_dims must be even and at most qk_dim");
        if (window_ < 0 || keep_ < 0) throw ConfigError(who_ + ": window and keep_first must not be negative");
        if (softcap_ < 0.0f) throw ConfigError(who_ + ": softcap must not be negative");
        if (v_is_k_ && d_ != e_) throw ConfigError(who_ + ": values that are keys have the keys' size");
        if (has_sink_ && unit_sink_) throw ConfigError(who_ + ": a learned sink or a one, not both");
        if (rot_dims_) {
            const Json* yarn = s.params.find(pre + "rot_yarn");
            const double base = s.get_double(pre + "rot_base");
            freq_host_ = yarn && yarn->is_object() ? yarn_frequencies(rot_dims_, base, *yarn, rot_scale_) : rotary_frequencies(rot_dims_, base, nullptr);
        }
    }
    int64_t cols() const { return (int64_t)H_ * d_ + kv_cols() + (out_gate_ ? (int64_t)H_ * e_ : 0); }      // of the wide product
    int64_t head_cols() const { return (int64_t)H_ * pad_; }                                              // of the output product
    bool bias() const { return bias_; }
    void requests(TensorRequests& r) const {
        r[pre_ + "q"] = want({(int64_t)H_ * d_, width_});
        if (bias_) r[pre_ + "q_bias"] = want({(int64_t)H_ * d_}, "bias");
        if (own_kv_) {
            r[pre_ + "k"] = want({(int64_t)G_ * d_, width_});
            if (bias_) r[pre_ + "k_bias"] = want({(int64_t)G_ * d_}, "bias");
            if (!v_is_k_) {
                r[pre_ + "v"] = want({(int64_t)G_ * e_, width_});
                if (bias_) r[pre_ + "v_bias"] = want({(int64_t)G_ * e_}, "bias");
            }
        }
        if (has_sink_) r[pre_ + "sink"] = want({(int64_t)H_}, "bias");
        if (out_gate_) r[pre_ + "gate"] = want({(int64_t)H_ * e_, width_});
        r[pre_ + "o"] = want({width_, (int64_t)H_ * e_});
    }
    // Its rows of the wide product's matrix, and their offsets (with bias).
    void add_rows(const TensorMap& t, std::vector<const HostTensor*>& rows, std::vector<HostTensor>& offsets) const {
        auto add = [&](const std::string& name) {
            rows.push_back(&t.at(pre_ + name));
            if (bias_) offsets.push_back(t.at(pre_ + name + "_bias"));
        };
        add("q");
        if (own_kv_) add("k");
        if (own_kv_ && !v_is_k_) add("v");
        if (out_gate_) {
            rows.push_back(&t.at(pre_ + "gate"));
            if (bias_) offsets.push_back(zeros((int64_t)H_ * e_));
        }
    }
    ColumnPart out_columns(const TensorMap& t) const { return {&t.at(pre_ + "o"), (int64_t)H_ * e_, e_, pad_}; }
    void bind(const TensorMap& t) {
        if (rot_dims_) freq_ = floats_to_device(freq_host_);
        if (unit_sink_) sink_ = floats_to_device(std::vector<float>((size_t)H_, 0.0f));      // exp(0) joins the denominator
        if (has_sink_) sink_ = to_device(t.at(pre_ + "sink"), DType::F32);
    }
    CacheSpec cache_spec() const { return CacheSpec::paged(G_, pad_, window_, keep_); }
    CacheSpec cache_spec_with_state(int64_t floats) const {
        CacheSpec c = CacheSpec::paged_with_state(G_, pad_, window_, {floats});
        c.keep_first = keep_;
        return c;
    }
    // wide: its columns of the wide product; heads: [T, head_cols()], its columns of the output product's input.
    void run(StepContext& ctx, const Tensor& wide, const LayerCall& call, Tensor& heads) {
        if (call.write_cache != own_kv_) throw ConfigError(who_ + ": a layer writes its cache entry when it has keys and values of its own");
        const int64_t T = wide.rows;
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        const KVView cache = ctx.caches->kv(call.cache);
        const int* table = ctx.block_tables.at((size_t)cache.group);
        Tensor q = ws.get("mix_q", T, head_cols(), ctx.compute_dtype);
        ops::AttentionExtras extras;
        ops::AttentionPrepare p;
        p.n_heads = H_; p.n_kv_heads = G_; p.qk_dim = d_; p.v_dim = e_;
        p.q_off = 0; p.k_off = H_ * d_; p.v_off = v_is_k_ ? p.k_off : (H_ + G_) * d_;
        p.freq = rot_dims_ ? (const float*)freq_.view.data : nullptr;
        p.rot_dims = rot_dims_;
        p.interleaved = interleaved_;
        p.rot_scale = rot_scale_;
        p.write_cache = call.write_cache;
        if (head_scale_ != 1.0f) {
            Tensor factor = ws.get("mix_head_gate", T, H_, DType::F32);
            p.gate_out = (float*)factor.data;
            p.gate_scale = head_scale_;
            extras.out_gate = (const float*)factor.data;
        }
        ops::attention_prepare(l, p, wide, cache, table, ctx.max_blocks, ctx.token_seq, ctx.positions, q);
        extras.sink = has_sink_ || unit_sink_ ? (const float*)sink_.view.data : nullptr;
        extras.keep_first = keep_;
        extras.softcap = softcap_;
        Tensor gate;
        if (out_gate_) {
            gate = wide.col_range(cols() - (int64_t)H_ * e_, cols());
            extras.elem_gate = &gate;
        }
        ops::attention(l, ctx.attention_step(cache.group, window_, keep_), q, cache, heads, H_, scale_, window_, ws, &extras);
    }
private:
    int64_t kv_cols() const { return own_kv_ ? (int64_t)G_ * (d_ + (v_is_k_ ? 0 : e_)) : 0; }
    std::string pre_, who_;
    int64_t width_;
    int H_, G_, d_, e_;
    float scale_;
    bool bias_;
    int rot_dims_;
    bool interleaved_;
    int window_, keep_;
    float softcap_;
    bool has_sink_, unit_sink_, out_gate_, own_kv_, v_is_k_;
    float head_scale_;
    int pad_;
    float rot_scale_ = 1.0f;
    std::vector<float> freq_host_;
    DeviceWeight freq_, sink_;
};

class WindowedAttention : public Mixer {
public:
    explicit WindowedAttention(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), path_(s, "", "windowed_attention"), wide_(width_, path_.cols(), path_.bias(), "out_in", "wide"),
          out_(path_.head_cols(), width_, false, "out_in", "out") {}
    TensorRequests requests() const override {
        TensorRequests r;
        path_.requests(r);
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        std::vector<const HostTensor*> rows;
        std::vector<HostTensor> offsets;
        path_.add_rows(t, rows, offsets);
        TensorMap m;
        m["wide.weight"] = stack_rows(rows, width_);
        if (path_.bias()) m["wide.bias"] = join_offsets(offsets, path_.cols());
        m["out.weight"] = join_columns({path_.out_columns(t)}, width_, path_.head_cols());
        wide_.bind(m, dtype);
        out_.bind(m, dtype);
        path_.bind(t);
    }
    size_t weight_bytes() const override { return wide_.weight_bytes() + out_.weight_bytes(); }
    CacheSpec cache_spec() const override { return path_.cache_spec(); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        Workspace& ws = *ctx.workspace;
        Tensor wide = ws.get("mix_wide", h.rows(), path_.cols(), ctx.compute_dtype);
        wide_.run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        Tensor heads = ws.get("mix_heads", h.rows(), path_.head_cols(), ctx.compute_dtype);
        path_.run(ctx, wide, call, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    int64_t width_;
    AttentionPath path_;
    Linear wide_, out_;
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
        const int64_t rank = shared_rank(t, "decay_in", "decay_out", "gated_linear_attention");
        TensorMap m;
        m["wide.weight"] = stack_rows({&t.at("q"), &t.at("k"), &t.at("v"), &t.at("gate")}, width_);
        m["out.weight"] = t.at("o");
        m["low.weight"] = t.at("decay_in");
        wide_.bind(m, dtype);
        out_.bind(m, dtype);
        low_.reset(new Linear(width_, rank, false, "out_in", "low"));
        low_->bind(m, dtype);
        w2t_ = turned_to_device(t.at("decay_out"));
        bias_ = to_device(t.at("decay_bias"), DType::F32);
        gain_ = to_device(t.at("norm"), DType::F32);
    }
    size_t weight_bytes() const override {
        return wide_.weight_bytes() + out_.weight_bytes() + (low_ ? low_->weight_bytes() : 0) + w2t_.bytes() + bias_.bytes();
    }
    CacheSpec cache_spec() const override { return CacheSpec::state({ops::fade_state_floats(shape())}); }
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
        ops::fade_scan(l, seqs_of(ctx), shape(), wide, low, w2t_.view, bias_.view, ctx.caches->state(call.cache), read, ctx.max_q_len, ws);
        Tensor heads = ws.get("mix_heads", T, (int64_t)H_ * e_, ctx.compute_dtype);
        Tensor gate = wide.col_range(n_wide_ - (int64_t)H_ * e_, n_wide_);
        ops::head_norm_gate(l, read, &gain_.view, &gate, ops::GateAct::Silu, 1.0f, eps_, H_, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    ops::FadeShape shape() const {
        ops::FadeShape m;
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

// ---- the delta rule with a decay per key channel ---------------------------------------------------------------------
// Parameters: width, eps, n_heads, n_qk_heads, qk_dim, v_dim, conv_taps, rank and gate_rank (0 or absent: as the tensors have).
// Tensors: q, k [G * qk_dim, width], v [H * v_dim, width], q_conv, k_conv, v_conv ([channels, taps], the last column is the
//   current token's), beta [H, width], decay_in [rank, width], decay_out [H * qk_dim, rank], dt_bias [H * qk_dim], a_log [H],
//   gate_in [gate_rank, width], gate_out [H * v_dim, gate_rank], norm [v_dim] (shared by the heads), o [width, H * v_dim].
//
// Per token: q, k, v = W h, each through a short causal convolution over time per channel and silu; q and k become unit vectors
//   per head (x / sqrt(sum x^2 + 1e-6)), q also times qk_dim^(-1/2); head h reads query/key head h / (H / G);
//   g = exp(-exp(a_log_h) softplus(W_out (W_in h) + dt_bias)), one per head and key channel; per head S <- diag(g) S,
//   u = sigmoid(w_beta . h) (v - S^T k), S <- S + k u^T, o = S^T q (csrc/gated_linear.cu); o over its root mean square, times the
//   gain, times sigmoid(W_gate_out (W_gate_in h)); x += W_o [heads].
// W_in h and w_beta . h are one product, written in float32; W_gate_in h is a part of the wide product (its columns come first
// and are padded to a multiple of 8, so that they are an operand of W_gate_out as they lie).
// A request's state: S [H][v_dim][qk_dim], then the last conv_taps - 1 inputs of the convolutions.
//
// ChannelDeltaPath is everything of it but the wide and the output product; `scale` is a factor on every head's output.
class ChannelDeltaPath {
public:
    ChannelDeltaPath(const PartSpec& s, const std::string& pre, const std::string& who, float scale = 1.0f)
        : pre_(pre), who_(who), width_(s.get_int("width")), eps_((float)s.get_double("eps")), H_((int)s.get_int(pre + "n_heads")),
          G_((int)s.get_int(pre + "n_qk_heads", s.get_int(pre + "n_heads"))), d_((int)s.get_int(pre + "qk_dim")), e_((int)s.get_int(pre + "v_dim")),
          taps_((int)s.get_int(pre + "conv_taps")), rank_(s.get_int(pre + "rank", 0)), gate_rank_(s.get_int(pre + "gate_rank", 0)), scale_(scale) {
        if (G_ <= 0 || H_ <= 0 || H_ % G_)
            throw ConfigError(who_ + ": " + std::to_string(H_) + " heads do not divide into " + std::to_string(G_) + " query/key heads");
        if (taps_ < 1 || taps_ > 8) throw ConfigError(who_ + ": 1 to 8 convolution taps are supported, got " + std::to_string(taps_));
        if (d_ <= 0 || e_ <= 0 || d_ > 256) throw ConfigError(who_ + ": head sizes must be positive, qk_dim at most 256");
        if (rank_ < 0 || rank_ > 512 || gate_rank_ < 0) throw ConfigError(who_ + ": the decay's rank is at most 512");
    }
    int64_t channels() const { return 2 * (int64_t)G_ * d_ + (int64_t)H_ * e_; }      // of the convolutions: q, k, v
    int64_t head_cols() const { return (int64_t)H_ * e_; }
    int64_t gate_cols() const { return gate_pad_; }                                   // after bind
    int64_t state_floats() const { return (int64_t)H_ * e_ * d_ + (int64_t)(taps_ - 1) * channels(); }
    void requests(TensorRequests& r) const {
        const int64_t rank = rank_ > 0 ? rank_ : -1, gate_rank = gate_rank_ > 0 ? gate_rank_ : -1;      // -1: as long as the file has it
        r[pre_ + "q"] = want({(int64_t)G_ * d_, width_});
        r[pre_ + "k"] = want({(int64_t)G_ * d_, width_});
        r[pre_ + "v"] = want({(int64_t)H_ * e_, width_});
        r[pre_ + "q_conv"] = want({(int64_t)G_ * d_, taps_});
        r[pre_ + "k_conv"] = want({(int64_t)G_ * d_, taps_});
        r[pre_ + "v_conv"] = want({(int64_t)H_ * e_, taps_});
        r[pre_ + "beta"] = want({(int64_t)H_, width_});
        r[pre_ + "decay_in"] = want({rank, width_});
        r[pre_ + "decay_out"] = want({(int64_t)H_ * d_, rank});
        r[pre_ + "dt_bias"] = want({(int64_t)H_ * d_}, "bias");
        r[pre_ + "a_log"] = want({(int64_t)H_}, "bias");
        r[pre_ + "gate_in"] = want({gate_rank, width_});
        r[pre_ + "gate_out"] = want({(int64_t)H_ * e_, gate_rank});
        r[pre_ + "norm"] = want({(int64_t)e_}, "gamma");
        r[pre_ + "o"] = want({width_, (int64_t)H_ * e_});
    }
    void bind(const TensorMap& t, DType dtype) {
        const int64_t rank = shared_rank(t, pre_ + "decay_in", pre_ + "decay_out", who_);
        const int64_t gate_rank = shared_rank(t, pre_ + "gate_in", pre_ + "gate_out", who_);
        gate_pad_ = round_up(gate_rank, 8);
        TensorMap m;
        m["narrow.weight"] = stack_rows({&t.at(pre_ + "beta"), &t.at(pre_ + "decay_in")}, width_);
        m["gate.weight"] = join_columns({{&t.at(pre_ + "gate_out"), gate_rank, 0, 0}}, head_cols(), gate_pad_);
        narrow_.reset(new Linear(width_, H_ + rank, false, "out_in", "narrow"));
        gate_.reset(new Linear(gate_pad_, head_cols(), false, "out_in", "gate"));
        narrow_->bind(m, dtype);
        gate_->bind(m, dtype);
        conv_ = to_device(stack_rows({&t.at(pre_ + "q_conv"), &t.at(pre_ + "k_conv"), &t.at(pre_ + "v_conv")}, taps_), DType::F32);
        w2t_ = turned_to_device(t.at(pre_ + "decay_out"));
        dt_bias_ = to_device(t.at(pre_ + "dt_bias"), DType::F32);
        a_log_ = to_device(t.at(pre_ + "a_log"), DType::F32);
        gain_ = to_device(t.at(pre_ + "norm"), DType::F32);
    }
    // Rows of the wide product's matrix: the gate's first (gate_cols of them, behind every other mixer's none), then q, k, v.
    HostTensor gate_rows(const TensorMap& t) const {
        const HostTensor& g = t.at(pre_ + "gate_in");
        const HostTensor pad = zeros((gate_pad_ - g.shape.at(0)) * width_);
        return gate_pad_ == g.shape.at(0) ? g : stack_rows({&g, &pad}, width_);
    }
    void add_rows(const TensorMap& t, std::vector<const HostTensor*>& rows) const {
        for (const char* n : {"q", "k", "v"}) rows.push_back(&t.at(pre_ + n));
    }
    ColumnPart out_columns(const TensorMap& t) const { return {&t.at(pre_ + "o"), head_cols(), 0, 0}; }
    size_t weight_bytes() const {
        return narrow_ ? narrow_->weight_bytes() + gate_->weight_bytes() + w2t_.bytes() + dt_bias_.bytes() + conv_.bytes() : 0;
    }
    // gate_low: the gate's columns of the wide product; qkv: the q, k, v columns; heads: [T, head_cols()].
    void run(StepContext& ctx, NormedInput& h, const Tensor& gate_low, const Tensor& qkv, const LayerCall& call, Tensor& heads) {
        const int64_t T = h.rows(), tail_off = (int64_t)H_ * e_ * d_;
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        const StateView state = ctx.caches->state(call.cache);
        Tensor narrow = ws.get("mix_gates", T, H_ + w2t_.view.rows, DType::F32);
        narrow_->run(ctx, &h, nullptr, narrow, ops::Act::None, nullptr);
        Tensor gate = ws.get("delta_gate", T, head_cols(), ctx.compute_dtype);
        gate_->run(ctx, nullptr, &gate_low, gate, ops::Act::None, nullptr);
        Tensor acted = ws.get("delta_qkv", T, channels(), DType::F32);
        const ops::DeltaShape ds{H_, G_, d_, e_, taps_};
        ops::delta_prepare(l, seqs_of(ctx), ds, qkv, conv_.view, nullptr, nullptr, nullptr, state, tail_off, 1.0f / std::sqrt((float)d_), acted,
                           nullptr, ctx.max_q_len);
        if (ctx.max_q_len != 1) ops::conv_tail(l, seqs_of(ctx), ds, qkv, state, tail_off);
        const Tensor beta = narrow.col_range(0, H_), low = narrow.col_range(H_, narrow.cols);
        ops::FadeShape m;
        m.n_heads = H_; m.n_qk_heads = G_; m.qk_dim = d_; m.v_dim = e_;
        m.q_off = 0; m.k_off = G_ * d_; m.v_off = 2 * G_ * d_;
        m.kind = ops::FadeKind::Delta;
        m.decay = ops::DecayForm::Softplus;
        m.a_log = (const float*)a_log_.view.data;
        m.beta = &beta;
        Tensor read = ws.get("mix_read", T, head_cols(), DType::F32);
        ops::fade_scan(l, seqs_of(ctx), m, acted, low, w2t_.view, dt_bias_.view, state, read, ctx.max_q_len, ws);
        ops::head_norm_gate(l, read, &gain_.view, &gate, ops::GateAct::Sigmoid, scale_, eps_, H_, heads);
    }
private:
    std::string pre_, who_;
    int64_t width_;
    float eps_;
    int H_, G_, d_, e_, taps_;
    int64_t rank_, gate_rank_, gate_pad_ = 0;
    float scale_;
    std::unique_ptr<Linear> narrow_, gate_;
    DeviceWeight conv_, w2t_, dt_bias_, a_log_, gain_;
};

class ChannelDelta : public Mixer {
public:
    explicit ChannelDelta(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), path_(s, "", "channel_delta"), out_(path_.head_cols(), width_, false, "out_in", "out") {}
    TensorRequests requests() const override {
        TensorRequests r;
        path_.requests(r);
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        path_.bind(t, dtype);
        const HostTensor gate = path_.gate_rows(t);
        std::vector<const HostTensor*> rows{&gate};
        path_.add_rows(t, rows);
        n_wide_ = round_up(path_.gate_cols() + path_.channels(), 8);
        const HostTensor pad = zeros((n_wide_ - path_.gate_cols() - path_.channels()) * width_);
        rows.push_back(&pad);
        TensorMap m;
        m["wide.weight"] = stack_rows(rows, width_);
        m["out.weight"] = t.at("o");
        wide_.reset(new Linear(width_, n_wide_, false, "out_in", "wide"));
        wide_->bind(m, dtype);
        out_.bind(m, dtype);
    }
    size_t weight_bytes() const override { return (wide_ ? wide_->weight_bytes() : 0) + out_.weight_bytes() + path_.weight_bytes(); }
    CacheSpec cache_spec() const override { return CacheSpec::state({path_.state_floats()}); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        Workspace& ws = *ctx.workspace;
        Tensor wide = ws.get("mix_wide", h.rows(), n_wide_, ctx.compute_dtype);
        wide_->run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        Tensor heads = ws.get("mix_heads", h.rows(), path_.head_cols(), ctx.compute_dtype);
        path_.run(ctx, h, wide.col_range(0, path_.gate_cols()), wide.col_range(path_.gate_cols(), path_.gate_cols() + path_.channels()), call, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    int64_t width_, n_wide_ = 0;
    ChannelDeltaPath path_;
    std::unique_ptr<Linear> wide_;
    Linear out_;
};

// ---- attention beside the delta rule -----------------------------------------------------------------------------------
// Parameters: width, eps, left_scale, right_scale, "left." those of windowed_attention, "right." those of channel_delta.
// Tensors: "left." and "right." theirs.
//
// Both read the same input: one wide product gives [right's gate | left's q, k, (v), (gate) | right's q, k, v].  The result is
// left_scale * left + right_scale * right; the output projections are one product over [left heads | right heads], with the
// scales as factors on the heads, in 32-bit before they are rounded.
class AttentionBesideChannelDelta : public Mixer {
public:
    explicit AttentionBesideChannelDelta(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")),
          left_(s, "left.", "attention_beside_channel_delta", (float)s.get_double("left_scale", 1.0)),
          right_(s, "right.", "attention_beside_channel_delta", (float)s.get_double("right_scale", 1.0)),
          k_right_(round_up(right_.head_cols(), 8)), out_(left_.head_cols() + k_right_, width_, false, "out_in", "out") {}
    TensorRequests requests() const override {
        TensorRequests r;
        left_.requests(r);
        right_.requests(r);
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        left_.bind(t);
        right_.bind(t, dtype);
        const HostTensor gate = right_.gate_rows(t);
        std::vector<const HostTensor*> rows{&gate};
        std::vector<HostTensor> offsets{zeros(right_.gate_cols())};
        left_.add_rows(t, rows, offsets);
        right_.add_rows(t, rows);
        const int64_t n = right_.gate_cols() + left_.cols() + right_.channels();
        n_wide_ = round_up(n, 8);
        const HostTensor pad = zeros((n_wide_ - n) * width_);
        rows.push_back(&pad);
        TensorMap m;
        m["wide.weight"] = stack_rows(rows, width_);
        if (left_.bias()) {
            offsets.push_back(zeros(n_wide_ - right_.gate_cols() - left_.cols()));
            m["wide.bias"] = join_offsets(offsets, n_wide_);
        }
        m["out.weight"] = join_columns({left_.out_columns(t), right_.out_columns(t)}, width_, left_.head_cols() + k_right_);
        wide_.reset(new Linear(width_, n_wide_, left_.bias(), "out_in", "wide"));
        wide_->bind(m, dtype);
        out_.bind(m, dtype);
    }
    size_t weight_bytes() const override { return (wide_ ? wide_->weight_bytes() : 0) + out_.weight_bytes() + right_.weight_bytes(); }
    CacheSpec cache_spec() const override { return left_.cache_spec_with_state(right_.state_floats()); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        const int64_t T = h.rows(), g = right_.gate_cols(), l = left_.cols(), kl = left_.head_cols();
        Workspace& ws = *ctx.workspace;
        Tensor wide = ws.get("mix_wide", T, n_wide_, ctx.compute_dtype);
        wide_->run(ctx, &h, nullptr, wide, ops::Act::None, nullptr);
        Tensor heads = ws.get("mix_heads", T, kl + k_right_, ctx.compute_dtype);
        if (k_right_ != right_.head_cols())      // the columns that only pad the product must not hold stale numbers
            cuda_check(cudaMemsetAsync(heads.data, 0, (size_t)heads.numel() * heads.elem_size(), ctx.launch.stream), "clearing padded heads");
        Tensor o_left = heads.col_range(0, kl), o_right = heads.col_range(kl, kl + right_.head_cols());
        left_.run(ctx, wide.col_range(g, g + l), call, o_left);
        right_.run(ctx, h, wide.col_range(0, g), wide.col_range(g + l, g + l + right_.channels()), call, o_right);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    int64_t width_, n_wide_ = 0;
    AttentionPath left_;
    ChannelDeltaPath right_;
    int64_t k_right_;
    std::unique_ptr<Linear> wide_;
    Linear out_;
};

// ---- time mixing ---------------------------------------------------------------------------------------------------------
// Parameters: width, eps, n_heads, dim, rank (0 or absent: as the tensors have).
// Tensors: mu_r, mu_k, mu_v, mu_g, mu_w [width]; r, k, v, gate [H * dim, width]; decay_in [rank, width], decay_out [H * dim, rank],
//   decay_bias [H * dim]; bonus [H, dim]; norm [H * dim]; o [width, H * dim].
//
// Per token, h being the normed stream row and h' the token before's (zeros at a request's first token): every projection reads
//   its own m_s = h + (h' - h) mu_s; r, k, v = W m; w = exp(-exp(W_out tanh(W_in m_w) + decay_bias)), one per head and channel; per
//   head o = (S + diag(bonus) k v^T)^T r, then S <- diag(w) S + k v^T (csrc/gated_linear.cu); o over its root mean square, times the
//   gain, times silu(W_gate m_g); x += W_o [heads].
// The norm and all five mixes are one pass over the stream; r, k, v and the gate are one launch in a decode step; W_in m_w is
// written in float32.  A request's state: h of its last token, then S [H][dim][dim].
class TimeMixing : public Mixer {
public:
    explicit TimeMixing(const PartSpec& s)
        : Mixer(s), width_(s.get_int("width")), eps_((float)s.get_double("eps")), H_((int)s.get_int("n_heads")), d_((int)s.get_int("dim")),
          rank_(s.get_int("rank", 0)), wide_(width_, 4 * (int64_t)H_ * d_, false, "out_in", "wide"), out_((int64_t)H_ * d_, width_, false, "out_in", "out") {
        if (H_ <= 0 || d_ <= 0 || d_ > 256) throw ConfigError("time_mixing: heads and dim must be positive, dim at most 256");
        if (rank_ < 0 || rank_ > 512) throw ConfigError("time_mixing: the decay's rank is at most 512");
    }
    TensorRequests requests() const override {
        TensorRequests r;
        const int64_t n = (int64_t)H_ * d_, rank = rank_ > 0 ? rank_ : -1;
        for (const char* m : {"mu_r", "mu_k", "mu_v", "mu_g", "mu_w"}) r[m] = want({width_}, "bias");
        for (const char* m : {"r", "k", "v", "gate"}) r[m] = want({n, width_});
        r["decay_in"] = want({rank, width_});
        r["decay_out"] = want({n, rank});
        r["decay_bias"] = want({n}, "bias");
        r["bonus"] = want({H_, d_}, "bias");
        r["norm"] = want({n}, "gamma");
        r["o"] = want({width_, n});
        return r;
    }
    void bind(const TensorMap& t, DType dtype) override {
        const int64_t rank = shared_rank(t, "decay_in", "decay_out", "time_mixing");
        TensorMap m;
        m["wide.weight"] = stack_rows({&t.at("r"), &t.at("k"), &t.at("v"), &t.at("gate")}, width_);
        m["low.weight"] = t.at("decay_in");
        m["out.weight"] = t.at("o");
        wide_.bind(m, dtype);
        low_.reset(new Linear(width_, rank, false, "out_in", "low"));
        low_->bind(m, dtype);
        out_.bind(m, dtype);
        mix_ = to_device(stack_rows({&t.at("mu_r"), &t.at("mu_k"), &t.at("mu_v"), &t.at("mu_g"), &t.at("mu_w")}, width_), DType::F32);
        w2t_ = turned_to_device(t.at("decay_out"));
        bias_ = to_device(t.at("decay_bias"), DType::F32);
        bonus_ = to_device(t.at("bonus"), DType::F32);
        gain_ = to_device(t.at("norm"), DType::F32);
    }
    size_t weight_bytes() const override {
        return wide_.weight_bytes() + out_.weight_bytes() + (low_ ? low_->weight_bytes() : 0) + w2t_.bytes() + bias_.bytes() + mix_.bytes();
    }
    CacheSpec cache_spec() const override { return CacheSpec::state({width_ + ops::fade_state_floats(shape())}); }
    bool can_overwrite() const override { return true; }
    void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) override {
        const int64_t T = h.rows(), n = (int64_t)H_ * d_;
        Workspace& ws = *ctx.workspace;
        const ops::Launch& l = ctx.launch;
        const StateView state = ctx.caches->state(call.cache);
        RmsNormParams norm;
        if (!h.rms(norm)) throw ConfigError("time_mixing: the token shift needs an RMS norm in front of the mixer");
        Tensor mixed = ws.get("mix_shifted", T, 5 * width_, ctx.compute_dtype);
        ops::rmsnorm_shift(l, seqs_of(ctx), norm.x, norm.gain, norm.eps, mix_.view, state, mixed, ctx.max_q_len);
        Tensor wide = ws.get("mix_wide", T, 4 * n, ctx.compute_dtype);
        wide_.run_groups(ctx, mixed.col_range(0, 4 * width_), 4, wide);
        const Tensor for_decay = mixed.col_range(4 * width_, 5 * width_);
        Tensor low = ws.get("mix_gates", T, w2t_.view.rows, DType::F32);
        low_->run(ctx, nullptr, &for_decay, low, ops::Act::None, nullptr);
        Tensor read = ws.get("mix_read", T, n, DType::F32);
        ops::fade_scan(l, seqs_of(ctx), shape(), wide, low, w2t_.view, bias_.view, state, read, ctx.max_q_len, ws);
        Tensor heads = ws.get("mix_heads", T, n, ctx.compute_dtype);
        Tensor gate = wide.col_range(3 * n, 4 * n);
        ops::head_norm_gate(l, read, &gain_.view, &gate, ops::GateAct::Silu, 1.0f, eps_, H_, heads);
        out_.run(ctx, nullptr, &heads, x, ops::Act::None, ctx.overwrite ? nullptr : &x);
    }
private:
    ops::FadeShape shape() const {
        ops::FadeShape m;
        m.n_heads = H_; m.qk_dim = d_; m.v_dim = d_;
        m.q_off = 0; m.k_off = H_ * d_; m.v_off = 2 * H_ * d_;
        m.kind = ops::FadeKind::Bonus;
        m.decay = ops::DecayForm::Exp;
        m.tanh_low = true;
        m.bonus = (const float*)bonus_.view.data;
        m.state_off = width_;
        return m;
    }
    int64_t width_;
    float eps_;
    int H_, d_;
    int64_t rank_;
    Linear wide_, out_;
    std::unique_ptr<Linear> low_;
    DeviceWeight mix_, w2t_, bias_, bonus_, gain_;
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
    register_part("mixer", "channel_delta", simple<ChannelDelta>());
    register_part("mixer", "attention_beside_channel_delta", simple<AttentionBesideChannelDelta>());
    register_part("mixer", "time_mixing", simple<TimeMixing>());
}

}  // namespace sandy
