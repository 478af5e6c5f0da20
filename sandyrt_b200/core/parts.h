// The parts a model is put together from, the per-step context they see, and their registry.
//
// A part is built from a PartSpec (its kind, its sizes and constants, the names of its tensors),
// says which tensors it needs (`requests`), receives them (`bind`) and then runs on the tokens of a
// step (`forward`).  It knows its own sizes and nothing of the model it sits in: layer indices,
// architecture names and config.json keys never reach it.
//
// Families and what each must provide:
//   Norm              forward(ctx, x, out, rows, n_rows)      out = norm(x[rows] or x)
//   PositionEncoding  table() -> tensor added at the embedding, or null
//                     rotate(ctx, q, k)  (in place), for encodings applied to queries and keys
//                     max_positions() -> limit or nullopt
//   Embedding         forward(ctx, x)                          x = the tokens' rows (+ position table)
//                     table() -> the bound token table
//   Head              forward(ctx, y, logits)                  float32 logits of the normed rows y
//   Mixer             cache_spec() -> pages, a fixed-size state, or nothing
//                     forward(ctx, h, x, call)                 x += mix(h), in place
//   FeedForward       forward(ctx, h, x)                       x += ff(h), in place
//   Block             forward(ctx, x, call)                    runs its norms, mixer, feed-forward
//   Remix             forward(ctx, x, x0)                      x <- f(x, x0), x0 the embedding's output
//   Wrap              read(ctx, X, ..) / write(ctx, X, ..)     how a sublayer reads the stream(s) and how its result joins
//                                                              them, for blocks whose sublayers do more than x += f(norm(x))
//
// `x` is the residual stream: float32 [tokens, width] in both compute dtypes, so the residual sum is
// always formed and kept in 32-bit.  `h` is a normed copy in the compute dtype, handed over as a
// NormedInput: a consumer either asks for the tensor (computed once) or, if its kernel can run the
// norm itself, takes the norm's parameters and never materialises it.
//
// A new kind is added with `register_part(family, kind, factory)`; no file of the engine changes.
// Kinds defined outside this library (the Python binding) register through the C interface and run
// as ForeignPart adapters around their callbacks.
#pragma once

#include <functional>
#include <map>
#include <memory>
#include <optional>
#include <string>
#include <vector>

#include "cache.h"
#include "device.h"
#include "ops.h"
#include "spec.h"
#include "weights.h"

namespace sandy {

class PositionEncoding;
class Wrap;

// Everything a part may read about the running step.  Device arrays are int32.
struct StepContext {
    int n_tokens = 0, n_seqs = 0, n_rows = 0;
    int* token_ids = nullptr;            // [T] the step's tokens, requests back to back
    int* positions = nullptr;            // [T] position of each token in its request
    const int* token_seq = nullptr;      // [T] which of the step's requests a token belongs to
    const int* seq_slots = nullptr;      // [S] state slot of each request
    const int* q_start = nullptr;        // [S+1] first token of each request in the step
    const int* kv_before = nullptr;      // [S] tokens each request had before the step
    const int* logit_rows = nullptr;     // [R] tokens whose logits are wanted
    std::vector<const int*> block_tables;    // per cache group: [S, max_blocks]
    int max_blocks = 0;
    DType compute_dtype = DType::F32;
    Workspace* workspace = nullptr;
    DeviceCaches* caches = nullptr;
    PositionEncoding* position = nullptr;    // the model's position encoding
    int embedding_cache = -1;                // the cache entry of the embedding's own state per request, or -1
    // A sublayer's result that its wrap has not written into the streams yet.  A block whose last sublayer sits in a wrap
    // may leave the write owed; whoever reads the streams next (the next block's first wrap, or the model before a stream
    // mix and before its final norm) does it in its own pass over them.  `y` and `gate` stay untouched until then.
    struct OwedWrite { Wrap* wrap = nullptr; Tensor y, gate; } owed;
    // Set by a block that norms a sublayer's output before it joins the stream: a mixer or feed-forward that
    // says `can_overwrite()` then writes its result over the tensor it is given instead of adding to it.
    bool overwrite = false;
    // host copies, for parts that plan their launches on the host
    std::vector<int> host_q_lens, host_kv_before, host_slots;
    int max_q_len = 0, max_kv_len = 0;
    ops::Launch launch;                  // stream and status words

    // `window` and `keep_first` of the layer that asks: the profile's figures count the keys it looks at
    ops::AttentionStep attention_step(int group, int window = 0, int keep_first = 0) const;
};

class Part {
public:
    explicit Part(const PartSpec& spec) : spec_(spec) {}
    virtual ~Part() = default;
    const PartSpec& spec() const { return spec_; }
    virtual TensorRequests requests() const { return {}; }             // local tensor name -> what is expected of it
    virtual void bind(const TensorMap& tensors, DType dtype) { (void)tensors; (void)dtype; }
    // Bytes of weights one step reads from this part (for roofline figures); parts with matrices override it.
    virtual size_t weight_bytes() const { return 0; }
    // A part whose `forward` only launches kernels that read the step's device arrays may be recorded
    // in a CUDA graph and replayed.  A part that decides anything from the step's host-side lists
    // must say false; the engine then runs every step of a model that holds such a part without graphs.
    virtual bool graph_safe() const { return true; }
protected:
    PartSpec spec_;
};

struct LayerNormParams { Tensor gamma; const Tensor* beta = nullptr; float eps = 0.0f; };
// An RMS norm's float32 input rows, gain (or null) and eps, for a consumer whose kernel runs the norm itself.
struct RmsNormParams { Tensor x; const Tensor* gain = nullptr; float eps = 0.0f; };

class Norm : public Part {
public:
    using Part::Part;
    virtual void forward(StepContext& ctx, const Tensor& x, Tensor& out, const int* rows, int n_rows) = 0;
    // Kernels that can run a LayerNorm inside themselves ask for its parameters here.
    virtual bool layernorm_params(LayerNormParams& out) const { (void)out; return false; }
    // ... and kernels that run an RMS norm inside themselves (a token shift behind the norm) here; `x` is left alone.
    virtual bool rms_params(RmsNormParams& out) const { (void)out; return false; }
    // x += mult * norm(y), both float32: a norm behind a sublayer.  Norms that cannot do this in 32-bit refuse.
    virtual void forward_add(StepContext& ctx, const Tensor& y, float mult, Tensor& x) {
        (void)ctx; (void)y; (void)mult; (void)x;
        throw ConfigError("norm kind '" + spec_.kind + "' cannot follow a sublayer");
    }
    // A part whose forward_add is x += mult * gain * y with one float32 factor per channel hands the factors out
    // here, so that a block can join several branches to the stream in one pass.
    virtual const Tensor* channel_gain() const { return nullptr; }
};

class PositionEncoding : public Part {
public:
    using Part::Part;
    virtual std::optional<int64_t> max_positions() const { return std::nullopt; }
    virtual const Tensor* table() const { return nullptr; }
    virtual bool rotates() const { return false; }                      // true for encodings that act on queries and keys
    virtual void rotate(StepContext& ctx, Tensor& q, Tensor* k) { (void)ctx; (void)q; (void)k; }
};

class Embedding : public Part {
public:
    using Part::Part;
    virtual const Tensor* table() const { return nullptr; }
    // A fixed-size state per request (something of the tokens before, kept between steps); the model's description
    // names the cache entry (ModelSpec::embedding_cache), the step hands it over as StepContext::embedding_cache.
    virtual CacheSpec cache_spec() const { return CacheSpec::none(); }
    virtual void forward(StepContext& ctx, Tensor& x) = 0;
};

class Head : public Part {
public:
    using Part::Part;
    virtual bool tied() const { return false; }        // shares the embedding's table: `bind` then receives it
    virtual void bind_head(const TensorMap& tensors, DType dtype, const Tensor* tied_weight) = 0;
    virtual void forward(StepContext& ctx, const Tensor& y, Tensor& logits) = 0;
};

// A normed view of the residual stream that has not been computed yet.
class NormedInput {
public:
    NormedInput(StepContext& ctx, Norm& norm, const Tensor& x) : ctx_(ctx), norm_(&norm), x_(x) {}
    // An input a block has computed already (a norm with something behind it): consumers get the tensor as it is.
    NormedInput(StepContext& ctx, const Tensor& computed) : ctx_(ctx), x_(computed), tensor_(computed), fixed_(true) {}
    int64_t rows() const { return x_.rows; }
    int64_t cols() const { return x_.cols; }
    const Tensor& tensor();                            // computed once and shared
    bool fusable(ops::FusedNorm& out) const;           // the norm's parameters, if it is a LayerNorm
    bool rms(RmsNormParams& out) const;                // the stream's rows and the norm's parameters, if it is an RMS norm
private:
    StepContext& ctx_;
    Norm* norm_ = nullptr;
    Tensor x_;
    Tensor tensor_;
    bool fixed_ = false;
};

class Mixer : public Part {
public:
    using Part::Part;
    virtual CacheSpec cache_spec() const { return CacheSpec::none(); }
    virtual void forward(StepContext& ctx, NormedInput& h, Tensor& x, const LayerCall& call) = 0;
    virtual bool can_overwrite() const { return false; }      // honours StepContext::overwrite
};

class FeedForward : public Part {
public:
    using Part::Part;
    virtual void forward(StepContext& ctx, NormedInput& h, Tensor& x) = 0;
    virtual bool can_overwrite() const { return false; }      // honours StepContext::overwrite
    virtual bool empty() const { return false; }              // a layer without a feed-forward
};

// Something that acts on the whole residual stream between layers, with the embedding's output at hand.
class Remix : public Part {
public:
    using Part::Part;
    virtual void forward(StepContext& ctx, Tensor& x, const Tensor& x0) = 0;
};

// What a block puts around one sublayer when that is more than x += f(norm(x)): how the sublayer's input is read from
// the stream(s) X (float32 [tokens, streams * width]) and how its result joins them.
class Wrap : public Part {
public:
    using Part::Part;
    // float32 numbers per request that the wrap keeps between steps (the block adds them to its layer's cache entry
    // and hands their place over as `state` and `offset`)
    virtual int64_t state_floats() const { return 0; }
    // What `read` hands back: `sublayer_in` is what the sublayer reads; `gate` whatever `write` needs again.
    struct Input { Tensor sublayer_in; Tensor gate; };
    // Reads the stream for this wrap's sublayer.  `before` / `before_y` / `before_in`: another wrap of the same block
    // whose write is still owed (its sublayer's result and what its read handed back); the read then does that write
    // first, in the same pass over the streams.
    virtual Input read(StepContext& ctx, Tensor& X, const StateView* state, int64_t offset, Wrap* before, const Tensor* before_y,
                       const Input* before_in) = 0;
    // X <- the streams with the sublayer's result y (float32 [tokens, width]) joined; with `sum_out` (float32 [tokens,
    // width]) also the sum of the streams after that.
    virtual void write(StepContext& ctx, Tensor& X, const Tensor& y, const Input& in, Tensor* sum_out = nullptr) = 0;
};

// An arrangement of norms, a mixer and a feed-forward (built from a LayerSpec).
class Block {
public:
    Block(std::unique_ptr<Mixer> mixer, std::unique_ptr<FeedForward> ff, std::map<std::string, std::unique_ptr<Norm>> norms,
          int64_t width)
        : mixer_(std::move(mixer)), ff_(std::move(ff)), norms_(std::move(norms)), width_(width) {}
    virtual ~Block() = default;
    virtual void forward(StepContext& ctx, Tensor& x, const LayerCall& call) = 0;
    // What the layer asks of the cache manager: the mixer's needs, plus whatever the block itself keeps per request.
    virtual CacheSpec cache_spec() const { return mixer_->cache_spec(); }
    // Whether `forward` itself does a write into the streams that the block before left owed (StepContext::owed); the
    // model settles it in front of every block that does not.
    virtual bool settles_owed() const { return false; }
    Mixer& mixer() { return *mixer_; }
    FeedForward& feed_forward() { return *ff_; }
    std::map<std::string, std::unique_ptr<Norm>>& norms() { return norms_; }
    std::map<std::string, std::unique_ptr<Wrap>>& wraps() { return wraps_; }
protected:
    std::unique_ptr<Mixer> mixer_;
    std::unique_ptr<FeedForward> ff_;
    std::map<std::string, std::unique_ptr<Norm>> norms_;
    std::map<std::string, std::unique_ptr<Wrap>> wraps_;
    int64_t width_;
};

// One weight matrix with its bias, and the choice of the kernel that multiplies by it.
//
// The weight file may store a matrix as [in, out] (GPT-2's Conv1D layout; the reference transposes
// these offline, scripts/run_gpt2.py:177-189) or as [out, in].  Both are read as they are: the
// 32-bit kernel takes either layout, and for the tensor-core kernels the matrix is brought into
// [out, in] once, when it is bound, which is the K-major operand layout those kernels read.
// Kernel choice per call, by dtype and row count: float32 -> the FFMA kernel; bfloat16 with up to 64
// rows (a decode step) -> the weight-streaming kernel, which can also run the norm before the
// product and write key/value columns into the cache; bfloat16 with more rows -> tcgen05.
class Linear {
public:
    Linear(int64_t in_features, int64_t out_features, bool bias, const std::string& layout, std::string name);
    TensorRequests requests() const;
    void bind(const TensorMap& tensors, DType dtype, const Tensor* shared_weight = nullptr);
    size_t weight_bytes() const;
    // out = act(a @ W + b) + residual.  `out` may be `residual` itself.  If `kv` is given and the
    // kernel used can write keys/values into the cache, it does and sets kv->written.
    void run(StepContext& ctx, NormedInput* lazy, const Tensor* a, Tensor& out, ops::Act act, const Tensor* residual,
             ops::KVTarget* kv = nullptr);
    // Several products of one shape whose weights are stacked in this one ([n_groups * N, in], layout "out_in", no bias): columns
    // g of out [T, n_groups * N] = columns g of a [T, n_groups * in] times rows g.  Up to 64 rows they are one launch.
    void run_groups(StepContext& ctx, const Tensor& a, int n_groups, Tensor& out);
    const Tensor& weight() const { return weight_.view; }
private:
    int64_t in_, out_;
    bool has_bias_, w_out_in_, use_tc_ = false;
    std::string layout_, name_;
    DeviceWeight weight_, bias_;
};

// ---- registry of part kinds ---------------------------------------------------------------------------
struct BlockParts {
    std::unique_ptr<Mixer> mixer;
    std::unique_ptr<FeedForward> feed_forward;
    std::map<std::string, std::unique_ptr<Norm>> norms;
    std::map<std::string, std::unique_ptr<Wrap>> wraps;
    int64_t width = 0;
    Json params = Json::object();          // the block's own constants (LayerSpec::block_params)
};
struct PartFactory {
    std::function<std::unique_ptr<Part>(const PartSpec&)> make;                // every family but "block"
    std::function<std::unique_ptr<Block>(BlockParts)> make_block;              // "block"
    std::vector<std::string> norm_names;                                       // "block": the norms it wants
};
// family: "mixer", "feed_forward", "norm", "position", "embedding", "head", "remix", "wrap" or "block"
void register_part(const std::string& family, const std::string& kind, PartFactory factory);
const PartFactory& get_part(const std::string& family, const std::string& kind);    // unknown -> ConfigError listing the known kinds
std::vector<std::string> part_kinds(const std::string& family);

// Kinds of parts_hybrid.cpp: RMS norm, gated feed-forward, norms on both sides of a sublayer, attention with a sink
// beside a matrix memory, the gated delta rule, the re-entry mix of a looped span.  Called once by the registry.
void register_hybrid_parts();
// Kinds of parts_capped.cpp: attention with normed queries, keys and values, a temperature per head, capped scores and
// chunks of positions, behind a token shift; the stream's re-entry into a looped span by addition.
void register_capped_parts();
// Kinds of parts_latent.cpp: attention over a latent of keys and values, a routed mixture of experts, a factor per
// channel behind a sublayer, the block whose two sublayers read one normed input.
void register_latent_parts();

// Kinds of parts_streams.cpp: a token embedding with a hashed pair-of-tokens table, the wrap and the block of a residual
// stream kept in several copies (with a short convolution on a sublayer's input and a gate on its result), attention
// with a learned bias by distance, and the state-space mixer with one decay per head.
void register_stream_parts();

// Kinds of parts_linear.cpp: attention with a sliding window that keeps the first tokens, a sink in the softmax's denominator
// and a gate by element; gated linear attention; the matrix memory as a mixer of its own; the delta rule with a decay per key
// channel, alone and beside attention; time mixing.
void register_linear_parts();

template <typename T>
std::unique_ptr<T> make_part(const std::string& family, const PartSpec& spec) {
    std::unique_ptr<Part> p = get_part(family, spec.kind).make(spec);
    T* typed = dynamic_cast<T*>(p.get());
    if (!typed) throw ConfigError("part kind '" + spec.kind + "' is not a " + family);
    p.release();
    return std::unique_ptr<T>(typed);
}

}  // namespace sandy
