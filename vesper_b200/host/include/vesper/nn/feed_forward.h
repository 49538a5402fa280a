// nn::FeedForward -- the second sublayer of a hybrid block -- and its kinds: nn::DenseMlp (squared ReLU, or a gate of ReLU /
// SiLU, with or without biases) and nn::MixtureOfExperts (sigmoid router with group choice, gated SiLU experts, a shared expert).
#pragma once
#include <vesper/core/json.h>
#include <vesper/core/tensor.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

namespace vesper::nn {

enum class Activation { SquaredRelu, GatedRelu, GatedSilu };

// What a design fixes about its feed-forwards and its configuration does not say.
struct FeedForwardStyle {
    Activation dense = Activation::SquaredRelu;
    bool dense_bias = false;
    bool experts = false;              // mixtures of experts may take a dense layer's place
};

// One call: M rows of `width` padded to the weights' row length; x in the model's dtype, y fp32.
struct FeedForwardStep {
    int64_t M = 0;
    const void* x = nullptr;
    float* y = nullptr;
    char* act = nullptr;               // [M, act_ld()]
    char* workspace = nullptr;
    int64_t workspace_bytes = 0;
};

// Rows that a feed-forward leaves to the norm after it: per token `count` bf16 rows of rows[gather[token, :]], to be added to y.
struct PendingRows {
    const void* rows = nullptr;
    const int32_t* gather = nullptr;
    int64_t count = 0;
};

class DenseMlp;

class FeedForward {
public:
    virtual ~FeedForward() = default;
    // Parameters below the layer's "mlp." prefix (gate biases are "gate.b" and so on).
    virtual std::map<std::string, std::vector<int64_t>> parameter_shapes() const = 0;
    virtual void load_parameter(const std::string& name, const float* host_values) = 0;
    virtual int64_t act_ld() const = 0;
    virtual int64_t workspace_bytes(int64_t M) const { (void)M; return 0; }
    virtual PendingRows forward(const FeedForwardStep& step) = 0;
    // The two projections, for a block that folds its norm and residual into them.
    virtual const DenseMlp* dense() const { return nullptr; }
};

class DenseMlp : public FeedForward {
public:
    DenseMlp(int64_t ff, Activation activation, bool bias, int64_t width, int64_t width_ld, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    int64_t act_ld() const override { return (ff_ + 7) / 8 * 8; }
    PendingRows forward(const FeedForwardStep& step) override;
    const DenseMlp* dense() const override { return this; }

    const Tensor& in_weight() const { return in_; }        // gate and up rows interleaved where there is a gate
    const Tensor& out_weight() const { return out_; }
    int64_t in_rows() const { return gated() ? 2 * ff_ : ff_; }
    int epilogue() const;

private:
    bool gated() const { return activation_ != Activation::SquaredRelu; }
    int64_t ff_, width_, width_ld_;
    Activation activation_;
    bool bias_;
    DType dtype_;
    Tensor in_, out_, in_bias_, out_bias_;
};

class MixtureOfExperts : public FeedForward {
public:
    struct Sizes {
        int64_t experts, top, groups = 0, keep = 0, ff, shared = 0;
        double scale;
        // expert {ff}, router {experts, top, scale, groups {count, keep} (optional)}, shared {ff} (optional)
        explicit Sizes(const Json& mlp);
    };
    MixtureOfExperts(const Json& mlp, int64_t width, int64_t width_ld, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    int64_t act_ld() const override { return 8; }          // its activations live in the workspace
    int64_t workspace_bytes(int64_t M) const override;
    PendingRows forward(const FeedForwardStep& step) override;

private:
    struct Args;
    Sizes z_;
    int64_t width_, width_ld_;
    DType dtype_;
    Tensor router_, correction_, in_, out_, shared_in_, shared_out_;
};

// Throws where a layer entry's "mlp" is of an unknown kind or its sizes do not fit together.  Needs no device.
void check_feed_forward(const Json& mlp, const FeedForwardStyle& style);
// The feed-forward of a layer entry's "mlp".
std::unique_ptr<FeedForward> make_feed_forward(const Json& mlp, const FeedForwardStyle& style, int64_t width, int64_t width_ld, DType dtype);

}  // namespace vesper::nn
