// models::HybridLM -- decoders whose layers each name their sequence mixer and feed-forward in the configuration.
//   "Nitenex"  token + bigram embedding, pre-norm layers (latent attention or Mamba-2, then dense squared ReLU), a range of
//              layers that may run several times with the same weights, RMSNorm and a tied output head
//   "Zudisun"  layers that read the stream itself and norm their outputs (sigmoid attention with mixed heads or Mamba-1, then a
//              ReLU-gated feed-forward with biases or a mixture of experts), RMSNorm and an output head of its own
//
// As in TransformerLM the residual stream is fp32, norms ahead of a projection are deferred into the GEMMs around them, and
// decode steps take positions from the device, so one step can be captured in a CUDA graph.  Each execution of a layer has a
// cache or recurrent state of its own; sequences live in slots of those.
#pragma once
#include <vesper/models/language_model.h>
#include <vesper/nn/feed_forward.h>
#include <vesper/nn/sequence_mixer.h>

namespace vesper::models {

// What an architecture fixes about its blocks and its configuration does not say.
struct HybridStyle {
    bool norm_outputs = false;     // x += norm(sublayer(x)) instead of x += sublayer(norm(x))
    bool tied_head = true;
    nn::FeedForwardStyle feed_forward;
};

struct HybridConfig {
    HybridStyle style;
    int64_t vocab = 0, width = 0;
    double eps = 1e-6;
    struct Layer {
        std::string type;          // mixer kind
        Json mixer;                // its sizes
        Json mlp;                  // its feed-forward, null = none
    };
    std::vector<Layer> layers;
    int64_t shared_value_cols = 0;                                          // of the layers that mix values, 0 = none
    struct { int64_t start = 0, stop = 0, times = 0; } loop;               // times 0 = no loop
    struct { int64_t buckets = 0, mul_prev = 0, mul_cur = 0; } bigram;     // buckets 0 = none
    static HybridConfig from_json(const Json& config, const HybridStyle& style);
};

class HybridLM : public LanguageModel {
public:
    HybridLM(const HybridConfig& config, const LoadOptions& options);
    ~HybridLM() override;

    int64_t vocab_size() const override { return config_.vocab; }
    int64_t max_seq_len() const override { return max_len_; }
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values, int64_t numel) override;

    // A recurrent state only continues where it stands: start_pos is 0 (new sequences) or the number of tokens the
    // rows have been given so far.
    Tensor forward_with_cache(const Tensor& tokens, int64_t start_pos, bool last_only = false) override;
    void init_cache(int64_t batch_size, Device device) override;
    void clear_cache() override;

    int64_t open_sequence() override;
    Tensor extend(int64_t sequence, const Tensor& tokens) override;
    void close_sequence(int64_t sequence) override;
    // The same for several sequences at once: row b of tokens [B, T] goes to sequences[b], all at one length.
    Tensor extend_batch(const std::vector<int64_t>& sequences, const Tensor& tokens);

    void decode_step(DecodeState& st) override;

    // The residual stream after every layer execution of the following forward calls goes to tap [executions, rows, width]
    // (fp32, rows = B * T of the call); an undefined tensor ends it.
    void set_layer_tap(Tensor tap) { tap_ = std::move(tap); }
    int64_t layer_executions() const { return static_cast<int64_t>(runs_.size()); }
    const HybridConfig& config() const { return config_; }

protected:
    const Tensor& last_logits() const override;
    int64_t logits_stride() const override;

private:
    struct Layer;
    struct Buffers;
    // One execution of a layer in a forward pass; at the head of a loop pass the loop's step vector (and, from the
    // second pass on, the embedding output) enters the residual stream first.
    struct Run {
        int64_t layer = 0;
        int64_t enter_pass = -1;
    };
    void allocate_slots(int64_t slots);
    void ensure_buffers(int64_t rows, const nn::MixerStep& step);
    // Runs the model on B x T ids with lengths in lens [B] (advanced); leaves the final residual stream, returns nothing.
    void run(const int32_t* ids, nn::MixerStep step, int32_t* lens);
    void run_pre_norm(const nn::MixerStep& step);
    void run_output_norm(const nn::MixerStep& step);
    void copy_to_tap(size_t run, int64_t rows);
    const float* step_vector(size_t run) const;         // of the loop pass that execution opens, or null
    void head(int64_t out_rows, int64_t first_row, int64_t row_stride);
    Tensor forward_rows(const Tensor& tokens, const std::vector<int64_t>& slots, int64_t start_pos, bool last_only);

    HybridConfig config_;
    DType dtype_;
    int64_t max_len_, max_sequences_, dim_;        // dim_: width padded to a multiple of 8
    double norm_eps_;                               // eps and (via the norm weights) scale of norms over padded rows
    float norm_gain_ = 1.0f;
    Tensor embed_, bigram_, final_norm_, loop_step_, head_;      // head_: undefined where tied
    std::map<std::string, std::vector<int64_t>> shapes_;
    std::vector<std::unique_ptr<Layer>> layers_;
    std::vector<Run> runs_;
    std::vector<std::unique_ptr<nn::SequenceState>> states_;     // one per run
    std::vector<int64_t> slot_len_;                 // tokens a slot's sequence has been given; -1 = free, -2 = known to the device only
    bool keep_embedding_ = false;
    Tensor prev_, lens_, slots_dev_;
    std::unique_ptr<Buffers> buf_;
    Tensor tap_;
};

}  // namespace vesper::models
