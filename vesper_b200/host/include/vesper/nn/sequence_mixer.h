// nn::SequenceMixer -- what stands between a hybrid block's input and output projections -- and its kinds:
// nn::LatentAttention (latent keys / values, sliding window, sinks), nn::SigmoidAttention (mixed heads, unnormalised
// sigmoid weights), nn::Mamba2 (state-space duality) and nn::Mamba1 (a state per channel).
//
// A mixer owns its weights and none of the sequences: a SequenceState, one per execution of the layer in a forward
// pass (a looped layer has one per pass), holds the slots' cache or recurrent state.  Weights and activations are
// BFloat16 or Float32; state that the recurrence carries is Float32 in both.
#pragma once
#include <vesper/core/json.h>
#include <vesper/core/tensor.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

namespace vesper::nn {

// Per-slot memory of one layer execution: latent ring [slots, ring, row], key and value rows [slots, longest, row], or
// convolution ring + state matrices.
struct SequenceState {
    Tensor ring;
    Tensor recurrent;
    Tensor values;
};

// Values that the first value-mixing layer of a forward step leaves to the later ones, [B*T, cols].
struct StepValues {
    char* data = nullptr;
    int64_t cols = 0;
    bool filled = false;
};

// One forward step: B rows of T new tokens; row b belongs to slot slots[b] (null: b) and starts at pos[b].
struct MixerStep {
    int64_t B = 0, T = 0;
    int64_t start_pos = 0;             // all rows' position when T > 1
    int64_t max_len = 0;               // longest length a one-token step can meet
    const int32_t* slots = nullptr;    // device
    const int32_t* pos = nullptr;      // device
    char* workspace = nullptr;
    int64_t workspace_bytes = 0;
    StepValues* values = nullptr;
};

class SequenceMixer {
public:
    virtual ~SequenceMixer() = default;
    // Parameters below the layer's "mix." prefix, as stored in a checkpoint; -1 = a size that the checkpoint's tensor gives.
    virtual std::map<std::string, std::vector<int64_t>> parameter_shapes() const = 0;
    virtual void load_parameter(const std::string& name, const float* host_values) = 0;
    // Told before load_parameter() how many values a parameter of free size has.
    virtual void set_free_size(const std::string& name, int64_t numel) { (void)name; (void)numel; }

    // Columns of the step's shared values this mixer takes part in, 0 = none.
    virtual int64_t shared_value_cols() const { return 0; }
    // True where a slot's memory grows with the longest sequence.
    virtual bool grows_with_length() const { return false; }
    virtual std::unique_ptr<SequenceState> make_state(int64_t slots, int64_t max_len) const = 0;
    virtual int64_t workspace_bytes(const MixerStep& step) const = 0;
    // projected [B*T, proj_ld()] (the input projection's output; may be modified) -> mixed [B*T, mixed_ld()].
    virtual void forward(const MixerStep& step, SequenceState& state, Tensor& projected, Tensor& mixed) = 0;

    // Input projection [proj_rows, width_ld], output projection [width_ld, mixed_ld]; rows are padded with zeros to a
    // multiple of 8 columns.
    const Tensor& in_weight() const { return in_weight_; }
    const Tensor& out_weight() const { return out_weight_; }
    int64_t proj_rows() const { return proj_rows_; }
    int64_t proj_ld() const { return (proj_rows_ + 7) / 8 * 8; }
    int64_t mixed_cols() const { return mixed_cols_; }
    int64_t mixed_ld() const { return (mixed_cols_ + 7) / 8 * 8; }

protected:
    SequenceMixer(int64_t width, int64_t width_ld, double eps, DType dtype) : width_(width), width_ld_(width_ld), eps_(eps), dtype_(dtype) {}
    int64_t width_, width_ld_, proj_rows_ = 0, mixed_cols_ = 0;
    double eps_;
    DType dtype_;
    Tensor in_weight_, out_weight_;
};

// Rows row0, row0 + step, ... of a zero-padded weight matrix from host fp32 values [rows, cols].
void load_rows(Tensor& dst, int64_t row0, int64_t rows, int64_t cols, const float* host_values, int64_t step = 1);
// Elements first, first + step, ... of an fp32 vector.
void load_vector(Tensor& dst, int64_t first, int64_t n, const float* host_values, int64_t step = 1);
// fp32 vector of a parameter.
Tensor vector_from_host(const float* host_values, int64_t n);

class LatentAttention : public SequenceMixer {
public:
    // mixer: heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}, mask {size}
    LatentAttention(const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    std::unique_ptr<SequenceState> make_state(int64_t slots, int64_t max_len) const override;
    int64_t workspace_bytes(const MixerStep& step) const override;
    void forward(const MixerStep& step, SequenceState& state, Tensor& projected, Tensor& mixed) override;

private:
    struct Args;
    int64_t heads_, dim_, rot_dim_, vdim_, rank_, window_;
    double scale_;
    Tensor inv_freq_;              // [rot_dim / 2] fp64
    Tensor latent_norm_, sink_;    // fp32
    Tensor expand_;                // [W_uk; W_uv], [heads * (dim + vdim), rank padded to 8]
};

class Mamba2 : public SequenceMixer {
public:
    // mixer: heads, vdim, state, groups, conv, norm_groups
    Mamba2(const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    std::unique_ptr<SequenceState> make_state(int64_t slots, int64_t max_len) const override;
    int64_t workspace_bytes(const MixerStep& step) const override;
    void forward(const MixerStep& step, SequenceState& state, Tensor& projected, Tensor& mixed) override;

private:
    struct Args;
    int64_t heads_, vdim_, state_, groups_, taps_, norm_groups_, channels_;
    Tensor conv_w_, conv_b_, dt_bias_, a_log_, d_, norm_;      // fp32
};

class SigmoidAttention : public SequenceMixer {
public:
    struct Sizes {
        int64_t heads, kv_heads, dim, vdim, temp_every = 0;
        double scale, reach, temp_coef = 0.0;
        bool value_mixing = false;
        // heads, kv_heads, dim, vdim, scale, bias_max, q_temp {coef, every} (optional), v_mix (optional)
        explicit Sizes(const Json& mixer);
        int64_t shared_value_cols() const { return value_mixing ? kv_heads * vdim : 0; }
    };
    SigmoidAttention(const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    void set_free_size(const std::string& name, int64_t numel) override;
    int64_t shared_value_cols() const override { return z_.shared_value_cols(); }
    bool grows_with_length() const override { return true; }
    std::unique_ptr<SequenceState> make_state(int64_t slots, int64_t max_len) const override;
    int64_t workspace_bytes(const MixerStep& step) const override;
    void forward(const MixerStep& step, SequenceState& state, Tensor& projected, Tensor& mixed) override;

private:
    struct Args;
    void fold_bias();
    Sizes z_;
    int64_t bias_rows_ = 0;
    float lambda_ = 0.0f;
    std::vector<float> host_rel_, host_talk_, host_offset_;      // until all three are known: the folded table needs them together
    Tensor talk_, bias_;                                         // fp32 [heads, heads], [heads, distances]
};

class Mamba1 : public SequenceMixer {
public:
    struct Sizes {
        int64_t inner, state, rank, taps;
        int64_t inner8, state8, rank8;           // padded to multiples of 8; the padding's weights are zero
        explicit Sizes(const Json& mixer);       // inner, state, dt_rank, conv
    };
    Mamba1(const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype);
    std::map<std::string, std::vector<int64_t>> parameter_shapes() const override;
    void load_parameter(const std::string& name, const float* host_values) override;
    std::unique_ptr<SequenceState> make_state(int64_t slots, int64_t max_len) const override;
    int64_t workspace_bytes(const MixerStep& step) const override;
    void forward(const MixerStep& step, SequenceState& state, Tensor& projected, Tensor& mixed) override;

private:
    struct Args;
    Sizes z_;
    Tensor w_x_, w_dt_;
    Tensor conv_w_, conv_b_, dt_bias_, a_, d_;                   // fp32; a = -exp(A_log)
};

// Row of a relative-bias table of `rows` rows for distance n: a row each below rows / 2, then logarithmic up to `reach`.
int64_t distance_bucket(int64_t n, int64_t rows, double reach);

// Throws where a layer entry's mixer is unknown or its sizes do not fit together; returns its shared value columns.  Needs no device.
int64_t check_mixer(const std::string& type, const Json& mixer);
// The mixer a layer entry's "type" names.
std::unique_ptr<SequenceMixer> make_mixer(const std::string& type, const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype);

}  // namespace vesper::nn
