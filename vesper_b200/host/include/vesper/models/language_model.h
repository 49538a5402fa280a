// models::LanguageModel -- what the generation loop, the command line and the C facade need of a decoder, and the
// registry that picks the class by config.json's "architecture".
#pragma once
#include <vesper/core/json.h>
#include <vesper/core/tensor.h>

#include <cstdint>
#include <functional>
#include <map>
#include <memory>
#include <string>
#include <vector>

namespace vesper::models {

class LanguageModel {
public:
    virtual ~LanguageModel() = default;

    virtual int64_t vocab_size() const = 0;
    virtual int64_t max_seq_len() const = 0;
    // -1: a size that the checkpoint's tensor gives.
    virtual std::map<std::string, std::vector<int64_t>> parameter_shapes() const = 0;
    // One parameter from host fp32 values.
    virtual void load_parameter(const std::string& name, const float* host_values, int64_t numel) = 0;

    // tokens [Batch, NewTokens] Int32 or Int64; fp32 logits [Batch, NewTokens, Vocab], or [Batch, 1, Vocab] of the last
    // position when last_only.  The returned tensor is valid until the next call.
    virtual Tensor forward_with_cache(const Tensor& tokens, int64_t start_pos, bool last_only = false) = 0;
    virtual void init_cache(int64_t batch_size, Device device) = 0;
    virtual void clear_cache() = 0;

    // ---- sequences one at a time, each with cache / state of its own ----
    // A new sequence; extend() feeds its next tokens and returns their logits [1, NewTokens, Vocab]; close_sequence()
    // gives back what it holds.  A model whose cache is one batch holds one sequence at a time.
    virtual int64_t open_sequence();
    virtual Tensor extend(int64_t sequence, const Tensor& tokens);
    virtual void close_sequence(int64_t sequence);

    // ---- device-resident decode step, used by generation::Generator ----
    // One greedy decode step for the whole batch with no host round trip: embeds ids_dev
    // [Batch] int32, runs every block at the per-sequence positions in the device length array
    // (advanced by one inside), writes logits and the arg-max ids back into ids_dev; appends the new
    // id to history_dev [Batch, history_ld] at column = the new length and updates done_dev.
    // All launches go to the current stream and are CUDA-graph capturable after one eager call.
    struct DecodeState {
        Tensor ids;        // [B] int32: in = token to process, out = next token
        Tensor lens;       // [B] int32: cached length per sequence
        Tensor history;    // [B, history_ld] int32
        Tensor done;       // [B] int32
        Tensor stop_ids;   // [n_stop] int32 (may be undefined)
        int64_t prompt_len = 0;
        int64_t min_new_tokens = 0;
        int64_t max_len = 0;          // upper bound of any sequence length during the loop (plans the split-KV launch)
    };
    // False where a decode step needs its position from the host (forward_with_cache then serves the loop).
    virtual bool device_decode() const { return true; }
    virtual void decode_step(DecodeState& st) = 0;
    // Greedy pick on the logits of the last forward_with_cache(..., last_only=true) or decode step: writes
    // st.ids, st.history[:, lens], st.done.
    void pick_from_last_logits(DecodeState& st);

protected:
    // Last logits [rows, row stride] fp32.
    virtual const Tensor& last_logits() const = 0;
    virtual int64_t logits_stride() const { return vocab_size(); }

private:
    int64_t single_len_ = -1;          // length of the one open sequence, -1 = none
};

struct LoadOptions {
    DType dtype = DType::BFloat16;     // BFloat16, or Float32 where the architecture has it
    int64_t max_seq_len = 0;           // longest sequence to provide for; 0 = the model's own limit
    int64_t max_sequences = 8;         // sequences open at a time
};

// An architecture's class from its configuration, without weights.
using ModelFactory = std::function<std::unique_ptr<LanguageModel>(const Json& config, const LoadOptions& options)>;
void register_architecture(const std::string& name, ModelFactory factory);
std::vector<std::string> architectures();
std::unique_ptr<LanguageModel> make_model(const Json& config, const LoadOptions& options);
// config.json and model.safetensors of a folder.
std::unique_ptr<LanguageModel> load_model(const std::string& folder, const LoadOptions& options);

}  // namespace vesper::models
