// The model registry, the greedy pick every model shares, and sequences over a one-batch cache.
#include <vesper/models/checkpoint.h>
#include <vesper/models/hybrid.h>
#include <vesper/models/language_model.h>
#include <vesper/models/transformer.h>

#include <vesper_b200_block.h>

#include <stdexcept>

namespace vesper::models {

int64_t LanguageModel::open_sequence() {
    if (single_len_ >= 0) throw std::runtime_error("this model holds one sequence at a time");
    init_cache(1, Device::CUDA);
    single_len_ = 0;
    return 0;
}

Tensor LanguageModel::extend(int64_t sequence, const Tensor& tokens) {
    if (sequence != 0 || single_len_ < 0) throw std::runtime_error("extend: no such sequence");
    Tensor y = forward_with_cache(tokens, single_len_);
    single_len_ += tokens.shape()[1];
    return y;
}

void LanguageModel::close_sequence(int64_t sequence) {
    if (sequence != 0 || single_len_ < 0) throw std::runtime_error("close_sequence: no such sequence");
    clear_cache();
    single_len_ = -1;
}

void LanguageModel::pick_from_last_logits(DecodeState& st) {
    const Tensor& logits = last_logits();
    vb200_greedy_args g{};
    g.struct_size = sizeof(g);
    g.device = logits.device_index();
    g.stream = Stream::current(Device::CUDA).raw_handle();
    g.logits = logits.data_ptr<float>();
    g.ld_logits = logits_stride();
    g.B = static_cast<int>(st.ids.shape()[0]);
    g.vocab = static_cast<int>(vocab_size());
    g.out_ids = st.ids.data_ptr<int32_t>();
    g.history = st.history.data_ptr<int32_t>();
    g.history_ld = st.history.strides()[0];
    g.pos_dev = st.lens.data_ptr<int32_t>();
    g.pos_base = static_cast<int>(st.prompt_len);
    if (st.stop_ids.defined() && st.stop_ids.numel() > 0) {
        g.stop_ids = st.stop_ids.data_ptr<int32_t>();
        g.n_stop = static_cast<int>(st.stop_ids.numel());
    }
    g.min_new_tokens = static_cast<int>(st.min_new_tokens);
    g.done = st.done.data_ptr<int32_t>();
    const int rc = vb200_greedy_step(&g);
    if (rc != VB200_OK) throw std::runtime_error(std::string("greedy_step: ") + vb200_strerror(rc) + ": " + vb200_last_error_detail());
}

namespace {

std::unique_ptr<LanguageModel> make_transformer(const Json& c, const LoadOptions& o) {
    if (o.dtype != DType::BFloat16) throw std::runtime_error("TransformerLM runs in bfloat16");
    TransformerConfig t;
    t.vocab_size = c.at("vocab_size").as_int();
    t.dim = c.at("dim").as_int();
    t.n_layers = c.at("n_layers").as_int();
    t.n_heads = c.at("n_heads").as_int();
    t.n_kv_heads = c.int_or("n_kv_heads", -1);
    t.max_seq_len = o.max_seq_len > 0 ? o.max_seq_len : c.int_or("max_seq_len", t.max_seq_len);
    t.ffn_hidden_dim = c.int_or("ffn_hidden_dim", 0);
    t.ffn_multiple_of = c.int_or("ffn_multiple_of", t.ffn_multiple_of);
    t.norm_eps = static_cast<float>(c.double_or("norm_eps", t.norm_eps));
    t.rope_base = static_cast<float>(c.double_or("rope_base", t.rope_base));
    return std::make_unique<TransformerLM>(t);
}

ModelFactory hybrid(const HybridStyle& style) {
    return [style](const Json& c, const LoadOptions& o) -> std::unique_ptr<LanguageModel> { return std::make_unique<HybridLM>(HybridConfig::from_json(c, style), o); };
}

std::map<std::string, ModelFactory>& registry() {
    static std::map<std::string, ModelFactory> r = {
        {"TransformerLM", make_transformer},
        {"Nitenex", hybrid(HybridStyle{})},
        {"Zudisun", hybrid(HybridStyle{true, false, {nn::Activation::GatedRelu, true, true}})},
    };
    return r;
}

}  // namespace

void register_architecture(const std::string& name, ModelFactory factory) { registry()[name] = std::move(factory); }

std::vector<std::string> architectures() {
    std::vector<std::string> out;
    for (const auto& kv : registry()) out.push_back(kv.first);
    return out;
}

std::unique_ptr<LanguageModel> make_model(const Json& config, const LoadOptions& options) {
    const std::string& name = config.at("architecture").as_string();
    auto it = registry().find(name);
    if (it == registry().end()) throw std::runtime_error("no model class for architecture '" + name + "'");
    return it->second(config, options);
}

std::unique_ptr<LanguageModel> load_model(const std::string& folder, const LoadOptions& options) {
    auto model = make_model(Json::parse(read_text_file(folder + "/config.json")), options);
    SafeTensors ckpt(folder + "/model.safetensors");
    for (const auto& kv : model->parameter_shapes()) {
        auto it = ckpt.entries().find(kv.first);
        if (it == ckpt.entries().end()) throw std::runtime_error("checkpoint has no tensor named " + kv.first);
        bool same = it->second.shape.size() == kv.second.size();
        for (size_t i = 0; same && i < kv.second.size(); ++i) same = kv.second[i] < 0 ? it->second.shape[i] > 0 : it->second.shape[i] == kv.second[i];
        if (!same) throw std::runtime_error("checkpoint tensor " + kv.first + " has another shape than the configuration gives");
        const std::vector<float> v = ckpt.read(kv.first);
        model->load_parameter(kv.first, v.data(), static_cast<int64_t>(v.size()));
    }
    return model;
}

}  // namespace vesper::models
