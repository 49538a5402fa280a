// models::HybridLM on the B200 operators.  Nothing here computes on the host.
#include <vesper/models/hybrid.h>

#include <vesper_b200_hybrid.h>

#include <cuda_runtime.h>

#include <algorithm>
#include <cmath>
#include <stdexcept>

namespace vesper::models {

namespace {

void check(int rc, const char* who) {
    if (rc != VB200_OK) throw std::runtime_error(std::string(who) + ": " + vb200_strerror(rc) + ": " + vb200_last_error_detail());
}
void* current_stream() { return Stream::current(Device::CUDA).raw_handle(); }
int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }

}  // namespace

HybridConfig HybridConfig::from_json(const Json& c, const HybridStyle& style) {
    HybridConfig h;
    h.style = style;
    h.vocab = c.at("vocab").as_int();
    h.width = c.at("width").as_int();
    h.eps = c.at("norm").at("eps").as_double();
    for (const Json& l : c.at("layers").as_array()) {
        Layer x;
        x.type = l.at("type").as_string();
        x.mixer = l.at("mixer");
        x.mlp = l.get("mlp");
        if (!x.mlp.is_null()) nn::check_feed_forward(x.mlp, style.feed_forward);
        const int64_t cols = nn::check_mixer(x.type, x.mixer);
        if (cols > 0 && h.shared_value_cols > 0 && cols != h.shared_value_cols) throw std::runtime_error("configuration: layers that mix values must have one number of value columns");
        h.shared_value_cols = std::max(h.shared_value_cols, cols);
        h.layers.push_back(x);
    }
    const Json& loop = c.get("loop");
    if (!loop.is_null()) {
        h.loop.start = loop.at("start").as_int();
        h.loop.stop = loop.at("stop").as_int();
        h.loop.times = loop.at("times").as_int();
        if (h.loop.start < 0 || h.loop.stop <= h.loop.start || h.loop.stop > static_cast<int64_t>(h.layers.size()) || h.loop.times < 1)
            throw std::runtime_error("configuration: the loop must cover existing layers at least once");
    }
    const Json& bigram = c.get("embedding").get("bigram");
    if (!bigram.is_null()) {
        h.bigram.buckets = bigram.at("buckets").as_int();
        h.bigram.mul_prev = bigram.at("mul_prev").as_int();
        h.bigram.mul_cur = bigram.at("mul_cur").as_int();
        if (h.bigram.buckets <= 0) throw std::runtime_error("configuration: 'buckets' must be positive");
    }
    if (style.norm_outputs && (h.loop.times > 0 || h.bigram.buckets > 0)) throw std::runtime_error("configuration: this architecture has no loop and no bigram embedding");
    if (h.vocab <= 0 || h.width <= 0) throw std::runtime_error("configuration: 'vocab' and 'width' must be positive");
    return h;
}

struct HybridLM::Layer {
    std::unique_ptr<nn::SequenceMixer> mixer;
    std::unique_ptr<nn::FeedForward> ff;       // null = none
    Tensor norm1, norm2;                       // [dim] fp32
};

struct HybridLM::Buffers {
    int64_t rows = 0;
    Tensor h, embed;               // [rows, dim] fp32: residual stream, embedding output (kept where a loop re-adds it)
    Tensor xn;                     // [rows, dim]: bf16(h * weight of the next norm) (bf16(h) where outputs are normed), or the normed rows in fp32
    Tensor y;                      // [rows, dim] fp32: a sublayer's output ahead of its norm
    Tensor values;                 // [rows, shared columns]: values that later layers mix in
    Tensor inv;                    // [rows] fp32
    Tensor proj, mixed, act;       // activations of the widest layer
    Tensor step_pos;               // [rows] int32
    Tensor logits;                 // [logit_rows, vocab padded to 4] fp32
    int64_t logit_rows = 0;
    Tensor workspace;              // bytes (as fp32)
};

HybridLM::HybridLM(const HybridConfig& config, const LoadOptions& options) : config_(config), dtype_(options.dtype) {
    if (dtype_ != DType::BFloat16 && dtype_ != DType::Float32) throw std::runtime_error("HybridLM: BFloat16 or Float32");
    max_sequences_ = std::max<int64_t>(1, options.max_sequences);
    // The residual stream is padded to rows of a multiple of 8 columns, the padding zero throughout.  A norm over the
    // padded row becomes the norm over the true one with eps and the weights rescaled:
    //   1 / sqrt(ss / width + eps) = sqrt(width / dim) / sqrt(ss / dim + eps * width / dim)
    dim_ = pad8(config_.width);
    const double r = static_cast<double>(config_.width) / static_cast<double>(dim_);
    // (norms that are kernels of their own divide by the true width instead)
    norm_eps_ = dtype_ == DType::Float32 ? config_.eps : config_.eps * r;
    norm_gain_ = dtype_ == DType::Float32 ? 1.0f : static_cast<float>(std::sqrt(r));
    embed_ = zeros({config_.vocab, dim_}, dtype_, Device::CUDA);
    final_norm_ = zeros({dim_}, DType::Float32, Device::CUDA);
    if (config_.bigram.buckets > 0) bigram_ = zeros({config_.bigram.buckets + 1, dim_}, dtype_, Device::CUDA);
    if (config_.loop.times > 0) loop_step_ = zeros({config_.loop.times, dim_}, DType::Float32, Device::CUDA);
    if (!config_.style.tied_head) head_ = zeros({config_.vocab, dim_}, dtype_, Device::CUDA);
    bool grows = false;
    for (const auto& l : config_.layers) {
        auto L = std::make_unique<Layer>();
        L->mixer = nn::make_mixer(l.type, l.mixer, config_.width, dim_, config_.eps, dtype_);
        L->norm1 = zeros({dim_}, DType::Float32, Device::CUDA);
        if (!l.mlp.is_null()) {
            L->norm2 = zeros({dim_}, DType::Float32, Device::CUDA);
            L->ff = nn::make_feed_forward(l.mlp, config_.style.feed_forward, config_.width, dim_, dtype_);
        }
        grows = grows || L->mixer->grows_with_length();
        layers_.push_back(std::move(L));
    }
    max_len_ = options.max_seq_len > 0 ? options.max_seq_len : grows ? 32768 : int64_t{1} << 20;
    const int64_t n = static_cast<int64_t>(config_.layers.size());
    const auto& loop = config_.loop;
    for (int64_t i = 0; i < (loop.times > 0 ? loop.start : n); ++i) runs_.push_back({i, -1});
    for (int64_t t = 0; t < loop.times; ++t)
        for (int64_t i = loop.start; i < loop.stop; ++i) runs_.push_back({i, i == loop.start ? t : -1});
    if (loop.times > 0)
        for (int64_t i = loop.stop; i < n; ++i) runs_.push_back({i, -1});
    keep_embedding_ = loop.times > 1;
    buf_ = std::make_unique<Buffers>();
    shapes_ = parameter_shapes();
}

HybridLM::~HybridLM() = default;

std::map<std::string, std::vector<int64_t>> HybridLM::parameter_shapes() const {
    const int64_t w = config_.width;
    std::map<std::string, std::vector<int64_t>> m;
    m["embed"] = {config_.vocab, w};
    m["final.norm"] = {w};
    if (!config_.style.tied_head) m["head"] = {config_.vocab, w};
    if (config_.bigram.buckets > 0) m["bigram"] = {config_.bigram.buckets + 1, w};
    if (config_.loop.times > 0) m["loop.step"] = {config_.loop.times, w};
    for (size_t i = 0; i < layers_.size(); ++i) {
        const std::string p = "l" + std::to_string(i) + ".";
        m[p + "norm1"] = {w};
        for (const auto& kv : layers_[i]->mixer->parameter_shapes()) m[p + "mix." + kv.first] = kv.second;
        if (layers_[i]->ff) {
            m[p + "norm2"] = {w};
            for (const auto& kv : layers_[i]->ff->parameter_shapes()) m[p + "mlp." + kv.first] = kv.second;
        }
    }
    return m;
}

void HybridLM::load_parameter(const std::string& name, const float* v, int64_t numel) {
    auto it = shapes_.find(name);
    if (it == shapes_.end()) throw std::runtime_error("HybridLM::load_parameter: no parameter named " + name);
    int64_t want = 1;
    bool free_size = false;
    for (auto d : it->second) {
        if (d < 0) free_size = true;
        else want *= d;
    }
    if (free_size ? numel <= 0 || numel % want != 0 : want != numel) throw std::runtime_error("HybridLM::load_parameter: size mismatch for " + name);
    const int64_t w = config_.width;
    auto norm = [&](Tensor& dst, bool of_output = false) {
        std::vector<float> g(static_cast<size_t>(dim_), 0.0f);
        for (int64_t i = 0; i < w; ++i) g[static_cast<size_t>(i)] = v[i] * (of_output ? 1.0f : norm_gain_);
        dst.copy_from_host(g.data());
    };
    if (name == "embed") return nn::load_rows(embed_, 0, config_.vocab, w, v);
    if (name == "head") return nn::load_rows(head_, 0, config_.vocab, w, v);
    if (name == "bigram") return nn::load_rows(bigram_, 0, config_.bigram.buckets + 1, w, v);
    if (name == "loop.step") return nn::load_rows(loop_step_, 0, config_.loop.times, w, v);
    if (name == "final.norm") return norm(final_norm_);
    const size_t dot = name.find('.');
    Layer& L = *layers_.at(static_cast<size_t>(std::stoll(name.substr(1, dot - 1))));
    const std::string rest = name.substr(dot + 1);
    if (rest == "norm1") norm(L.norm1, config_.style.norm_outputs);
    else if (rest == "norm2") norm(L.norm2, config_.style.norm_outputs);
    else if (rest.compare(0, 4, "mlp.") == 0) L.ff->load_parameter(rest.substr(4), v);
    else {
        if (free_size) L.mixer->set_free_size(rest.substr(4), numel);
        L.mixer->load_parameter(rest.substr(4), v);
    }
}

void HybridLM::allocate_slots(int64_t slots) {
    states_.clear();
    for (const Run& r : runs_) states_.push_back(layers_[static_cast<size_t>(r.layer)]->mixer->make_state(slots, max_len_));
    slot_len_.assign(static_cast<size_t>(slots), -1);
    prev_ = zeros({slots}, DType::Int32, Device::CUDA);
    lens_ = zeros({slots}, DType::Int32, Device::CUDA);
    slots_dev_ = zeros({slots}, DType::Int32, Device::CUDA);
    Stream::current(Device::CUDA).synchronize();
}

void HybridLM::init_cache(int64_t batch_size, Device device) {
    if (device != Device::CUDA) throw std::runtime_error("HybridLM::init_cache: this library is the CUDA backend");
    allocate_slots(batch_size);
}

void HybridLM::clear_cache() {
    states_.clear();
    slot_len_.clear();
}

int64_t HybridLM::open_sequence() {
    if (states_.empty()) allocate_slots(max_sequences_);
    for (size_t i = 0; i < slot_len_.size(); ++i)
        if (slot_len_[i] == -1) { slot_len_[i] = 0; return static_cast<int64_t>(i); }
    throw std::runtime_error("HybridLM: all " + std::to_string(slot_len_.size()) + " sequence slots are in use");
}

void HybridLM::close_sequence(int64_t s) {
    if (s < 0 || s >= static_cast<int64_t>(slot_len_.size()) || slot_len_[static_cast<size_t>(s)] == -1) throw std::runtime_error("close_sequence: no such sequence");
    slot_len_[static_cast<size_t>(s)] = -1;          // position 0 ignores what a slot holds: nothing to clear
}

Tensor HybridLM::extend(int64_t sequence, const Tensor& tokens) { return extend_batch({sequence}, tokens); }

Tensor HybridLM::extend_batch(const std::vector<int64_t>& sequences, const Tensor& tokens) {
    if (tokens.ndim() != 2 || tokens.shape()[0] != static_cast<int64_t>(sequences.size())) throw std::runtime_error("extend: tokens must be [Sequences, NewTokens]");
    int64_t len = -1;
    for (size_t i = 0; i < sequences.size(); ++i) {
        const int64_t s = sequences[i];
        if (s < 0 || s >= static_cast<int64_t>(slot_len_.size()) || slot_len_[static_cast<size_t>(s)] < 0) throw std::runtime_error("extend: no such sequence");
        if (i > 0 && slot_len_[static_cast<size_t>(s)] != len) throw std::runtime_error("extend: the sequences of a batch must have one length");
        if (std::find(sequences.begin(), sequences.begin() + static_cast<std::ptrdiff_t>(i), s) != sequences.begin() + static_cast<std::ptrdiff_t>(i))
            throw std::runtime_error("extend: a sequence occurs twice");
        len = slot_len_[static_cast<size_t>(s)];
    }
    return forward_rows(tokens, sequences, len, false);
}

Tensor HybridLM::forward_with_cache(const Tensor& tokens, int64_t start_pos, bool last_only) {
    if (states_.empty()) throw std::runtime_error("KV cache not initialized. Call init_cache first.");
    if (tokens.ndim() != 2) throw std::runtime_error("HybridLM::forward_with_cache: tokens must be [Batch, NewTokens]");
    const int64_t B = tokens.shape()[0];
    if (B > static_cast<int64_t>(slot_len_.size())) throw std::runtime_error("HybridLM::forward_with_cache: more rows than init_cache made room for");
    if (start_pos > 0)
        for (int64_t b = 0; b < B; ++b)
            if (slot_len_[static_cast<size_t>(b)] != start_pos)
                throw std::runtime_error("HybridLM::forward_with_cache: the recurrent state does not stand at position " + std::to_string(start_pos));
    std::vector<int64_t> slots(static_cast<size_t>(B));
    for (int64_t b = 0; b < B; ++b) slots[static_cast<size_t>(b)] = b;
    return forward_rows(tokens, slots, start_pos, last_only);
}

void HybridLM::ensure_buffers(int64_t rows, const nn::MixerStep& step) {
    Buffers& b = *buf_;
    int64_t ws = 256;
    for (auto& L : layers_) {
        ws = std::max(ws, L->mixer->workspace_bytes(step));
        if (L->ff) ws = std::max(ws, L->ff->workspace_bytes(rows));
    }
    const int64_t have = b.workspace.defined() ? static_cast<int64_t>(b.workspace.numel()) * 4 : 0;
    if (ws > have) b.workspace = empty({(ws + 255) / 256 * 64}, DType::Float32, Device::CUDA);
    if (rows <= b.rows) return;
    int64_t proj = 8, mixed = 8, act = 8;
    for (auto& L : layers_) {
        proj = std::max(proj, L->mixer->proj_ld());
        mixed = std::max(mixed, L->mixer->mixed_ld());
        if (L->ff) act = std::max(act, L->ff->act_ld());
    }
    // zeroed once: padding columns are multiplied with zero weights and must hold finite numbers
    b.h = zeros({rows, dim_}, DType::Float32, Device::CUDA);
    if (keep_embedding_) b.embed = zeros({rows, dim_}, DType::Float32, Device::CUDA);
    b.xn = zeros({rows, dim_}, dtype_, Device::CUDA);
    if (config_.style.norm_outputs) b.y = zeros({rows, dim_}, DType::Float32, Device::CUDA);
    if (config_.shared_value_cols > 0) b.values = zeros({rows, config_.shared_value_cols}, dtype_, Device::CUDA);
    b.inv = zeros({rows}, DType::Float32, Device::CUDA);
    b.proj = zeros({rows, proj}, dtype_, Device::CUDA);
    b.mixed = zeros({rows, mixed}, dtype_, Device::CUDA);
    b.act = zeros({rows, act}, dtype_, Device::CUDA);
    b.step_pos = zeros({rows}, DType::Int32, Device::CUDA);
    b.rows = rows;
}

const float* HybridLM::step_vector(size_t r) const {
    return r < runs_.size() && runs_[r].enter_pass >= 0 ? loop_step_.data_ptr<float>() + runs_[r].enter_pass * dim_ : nullptr;
}

void HybridLM::copy_to_tap(size_t r, int64_t M) {
    const size_t row = static_cast<size_t>(config_.width) * 4;
    if (tap_.numel() < runs_.size() * static_cast<size_t>(M) * static_cast<size_t>(config_.width)) throw std::runtime_error("HybridLM: layer tap too small");
    if (cudaMemcpy2DAsync(tap_.data_ptr<float>() + static_cast<int64_t>(r) * M * config_.width, row, buf_->h.data_ptr<float>(), static_cast<size_t>(dim_) * 4, row,
                          static_cast<size_t>(M), cudaMemcpyDeviceToDevice, static_cast<cudaStream_t>(current_stream())) != cudaSuccess)
        throw std::runtime_error("HybridLM: layer tap copy failed");
}

void HybridLM::run(const int32_t* ids, nn::MixerStep step, int32_t* lens) {
    Buffers& b = *buf_;
    const bool f32 = dtype_ == DType::Float32;
    step.pos = b.step_pos.data_ptr<int32_t>();
    step.workspace = b.workspace.data_ptr<char>();
    step.workspace_bytes = static_cast<int64_t>(b.workspace.numel()) * 4;
    nn::StepValues values;
    if (config_.shared_value_cols > 0) {
        values.data = b.values.data_ptr<char>();
        values.cols = config_.shared_value_cols;
        step.values = &values;
    }

    vb200_embed_args e{};
    e.struct_size = sizeof(e);
    e.device = b.h.device_index(); e.stream = current_stream(); e.dtype = f32 ? VB200_F32 : VB200_BF16;
    e.ids = ids; e.B = static_cast<int>(step.B); e.T = static_cast<int>(step.T); e.dim = static_cast<int>(dim_); e.vocab = static_cast<int>(config_.vocab);
    e.table = embed_.data_ptr<char>();
    if (bigram_.defined()) {
        e.bigram = bigram_.data_ptr<char>();
        e.buckets = config_.bigram.buckets; e.mul_prev = config_.bigram.mul_prev; e.mul_cur = config_.bigram.mul_cur;
    }
    e.slots = step.slots; e.lens = lens; e.step_pos = b.step_pos.data_ptr<int32_t>(); e.prev = prev_.data_ptr<int32_t>();
    e.h = b.h.data_ptr<float>();
    e.embed_copy = keep_embedding_ ? b.embed.data_ptr<float>() : nullptr;
    e.add = step_vector(0);
    if (!f32) {
        if (!config_.style.norm_outputs) e.scale = (runs_.empty() ? final_norm_ : layers_[static_cast<size_t>(runs_[0].layer)]->norm1).data_ptr<float>();
        else if (runs_.empty()) e.scale = final_norm_.data_ptr<float>();
        e.scaled_out = b.xn.data_ptr<char>();
    }
    check(vb200_embed_sequence(&e), "embedding");
    if (config_.style.norm_outputs) run_output_norm(step);
    else run_pre_norm(step);
}

// x += norm1(mixer(x)), x += norm2(feed-forward(x)): the sublayers read the stream itself (its bf16 copy), and one kernel per sublayer
// norms the finished rows, adds them and leaves the next operand (scaled for the head's deferred norm at the end).
void HybridLM::run_output_norm(const nn::MixerStep& step) {
    Buffers& b = *buf_;
    void* s = current_stream();
    const int dev = b.h.device_index(), M = static_cast<int>(step.B * step.T), dim = static_cast<int>(dim_);
    const bool f32 = dtype_ == DType::Float32;
    const void* x = f32 ? static_cast<const void*>(b.h.data_ptr<float>()) : b.xn.data_ptr<char>();
    auto linear = [&](const void* in, int64_t K, const Tensor& w, void* out, int64_t ldo, int64_t N, int epilogue, const char* who) {
        if (f32)
            check(vb200_linear_f32(dev, s, static_cast<const float*>(in), K, w.data_ptr<float>(), K, nullptr, static_cast<float*>(out), ldo, M, static_cast<int>(N), static_cast<int>(K)), who);
        else
            check(vb200_linear(dev, s, in, K, w.data_ptr<char>(), K, out, ldo, M, static_cast<int>(N), static_cast<int>(K), epilogue, 0), who);
    };
    auto norm_add = [&](const Tensor& w, const nn::PendingRows& pending, bool last) {
        vb200_norm_add_args a{};
        a.struct_size = sizeof(a);
        a.device = dev; a.stream = s;
        a.M = M; a.dim = dim; a.count = static_cast<int>(config_.width); a.eps = static_cast<float>(config_.eps);
        a.x = b.h.data_ptr<float>(); a.y = b.y.data_ptr<float>(); a.w = w.data_ptr<float>();
        if (pending.count > 0) { a.rows = pending.rows; a.gather = pending.gather; a.n_gather = static_cast<int>(pending.count); }
        if (!f32) {
            a.copy_out = b.xn.data_ptr<char>();
            if (last) a.scale = final_norm_.data_ptr<float>();
        }
        check(vb200_norm_add(&a), "norm + residual");
    };
    for (size_t r = 0; r < runs_.size(); ++r) {
        Layer& L = *layers_[static_cast<size_t>(runs_[r].layer)];
        nn::SequenceMixer& mix = *L.mixer;
        const bool last = r + 1 == runs_.size();
        linear(x, dim, mix.in_weight(), b.proj.data_ptr<char>(), mix.proj_ld(), mix.proj_rows(), VB200_EPI_BF16, "linear(mixer in)");
        mix.forward(step, *states_[r], b.proj, b.mixed);
        linear(b.mixed.data_ptr<char>(), mix.mixed_ld(), mix.out_weight(), b.y.data_ptr<float>(), dim, dim, VB200_EPI_F32, "linear(mixer out)");
        norm_add(L.norm1, {}, last && !L.ff);
        if (L.ff) {
            nn::FeedForwardStep f;
            f.M = M; f.x = x; f.y = b.y.data_ptr<float>(); f.act = b.act.data_ptr<char>();
            f.workspace = step.workspace; f.workspace_bytes = step.workspace_bytes;
            const nn::PendingRows pending = L.ff->forward(f);
            norm_add(L.norm2, pending, last);
        }
        if (tap_.defined()) copy_to_tap(r, M);
    }
}

// x += mixer(norm1(x)), x += feed-forward(norm2(x)), both norms folded into the products around them.
void HybridLM::run_pre_norm(const nn::MixerStep& step) {
    Buffers& b = *buf_;
    void* s = current_stream();
    const int dev = b.h.device_index();
    const int M = static_cast<int>(step.B * step.T), dim = static_cast<int>(dim_);
    const float eps = static_cast<float>(norm_eps_);
    const bool f32 = dtype_ == DType::Float32;

    // out = norm(h) W^T: the norm's weight is already in xn, its 1/rms is applied to the product (bf16); fp32 norms first
    auto consume = [&](const Tensor& norm, const Tensor& w, void* out, int64_t ldo, int64_t N, int epilogue, const char* who) {
        if (f32) {
            check(vb200_rms_norm_f32(dev, s, b.h.data_ptr<float>(), norm.data_ptr<float>(), b.xn.data_ptr<float>(), M, dim, static_cast<int>(config_.width), eps), "rms_norm");
            check(vb200_linear_f32_ex(dev, s, b.xn.data_ptr<float>(), dim, w.data_ptr<float>(), dim, nullptr, nullptr, static_cast<float*>(out), ldo, M, static_cast<int>(N), dim,
                                      epilogue == VB200_EPI_BF16 ? VB200_EPI_F32 : epilogue), who);
            return;
        }
        vb200_linear_args a{};
        a.struct_size = sizeof(a);
        a.device = dev; a.stream = s;
        a.x = b.xn.data_ptr<char>(); a.ldx = dim; a.w = w.data_ptr<char>(); a.ldw = dim; a.out = out; a.ldo = ldo;
        a.M = M; a.N = static_cast<int>(N); a.K = dim; a.epilogue = epilogue;
        if (M <= 64) { a.rms_rows = b.h.data_ptr<float>(); a.rms_dim = dim; a.rms_ld = dim; a.rms_eps = eps; }
        else {
            check(vb200_row_inv_rms(dev, s, b.h.data_ptr<float>(), dim, b.inv.data_ptr<float>(), M, dim, eps), "row_inv_rms");
            a.row_scale = b.inv.data_ptr<float>();
        }
        check(vb200_linear_ex(&a), who);
    };
    // h += x W^T (+ what enters the residual stream before the next layer); xn = bf16(h * weight of the next norm)
    auto produce = [&](const void* x, int64_t K, const Tensor& w, const Tensor& next_norm, const float* bias, const float* addend, const char* who) {
        if (f32) {
            check(vb200_linear_f32_ex(dev, s, static_cast<const float*>(x), K, w.data_ptr<float>(), K, bias, addend, b.h.data_ptr<float>(), dim, M, dim, static_cast<int>(K),
                                      VB200_EPI_ADD_F32), who);
            return;
        }
        vb200_linear_args a{};
        a.struct_size = sizeof(a);
        a.device = dev; a.stream = s;
        a.x = x; a.ldx = K; a.w = w.data_ptr<char>(); a.ldw = K; a.out = b.h.data_ptr<float>(); a.ldo = dim;
        a.M = M; a.N = dim; a.K = static_cast<int>(K); a.epilogue = VB200_EPI_ADD_F32;
        a.bias = bias; a.addend = addend;
        a.scaled_copy = b.xn.data_ptr<char>(); a.copy_scale = next_norm.data_ptr<float>();
        check(vb200_linear_ex(&a), who);
    };
    auto entry_norm = [&](size_t r) -> const Tensor& { return r < runs_.size() ? layers_[static_cast<size_t>(runs_[r].layer)]->norm1 : final_norm_; };
    auto embedding_again = [&](size_t r) -> const float* { return r < runs_.size() && runs_[r].enter_pass > 0 ? b.embed.data_ptr<float>() : nullptr; };

    for (size_t r = 0; r < runs_.size(); ++r) {
        Layer& L = *layers_[static_cast<size_t>(runs_[r].layer)];
        nn::SequenceMixer& mix = *L.mixer;
        const bool tap = tap_.defined();          // a tap wants the stream before anything else enters it
        const Tensor& next = entry_norm(r + 1);
        const float* bias = tap ? nullptr : step_vector(r + 1);
        const float* addend = tap ? nullptr : embedding_again(r + 1);
        consume(L.norm1, mix.in_weight(), b.proj.data_ptr<char>(), mix.proj_ld(), mix.proj_rows(), VB200_EPI_BF16, "linear(mixer in)");
        mix.forward(step, *states_[r], b.proj, b.mixed);
        const nn::DenseMlp* ff = L.ff ? L.ff->dense() : nullptr;
        const bool last = ff == nullptr;
        produce(b.mixed.data_ptr<char>(), mix.mixed_ld(), mix.out_weight(), last ? next : L.norm2, last ? bias : nullptr, last ? addend : nullptr, "linear(mixer out) + residual");
        if (!last) {
            consume(L.norm2, ff->in_weight(), b.act.data_ptr<char>(), ff->act_ld(), ff->in_rows(), ff->epilogue(), "linear(up)");
            produce(b.act.data_ptr<char>(), ff->act_ld(), ff->out_weight(), next, bias, addend, "linear(down) + residual");
        }
        if (tap) {
            copy_to_tap(r, M);
            if (step_vector(r + 1) || embedding_again(r + 1))
                check(vb200_residual_add(dev, s, b.h.data_ptr<float>(), embedding_again(r + 1), step_vector(r + 1), M, dim, f32 ? nullptr : next.data_ptr<float>(),
                                         f32 ? nullptr : b.xn.data_ptr<char>()), "residual_add");
        }
    }
}

int64_t HybridLM::logits_stride() const { return (config_.vocab + 3) / 4 * 4; }
const Tensor& HybridLM::last_logits() const { return buf_->logits; }

// Logits of out_rows rows of the residual stream, the first at first_row, row_stride rows apart.
void HybridLM::head(int64_t out_rows, int64_t first_row, int64_t row_stride) {
    Buffers& b = *buf_;
    void* s = current_stream();
    const int dev = b.h.device_index(), dim = static_cast<int>(dim_), vocab = static_cast<int>(config_.vocab), M = static_cast<int>(out_rows);
    const float eps = static_cast<float>(norm_eps_);
    const int64_t first = first_row * dim_, ld = row_stride * dim_;
    const Tensor& w = head_.defined() ? head_ : embed_;
    if (b.logit_rows < out_rows) {
        b.logits = empty({out_rows, logits_stride()}, DType::Float32, Device::CUDA);
        b.logit_rows = out_rows;
    }
    if (dtype_ == DType::Float32) {
        // every row is normed; the product takes the wanted ones by their stride
        check(vb200_rms_norm_f32(dev, s, b.h.data_ptr<float>(), final_norm_.data_ptr<float>(), b.xn.data_ptr<float>(), static_cast<int>(first_row + (out_rows - 1) * row_stride + 1),
                                 dim, static_cast<int>(config_.width), eps), "rms_norm");
        check(vb200_linear_f32_ex(dev, s, b.xn.data_ptr<float>() + first, ld, w.data_ptr<float>(), dim, nullptr, nullptr, b.logits.data_ptr<float>(), logits_stride(), M, vocab, dim,
                                  VB200_EPI_F32), "linear(output)");
        return;
    }
    vb200_linear_args a{};
    a.struct_size = sizeof(a);
    a.device = dev; a.stream = s;
    a.x = b.xn.data_ptr<uint16_t>() + first; a.ldx = ld;
    a.w = w.data_ptr<char>(); a.ldw = dim; a.out = b.logits.data_ptr<float>(); a.ldo = logits_stride();
    a.M = M; a.N = vocab; a.K = dim; a.epilogue = VB200_EPI_F32;
    if (M <= 64) { a.rms_rows = b.h.data_ptr<float>() + first; a.rms_ld = ld; a.rms_dim = dim; a.rms_eps = eps; }
    else {
        check(vb200_row_inv_rms(dev, s, b.h.data_ptr<float>() + first, ld, b.inv.data_ptr<float>(), M, dim, eps), "row_inv_rms");
        a.row_scale = b.inv.data_ptr<float>();
    }
    check(vb200_linear_ex(&a), "linear(output)");
}

Tensor HybridLM::forward_rows(const Tensor& tokens, const std::vector<int64_t>& slots, int64_t start_pos, bool last_only) {
    if (tokens.dtype() != DType::Int32 && tokens.dtype() != DType::Int64) throw std::runtime_error("HybridLM: tokens must be Int32 or Int64");
    const int64_t B = tokens.shape()[0], T = tokens.shape()[1];
    if (B < 1 || T < 1) throw std::runtime_error("HybridLM: no tokens");
    if (start_pos < 0 || start_pos + T > max_len_)
        throw std::runtime_error("Sequence length " + std::to_string(start_pos + T) + " exceeds maximum " + std::to_string(max_len_));
    nn::MixerStep step;
    step.B = B; step.T = T; step.start_pos = start_pos; step.max_len = start_pos + T;
    ensure_buffers(B * T, step);
    Tensor ids = tokens.is_contiguous() ? tokens : tokens.contiguous();
    if (ids.dtype() == DType::Int64) {
        Tensor host = ids.to(Device::CPU);
        std::vector<int32_t> v(ids.numel());
        for (size_t i = 0; i < v.size(); ++i) v[i] = static_cast<int32_t>(host.data_ptr<int64_t>()[i]);
        ids = empty({B, T}, DType::Int32, Device::CUDA);
        ids.copy_from_host(v.data());
    } else if (ids.device() != Device::CUDA) ids = ids.to(Device::CUDA);
    // where the rows live and stand: B integers each, staged by the copy call itself
    std::vector<int32_t> host(static_cast<size_t>(B), static_cast<int32_t>(start_pos));
    cudaStream_t cs = static_cast<cudaStream_t>(current_stream());
    bool identity = true;
    for (int64_t b = 0; b < B; ++b) identity = identity && slots[static_cast<size_t>(b)] == b;
    cudaError_t rc = cudaMemcpyAsync(lens_.data_ptr<int32_t>(), host.data(), host.size() * 4, cudaMemcpyHostToDevice, cs);
    if (!identity && rc == cudaSuccess) {
        for (int64_t b = 0; b < B; ++b) host[static_cast<size_t>(b)] = static_cast<int32_t>(slots[static_cast<size_t>(b)]);
        rc = cudaMemcpyAsync(slots_dev_.data_ptr<int32_t>(), host.data(), host.size() * 4, cudaMemcpyHostToDevice, cs);
        step.slots = slots_dev_.data_ptr<int32_t>();
    }
    if (rc != cudaSuccess) throw std::runtime_error(std::string("HybridLM: ") + cudaGetErrorString(rc));
    run(ids.data_ptr<int32_t>(), step, lens_.data_ptr<int32_t>());
    for (int64_t v : slots) slot_len_[static_cast<size_t>(v)] = start_pos + T;
    const int64_t out_rows = last_only ? B : B * T;
    head(out_rows, last_only ? T - 1 : 0, last_only ? T : 1);
    Tensor out = buf_->logits.narrow(0, 0, out_rows);
    if (logits_stride() != config_.vocab) {           // an odd vocabulary: without the row padding
        Tensor dense = empty({out_rows, config_.vocab}, DType::Float32, Device::CUDA);
        const size_t row = static_cast<size_t>(config_.vocab) * 4;
        if (cudaMemcpy2DAsync(dense.data_ptr<float>(), row, out.data_ptr<float>(), static_cast<size_t>(logits_stride()) * 4, row, static_cast<size_t>(out_rows),
                              cudaMemcpyDeviceToDevice, cs) != cudaSuccess)
            throw std::runtime_error("HybridLM: logits copy failed");
        out = dense;
    }
    return out.view({B, last_only ? 1 : T, config_.vocab});
}

void HybridLM::decode_step(DecodeState& st) {
    if (states_.empty()) throw std::runtime_error("KV cache not initialized. Call init_cache first.");
    const int64_t B = st.ids.shape()[0];
    if (B > static_cast<int64_t>(slot_len_.size())) throw std::runtime_error("HybridLM::decode_step: more rows than init_cache made room for");
    nn::MixerStep step;
    step.B = B; step.T = 1; step.max_len = st.max_len;
    ensure_buffers(B, step);
    run(st.ids.data_ptr<int32_t>(), step, st.lens.data_ptr<int32_t>());
    for (int64_t b = 0; b < B; ++b) slot_len_[static_cast<size_t>(b)] = -2;
    head(B, 0, 1);
    pick_from_last_logits(st);
}

}  // namespace vesper::models
