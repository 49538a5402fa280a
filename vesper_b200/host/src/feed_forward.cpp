// nn::DenseMlp and nn::MixtureOfExperts over the C ABI of vesper_b200_hybrid.h.
#include <vesper/nn/feed_forward.h>
#include <vesper/nn/sequence_mixer.h>

#include <vesper_b200_hybrid.h>

#include <stdexcept>

namespace vesper::nn {

namespace {

void check(int rc, const char* who) {
    if (rc != VB200_OK) throw std::runtime_error(std::string(who) + ": " + vb200_strerror(rc) + ": " + vb200_last_error_detail());
}
void* current_stream() { return Stream::current(Device::CUDA).raw_handle(); }
int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }
int64_t positive(const Json& m, const char* key) {
    const int64_t v = m.at(key).as_int();
    if (v <= 0) throw std::runtime_error(std::string("configuration: '") + key + "' must be positive");
    return v;
}
const float* ptr_or_null(const Tensor& t) { return t.defined() ? t.data_ptr<float>() : nullptr; }

// out = x W^T (+ bias) with an epilogue; x and W in `dtype`, bf16 or fp32 out as the epilogue says.
void linear(DType dtype, const void* x, int64_t ldx, const Tensor& w, const Tensor& bias, void* out, int64_t ldo, int64_t M, int64_t N, int epilogue, const char* who) {
    const int dev = w.device_index();
    const int64_t K = w.shape()[1];
    if (dtype == DType::Float32) {
        check(vb200_linear_f32_ex(dev, current_stream(), static_cast<const float*>(x), ldx, w.data_ptr<float>(), K, ptr_or_null(bias), nullptr, static_cast<float*>(out), ldo,
                                  static_cast<int>(M), static_cast<int>(N), static_cast<int>(K), epilogue), who);
        return;
    }
    check(vb200_linear_bias(dev, current_stream(), x, ldx, w.data_ptr<char>(), K, ptr_or_null(bias), out, ldo, static_cast<int>(M), static_cast<int>(N), static_cast<int>(K), epilogue, 0), who);
}

}  // namespace

// ---- dense -----------------------------------------------------------------------------------------

DenseMlp::DenseMlp(int64_t ff, Activation activation, bool bias, int64_t width, int64_t width_ld, DType dtype)
    : ff_(ff), width_(width), width_ld_(width_ld), activation_(activation), bias_(bias), dtype_(dtype) {
    in_ = zeros({in_rows(), width_ld}, dtype, Device::CUDA);
    out_ = zeros({width_ld, act_ld()}, dtype, Device::CUDA);
    if (bias) {
        in_bias_ = zeros({in_rows()}, DType::Float32, Device::CUDA);
        out_bias_ = zeros({width_ld}, DType::Float32, Device::CUDA);
    }
}

int DenseMlp::epilogue() const {
    return activation_ == Activation::GatedRelu ? VB200_EPI_REGLU : activation_ == Activation::GatedSilu ? VB200_EPI_SWIGLU : VB200_EPI_RELU2;
}

std::map<std::string, std::vector<int64_t>> DenseMlp::parameter_shapes() const {
    std::map<std::string, std::vector<int64_t>> m = {{"up", {ff_, width_}}, {"down", {width_, ff_}}};
    if (gated()) m["gate"] = {ff_, width_};
    if (bias_) {
        m["up.b"] = {ff_};
        m["down.b"] = {width_};
        if (gated()) m["gate.b"] = {ff_};
    }
    return m;
}

void DenseMlp::load_parameter(const std::string& name, const float* v) {
    const int64_t step = gated() ? 2 : 1, up0 = gated() ? 1 : 0;
    if (name == "up") load_rows(in_, up0, ff_, width_, v, step);
    else if (name == "gate") load_rows(in_, 0, ff_, width_, v, step);
    else if (name == "down") load_rows(out_, 0, width_, ff_, v);
    else if (name == "up.b") load_vector(in_bias_, up0, ff_, v, step);
    else if (name == "gate.b") load_vector(in_bias_, 0, ff_, v, step);
    else if (name == "down.b") load_vector(out_bias_, 0, width_, v);
    else throw std::runtime_error("DenseMlp: no parameter named " + name);
}

PendingRows DenseMlp::forward(const FeedForwardStep& s) {
    linear(dtype_, s.x, width_ld_, in_, in_bias_, s.act, act_ld(), s.M, in_rows(), epilogue(), "linear(gate, up)");
    linear(dtype_, s.act, act_ld(), out_, out_bias_, s.y, width_ld_, s.M, width_ld_, VB200_EPI_F32, "linear(down)");
    return {};
}

// ---- mixture of experts ----------------------------------------------------------------------------

MixtureOfExperts::Sizes::Sizes(const Json& m) {
    const Json& r = m.at("router");
    experts = positive(r, "experts");
    top = positive(r, "top");
    scale = r.at("scale").as_double();
    ff = positive(m.at("expert"), "ff");
    const Json& g = r.get("groups");
    if (!g.is_null()) {
        groups = positive(g, "count");
        keep = positive(g, "keep");
        if (experts % groups != 0 || keep > groups || top > keep * (experts / groups))
            throw std::runtime_error("configuration: the experts must divide into the groups, and the kept groups hold 'top' experts");
    }
    if (top > experts) throw std::runtime_error("configuration: 'top' exceeds the number of experts");
    const Json& s = m.get("shared");
    if (!s.is_null()) shared = positive(s, "ff");
}

MixtureOfExperts::MixtureOfExperts(const Json& mlp, int64_t width, int64_t width_ld, DType dtype) : z_(mlp), width_(width), width_ld_(width_ld), dtype_(dtype) {
    router_ = zeros({z_.experts, width_ld}, dtype, Device::CUDA);
    correction_ = zeros({z_.experts}, DType::Float32, Device::CUDA);
    in_ = zeros({z_.experts * 2 * z_.ff, width_ld}, dtype, Device::CUDA);
    out_ = zeros({z_.experts * width_ld, pad8(z_.ff)}, dtype, Device::CUDA);
    if (z_.shared > 0) {
        shared_in_ = zeros({2 * z_.shared, width_ld}, dtype, Device::CUDA);
        shared_out_ = zeros({width_ld, pad8(z_.shared)}, dtype, Device::CUDA);
    }
}

std::map<std::string, std::vector<int64_t>> MixtureOfExperts::parameter_shapes() const {
    std::map<std::string, std::vector<int64_t>> m = {{"router", {z_.experts, width_}}, {"correction", {z_.experts}}};
    auto expert = [&](const std::string& p, int64_t ff) {
        m[p + ".gate"] = {ff, width_};
        m[p + ".up"] = {ff, width_};
        m[p + ".down"] = {width_, ff};
    };
    for (int64_t e = 0; e < z_.experts; ++e) expert("e" + std::to_string(e), z_.ff);
    if (z_.shared > 0) expert("shared", z_.shared);
    return m;
}

void MixtureOfExperts::load_parameter(const std::string& name, const float* v) {
    if (name == "router") return load_rows(router_, 0, z_.experts, width_, v);
    if (name == "correction") return load_vector(correction_, 0, z_.experts, v);
    const size_t dot = name.find('.');
    const std::string who = name.substr(0, dot), what = dot == std::string::npos ? "" : name.substr(dot + 1);
    const bool shared = who == "shared";
    const int64_t e = shared ? 0 : std::stoll(who.substr(1)), ff = shared ? z_.shared : z_.ff;
    Tensor &in = shared ? shared_in_ : in_, &out = shared ? shared_out_ : out_;
    if (what == "gate") load_rows(in, e * 2 * ff, ff, width_, v, 2);
    else if (what == "up") load_rows(in, e * 2 * ff + 1, ff, width_, v, 2);
    else if (what == "down") load_rows(out, e * width_ld_, width_, ff, v);
    else throw std::runtime_error("MixtureOfExperts: no parameter named " + name);
}

struct MixtureOfExperts::Args {
    vb200_moe_args a{};
    Args(const MixtureOfExperts& m, int64_t M) {
        a.struct_size = sizeof(a);
        a.device = m.router_.device_index();
        a.stream = current_stream();
        a.dtype = m.dtype_ == DType::Float32 ? VB200_F32 : VB200_BF16;
        a.M = static_cast<int>(M); a.dim = static_cast<int>(m.width_ld_); a.ff = static_cast<int>(m.z_.ff); a.ff_shared = static_cast<int>(m.z_.shared);
        a.experts = static_cast<int>(m.z_.experts); a.top = static_cast<int>(m.z_.top); a.groups = static_cast<int>(m.z_.groups); a.keep = static_cast<int>(m.z_.keep);
        a.scale = static_cast<float>(m.z_.scale);
        a.w_router = m.router_.data_ptr<char>();
        a.correction = m.correction_.data_ptr<float>();
        a.w_in = m.in_.data_ptr<char>();
        a.w_out = m.out_.data_ptr<char>();
        a.ld_out = m.out_.shape()[1];
        if (m.z_.shared > 0) {
            a.w_shared_in = m.shared_in_.data_ptr<char>();
            a.w_shared_out = m.shared_out_.data_ptr<char>();
            a.ld_shared = m.shared_out_.shape()[1];
        }
    }
};

int64_t MixtureOfExperts::workspace_bytes(int64_t M) const {
    const Args x(*this, M);
    return static_cast<int64_t>(vb200_moe_workspace_bytes(&x.a));
}

PendingRows MixtureOfExperts::forward(const FeedForwardStep& s) {
    Args x(*this, s.M);
    x.a.x = s.x;
    x.a.y = s.y;
    x.a.workspace = s.workspace;
    x.a.workspace_bytes = static_cast<size_t>(s.workspace_bytes);
    check(vb200_moe_forward(&x.a), "mixture of experts");
    PendingRows p;
    p.count = vb200_moe_rows(&x.a);
    if (p.count > 0) check(vb200_moe_rows_of(&x.a, &p.rows, &p.gather), "mixture of experts");
    return p;
}

void check_feed_forward(const Json& mlp, const FeedForwardStyle& style) {
    const std::string& kind = mlp.at("kind").as_string();
    if (kind == "dense") (void)positive(mlp, "ff");
    else if (kind == "moe" && style.experts) (void)MixtureOfExperts::Sizes(mlp);
    else throw std::runtime_error("configuration: no feed-forward of kind '" + kind + "'");
}

std::unique_ptr<FeedForward> make_feed_forward(const Json& mlp, const FeedForwardStyle& style, int64_t width, int64_t width_ld, DType dtype) {
    check_feed_forward(mlp, style);
    if (mlp.at("kind").as_string() == "dense") return std::make_unique<DenseMlp>(positive(mlp, "ff"), style.dense, style.dense_bias, width, width_ld, dtype);
    return std::make_unique<MixtureOfExperts>(mlp, width, width_ld, dtype);
}

}  // namespace vesper::nn
