// nn::LatentAttention and nn::Mamba2 over the C ABI of vesper_b200_hybrid.h.
#include <vesper/nn/sequence_mixer.h>

#include <vesper_b200_hybrid.h>

#include <algorithm>
#include <cmath>
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

}  // namespace

void load_rows(Tensor& dst, int64_t row0, int64_t rows, int64_t cols, const float* host_values) {
    const int64_t ld = dst.shape()[1];
    Tensor part = dst.narrow(0, row0, rows);
    if (dst.dtype() == DType::Float32) {
        std::vector<float> tmp(static_cast<size_t>(rows * ld), 0.0f);
        for (int64_t r = 0; r < rows; ++r) std::copy(host_values + r * cols, host_values + (r + 1) * cols, tmp.begin() + r * ld);
        part.copy_from_host(tmp.data());
    } else {
        std::vector<uint16_t> tmp(static_cast<size_t>(rows * ld), 0);
        for (int64_t r = 0; r < rows; ++r)
            for (int64_t c = 0; c < cols; ++c) tmp[static_cast<size_t>(r * ld + c)] = float_to_bf16(host_values[r * cols + c]);
        part.copy_from_host(tmp.data());
    }
}

Tensor vector_from_host(const float* host_values, int64_t n) {
    Tensor t = empty({n}, DType::Float32, Device::CUDA);
    t.copy_from_host(host_values);
    return t;
}

// ---- latent attention ----------------------------------------------------------------------------

LatentAttention::LatentAttention(const Json& m, int64_t width, int64_t width_ld, double eps, DType dtype) : SequenceMixer(width, width_ld, eps, dtype) {
    heads_ = positive(m, "heads");
    dim_ = positive(m, "dim");
    rot_dim_ = positive(m, "rot_dim");
    vdim_ = positive(m, "vdim");
    rank_ = positive(m, "kv_rank");
    window_ = positive(m.at("mask"), "size");
    scale_ = m.at("scale").as_double();
    const Json& rot = m.at("rot");
    if (rot.int_or("dims", rot_dim_) != rot_dim_) throw std::runtime_error("configuration: latent attention rotates all of rot_dim, but rot.dims differs");
    if (rot_dim_ % 2 != 0) throw std::runtime_error("configuration: rot_dim must be even");
    const double base = rot.at("base").as_double();
    std::vector<double> f(static_cast<size_t>(rot_dim_ / 2));
    for (size_t i = 0; i < f.size(); ++i) f[i] = std::pow(base, -2.0 * static_cast<double>(i) / static_cast<double>(rot_dim_));
    inv_freq_ = empty({rot_dim_ / 2}, DType::Float64, Device::CUDA);
    inv_freq_.copy_from_host(f.data());
    proj_rows_ = heads_ * (dim_ + rot_dim_) + rank_ + rot_dim_;
    mixed_cols_ = heads_ * vdim_;
    in_weight_ = zeros({proj_rows_, width_ld}, dtype, Device::CUDA);
    out_weight_ = zeros({width_ld, mixed_ld()}, dtype, Device::CUDA);
    expand_ = zeros({heads_ * (dim_ + vdim_), pad8(rank_)}, dtype, Device::CUDA);
    latent_norm_ = zeros({rank_}, DType::Float32, Device::CUDA);
    sink_ = zeros({heads_}, DType::Float32, Device::CUDA);
}

std::map<std::string, std::vector<int64_t>> LatentAttention::parameter_shapes() const {
    return {{"q", {heads_ * (dim_ + rot_dim_), width_}}, {"dkv", {rank_ + rot_dim_, width_}}, {"dkv.norm", {rank_}}, {"uk", {heads_ * dim_, rank_}},
            {"uv", {heads_ * vdim_, rank_}}, {"sink", {heads_}}, {"o", {width_, heads_ * vdim_}}};
}

void LatentAttention::load_parameter(const std::string& name, const float* v) {
    if (name == "q") load_rows(in_weight_, 0, heads_ * (dim_ + rot_dim_), width_, v);
    else if (name == "dkv") load_rows(in_weight_, heads_ * (dim_ + rot_dim_), rank_ + rot_dim_, width_, v);
    else if (name == "uk") load_rows(expand_, 0, heads_ * dim_, rank_, v);
    else if (name == "uv") load_rows(expand_, heads_ * dim_, heads_ * vdim_, rank_, v);
    else if (name == "o") load_rows(out_weight_, 0, width_, heads_ * vdim_, v);
    else if (name == "dkv.norm") latent_norm_ = vector_from_host(v, rank_);
    else if (name == "sink") sink_ = vector_from_host(v, heads_);
    else throw std::runtime_error("LatentAttention: no parameter named " + name);
}

std::unique_ptr<SequenceState> LatentAttention::make_state(int64_t slots, int64_t max_len) const {
    auto st = std::make_unique<SequenceState>();
    const int64_t ring = std::min(window_, max_len);
    st->ring = zeros({slots, ring, vb200_latent_row(static_cast<int>(rank_), static_cast<int>(rot_dim_))}, dtype_, Device::CUDA);
    return st;
}

struct LatentAttention::Args {
    vb200_latent_args a{};
    int64_t ctx = 0, ldkv = 0;
    int64_t latent_bytes = 0, kv_bytes = 0, split_bytes = 0;
    Args(const LatentAttention& m, const MixerStep& st, int64_t ring) {
        const int64_t esz = m.dtype_ == DType::Float32 ? 4 : 2;
        a.struct_size = sizeof(a);
        a.device = m.in_weight_.device_index();
        a.stream = current_stream();
        a.dtype = m.dtype_ == DType::Float32 ? VB200_F32 : VB200_BF16;
        a.B = static_cast<int>(st.B); a.T = static_cast<int>(st.T); a.H = static_cast<int>(m.heads_);
        a.dim = static_cast<int>(m.dim_); a.rot_dim = static_cast<int>(m.rot_dim_); a.vdim = static_cast<int>(m.vdim_); a.rank = static_cast<int>(m.rank_);
        a.window = static_cast<int>(std::min<int64_t>(m.window_, INT32_MAX)); a.ring = static_cast<int>(ring);
        a.scale = static_cast<float>(m.scale_); a.eps = static_cast<float>(m.eps_);
        a.inv_freq = m.inv_freq_.data_ptr<double>();
        a.c_norm = m.latent_norm_.data_ptr<float>();
        a.w_uk = m.expand_.data_ptr<char>();
        a.ldu = m.expand_.shape()[1];
        a.w_uv = m.expand_.data_ptr<char>() + m.heads_ * m.dim_ * a.ldu * esz;
        a.sink = m.sink_.data_ptr<float>();
        a.slots = st.slots; a.pos = st.pos;
        a.ldp = m.proj_ld(); a.ldo = m.mixed_ld();
        a.ldc = vb200_latent_row(a.rank, a.rot_dim);
        a.start_pos = static_cast<int>(st.start_pos);
        a.max_len = static_cast<int>(std::min<int64_t>(st.max_len, INT32_MAX));
        if (st.T > 1) {
            ctx = vb200_latent_context(a.start_pos, a.T, a.window);
            ldkv = pad8(m.heads_ * (m.dim_ + m.vdim_));
            a.ldkv = ldkv;
            latent_bytes = (st.B * ctx * a.ldc * esz + 255) / 256 * 256;
            kv_bytes = (st.B * ctx * ldkv * esz + 255) / 256 * 256;
        } else {
            split_bytes = static_cast<int64_t>(vb200_latent_workspace_bytes(&a));
        }
    }
};

int64_t LatentAttention::workspace_bytes(const MixerStep& st) const {
    const Args x(*this, st, window_ < INT32_MAX ? window_ : INT32_MAX);
    return x.latent_bytes + x.kv_bytes + x.split_bytes;
}

void LatentAttention::forward(const MixerStep& st, SequenceState& state, Tensor& projected, Tensor& mixed) {
    Args x(*this, st, state.ring.shape()[1]);
    vb200_latent_args& a = x.a;
    if (st.workspace_bytes < x.latent_bytes + x.kv_bytes + x.split_bytes) throw std::runtime_error("LatentAttention: workspace too small");
    a.proj = projected.data_ptr<char>();
    a.cache = state.ring.data_ptr<char>();
    a.out = mixed.data_ptr<char>();
    if (st.T == 1) {
        a.workspace = st.workspace;
        a.workspace_bytes = static_cast<size_t>(st.workspace_bytes);
        check(vb200_latent_decode(&a), "latent attention(decode)");
        return;
    }
    a.ctx_latent = st.workspace;
    a.ctx_kv = st.workspace + x.latent_bytes;
    check(vb200_latent_append(&a), "latent attention(append)");
    const int M = static_cast<int>(st.B * x.ctx), N = static_cast<int>(heads_ * (dim_ + vdim_)), K = static_cast<int>(a.ldu);
    if (dtype_ == DType::Float32)
        check(vb200_linear_f32(a.device, a.stream, static_cast<const float*>(a.ctx_latent), a.ldc, expand_.data_ptr<float>(), a.ldu, nullptr,
                               static_cast<float*>(a.ctx_kv), x.ldkv, M, N, static_cast<int>(rank_)), "linear(keys, values)");
    else
        check(vb200_linear(a.device, a.stream, a.ctx_latent, a.ldc, expand_.data_ptr<char>(), a.ldu, a.ctx_kv, x.ldkv, M, N, K, VB200_EPI_BF16, 0),
              "linear(keys, values)");
    check(vb200_latent_prefill(&a), "latent attention(prefill)");
}

// ---- Mamba-2 -------------------------------------------------------------------------------------

Mamba2::Mamba2(const Json& m, int64_t width, int64_t width_ld, double eps, DType dtype) : SequenceMixer(width, width_ld, eps, dtype) {
    heads_ = positive(m, "heads");
    vdim_ = positive(m, "vdim");
    state_ = positive(m, "state");
    groups_ = positive(m, "groups");
    taps_ = positive(m, "conv");
    norm_groups_ = positive(m, "norm_groups");
    if (heads_ % groups_ != 0) throw std::runtime_error("configuration: heads must be divisible by groups");
    if ((heads_ * vdim_) % norm_groups_ != 0) throw std::runtime_error("configuration: heads * vdim must be divisible by norm_groups");
    channels_ = heads_ * vdim_ + 2 * groups_ * state_;
    proj_rows_ = 2 * heads_ * vdim_ + 2 * groups_ * state_ + heads_;
    mixed_cols_ = heads_ * vdim_;
    in_weight_ = zeros({proj_rows_, width_ld}, dtype, Device::CUDA);
    out_weight_ = zeros({width_ld, mixed_ld()}, dtype, Device::CUDA);
    conv_w_ = zeros({channels_ * taps_}, DType::Float32, Device::CUDA);
    conv_b_ = zeros({channels_}, DType::Float32, Device::CUDA);
    dt_bias_ = zeros({heads_}, DType::Float32, Device::CUDA);
    a_log_ = zeros({heads_}, DType::Float32, Device::CUDA);
    d_ = zeros({heads_}, DType::Float32, Device::CUDA);
    norm_ = zeros({heads_ * vdim_}, DType::Float32, Device::CUDA);
}

std::map<std::string, std::vector<int64_t>> Mamba2::parameter_shapes() const {
    return {{"in", {proj_rows_, width_}}, {"conv", {channels_, taps_}}, {"conv.b", {channels_}}, {"dt_bias", {heads_}}, {"A_log", {heads_}}, {"D", {heads_}},
            {"norm", {heads_ * vdim_}}, {"o", {width_, heads_ * vdim_}}};
}

void Mamba2::load_parameter(const std::string& name, const float* v) {
    if (name == "in") load_rows(in_weight_, 0, proj_rows_, width_, v);
    else if (name == "o") load_rows(out_weight_, 0, width_, heads_ * vdim_, v);
    else if (name == "conv") conv_w_ = vector_from_host(v, channels_ * taps_);
    else if (name == "conv.b") conv_b_ = vector_from_host(v, channels_);
    else if (name == "dt_bias") dt_bias_ = vector_from_host(v, heads_);
    else if (name == "A_log") a_log_ = vector_from_host(v, heads_);
    else if (name == "D") d_ = vector_from_host(v, heads_);
    else if (name == "norm") norm_ = vector_from_host(v, heads_ * vdim_);
    else throw std::runtime_error("Mamba2: no parameter named " + name);
}

std::unique_ptr<SequenceState> Mamba2::make_state(int64_t slots, int64_t) const {
    auto st = std::make_unique<SequenceState>();
    st->ring = zeros({slots, taps_, channels_}, dtype_, Device::CUDA);
    st->recurrent = zeros({slots, heads_, state_, (vdim_ + 3) / 4 * 4}, DType::Float32, Device::CUDA);
    return st;
}

struct Mamba2::Args {
    vb200_ssd_args a{};
    Args(const Mamba2& m, const MixerStep& st) {
        a.struct_size = sizeof(a);
        a.device = m.in_weight_.device_index();
        a.stream = current_stream();
        a.dtype = m.dtype_ == DType::Float32 ? VB200_F32 : VB200_BF16;
        a.B = static_cast<int>(st.B); a.T = static_cast<int>(st.T); a.H = static_cast<int>(m.heads_); a.P = static_cast<int>(m.vdim_);
        a.N = static_cast<int>(m.state_); a.G = static_cast<int>(m.groups_); a.taps = static_cast<int>(m.taps_); a.norm_groups = static_cast<int>(m.norm_groups_);
        a.eps = static_cast<float>(m.eps_);
        a.ldp = m.proj_ld(); a.ldo = m.mixed_ld();
        a.conv_w = m.conv_w_.data_ptr<float>(); a.conv_b = m.conv_b_.data_ptr<float>();
        a.dt_bias = m.dt_bias_.data_ptr<float>(); a.A_log = m.a_log_.data_ptr<float>(); a.D = m.d_.data_ptr<float>(); a.norm_w = m.norm_.data_ptr<float>();
        a.slots = st.slots; a.pos = st.pos;
    }
};

int64_t Mamba2::workspace_bytes(const MixerStep& st) const {
    const Args x(*this, st);
    return static_cast<int64_t>(vb200_ssd_workspace_bytes(&x.a));
}

void Mamba2::forward(const MixerStep& st, SequenceState& state, Tensor& projected, Tensor& mixed) {
    Args x(*this, st);
    x.a.proj = projected.data_ptr<char>();
    x.a.conv_state = state.ring.data_ptr<char>();
    x.a.state = state.recurrent.data_ptr<float>();
    x.a.out = mixed.data_ptr<char>();
    x.a.workspace = st.workspace;
    x.a.workspace_bytes = static_cast<size_t>(st.workspace_bytes);
    check(vb200_ssd_forward(&x.a), "mamba2");
}

std::unique_ptr<SequenceMixer> make_mixer(const std::string& type, const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype) {
    if (type == "latent_attention") return std::make_unique<LatentAttention>(mixer, width, width_ld, eps, dtype);
    if (type == "mamba2") return std::make_unique<Mamba2>(mixer, width, width_ld, eps, dtype);
    throw std::runtime_error("configuration: no sequence mixer of type '" + type + "'");
}

}  // namespace vesper::nn
