// nn::LatentAttention, nn::SigmoidAttention, nn::Mamba2 and nn::Mamba1 over the C ABI of vesper_b200_hybrid.h.
#include <vesper/nn/sequence_mixer.h>

#include <vesper_b200_hybrid.h>

#include <cuda_runtime.h>

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

namespace {
// rows of `bytes` host bytes, to device rows `step` apart
void copy_rows(char* dst, int64_t bytes, int64_t step, const void* src, int64_t rows) {
    const size_t n = static_cast<size_t>(bytes);
    const cudaError_t rc = cudaMemcpy2D(dst, n * static_cast<size_t>(step), src, n, n, static_cast<size_t>(rows), cudaMemcpyHostToDevice);
    if (rc != cudaSuccess) throw std::runtime_error(std::string("loading a parameter: ") + cudaGetErrorString(rc));
}
}  // namespace

void load_rows(Tensor& dst, int64_t row0, int64_t rows, int64_t cols, const float* host_values, int64_t step) {
    const int64_t ld = dst.shape()[1], esz = dst.dtype() == DType::Float32 ? 4 : 2;
    if (row0 < 0 || cols > ld || row0 + (rows - 1) * step >= dst.shape()[0]) throw std::runtime_error("load_rows: rows outside the matrix");
    char* base = dst.data_ptr<char>() + row0 * ld * esz;
    if (esz == 4) {
        std::vector<float> tmp(static_cast<size_t>(rows * ld), 0.0f);
        for (int64_t r = 0; r < rows; ++r) std::copy(host_values + r * cols, host_values + (r + 1) * cols, tmp.begin() + r * ld);
        copy_rows(base, ld * esz, step, tmp.data(), rows);
    } else {
        std::vector<uint16_t> tmp(static_cast<size_t>(rows * ld), 0);
        for (int64_t r = 0; r < rows; ++r)
            for (int64_t c = 0; c < cols; ++c) tmp[static_cast<size_t>(r * ld + c)] = float_to_bf16(host_values[r * cols + c]);
        copy_rows(base, ld * esz, step, tmp.data(), rows);
    }
}

void load_vector(Tensor& dst, int64_t first, int64_t n, const float* host_values, int64_t step) {
    if (first < 0 || first + (n - 1) * step >= static_cast<int64_t>(dst.numel())) throw std::runtime_error("load_vector: outside the vector");
    copy_rows(dst.data_ptr<char>() + first * 4, 4, step, host_values, n);
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

// ---- sigmoid attention with mixed heads ------------------------------------------------------------

int64_t distance_bucket(int64_t n, int64_t rows, double reach) {
    const int64_t half = rows / 2;
    if (n < half) return n;
    if (half == 0 || reach <= static_cast<double>(half)) return rows - 1;
    // the quotient of two logarithms may round below an edge it lands on exactly
    const double x = std::log(static_cast<double>(n) / static_cast<double>(half)) / std::log(reach / static_cast<double>(half)) * static_cast<double>(rows - half);
    return std::min(rows - 1, half + static_cast<int64_t>(std::floor(x + 1e-9)));
}

SigmoidAttention::Sizes::Sizes(const Json& m) {
    heads = positive(m, "heads");
    kv_heads = positive(m, "kv_heads");
    dim = positive(m, "dim");
    vdim = positive(m, "vdim");
    if (heads % kv_heads != 0) throw std::runtime_error("configuration: heads must be divisible by kv_heads");
    scale = m.at("scale").as_double();
    reach = m.at("bias_max").as_double();
    const Json& temp = m.get("q_temp");
    if (!temp.is_null()) {
        temp_coef = temp.at("coef").as_double();
        temp_every = positive(temp, "every");
    }
    const Json& mix = m.get("v_mix");
    value_mixing = !mix.is_null() && mix.as_bool();
}

SigmoidAttention::SigmoidAttention(const Json& m, int64_t width, int64_t width_ld, double eps, DType dtype) : SequenceMixer(width, width_ld, eps, dtype), z_(m) {
    proj_rows_ = z_.heads * (z_.dim + 1) + z_.kv_heads * (z_.dim + z_.vdim);
    mixed_cols_ = z_.heads * z_.vdim;
    in_weight_ = zeros({proj_rows_, width_ld}, dtype, Device::CUDA);
    out_weight_ = zeros({width_ld, mixed_ld()}, dtype, Device::CUDA);
    talk_ = zeros({z_.heads, z_.heads}, DType::Float32, Device::CUDA);
    bias_ = zeros({z_.heads, 1}, DType::Float32, Device::CUDA);
}

std::map<std::string, std::vector<int64_t>> SigmoidAttention::parameter_shapes() const {
    std::map<std::string, std::vector<int64_t>> m = {{"q", {z_.heads * z_.dim, width_}}, {"k", {z_.kv_heads * z_.dim, width_}}, {"v", {z_.kv_heads * z_.vdim, width_}}, {"g", {z_.heads, width_}},
                                                     {"rel", {-1, z_.heads}}, {"talk", {z_.heads, z_.heads}}, {"pb", {z_.heads}}, {"o", {width_, z_.heads * z_.vdim}}};
    if (z_.value_mixing) m["vmix"] = {};
    return m;
}

void SigmoidAttention::set_free_size(const std::string& name, int64_t numel) {
    if (name == "rel") bias_rows_ = numel / z_.heads;
}

void SigmoidAttention::load_parameter(const std::string& name, const float* v) {
    const int64_t q = z_.heads * z_.dim, k = z_.kv_heads * z_.dim, vv = z_.kv_heads * z_.vdim;
    if (name == "q") load_rows(in_weight_, 0, q, width_, v);
    else if (name == "k") load_rows(in_weight_, q, k, width_, v);
    else if (name == "v") load_rows(in_weight_, q + k, vv, width_, v);
    else if (name == "g") load_rows(in_weight_, q + k + vv, z_.heads, width_, v);
    else if (name == "o") load_rows(out_weight_, 0, width_, mixed_cols_, v);
    else if (name == "vmix") lambda_ = v[0];
    else if (name == "rel") { host_rel_.assign(v, v + bias_rows_ * z_.heads); fold_bias(); }
    else if (name == "pb") { host_offset_.assign(v, v + z_.heads); fold_bias(); }
    else if (name == "talk") { host_talk_.assign(v, v + z_.heads * z_.heads); load_vector(talk_, 0, z_.heads * z_.heads, v); fold_bias(); }
    else throw std::runtime_error("SigmoidAttention: no parameter named " + name);
}

// What a score gets that depends on its head and distance only, [heads, distances]: the relative bias mixed like the scores, plus the
// head's offset.  The last distance stands for all beyond it.
void SigmoidAttention::fold_bias() {
    if (host_rel_.empty() || host_talk_.empty() || host_offset_.empty()) return;
    std::vector<int64_t> bucket;
    for (int64_t n = 0;; ++n) {
        bucket.push_back(distance_bucket(n, bias_rows_, z_.reach));
        if (bucket.back() == bias_rows_ - 1) break;
    }
    const int64_t len = static_cast<int64_t>(bucket.size());
    std::vector<float> folded(static_cast<size_t>(z_.heads * len));
    for (int64_t h = 0; h < z_.heads; ++h) {
        std::vector<float> by_row(static_cast<size_t>(bias_rows_));
        for (int64_t r = 0; r < bias_rows_; ++r) {
            double x = host_offset_[static_cast<size_t>(h)];
            for (int64_t g = 0; g < z_.heads; ++g) x += static_cast<double>(host_talk_[static_cast<size_t>(h * z_.heads + g)]) * host_rel_[static_cast<size_t>(r * z_.heads + g)];
            by_row[static_cast<size_t>(r)] = static_cast<float>(x);
        }
        for (int64_t n = 0; n < len; ++n) folded[static_cast<size_t>(h * len + n)] = by_row[static_cast<size_t>(bucket[static_cast<size_t>(n)])];
    }
    bias_ = empty({z_.heads, len}, DType::Float32, Device::CUDA);
    bias_.copy_from_host(folded.data());
}

std::unique_ptr<SequenceState> SigmoidAttention::make_state(int64_t slots, int64_t max_len) const {
    auto st = std::make_unique<SequenceState>();
    st->ring = zeros({slots, max_len, pad8(z_.kv_heads * z_.dim)}, dtype_, Device::CUDA);
    st->values = zeros({slots, max_len, pad8(z_.kv_heads * z_.vdim)}, dtype_, Device::CUDA);
    return st;
}

struct SigmoidAttention::Args {
    vb200_sigattn_args a{};
    Args(const SigmoidAttention& m, const MixerStep& st, int64_t cap) {
        a.struct_size = sizeof(a);
        a.device = m.in_weight_.device_index();
        a.stream = current_stream();
        a.dtype = m.dtype_ == DType::Float32 ? VB200_F32 : VB200_BF16;
        a.B = static_cast<int>(st.B); a.T = static_cast<int>(st.T);
        a.H = static_cast<int>(m.z_.heads); a.G = static_cast<int>(m.z_.kv_heads); a.dim = static_cast<int>(m.z_.dim); a.vdim = static_cast<int>(m.z_.vdim);
        a.scale = static_cast<float>(m.z_.scale); a.eps = static_cast<float>(m.eps_);
        a.temp_coef = static_cast<float>(m.z_.temp_coef); a.temp_every = static_cast<int>(std::min<int64_t>(m.z_.temp_every, INT32_MAX));
        a.ldp = m.proj_ld(); a.ldo = m.mixed_ld();
        a.ldk = pad8(m.z_.kv_heads * m.z_.dim); a.ldv = pad8(m.z_.kv_heads * m.z_.vdim);
        a.talk = m.talk_.data_ptr<float>(); a.bias = m.bias_.data_ptr<float>(); a.n_bias = static_cast<int>(m.bias_.shape()[1]);
        a.lambda = m.lambda_;
        a.slots = st.slots; a.pos = st.pos;
        a.cap = static_cast<int>(std::min<int64_t>(cap, INT32_MAX));
        a.start_pos = static_cast<int>(st.start_pos);
        a.max_len = static_cast<int>(std::min<int64_t>(st.max_len, INT32_MAX));
    }
};

int64_t SigmoidAttention::workspace_bytes(const MixerStep& st) const {
    const Args x(*this, st, INT32_MAX);
    return static_cast<int64_t>(vb200_sigattn_workspace_bytes(&x.a));
}

void SigmoidAttention::forward(const MixerStep& st, SequenceState& state, Tensor& projected, Tensor& mixed) {
    Args x(*this, st, state.ring.shape()[1]);
    x.a.proj = projected.data_ptr<char>();
    x.a.k_cache = state.ring.data_ptr<char>();
    x.a.v_cache = state.values.data_ptr<char>();
    x.a.out = mixed.data_ptr<char>();
    x.a.workspace = st.workspace;
    x.a.workspace_bytes = static_cast<size_t>(st.workspace_bytes);
    if (z_.value_mixing) {
        if (!st.values) throw std::runtime_error("SigmoidAttention: value mixing needs the step's shared values");
        x.a.first_values = st.values->data;
        x.a.value_role = st.values->filled ? 2 : 1;
        st.values->filled = true;
    }
    check(vb200_sigattn_forward(&x.a), "sigmoid attention");
}

// ---- Mamba-1 -------------------------------------------------------------------------------------

Mamba1::Sizes::Sizes(const Json& m) {
    inner = positive(m, "inner");
    state = positive(m, "state");
    rank = positive(m, "dt_rank");
    taps = positive(m, "conv");
    inner8 = pad8(inner); state8 = pad8(state); rank8 = pad8(rank);
}

Mamba1::Mamba1(const Json& m, int64_t width, int64_t width_ld, double eps, DType dtype) : SequenceMixer(width, width_ld, eps, dtype), z_(m) {
    proj_rows_ = 2 * z_.inner8;
    mixed_cols_ = z_.inner;
    in_weight_ = zeros({proj_rows_, width_ld}, dtype, Device::CUDA);
    out_weight_ = zeros({width_ld, mixed_ld()}, dtype, Device::CUDA);
    w_x_ = zeros({z_.rank8 + 2 * z_.state8, z_.inner8}, dtype, Device::CUDA);
    w_dt_ = zeros({z_.inner8, z_.rank8}, dtype, Device::CUDA);
    conv_w_ = zeros({z_.inner8, z_.taps}, DType::Float32, Device::CUDA);
    conv_b_ = zeros({z_.inner8}, DType::Float32, Device::CUDA);
    dt_bias_ = zeros({z_.inner8}, DType::Float32, Device::CUDA);
    a_ = zeros({z_.inner8, z_.state8}, DType::Float32, Device::CUDA);
    d_ = zeros({z_.inner8}, DType::Float32, Device::CUDA);
}

std::map<std::string, std::vector<int64_t>> Mamba1::parameter_shapes() const {
    return {{"in", {2 * z_.inner, width_}}, {"conv", {z_.inner, z_.taps}}, {"conv.b", {z_.inner}}, {"x", {z_.rank + 2 * z_.state, z_.inner}}, {"dt", {z_.inner, z_.rank}}, {"dt.b", {z_.inner}},
            {"A_log", {z_.inner, z_.state}}, {"D", {z_.inner}}, {"o", {width_, z_.inner}}};
}

void Mamba1::load_parameter(const std::string& name, const float* v) {
    if (name == "in") {
        load_rows(in_weight_, 0, z_.inner, width_, v);
        load_rows(in_weight_, z_.inner8, z_.inner, width_, v + z_.inner * width_);
    } else if (name == "x") {
        load_rows(w_x_, 0, z_.rank, z_.inner, v);
        load_rows(w_x_, z_.rank8, z_.state, z_.inner, v + z_.rank * z_.inner);
        load_rows(w_x_, z_.rank8 + z_.state8, z_.state, z_.inner, v + (z_.rank + z_.state) * z_.inner);
    } else if (name == "A_log") {
        std::vector<float> a(static_cast<size_t>(z_.inner * z_.state));
        for (size_t i = 0; i < a.size(); ++i) a[i] = static_cast<float>(-std::exp(static_cast<double>(v[i])));
        load_rows(a_, 0, z_.inner, z_.state, a.data());
    } else if (name == "conv") load_rows(conv_w_, 0, z_.inner, z_.taps, v);
    else if (name == "conv.b") load_vector(conv_b_, 0, z_.inner, v);
    else if (name == "dt") load_rows(w_dt_, 0, z_.inner, z_.rank, v);
    else if (name == "dt.b") load_vector(dt_bias_, 0, z_.inner, v);
    else if (name == "D") load_vector(d_, 0, z_.inner, v);
    else if (name == "o") load_rows(out_weight_, 0, width_, z_.inner, v);
    else throw std::runtime_error("Mamba1: no parameter named " + name);
}

std::unique_ptr<SequenceState> Mamba1::make_state(int64_t slots, int64_t) const {
    auto st = std::make_unique<SequenceState>();
    st->ring = zeros({slots, z_.taps, z_.inner8}, dtype_, Device::CUDA);
    st->recurrent = zeros({slots, z_.inner8, z_.state8}, DType::Float32, Device::CUDA);
    return st;
}

struct Mamba1::Args {
    vb200_selective_args a{};
    Args(const Mamba1& m, const MixerStep& st) {
        a.struct_size = sizeof(a);
        a.device = m.in_weight_.device_index();
        a.stream = current_stream();
        a.dtype = m.dtype_ == DType::Float32 ? VB200_F32 : VB200_BF16;
        a.B = static_cast<int>(st.B); a.T = static_cast<int>(st.T); a.inner = static_cast<int>(m.z_.inner8); a.N = static_cast<int>(m.z_.state8);
        a.rank = static_cast<int>(m.z_.rank8); a.taps = static_cast<int>(m.z_.taps);
        a.ldp = m.proj_ld(); a.ldo = m.mixed_ld();
        a.conv_w = m.conv_w_.data_ptr<float>(); a.conv_b = m.conv_b_.data_ptr<float>();
        a.w_x = m.w_x_.data_ptr<char>(); a.w_dt = m.w_dt_.data_ptr<char>();
        a.dt_bias = m.dt_bias_.data_ptr<float>(); a.A = m.a_.data_ptr<float>(); a.D = m.d_.data_ptr<float>();
        a.slots = st.slots; a.pos = st.pos;
    }
};

int64_t Mamba1::workspace_bytes(const MixerStep& st) const {
    const Args x(*this, st);
    return static_cast<int64_t>(vb200_selective_workspace_bytes(&x.a));
}

void Mamba1::forward(const MixerStep& st, SequenceState& state, Tensor& projected, Tensor& mixed) {
    Args x(*this, st);
    x.a.proj = projected.data_ptr<char>();
    x.a.conv_state = state.ring.data_ptr<char>();
    x.a.state = state.recurrent.data_ptr<float>();
    x.a.out = mixed.data_ptr<char>();
    x.a.workspace = st.workspace;
    x.a.workspace_bytes = static_cast<size_t>(st.workspace_bytes);
    check(vb200_selective_forward(&x.a), "mamba1");
}

int64_t check_mixer(const std::string& type, const Json& mixer) {
    if (type == "attention") return SigmoidAttention::Sizes(mixer).shared_value_cols();
    if (type == "mamba1") (void)Mamba1::Sizes(mixer);
    else if (type != "latent_attention" && type != "mamba2") throw std::runtime_error("configuration: no sequence mixer of type '" + type + "'");
    return 0;
}

std::unique_ptr<SequenceMixer> make_mixer(const std::string& type, const Json& mixer, int64_t width, int64_t width_ld, double eps, DType dtype) {
    if (type == "latent_attention") return std::make_unique<LatentAttention>(mixer, width, width_ld, eps, dtype);
    if (type == "attention") return std::make_unique<SigmoidAttention>(mixer, width, width_ld, eps, dtype);
    if (type == "mamba1") return std::make_unique<Mamba1>(mixer, width, width_ld, eps, dtype);
    if (type == "mamba2") return std::make_unique<Mamba2>(mixer, width, width_ld, eps, dtype);
    throw std::runtime_error("configuration: no sequence mixer of type '" + type + "'");
}

}  // namespace vesper::nn
