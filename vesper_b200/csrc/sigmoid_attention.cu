// Sigmoid attention with mixed heads: everything around the tensor-core kernels, and the CUDA-core form of the attention
// itself (fp32, and sizes those kernels do not take).
//
// The scores of head h are sum_g talk[h, g] * scale * (q_g . k_group(g)).  The sum over the query heads of one key / value head is
// taken before the product with the keys, q'[h, group, :] = scale * sum_{g in group} talk[h, g] q_g, so a score is one dot product of
// q'_h [G * dim] with the concatenated keys of a position, and mixing costs no exchange between heads.
#include "hybrid.cuh"

#include <type_traits>

namespace vb200 {
namespace {

struct SigParams {
    int B, T, H, G, dim, vdim, R;         // R = H / G
    float scale, eps, temp_coef;
    int temp_every, n_bias, cap, qld, splits;
    long long ldp, ldk, ldv, ldo;
    int value_role;
    float lambda;
    const float *talk, *bias;
    const int *slots, *pos;
    int *status;
};

constexpr int kAppendThreads = 128, kHeadSlice = 4;

// grid (ceil(T / tokens), B, G), a few tokens and one key / value head with its query heads: norms, temperature, the new cache rows, and that
// group's columns of q' for every head.  RM: query heads of a group, rounded up to a power of two (0: more than eight, or an odd head size).
template <typename T, typename QT, int RM>
__global__ void __launch_bounds__(kAppendThreads)
sig_append_kernel(SigParams p, int tokens, const T* __restrict__ proj, T* __restrict__ kc, T* __restrict__ vc, T* __restrict__ first, QT* __restrict__ qm) {
    extern __shared__ __align__(16) float qs[];          // [tokens][R * dim] scaled queries, then this group's columns of talk [H, RM]
    const int q_ld = (p.R * p.dim + 3) / 4 * 4;
    float* tk = qs + tokens * q_ld;
    const int t0 = blockIdx.x * tokens, b = blockIdx.y, g = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nt = min(tokens, p.T - t0);
    const int t_ld = RM > 0 ? RM : p.R;
    for (int i = tid; i < p.H * t_ld; i += kAppendThreads) {
        const int h = i / t_ld, r = i - h * t_ld;
        tk[i] = r < p.R ? __ldg(p.talk + h * p.H + g * p.R + r) : 0.f;
    }
    pdl_begin();
    const long long m0 = static_cast<long long>(b) * p.T + t0;
    const int pos0 = p.pos[b] + t0, fit = min(nt, p.cap - pos0);                     // tokens that the cache has room for
    const long long row0 = static_cast<long long>(p.slots ? p.slots[b] : b) * p.cap + pos0;
    const int vcols = p.G * p.vdim;
    if (fit < nt && g == 0 && tid == 0) atomicCAS(p.status, 0, (2 << 24) | b);
    const T* vsrc = proj + m0 * p.ldp + (p.H + p.G) * p.dim + g * p.vdim;
    for (int u = 0; u < nt; ++u)
        for (int i = tid; i < p.vdim; i += kAppendThreads) {
            const T raw = vsrc[u * p.ldp + i];
            const long long shared = (m0 + u) * vcols + g * p.vdim + i;
            float v = Elem<T>::to_f(raw);
            if (p.value_role == 1) first[shared] = raw;
            else if (p.value_role == 2) v = (1.0f - p.lambda) * v + p.lambda * Elem<T>::to_f(first[shared]);
            if (u < fit) vc[(row0 + u) * p.ldv + g * p.vdim + i] = Elem<T>::from_f(v);
        }
    const float scale = p.scale * (sizeof(QT) == 2 ? -kLog2e : 1.0f);                // the tensor-core kernels compute 2^(-score log2 e)
    for (int k = warp; k < nt * (p.R + 1); k += kAppendThreads / 32) {               // a token's query heads of the group, then its key head
        const int u = k / (p.R + 1), h = k - u * (p.R + 1);
        const T* x = proj + (m0 + u) * p.ldp + (h < p.R ? g * p.R + h : p.H + g) * p.dim;
        float keep[4], ss = 0.f;                         // the first 128 columns stay in registers
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = lane + 32 * j;
            keep[j] = i < p.dim ? Elem<T>::to_f(x[i]) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) ss = fmaf(keep[j], keep[j], ss);
        for (int i = lane + 128; i < p.dim; i += 32) { const float v = Elem<T>::to_f(x[i]); ss = fmaf(v, v, ss); }
        float f = 1.0f / sqrtf(warp_sum_f(ss) / static_cast<float>(p.dim) + p.eps);
        if (h < p.R) {
            f *= scale;
            if (p.temp_every > 0) f *= 1.0f + p.temp_coef * logf(static_cast<float>((pos0 + u + 1) / p.temp_every) + 1.0f);
            float* dst = qs + u * q_ld + h * p.dim;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (lane + 32 * j < p.dim) dst[lane + 32 * j] = keep[j] * f;
            for (int i = lane + 128; i < p.dim; i += 32) dst[i] = Elem<T>::to_f(x[i]) * f;
        } else if (u < fit) {
            T* dst = kc + (row0 + u) * p.ldk + g * p.dim;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (lane + 32 * j < p.dim) dst[lane + 32 * j] = Elem<T>::from_f(keep[j] * f);
            for (int i = lane + 128; i < p.dim; i += 32) dst[i] = Elem<T>::from_f(Elem<T>::to_f(x[i]) * f);
        }
    }
    __syncthreads();
    const long long token_ld = static_cast<long long>(p.H) * p.qld;
    QT* out = qm + m0 * token_ld + g * p.dim;
    if constexpr (RM > 0) {                              // two columns and a slice of the heads per step, whose mixing weights serve all tokens
        const int slices = (p.H + kHeadSlice - 1) / kHeadSlice, pairs = p.dim / 2;
        for (int i = tid; i < pairs * slices; i += kAppendThreads) {
            const int sl = i / pairs, d = (i - sl * pairs) * 2, h0 = sl * kHeadSlice, nh = min(kHeadSlice, p.H - h0);
            float w[kHeadSlice][RM];                     // talk is padded to RM columns with zeros
#pragma unroll
            for (int e = 0; e < kHeadSlice; ++e)
#pragma unroll
                for (int r = 0; r < RM; ++r) w[e][r] = e < nh ? tk[(h0 + e) * RM + r] : 0.f;
            QT* dst = out + static_cast<long long>(h0) * p.qld + d;
            for (int u = 0; u < nt; ++u, dst += token_ld) {
                float2 qr[RM];
#pragma unroll
                for (int r = 0; r < RM; ++r) qr[r] = r < p.R ? *reinterpret_cast<const float2*>(qs + u * q_ld + r * p.dim + d) : make_float2(0.f, 0.f);
#pragma unroll
                for (int e = 0; e < kHeadSlice; ++e) {
                    if (e >= nh) break;
                    float2 a = make_float2(0.f, 0.f);
#pragma unroll
                    for (int r = 0; r < RM; ++r) a = __ffma2_rn(make_float2(w[e][r], w[e][r]), qr[r], a);
                    if constexpr (sizeof(QT) == 2) *reinterpret_cast<uint32_t*>(dst + e * p.qld) = Elem<__nv_bfloat16>::pack2(a.x, a.y);
                    else *reinterpret_cast<float2*>(dst + e * p.qld) = a;
                }
            }
        }
    } else {
        for (int i = tid; i < p.dim * p.H; i += kAppendThreads) {
            const int h = i / p.dim, d = i - h * p.dim;
            for (int u = 0; u < nt; ++u) {
                float a = 0.f;
                for (int r = 0; r < p.R; ++r) a = fmaf(tk[h * p.R + r], qs[u * q_ld + r * p.dim + d], a);
                out[u * token_ld + static_cast<long long>(h) * p.qld + d] = Elem<QT>::from_f(a);
            }
        }
    }
    const int pad = p.qld - p.G * p.dim;                 // columns past the last group
    if (g == p.G - 1)
        for (int i = tid; i < nt * pad * p.H; i += kAppendThreads) out[static_cast<long long>(i / pad) * p.qld + p.dim + i % pad] = Elem<QT>::from_f(0.f);
}

__device__ __forceinline__ float sigmoid_exact(float x) { return 1.0f / (1.0f + expf(-x)); }

// grid (key splits, H * ceil(T / 4), B), a warp per query over one split of the keys: a lane per key for the scores, a lane per value
// column for the sum.  Prompts run with one split and write the gated output; decode steps write partial sums.
template <typename T>
__global__ void __launch_bounds__(128)
sig_attend_generic_kernel(SigParams p, const T* __restrict__ proj, const T* __restrict__ kc, const T* __restrict__ vc, const float* __restrict__ qm, float* __restrict__ part,
                          T* __restrict__ out) {
    pdl_begin();
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kcols = p.G * p.dim;
    const int n_t = (p.T + 3) / 4, h = blockIdx.y / n_t, t = (blockIdx.y - h * n_t) * 4 + warp, b = blockIdx.z, split = blockIdx.x;
    if (t >= p.T) return;
    float* q = sm + warp * (kcols + p.vdim);
    float* acc = q + kcols;
    const long long m = static_cast<long long>(b) * p.T + t;
    const float* qr = qm + (m * p.H + h) * p.qld;
    for (int i = lane; i < kcols; i += 32) q[i] = qr[i];
    for (int i = lane; i < p.vdim; i += 32) acc[i] = 0.f;
    __syncwarp();
    const int me = min(p.pos[b] + t, p.cap - 1), n = me + 1, chunk = (n + p.splits - 1) / p.splits, lo = split * chunk, hi = min(n, lo + chunk);
    const long long base = static_cast<long long>(p.slots ? p.slots[b] : b) * p.cap;
    const float* bias = p.bias + static_cast<long long>(h) * p.n_bias;
    const int vcol = (h / p.R) * p.vdim;
    for (int j0 = lo; j0 < hi; j0 += 32) {
        const int j = j0 + lane;
        float w = 0.f;
        if (j < hi) {
            const T* kr = kc + (base + j) * p.ldk;
            float d = 0.f;
            for (int i0 = 0; i0 < kcols; i0 += 16) {                     // sums of 16 products at a time: shorter chains of roundings
                float e = 0.f;
                for (int i = i0; i < min(kcols, i0 + 16); ++i) e = fmaf(q[i], Elem<T>::to_f(kr[i]), e);
                d += e;
            }
            w = sigmoid_exact(d + bias[min(me - j, p.n_bias - 1)]);
        }
        const int nt = min(32, hi - j0);
        for (int i0 = 0; i0 < p.vdim; i0 += 32) {
            const int i = i0 + lane;
            float e = 0.f;
            for (int k = 0; k < nt; ++k) {
                const float wk = __shfl_sync(0xFFFFFFFFu, w, k);
                if (i < p.vdim) e = fmaf(wk, Elem<T>::to_f(vc[(base + j0 + k) * p.ldv + vcol + i]), e);
            }
            if (i < p.vdim) acc[i] += e;
        }
    }
    if (part != nullptr) {
        float* o = part + ((m * p.H + h) * p.splits + split) * p.vdim;
        for (int i = lane; i < p.vdim; i += 32) o[i] = acc[i];
        return;
    }
    const float gate = sigmoid_exact(Elem<T>::to_f(proj[m * p.ldp + p.H * p.dim + kcols + p.G * p.vdim + h]));
    T* o = out + m * p.ldo + h * p.vdim;
    for (int i = lane; i < p.vdim; i += 32) o[i] = Elem<T>::from_f(acc[i] * gate);
}

// grid (H, B), 128 threads: the splits of a decode step added in order, times the gate.
template <typename T>
__global__ void __launch_bounds__(128)
sig_combine_kernel(SigParams p, const T* __restrict__ proj, const float* __restrict__ part, T* __restrict__ out) {
    pdl_begin();
    const int h = blockIdx.x, b = blockIdx.y;
    const float gate = sigmoid_exact(Elem<T>::to_f(proj[b * p.ldp + p.H * p.dim + p.G * (p.dim + p.vdim) + h]));
    const float* src = part + (static_cast<long long>(b) * p.H + h) * p.splits * p.vdim;
    for (int i = threadIdx.x; i < p.vdim; i += 128) {
        float a = 0.f;
        for (int s0 = 0; s0 < p.splits; s0 += 8) {
            float r[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) r[u] = src[static_cast<long long>(min(s0 + u, p.splits - 1)) * p.vdim + i];
#pragma unroll
            for (int u = 0; u < 8; ++u) a += s0 + u < p.splits ? r[u] : 0.f;
        }
        out[b * p.ldo + h * p.vdim + i] = Elem<T>::from_f(a * gate);
    }
}

}  // namespace

SigPlan plan_sigattn(const vb200_sigattn_args& a) {
    SigPlan pl{};
    pl.qld = pad_to(a.G * a.dim, 16);
    pl.mma = a.form != 1 && (a.T > 1 ? sig_prefill_sm100_supported(a) : sig_decode_mma_supported(a));
    pl.splits = 1;
    if (a.T == 1) {
        const int n_max = a.max_len > 0 && a.max_len < a.cap ? a.max_len : a.cap;
        const long long units = static_cast<long long>(a.B) * (pl.mma ? (a.H + 15) / 16 : a.H);
        long long want = (pl.mma ? sig_decode_ctas_per_sm(a) : 4LL) * device_sm_count() / units;         // rounded down: a few CTAs more would be a second wave
        const long long most = (n_max + 63) / 64;
        if (want > most) want = most;
        if (want > 128) want = 128;
        pl.splits = want < 1 ? 1 : static_cast<int>(want);
    }
    auto up = [](size_t x) { return (x + 255) / 256 * 256; };
    pl.q_bytes = up(static_cast<size_t>(a.B) * a.T * a.H * pl.qld * (pl.mma ? 2 : 4));
    pl.part_bytes = a.T == 1 ? up(static_cast<size_t>(a.B) * a.H * pl.splits * a.vdim * 4) : 0;
    pl.total = pl.q_bytes + pl.part_bytes;
    return pl;
}

int launch_sigattn(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, int* status) {
    SigParams p{};
    p.B = a.B; p.T = a.T; p.H = a.H; p.G = a.G; p.dim = a.dim; p.vdim = a.vdim; p.R = a.H / a.G;
    p.scale = a.scale; p.eps = a.eps; p.temp_coef = a.temp_coef; p.temp_every = a.temp_every; p.n_bias = a.n_bias; p.cap = a.cap; p.qld = pl.qld; p.splits = pl.splits;
    p.ldp = a.ldp; p.ldk = a.ldk; p.ldv = a.ldv; p.ldo = a.ldo; p.value_role = a.value_role; p.lambda = a.lambda;
    p.talk = a.talk; p.bias = a.bias; p.slots = a.slots; p.pos = a.pos; p.status = status;
    void* q = a.workspace;
    float* part = reinterpret_cast<float*>(static_cast<uint8_t*>(a.workspace) + pl.q_bytes);
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        T *kc = static_cast<T*>(a.k_cache), *vc = static_cast<T*>(a.v_cache), *first = static_cast<T*>(a.first_values), *out = static_cast<T*>(a.out);
        const T* proj = static_cast<const T*>(a.proj);
        const size_t q_floats = (static_cast<size_t>(p.R) * a.dim + 3) / 4 * 4;
        const int tokens = a.T >= 16 && q_floats <= 1024 ? 4 : 1;
        const dim3 grid(static_cast<unsigned>((a.T + tokens - 1) / tokens), static_cast<unsigned>(a.B), static_cast<unsigned>(a.G));
        const int rm = a.dim % 2 != 0 || p.R > 8 ? 0 : p.R <= 1 ? 1 : p.R <= 2 ? 2 : p.R <= 4 ? 4 : 8;
        const size_t smem = sizeof(float) * (tokens * q_floats + static_cast<size_t>(a.H) * (rm > 0 ? rm : p.R));
        auto append = [&](auto* qm) -> int {
            using QT = std::remove_pointer_t<decltype(qm)>;
            auto kernel = rm == 0 ? sig_append_kernel<T, QT, 0> : rm == 1 ? sig_append_kernel<T, QT, 1> : rm == 2 ? sig_append_kernel<T, QT, 2> : rm == 4 ? sig_append_kernel<T, QT, 4>
                                                                                                                                  : sig_append_kernel<T, QT, 8>;
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_pdl(kernel, grid, dim3(kAppendThreads), smem, s, p, tokens, proj, kc, vc, first, qm);
        };
        if (int rc = pl.mma ? append(static_cast<__nv_bfloat16*>(q)) : append(static_cast<float*>(q))) return rc;
        int rc;
        profile_mark_begin(s);
        if (pl.mma) {
            rc = a.T > 1 ? launch_sig_prefill_sm100(s, a, pl, q, status) : launch_sig_decode_mma(s, a, pl, q, part, status);
            if (a.T == 1) note_sigattn_kernel("sig_decode_mma_kernel");
        } else {
            const size_t sm = sizeof(float) * 4 * (a.G * a.dim + a.vdim);
            rc = allow_smem(sig_attend_generic_kernel<T>, sm);
            if (rc == VB200_OK)
                rc = launch_pdl(sig_attend_generic_kernel<T>, dim3(static_cast<unsigned>(pl.splits), static_cast<unsigned>(a.H * ((a.T + 3) / 4)), static_cast<unsigned>(a.B)),
                                dim3(128), sm, s, p, proj, kc, vc, static_cast<const float*>(q), a.T == 1 ? part : nullptr, out);
            note_sigattn_kernel("sig_attend_generic_kernel");
        }
        profile_mark_end(s);
        if (rc || a.T > 1) return rc;
        return launch_pdl(sig_combine_kernel<T>, dim3(static_cast<unsigned>(a.H), static_cast<unsigned>(a.B)), dim3(128), 0, s, p, proj, part, out);
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace vb200
