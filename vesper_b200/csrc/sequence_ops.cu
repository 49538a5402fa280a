// Row operators of hybrid decoders: the embedding of a step (token row + bigram row, sequence bookkeeping), the
// re-entry into a looped range of layers, and the fp32 RMSNorm.
#include "hybrid.cuh"

namespace vb200 {
namespace {

// One CTA per token row.  Only the row of a sequence's first new token touches the sequence's state (length,
// previous id), so the same CTA can advance it: every other row takes its previous id from the call's own ids.
template <typename T>
__global__ void __launch_bounds__(256)
embed_sequence_kernel(const int* __restrict__ ids, int tokens, int dim, int vocab, const T* __restrict__ table, const T* __restrict__ bigram,
                      long long buckets, long long mul_prev, long long mul_cur, const int* __restrict__ slots, int* lens, int* step_pos, int* prev,
                      float* __restrict__ h, float* __restrict__ embed_copy, const float* __restrict__ add, const float* __restrict__ scale,
                      __nv_bfloat16* __restrict__ scaled_out, int* status) {
    pdl_begin();
    const int m = blockIdx.x, b = m / tokens, t = m - b * tokens;
    const long long id = ids[m];
    __shared__ long long s_row;
    if (threadIdx.x == 0) {
        long long row = -1;
        if (bigram != nullptr) {
            const int slot = slots ? slots[b] : b;
            if (t > 0) row = (ids[m - 1] * mul_prev + id * mul_cur) % buckets;
            else row = lens[b] == 0 ? buckets : (prev[slot] * mul_prev + id * mul_cur) % buckets;
            if (row < 0) row += buckets;
        }
        if (t == 0) {
            const int p = lens[b];
            step_pos[b] = p;
            lens[b] = p + tokens;
            prev[slots ? slots[b] : b] = ids[m + tokens - 1];
        }
        if (id < 0 || id >= vocab) atomicCAS(status, 0, (2 << 24) | 0x62);
        s_row = row;
    }
    __syncthreads();
    const bool bad = id < 0 || id >= vocab;
    const T* src = table + (bad ? 0 : id) * dim;
    const T* src2 = bigram != nullptr ? bigram + s_row * dim : nullptr;
    const long long base = static_cast<long long>(m) * dim;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float v = bad ? 0.f : Elem<T>::to_f(src[i]);
        if (src2 != nullptr) v += Elem<T>::to_f(src2[i]);
        if (embed_copy != nullptr) embed_copy[base + i] = v;
        if (add != nullptr) v += add[i];
        h[base + i] = v;
        if (scaled_out != nullptr) scaled_out[base + i] = __float2bfloat16_rn(scale != nullptr ? v * scale[i] : v);
    }
}

__global__ void __launch_bounds__(256)
residual_add_kernel(float* __restrict__ h, const float* __restrict__ addend, const float* __restrict__ vec, long long total, int dim,
                    const float* __restrict__ scale, __nv_bfloat16* __restrict__ scaled_out) {
    pdl_begin();
    for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < total; i += static_cast<long long>(gridDim.x) * blockDim.x) {
        const int c = static_cast<int>(i % dim);
        float v = h[i];
        if (addend != nullptr) v += addend[i];
        if (vec != nullptr) v += vec[c];
        h[i] = v;
        if (scaled_out != nullptr) scaled_out[i] = __float2bfloat16_rn(v * scale[c]);
    }
}

__global__ void __launch_bounds__(256)
rms_norm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ out, int dim, int count, float eps) {
    pdl_begin();
    const float* xr = x + static_cast<long long>(blockIdx.x) * dim;
    float ss = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) ss += xr[i] * xr[i];
    __shared__ float part[8];
    const float inv = 1.0f / sqrtf(block_sum<8>(ss, part) / static_cast<float>(count) + eps);
    float* o = out + static_cast<long long>(blockIdx.x) * dim;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) o[i] = xr[i] * inv * w[i];
}

// One CTA per row.  The row to be normed stays in registers between the two passes (up to 256 * 4 * kNormVec columns; wider rows are
// gathered twice).
constexpr int kNormVec = 8;

__global__ void __launch_bounds__(256)
norm_add_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, int dim, int count, float eps, const __nv_bfloat16* __restrict__ rows,
                const int* __restrict__ gather, int n_gather, const float* __restrict__ scale, __nv_bfloat16* __restrict__ copy_out) {
    pdl_begin();
    const long long m = blockIdx.x, base = m * dim;
    const int nv = dim / 4;
    __shared__ float part[8];
    auto load = [&](int c) {
        float4 v = y != nullptr ? *reinterpret_cast<const float4*>(y + base + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < n_gather; ++k) {
            const uint2 u = *reinterpret_cast<const uint2*>(rows + static_cast<long long>(gather[m * n_gather + k]) * dim + c * 4);
            const float2 a = Elem<__nv_bfloat16>::unpack2(u.x), b = Elem<__nv_bfloat16>::unpack2(u.y);
            v.x += a.x; v.y += a.y; v.z += b.x; v.w += b.y;
        }
        return v;
    };
    float4 v[kNormVec];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kNormVec; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < nv) { v[i] = load(c); ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w; }
    }
    for (int c = threadIdx.x + kNormVec * 256; c < nv; c += 256) { const float4 t = load(c); ss += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w; }
    const float inv = 1.0f / sqrtf(block_sum<8>(ss, part) / static_cast<float>(count) + eps);
    auto finish = [&](int c, const float4& t) {
        const float4 g = *reinterpret_cast<const float4*>(w + c * 4);
        float4 h = *reinterpret_cast<const float4*>(x + base + c * 4);
        h.x += t.x * inv * g.x; h.y += t.y * inv * g.y; h.z += t.z * inv * g.z; h.w += t.w * inv * g.w;
        *reinterpret_cast<float4*>(x + base + c * 4) = h;
        if (copy_out != nullptr) {
            if (scale != nullptr) {
                const float4 s4 = *reinterpret_cast<const float4*>(scale + c * 4);
                h.x *= s4.x; h.y *= s4.y; h.z *= s4.z; h.w *= s4.w;
            }
            uint2 u;
            u.x = Elem<__nv_bfloat16>::pack2(h.x, h.y); u.y = Elem<__nv_bfloat16>::pack2(h.z, h.w);
            *reinterpret_cast<uint2*>(copy_out + base + c * 4) = u;
        }
    };
#pragma unroll
    for (int i = 0; i < kNormVec; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < nv) finish(c, v[i]);
    }
    for (int c = threadIdx.x + kNormVec * 256; c < nv; c += 256) finish(c, load(c));
}

}  // namespace

int launch_norm_add(cudaStream_t s, const vb200_norm_add_args& a) {
    return launch_pdl(norm_add_kernel, dim3(static_cast<unsigned>(a.M)), dim3(256), 0, s, a.x, a.y, a.w, a.dim, a.count, a.eps, static_cast<const __nv_bfloat16*>(a.rows),
                      a.gather, a.gather != nullptr ? a.n_gather : 0, a.scale, static_cast<__nv_bfloat16*>(a.copy_out));
}

int launch_embed_sequence(cudaStream_t s, const vb200_embed_args& a, int* status) {
    const dim3 grid(static_cast<unsigned>(a.B * a.T));
    auto go = [&](auto tag) {
        using T = decltype(tag);
        return launch_pdl(embed_sequence_kernel<T>, grid, dim3(256), 0, s, a.ids, a.T, a.dim, a.vocab, static_cast<const T*>(a.table), static_cast<const T*>(a.bigram),
                          static_cast<long long>(a.buckets), static_cast<long long>(a.mul_prev), static_cast<long long>(a.mul_cur), a.slots, a.lens, a.step_pos,
                          a.prev, a.h, a.embed_copy, a.add, a.scale, static_cast<__nv_bfloat16*>(a.scaled_out), status);
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int launch_residual_add(cudaStream_t s, float* h, const float* addend, const float* vec, int M, int dim, const float* scale, void* scaled_out) {
    const long long total = static_cast<long long>(M) * dim;
    long long blocks = (total + 1023) / 1024;
    if (blocks > 148 * 8) blocks = 148 * 8;
    return launch_pdl(residual_add_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, s, h, addend, vec, total, dim, scale,
                      static_cast<__nv_bfloat16*>(scaled_out));
}

int launch_rms_norm_f32(cudaStream_t s, const float* x, const float* w, float* out, int M, int dim, int count, float eps) {
    return launch_pdl(rms_norm_f32_kernel, dim3(static_cast<unsigned>(M)), dim3(256), 0, s, x, w, out, dim, count, eps);
}

}  // namespace vb200
