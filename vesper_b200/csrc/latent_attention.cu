// Latent attention: the pieces around the two tuned kernels, and forms of both for any sizes and for fp32.
//
//   latent_append_kernel   prompt pass: RMSNorm of the new latents, rotation of their key part and of q, the ring
//                          update, and the contiguous context rows the keys / values are expanded from
//   latent_query_kernel    decode: q' = W_uk_h^T q (so that attention runs on the latents themselves), its rotated
//                          part, and the new latent row, in one launch
//   latent_split_generic   decode attention over a slice of the ring on CUDA cores, any sizes, fp32 or bf16
//   latent_value_kernel    decode: merges the slices, adds the sink to the denominator, applies W_uv_h
//   latent_prefill_generic prompt attention on CUDA cores, any sizes, fp32 or bf16
//
// The ring holds exactly the positions a decode step may see (row p mod ring), so the step attends to its first
// min(p + 1, ring) rows in any order and needs no mask.  Scores are kept in log2 units (scale * log2 e folded into q').
#include "hybrid.cuh"

namespace vb200 {
namespace {

struct LatentParams {
    int B, T, H, dim, rot, vdim, rank, window, ring;
    float scale, eps;
    const double* inv_freq;
    long long ldp, ldu, ldc, ldo, ldkv;
    const float *c_norm, *sink;
    const int *slots, *pos;
    int start_pos, n_ctx;
    int splits, rank16, rot16, qld, part_ld;
    int n_rc;                    // 128-column blocks of a latent
    int rot_off;
    int src_aligned;             // latents start at 16-byte boundaries of a projection row
};

// One latent row: c = rmsnorm(src[0..rank)) * w, key part rotated.  ring_row receives it (nullable), after the row it
// replaces has been copied to old_copy (nullable); ctx_row receives it too (nullable).
template <typename T, int W>
__device__ void latent_row(const LatentParams& p, const T* __restrict__ src, const float2* cs, T* ring_row, T* old_copy, T* ctx_row, float* part) {
    float ss = 0.f;
    if (p.rank % 8 == 0 && p.rank <= W * 256 && p.src_aligned) {          // eight columns per thread, one pass
        const int i = threadIdx.x * 8;
        const bool on = i < p.rank;
        float v[8] = {}, w[8] = {};
        if (on) {
            load8(src + i, v);
#pragma unroll
            for (int e = 0; e < 8; ++e) { w[e] = p.c_norm[i + e]; ss += v[e] * v[e]; }
        }
        const float inv = 1.0f / sqrtf(block_sum<W>(ss, part) / static_cast<float>(p.rank) + p.eps);
        if (on) {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = v[e] * inv * w[e];
            if (old_copy != nullptr) { float o[8]; load8(ring_row + i, o); store8(old_copy + i, o); }
            if (ring_row != nullptr) store8(ring_row + i, v);
            if (ctx_row != nullptr) store8(ctx_row + i, v);
        }
    } else {
    for (int i = threadIdx.x; i < p.rank; i += W * 32) { const float v = Elem<T>::to_f(src[i]); ss += v * v; }
    const float inv = 1.0f / sqrtf(block_sum<W>(ss, part) / static_cast<float>(p.rank) + p.eps);
    for (int i = threadIdx.x; i < p.rank; i += W * 32) {
        const T v = Elem<T>::from_f(Elem<T>::to_f(src[i]) * inv * p.c_norm[i]);
        if (old_copy != nullptr) old_copy[i] = ring_row[i];
        if (ring_row != nullptr) ring_row[i] = v;
        if (ctx_row != nullptr) ctx_row[i] = v;
    }
    }
    for (int i = p.rank + threadIdx.x; i < p.rot_off; i += W * 32) {      // context rows feed a product over the padded width
        if (old_copy != nullptr) old_copy[i] = Elem<T>::from_f(0.f);
        if (ctx_row != nullptr) ctx_row[i] = Elem<T>::from_f(0.f);
    }
    const int half = p.rot / 2;
    for (int i = threadIdx.x; i < half; i += W * 32) {
        const float u = Elem<T>::to_f(src[p.rank + i]), v = Elem<T>::to_f(src[p.rank + half + i]);
        const T a = Elem<T>::from_f(u * cs[i].x - v * cs[i].y), b = Elem<T>::from_f(v * cs[i].x + u * cs[i].y);
        const int ia = p.rot_off + i, ib = ia + half;
        if (old_copy != nullptr) { old_copy[ia] = ring_row[ia]; old_copy[ib] = ring_row[ib]; }
        if (ring_row != nullptr) { ring_row[ia] = a; ring_row[ib] = b; }
        if (ctx_row != nullptr) { ctx_row[ia] = a; ctx_row[ib] = b; }
    }
}

// grid (T + earlier context rows, B).  A ring row is written by one CTA, the one of the newest token that maps to it;
// that CTA first saves the row's old content to the context.  Old rows nobody overwrites are copied by CTAs of their own.
template <typename T>
__global__ void __launch_bounds__(128)
latent_append_kernel(LatentParams p, T* __restrict__ proj, T* __restrict__ cache, T* __restrict__ ctx) {
    pdl_begin();
    extern __shared__ float2 cs[];
    __shared__ float part[4];
    const int b = blockIdx.y, start = p.pos[b], last = start + p.T - 1;
    const int n_old = p.n_ctx - p.T, ctx0 = start - n_old;       // position of context row 0
    const int slot = p.slots ? p.slots[b] : b;
    T* ring = cache + static_cast<long long>(slot) * p.ring * p.ldc;
    T* crow = ctx + static_cast<long long>(b) * p.n_ctx * p.ldc;
    if (static_cast<int>(blockIdx.x) >= p.T) {
        const int i = blockIdx.x - p.T, q = ctx0 + i;            // an earlier position
        if (q < 0 || q + p.ring <= last) return;                  // its row is overwritten in this pass: saved there
        const T* src = ring + static_cast<long long>(q % p.ring) * p.ldc;
        for (int j = threadIdx.x; j < p.ldc; j += blockDim.x) crow[static_cast<long long>(i) * p.ldc + j] = src[j];
        return;
    }
    const int t = blockIdx.x, pos = start + t, half = p.rot / 2;
    for (int i = threadIdx.x; i < half; i += blockDim.x) cs[i] = rope_cs(pos, p.inv_freq[i]);
    __syncthreads();
    T* row = proj + (static_cast<long long>(b) * p.T + t) * p.ldp;
    T* ring_row = nullptr;
    T* old_copy = nullptr;
    if (pos + p.ring > last) {                                    // the newest token of its ring row
        const int r = pos % p.ring;
        ring_row = ring + static_cast<long long>(r) * p.ldc;
        if (start > 0) {
            const int q = start - 1 - ((start - 1 - r) % p.ring + p.ring) % p.ring;      // the newest earlier position there
            if (q >= ctx0 && q >= 0) old_copy = crow + static_cast<long long>(q - ctx0) * p.ldc;
        }
    }
    const int hq = p.dim + p.rot;
    if (half % 8 == 0 && p.dim % 8 == 0 && p.ldp % 8 == 0) {        // eight pairs per thread
        const int groups = half / 8;
        for (int i = threadIdx.x; i < p.H * groups; i += blockDim.x) {
            const int h = i / groups, j = (i - h * groups) * 8;
            T* q = row + static_cast<long long>(h) * hq + p.dim + j;
            float u[8], v[8], a[8], c[8];
            load8(q, u);
            load8(q + half, v);
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float2 w = cs[j + e];
                a[e] = u[e] * w.x - v[e] * w.y;
                c[e] = v[e] * w.x + u[e] * w.y;
            }
            store8(q, a);
            store8(q + half, c);
        }
    } else {
        for (int i = threadIdx.x; i < p.H * half; i += blockDim.x) {
            const int h = i / half, j = i - h * half;
            T* q = row + static_cast<long long>(h) * hq + p.dim;
            const float u = Elem<T>::to_f(q[j]), v = Elem<T>::to_f(q[j + half]);
            q[j] = Elem<T>::from_f(u * cs[j].x - v * cs[j].y);
            q[j + half] = Elem<T>::from_f(v * cs[j].x + u * cs[j].y);
        }
    }
    latent_row<T, 4>(p, row + static_cast<long long>(p.H) * hq, cs, ring_row, old_copy, crow + static_cast<long long>(n_old + t) * p.ldc, part);
}

constexpr int kBT = 4;           // batch rows per CTA of the two per-head products (their weights are read once per CTA)

// grid (H * n_rc + kBT, ceil(B / kBT)), 256 threads: thread = 8 latent columns x one sixteenth of the head dimension.
template <typename T>
__global__ void __launch_bounds__(256)
latent_query_kernel(LatentParams p, const T* __restrict__ proj, const T* __restrict__ w_uk, T* __restrict__ cache, float* __restrict__ qa) {
    extern __shared__ float sm[];
    __shared__ float part[8];
    // weights do not depend on the previous kernel: the first eight rows of this thread stream while it finishes
    constexpr int kAhead = 8;
    Raw8<T> ahead[kAhead];
    const int cg = threadIdx.x & 15, dg = threadIdx.x >> 4, c0 = (blockIdx.x % p.n_rc) * 128 + cg * 8;
    const bool mine = static_cast<int>(blockIdx.x) < p.H * p.n_rc && c0 < (p.rank + 7) / 8 * 8;
    const T* wrow = w_uk + static_cast<long long>(blockIdx.x / p.n_rc) * p.dim * p.ldu + c0;
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (mine && dg + 16 * i < p.dim) ahead[i].load(wrow + static_cast<long long>(dg + 16 * i) * p.ldu);
    pdl_begin();
    const int b0 = blockIdx.y * kBT, hq = p.dim + p.rot, half = p.rot / 2;
    if (static_cast<int>(blockIdx.x) >= p.H * p.n_rc) {           // the new latent row of one sequence
        const int b = b0 + blockIdx.x - p.H * p.n_rc;
        if (b >= p.B) return;
        float2* cs = reinterpret_cast<float2*>(sm);
        const int pos = p.pos[b], slot = p.slots ? p.slots[b] : b;
        for (int i = threadIdx.x; i < half; i += blockDim.x) cs[i] = rope_cs(pos, p.inv_freq[i]);
        __syncthreads();
        T* ring_row = cache + (static_cast<long long>(slot) * p.ring + pos % p.ring) * p.ldc;
        latent_row<T, 8>(p, proj + static_cast<long long>(b) * p.ldp + static_cast<long long>(p.H) * hq, cs, ring_row, nullptr, nullptr, part);
        return;
    }
    const int h = blockIdx.x / p.n_rc, rc = blockIdx.x % p.n_rc;
    float* qs = sm;                                  // [kBT][dim]
    float* red = sm + kBT * p.dim;                   // [8 warps][kBT][128]
    const int nb = min(kBT, p.B - b0);
    for (int i = threadIdx.x; i < kBT * p.dim; i += 256) {
        const int b = i / p.dim, d = i - b * p.dim;
        qs[i] = b < nb ? Elem<T>::to_f(proj[static_cast<long long>(b0 + b) * p.ldp + static_cast<long long>(h) * hq + d]) : 0.f;
    }
    __syncthreads();
    float acc[kBT][8] = {};
    if (mine) {
        auto add = [&](int d, const float (&wv)[8]) {
#pragma unroll
            for (int b = 0; b < kBT; ++b) {
                const float q = qs[b * p.dim + d];
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[b][j] = fmaf(q, wv[j], acc[b][j]);
            }
        };
        float wv[8];
#pragma unroll
        for (int i = 0; i < kAhead; ++i)
            if (dg + 16 * i < p.dim) { ahead[i].get(wv); add(dg + 16 * i, wv); }
        for (int d = dg + 16 * kAhead; d < p.dim; d += 16) { load8(wrow + static_cast<long long>(d) * p.ldu, wv); add(d, wv); }
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
    for (int b = 0; b < kBT; ++b)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const float v = acc[b][j] + __shfl_xor_sync(0xFFFFFFFFu, acc[b][j], 16);
            if (lane < 16) red[(warp * kBT + b) * 128 + cg * 8 + j] = v;
        }
    __syncthreads();
    const float sc = p.scale * kLog2e;
    for (int i = threadIdx.x; i < nb * 128; i += 256) {
        const int b = i >> 7, c = i & 127, col = rc * 128 + c;
        if (col >= p.rank16) continue;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += red[(w * kBT + b) * 128 + c];
        qa[(static_cast<long long>(b0 + b) * p.H + h) * p.qld + col] = col < p.rank ? v * sc : 0.f;
    }
    if (rc == 0) {
        for (int i = threadIdx.x; i < nb * p.rot16; i += 256) {
            const int b = i / p.rot16, j = i - b * p.rot16;
            float v = 0.f;
            if (j < p.rot) {
                const int k = j < half ? j : j - half;
                const T* q = proj + static_cast<long long>(b0 + b) * p.ldp + static_cast<long long>(h) * hq + p.dim;
                const float2 cs = rope_cs(p.pos[b0 + b], p.inv_freq[k]);
                const float a = Elem<T>::to_f(q[k]), c = Elem<T>::to_f(q[k + half]);
                v = (j < half ? a * cs.x - c * cs.y : c * cs.x + a * cs.y) * sc;
            }
            qa[(static_cast<long long>(b0 + b) * p.H + h) * p.qld + p.rank16 + j] = v;
        }
    }
}

// grid (splits, H, B), 128 threads: a warp per key for the scores, a thread per latent column for the sum.
template <typename T>
__global__ void __launch_bounds__(128)
latent_split_generic_kernel(LatentParams p, const float* __restrict__ qa, const T* __restrict__ cache, float* __restrict__ part) {
    pdl_begin();
    extern __shared__ float sm[];
    float* q = sm;                       // [qld]
    float* acc = q + p.qld;              // [rank]
    float* sc = acc + p.rank;            // [64]
    const int split = blockIdx.x, h = blockIdx.y, b = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n = min(p.pos[b] + 1, p.ring), chunk = (n + p.splits - 1) / p.splits;
    const int k0 = split * chunk, k1 = min(n, k0 + chunk);
    const T* ring = cache + static_cast<long long>(p.slots ? p.slots[b] : b) * p.ring * p.ldc;
    const float* qrow = qa + (static_cast<long long>(b) * p.H + h) * p.qld;
    for (int i = threadIdx.x; i < p.qld; i += 128) q[i] = qrow[i];
    for (int i = threadIdx.x; i < p.rank; i += 128) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int t0 = k0; t0 < k1; t0 += 64) {
        const int nt = min(64, k1 - t0);
        __syncthreads();
        for (int k = warp; k < nt; k += 4) {
            const T* row = ring + static_cast<long long>(t0 + k) * p.ldc;
            float d = 0.f;
            for (int i = lane; i < p.rank; i += 32) d = fmaf(q[i], Elem<T>::to_f(row[i]), d);
            for (int i = lane; i < p.rot; i += 32) d = fmaf(q[p.rank16 + i], Elem<T>::to_f(row[p.rot_off + i]), d);
            d = warp_sum_f(d);
            if (lane == 0) sc[k] = d;
        }
        __syncthreads();
        float mt = m;
        for (int k = 0; k < nt; ++k) mt = fmaxf(mt, sc[k]);
        __syncthreads();
        if (threadIdx.x < nt) sc[threadIdx.x] = exp2f(sc[threadIdx.x] - mt);
        __syncthreads();
        const float alpha = exp2f(m - mt);
        float ls = 0.f;
        for (int k = 0; k < nt; ++k) ls += sc[k];
        l = l * alpha + ls;
        m = mt;
        for (int i = threadIdx.x; i < p.rank; i += 128) {
            float a = acc[i] * alpha;
            for (int k = 0; k < nt; ++k) a = fmaf(sc[k], Elem<T>::to_f(ring[static_cast<long long>(t0 + k) * p.ldc + i]), a);
            acc[i] = a;
        }
    }
    __syncthreads();
    float* out = part + ((static_cast<long long>(b) * p.H + h) * p.splits + split) * p.part_ld;
    for (int i = threadIdx.x; i < p.rank16; i += 128) out[i] = i < p.rank ? acc[i] : 0.f;
    if (threadIdx.x == 0) { out[p.rank16] = m; out[p.rank16 + 1] = l; }
}

constexpr int kValueRows = 32;           // rows of W_uv_h per CTA

// grid (H * ceil(vdim / 32), ceil(B / kBT)), 256 threads: a warp has four rows of W_uv_h, fetched before the wait for
// latents of up to 512 columns.
template <typename T>
__global__ void __launch_bounds__(256)
latent_value_kernel(LatentParams p, const float* __restrict__ part, const T* __restrict__ w_uv, T* __restrict__ out) {
    extern __shared__ float sm[];
    float* o = sm;                               // [kBT][rank16]
    float* coef = o + kBT * p.rank16;            // [kBT][splits]
    const int n_vc = (p.vdim + kValueRows - 1) / kValueRows;
    const int h = blockIdx.x / n_vc, v0 = (blockIdx.x % n_vc) * kValueRows, b0 = blockIdx.y * kBT;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nb = min(kBT, p.B - b0);
    const int rank8 = (p.rank + 7) / 8 * 8;
    constexpr int kRowsPerWarp = kValueRows / 8, kPieces = 2;
    Raw8<T> ahead[kRowsPerWarp][kPieces];
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; ++r)
#pragma unroll
        for (int k = 0; k < kPieces; ++k) {
            const int v = v0 + warp + 8 * r, c = lane * 8 + 256 * k;
            if (v < p.vdim && c < rank8) ahead[r][k].load(w_uv + (static_cast<long long>(h) * p.vdim + v) * p.ldu + c);
        }
    pdl_begin();
    if (warp < nb) {
        const float* rec = part + (static_cast<long long>(b0 + warp) * p.H + h) * p.splits * p.part_ld + p.rank16;
        const float sink = p.sink ? p.sink[h] * kLog2e : -INFINITY;
        float m = sink;
        for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, rec[static_cast<long long>(s) * p.part_ld]);
        m = warp_max_f(m);
        float l = 0.f;
        for (int s = lane; s < p.splits; s += 32) {
            const float2 ml = *reinterpret_cast<const float2*>(rec + static_cast<long long>(s) * p.part_ld);
            const float c = exp2f(ml.x - m);
            coef[warp * p.splits + s] = c;
            l += c * ml.y;
        }
        l = warp_sum_f(l) + (p.sink ? exp2f(sink - m) : 0.f);
        const float inv = 1.0f / l;
        for (int s = lane; s < p.splits; s += 32) coef[warp * p.splits + s] *= inv;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < kBT * p.rank16 / 4; i += 256) {        // four columns of one sequence, many slices' loads in flight
        const int b = i / (p.rank16 / 4), c = (i - b * (p.rank16 / 4)) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (b < nb) {
            const float* rec = part + (static_cast<long long>(b0 + b) * p.H + h) * p.splits * p.part_ld + c;
            constexpr int kBatch = 8;
            for (int s0 = 0; s0 < p.splits; s0 += kBatch) {
                float4 r[kBatch];
#pragma unroll
                for (int u = 0; u < kBatch; ++u) r[u] = *reinterpret_cast<const float4*>(rec + static_cast<long long>(min(s0 + u, p.splits - 1)) * p.part_ld);
#pragma unroll
                for (int u = 0; u < kBatch; ++u) {
                    const float w = s0 + u < p.splits ? coef[b * p.splits + s0 + u] : 0.f;
                    v.x = fmaf(w, r[u].x, v.x); v.y = fmaf(w, r[u].y, v.y); v.z = fmaf(w, r[u].z, v.z); v.w = fmaf(w, r[u].w, v.w);
                }
            }
        }
        *reinterpret_cast<float4*>(o + b * p.rank16 + c) = v;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; ++r) {
        const int v = v0 + warp + 8 * r;
        if (v >= p.vdim) break;
        float acc[kBT] = {};
        auto add = [&](int c, const float (&wv)[8]) {
#pragma unroll
            for (int b = 0; b < kBT; ++b) {
                const float4 x = *reinterpret_cast<const float4*>(o + b * p.rank16 + c), y = *reinterpret_cast<const float4*>(o + b * p.rank16 + c + 4);
                acc[b] = fmaf(wv[0], x.x, fmaf(wv[1], x.y, fmaf(wv[2], x.z, fmaf(wv[3], x.w, acc[b]))));
                acc[b] = fmaf(wv[4], y.x, fmaf(wv[5], y.y, fmaf(wv[6], y.z, fmaf(wv[7], y.w, acc[b]))));
            }
        };
        float wv[8];
#pragma unroll
        for (int k = 0; k < kPieces; ++k) {
            const int c = lane * 8 + 256 * k;
            if (c < rank8) { ahead[r][k].get(wv); add(c, wv); }
        }
        for (int c = lane * 8 + 256 * kPieces; c < rank8; c += 256) { load8(w_uv + (static_cast<long long>(h) * p.vdim + v) * p.ldu + c, wv); add(c, wv); }
#pragma unroll
        for (int b = 0; b < kBT; ++b) {
            const float x = warp_sum_f(acc[b]);
            if (lane == 0 && b < nb) out[static_cast<long long>(b0 + b) * p.ldo + static_cast<long long>(h) * p.vdim + v] = Elem<T>::from_f(x);
        }
    }
}

// grid (ceil(T / 4), H, B), a warp per query: a lane per key for the scores, a lane per value column for the sum.
template <typename T>
__global__ void __launch_bounds__(128)
latent_prefill_generic_kernel(LatentParams p, const T* __restrict__ proj, const T* __restrict__ ctx, const T* __restrict__ kv, T* __restrict__ out) {
    pdl_begin();
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hq = p.dim + p.rot;
    const int t = blockIdx.x * 4 + warp, h = blockIdx.y, b = blockIdx.z;
    float* q = sm + warp * (hq + p.vdim);
    float* acc = q + hq;
    if (t >= p.T) return;
    const T* qr = proj + (static_cast<long long>(b) * p.T + t) * p.ldp + static_cast<long long>(h) * hq;
    for (int i = lane; i < hq; i += 32) q[i] = Elem<T>::to_f(qr[i]);
    for (int i = lane; i < p.vdim; i += 32) acc[i] = 0.f;
    __syncwarp();
    const int me = p.n_ctx - p.T + t;                             // context row of this query's own token
    const int lo = max(0, me - p.window + 1);
    const T* kvb = kv + static_cast<long long>(b) * p.n_ctx * p.ldkv;
    const T* cb = ctx + static_cast<long long>(b) * p.n_ctx * p.ldc;
    const float sc = p.scale * kLog2e;
    float m = p.sink ? p.sink[h] * kLog2e : -INFINITY, l = p.sink ? 1.f : 0.f;
    for (int j0 = lo; j0 <= me; j0 += 32) {
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j <= me) {
            const T* kr = kvb + static_cast<long long>(j) * p.ldkv + static_cast<long long>(h) * p.dim;
            const T* rr = cb + static_cast<long long>(j) * p.ldc + p.rot_off;
            float d = 0.f;
            for (int i = 0; i < p.dim; ++i) d = fmaf(q[i], Elem<T>::to_f(kr[i]), d);
            for (int i = 0; i < p.rot; ++i) d = fmaf(q[p.dim + i], Elem<T>::to_f(rr[i]), d);
            s = d * sc;
        }
        const float mn = fmaxf(m, warp_max_f(s));
        const float e = exp2f(s - mn), alpha = exp2f(m - mn);
        l = l * alpha + warp_sum_f(e);
        m = mn;
        const int nt = min(32, me - j0 + 1);
        for (int i = lane; i < p.vdim; i += 32) acc[i] *= alpha;
        for (int k = 0; k < nt; ++k) {
            const float w = __shfl_sync(0xFFFFFFFFu, e, k);
            const T* vr = kvb + static_cast<long long>(j0 + k) * p.ldkv + static_cast<long long>(p.H) * p.dim + static_cast<long long>(h) * p.vdim;
            for (int i = lane; i < p.vdim; i += 32) acc[i] = fmaf(w, Elem<T>::to_f(vr[i]), acc[i]);
        }
    }
    const float inv = 1.0f / l;
    T* o = out + (static_cast<long long>(b) * p.T + t) * p.ldo + static_cast<long long>(h) * p.vdim;
    for (int i = lane; i < p.vdim; i += 32) o[i] = Elem<T>::from_f(acc[i] * inv);
}

LatentParams params_of(const vb200_latent_args& a) {
    LatentParams p{};
    p.B = a.B; p.T = a.T; p.H = a.H; p.dim = a.dim; p.rot = a.rot_dim; p.vdim = a.vdim; p.rank = a.rank;
    p.window = a.window; p.ring = a.ring; p.scale = a.scale; p.eps = a.eps; p.inv_freq = a.inv_freq;
    p.ldp = a.ldp; p.ldu = a.ldu; p.ldc = a.ldc; p.ldo = a.ldo; p.ldkv = a.ldkv;
    p.c_norm = a.c_norm; p.sink = a.sink; p.slots = a.slots; p.pos = a.pos;
    p.start_pos = a.start_pos;
    p.n_ctx = vb200_latent_context(a.start_pos, a.T, a.window);
    p.rot_off = vb200_latent_rot_offset(a.rank);
    const LatentPlan pl = plan_latent(a);
    p.splits = pl.splits; p.rank16 = pl.rank16; p.rot16 = pl.rot16; p.qld = pl.qld; p.part_ld = pl.part_ld;
    p.n_rc = (p.rank16 + 127) / 128;
    p.src_aligned = a.ldp % 8 == 0 && (static_cast<long long>(a.H) * (a.dim + a.rot_dim)) % 8 == 0;
    return p;
}

}  // namespace

LatentPlan plan_latent(const vb200_latent_args& a) {
    LatentPlan pl{};
    pl.n_max = a.max_len > 0 && a.max_len < a.ring ? a.max_len : a.ring;
    pl.rank16 = pad_to(a.rank, 16);
    pl.rot16 = pad_to(a.rot_dim, 16);
    pl.qld = pl.rank16 + pl.rot16;
    pl.part_ld = pl.rank16 + 4;
    // two CTAs per SM, at least 64 keys each
    const bool mma = latent_mma_supported(a);
    const long long units = static_cast<long long>(a.B) * (mma ? (a.H + 15) / 16 : a.H);
    long long want = 2LL * device_sm_count() / units;           // rounded down: a few CTAs more would be a second wave
    const long long most = (pl.n_max + 63) / 64;
    if (want > most) want = most;
    if (want > 128) want = 128;
    pl.splits = want < 1 ? 1 : static_cast<int>(want);
    pl.q_floats = static_cast<size_t>(a.B) * a.H * pl.qld;
    pl.part_floats = static_cast<size_t>(a.B) * a.H * pl.splits * pl.part_ld;
    return pl;
}

int launch_latent_append(cudaStream_t s, const vb200_latent_args& a) {
    const LatentParams p = params_of(a);
    const dim3 grid(static_cast<unsigned>(p.n_ctx), static_cast<unsigned>(p.B));
    const size_t smem = sizeof(float2) * (a.rot_dim / 2 + 1);
    auto go = [&](auto tag) {
        using T = decltype(tag);
        return launch_pdl(latent_append_kernel<T>, grid, dim3(128), smem, s, p, static_cast<T*>(a.proj), static_cast<T*>(a.cache), static_cast<T*>(a.ctx_latent));
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int launch_latent_prefill_generic(cudaStream_t s, const vb200_latent_args& a) {
    const LatentParams p = params_of(a);
    const dim3 grid(static_cast<unsigned>((p.T + 3) / 4), static_cast<unsigned>(p.H), static_cast<unsigned>(p.B));
    const size_t smem = sizeof(float) * 4 * (p.dim + p.rot + p.vdim);
    auto go = [&](auto tag) {
        using T = decltype(tag);
        if (int rc = allow_smem(latent_prefill_generic_kernel<T>, smem)) return rc;
        return launch_pdl(latent_prefill_generic_kernel<T>, grid, dim3(128), smem, s, p, static_cast<const T*>(a.proj), static_cast<const T*>(a.ctx_latent),
                          static_cast<const T*>(a.ctx_kv), static_cast<T*>(a.out));
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int launch_latent_decode(cudaStream_t s, const vb200_latent_args& a, int* status) {
    const LatentParams p = params_of(a);
    const LatentPlan pl = plan_latent(a);
    float* qa = static_cast<float*>(a.workspace);
    float* part = qa + (pl.q_floats + 63) / 64 * 64;
    const unsigned bg = static_cast<unsigned>((p.B + kBT - 1) / kBT);
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        const size_t q_smem = sizeof(float) * (kBT * p.dim + 8 * kBT * 128) + sizeof(float2) * p.rot;
        if (int rc = allow_smem(latent_query_kernel<T>, q_smem)) return rc;
        if (int rc = launch_pdl(latent_query_kernel<T>, dim3(static_cast<unsigned>(p.H * p.n_rc + kBT), bg), dim3(256), q_smem, s, p, static_cast<const T*>(a.proj),
                                static_cast<const T*>(a.w_uk), static_cast<T*>(a.cache), qa)) return rc;
        profile_mark_begin(s);
        if (latent_mma_supported(a)) {
            if (int rc = launch_latent_split_mma(s, a, pl, qa, part, status)) return rc;
        } else {
            const size_t smem = sizeof(float) * (p.qld + p.rank + 64);
            if (int rc = allow_smem(latent_split_generic_kernel<T>, smem)) return rc;
            if (int rc = launch_pdl(latent_split_generic_kernel<T>, dim3(static_cast<unsigned>(p.splits), static_cast<unsigned>(p.H), static_cast<unsigned>(p.B)), dim3(128),
                                    smem, s, p, qa, static_cast<const T*>(a.cache), part)) return rc;
            note_latent_kernel("latent_split_generic_kernel");
        }
        profile_mark_end(s);
        const size_t v_smem = sizeof(float) * kBT * (p.rank16 + p.splits);
        if (int rc = allow_smem(latent_value_kernel<T>, v_smem)) return rc;
        const unsigned gx = static_cast<unsigned>(p.H * ((p.vdim + kValueRows - 1) / kValueRows));
        return launch_pdl(latent_value_kernel<T>, dim3(gx, bg), dim3(256), v_smem, s, p, part, static_cast<const T*>(a.w_uv), static_cast<T*>(a.out));
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace vb200
