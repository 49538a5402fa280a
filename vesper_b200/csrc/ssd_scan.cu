// The Mamba-2 mixer around its projections: causal convolution, the recurrence token by token (any sizes, fp32 or bf16;
// decode steps and short portions), and the gated group RMSNorm.  The chunked form of the recurrence for prompts is in
// ssd_chunk.cu.  (The convolution of a decode step is a launch of its own: inside the recurrence every head of a group
// would repeat it for B and C, and measured slower.)
#include "hybrid.cuh"

namespace vb200 {
namespace {

struct SsdParams {
    int B, T, H, P, N, G, taps, channels, Pp;
    long long ldp;
    const float *conv_w, *conv_b, *dt_bias, *A_log, *D;
    const int *slots, *pos;
    int slices, p4s, rows;      // scan kernel: slices of a head's columns, float4 columns per slice, state rows per pass
};

struct ConvTask {
    int T, taps, channels;
    long long ldp;
    const float *conv_w, *conv_b;
    const int *slots, *pos;
    long long col;              // first convolved column of a projection row
};

constexpr int kConvTile = 32;   // tokens per CTA
constexpr int kAhead = 8;       // tokens whose loads are in flight

__device__ __forceinline__ void load2(const __nv_bfloat16* p, float (&v)[2]) {
    const float2 f = Elem<__nv_bfloat16>::unpack2(*reinterpret_cast<const uint32_t*>(p));
    v[0] = f.x; v[1] = f.y;
}
__device__ __forceinline__ void load2(const float* p, float (&v)[2]) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
}
__device__ __forceinline__ void store2(__nv_bfloat16* p, const float (&v)[2]) { *reinterpret_cast<uint32_t*>(p) = Elem<__nv_bfloat16>::pack2(v[0], v[1]); }
__device__ __forceinline__ void store2(float* p, const float (&v)[2]) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }

// grid (channel blocks, token tiles, B); a thread owns VEC channels.  Only the first tile's CTA reads the state (the
// inputs ahead of the portion) and it alone writes it, after its own reads.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
ssd_conv_kernel(ConvTask p, const T* __restrict__ proj, T* __restrict__ state, T* __restrict__ out) {
    pdl_begin();
    const int c0 = (blockIdx.x * 128 + threadIdx.x) * VEC;
    if (c0 >= p.channels) return;
    const int b = blockIdx.z, t0 = blockIdx.y * kConvTile, t1 = min(p.T, t0 + kConvTile);
    const int taps = TAPS > 0 ? TAPS : p.taps;
    const int pos = p.pos[b], slot = p.slots ? p.slots[b] : b;
    const T* in = proj + static_cast<long long>(b) * p.T * p.ldp + p.col + c0;
    T* st = state + static_cast<long long>(slot) * taps * p.channels + c0;
    T* o = out + static_cast<long long>(b) * p.T * p.channels + c0;
    auto fetch = [&](int t, float (&v)[VEC]) {           // the input of portion token t, which may lie ahead of the portion
        const T* src = t >= 0 ? in + static_cast<long long>(t) * p.ldp
                              : (pos + t >= 0 ? st + static_cast<long long>((pos + t) % taps) * p.channels : nullptr);
        if (src == nullptr) {
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = 0.f;
        } else if constexpr (VEC == 2) {
            load2(src, v);
        } else {
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = Elem<T>::to_f(src[j]);
        }
    };
    auto emit = [&](int t, float (&a)[VEC]) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) a[j] = silu_for<T>(a[j]);
        T* dst = o + static_cast<long long>(t) * p.channels;
        if constexpr (VEC == 2) store2(dst, a);
        else {
#pragma unroll
            for (int j = 0; j < VEC; ++j) dst[j] = Elem<T>::from_f(a[j]);
        }
    };
    float bias[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) bias[j] = p.conv_b[c0 + j];
    if constexpr (TAPS > 0) {
        float w[TAPS][VEC], x[TAPS - 1 + kAhead][VEC];           // a window of inputs: the taps before a block, then the block
#pragma unroll
        for (int j = 0; j < VEC; ++j)
#pragma unroll
            for (int k = 0; k < TAPS; ++k) w[k][j] = p.conv_w[static_cast<long long>(c0 + j) * TAPS + k];
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k) fetch(t0 - (TAPS - 1) + k, x[k]);
        for (int tb = t0; tb < t1; tb += kAhead) {
            const int n = min(kAhead, t1 - tb);
            const T* src = in + static_cast<long long>(tb) * p.ldp;
#pragma unroll
            for (int u = 0; u < kAhead; ++u) {
                const T* q = src + static_cast<long long>(min(u, n - 1)) * p.ldp;
                if constexpr (VEC == 2) load2(q, x[TAPS - 1 + u]);
                else x[TAPS - 1 + u][0] = Elem<T>::to_f(q[0]);
            }
#pragma unroll
            for (int u = 0; u < kAhead; ++u) {
                float a[VEC];
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    a[j] = bias[j];
#pragma unroll
                    for (int k = 0; k < TAPS; ++k) a[j] = fmaf(w[k][j], x[u + k][j], a[j]);
                }
                if (u < n) emit(tb + u, a);
            }
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
                for (int j = 0; j < VEC; ++j) x[k][j] = x[kAhead + k][j];
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            float a[VEC];
#pragma unroll
            for (int j = 0; j < VEC; ++j) a[j] = bias[j];
            for (int k = 0; k < taps; ++k) {
                float v[VEC];
                fetch(t - (taps - 1) + k, v);
#pragma unroll
                for (int j = 0; j < VEC; ++j) a[j] = fmaf(p.conv_w[static_cast<long long>(c0 + j) * taps + k], v[j], a[j]);
            }
            emit(t, a);
        }
    }
    if (t0 == 0) {
        for (int t = max(0, p.T - (taps - 1)); t < p.T; ++t) {
            T* dst = st + static_cast<long long>((pos + t) % taps) * p.channels;
#pragma unroll
            for (int j = 0; j < VEC; ++j) dst[j] = in[static_cast<long long>(t) * p.ldp + j];
        }
    }
}

// grid (H * slices, B), 256 threads: thread = one float4 column of the slice x every `rows`-th state row, the state in
// registers over the whole portion (decode: one token).
template <typename T, int NI>
__global__ void __launch_bounds__(256, NI <= 4 ? 4 : NI <= 8 ? 3 : 2)
ssd_scan_kernel(SsdParams p, const T* __restrict__ proj, const T* __restrict__ xbc, float* __restrict__ state, float* __restrict__ gated) {
    pdl_begin();
    extern __shared__ float sm[];
    const int h = blockIdx.x / p.slices, sl = blockIdx.x - h * p.slices, b = blockIdx.y;
    const int g = h / (p.H / p.G), inner = p.H * p.P;
    const int pos = p.pos[b], slot = p.slots ? p.slots[b] : b;
    const int pc0 = sl * p.p4s * 4, pcn = min(p.P - pc0, p.p4s * 4);          // this slice's columns
    const int width = p.p4s * 4, buf_floats = width + 2 * p.N;
    float* red = sm + 2 * buf_floats;                                          // [rows][width]
    const int c4 = threadIdx.x % p.p4s, r = threadIdx.x / p.p4s;
    const bool active = r < p.rows && pc0 + c4 * 4 < p.Pp;
    float* sp = state + (static_cast<long long>(slot) * p.H + h) * p.N * p.Pp + pc0 + c4 * 4;
    float4 S[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = r + i * p.rows;
        S[i] = active && n < p.N && pos > 0 ? *reinterpret_cast<const float4*>(sp + static_cast<long long>(n) * p.Pp) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float nA = -expf(p.A_log[h]), dtb = p.dt_bias[h], Dh = p.D[h];
    for (int t = 0; t < p.T; ++t) {
        const long long m = static_cast<long long>(b) * p.T + t;
        const T* prow = proj + m * p.ldp;
        float* buf = sm + (t & 1) * buf_floats;
        float *xs = buf, *Bs = buf + width, *Cs = Bs + p.N;
        for (int i = threadIdx.x; i < width + 2 * p.N; i += 256) {
            int ch;
            if (i < width) {
                if (i >= pcn) { buf[i] = 0.f; continue; }
                ch = h * p.P + pc0 + i;
            } else {
                const int k = i - width;
                ch = inner + (k < p.N ? g * p.N + k : p.G * p.N + g * p.N + k - p.N);
            }
            buf[i] = Elem<T>::to_f(xbc[m * p.channels + ch]);
        }
        const float dt = softplus_f(Elem<T>::to_f(prow[2 * inner + 2 * p.G * p.N + h]) + dtb), decay = expf(nA * dt);
        __syncthreads();
        if (active) {
            const float4 x4 = *reinterpret_cast<const float4*>(xs + c4 * 4);
            const float4 dx = make_float4(dt * x4.x, dt * x4.y, dt * x4.z, dt * x4.w);
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int n = r + i * p.rows;
                if (n < p.N) {
                    const float bn = Bs[n], cn = Cs[n];
                    S[i].x = fmaf(decay, S[i].x, bn * dx.x); S[i].y = fmaf(decay, S[i].y, bn * dx.y);
                    S[i].z = fmaf(decay, S[i].z, bn * dx.z); S[i].w = fmaf(decay, S[i].w, bn * dx.w);
                    y.x = fmaf(cn, S[i].x, y.x); y.y = fmaf(cn, S[i].y, y.y);
                    y.z = fmaf(cn, S[i].z, y.z); y.w = fmaf(cn, S[i].w, y.w);
                }
            }
            *reinterpret_cast<float4*>(red + r * width + c4 * 4) = y;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < pcn; i += 256) {
            float y = 0.f;
            for (int k = 0; k < p.rows; ++k) y += red[k * width + i];
            y = fmaf(Dh, xs[i], y);
            const int col = h * p.P + pc0 + i;
            gated[m * inner + col] = y * silu_for<T>(Elem<T>::to_f(prow[col]));
        }
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = r + i * p.rows;
        if (active && n < p.N) *reinterpret_cast<float4*>(sp + static_cast<long long>(n) * p.Pp) = S[i];
    }
}

// grid (norm groups, rows), 128 threads.  VEC: eight elements at a time, up to 64 per thread held in registers.
template <typename GT, typename T, bool VEC>
__global__ void __launch_bounds__(128)
gated_group_norm_kernel(const GT* __restrict__ gated, int inner, int part_len, const float* __restrict__ w, float eps, T* __restrict__ out, long long ldo) {
    pdl_begin();
    const long long m = blockIdx.y;
    const int c0 = blockIdx.x * part_len;
    const GT* src = gated + m * inner + c0;
    T* dst = out + m * ldo + c0;
    __shared__ float part[4];
    float ss = 0.f;
    if constexpr (VEC) {
        constexpr int kMax = 8;
        float v[kMax][8];
        const int n8 = part_len / 8;
#pragma unroll
        for (int i = 0; i < kMax; ++i) {
            const int k = threadIdx.x + i * 128;
            if (k < n8) load8(src + k * 8, v[i]);
        }
#pragma unroll
        for (int i = 0; i < kMax; ++i)
            if (threadIdx.x + i * 128 < n8) {
#pragma unroll
                for (int e = 0; e < 8; ++e) ss += v[i][e] * v[i][e];
            }
        const float inv = 1.0f / sqrtf(block_sum<4>(ss, part) / static_cast<float>(part_len) + eps);
#pragma unroll
        for (int i = 0; i < kMax; ++i) {
            const int k = threadIdx.x + i * 128;
            if (k >= n8) break;
            float wv[8];
            load8(w + c0 + k * 8, wv);
#pragma unroll
            for (int e = 0; e < 8; ++e) wv[e] *= v[i][e] * inv;
            store8(dst + k * 8, wv);
        }
    } else {
        for (int i = threadIdx.x; i < part_len; i += 128) { const float v = Elem<GT>::to_f(src[i]); ss += v * v; }
        const float inv = 1.0f / sqrtf(block_sum<4>(ss, part) / static_cast<float>(part_len) + eps);
        for (int i = threadIdx.x; i < part_len; i += 128) dst[i] = Elem<T>::from_f(Elem<GT>::to_f(src[i]) * inv * w[c0 + i]);
    }
}

template <typename GT, typename T>
int launch_group_norm(cudaStream_t s, const vb200_ssd_args& a, const void* gated) {
    const int inner = a.H * a.P, len = inner / a.norm_groups;
    const bool vec = len % 8 == 0 && len <= 8192 && a.ldo % 8 == 0 && reinterpret_cast<uintptr_t>(a.norm_w) % 16 == 0 && reinterpret_cast<uintptr_t>(a.out) % 16 == 0;
    const dim3 grid(static_cast<unsigned>(a.norm_groups), static_cast<unsigned>(a.B * a.T));
    return launch_pdl(vec ? gated_group_norm_kernel<GT, T, true> : gated_group_norm_kernel<GT, T, false>, grid, dim3(128), 0, s, static_cast<const GT*>(gated), inner, len,
                      a.norm_w, a.eps, static_cast<T*>(a.out), static_cast<long long>(a.ldo));
}

}  // namespace

SsdPlan plan_ssd(const vb200_ssd_args& a) {
    SsdPlan pl{};
    pl.channels = a.H * a.P + 2 * a.G * a.N;
    pl.Pp = pad_to(a.P, 4);
    pl.chunked = a.T > 1 && a.form != 1 && ssd_chunk_supported(a) && (a.form >= 2 || a.T >= 16);
    const size_t esz = a.dtype == VB200_F32 ? 4 : 2, M = static_cast<size_t>(a.B) * a.T;
    auto up = [](size_t x) { return (x + 255) / 256 * 256; };
    pl.conv_bytes = up(M * pl.channels * esz);
    pl.gated_bytes = up(M * a.H * a.P * (pl.chunked ? 2 : 4));
    if (pl.chunked) {
        int slices, n_seg, seg_chunks;
        plan_ssd_chunks(a, &slices, &n_seg, &seg_chunks);
        if (n_seg > 1) pl.chunk_bytes = up(sizeof(float) * (static_cast<size_t>(a.B) * n_seg * a.H * (static_cast<size_t>(a.N) * pl.Pp + 1) + 64));
    }
    pl.total = pl.conv_bytes + pl.gated_bytes + pl.chunk_bytes;
    return pl;
}

int launch_causal_conv(cudaStream_t s, const ConvLaunch& c) {
    const ConvTask p{c.T, c.taps, c.channels, c.ldp, c.w, c.b, c.slots, c.pos, c.col};
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        const bool vec = c.col % 2 == 0 && c.channels % 2 == 0 && c.ldp % 2 == 0;
        auto conv = [&](auto kernel, int v) {
            const dim3 grid(static_cast<unsigned>((c.channels + 128 * v - 1) / (128 * v)), static_cast<unsigned>((c.T + kConvTile - 1) / kConvTile), static_cast<unsigned>(c.B));
            return launch_pdl(kernel, grid, dim3(128), 0, s, p, static_cast<const T*>(c.proj), static_cast<T*>(c.state), static_cast<T*>(c.out));
        };
        return vec ? (c.taps == 4 ? conv(ssd_conv_kernel<T, 2, 4>, 2) : conv(ssd_conv_kernel<T, 2, 0>, 2))
                   : (c.taps == 4 ? conv(ssd_conv_kernel<T, 1, 4>, 1) : conv(ssd_conv_kernel<T, 1, 0>, 1));
    };
    return c.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

int launch_ssd(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, int* status) {
    SsdParams p{};
    p.B = a.B; p.T = a.T; p.H = a.H; p.P = a.P; p.N = a.N; p.G = a.G; p.taps = a.taps; p.channels = pl.channels; p.Pp = pl.Pp;
    p.ldp = a.ldp; p.conv_w = a.conv_w; p.conv_b = a.conv_b; p.dt_bias = a.dt_bias; p.A_log = a.A_log; p.D = a.D; p.slots = a.slots; p.pos = a.pos;
    // slices: few enough state rows per thread for registers, and enough CTAs for the machine
    const int P4 = pl.Pp / 4;
    int slices = (P4 + 255) / 256;
    auto per_thread = [&](int sl) { const int w = (P4 + sl - 1) / sl; return (a.N + 256 / w - 1) / (256 / w); };
    while (slices < P4 && per_thread(slices) > 16) ++slices;
    if (per_thread(slices) > 16) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_ssd_forward: state size above 4096");
    while (2 * slices <= P4 && static_cast<long long>(a.B) * a.H * slices * 2 <= device_sm_count()) slices *= 2;
    p.slices = slices;
    p.p4s = (P4 + slices - 1) / slices;
    p.rows = 256 / p.p4s;
    const int ni = (a.N + p.rows - 1) / p.rows;
    uint8_t* ws = static_cast<uint8_t*>(a.workspace);
    void* xbc = ws;
    void* gated = ws + pl.conv_bytes;
    float* states = reinterpret_cast<float*>(ws + pl.conv_bytes + pl.gated_bytes);

    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        const T* proj = static_cast<const T*>(a.proj);
        if (int rc = launch_causal_conv(s, ConvLaunch{a.dtype, a.B, a.T, p.channels, a.taps, a.proj, a.ldp, static_cast<long long>(a.H) * a.P, a.conv_w, a.conv_b, a.slots,
                                                      a.pos, a.conv_state, xbc})) return rc;
        if constexpr (sizeof(T) == 2) {
            if (pl.chunked) {
                if (int rc = launch_ssd_chunks(s, a, pl, xbc, gated, states, status)) return rc;
                return launch_group_norm<__nv_bfloat16, T>(s, a, gated);
            }
        }
        const size_t smem = sizeof(float) * (2 * (p.p4s * 4 + 2 * a.N) + p.rows * p.p4s * 4);
        const dim3 grid(static_cast<unsigned>(a.H * p.slices), static_cast<unsigned>(a.B));
        auto scan = [&](auto kernel) -> int {
            if (int rc = allow_smem(kernel, smem)) return rc;
            return launch_pdl(kernel, grid, dim3(256), smem, s, p, proj, static_cast<const T*>(xbc), a.state, static_cast<float*>(gated));
        };
        int rc;
        profile_mark_begin(s);
        rc = ni <= 4 ? scan(ssd_scan_kernel<T, 4>) : ni <= 8 ? scan(ssd_scan_kernel<T, 8>) : scan(ssd_scan_kernel<T, 16>);
        profile_mark_end(s);
        if (rc) return rc;
        note_ssd_kernel("ssd_scan_kernel");
        return launch_group_norm<float, T>(s, a, gated);
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace vb200
