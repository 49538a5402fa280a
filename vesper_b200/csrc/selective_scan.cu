// The selective state-space mixer with a state of its own per channel (Mamba-1): convolution and projections of the recurrence's inputs,
// and the recurrence
//
//   S[c, n] = exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,    y_c = sum_n S[c, n] C_n + D_c x_c,    out = y * silu(z).
//
// Every (channel, state) pair has its own decay, so a chunk of tokens is no matrix product: the work is one exponential and two
// multiply-adds per pair and token.  LP lanes share a channel, each holding NI of its states in registers over the whole portion; the
// tokens come in tiles through a two-stage shared-memory ring filled with cp.async while the tile before is walked.
#include "hybrid.cuh"

#include <type_traits>

namespace vb200 {
namespace {

constexpr int kThreads = 128;

struct ScanParams {
    int B, T, inner, N, rank;
    long long ldp, ldx, ldo;       // rows of proj, of [dt | B | C], of out
    const float *A, *D, *dt_bias;
    const int *slots, *pos;
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// exp(dt * a) * s + u.  fp32 form: s + (exp(dt * a) - 1) * s, because the rounding of a factor close to one would add up over a long
// memory.  Where activations are bf16: the base-2 instruction (2 ulp), dt then carries log2 e.
template <typename T> __device__ __forceinline__ float decayed(float s, float dt, float a, float u) {
    if constexpr (sizeof(T) == 4) return s + fmaf(expm1f(dt * a), s, u);
    else return fmaf(fast_exp2(dt * a), s, u);
}
template <typename T> __device__ __forceinline__ float decay_dt(float dt) { return sizeof(T) == 4 ? dt : dt * kLog2e; }

// log(1 + exp(x)).  bf16 form: log(1 + u) = 2 artanh(u / (2 + u)) with u = exp(-|x|) <= 1, the series up to the 13th power (its
// remainder is below 1e-8 of the sum at u = 1).
template <typename T> __device__ __forceinline__ float softplus_for(float x) {
    if constexpr (sizeof(T) == 4) return softplus_f(x);
    const float u = fast_exp2(-fabsf(x) * kLog2e), s = __fdividef(u, 2.0f + u), q = s * s;
    float r = 2.0f / 13.0f;
    r = fmaf(r, q, 2.0f / 11.0f); r = fmaf(r, q, 2.0f / 9.0f); r = fmaf(r, q, 2.0f / 7.0f);
    r = fmaf(r, q, 2.0f / 5.0f); r = fmaf(r, q, 2.0f / 3.0f); r = fmaf(r, q, 2.0f);
    return fmaxf(x, 0.f) + s * r;
}

template <int N> __device__ __forceinline__ void load_states(const __nv_bfloat16* p, float (&v)[N]) {
    static_assert(N % 4 == 0, "four at a time");
#pragma unroll
    for (int i = 0; i < N; i += 4) {
        const uint2 u = *reinterpret_cast<const uint2*>(p + i);
        const float2 a = Elem<__nv_bfloat16>::unpack2(u.x), b = Elem<__nv_bfloat16>::unpack2(u.y);
        v[i] = a.x; v[i + 1] = a.y; v[i + 2] = b.x; v[i + 3] = b.y;
    }
}
template <int N> __device__ __forceinline__ void load_states(const float* p, float (&v)[N]) {
    if constexpr (N == 2) {
        const float2 a = *reinterpret_cast<const float2*>(p);
        v[0] = a.x; v[1] = a.y;
    } else
#pragma unroll
    for (int i = 0; i < N; i += 4) {
        const float4 a = *reinterpret_cast<const float4*>(p + i);
        v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
    }
}

// a lane's states from / to memory; those from `count` on do not exist (zero, not stored)
template <int N> __device__ __forceinline__ void load_state(const float* p, int count, float (&v)[N]) {
    constexpr int W = N < 4 ? 2 : 4;
#pragma unroll
    for (int i = 0; i < N; i += W) {
        if constexpr (W == 2) {
            const float2 u = i < count ? *reinterpret_cast<const float2*>(p + i) : make_float2(0.f, 0.f);
            v[i] = u.x; v[i + 1] = u.y;
        } else {
            const float4 u = i < count ? *reinterpret_cast<const float4*>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            v[i] = u.x; v[i + 1] = u.y; v[i + 2] = u.z; v[i + 3] = u.w;
        }
    }
}
template <int N> __device__ __forceinline__ void store_state(float* p, int count, const float (&v)[N]) {
    constexpr int W = N < 4 ? 2 : 4;
#pragma unroll
    for (int i = 0; i < N; i += W) {
        if (i >= count) break;
        if constexpr (W == 2) *reinterpret_cast<float2*>(p + i) = make_float2(v[i], v[i + 1]);
        else *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
}

template <typename T, int LP, int NI>
struct ScanTile {
    static constexpr int kCh = kThreads / LP;                  // channels per CTA
    static constexpr int kStates = LP * NI;
    static constexpr int kTile = kStates > 256 ? 8 : 32;      // tokens per shared-memory tile
    struct Stage {
        alignas(16) T x[kTile][kCh], z[kTile][kCh];
        alignas(16) float dt[kTile][kCh];
        alignas(16) T bc[2][kTile][kStates];                   // B, C
    };
    Stage st[2];
    // of the tile being walked: step size (times log2 e in the bf16 form) and step size * input; B, C in fp32; y
    alignas(16) float2 dd[kTile][kCh];
    alignas(16) float bc[2][sizeof(T) == 2 ? kTile : 1][kStates];          // (fp32 inputs are read where they landed)
    alignas(16) float y[kTile][kCh + 1];
};

// grid (ceil(inner / kCh), B).  dt holds the step sizes before bias and softplus.
template <typename T, int LP, int NI>
__global__ void __launch_bounds__(kThreads)
selective_scan_kernel(ScanParams p, const T* __restrict__ proj, const T* __restrict__ xc, const T* __restrict__ xdbl, const float* __restrict__ dt, float* __restrict__ state,
                      T* __restrict__ out) {
    using S = ScanTile<T, LP, NI>;
    constexpr int CH = S::kCh, V = 16 / sizeof(T), kTile = S::kTile, U = NI <= 4 ? 4 : NI <= 8 ? 2 : 1;
    extern __shared__ __align__(16) uint8_t raw[];
    S& sm = *reinterpret_cast<S*>(raw);
    const int tid = threadIdx.x, lane = tid % LP, ch = tid / LP, b = blockIdx.y, c0 = blockIdx.x * CH, c = c0 + ch;
    const bool live = c < p.inner;
    // weights do not depend on the launch before
    float a[NI], S_[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int n = lane * NI + i;
        a[i] = live && n < p.N ? __ldg(p.A + static_cast<long long>(c) * p.N + n) : 0.f;
    }
    // the gating pass gives a thread the same two channels in every tile: kThreads is a multiple of CH / 2
    const int gk = (tid % (CH / 2)) * 2;
    const float Ds[2] = {c0 + gk < p.inner ? __ldg(p.D + c0 + gk) : 0.f, c0 + gk + 1 < p.inner ? __ldg(p.D + c0 + gk + 1) : 0.f};
    pdl_begin();
    const int pos = p.pos[b], slot = p.slots ? p.slots[b] : b;
    float* sp = state + (static_cast<long long>(slot) * p.inner + c) * p.N + lane * NI;
    load_state(sp, live && pos > 0 ? p.N - lane * NI : 0, S_);
    const long long m0 = static_cast<long long>(b) * p.T;
    auto load_tile = [&](int t0, int s) {
        typename S::Stage& st = sm.st[s];
        for (int i = tid; i < kTile * (CH / V); i += kThreads) {
            const int t = i / (CH / V), k = (i - t * (CH / V)) * V;
            const bool ok = t0 + t < p.T && c0 + k < p.inner;
            const long long m = ok ? m0 + t0 + t : m0;
            const int col = ok ? c0 + k : 0;
            cp_async16(&st.x[t][k], xc + m * p.inner + col, ok);
            cp_async16(&st.z[t][k], proj + m * p.ldp + p.inner + col, ok);
        }
        for (int i = tid; i < kTile * (CH / 4); i += kThreads) {
            const int t = i / (CH / 4), k = (i - t * (CH / 4)) * 4;
            const bool ok = t0 + t < p.T && c0 + k < p.inner;
            cp_async16(&st.dt[t][k], dt + (ok ? (m0 + t0 + t) * p.inner + c0 + k : 0), ok);
        }
        constexpr int kVs = (S::kStates + V - 1) / V;
        for (int i = tid; i < 2 * kTile * kVs; i += kThreads) {
            const int w = i / (kTile * kVs), j = i - w * (kTile * kVs), t = j / kVs, k = (j - t * kVs) * V;
            const bool ok = t0 + t < p.T && k < p.N;
            cp_async16(&st.bc[w][t][k], xdbl + (ok ? (m0 + t0 + t) * p.ldx + p.rank + w * p.N + k : 0), ok);
        }
        cp_async_commit();
    };
    const int n_tiles = (p.T + kTile - 1) / kTile;
    load_tile(0, 0);
    for (int it = 0; it < n_tiles; ++it) {
        const int t0 = it * kTile, nt = min(kTile, p.T - t0);
        if (it + 1 < n_tiles) { load_tile(t0 + kTile, (it + 1) & 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        typename S::Stage& st = sm.st[it & 1];
        // once per (token, channel): the softplus of the step size and its products; past the portion a step size of 0 keeps the state
        for (int i = tid; i < kTile * CH; i += kThreads) {
            const int t = i / CH, k = i - t * CH;
            const float bk = c0 + k < p.inner ? __ldg(p.dt_bias + c0 + k) : 0.f;
            const float d = t < nt ? softplus_for<T>(st.dt[t][k] + bk) : 0.f;
            sm.dd[t][k] = make_float2(decay_dt<T>(d), d * Elem<T>::to_f(st.x[t][k]));
        }
        if constexpr (sizeof(T) == 2) {
            for (int i = tid; i < kTile * S::kStates / 2; i += kThreads) {       // four of B and C's 2 * kTile * kStates values at a time
                float v[4];
                load_states(&st.bc[0][0][0] + i * 4, v);
                *reinterpret_cast<float4*>(&sm.bc[0][0][0] + i * 4) = make_float4(v[0], v[1], v[2], v[3]);
            }
        }
        __syncthreads();
        if constexpr (sizeof(T) == 2) {
            // U tokens at a time: their loads, exponentials and sums are independent, only S += is a chain.  In the smallest shape, which
            // runs with few warps, the next tokens' loads and exponentials are under way while the sums of these are finished.
            const float2* __restrict__ dd = &sm.dd[0][ch];
            const float *__restrict__ Bs = &sm.bc[0][0][lane * NI], *__restrict__ Cs = &sm.bc[1][0][lane * NI];
            float* __restrict__ ys = &sm.y[0][ch];
            struct Batch { float2 e[U][NI / 2], bx[U][NI / 2], c[U][NI / 2]; };
            auto prepare = [&](int tb, Batch& q) {
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const float2 d = dd[(tb + u) * CH];
                    float bn[NI], cn[NI];
                    load_states(Bs + (tb + u) * S::kStates, bn);
                    load_states(Cs + (tb + u) * S::kStates, cn);
                    const float2 dl2 = make_float2(d.x, d.x), dx2 = make_float2(d.y, d.y);
#pragma unroll
                    for (int i = 0; i < NI / 2; ++i) {
                        const float2 m = __fmul2_rn(dl2, make_float2(a[2 * i], a[2 * i + 1]));
                        q.e[u][i] = make_float2(fast_exp2(m.x), fast_exp2(m.y));
                        q.bx[u][i] = __fmul2_rn(dx2, make_float2(bn[2 * i], bn[2 * i + 1]));
                        q.c[u][i] = make_float2(cn[2 * i], cn[2 * i + 1]);
                    }
                }
            };
            auto finish = [&](int tb, const Batch& q) {
                float y[U];
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
                    for (int i = 0; i < NI / 2; ++i) {
                        const float2 n = __ffma2_rn(q.e[u][i], make_float2(S_[2 * i], S_[2 * i + 1]), q.bx[u][i]);
                        S_[2 * i] = n.x; S_[2 * i + 1] = n.y;
                        acc = __ffma2_rn(n, q.c[u][i], acc);
                    }
                    y[u] = acc.x + acc.y;
                }
                // sums over the channel's lanes: halves of the tokens are exchanged until every lane holds one of them
                if constexpr (U == 4 && LP >= 4) {
                    float z[2];
                    const bool odd = lane & 1, high = lane & 2;
#pragma unroll
                    for (int k = 0; k < 2; ++k) {        // tokens 0, 1 stay with even lanes, 2, 3 with odd ones
                        const float send = odd ? y[k] : y[k + 2], keep = odd ? y[k + 2] : y[k];
                        z[k] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, 1);
                    }
                    const float send = high ? z[0] : z[1], keep = high ? z[1] : z[0];
                    float v = keep + __shfl_xor_sync(0xFFFFFFFFu, send, 2);
#pragma unroll
                    for (int o = 4; o < LP; o <<= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
                    if (lane < 4) ys[(tb + (lane & 1) * 2 + ((lane >> 1) & 1)) * (CH + 1)] = v;
                } else {
#pragma unroll
                    for (int u = 0; u < U; ++u) {
#pragma unroll
                        for (int o = LP / 2; o > 0; o >>= 1) y[u] += __shfl_xor_sync(0xFFFFFFFFu, y[u], o);
                        if (lane == 0) ys[(tb + u) * (CH + 1)] = y[u];
                    }
                }
            };
            if constexpr (NI == 2) {
                Batch q[2];
                prepare(0, q[0]);
                for (int tb = 0; tb < nt; tb += 2 * U) { // kTile is a multiple of 2 U; tokens past the portion change nothing
                    prepare(tb + U, q[1]);
                    finish(tb, q[0]);
                    if (tb + 2 * U < nt) prepare(tb + 2 * U, q[0]);
                    finish(tb + U, q[1]);
                }
            } else {
                for (int tb = 0; tb < nt; tb += U) {
                    Batch q;
                    prepare(tb, q);
                    finish(tb, q);
                }
            }
        } else {
            for (int t = 0; t < nt; ++t) {
                const float2 d = sm.dd[t][ch];
                float bn[NI], cn[NI], y = 0.f;
                load_states(&st.bc[0][t][lane * NI], bn);
                load_states(&st.bc[1][t][lane * NI], cn);
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    S_[i] = decayed<T>(S_[i], d.x, a[i], d.y * bn[i]);
                    y = fmaf(S_[i], cn[i], y);
                }
#pragma unroll
                for (int o = LP / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xFFFFFFFFu, y, o);
                if (lane == 0) sm.y[t][ch] = y;
            }
        }
        __syncthreads();
        // gate and store, two channels per thread
        for (int i = tid; i < nt * (CH / 2); i += kThreads) {
            const int t = i / (CH / 2), k = gk;
            if (c0 + k >= p.inner) continue;
            const float v0 = fmaf(Ds[0], Elem<T>::to_f(st.x[t][k]), sm.y[t][k]) * silu_for<T>(Elem<T>::to_f(st.z[t][k]));
            const float v1 = fmaf(Ds[1], Elem<T>::to_f(st.x[t][k + 1]), sm.y[t][k + 1]) * silu_for<T>(Elem<T>::to_f(st.z[t][k + 1]));
            T* dst = out + (m0 + t0 + t) * p.ldo + c0 + k;
            if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst) = Elem<__nv_bfloat16>::pack2(v0, v1);
            else *reinterpret_cast<float2*>(dst) = make_float2(v0, v1);
        }
        __syncthreads();           // the stage after next is refilled at the top
    }
    store_state(sp, live ? p.N - lane * NI : 0, S_);
}

constexpr int kStepRows = 2;       // sequences that a CTA of the decode step takes in turn

// One token per sequence: grid (ceil(inner / kCh), ceil(B / rows)).  dt (nullable) holds the step sizes before bias and softplus; without it
// they are computed here: the LP lanes of a channel share its row of W_dt, which is fetched ahead of the wait and kept for all rows.
template <typename T, int LP, int NI>
__global__ void __launch_bounds__(kThreads)
selective_step_kernel(ScanParams p, int rows, const T* __restrict__ proj, const T* __restrict__ xc, const T* __restrict__ xdbl, const T* __restrict__ w_dt,
                      const float* __restrict__ dt, float* __restrict__ state, T* __restrict__ out) {
    constexpr int CH = kThreads / LP;
    extern __shared__ __align__(16) uint8_t raw[];
    float* sm = reinterpret_cast<float*>(raw);         // [rows][(dt |) B | C]
    const int tid = threadIdx.x, lane = tid % LP, b0 = blockIdx.y * rows, nb = min(rows, p.B - b0), c = blockIdx.x * CH + tid / LP, cc = min(c, p.inner - 1);
    const bool live = c < p.inner;
    float a[NI];
    load_state(p.A + static_cast<long long>(cc) * p.N + lane * NI, p.N - lane * NI, a);
    const float bias = __ldg(p.dt_bias + cc), Dc = __ldg(p.D + cc);
    constexpr int kAhead = 4;                          // pieces of W_dt kept in registers
    const int n8 = dt != nullptr ? 0 : p.rank / 8, skip = dt != nullptr ? p.rank : 0, ld = p.rank + 2 * p.N - skip;      // staged columns
    const T* wr = w_dt + static_cast<long long>(cc) * p.rank;
    Raw8<T> w[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (lane + i * LP < n8) w[i].load(wr + (lane + i * LP) * 8);
    pdl_begin();
    for (int r = 0; r < nb; ++r)
        for (int i = tid; i < ld; i += kThreads) sm[r * ld + i] = Elem<T>::to_f(xdbl[(b0 + r) * p.ldx + skip + i]);
    for (int r = 0; r < nb; ++r) {
        const int b = b0 + r, slot = p.slots ? p.slots[b] : b;
        float* sp = state + (static_cast<long long>(slot) * p.inner + cc) * p.N + lane * NI;
        float S_[NI];
        load_state(sp, p.N - lane * NI, S_);
        if (p.pos[b] == 0) {                           // a new sequence ignores what its slot holds
#pragma unroll
            for (int i = 0; i < NI; ++i) S_[i] = 0.f;
        }
        const float x = Elem<T>::to_f(xc[static_cast<long long>(b) * p.inner + cc]), z = Elem<T>::to_f(proj[b * p.ldp + p.inner + cc]);
        if (r == 0) __syncthreads();
        const float* row = sm + r * ld;
        float d = 0.f;
        auto dot8 = [&](const float (&wv)[8], int k) {
            const float4 u = *reinterpret_cast<const float4*>(row + k * 8), v = *reinterpret_cast<const float4*>(row + k * 8 + 4);
            d = fmaf(wv[0], u.x, fmaf(wv[1], u.y, fmaf(wv[2], u.z, fmaf(wv[3], u.w, d))));
            d = fmaf(wv[4], v.x, fmaf(wv[5], v.y, fmaf(wv[6], v.z, fmaf(wv[7], v.w, d))));
        };
#pragma unroll
        for (int i = 0; i < kAhead; ++i)
            if (lane + i * LP < n8) { float wv[8]; w[i].get(wv); dot8(wv, lane + i * LP); }
#pragma unroll 1
        for (int k = lane + kAhead * LP; k < n8; k += LP) { float wv[8]; load8(wr + k * 8, wv); dot8(wv, k); }
        if (dt != nullptr) d = dt[static_cast<long long>(b) * p.inner + cc];
        else {
#pragma unroll
            for (int o = LP / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xFFFFFFFFu, d, o);
        }
        d = softplus_for<T>(d + bias);
        const float dx = d * x, dl = decay_dt<T>(d);
        const float *Bn = row + ld - 2 * p.N + lane * NI, *Cn = Bn + p.N;
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            if (lane * NI + i < p.N) {
                S_[i] = decayed<T>(S_[i], dl, a[i], dx * Bn[i]);
                y = fmaf(S_[i], Cn[i], y);
            }
        }
#pragma unroll
        for (int o = LP / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xFFFFFFFFu, y, o);
        if (!live) continue;
        store_state(sp, p.N - lane * NI, S_);
        if (lane == 0) out[(b0 + r) * p.ldo + c] = Elem<T>::from_f(fmaf(Dc, x, y) * silu_for<T>(z));
    }
}

// Calls f(LP, NI) with compile-time sizes that hold N states; the fewer CTAs there would be, the fewer states per lane (a decode step: four).
template <typename F>
int with_shape(int N, long long pairs, bool step, F f) {
    const long long sms = device_sm_count();
    const bool wide = step || pairs < 4 * 8 * kThreads * sms, widest = !step && pairs < 2 * 4 * kThreads * sms;
    using std::integral_constant;
    auto lanes = [&](auto ni) -> int {
        const int need = (N + decltype(ni)::value - 1) / decltype(ni)::value;
        if (need <= 2) return f(integral_constant<int, 2>{}, ni);
        if (need <= 4) return f(integral_constant<int, 4>{}, ni);
        if (need <= 8) return f(integral_constant<int, 8>{}, ni);
        return f(integral_constant<int, 16>{}, ni);
    };
    if (N <= 32 && widest) return lanes(integral_constant<int, 2>{});
    if (N <= 64 && (wide || N == 8)) return lanes(integral_constant<int, 4>{});
    if (N <= 128) return lanes(integral_constant<int, 8>{});
    if (N <= 256) return f(integral_constant<int, 16>{}, integral_constant<int, 16>{});
    return f(integral_constant<int, 16>{}, integral_constant<int, 32>{});
}

int product(cudaStream_t s, int dtype, const void* x, long long ldx, const void* w, long long ldw, void* out, long long ldo, int M, int N, int K, bool f32_out, int* status) {
    if (dtype == VB200_F32)
        return launch_linear_f32(s, static_cast<const float*>(x), ldx, static_cast<const float*>(w), ldw, nullptr, static_cast<float*>(out), ldo, M, N, K);
    LinearParams p{};
    p.x = x; p.ldx = ldx; p.w = w; p.ldw = ldw; p.out = out; p.ldo = ldo; p.M = M; p.N = N; p.K = K;
    p.epilogue = f32_out ? VB200_EPI_F32 : VB200_EPI_BF16;
    p.status = status;
    return launch_linear(s, p);
}

}  // namespace

SelectivePlan plan_selective(const vb200_selective_args& a) {
    SelectivePlan pl{};
    auto up = [](size_t x) { return (x + 255) / 256 * 256; };
    const size_t esz = a.dtype == VB200_F32 ? 4 : 2, M = static_cast<size_t>(a.B) * a.T;
    pl.dt_gemm = a.T > 1 || a.B >= 16;          // few rows: W_dt streams through the step kernel instead
    pl.conv_bytes = up(M * a.inner * esz);
    pl.xdbl_bytes = up(M * (a.rank + 2 * a.N) * esz);
    pl.dt_bytes = pl.dt_gemm ? up(M * a.inner * 4) : 0;
    pl.total = pl.conv_bytes + pl.xdbl_bytes + pl.dt_bytes;
    return pl;
}

int launch_selective(cudaStream_t s, const vb200_selective_args& a, const SelectivePlan& pl, int* status) {
    uint8_t* ws = static_cast<uint8_t*>(a.workspace);
    void *xc = ws, *xdbl = ws + pl.conv_bytes;
    float* dt = reinterpret_cast<float*>(ws + pl.conv_bytes + pl.xdbl_bytes);
    const int M = a.B * a.T, ldx = a.rank + 2 * a.N;
    if (int rc = launch_causal_conv(s, ConvLaunch{a.dtype, a.B, a.T, a.inner, a.taps, a.proj, a.ldp, 0, a.conv_w, a.conv_b, a.slots, a.pos, a.conv_state, xc})) return rc;
    if (int rc = product(s, a.dtype, xc, a.inner, a.w_x, a.inner, xdbl, ldx, M, ldx, a.inner, false, status)) return rc;
    if (pl.dt_gemm)
        if (int rc = product(s, a.dtype, xdbl, ldx, a.w_dt, a.rank, dt, a.inner, M, a.inner, a.rank, true, status)) return rc;
    ScanParams p{};
    p.B = a.B; p.T = a.T; p.inner = a.inner; p.N = a.N; p.rank = a.rank; p.ldp = a.ldp; p.ldx = ldx; p.ldo = a.ldo;
    p.A = a.A; p.D = a.D; p.dt_bias = a.dt_bias; p.slots = a.slots; p.pos = a.pos;
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        const T *proj = static_cast<const T*>(a.proj), *x = static_cast<const T*>(xc), *d = static_cast<const T*>(xdbl);
        T* out = static_cast<T*>(a.out);
        return with_shape(a.N, static_cast<long long>(a.B) * a.inner * a.N, a.T == 1, [&](auto lp, auto ni) -> int {
            constexpr int LP = decltype(lp)::value, NI = decltype(ni)::value, CH = kThreads / LP;
            const dim3 grid(static_cast<unsigned>((a.inner + CH - 1) / CH), static_cast<unsigned>(a.B));
            profile_mark_begin(s);
            int rc;
            if (a.T == 1) {
                // rows per CTA: W_dt and A are read once for them, as long as six CTAs per SM remain
                int rows = 1;
                while (rows < kStepRows && rows < a.B && static_cast<long long>(grid.x) * ((a.B + 2 * rows - 1) / (2 * rows)) >= 6 * device_sm_count()) rows *= 2;
                const dim3 step_grid(grid.x, static_cast<unsigned>((a.B + rows - 1) / rows));
                const size_t smem = sizeof(float) * ldx * rows;
                rc = allow_smem(selective_step_kernel<T, LP, NI>, smem);
                if (rc == VB200_OK) rc = launch_pdl(selective_step_kernel<T, LP, NI>, step_grid, dim3(kThreads), smem, s, p, rows, proj, x, d, static_cast<const T*>(a.w_dt), static_cast<const float*>(pl.dt_gemm ? dt : nullptr), a.state, out);
                note_selective_kernel("selective_step_kernel");
            } else {
                const size_t smem = sizeof(ScanTile<T, LP, NI>);
                rc = allow_smem(selective_scan_kernel<T, LP, NI>, smem);
                // no programmatic launch: scheduled while the product before drains, the CTAs would pile up on the SMs that finish first
                if (rc == VB200_OK) {
                    selective_scan_kernel<T, LP, NI><<<grid, kThreads, smem, s>>>(p, proj, x, d, dt, a.state, out);
                    note_launch();
                    VB200_CUDA_TRY(cudaPeekAtLastError());
                }
                note_selective_kernel("selective_scan_kernel");
            }
            profile_mark_end(s);
            return rc;
        });
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace vb200
