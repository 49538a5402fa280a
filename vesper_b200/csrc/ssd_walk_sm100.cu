// The chunked Mamba-2 walk (ssd_chunk.cu has the equations) on the sm_100a tensor cores: heads of up to 64 columns and
// 128 state rows, chunks of 128 tokens, one CTA per (batch, head) and segment, one CTA per SM.
//
//   G  = C B^T                      128 x 128 x N     A, B from shared memory
//   Y  = C S                        128 x 64 x N      S = hi + lo bf16 halves in shared memory
//   Y  = 2^la Y + M x               128 x 64 x 128    M = mask(G) 2^(la_i - la_j) dt_j = hi + lo, from TMEM
//   S += B^T (w x)                  N x 64 x 128      A = the B tile read MN-major; w x = hi + lo in shared memory
//
// S stays in TMEM (fp32) over the whole walk; before a chunk's update it is scaled by the chunk's decay and published to
// shared memory as the next C S operand.  The decays touch fp32 values only; every product operand they enter is split.
//   warps 0-7  compute: row = TMEM lane, the two warpgroups share a row's columns
//   warp  8    TMA: C, B and x of the next chunk into the second buffers (128-byte swizzle)
//   warp  9    tcgen05.mma issuer, TMEM owner
// TMEM (512 columns): G [0,128) Y [128,192) S [192,256) M [256,384): hi in its first 64 columns, lo in the others.
// All hand-overs are mbarriers with bounded waits; there is no CTA barrier inside the walk.
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kL = 128;                   // tokens per chunk
constexpr int kBox = kL * 128;            // one [128 rows x 64 columns] box
constexpr int kStage = 5 * kBox;          // C (2 boxes), B (2), x (1)
constexpr int kSmem = 2 * kStage + 4 * kBox;          // + w x (hi, lo), S (hi, lo)
constexpr int kThreads = 320;

struct WalkMaps { CUtensorMap x, b, c; };

struct WalkParams {
    int T, H, P, N, G, Pp, nk, n_seg, seg_chunks;          // seg_chunks: 128-token chunks per segment
    long long ldp;
    const __nv_bfloat16* proj;
    const float *dt_bias, *A_log, *D;
    const int *slots, *pos;
    float* state;
    const float* seg_state;
    __nv_bfloat16* gated;
    int* status;
};

struct WalkBars {
    float la[2][kL], dt[2][kL];           // running log2-decays and step sizes of a chunk
    uint64_t tiles_full[2], tiles_empty[2], dt_ready, g_full, cs_full, xw_ready, p_ready, s_ready, u_full, y_full, y_free, drain;
    uint32_t tmem;
    int abort_flag;
};

__global__ void __launch_bounds__(kThreads, 1)
ssd_walk_sm100_kernel(const __grid_constant__ WalkMaps maps, WalkParams p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ WalkBars bar;
    uint8_t* xw = smem + 2 * kStage;                 // hi, lo
    uint8_t* ss = xw + 2 * kBox;                     // hi, lo
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seg = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
    const int c_begin = seg * p.seg_chunks, n_chunk = min((p.T + kL - 1) / kL, c_begin + p.seg_chunks) - c_begin;
    const WaitCtx ctx{&bar.abort_flag, p.status};

    if (threadIdx.x == 0) {
        bar.abort_flag = 0;
        for (int i = 0; i < 2; ++i) { mbar_init(&bar.tiles_full[i], 1); mbar_init(&bar.tiles_empty[i], 1 + 256); }
        mbar_init(&bar.dt_ready, 32);
        mbar_init(&bar.g_full, 1); mbar_init(&bar.cs_full, 1); mbar_init(&bar.u_full, 1); mbar_init(&bar.y_full, 1);
        mbar_init(&bar.xw_ready, 256); mbar_init(&bar.p_ready, 256); mbar_init(&bar.s_ready, 256); mbar_init(&bar.y_free, 256);
        mbar_init(&bar.drain, 1);
        mbar_fence_init();
        if ((smem_u32(smem) & 1023) != 0) { bar.abort_flag = 1; atomicCAS(p.status, 0, (3 << 24) | 0x3); }      // the swizzle needs 1024-byte tiles
    }
    if (warp == 9) { tmem_alloc(&bar.tmem, 512); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bar.tmem, t_y = tmem + 128, t_s = tmem + 192, t_m = tmem + 256;
    const bool dead = *static_cast<volatile int*>(&bar.abort_flag) != 0;
    __syncthreads();
    pdl_begin();

    if (dead) {
    } else if (warp == 8) {
        if (lane == 0) {
            const int grp = h / (p.H / p.G);
            for (int k = 0; k < n_chunk; ++k) {
                const int q = k & 1, t0 = (c_begin + k) * kL;
                if (k >= 2 && !mbar_wait(&bar.tiles_empty[q], (k / 2 - 1) & 1, ctx, 0xD1)) break;
                uint8_t* st = smem + q * kStage;
                mbar_arrive_expect_tx(&bar.tiles_full[q], kStage);
                for (int i = 0; i < 2; ++i) tma_load_4d(st + i * kBox, &maps.c, &bar.tiles_full[q], i * 64, grp, t0, b);
                for (int i = 0; i < 2; ++i) tma_load_4d(st + (2 + i) * kBox, &maps.b, &bar.tiles_full[q], i * 64, grp, t0, b);
                tma_load_4d(st + 4 * kBox, &maps.x, &bar.tiles_full[q], 0, h, t0, b);
            }
        }
    } else if (warp == 9) {
        if (lane == 0) {
            constexpr uint32_t id_g = make_idesc_f16(1, 0, 0, 128, 128), id_cs = make_idesc_f16(1, 0, 1, 128, 64), id_u = make_idesc_f16(1, 1, 1, 128, 64);
            const uint32_t xw_a = smem_u32(xw), ss_a = smem_u32(ss);
            for (int k = 0; k < n_chunk; ++k) {
                const int q = k & 1, ph = k & 1;
                if (!mbar_wait(&bar.tiles_full[q], (k / 2) & 1, ctx, 0xD2)) break;
                tc_fence_after();
                const uint32_t c_a = smem_u32(smem + q * kStage), b_a = c_a + 2 * kBox, x_a = c_a + 4 * kBox;
                for (int kk = 0; kk < p.nk; ++kk) {
                    const uint32_t off = (kk >> 2) * kBox + (kk & 3) * 32;
                    umma_ss(tmem, make_smem_desc_sw128(c_a + off, 16, 1024), make_smem_desc_sw128(b_a + off, 16, 1024), id_g, kk > 0 ? 1u : 0u);
                }
                umma_commit(&bar.g_full);
                if (!mbar_wait(&bar.s_ready, ph, ctx, 0xD3)) break;
                if (k > 0 && !mbar_wait(&bar.y_free, (k - 1) & 1, ctx, 0xD4)) break;
                tc_fence_after();
                for (int half = 0; half < 2; ++half)
                    for (int kk = 0; kk < p.nk; ++kk)
                        umma_ss(t_y, make_smem_desc_sw128(c_a + (kk >> 2) * kBox + (kk & 3) * 32, 16, 1024), make_smem_desc_sw128(ss_a + half * kBox + kk * 2048, kBox, 1024), id_cs,
                                (half | kk) ? 1u : 0u);
                umma_commit(&bar.cs_full);
                if (!mbar_wait(&bar.xw_ready, ph, ctx, 0xD5)) break;
                tc_fence_after();
                for (int half = 0; half < 2; ++half)
                    for (int kk = 0; kk < kL / 16; ++kk)
                        umma_ss(t_s, make_smem_desc_sw128(b_a + kk * 2048, kBox, 1024), make_smem_desc_sw128(xw_a + half * kBox + kk * 2048, kBox, 1024), id_u, 1u);
                umma_commit(&bar.u_full);
                if (!mbar_wait(&bar.p_ready, ph, ctx, 0xD6)) break;
                tc_fence_after();
                for (int half = 0; half < 2; ++half)
                    for (int kk = 0; kk < kL / 16; ++kk)
                        umma_ts(t_y, t_m + half * 64 + kk * 8, make_smem_desc_sw128(x_a + kk * 2048, kBox, 1024), id_cs, 1u);
                umma_commit(&bar.y_full);
                umma_commit(&bar.tiles_empty[q]);
            }
            umma_commit(&bar.drain);                 // nothing may be in flight when TMEM is freed
            mbar_wait(&bar.drain, 0, ctx, 0xD7);
        }
    } else {
        const int r = threadIdx.x & 127, half = threadIdx.x >> 7;           // TMEM lane, column half
        const uint32_t lane_base = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const int inner = p.H * p.P, slot = p.slots ? p.slots[b] : b, col0 = half * 32;
        const float nA2 = -expf(p.A_log[h]) * kLog2e, dtb = p.dt_bias[h], Dh = p.D[h];
        const __nv_bfloat16* proj = p.proj + static_cast<long long>(b) * p.T * p.ldp;
        const long long state_row = ((static_cast<long long>(slot) * p.H + h) * p.N + r) * p.Pp;
        // step sizes and running log-decays of a chunk: warp 0, four tokens per lane
        float raw[4] = {0.f, 0.f, 0.f, 0.f};
        auto fetch_dt = [&](int k) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = (c_begin + k) * kL + lane * 4 + e;
                raw[e] = t < p.T ? __bfloat162float(proj[static_cast<long long>(t) * p.ldp + 2 * inner + 2 * p.G * p.N + h]) : 0.f;
            }
        };
        auto scan_dt = [&](int k) {
            float d[4], a[4], s = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                d[e] = (c_begin + k) * kL + lane * 4 + e < p.T ? softplus_f(raw[e] + dtb) : 0.f;
                s += nA2 * d[e];
                a[e] = s;
            }
            float inc = s;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xFFFFFFFFu, inc, o);
                if (lane >= o) inc += v;
            }
            const float before = inc - s;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                bar.la[k & 1][lane * 4 + e] = before + a[e];
                bar.dt[k & 1][lane * 4 + e] = d[e];
            }
            mbar_arrive(&bar.dt_ready);
        };
        // the state row of this thread (32 columns) as operand of the next C S, and scaled by the next chunk's decay in TMEM
        auto publish = [&](uint32_t (&s)[32], float decay) {
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                uint4 hi, lo;
                split_hi_lo(__uint_as_float(s[c * 8]), __uint_as_float(s[c * 8 + 1]), hi.x, lo.x);
                split_hi_lo(__uint_as_float(s[c * 8 + 2]), __uint_as_float(s[c * 8 + 3]), hi.y, lo.y);
                split_hi_lo(__uint_as_float(s[c * 8 + 4]), __uint_as_float(s[c * 8 + 5]), hi.z, lo.z);
                split_hi_lo(__uint_as_float(s[c * 8 + 6]), __uint_as_float(s[c * 8 + 7]), hi.w, lo.w);
                const int at = r * 128 + (((half * 4 + c) ^ (r & 7)) << 4);
                *reinterpret_cast<uint4*>(ss + at) = hi;
                *reinterpret_cast<uint4*>(ss + kBox + at) = lo;
            }
#pragma unroll
            for (int i = 0; i < 32; ++i) s[i] = __float_as_uint(__uint_as_float(s[i]) * decay);
            tmem_st32(t_s + lane_base + col0, s);
            tmem_st_wait();
            tc_fence_before();
            fence_proxy_async_smem();
            mbar_arrive(&bar.s_ready);
        };
        if (warp == 0) { fetch_dt(0); scan_dt(0); }
        bool ok = mbar_wait_warp(&bar.dt_ready, 0, ctx, 0xDD);
        if (ok) {
            uint32_t s[32];
            const float* src = p.n_seg > 1 ? p.seg_state + ((static_cast<long long>(b) * p.n_seg + seg) * p.H + h) * p.N * p.Pp + static_cast<long long>(r) * p.Pp
                                           : (p.pos[b] > 0 ? p.state + state_row : nullptr);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                float v[8] = {};
                if (src != nullptr && r < p.N && col0 + c * 8 < p.P) load8(src + col0 + c * 8, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) s[c * 8 + e] = __float_as_uint(v[e]);
            }
            publish(s, fast_exp2(bar.la[0][kL - 1]));
        }
        for (int k = 0; k < n_chunk && ok; ++k) {
            const int q = k & 1, ph = k & 1, t0 = (c_begin + k) * kL, tn = min(kL, p.T - t0);
            const long long m = static_cast<long long>(b) * p.T + t0 + r;
            const float *la = bar.la[q], *dt = bar.dt[q];
            const bool more = k + 1 < n_chunk;
            uint4 z[4];
#pragma unroll
            for (int c = 0; c < 4; ++c)
                z[c] = r < tn && col0 + c * 8 < p.P ? *reinterpret_cast<const uint4*>(p.proj + m * p.ldp + h * p.P + col0 + c * 8) : make_uint4(0, 0, 0, 0);
            if (warp == 0 && more) fetch_dt(k + 1);
            ok = mbar_wait_warp(&bar.tiles_full[q], (k / 2) & 1, ctx, 0xD8);
            if (!ok) break;
            // ---- w x: token r, this half's columns.  (The last update has read the previous one: its completion was awaited.) ----
            const uint8_t* xt = smem + q * kStage + 4 * kBox;
            uint4 xv[4];
            const float lar = la[r], wr = dt[r] * fast_exp2(la[kL - 1] - lar);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int at = r * 128 + (((half * 4 + c) ^ (r & 7)) << 4);
                xv[c] = *reinterpret_cast<const uint4*>(xt + at);
                uint4 hi, lo;
                float2 f = Elem<__nv_bfloat16>::unpack2(xv[c].x);
                split_hi_lo(f.x * wr, f.y * wr, hi.x, lo.x);
                f = Elem<__nv_bfloat16>::unpack2(xv[c].y);
                split_hi_lo(f.x * wr, f.y * wr, hi.y, lo.y);
                f = Elem<__nv_bfloat16>::unpack2(xv[c].z);
                split_hi_lo(f.x * wr, f.y * wr, hi.z, lo.z);
                f = Elem<__nv_bfloat16>::unpack2(xv[c].w);
                split_hi_lo(f.x * wr, f.y * wr, hi.w, lo.w);
                *reinterpret_cast<uint4*>(xw + at) = hi;
                *reinterpret_cast<uint4*>(xw + kBox + at) = lo;
            }
            fence_proxy_async_smem();
            mbar_arrive(&bar.xw_ready);
            mbar_arrive(&bar.tiles_empty[q]);        // this thread reads the tiles no more (the products' part is the commit)
            // ---- M: row r of G, 64 columns ----
            ok = mbar_wait_warp(&bar.g_full, ph, ctx, 0xD9);
            if (!ok) break;
            tc_fence_after();
#pragma unroll
            for (int cc = 0; cc < 2; ++cc) {
                const int j0 = half * 64 + cc * 32;
                uint32_t hi[16], lo[16];
                if (j0 > (warp & 3) * 32 + 31) {     // every column lies after every row of this warp
#pragma unroll
                    for (int i = 0; i < 16; ++i) { hi[i] = 0u; lo[i] = 0u; }
                } else {
                    uint32_t gv[32];
                    tmem_ld32(tmem + lane_base + j0, gv);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; i += 4) {
                        const float4 l4 = *reinterpret_cast<const float4*>(la + j0 + i), d4 = *reinterpret_cast<const float4*>(dt + j0 + i);
                        const float w0 = j0 + i <= r ? __uint_as_float(gv[i]) * (fast_exp2(lar - l4.x) * d4.x) : 0.f;
                        const float w1 = j0 + i + 1 <= r ? __uint_as_float(gv[i + 1]) * (fast_exp2(lar - l4.y) * d4.y) : 0.f;
                        const float w2 = j0 + i + 2 <= r ? __uint_as_float(gv[i + 2]) * (fast_exp2(lar - l4.z) * d4.z) : 0.f;
                        const float w3 = j0 + i + 3 <= r ? __uint_as_float(gv[i + 3]) * (fast_exp2(lar - l4.w) * d4.w) : 0.f;
                        split_hi_lo(w0, w1, hi[i / 2], lo[i / 2]);
                        split_hi_lo(w2, w3, hi[i / 2 + 1], lo[i / 2 + 1]);
                    }
                }
                tmem_st16(t_m + lane_base + j0 / 2, hi);
                tmem_st16(t_m + lane_base + 64 + j0 / 2, lo);
            }
            // ---- 2^la C S ----
            ok = mbar_wait_warp(&bar.cs_full, ph, ctx, 0xDA);
            if (!ok) break;
            tc_fence_after();
            {
                uint32_t y[32];
                const float e = fast_exp2(lar);
                tmem_ld32(t_y + lane_base + col0, y);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) y[i] = __float_as_uint(__uint_as_float(y[i]) * e);
                tmem_st32(t_y + lane_base + col0, y);
            }
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(&bar.p_ready);
            // ---- the state after this chunk.  (C S of this chunk is complete, so every thread has left the chunk before:
            // the other set of step sizes is free.) ----
            if (more) {
                if (warp == 0) scan_dt(k + 1);
                ok = mbar_wait_warp(&bar.dt_ready, (k + 1) & 1, ctx, 0xDE);
                if (!ok) break;
            }
            ok = mbar_wait_warp(&bar.u_full, ph, ctx, 0xDB);
            if (!ok) break;
            tc_fence_after();
            {
                uint32_t s[32];
                tmem_ld32(t_s + lane_base + col0, s);
                tmem_ld_wait();
                if (more) publish(s, fast_exp2(bar.la[q ^ 1][kL - 1]));
                else if (seg + 1 == p.n_seg && r < p.N) {
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        float v[8];
#pragma unroll
                        for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(s[c * 8 + e]);
                        if (col0 + c * 8 < p.P) store8(p.state + state_row + col0 + c * 8, v);
                    }
                }
            }
            // ---- outputs ----
            ok = mbar_wait_warp(&bar.y_full, ph, ctx, 0xDC);
            if (!ok) break;
            tc_fence_after();
            uint32_t y[32];
            tmem_ld32(t_y + lane_base + col0, y);
            tmem_ld_wait();
            tc_fence_before();
            mbar_arrive(&bar.y_free);
            if (r < tn) {
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    if (col0 + c * 8 >= p.P) break;
                    const uint32_t xs[4] = {xv[c].x, xv[c].y, xv[c].z, xv[c].w}, zs[4] = {z[c].x, z[c].y, z[c].z, z[c].w};
                    float v[8];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float2 xf = Elem<__nv_bfloat16>::unpack2(xs[e]), zf = Elem<__nv_bfloat16>::unpack2(zs[e]);
                        v[2 * e] = fmaf(Dh, xf.x, __uint_as_float(y[c * 8 + 2 * e])) * silu_for<__nv_bfloat16>(zf.x);
                        v[2 * e + 1] = fmaf(Dh, xf.y, __uint_as_float(y[c * 8 + 2 * e + 1])) * silu_for<__nv_bfloat16>(zf.y);
                    }
                    store8(p.gated + m * inner + h * p.P + col0 + c * 8, v);
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 9) tmem_dealloc(tmem, 512);
    abort_linger(&bar.abort_flag);
}

}  // namespace

bool ssd_walk_supported(const vb200_ssd_args& a) {
    return ssd_chunk_supported(a) && a.P <= 64 && a.N <= 128 && a.T >= 96 && a.B <= 65535 && a.H <= 65535;
}

int launch_ssd_walk(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, const void* xbc, void* gated, const float* seg_state, int n_seg, int seg_chunks64, int* status) {
    const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(xbc);
    const long long ch = pl.channels, batch = ch * a.T, inner = static_cast<long long>(a.H) * a.P;
    WalkMaps maps;
    if (int rc = make_map_4d(&maps.x, base, a.P, a.H, a.T, a.B, a.P, ch, batch, kL)) return rc;
    if (int rc = make_map_4d(&maps.b, base + inner, a.N, a.G, a.T, a.B, a.N, ch, batch, kL)) return rc;
    if (int rc = make_map_4d(&maps.c, base + inner + static_cast<long long>(a.G) * a.N, a.N, a.G, a.T, a.B, a.N, ch, batch, kL)) return rc;
    WalkParams p{};
    p.T = a.T; p.H = a.H; p.P = a.P; p.N = a.N; p.G = a.G; p.Pp = pl.Pp; p.nk = (a.N + 15) / 16;
    p.n_seg = n_seg; p.seg_chunks = n_seg > 1 ? seg_chunks64 / 2 : (a.T + kL - 1) / kL;
    p.ldp = a.ldp; p.proj = static_cast<const __nv_bfloat16*>(a.proj);
    p.dt_bias = a.dt_bias; p.A_log = a.A_log; p.D = a.D; p.slots = a.slots; p.pos = a.pos;
    p.state = a.state; p.seg_state = seg_state; p.gated = static_cast<__nv_bfloat16*>(gated); p.status = status;
    if (int rc = allow_smem(ssd_walk_sm100_kernel, kSmem)) return rc;
    note_ssd_kernel("ssd_walk_sm100_kernel");
    return launch_pdl(ssd_walk_sm100_kernel, dim3(static_cast<unsigned>(n_seg), static_cast<unsigned>(a.H), static_cast<unsigned>(a.B)), dim3(kThreads), kSmem, s, maps, p);
}

}  // namespace vb200
