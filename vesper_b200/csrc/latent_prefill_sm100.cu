// Prompt attention of latent-attention layers on sm_100a: causal with a sliding window, keys of two parts (per-head
// columns expanded from the latents, and one rotated part shared by all heads), a per-head sink in the denominator.
//
//   s_ij = scale * (qn_i . kn_j + qr_i . kr_j),   visible iff 0 <= i - j < window
//   O_i  = sum_j exp(s_ij) v_j / (exp(sink) + sum_j exp(s_ij))
//
// One CTA per 128 query rows of one (batch, head), two CTAs per SM so that one computes products while the other is in
// its softmax.  The context is walked in blocks of 64 keys, from the first block the window of the tile's first row
// reaches to the tile's last own key.
//   warps 0-3  softmax, correction, epilogue: one thread per query row = TMEM lane
//   warp  4    TMA producer: Q once (both parts), rings of K blocks (both parts) and V blocks, 128-byte swizzle
//   warp  5    tcgen05.mma issuer, TMEM owner
// TMEM (256 columns): S0 [0,64) S1 [64,128) O [128, 128 + vdim).  QK of block j+1 is issued before PV of block j.
// The weights stay fp32-class in the second product: P = hi + lo, both bf16, packed over their S (hi in its first 32
// columns, lo in the other 32), two MMAs per 16 keys.  The sink enters as the initial state of the online softmax
// (reference maximum = sink, sum = 1), so no key and no value belong to it.
// Head sizes are runtime values: the 64-column boxes zero-fill past a part's width.
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kRows = 128;            // query rows per CTA
constexpr int kKeys = 64;             // keys per block
constexpr int kQBox = kRows * 128;    // one [rows x 64 columns] box
constexpr int kKBox = kKeys * 128;
constexpr int kMaxStages = 4;
constexpr int kThreads = 192;
constexpr float kGrow = 8.0f;         // rescale O only when a row maximum grows by more than 2^8

struct LatentMaps { CUtensorMap qn, qr, kn, kr, v; };

struct LatentTileParams {
    int T, n_ctx, window, vdim;
    int ks_n, ks_r;                   // 16-column steps of the two key parts
    int nb_n, nb_r, nb_v;             // 64-column boxes
    int n_pv;                         // columns of the PV product
    int k_stages, v_stages;
    float scale_log2;
    const float* sink;
    __nv_bfloat16* out;
    long long ldo;
    int* status;
};

struct LatentBars {
    uint64_t q_full, k_full[kMaxStages], k_empty[kMaxStages], v_full[kMaxStages], v_empty[kMaxStages], s_full[2], p_ready[2], o_done[2], drain;
    uint32_t tmem;
    int abort_flag;
};

__global__ void __launch_bounds__(kThreads, 2)
latent_prefill_sm100_kernel(const __grid_constant__ LatentMaps maps, LatentTileParams p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ LatentBars bar;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r0 = static_cast<int>(gridDim.z - 1 - blockIdx.z) * kRows, h = blockIdx.x, b = blockIdx.y;      // tiles with most keys first
    const int n_old = p.n_ctx - p.T;
    const int first_lo = max(0, n_old + r0 - p.window + 1);
    const int last_key = min(n_old + r0 + kRows - 1, p.n_ctx - 1);
    const int blk0 = first_lo / kKeys, n_blk = last_key / kKeys - blk0 + 1;
    const int nb_k = p.nb_n + p.nb_r;
    uint8_t* q_smem = smem;
    uint8_t* k_smem = q_smem + nb_k * kQBox;
    uint8_t* v_smem = k_smem + p.k_stages * nb_k * kKBox;
    const WaitCtx ctx{&bar.abort_flag, p.status};

    if (threadIdx.x == 0) {
        bar.abort_flag = 0;
        mbar_init(&bar.q_full, 1);
        for (int i = 0; i < kMaxStages; ++i) { mbar_init(&bar.k_full[i], 1); mbar_init(&bar.k_empty[i], 1); mbar_init(&bar.v_full[i], 1); mbar_init(&bar.v_empty[i], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&bar.s_full[i], 1); mbar_init(&bar.p_ready[i], kRows); mbar_init(&bar.o_done[i], 1); }
        mbar_init(&bar.drain, 1);
        mbar_fence_init();
        if ((smem_u32(smem) & 1023) != 0) { bar.abort_flag = 1; atomicCAS(p.status, 0, (3 << 24) | 0x2); }      // the swizzle needs 1024-byte tiles
    }
    if (warp == 5) { tmem_alloc(&bar.tmem, 256); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bar.tmem;
    const bool dead = *static_cast<volatile int*>(&bar.abort_flag) != 0;
    pdl_begin();

    if (dead) {
    } else if (warp == 4) {
        if (lane == 0) {
            mbar_arrive_expect_tx(&bar.q_full, nb_k * kQBox);
            for (int i = 0; i < p.nb_n; ++i) tma_load_4d(q_smem + i * kQBox, &maps.qn, &bar.q_full, i * 64, h, r0, b);
            for (int i = 0; i < p.nb_r; ++i) tma_load_4d(q_smem + (p.nb_n + i) * kQBox, &maps.qr, &bar.q_full, i * 64, h, r0, b);
            bool ok = true;
            auto load_k = [&](int j) {
                const int s = j % p.k_stages;
                if (j >= p.k_stages) ok = mbar_wait(&bar.k_empty[s], (j / p.k_stages - 1) & 1, ctx, 0xB1);
                if (!ok) return;
                uint8_t* st = k_smem + s * nb_k * kKBox;
                mbar_arrive_expect_tx(&bar.k_full[s], nb_k * kKBox);
                for (int i = 0; i < p.nb_n; ++i) tma_load_4d(st + i * kKBox, &maps.kn, &bar.k_full[s], i * 64, h, (blk0 + j) * kKeys, b);
                for (int i = 0; i < p.nb_r; ++i) tma_load_4d(st + (p.nb_n + i) * kKBox, &maps.kr, &bar.k_full[s], i * 64, 0, (blk0 + j) * kKeys, b);
            };
            load_k(0);
            for (int j = 0; j < n_blk && ok; ++j) {
                if (j + 1 < n_blk) load_k(j + 1);
                if (!ok) break;
                const int s = j % p.v_stages;
                if (j >= p.v_stages) ok = mbar_wait(&bar.v_empty[s], (j / p.v_stages - 1) & 1, ctx, 0xB2);
                if (!ok) break;
                mbar_arrive_expect_tx(&bar.v_full[s], p.nb_v * kKBox);
                for (int i = 0; i < p.nb_v; ++i) tma_load_4d(v_smem + (s * p.nb_v + i) * kKBox, &maps.v, &bar.v_full[s], i * 64, h, (blk0 + j) * kKeys, b);
            }
        }
    } else if (warp == 5) {
        if (lane == 0) {
            const uint32_t idesc_qk = make_idesc_f16(1, 0, 0, kRows, kKeys);
            const uint32_t idesc_pv = make_idesc_f16(1, 0, 1, kRows, p.n_pv);
            const uint32_t q_addr = smem_u32(q_smem), k_addr = smem_u32(k_smem), v_addr = smem_u32(v_smem);
            bool ok = mbar_wait(&bar.q_full, 0, ctx, 0xB3);
            auto issue_qk = [&](int j) {
                const int s = j % p.k_stages;
                ok = mbar_wait(&bar.k_full[s], (j / p.k_stages) & 1, ctx, 0xB4);
                if (!ok) return;
                tc_fence_after();
                const uint32_t kb = k_addr + s * nb_k * kKBox, d = tmem + (j & 1) * kKeys;
                for (int kk = 0; kk < p.ks_n + p.ks_r; ++kk) {
                    const int box = kk < p.ks_n ? kk >> 2 : p.nb_n + ((kk - p.ks_n) >> 2), off = (kk < p.ks_n ? kk & 3 : (kk - p.ks_n) & 3) * 32;
                    umma_ss(d, make_smem_desc_sw128(q_addr + box * kQBox + off, 16, 1024), make_smem_desc_sw128(kb + box * kKBox + off, 16, 1024), idesc_qk, kk > 0 ? 1u : 0u);
                }
                umma_commit(&bar.s_full[j & 1]);
                umma_commit(&bar.k_empty[s]);
            };
            if (ok) issue_qk(0);
            for (int j = 0; j < n_blk && ok; ++j) {
                if (j + 1 < n_blk) issue_qk(j + 1);      // its S held P of block j-1, whose product was issued before
                if (!ok) break;
                const int s = j % p.v_stages;
                ok = mbar_wait(&bar.v_full[s], (j / p.v_stages) & 1, ctx, 0xB5) && mbar_wait(&bar.p_ready[j & 1], (j >> 1) & 1, ctx, 0xB6);
                if (!ok) break;
                tc_fence_after();
                const uint32_t vb = v_addr + s * p.nb_v * kKBox, a = tmem + (j & 1) * kKeys;
                for (int half = 0; half < 2; ++half)
                    for (int kk = 0; kk < kKeys / 16; ++kk)
                        umma_ts(tmem + 2 * kKeys, a + half * 32 + kk * 8, make_smem_desc_sw128(vb + kk * 2048, kKBox, 1024), idesc_pv, (j | half | kk) ? 1u : 0u);
                umma_commit(&bar.o_done[j & 1]);
                umma_commit(&bar.v_empty[s]);
            }
            umma_commit(&bar.drain);                     // nothing may be in flight when TMEM is freed
            mbar_wait(&bar.drain, 0, ctx, 0xB7);
        }
    } else {
        const int r = threadIdx.x;                       // row of the tile = TMEM lane
        const uint32_t lane_base = static_cast<uint32_t>(warp * 32) << 16, o_addr = tmem + lane_base + 2 * kKeys;
        const int me = n_old + r0 + r, lo = me - p.window + 1;
        float m_ref = -1e30f, l_sum = 0.f;
        if (p.sink != nullptr) { m_ref = p.sink[h] * kLog2e; l_sum = 1.f; }
        bool ok = true;
        for (int j = 0; j < n_blk; ++j) {
            ok = mbar_wait_warp(&bar.s_full[j & 1], (j >> 1) & 1, ctx, 0xB8);
            if (!ok) break;
            tc_fence_after();
            const uint32_t s_addr = tmem + lane_base + (j & 1) * kKeys;
            uint32_t s[2][32];
            tmem_ld32(s_addr, s[0]);
            tmem_ld32(s_addr + 32, s[1]);
            tmem_ld_wait();
            const int k0 = (blk0 + j) * kKeys;
            if (k0 + kKeys - 1 > n_old + r0 || k0 < n_old + r0 + kRows - p.window) {
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        const int k = k0 + c * 32 + i;
                        if (k > me || k < lo) s[c][i] = 0xFF800000u;     // -inf
                    }
            }
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int i = 0; i < 32; i += 2) mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], __uint_as_float(s[c][i]), __uint_as_float(s[c][i + 1]));
            const float m_cand = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
            const bool grow = m_cand > m_ref + kGrow;
            if (__any_sync(0xFFFFFFFFu, grow)) {
                const float m_new = grow ? m_cand : m_ref;
                const float alpha = fast_exp2(m_ref - m_new);
                if (j > 0) {
                    ok = mbar_wait_warp(&bar.o_done[(j - 1) & 1], ((j - 1) >> 1) & 1, ctx, 0xB9);
                    if (!ok) break;
                    tc_fence_after();
                    for (int c = 0; c < p.n_pv; c += 32) {
                        uint32_t o[32];
                        tmem_ld32(o_addr + c, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                        tmem_st32(o_addr + c, o);
                    }
                    tmem_st_wait();
                }
                l_sum *= alpha;
                m_ref = m_new;
            }
            float2 rs[2] = {{0.f, 0.f}, {0.f, 0.f}};
            const float2 sc2 = make_float2(p.scale_log2, p.scale_log2), nm2 = make_float2(-m_ref, -m_ref);
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                uint32_t hi[16], lo16[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float2 e = __ffma2_rn(make_float2(__uint_as_float(s[c][2 * i]), __uint_as_float(s[c][2 * i + 1])), sc2, nm2);
                    const float2 pp = make_float2(fast_exp2(e.x), fast_exp2(e.y));
                    rs[i & 1] = __fadd2_rn(rs[i & 1], pp);
                    split_hi_lo(pp.x, pp.y, hi[i], lo16[i]);
                }
                tmem_st16(s_addr + c * 16, hi);
                tmem_st16(s_addr + 32 + c * 16, lo16);
            }
            l_sum += (rs[0].x + rs[0].y) + (rs[1].x + rs[1].y);
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(&bar.p_ready[j & 1]);
        }
        if (ok) ok = mbar_wait_warp(&bar.o_done[(n_blk - 1) & 1], ((n_blk - 1) >> 1) & 1, ctx, 0xBA);
        if (ok) {
            tc_fence_after();
            const float inv = 1.0f / l_sum;
            __nv_bfloat16* orow = p.out + (static_cast<long long>(b) * p.T + r0 + r) * p.ldo + static_cast<long long>(h) * p.vdim;
            for (int c = 0; c < p.vdim; c += 32) {
                uint32_t o[32];
                tmem_ld32(o_addr + c, o);
                tmem_ld_wait();
                if (r0 + r < p.T) {
#pragma unroll
                    for (int v = 0; v < 4; ++v) {
                        if (c + v * 8 >= p.vdim) break;
                        float f[8];
#pragma unroll
                        for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[v * 8 + e]) * inv;
                        store8(orow + c + v * 8, f);
                    }
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 5) tmem_dealloc(tmem, 256);
    abort_linger(&bar.abort_flag);
}

}  // namespace

bool latent_sm100_supported(const vb200_latent_args& a) {
    return a.dtype == VB200_BF16 && a.dim % 8 == 0 && a.rot_dim % 8 == 0 && a.rot_dim > 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.rot_dim <= 64 && a.vdim <= 128 &&
           a.scale > 0.f && a.T <= 65535 * kRows && a.ldp % 8 == 0 && a.ldkv % 8 == 0 && a.ldo % 8 == 0 && reinterpret_cast<uintptr_t>(a.ctx_kv) % 16 == 0 &&
           reinterpret_cast<uintptr_t>(a.ctx_latent) % 16 == 0 && reinterpret_cast<uintptr_t>(a.out) % 16 == 0;
}

int launch_latent_prefill_sm100(cudaStream_t s, const vb200_latent_args& a, int* status) {
    const int n_ctx = vb200_latent_context(a.start_pos, a.T, a.window);
    const int hq = a.dim + a.rot_dim;
    const __nv_bfloat16 *q = static_cast<const __nv_bfloat16*>(a.proj), *kv = static_cast<const __nv_bfloat16*>(a.ctx_kv), *lat = static_cast<const __nv_bfloat16*>(a.ctx_latent);
    LatentMaps maps;
    if (int rc = make_map_4d(&maps.qn, q, a.dim, a.H, a.T, a.B, hq, a.ldp, a.ldp * a.T, kRows)) return rc;
    if (int rc = make_map_4d(&maps.qr, q + a.dim, a.rot_dim, a.H, a.T, a.B, hq, a.ldp, a.ldp * a.T, kRows)) return rc;
    if (int rc = make_map_4d(&maps.kn, kv, a.dim, a.H, n_ctx, a.B, a.dim, a.ldkv, a.ldkv * n_ctx, kKeys)) return rc;
    if (int rc = make_map_4d(&maps.kr, lat + vb200_latent_rot_offset(a.rank), a.rot_dim, 1, n_ctx, a.B, a.rot_dim, a.ldc, a.ldc * n_ctx, kKeys)) return rc;
    if (int rc = make_map_4d(&maps.v, kv + static_cast<long long>(a.H) * a.dim, a.vdim, a.H, n_ctx, a.B, a.vdim, a.ldkv, a.ldkv * n_ctx, kKeys)) return rc;
    LatentTileParams p{};
    p.T = a.T; p.n_ctx = n_ctx; p.window = a.window; p.vdim = a.vdim;
    p.ks_n = (a.dim + 15) / 16; p.ks_r = (a.rot_dim + 15) / 16;
    p.nb_n = (a.dim + 63) / 64; p.nb_r = (a.rot_dim + 63) / 64; p.nb_v = (a.vdim + 63) / 64;
    p.n_pv = pad_to(a.vdim, 16);
    p.scale_log2 = a.scale * kLog2e;
    p.sink = a.sink; p.out = static_cast<__nv_bfloat16*>(a.out); p.ldo = a.ldo; p.status = status;
    // ring depths: what fits beside Q with two CTAs on an SM (228 KB, 1 KB reserved per CTA, barriers static)
    const int nb_k = p.nb_n + p.nb_r, budget = 112 * 1024 - nb_k * kQBox;
    p.k_stages = 1; p.v_stages = 1;
    auto used = [&] { return (p.k_stages * nb_k + p.v_stages * p.nb_v) * kKBox; };
    for (bool grew = true; grew;) {
        grew = false;
        if (p.k_stages < kMaxStages && p.k_stages <= p.v_stages) { ++p.k_stages; if (used() <= budget) grew = true; else --p.k_stages; }
        if (p.v_stages < kMaxStages && p.v_stages < p.k_stages) { ++p.v_stages; if (used() <= budget) grew = true; else --p.v_stages; }
    }
    size_t smem = static_cast<size_t>(nb_k) * kQBox + used();
    if (smem < 80 * 1024) smem = 80 * 1024;          // never a third CTA on an SM: it would find no TMEM
    if (int rc = allow_smem(latent_prefill_sm100_kernel, smem)) return rc;
    return launch_pdl(latent_prefill_sm100_kernel, dim3(static_cast<unsigned>(a.H), static_cast<unsigned>(a.B), static_cast<unsigned>((a.T + kRows - 1) / kRows)), dim3(kThreads),
                      smem, s, maps, p);
}

}  // namespace vb200
