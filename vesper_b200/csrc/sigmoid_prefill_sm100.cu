// Prompt attention of sigmoid-attention layers on sm_100a.
//
//   O_i[h] = gate * sum_{j <= i} sigmoid(s_ij) v_j[group of h],   s_ij = q'_i[h] . k_j + bias[h, min(i - j, last)]
//
// q' holds the mixed queries of a head against the concatenated keys of all groups (kd = G * dim columns), already times -log2(e):
// sigmoid(s) = 1 / (1 + 2^(s')).  Weights are not normalised, so there is no running maximum, no correction of O, and two warps
// can share a row: nothing has to be reduced over keys.
//
// One CTA per 128 query rows of one (batch, head), one CTA per SM; keys in blocks of 128.  The key rows are as wide as all groups
// together, so with one tile per CTA they come from L2 faster than it delivers; where two neighbouring heads share their values (PAIR), the
// CTAs of the two heads form a cluster that runs every product as one tcgen05.mma.cta_group::2 of 256 rows, and each loads half of the keys
// (64 of a block's 128) and half of the value columns.  The cluster's rank 0 issues the products; its barriers collect both CTAs' copies
// and arrivals, its commits go to both.
//   warps 0-7  weights and epilogue: warps w and w + 4 own the same 32 rows (TMEM lanes), and 64 keys of a block each
//   warp  8    TMA producer: Q once, then a ring of K stages (a few boxes of 64 columns) and one of V blocks
//   warp  9    tcgen05.mma issuer, TMEM owner
// TMEM (512 columns): S0 [0, 128) S1 [128, 256) O [256, 256 + vdim).  QK of block j+1 is issued before PV of block j.  The weights stay
// fp32-class in the second product: each half of a block is packed over its own 64 columns of S as bf16 hi (32 columns) and lo (32).
// Two elements share one reciprocal: 1/a = b * (1/(ab)); 2^(s') is cut at 2^60, which leaves a weight below 1e-18.
#include "cluster_pair.cuh"
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kRows = 128, kKeys = 128;
constexpr int kBox = 128 * 128;               // [128 rows x 64 columns]
constexpr int kMaxStages = 8;
constexpr int kBoxesPerSm = 14;               // of 16 KB: Q, K ring and V ring of the one CTA
constexpr int kWeightThreads = 256;
constexpr int kThreads = kWeightThreads + 64;
constexpr float kCut = 60.0f;

struct SigMaps { CUtensorMap q, k, v; };

struct SigTileParams {
    int T, start_pos, vdim, R, n_bias, gate_col;
    int nb_k, nb_v, n_pv;                     // 64-column boxes of a key and a value row, columns of the second product
    int kbs, k_stages, v_stages;              // boxes per K stage, ring depths
    int v_half;                               // PAIR: value columns of one CTA
    const float* bias;
    const __nv_bfloat16* proj;
    __nv_bfloat16* out;
    long long ldp, ldo;
    const int* slots;
    int* status;
};

struct SigBars {
    uint64_t q_full[kMaxStages], k_full[kMaxStages], k_empty[kMaxStages], v_full[kMaxStages], v_empty[kMaxStages], s_full[2], p_ready[2], o_done, drain;
    uint32_t tmem;
    int abort_flag;
};

__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <bool PAIR>
__global__ void __launch_bounds__(kThreads, 1)
sig_prefill_sm100_kernel(const __grid_constant__ SigMaps maps, SigTileParams p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ SigBars bar;
    constexpr int kKBox = PAIR ? kBox / 2 : kBox;         // this CTA's keys of a block x 64 columns
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r0 = static_cast<int>(gridDim.z - 1 - blockIdx.z) * kRows, h = blockIdx.x, b = blockIdx.y;      // tiles with most keys first
    const int cta = PAIR ? static_cast<int>(cluster_ctarank()) : 0;
    const int last_key = p.start_pos + min(r0 + kRows, p.T) - 1, n_blk = last_key / kKeys + 1;
    uint8_t* q_smem = smem;
    uint8_t* k_ring = q_smem + p.nb_k * kBox;
    uint8_t* v_ring = k_ring + p.k_stages * p.kbs * kKBox;
    const WaitCtx ctx{&bar.abort_flag, p.status};
    // copies credit the issuing CTA's barrier, commits go to both CTAs
    auto load = [&](void* dst, const CUtensorMap* m, uint64_t* full, int c0, int c1, int c2, int c3) {
        if constexpr (PAIR) tma_load_4d_pair(dst, m, map_to_cta(smem_u32(full), 0), c0, c1, c2, c3);
        else tma_load_4d(dst, m, full, c0, c1, c2, c3);
    };
    auto expect = [&](uint64_t* full, int bytes) {
        if (cta == 0) mbar_arrive_expect_tx(full, PAIR ? 2 * bytes : bytes);
    };
    auto commit = [&](uint64_t* to) {
        if constexpr (PAIR) umma2_commit(to);
        else umma_commit(to);
    };

    if (threadIdx.x == 0) {
        bar.abort_flag = 0;
        for (int i = 0; i < kMaxStages; ++i) {
            mbar_init(&bar.q_full[i], 1);
            mbar_init(&bar.k_full[i], 1); mbar_init(&bar.k_empty[i], 1); mbar_init(&bar.v_full[i], 1); mbar_init(&bar.v_empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) { mbar_init(&bar.s_full[i], 1); mbar_init(&bar.p_ready[i], (PAIR ? 2 : 1) * kWeightThreads / 32); }
        mbar_init(&bar.o_done, 1);
        mbar_init(&bar.drain, 1);
        mbar_fence_init();
        if ((smem_u32(smem) & 1023) != 0) { bar.abort_flag = 1; atomicCAS(p.status, 0, (3 << 24) | 0x3); }      // the swizzle needs 1024-byte tiles
    }
    if (warp == 9) {
        __syncwarp();
        if constexpr (PAIR) { tmem_alloc2(&bar.tmem, 512); tmem_relinquish2(); }
        else { tmem_alloc(&bar.tmem, 512); tmem_relinquish(); }
    }
    tc_fence_before();
    __syncthreads();
    if constexpr (PAIR) { cluster_arrive(); cluster_wait(); }        // both CTAs' barriers exist before anything crosses the pair
    tc_fence_after();
    const uint32_t tmem = bar.tmem;
    const bool dead = *static_cast<volatile int*>(&bar.abort_flag) != 0;
    pdl_begin();

    if (dead) {
    } else if (warp == 8) {
        if (lane == 0) {
            const int slot = p.slots ? p.slots[b] : b;
            bool ok = true;
            int ks = 0, vs = 0;
            uint32_t k_phase = 1, v_phase = 1;           // parity 1: the first round finds every stage free
            auto load_k = [&](int j) {
                for (int i = 0; i < p.nb_k; i += p.kbs) {
                    if (j == 0) {                        // the queries come along with the first block's keys, stage by stage
                        uint64_t* full = &bar.q_full[i / p.kbs];
                        expect(full, p.kbs * kBox);
                        for (int x = 0; x < p.kbs; ++x) load(q_smem + (i + x) * kBox, &maps.q, full, (i + x) * 64, h, r0, b);
                    }
                    ok = mbar_wait(&bar.k_empty[ks], k_phase, ctx, 0xD1);
                    if (!ok) return;
                    expect(&bar.k_full[ks], p.kbs * kKBox);
                    for (int x = 0; x < p.kbs; ++x) load(k_ring + (ks * p.kbs + x) * kKBox, &maps.k, &bar.k_full[ks], (i + x) * 64, 0, j * kKeys + 64 * cta, slot);
                    if (++ks == p.k_stages) { ks = 0; k_phase ^= 1; }
                }
            };
            load_k(0);
            for (int j = 0; j < n_blk && ok; ++j) {
                if (j + 1 < n_blk) load_k(j + 1);
                if (!ok) break;
                ok = mbar_wait(&bar.v_empty[vs], v_phase, ctx, 0xD8);
                if (!ok) break;
                expect(&bar.v_full[vs], p.nb_v * kBox);
                for (int i = 0; i < p.nb_v; ++i) load(v_ring + (vs * p.nb_v + i) * kBox, &maps.v, &bar.v_full[vs], PAIR ? p.v_half * cta : i * 64, h / p.R, j * kKeys, slot);
                if (++vs == p.v_stages) { vs = 0; v_phase ^= 1; }
            }
        }
    } else if (warp == 9) {
        if (lane == 0 && cta == 0) {
            constexpr int kM = PAIR ? 2 * kRows : kRows;
            const uint32_t idesc_qk = make_idesc_f16(1, 0, 0, kM, kKeys);
            const uint32_t idesc_pv = make_idesc_f16(1, 0, 1, kM, p.n_pv);
            // what this one thread executes between two products is what holds the tensor pipe up: descriptors are built once (only the
            // start address, in units of 16 bytes, moves), stages and parities are counted, the steps of a box are unrolled.  Columns
            // past kd are zero in both operands, so every box takes its four steps.
            const uint64_t q_desc = make_smem_desc_sw128(smem_u32(q_smem), 16, 1024), k_desc = make_smem_desc_sw128(smem_u32(k_ring), 16, 1024);
            const uint64_t v_desc = make_smem_desc_sw128(smem_u32(v_ring), kBox, 1024);
            const uint32_t k_stage16 = p.kbs * (kKBox >> 4), v_stage16 = p.nb_v * (kBox >> 4);
            bool ok = true;
            int ks = 0, vs = 0;
            uint32_t k_phase = 0, v_phase = 0;
            auto issue_qk = [&](int j) {
                const uint32_t d = tmem + (j & 1) * kKeys;
                uint64_t qd = q_desc;
                uint32_t acc = 0;
                for (int i = 0; i < p.nb_k; i += p.kbs) {
                    if (j == 0) ok = mbar_wait(&bar.q_full[i / p.kbs], 0, ctx, 0xD2);
                    ok = ok && mbar_wait(&bar.k_full[ks], k_phase, ctx, 0xD3);
                    if (!ok) return;
                    tc_fence_after();
                    uint64_t kd = k_desc + ks * k_stage16;
                    for (int x = 0; x < p.kbs; ++x) {
#pragma unroll
                        for (int kk = 0; kk < 4; ++kk) {
                            if constexpr (PAIR) umma2_ss(d, qd + 2 * kk, kd + 2 * kk, idesc_qk, kk > 0 ? 1u : acc);
                            else umma_ss(d, qd + 2 * kk, kd + 2 * kk, idesc_qk, kk > 0 ? 1u : acc);
                        }
                        acc = 1;
                        qd += kBox >> 4;
                        kd += kKBox >> 4;
                    }
                    commit(&bar.k_empty[ks]);
                    if (++ks == p.k_stages) { ks = 0; k_phase ^= 1; }
                }
                commit(&bar.s_full[j & 1]);
            };
            if (ok) issue_qk(0);
            for (int j = 0; j < n_blk && ok; ++j) {
                if (j + 1 < n_blk) issue_qk(j + 1);      // its S held the weights of block j-1, whose product was issued before
                if (!ok) break;
                ok = mbar_wait(&bar.v_full[vs], v_phase, ctx, 0xD9) && mbar_wait(&bar.p_ready[j & 1], (j >> 1) & 1, ctx, 0xD4);
                if (!ok) break;
                tc_fence_after();
                const uint32_t w = tmem + (j & 1) * kKeys, o = tmem + 2 * kKeys, acc = j > 0 ? 1u : 0u;
                const uint64_t vd = v_desc + vs * v_stage16;
#pragma unroll
                for (int i = 0; i < 2 * (kKeys / 16); ++i) {             // hi, then lo
                    const int half = i / (kKeys / 16), kk = i % (kKeys / 16);
                    const uint32_t at = w + (kk >> 2) * 64 + half * 32 + (kk & 3) * 8;
                    if constexpr (PAIR) umma2_ts(o, at, vd + kk * (2048 >> 4), idesc_pv, i > 0 ? 1u : acc);
                    else umma_ts(o, at, vd + kk * (2048 >> 4), idesc_pv, i > 0 ? 1u : acc);
                }
                commit(&bar.v_empty[vs]);
                if (++vs == p.v_stages) { vs = 0; v_phase ^= 1; }
            }
            if (ok) commit(&bar.o_done);
            commit(&bar.drain);                          // nothing may be in flight when TMEM is freed
        }
        if (lane == 0) mbar_wait(&bar.drain, 0, ctx, 0xD5);
        __syncwarp();
    } else {
        const int r = (warp & 3) * 32 + lane, half = warp >> 2;          // row of the tile = TMEM lane; half of a block's keys
        const uint32_t lane_base = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const int me = p.start_pos + r0 + r;
        const float* bias = p.bias + static_cast<long long>(h) * p.n_bias;
        const float far = -kLog2e * __ldg(bias + p.n_bias - 1);
        bool ok = true;
        for (int j = 0; j < n_blk; ++j) {
            ok = mbar_wait_warp(&bar.s_full[j & 1], (j >> 1) & 1, ctx, 0xD6);
            if (!ok) break;
            tc_fence_after();
            const uint32_t s_addr = tmem + lane_base + (j & 1) * kKeys + half * 64;
            const int k0 = j * kKeys + half * 64;
            const int nearest = p.start_pos + r0 + (warp & 3) * 32 - (k0 + 63);         // smallest distance this warp meets in its half
            uint32_t s[2][32];
            tmem_ld32(s_addr, s[0]);
            tmem_ld32(s_addr + 32, s[1]);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                if (nearest >= p.n_bias - 1) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) s[c][i] = __float_as_uint(__uint_as_float(s[c][i]) + far);
                } else {
                    const int n0 = me - (k0 + c * 32);
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        const int n = n0 - i;
                        const float bv = __ldg(bias + min(max(n, 0), p.n_bias - 1));
                        s[c][i] = __float_as_uint(fmaf(bv, -kLog2e, __uint_as_float(s[c][i])));
                    }
                }
                uint32_t hi[16], lo[16];
                const bool diagonal = nearest < 0;
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float a = 1.0f + fast_exp2(fminf(__uint_as_float(s[c][2 * i]), kCut)), d = 1.0f + fast_exp2(fminf(__uint_as_float(s[c][2 * i + 1]), kCut));
                    const float inv = rcp_approx(a * d);
                    float w0 = inv * d, w1 = inv * a;
                    if (diagonal) {
                        const int n = me - (k0 + c * 32 + 2 * i);
                        if (n < 0) w0 = 0.f;
                        if (n < 1) w1 = 0.f;
                    }
                    split_hi_lo(w0, w1, hi[i], lo[i]);
                }
                tmem_st16(s_addr + c * 16, hi);
                tmem_st16(s_addr + 32 + c * 16, lo);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) {
                if constexpr (PAIR) mbar_arrive_cluster(map_to_cta(smem_u32(&bar.p_ready[j & 1]), 0));
                else mbar_arrive(&bar.p_ready[j & 1]);
            }
        }
        if (ok) ok = mbar_wait_warp(&bar.o_done, 0, ctx, 0xD7);
        if (ok) {
            tc_fence_after();
            const bool live = r0 + r < p.T;
            const long long m = static_cast<long long>(b) * p.T + r0 + r;
            float gate = 0.f;
            if (live) gate = 1.0f / (1.0f + __expf(-__bfloat162float(p.proj[m * p.ldp + p.gate_col + h])));
            __nv_bfloat16* orow = p.out + m * p.ldo + static_cast<long long>(h) * p.vdim;
            for (int c = half * 32; c < p.vdim; c += 64) {
                uint32_t o[32];
                tmem_ld32(tmem + lane_base + 2 * kKeys + c, o);
                tmem_ld_wait();
                if (live) {
#pragma unroll
                    for (int v = 0; v < 4; ++v) {
                        if (c + v * 8 >= p.vdim) break;
                        float f[8];
#pragma unroll
                        for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[v * 8 + e]) * gate;
                        store8(orow + c + v * 8, f);
                    }
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if constexpr (PAIR) { cluster_arrive(); cluster_wait(); }        // nobody signals the peer any more
    if (warp == 9) {
        tc_fence_after();
        if constexpr (PAIR) tmem_dealloc2(tmem, 512);
        else tmem_dealloc(tmem, 512);
    }
    abort_linger(&bar.abort_flag);
}

}  // namespace

bool sig_prefill_sm100_supported(const vb200_sigattn_args& a) {
    return a.dtype == VB200_BF16 && a.G * a.dim <= 512 && a.vdim % 8 == 0 && a.vdim <= 256 && a.ldo % 8 == 0 && a.T <= 65535 * kRows &&
           reinterpret_cast<uintptr_t>(a.out) % 16 == 0;
}

int launch_sig_prefill_sm100(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, const void* q, int* status) {
    const int kd = a.G * a.dim, n_ctx = a.start_pos + a.T, slots = a.slots ? 1 << 20 : a.B;      // a row's slot is the caller's promise
    if (n_ctx > a.cap) return set_detail(VB200_ERR_INVALID_ARG, "vb200_sigattn_forward: the prompt does not fit the cache");
    // two SMs per pair of heads that share their values; narrow keys are not what bounds the single form
    const bool pair = (a.H / a.G) % 2 == 0 && (a.vdim == 64 || a.vdim == 128) && kd >= 192 && a.form != 2;
    SigMaps maps;
    if (int rc = make_map_4d(&maps.q, q, kd, a.H, a.T, a.B, pl.qld, static_cast<long long>(a.H) * pl.qld, static_cast<long long>(a.T) * a.H * pl.qld, kRows)) return rc;
    if (int rc = make_map_4d(&maps.k, a.k_cache, kd, 1, n_ctx, slots, a.ldk, a.ldk, a.ldk * a.cap, pair ? kKeys / 2 : kKeys)) return rc;
    if (int rc = make_map_4d(&maps.v, a.v_cache, a.vdim, a.G, n_ctx, slots, a.vdim, a.ldv, a.ldv * a.cap, kKeys)) return rc;
    SigTileParams p{};
    p.T = a.T; p.start_pos = a.start_pos; p.vdim = a.vdim; p.R = a.H / a.G; p.n_bias = a.n_bias;
    p.gate_col = a.H * a.dim + a.G * (a.dim + a.vdim);
    p.nb_k = (kd + 63) / 64; p.nb_v = pair ? 1 : (a.vdim + 63) / 64; p.v_half = a.vdim / 2;
    p.bias = a.bias; p.proj = static_cast<const __nv_bfloat16*>(a.proj); p.out = static_cast<__nv_bfloat16*>(a.out);
    p.ldp = a.ldp; p.ldo = a.ldo; p.slots = a.slots; p.status = status;
    p.n_pv = pad_to(a.vdim, 16);
    // rings: what Q leaves.  Several boxes per K stage: every commit between products costs; V needs depth only where K is short
    const int k_box = pair ? kBox / 2 : kBox;
    int left = (kBoxesPerSm - p.nb_k) * kBox;
    p.v_stages = pair || left - 2 * p.nb_v * kBox >= 4 * kBox ? 2 : 1;
    left -= p.v_stages * p.nb_v * kBox;
    p.kbs = p.nb_k % 4 == 0 && left >= 8 * k_box ? 4 : p.nb_k % 2 == 0 ? 2 : 1;
    p.k_stages = left / (p.kbs * k_box);
    if (p.k_stages > kMaxStages) p.k_stages = kMaxStages;
    size_t smem = static_cast<size_t>(p.nb_k + p.v_stages * p.nb_v) * kBox + static_cast<size_t>(p.k_stages) * p.kbs * k_box;
    if (smem < 120 * 1024) smem = 120 * 1024;            // never a second CTA on an SM: it would find no TMEM
    auto kernel = pair ? sig_prefill_sm100_kernel<true> : sig_prefill_sm100_kernel<false>;
    if (int rc = allow_smem(kernel, smem)) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(static_cast<unsigned>(a.H), static_cast<unsigned>(a.B), static_cast<unsigned>((a.T + kRows - 1) / kRows));
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = 2;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pair ? 2 : 1;
    VB200_CUDA_TRY(cudaLaunchKernelEx(&cfg, kernel, maps, p));
    note_launch();
    note_sigattn_kernel(pair ? "sig_prefill_sm100_kernel (pair)" : "sig_prefill_sm100_kernel");
    return VB200_OK;
}

}  // namespace vb200
