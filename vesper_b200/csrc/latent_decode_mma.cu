// Decode attention over latents (one token per sequence, absorbed queries) with warp-level MMAs.
//
// Every head reads the same latent rows, so up to 16 heads of a sequence form the rows of m16n8k16 products and each row
// of the ring is fetched once per 16 heads.  The queries (fp32, scale * log2 e folded in) are rounded to bf16 like any
// projection's output; scores and softmax stay fp32, and the weights enter the second product as hi + lo bf16 halves.
//
//   S[head, key] = q'[head, :] . row[key, :]     the 8 consumer warps take 16-column steps in turn (A in registers,
//                                                B = rows by ldmatrix) and add their partial S through shared memory
//   O[head, c]  += P[head, key] row[key, c]      each warp owns 16-column blocks of the latent (B by ldmatrix.trans)
// A 32-key tile arrives as TMA boxes of [32 keys x 64 columns] with the 128-byte swizzle (4-D maps over the ring, zero
// fill past the latent's and the rotated part's width), in a ring of stages that thread 0 refills: the barrier after
// the scores of a tile tells it that every warp is done with the tile before.
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kTile = 32;                // keys per stage
constexpr int kBox = kTile * 128;
constexpr int kWarps = 8;                // consumer warps
constexpr int kStagesMax = 6;
constexpr int kRedLd = 40;               // floats per row of a partial score tile: 8-row float2 accesses without conflicts
constexpr float kGrow = 8.0f;
constexpr int kPLd = 40;                 // bf16 per row of a weight tile: ldmatrix phases without conflicts

struct LatentCacheMaps { CUtensorMap c, r; };

struct LatentSplitParams {
    int H, ring, rank, ksc, ks, nbc, nbox, splits, stages;
    long long qld, part_ld;
    int rank16;
    const int *slots, *pos;
    const float* q;
    float* part;
    int* status;
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void consumers_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// The same barrier, returning to every consumer whether any of them passed true.
__device__ __forceinline__ bool consumers_sync_any(bool v) {
    uint32_t r;
    asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.b32 p, %1, 0;\n\tbar.red.or.pred q, 1, 256, p;\n\tselp.b32 %0, 1, 0, q;\n\t}" : "=r"(r) : "r"(static_cast<uint32_t>(v)) : "memory");
    return r != 0;
}

struct __align__(16) LatentSplitSmem {
    float red[kWarps][16][kRedLd];
    __nv_bfloat16 p_hi[16][kPLd], p_lo[16][kPLd];
    float alpha[16];
    uint64_t full[kStagesMax];
    int abort_flag;
};

// KS: 16-column steps per warp; NP: 16-column output blocks per warp.
template <int KS, int NP>
__global__ void __launch_bounds__(kWarps * 32, 2)
latent_split_mma_kernel(const __grid_constant__ LatentCacheMaps maps, LatentSplitParams p) {
    extern __shared__ uint8_t raw[];
    uint8_t* tiles = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~static_cast<uintptr_t>(1023));
    const int stage_bytes = p.nbox * kBox;
    LatentSplitSmem& sm = *reinterpret_cast<LatentSplitSmem*>(tiles + p.stages * stage_bytes);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, h0 = blockIdx.y * 16, b = blockIdx.z;
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) mbar_init(&sm.full[i], 1);
        sm.abort_flag = 0;
        mbar_fence_init();
    }
    __syncthreads();
    pdl_begin();
    const WaitCtx ctx{&sm.abort_flag, p.status};
    const int n = min(p.pos[b] + 1, p.ring), chunk = (n + p.splits - 1) / p.splits;
    const int k0 = split * chunk, k1 = min(n, k0 + chunk);
    const int n_tiles = k1 > k0 ? (k1 - k0 + kTile - 1) / kTile : 0;
    const int slot = p.slots ? p.slots[b] : b;
    auto load_tile = [&](int i) {
        const int s = i % p.stages;
        uint8_t* st = tiles + s * stage_bytes;
        mbar_arrive_expect_tx(&sm.full[s], stage_bytes);
        for (int x = 0; x < p.nbox; ++x) {
            const bool rot = x >= p.nbc;
            tma_load_4d(st + x * kBox, rot ? &maps.r : &maps.c, &sm.full[s], (rot ? x - p.nbc : x) * 64, 0, k0 + i * kTile, slot);
        }
    };
    if (tid == 0)
        for (int i = 0; i < min(p.stages, n_tiles); ++i) load_tile(i);

    {
        const int g = lane >> 2, t = lane & 3;
        // A fragments of this warp's steps: rows = heads h0 + g, h0 + g + 8
        uint32_t qh[KS][4];
#pragma unroll
        for (int i = 0; i < KS; ++i) {
            const int kk = warp + i * kWarps;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int h = h0 + g + (e & 1) * 8;
                float2 v = make_float2(0.f, 0.f);
                if (kk < p.ks && h < p.H) v = *reinterpret_cast<const float2*>(p.q + (static_cast<long long>(b) * p.H + h) * p.qld + kk * 16 + (e >> 1) * 8 + t * 2);
                qh[i][e] = Elem<__nv_bfloat16>::pack2(v.x, v.y);
            }
        }
        float o[NP][2][4];
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[i][x][e] = 0.f;
        const int row = tid >> 4, kp = (tid & 15) * 2;           // softmax: this thread's head and two keys
        float m = -1e30f, l = 0.f;
        // ldmatrix offsets inside a tile: this lane addresses row mr (mod 8) of matrix mi; 16 keys on = 2048 bytes
        const int mi = lane >> 3, mr = lane & 7;
        uint32_t s_off[KS], v_off[NP];
#pragma unroll
        for (int i = 0; i < KS; ++i) {
            const int kk = min(warp + i * kWarps, p.ks - 1), kc = kk < p.ksc ? kk : kk - p.ksc, box = (kk < p.ksc ? 0 : p.nbc) + (kc >> 2), ch = (kc & 3) * 2 + (mi & 1);
            s_off[i] = box * kBox + ((mi >> 1) * 8 + mr) * 128 + ((ch ^ mr) << 4);
        }
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int blk = min(warp + i * kWarps, p.ksc - 1), ch = (blk & 3) * 2 + (mi >> 1);      // a block too many is computed and dropped
            v_off[i] = (blk >> 2) * kBox + ((mi & 1) * 8 + mr) * 128 + ((ch ^ mr) << 4);
        }
        const uint32_t p_hi_a = smem_u32(&sm.p_hi[(mi & 1) * 8 + mr][(mi >> 1) * 8]), p_lo_a = smem_u32(&sm.p_lo[(mi & 1) * 8 + mr][(mi >> 1) * 8]);
        for (int it = 0; it < n_tiles; ++it) {
            const int s = it % p.stages, valid = min(kTile, k1 - k0 - it * kTile);
            const bool ok = mbar_wait_warp(&sm.full[s], (it / p.stages) & 1, ctx, 0xC2);
            uint8_t* tile = tiles + s * stage_bytes;
            const uint32_t tile_a = smem_u32(tile);
            float c[4][4] = {};
            if (ok) {
#pragma unroll
                for (int i = 0; i < KS; ++i) {                   // steps past the last one have zero queries
                    uint32_t bq[2][4];
                    ldmatrix4(bq[0], tile_a + s_off[i]);
                    ldmatrix4(bq[1], tile_a + s_off[i] + 2048);
#pragma unroll
                    for (int x = 0; x < 4; ++x) mma_bf16(c[x], qh[i], bq[x >> 1][(x & 1) * 2], bq[x >> 1][(x & 1) * 2 + 1]);
                }
                if (valid < kTile) {
                    // rows past the slice hold other tokens (or another sequence's): their weight is zero, and so must their
                    // values be.  Each warp clears the columns it alone has read so far.
                    __syncwarp();
                    for (int i = 0; i < KS; ++i) {
                        const int kk = warp + i * kWarps;
                        if (kk >= p.ksc) break;
                        for (int x = lane; x < (kTile - valid) * 2; x += 32) {
                            const int key = valid + (x >> 1), ch = (kk & 3) * 2 + (x & 1);
                            *reinterpret_cast<uint4*>(tile + (kk >> 2) * kBox + key * 128 + ((ch ^ (key & 7)) << 4)) = make_uint4(0, 0, 0, 0);
                        }
                    }
                }
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                *reinterpret_cast<float2*>(&sm.red[warp][g][x * 8 + t * 2]) = make_float2(c[x][0], c[x][1]);
                *reinterpret_cast<float2*>(&sm.red[warp][g + 8][x * 8 + t * 2]) = make_float2(c[x][2], c[x][3]);
            }
            if (consumers_sync_any(!ok)) break;                  // a wait ran out: all consumers leave together
            if (tid == 0 && it > 0 && it - 1 + p.stages < n_tiles) load_tile(it - 1 + p.stages);
            float2 sv = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < kWarps; ++w) {
                const float2 v = *reinterpret_cast<const float2*>(&sm.red[w][row][kp]);
                sv.x += v.x; sv.y += v.y;
            }
            if (kp >= valid) sv.x = -INFINITY;
            if (kp + 1 >= valid) sv.y = -INFINITY;
            float mt = fmaxf(sv.x, sv.y);
#pragma unroll
            for (int x = 8; x > 0; x >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xFFFFFFFFu, mt, x));
            // the reference maximum follows only when a row grows by more than 2^8 beyond it: most tiles rescale nothing
            const float m_new = mt > m + kGrow ? mt : m, alpha = fast_exp2(m - m_new);
            const float p0 = fast_exp2(sv.x - m_new), p1 = fast_exp2(sv.y - m_new);
            float ls = p0 + p1;
#pragma unroll
            for (int x = 8; x > 0; x >>= 1) ls += __shfl_xor_sync(0xFFFFFFFFu, ls, x);
            l = l * alpha + ls;
            m = m_new;
            uint32_t hi, lo;
            split_hi_lo(p0, p1, hi, lo);
            *reinterpret_cast<uint32_t*>(&sm.p_hi[row][kp]) = hi;
            *reinterpret_cast<uint32_t*>(&sm.p_lo[row][kp]) = lo;
            if ((tid & 15) == 0) sm.alpha[row] = alpha;
            consumers_sync();
            const float a0 = sm.alpha[g], a1 = sm.alpha[g + 8];
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                ldmatrix4(ph[ks], p_hi_a + ks * 32);
                ldmatrix4(pl[ks], p_lo_a + ks * 32);
            }
            if (__any_sync(0xFFFFFFFFu, a0 != 1.0f || a1 != 1.0f)) {
#pragma unroll
                for (int i = 0; i < NP; ++i)
#pragma unroll
                    for (int x = 0; x < 2; ++x) { o[i][x][0] *= a0; o[i][x][1] *= a0; o[i][x][2] *= a1; o[i][x][3] *= a1; }
            }
#pragma unroll
            for (int ks = 0; ks < 2; ++ks) {
                uint32_t bv[NP][4];
#pragma unroll
                for (int i = 0; i < NP; ++i) ldmatrix4_trans(bv[i], tile_a + v_off[i] + ks * 2048);
#pragma unroll
                for (int i = 0; i < NP; ++i) { mma_bf16(o[i][0], ph[ks], bv[i][0], bv[i][1]); mma_bf16(o[i][1], ph[ks], bv[i][2], bv[i][3]); }
#pragma unroll
                for (int i = 0; i < NP; ++i) { mma_bf16(o[i][0], pl[ks], bv[i][0], bv[i][1]); mma_bf16(o[i][1], pl[ks], bv[i][2], bv[i][3]); }
            }
        }
        float* out = p.part + ((static_cast<long long>(b) * p.H) * p.splits + split) * p.part_ld;
        const long long head_ld = static_cast<long long>(p.splits) * p.part_ld;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int blk = warp + i * kWarps;
            if (blk >= p.ksc) break;
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int col = blk * 16 + x * 8 + t * 2;
                if (h0 + g < p.H) *reinterpret_cast<float2*>(out + (h0 + g) * head_ld + col) = make_float2(o[i][x][0], o[i][x][1]);
                if (h0 + g + 8 < p.H) *reinterpret_cast<float2*>(out + (h0 + g + 8) * head_ld + col) = make_float2(o[i][x][2], o[i][x][3]);
            }
        }
        if ((tid & 15) == 0 && h0 + row < p.H) {
            out[(h0 + row) * head_ld + p.rank16] = m;
            out[(h0 + row) * head_ld + p.rank16 + 1] = l;
        }
    }
    __syncthreads();
    abort_linger(&sm.abort_flag);
}

}  // namespace

bool latent_mma_supported(const vb200_latent_args& a) { return a.dtype == VB200_BF16 && a.rank <= 512 && a.rot_dim <= 128 && a.rot_dim > 0; }

int launch_latent_split_mma(cudaStream_t s, const vb200_latent_args& a, const LatentPlan& pl, const float* q, float* part, int* status) {
    const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(a.cache);
    const int slots = a.slots ? 1 << 20 : a.B;                  // a row's slot is the caller's promise; its ring rows are bounded
    LatentCacheMaps maps;
    if (int rc = make_map_4d(&maps.c, cache, a.rank, 1, a.ring, slots, a.ldc, a.ldc, a.ldc * a.ring, kTile)) return rc;
    if (int rc = make_map_4d(&maps.r, cache + vb200_latent_rot_offset(a.rank), a.rot_dim, 1, a.ring, slots, a.ldc, a.ldc, a.ldc * a.ring, kTile)) return rc;
    LatentSplitParams p{};
    p.H = a.H; p.ring = a.ring; p.rank = a.rank; p.rank16 = pl.rank16;
    p.ksc = pl.rank16 / 16; p.ks = p.ksc + pl.rot16 / 16;
    p.nbc = (a.rank + 63) / 64; p.nbox = p.nbc + (a.rot_dim + 63) / 64;
    p.splits = pl.splits; p.qld = pl.qld; p.part_ld = pl.part_ld;
    p.slots = a.slots; p.pos = a.pos; p.q = q; p.part = part; p.status = status;
    const int stage = p.nbox * kBox;
    p.stages = 80 * 1024 / stage;
    if (p.stages > kStagesMax) p.stages = kStagesMax;
    const size_t smem = 1024 + static_cast<size_t>(p.stages) * stage + sizeof(LatentSplitSmem);
    auto go = [&](auto kernel) -> int {
        if (int rc = allow_smem(kernel, smem)) return rc;
        return launch_pdl(kernel, dim3(static_cast<unsigned>(pl.splits), static_cast<unsigned>((a.H + 15) / 16), static_cast<unsigned>(a.B)), dim3(kWarps * 32), smem, s, maps, p);
    };
    note_latent_kernel("latent_split_mma_kernel");
    if (p.ks <= 16 && p.ksc <= 8) return go(latent_split_mma_kernel<2, 1>);
    if (p.ks <= 24 && p.ksc <= 16) return go(latent_split_mma_kernel<3, 2>);
    return go(latent_split_mma_kernel<5, 4>);
}

}  // namespace vb200
