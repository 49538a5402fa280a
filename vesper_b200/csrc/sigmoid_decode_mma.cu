// Decode attention of sigmoid-attention layers (one token per sequence) with warp-level MMAs.
//
// A mixed score takes the keys of all groups, so up to 16 heads of a sequence form the rows of m16n8k16 products against the whole
// key row [G * dim], and each cache row is fetched once per 16 heads.  Weights are not normalised: no maximum, no rescaling, and the
// splits of the keys simply add.
//
//   S[head, key]  = q'[head, :] . k[key, :]      the 8 warps take 16-column steps in turn (A in registers, B = rows by ldmatrix) and add
//                                                their partial S through shared memory; q' carries -log2(e)
//   O[head, c]   += W[head, key] v[key, c]       each warp owns 16-column blocks of the value row [G * vdim] (B by ldmatrix.trans), W = hi + lo
//                                                bf16; of a block's rows, those of its group are kept
// A 32-key tile arrives as TMA boxes of [32 keys x 64 columns] with the 128-byte swizzle, in a ring of stages that thread 0 refills: the
// barrier after the scores of a tile tells it that every warp is done with the tile before.
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kTile = 32;                // keys per stage
constexpr int kBox = kTile * 128;
constexpr int kWarps = 8;
constexpr int kStagesMax = 6;
constexpr int kRedLd = 40;               // floats per row of a partial score tile: 8-row float2 accesses without conflicts
constexpr int kPLd = 40;                 // bf16 per row of a weight tile: ldmatrix phases without conflicts

struct SigCacheMaps { CUtensorMap k, v; };

struct SigSplitParams {
    int H, R, vdim, n_bias, cap, ks, nvb, nbk, nbox, splits, stages, qld;
    const int *slots, *pos;
    const float* bias;
    const __nv_bfloat16* q;
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

struct __align__(16) SigSplitSmem {
    float red[kWarps][16][kRedLd];
    __nv_bfloat16 w_hi[16][kPLd], w_lo[16][kPLd];
    uint64_t full[kStagesMax];
    int abort_flag;
};

// grid (splits, ceil(H / 16), B).  KS: 16-column key steps per warp; NP: 16-column value blocks per warp.
template <int KS, int NP>
__global__ void __launch_bounds__(kWarps * 32, 2)
sig_decode_mma_kernel(const __grid_constant__ SigCacheMaps maps, SigSplitParams p) {
    extern __shared__ uint8_t raw[];
    uint8_t* tiles = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~static_cast<uintptr_t>(1023));
    const int stage_bytes = p.nbox * kBox;
    SigSplitSmem& sm = *reinterpret_cast<SigSplitSmem*>(tiles + p.stages * stage_bytes);
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
    const int me = min(p.pos[b], p.cap - 1), n = me + 1, chunk = (n + p.splits - 1) / p.splits;
    const int k0 = split * chunk, k1 = min(n, k0 + chunk);
    const int n_tiles = k1 > k0 ? (k1 - k0 + kTile - 1) / kTile : 0;
    const int slot = p.slots ? p.slots[b] : b;
    auto load_tile = [&](int i) {
        const int s = i % p.stages;
        uint8_t* st = tiles + s * stage_bytes;
        mbar_arrive_expect_tx(&sm.full[s], stage_bytes);
        for (int x = 0; x < p.nbox; ++x) {
            const bool val = x >= p.nbk;
            tma_load_4d(st + x * kBox, val ? &maps.v : &maps.k, &sm.full[s], (val ? x - p.nbk : x) * 64, 0, k0 + i * kTile, slot);
        }
    };
    if (tid == 0)
        for (int i = 0; i < min(p.stages, n_tiles); ++i) load_tile(i);

    const int g = lane >> 2, t = lane & 3;
    // A fragments of this warp's steps: rows = heads h0 + g, h0 + g + 8
    uint32_t qa[KS][4];
#pragma unroll
    for (int i = 0; i < KS; ++i) {
        const int kk = warp + i * kWarps;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int h = h0 + g + (e & 1) * 8;
            qa[i][e] = kk < p.ks && h < p.H ? *reinterpret_cast<const uint32_t*>(p.q + (static_cast<long long>(b) * p.H + h) * p.qld + kk * 16 + (e >> 1) * 8 + t * 2) : 0u;
        }
    }
    float o[NP][2][4];
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][x][e] = 0.f;
    const int row = tid >> 4, kp = (tid & 15) * 2;                       // weights: this thread's head and two keys of a tile
    const float* bias = p.bias + static_cast<long long>(min(h0 + row, p.H - 1)) * p.n_bias;
    // ldmatrix offsets inside a tile: this lane addresses row mr (mod 8) of matrix mi; 16 keys on = 2048 bytes
    const int mi = lane >> 3, mr = lane & 7;
    uint32_t s_off[KS], v_off[NP];
#pragma unroll
    for (int i = 0; i < KS; ++i) {
        const int kk = min(warp + i * kWarps, p.ks - 1), ch = (kk & 3) * 2 + (mi & 1);
        s_off[i] = (kk >> 2) * kBox + ((mi >> 1) * 8 + mr) * 128 + ((ch ^ mr) << 4);
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int blk = min(warp + i * kWarps, p.nvb - 1), ch = (blk & 3) * 2 + (mi >> 1);            // a block too many is computed and dropped
        v_off[i] = (p.nbk + (blk >> 2)) * kBox + ((mi & 1) * 8 + mr) * 128 + ((ch ^ mr) << 4);
    }
    const uint32_t hi_a = smem_u32(&sm.w_hi[(mi & 1) * 8 + mr][(mi >> 1) * 8]), lo_a = smem_u32(&sm.w_lo[(mi & 1) * 8 + mr][(mi >> 1) * 8]);
    for (int it = 0; it < n_tiles; ++it) {
        const int s = it % p.stages, first = k0 + it * kTile, valid = min(kTile, k1 - first);
        const bool ok = mbar_wait_warp(&sm.full[s], (it / p.stages) & 1, ctx, 0xE1);
        uint8_t* tile = tiles + s * stage_bytes;
        const uint32_t tile_a = smem_u32(tile);
        const int d = me - (first + kp);                                 // distances of this thread's keys: d, d - 1
        const float b0 = bias[min(max(d, 0), p.n_bias - 1)], b1 = bias[min(max(d - 1, 0), p.n_bias - 1)];
        float c[4][4] = {};
        if (ok) {
#pragma unroll
            for (int i = 0; i < KS; ++i) {                               // steps past the last one have zero queries
                uint32_t bq[2][4];
                ldmatrix4(bq[0], tile_a + s_off[i]);
                ldmatrix4(bq[1], tile_a + s_off[i] + 2048);
#pragma unroll
                for (int x = 0; x < 4; ++x) mma_bf16(c[x], qa[i], bq[x >> 1][(x & 1) * 2], bq[x >> 1][(x & 1) * 2 + 1]);
            }
            if (valid < kTile) {
                // rows past the slice hold other tokens: their weight is zero, and so must their values be.  Each warp clears the
                // columns that it alone reads.
                for (int i = 0; i < NP; ++i) {
                    const int blk = warp + i * kWarps;
                    if (blk >= p.nvb) break;
                    for (int x = lane; x < (kTile - valid) * 2; x += 32) {
                        const int key = valid + (x >> 1), ch = (blk & 3) * 2 + (x & 1);
                        *reinterpret_cast<uint4*>(tile + (p.nbk + (blk >> 2)) * kBox + key * 128 + ((ch ^ (key & 7)) << 4)) = make_uint4(0, 0, 0, 0);
                    }
                }
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            *reinterpret_cast<float2*>(&sm.red[warp][g][x * 8 + t * 2]) = make_float2(c[x][0], c[x][1]);
            *reinterpret_cast<float2*>(&sm.red[warp][g + 8][x * 8 + t * 2]) = make_float2(c[x][2], c[x][3]);
        }
        if (__syncthreads_or(!ok)) break;                                // a wait ran out: all leave together
        if (tid == 0 && it > 0 && it - 1 + p.stages < n_tiles) load_tile(it - 1 + p.stages);
        float2 sv = make_float2(0.f, 0.f);
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
            const float2 v = *reinterpret_cast<const float2*>(&sm.red[w][row][kp]);
            sv.x += v.x; sv.y += v.y;
        }
        // sigmoid(s + bias) = 1 / (1 + 2^(-(s + bias) log2 e)), s with its factor already
        float w0 = __fdividef(1.0f, 1.0f + fast_exp2(fminf(fmaf(b0, -kLog2e, sv.x), 100.0f))), w1 = __fdividef(1.0f, 1.0f + fast_exp2(fminf(fmaf(b1, -kLog2e, sv.y), 100.0f)));
        if (kp >= valid) w0 = 0.f;
        if (kp + 1 >= valid) w1 = 0.f;
        uint32_t hi, lo;
        split_hi_lo(w0, w1, hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.w_hi[row][kp]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.w_lo[row][kp]) = lo;
        __syncthreads();
        uint32_t ph[2][4], pl[2][4];
#pragma unroll
        for (int ks = 0; ks < 2; ++ks) {
            ldmatrix4(ph[ks], hi_a + ks * 32);
            ldmatrix4(pl[ks], lo_a + ks * 32);
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
    float* out = p.part + ((static_cast<long long>(b) * p.H) * p.splits + split) * p.vdim;
    const long long head_ld = static_cast<long long>(p.splits) * p.vdim;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int blk = warp + i * kWarps;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int col = blk * 16 + x * 8 + t * 2, group = (blk * 16 + x * 8) / p.vdim, v = col - group * p.vdim;      // vdim % 8 == 0: one group per 8 columns
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int h = h0 + g + e * 8;
                if (h < p.H && h / p.R == group) *reinterpret_cast<float2*>(out + h * head_ld + v) = make_float2(o[i][x][2 * e], o[i][x][2 * e + 1]);
            }
        }
    }
    __syncthreads();
    abort_linger(&sm.abort_flag);
}

int boxes(int cols) { return (cols + 63) / 64; }
int stage_bytes_of(const vb200_sigattn_args& a) { return (boxes(a.G * a.dim) + boxes(a.G * a.vdim)) * kBox; }

}  // namespace

bool sig_decode_mma_supported(const vb200_sigattn_args& a) { return a.dtype == VB200_BF16 && a.G * a.dim <= 512 && a.G * a.vdim <= 512 && a.vdim % 8 == 0; }

int sig_decode_ctas_per_sm(const vb200_sigattn_args& a) { return stage_bytes_of(a) <= 40 * 1024 ? 2 : 1; }

int launch_sig_decode_mma(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, const void* q, float* part, int* status) {
    const int kd = a.G * a.dim, vd = a.G * a.vdim, slots = a.slots ? 1 << 20 : a.B;          // a row's slot is the caller's promise
    SigCacheMaps maps;
    if (int rc = make_map_4d(&maps.k, a.k_cache, kd, 1, a.cap, slots, a.ldk, a.ldk, a.ldk * a.cap, kTile)) return rc;
    if (int rc = make_map_4d(&maps.v, a.v_cache, vd, 1, a.cap, slots, a.ldv, a.ldv, a.ldv * a.cap, kTile)) return rc;
    SigSplitParams p{};
    p.H = a.H; p.R = a.H / a.G; p.vdim = a.vdim; p.n_bias = a.n_bias; p.cap = a.cap;
    p.ks = (kd + 15) / 16; p.nvb = (vd + 15) / 16; p.nbk = boxes(kd); p.nbox = p.nbk + boxes(vd);
    p.splits = pl.splits; p.qld = pl.qld; p.slots = a.slots; p.pos = a.pos; p.bias = a.bias;
    p.q = static_cast<const __nv_bfloat16*>(q); p.part = part; p.status = status;
    const int stage = stage_bytes_of(a), budget = sig_decode_ctas_per_sm(a) == 2 ? 84 * 1024 : 200 * 1024;
    p.stages = budget / stage;
    if (p.stages > kStagesMax) p.stages = kStagesMax;
    const size_t smem = 1024 + static_cast<size_t>(p.stages) * stage + sizeof(SigSplitSmem);
    auto go = [&](auto kernel) -> int {
        if (int rc = allow_smem(kernel, smem)) return rc;
        return launch_pdl(kernel, dim3(static_cast<unsigned>(pl.splits), static_cast<unsigned>((a.H + 15) / 16), static_cast<unsigned>(a.B)), dim3(kWarps * 32), smem, s, maps, p);
    };
    const int widest = p.ks > p.nvb ? p.ks : p.nvb;
    if (widest <= 8) return go(sig_decode_mma_kernel<1, 1>);
    if (widest <= 16) return go(sig_decode_mma_kernel<2, 2>);
    return go(sig_decode_mma_kernel<4, 4>);
}

}  // namespace vb200
