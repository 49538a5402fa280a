// The Mamba-2 recurrence over a prompt in chunks of 64 tokens, as matrix products (bf16 inputs):
//
//   la_i = log2 of the decay from the chunk's start through token i        (fp32 running sum of -exp(A) dt)
//   y_i  = 2^la_i C_i S  +  sum_{j <= i} (C_i . B_j) 2^(la_i - la_j) dt_j x_j  +  D x_i
//   S   <- 2^la_last S   +  sum_j 2^(la_last - la_j) dt_j B_j x_j^T
//
// One CTA of eight warps walks the chunks of one (batch, head, column slice) with S in its MMA accumulators: warp-level
// m16n8k16 products, fp32 accumulation.  C, B and x are bf16 values as they come from the convolution; everything the
// decays touch (the weights of the second sum, the weighted B of the state update, S itself as a right operand) enters
// as hi + lo bf16 halves, so the recurrence keeps fp32-class accuracy.
// Heads of up to 64 columns and 128 state rows take the tcgen05 walk (ssd_walk_sm100.cu) instead; this file's kernel then
// only computes what segments add.
// When batch x heads does not fill the machine the portion is cut into segments: a first pass computes what each
// segment adds to the state, a small kernel chains them, and the walk starts every segment from its own state.
#include "hybrid.cuh"

namespace vb200 {
namespace {

constexpr int kChunk = 64;
constexpr int kThreads = 256;
constexpr int kPad = 8;                  // bf16 of row padding: ldmatrix rows fall into distinct banks

struct ChunkParams {
    int T, H, P, N, G, channels, Pp, N16, slices, pw;       // pw: columns per slice
    int n_seg, seg_chunks;
    long long ldp;
    const __nv_bfloat16 *proj, *xbc;
    const float *dt_bias, *A_log, *D;
    const int *slots, *pos;
    float* state;                        // [slots, H, N, Pp]
    float *seg_state, *seg_decay;        // [B, n_seg, H, N, Pp], [B, n_seg, H] (n_seg > 1)
    __nv_bfloat16* gated;                // [B*T, H * P]
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], const __nv_bfloat16* ptr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(ptr)) : "memory");
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], const __nv_bfloat16* ptr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(ptr)) : "memory");
}

__device__ __forceinline__ void cp_async16(const __nv_bfloat16* dst, const void* src, bool ok) {       // zeros when !ok
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// MT: 16-row tiles of S per warp (rows dealt to the eight warps in turn); PT: 8-column tiles of the slice.  In the
// output products warp w has token rows 16 (w & 3) .. and column half w >> 2.
// OUT: the walk (outputs and, in the last segment, the final state); else the first pass (what a segment adds to S).
// B and x of the next chunk are copied (cp.async) into second buffers while this one computes, C once its last reader
// is through; step sizes and gates are fetched ahead into registers.
template <int MT, int PT, bool OUT>
__global__ void __launch_bounds__(kThreads, 2)
ssd_chunk_kernel(ChunkParams p) {
    pdl_begin();
    extern __shared__ __align__(16) uint8_t smem[];
    const int ldn = p.N16 + kPad;
    constexpr int kPw = PT * 8, ldp_s = kPw + kPad, HT = PT / 2;
    const int b_size = kChunk * ldn;
    constexpr int x_size = kChunk * ldp_s;
    __nv_bfloat16* Bbuf = reinterpret_cast<__nv_bfloat16*>(smem);      // 2 x [64][ldn]
    __nv_bfloat16* xbuf = Bbuf + 2 * b_size;                           // 2 x [64][ldp_s]
    __nv_bfloat16* Cs = xbuf + 2 * x_size;                             // [64][ldn]
    __nv_bfloat16* Sh = Cs + b_size;                                   // [N16][ldp_s] high halves, then low halves
    __nv_bfloat16* Sl = Sh + p.N16 * ldp_s;
    __shared__ float s_la[2][kChunk], s_dt[2][kChunk], s_w[2][kChunk];

    const int seg = blockIdx.x, h = blockIdx.y / p.slices, sl = blockIdx.y % p.slices, b = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, mr = lane & 7;
    const int grp = h / (p.H / p.G), inner = p.H * p.P, p0 = sl * kPw, pn = min(p.P - p0, kPw);
    const int slot = p.slots ? p.slots[b] : b;
    const float nA2 = -expf(p.A_log[h]) * kLog2e, dtb = p.dt_bias[h], Dh = OUT ? p.D[h] : 0.f;
    const long long seg_row = (static_cast<long long>(b) * p.n_seg + seg) * p.H + h;
    const int c_begin = seg * p.seg_chunks, c_end = min((p.T + kChunk - 1) / kChunk, c_begin + p.seg_chunks);
    const __nv_bfloat16* xbc = p.xbc + static_cast<long long>(b) * p.T * p.channels;
    const __nv_bfloat16* proj = p.proj + static_cast<long long>(b) * p.T * p.ldp;

    // ---- tile copies: 16-byte pieces, zero past the portion and past a matrix's width ----
    // this thread's first piece and the step between its pieces, in (row, column) of a tile
    const int nv = p.N16 / 8;
    const int nb_r0 = threadIdx.x / nv, nb_c0 = (threadIdx.x % nv) * 8, nb_dr = kThreads / nv, nb_dc = (kThreads % nv) * 8;
    auto copy_nb = [&](const __nv_bfloat16* dst, int ch, int col0) {
        const __nv_bfloat16* src = xbc + static_cast<long long>(ch) * kChunk * p.channels + col0;
        const int rows = p.T - ch * kChunk;
        int c = nb_c0;
        for (int r = nb_r0; r < kChunk; r += nb_dr) {
            const bool ok = r < rows && c < p.N;
            cp_async16(dst + r * ldn + c, ok ? src + static_cast<long long>(r) * p.channels + c : xbc, ok);
            c += nb_dc;
            if (c >= p.N16) { c -= p.N16; ++r; }
        }
    };
    constexpr int pv = kPw / 8;
    const int x_r0 = threadIdx.x / pv, x_c = (threadIdx.x % pv) * 8;
    auto copy_x = [&](const __nv_bfloat16* dst, int ch) {
        const __nv_bfloat16* src = xbc + static_cast<long long>(ch) * kChunk * p.channels + h * p.P + p0 + x_c;
        const int rows = x_c < pn ? p.T - ch * kChunk : 0;
#pragma unroll
        for (int r = x_r0; r < kChunk; r += kThreads / pv) {
            const bool ok = r < rows;
            cp_async16(dst + r * ldp_s + x_c, ok ? src + static_cast<long long>(r) * p.channels : xbc, ok);
        }
    };
    const int col_b = inner + grp * p.N, col_c = col_b + p.G * p.N, col_dt = 2 * inner + 2 * p.G * p.N + h;
    // step sizes and the running log-decay of a chunk: warp 7, two tokens per lane
    auto fetch_dt = [&](int ch, float (&raw)[2]) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = ch * kChunk + lane * 2 + e;
            raw[e] = t < p.T ? __bfloat162float(proj[static_cast<long long>(t) * p.ldp + col_dt]) : 0.f;
        }
    };
    auto scan_dt = [&](int ch, const float (&raw)[2]) {
        float d[2], a[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            d[e] = ch * kChunk + lane * 2 + e < p.T ? softplus_f(raw[e] + dtb) : 0.f;
            a[e] = nA2 * d[e];
        }
        float s = a[0] + a[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xFFFFFFFFu, s, o);
            if (lane >= o) s += v;
        }
        const float excl = s - (a[0] + a[1]), l0 = excl + a[0], l1 = l0 + a[1], last = __shfl_sync(0xFFFFFFFFu, l1, 31);
        const int q = ch & 1;
        s_la[q][lane * 2] = l0; s_la[q][lane * 2 + 1] = l1;
        s_dt[q][lane * 2] = d[0]; s_dt[q][lane * 2 + 1] = d[1];
        s_w[q][lane * 2] = d[0] * fast_exp2(last - l0); s_w[q][lane * 2 + 1] = d[1] * fast_exp2(last - l1);
    };
    float raw_dt[2] = {0.f, 0.f};
    copy_nb(Bbuf + (c_begin & 1) * b_size, c_begin, col_b);
    copy_x(xbuf + (c_begin & 1) * x_size, c_begin);
    if (OUT) copy_nb(Cs, c_begin, col_c);
    cp_commit();
    if (warp == 7) { fetch_dt(c_begin, raw_dt); scan_dt(c_begin, raw_dt); }

    // rows mt*16 + g, +8 and columns p0 + pt*8 + 2*t4 of the state
    float S[MT][PT][4];
    float* sp = p.state + (static_cast<long long>(slot) * p.H + h) * p.N * p.Pp + p0;
    {
        const float* src = nullptr;
        if (OUT) src = p.n_seg > 1 ? p.seg_state + seg_row * p.N * p.Pp + p0 : (p.pos[b] > 0 ? sp : nullptr);
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int x = 0; x < PT; ++x)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int n = (warp + 8 * i) * 16 + g + hf * 8, c = x * 8 + t4 * 2;
                    float2 v = make_float2(0.f, 0.f);
                    if (src != nullptr && n < p.N && c < pn) v = *reinterpret_cast<const float2*>(src + static_cast<long long>(n) * p.Pp + c);
                    S[i][x][hf * 2] = v.x; S[i][x][hf * 2 + 1] = v.y;
                }
    }
    auto publish_state = [&] {                      // S as the right operand of the next chunk's C S
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            if ((warp + 8 * i) * 16 >= p.N16) break;
            const int at0 = ((warp + 8 * i) * 16 + g) * ldp_s + t4 * 2;
#pragma unroll
            for (int x = 0; x < PT; ++x)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    uint32_t hi, lo;
                    split_hi_lo(S[i][x][hf * 2], S[i][x][hf * 2 + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(Sh + at0 + hf * 8 * ldp_s + x * 8) = hi;
                    *reinterpret_cast<uint32_t*>(Sl + at0 + hf * 8 * ldp_s + x * 8) = lo;
                }
        }
    };
    if (OUT) publish_state();
    float log_decay = 0.f;
    for (int ch = c_begin; ch < c_end; ++ch) {
        const int tn = min(kChunk, p.T - ch * kChunk), q = ch & 1;
        const long long m0 = static_cast<long long>(b) * p.T + ch * kChunk;
        const __nv_bfloat16 *Bs = Bbuf + q * b_size, *xs = xbuf + q * x_size;
        const float *la = s_la[q], *dtv = s_dt[q], *wv = s_w[q];
        cp_wait_all();
        __syncthreads();                            // tiles, step sizes and S of this chunk are in place; the other buffers are free
        const bool more = ch + 1 < c_end;
        if (more) {
            copy_nb(Bbuf + (q ^ 1) * b_size, ch + 1, col_b);
            copy_x(xbuf + (q ^ 1) * x_size, ch + 1);
            cp_commit();
            if (warp == 7) fetch_dt(ch + 1, raw_dt);
        }
        const float last = la[kChunk - 1];
        if (OUT) {
            const int rt = warp & 3, x0 = (warp >> 2) * HT;        // this warp's 16 tokens and column tiles
            const int ra = rt * 16 + g, rb = ra + 8;
            uint32_t z[HT][2];
            const __nv_bfloat16* zrow = p.proj + m0 * p.ldp + h * p.P + p0 + x0 * 8 + t4 * 2;
#pragma unroll
            for (int x = 0; x < HT; ++x)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int r = hf ? rb : ra;
                    z[x][hf] = r < tn && (x0 + x) * 8 < pn ? *reinterpret_cast<const uint32_t*>(zrow + static_cast<long long>(r) * p.ldp + x * 8) : 0u;
                }
            float y[HT][4] = {};
            const __nv_bfloat16* crow = Cs + (rt * 16 + (mi & 1) * 8 + mr) * ldn + (mi >> 1) * 8;
            const int s_at = ((mi & 1) * 8 + mr) * ldp_s + x0 * 8 + (mi >> 1) * 8;
            const int nk = p.N16 / 16;
#pragma unroll 2
            for (int ks = 0; ks < nk; ++ks) {
                uint32_t a[4], bh[HT / 2][4], bl[HT / 2][4];
                ldmatrix4(a, crow + ks * 16);
#pragma unroll
                for (int x = 0; x < HT / 2; ++x) {
                    ldmatrix4_trans(bh[x], Sh + s_at + ks * 16 * ldp_s + x * 16);
                    ldmatrix4_trans(bl[x], Sl + s_at + ks * 16 * ldp_s + x * 16);
                }
#pragma unroll
                for (int x = 0; x < HT; ++x) mma_bf16(y[x], a, bh[x / 2][(x & 1) * 2], bh[x / 2][(x & 1) * 2 + 1]);
#pragma unroll
                for (int x = 0; x < HT; ++x) mma_bf16(y[x], a, bl[x / 2][(x & 1) * 2], bl[x / 2][(x & 1) * 2 + 1]);
            }
            const float laa = la[ra], lab = la[rb], ea = fast_exp2(laa), eb = fast_exp2(lab);
#pragma unroll
            for (int x = 0; x < HT; ++x) { y[x][0] *= ea; y[x][1] *= ea; y[x][2] *= eb; y[x][3] *= eb; }
            for (int jb = 0; jb <= rt; ++jb) {
                float gm[2][2][4] = {};                            // even and odd steps of the inner dimension
                const __nv_bfloat16* brow = Bs + (jb * 16 + (mi >> 1) * 8 + mr) * ldn + (mi & 1) * 8;
                auto step = [&](int ks, float (&acc)[2][4]) {
                    uint32_t a[4], bq[4];
                    ldmatrix4(a, crow + ks * 16);
                    ldmatrix4(bq, brow + ks * 16);
                    mma_bf16(acc[0], a, bq[0], bq[1]);
                    mma_bf16(acc[1], a, bq[2], bq[3]);
                };
#pragma unroll 2
                for (int ks = 0; ks + 1 < nk; ks += 2) { step(ks, gm[0]); step(ks + 1, gm[1]); }
                if (nk & 1) step(nk - 1, gm[0]);
                uint32_t ah[4], al[4];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const int j = jb * 16 + x * 8 + t4 * 2;
                    const float2 l = *reinterpret_cast<const float2*>(la + j), d = *reinterpret_cast<const float2*>(dtv + j);
                    float w00 = (gm[0][x][0] + gm[1][x][0]) * (fast_exp2(laa - l.x) * d.x), w01 = (gm[0][x][1] + gm[1][x][1]) * (fast_exp2(laa - l.y) * d.y);
                    float w10 = (gm[0][x][2] + gm[1][x][2]) * (fast_exp2(lab - l.x) * d.x), w11 = (gm[0][x][3] + gm[1][x][3]) * (fast_exp2(lab - l.y) * d.y);
                    if (jb == rt) {                                // the diagonal block: later tokens have no weight
                        if (j > ra) w00 = 0.f;
                        if (j + 1 > ra) w01 = 0.f;
                        if (j > rb) w10 = 0.f;
                        if (j + 1 > rb) w11 = 0.f;
                    }
                    split_hi_lo(w00, w01, ah[x * 2], al[x * 2]);
                    split_hi_lo(w10, w11, ah[x * 2 + 1], al[x * 2 + 1]);
                }
                uint32_t bx[HT / 2][4];
#pragma unroll
                for (int x = 0; x < HT / 2; ++x) ldmatrix4_trans(bx[x], xs + (jb * 16 + (mi & 1) * 8 + mr) * ldp_s + (x0 + 2 * x) * 8 + (mi >> 1) * 8);
#pragma unroll
                for (int x = 0; x < HT; ++x) mma_bf16(y[x], ah, bx[x / 2][(x & 1) * 2], bx[x / 2][(x & 1) * 2 + 1]);
#pragma unroll
                for (int x = 0; x < HT; ++x) mma_bf16(y[x], al, bx[x / 2][(x & 1) * 2], bx[x / 2][(x & 1) * 2 + 1]);
            }
            __nv_bfloat16* grow = p.gated + m0 * inner + h * p.P + p0 + x0 * 8 + t4 * 2;
#pragma unroll
            for (int x = 0; x < HT; ++x)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int r = hf ? rb : ra;
                    if (r >= tn || (x0 + x) * 8 >= pn) continue;
                    const float2 xv = Elem<__nv_bfloat16>::unpack2(*reinterpret_cast<const uint32_t*>(xs + r * ldp_s + (x0 + x) * 8 + t4 * 2));
                    const float2 zv = Elem<__nv_bfloat16>::unpack2(z[x][hf]);
                    *reinterpret_cast<uint32_t*>(grow + static_cast<long long>(r) * inner + x * 8) =
                        Elem<__nv_bfloat16>::pack2(fmaf(Dh, xv.x, y[x][hf * 2]) * silu_for<__nv_bfloat16>(zv.x), fmaf(Dh, xv.y, y[x][hf * 2 + 1]) * silu_for<__nv_bfloat16>(zv.y));
                }
            if (more) {
                __syncthreads();                    // C and the published S have been read
                copy_nb(Cs, ch + 1, col_c);
                cp_commit();
            }
        }
        if (more && warp == 7) scan_dt(ch + 1, raw_dt);
        // ---- state update ----
        const float decay = fast_exp2(last);
        log_decay += last;
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            const int n0 = (warp + 8 * i) * 16;
            if (n0 >= p.N16) break;
#pragma unroll
            for (int x = 0; x < PT; ++x)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[i][x][e] *= decay;
#pragma unroll
            for (int ks = 0; ks < kChunk / 16; ++ks) {
                uint32_t a[4], ah[4], al[4], bx[PT / 2][4];
                ldmatrix4_trans(a, Bs + (ks * 16 + (mi >> 1) * 8 + mr) * ldn + n0 + (mi & 1) * 8);
#pragma unroll
                for (int x = 0; x < PT / 2; ++x) ldmatrix4_trans(bx[x], xs + (ks * 16 + (mi & 1) * 8 + mr) * ldp_s + x * 16 + (mi >> 1) * 8);
                const float2 w0 = *reinterpret_cast<const float2*>(wv + ks * 16 + t4 * 2), w1 = *reinterpret_cast<const float2*>(wv + ks * 16 + 8 + t4 * 2);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 v = Elem<__nv_bfloat16>::unpack2(a[e]), w = e < 2 ? w0 : w1;
                    split_hi_lo(v.x * w.x, v.y * w.y, ah[e], al[e]);
                }
#pragma unroll
                for (int x = 0; x < PT; ++x) mma_bf16(S[i][x], ah, bx[x / 2][(x & 1) * 2], bx[x / 2][(x & 1) * 2 + 1]);
#pragma unroll
                for (int x = 0; x < PT; ++x) mma_bf16(S[i][x], al, bx[x / 2][(x & 1) * 2], bx[x / 2][(x & 1) * 2 + 1]);
            }
        }
        if (OUT && more) publish_state();
    }
    if (OUT && seg + 1 < p.n_seg) return;
    float* dst = OUT ? sp : p.seg_state + seg_row * p.N * p.Pp + p0;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int x = 0; x < PT; ++x)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int n = (warp + 8 * i) * 16 + g + hf * 8, c = x * 8 + t4 * 2;
                if (n < p.N && c < pn) *reinterpret_cast<float2*>(dst + static_cast<long long>(n) * p.Pp + c) = make_float2(S[i][x][hf * 2], S[i][x][hf * 2 + 1]);
            }
    if (!OUT && sl == 0 && threadIdx.x == 0) p.seg_decay[seg_row] = log_decay;
}

// seg_state[seg] <- the state every segment starts from.  grid (blocks of a head's state, H, B).
__global__ void __launch_bounds__(256)
ssd_segment_scan_kernel(ChunkParams p) {
    pdl_begin();
    const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, b = blockIdx.z, size = p.N * p.Pp;
    if (i >= size) return;
    float run = p.pos[b] > 0 ? p.state[(static_cast<long long>(p.slots ? p.slots[b] : b) * p.H + h) * size + i] : 0.f;
    for (int s = 0; s < p.n_seg; ++s) {
        const long long row = (static_cast<long long>(b) * p.n_seg + s) * p.H + h;
        const float add = s + 1 < p.n_seg ? p.seg_state[row * size + i] : 0.f;
        p.seg_state[row * size + i] = run;
        if (s + 1 < p.n_seg) run = fmaf(exp2f(p.seg_decay[row]), run, add);
    }
}

}  // namespace

bool ssd_chunk_supported(const vb200_ssd_args& a) {
    return a.dtype == VB200_BF16 && a.P % 8 == 0 && a.N % 8 == 0 && a.N <= 256 && a.ldp % 8 == 0 && a.H * ((a.P + 31) / 32) <= 65535;
}

// Column slices of a head and segments of a portion.
void plan_ssd_chunks(const vb200_ssd_args& a, int* slices, int* n_seg, int* seg_chunks) {
    const int pw = a.N <= 128 ? 64 : 32, chunks = (a.T + kChunk - 1) / kChunk;
    *slices = (a.P + pw - 1) / pw;
    const long long ctas = static_cast<long long>(a.B) * a.H * *slices;
    const bool walk = a.form != 3 && ssd_walk_supported(a);         // chunks of 128 tokens, one CTA per SM
    long long want = walk ? device_sm_count() / ctas : (2LL * device_sm_count() + ctas - 1) / ctas;
    const int unit = walk ? 4 : 2;                                   // fewest 64-token chunks of a segment
    if (want > chunks / unit) want = chunks / unit;
    if (want < 1) want = 1;
    *seg_chunks = static_cast<int>((chunks + want - 1) / want);
    if (walk) *seg_chunks = (*seg_chunks + 1) / 2 * 2;
    *n_seg = (chunks + *seg_chunks - 1) / *seg_chunks;
}

int launch_ssd_chunks(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, const void* xbc, void* gated, float* states, int* status) {
    ChunkParams p{};
    p.T = a.T; p.H = a.H; p.P = a.P; p.N = a.N; p.G = a.G; p.channels = pl.channels; p.Pp = pl.Pp; p.N16 = pad_to(a.N, 16);
    plan_ssd_chunks(a, &p.slices, &p.n_seg, &p.seg_chunks);
    p.ldp = a.ldp;
    p.proj = static_cast<const __nv_bfloat16*>(a.proj); p.xbc = static_cast<const __nv_bfloat16*>(xbc);
    p.dt_bias = a.dt_bias; p.A_log = a.A_log; p.D = a.D; p.slots = a.slots; p.pos = a.pos; p.state = a.state;
    p.seg_decay = states;
    p.seg_state = states + (static_cast<long long>(a.B) * p.n_seg * a.H + 63) / 64 * 64;
    p.gated = static_cast<__nv_bfloat16*>(gated);
    auto go = [&](auto first, auto walk, int pt) -> int {
        const size_t nb = static_cast<size_t>(kChunk) * (p.N16 + kPad), xb = static_cast<size_t>(kChunk) * (pt * 8 + kPad);
        const size_t tiles = 2 * (2 * nb + 2 * xb), all = tiles + 2 * (nb + 2 * static_cast<size_t>(p.N16) * (pt * 8 + kPad));
        const unsigned hs = static_cast<unsigned>(a.H * p.slices), bs = static_cast<unsigned>(a.B);
        if (int rc = allow_smem(first, tiles)) return rc;
        if (int rc = allow_smem(walk, all)) return rc;
        if (p.n_seg > 1) {
            if (int rc = launch_pdl(first, dim3(static_cast<unsigned>(p.n_seg - 1), hs, bs), dim3(kThreads), tiles, s, p)) return rc;
            if (int rc = launch_pdl(ssd_segment_scan_kernel, dim3(static_cast<unsigned>((a.N * p.Pp + 255) / 256), static_cast<unsigned>(a.H), bs), dim3(256), 0, s, p)) return rc;
        }
        profile_mark_begin(s);
        const int rc = a.form != 3 && ssd_walk_supported(a) ? launch_ssd_walk(s, a, pl, xbc, gated, p.seg_state, p.n_seg, p.seg_chunks, status) : launch_pdl(walk, dim3(static_cast<unsigned>(p.n_seg), hs, bs), dim3(kThreads), all, s, p);
        profile_mark_end(s);
        return rc;
    };
    note_ssd_kernel("ssd_chunk_kernel");
    return a.N <= 128 ? go(ssd_chunk_kernel<1, 8, false>, ssd_chunk_kernel<1, 8, true>, 8) : go(ssd_chunk_kernel<2, 4, false>, ssd_chunk_kernel<2, 4, true>, 4);
}

}  // namespace vb200
