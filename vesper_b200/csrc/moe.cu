// Mixture of experts: the router's choice, and the experts' products in two forms.
//   token by token (any sizes, fp32 or bf16; decode steps)   every (token, chosen expert) pair streams its expert's weights through
//                                                            CUDA cores; the shared expert is one more pair per token
//   grouped (bf16 prompts)                                   (token, expert) pairs are sorted by expert and the rows of one expert form
//                                                            128-row tiles of the tcgen05 product in linear_sm100.cu
#include "hybrid.cuh"

namespace vb200 {
namespace {

// ---- the choice: one warp per token ----
constexpr int kRouteWarps = 4;

struct Pick { float v; int i; };
__device__ __forceinline__ Pick warp_argmax(Pick a) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xFFFFFFFFu, a.v, o);
        const int i = __shfl_xor_sync(0xFFFFFFFFu, a.i, o);
        if (v > a.v || (v == a.v && i < a.i)) { a.v = v; a.i = i; }
    }
    return a;
}

// s, choice [E], group [groups]: this warp's shared memory; choice is consumed
__device__ __forceinline__ void route_token(const float* __restrict__ logits, const float* __restrict__ correction, int E, int top, int groups, int keep, float scale,
                                            float* s, float* choice, float* group, int* __restrict__ ids, float* __restrict__ weights) {
    const int lane = threadIdx.x & 31;
    for (int e = lane; e < E; e += 32) {
        const float v = 1.0f / (1.0f + expf(-logits[e]));
        s[e] = v;
        choice[e] = v + (correction != nullptr ? correction[e] : 0.f);
    }
    __syncwarp();
    if (groups > 0) {
        const int per = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;          // the two largest
            for (int i = 0; i < per; ++i) {
                const float v = choice[g * per + i];
                if (v > a) { b = a; a = v; }
                else if (v > b) b = v;
            }
            group[g] = per > 1 ? a + b : a;
        }
        __syncwarp();
        // a kept group is marked by NaN
        for (int k = 0; k < keep; ++k) {
            Pick best{-INFINITY, 0x7FFFFFFF};
            for (int g = lane; g < groups; g += 32)
                if (group[g] > best.v || (group[g] == best.v && best.i == 0x7FFFFFFF)) best = Pick{group[g], g};
            best = warp_argmax(best);
            if (lane == 0 && best.i < groups) group[best.i] = NAN;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (!isnan(group[e / per])) choice[e] = -INFINITY;
        __syncwarp();
    }
    float sum = 0.f, mine = 0.f;
    int my_id = 0;
    for (int k = 0; k < top; ++k) {
        Pick best{-INFINITY, 0x7FFFFFFF};
        for (int e = lane; e < E; e += 32)
            if (choice[e] > best.v) best = Pick{choice[e], e};
        best = warp_argmax(best);
        const int id = best.i < E ? best.i : 0;
        const float v = s[id];
        sum += v;
        if (lane == (k & 31)) { mine = v; my_id = id; }
        if (lane == 0) choice[id] = -INFINITY;
        if ((k & 31) == 31 || k + 1 == top) {            // park up to 32 picks, scaled below
            const int k0 = k & ~31;
            if (k0 + lane <= k) { ids[k0 + lane] = my_id; weights[k0 + lane] = mine; }
        }
        __syncwarp();
    }
    const float f = scale / (sum + 1e-20f);
    for (int k = lane; k < top; k += 32) weights[k] *= f;
}

__global__ void __launch_bounds__(kRouteWarps * 32)
moe_route_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ correction, int M, int E, int top, int groups, int keep, float scale, int* __restrict__ ids,
                 float* __restrict__ weights) {
    pdl_begin();
    extern __shared__ float sm[];
    const int warp = threadIdx.x >> 5, m = blockIdx.x * kRouteWarps + warp;
    if (m >= M) return;
    float* s = sm + warp * (2 * E + groups);
    route_token(logits + static_cast<long long>(m) * ld, correction, E, top, groups, keep, scale, s, s + E, s + 2 * E, ids + static_cast<long long>(m) * top,
                weights + static_cast<long long>(m) * top);
}

// ---- token by token ----
struct MoeParams {
    int M, dim, ff, ff_shared, E, top;
    long long ld_out, ld_shared;
    int act_ld;                  // activations of one (token, expert) pair
};

constexpr int kAhead = 4;        // 16-byte (fp32: 32-byte) pieces of a weight row that a lane has in flight

__device__ __forceinline__ float dot8(const float (&v)[8], const float* x, float a) {
    const float4 x0 = *reinterpret_cast<const float4*>(x), x1 = *reinterpret_cast<const float4*>(x + 4);
    a = fmaf(v[0], x0.x, fmaf(v[1], x0.y, fmaf(v[2], x0.z, fmaf(v[3], x0.w, a))));
    return fmaf(v[4], x1.x, fmaf(v[5], x1.y, fmaf(v[6], x1.z, fmaf(v[7], x1.w, a))));
}

// Warp-wide dot product of n8 pieces of eight columns with x in shared memory; row(i) is the address of piece i.
template <typename T, int ROWS, typename F>
__device__ __forceinline__ void piece_dots(int n8, const float* x, float (&sum)[ROWS], F row) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) sum[r] = 0.f;
    for (int i0 = lane; i0 < n8; i0 += 32 * kAhead) {
        Raw8<T> w[kAhead][ROWS];
#pragma unroll
        for (int u = 0; u < kAhead; ++u)
            if (i0 + 32 * u < n8) {
#pragma unroll
                for (int r = 0; r < ROWS; ++r) w[u][r].load(row(i0 + 32 * u, r));
            }
#pragma unroll
        for (int u = 0; u < kAhead; ++u)
            if (i0 + 32 * u < n8) {
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    float v[8];
                    w[u][r].get(v);
                    sum[r] = dot8(v, x + (i0 + 32 * u) * 8, sum[r]);
                }
            }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) sum[r] = warp_sum_f(sum[r]);      // every lane has them
}

constexpr int kRouterThreads = 1024;

// Router logits and choice of one token: grid M (few tokens; prompts take the product of linear_sm100.cu).
template <typename T>
__global__ void __launch_bounds__(kRouterThreads)
moe_router_kernel(const T* __restrict__ x, const T* __restrict__ w, const float* __restrict__ correction, int dim, int E, int top, int groups, int keep, float scale,
                  int* __restrict__ ids, float* __restrict__ weights) {
    pdl_begin();
    extern __shared__ __align__(16) float sm[];          // [dim] x | [E] logits | [2 E + groups] of the choice
    float* logits = sm + dim;
    const long long m = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = threadIdx.x * 8; i < dim; i += kRouterThreads * 8) {
        float v[8];
        load8(x + m * dim + i, v);
        store8(sm + i, v);
    }
    __syncthreads();
    for (int e = 2 * warp; e < E; e += kRouterThreads / 16) {
        const int second = min(e + 1, E - 1);
        float z[2];
        piece_dots<T, 2>(dim / 8, sm, z, [&](int i, int r) { return w + static_cast<long long>(r ? second : e) * dim + i * 8; });
        if (lane < 2 && e + lane < E) logits[e + lane] = z[lane];
    }
    __syncthreads();
    if (warp == 0) route_token(logits, correction, E, top, groups, keep, scale, logits + E, logits + 2 * E, logits + 3 * E, ids + m * top, weights + m * top);
}

constexpr int kPairRows = 16;    // hidden units per CTA: two per warp

// grid (ceil(max(ff, ff_shared) / kPairRows), top + (shared ? 1 : 0), M), 256 threads
template <typename T>
__global__ void __launch_bounds__(256)
moe_pair_in_kernel(MoeParams p, const T* __restrict__ x, const int* __restrict__ ids, const T* __restrict__ w_in, const T* __restrict__ w_shared, T* __restrict__ act) {
    pdl_begin();
    extern __shared__ __align__(16) float xs[];
    const int k = blockIdx.y, m = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool shared = k == p.top;
    const int ff = shared ? p.ff_shared : p.ff, j0 = blockIdx.x * kPairRows;
    if (j0 >= ff) return;
    const T* w = shared ? w_shared : w_in + static_cast<long long>(ids[m * p.top + k]) * 2 * p.ff * p.dim;
    for (int i = threadIdx.x * 8; i < p.dim; i += 256 * 8) {
        float v[8];
        load8(x + static_cast<long long>(m) * p.dim + i, v);
        store8(xs + i, v);
    }
    __syncthreads();
    T* dst = act + (static_cast<long long>(m) * (p.top + 1) + k) * p.act_ld;
    for (int j = j0 + warp; j < min(ff, j0 + kPairRows); j += 8) {
        const T* rows = w + static_cast<long long>(2 * j) * p.dim;
        float gu[2];
        piece_dots<T, 2>(p.dim / 8, xs, gu, [&](int i, int r) { return rows + r * p.dim + i * 8; });
        if (lane == 0) dst[j] = Elem<T>::from_f(silu_for<T>(gu[0]) * gu[1]);
    }
    // the padding up to a multiple of eight is multiplied with zero weights and must be finite
    if (j0 + kPairRows >= ff && threadIdx.x < 8 && ff + threadIdx.x < (ff + 7) / 8 * 8) dst[ff + threadIdx.x] = Elem<T>::from_f(0.f);
}

constexpr int kOutRows = 16;

// grid (ceil(dim / kOutRows), M), 256 threads: an output row is one dot product over the hidden units of all its token's experts, weighted ahead
template <typename T>
__global__ void __launch_bounds__(256)
moe_pair_out_kernel(MoeParams p, const int* __restrict__ ids, const float* __restrict__ weights, const T* __restrict__ w_out, const T* __restrict__ w_shared, const T* __restrict__ act,
                    float* __restrict__ y) {
    pdl_begin();
    extern __shared__ __align__(16) float as[];
    const int m = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, d0 = blockIdx.x * kOutRows;
    const int f8 = (p.ff + 7) / 8, s8 = (p.ff_shared + 7) / 8, n8 = p.top * f8 + s8;
    const T* src = act + static_cast<long long>(m) * (p.top + 1) * p.act_ld;
    for (int i = threadIdx.x; i < n8; i += 256) {
        const int k = min(i / f8, p.top), c = i - k * f8;
        const float w = k < p.top ? weights[m * p.top + k] : 1.0f;
        float v[8];
        load8(src + k * p.act_ld + c * 8, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= w;
        store8(as + i * 8, v);
    }
    __syncthreads();
    for (int d = d0 + 2 * warp; d < min(p.dim, d0 + kOutRows); d += 16) {            // two rows at a time (dim is a multiple of 8)
        float t[2];
        piece_dots<T, 2>(n8, as, t, [&](int i, int r) {
            const int k = min(i / f8, p.top), c = i - k * f8;
            return k < p.top ? w_out + (static_cast<long long>(ids[m * p.top + k]) * p.dim + d + r) * p.ld_out + c * 8 : w_shared + static_cast<long long>(d + r) * p.ld_shared + c * 8;
        });
        if (lane == 0) *reinterpret_cast<float2*>(y + static_cast<long long>(m) * p.dim + d) = make_float2(t[0], t[1]);
    }
}

// ---- grouped by expert ----
// grid E, 1024 threads: every CTA counts all pairs, then places its own expert's in their order.  gather[pair] = sorted row; token / weight of
// every sorted row; the row tiles of the grouped products.
constexpr int kSortThreads = 1024;

__global__ void __launch_bounds__(kSortThreads)
moe_sort_kernel(const int* __restrict__ ids, const float* __restrict__ weights, int pairs, int E, int* __restrict__ gather, float* __restrict__ row_weight, int4* __restrict__ tiles,
                int* __restrict__ tile_count) {
    pdl_begin();
    extern __shared__ int count[];               // [E]
    __shared__ int warp_sum[kSortThreads / 32], base[3];
    const int e = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < E; i += kSortThreads) count[i] = 0;
    __syncthreads();
    const int per = (pairs + kSortThreads - 1) / kSortThreads, i0 = min(pairs, tid * per), i1 = min(pairs, i0 + per);
    int mine = 0;
    for (int i = i0; i < i1; ++i) {
        const int id = ids[i];
        atomicAdd(&count[id], 1);
        mine += id == e;
    }
    int scan = mine;                             // inclusive over the warp
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xFFFFFFFFu, scan, o); if (lane >= o) scan += v; }
    if (lane == 31) warp_sum[warp] = scan;
    __syncthreads();
    if (warp == 0) {
        int row = 0, tile = 0, all = 0;
        for (int i = lane; i < E; i += 32) {
            const int t = (count[i] + 127) / 128;
            if (i < e) { row += count[i]; tile += t; }
            all += t;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            row += __shfl_xor_sync(0xFFFFFFFFu, row, o);
            tile += __shfl_xor_sync(0xFFFFFFFFu, tile, o);
            all += __shfl_xor_sync(0xFFFFFFFFu, all, o);
        }
        if (lane == 0) { base[0] = row; base[1] = tile; base[2] = all; }
    } else if (warp == 1) {
        const int v0 = warp_sum[lane];
        int v = v0;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const int u = __shfl_up_sync(0xFFFFFFFFu, v, o); if (lane >= o) v += u; }
        warp_sum[lane] = v - v0;
    }
    __syncthreads();
    int at = base[0] + warp_sum[warp] + scan - mine;
    for (int i = i0; i < i1; ++i)
        if (ids[i] == e) { gather[i] = at; row_weight[at] = weights[i]; ++at; }
    const int n = count[e], row_end = base[0] + n;
    for (int t = tid; t < (n + 127) / 128; t += kSortThreads) tiles[base[1] + t] = make_int4(base[0] + t * 128, row_end, e, 0);
    if (e == 0 && tid == 0) *tile_count = base[2];
}

// grid M, 128 threads: a token's row to its `top` places
__global__ void __launch_bounds__(128)
moe_scatter_rows_kernel(const uint4* __restrict__ x, const int* __restrict__ gather, int top, int n16, uint4* __restrict__ sorted) {
    pdl_begin();
    const long long m = blockIdx.x;
    for (int c = threadIdx.x; c < n16; c += 128) {
        const uint4 v = x[m * n16 + c];
        for (int k = 0; k < top; ++k) sorted[static_cast<long long>(gather[m * top + k]) * n16 + c] = v;
    }
}

int router_logits(cudaStream_t s, const vb200_moe_args& a, float* logits, int* status) {
    if (a.dtype == VB200_F32)
        return launch_linear_f32(s, static_cast<const float*>(a.x), a.dim, static_cast<const float*>(a.w_router), a.dim, nullptr, logits, pad_to(a.experts, 4), a.M, a.experts, a.dim);
    LinearParams p{};
    p.x = a.x; p.ldx = a.dim; p.w = a.w_router; p.ldw = a.dim; p.out = logits; p.ldo = pad_to(a.experts, 4); p.M = a.M; p.N = a.experts; p.K = a.dim;
    p.epilogue = VB200_EPI_F32;
    p.status = status;
    return launch_linear(s, p);
}

int launch_grouped(cudaStream_t s, const vb200_moe_args& a, const MoePlan& pl, const int* ids, const float* weights, int* status) {
    uint8_t* ws = static_cast<uint8_t*>(a.workspace);
    const int pairs = a.M * a.top;
    int *gather = reinterpret_cast<int*>(ws + pl.gather), *tile_count = reinterpret_cast<int*>(ws + pl.tiles);
    float* row_weight = reinterpret_cast<float*>(ws + pl.row_weight);
    int4* tiles = reinterpret_cast<int4*>(ws + pl.tiles + 16);
    if (int rc = launch_pdl(moe_sort_kernel, dim3(static_cast<unsigned>(a.experts)), dim3(kSortThreads), sizeof(int) * a.experts, s, ids, weights, pairs, a.experts, gather, row_weight,
                            tiles, tile_count)) return rc;
    if (int rc = launch_pdl(moe_scatter_rows_kernel, dim3(static_cast<unsigned>(a.M)), dim3(128), 0, s, static_cast<const uint4*>(a.x), static_cast<const int*>(gather), a.top, a.dim / 8,
                            reinterpret_cast<uint4*>(ws + pl.sorted_x))) return rc;
    LinearParams p{};
    p.status = status;
    p.group_tiles = tiles; p.group_tile_count = tile_count; p.group_tile_max = pl.max_tiles; p.groups = a.experts;
    p.x = ws + pl.sorted_x; p.ldx = a.dim; p.w = a.w_in; p.ldw = a.dim; p.out = ws + pl.sorted_act; p.ldo = pad_to(a.ff, 8);
    p.M = pairs; p.N = 2 * a.ff; p.K = a.dim; p.group_rows = 2 * a.ff;
    p.epilogue = VB200_EPI_SWIGLU;
    profile_mark_begin(s);
    if (int rc = launch_linear_grouped(s, p)) return rc;
    p.x = ws + pl.sorted_act; p.ldx = pad_to(a.ff, 8); p.w = a.w_out; p.ldw = a.ld_out; p.out = ws + pl.sorted_y; p.ldo = a.dim;
    p.N = a.dim; p.K = a.ff; p.group_rows = a.dim; p.row_scale = row_weight;
    p.epilogue = VB200_EPI_BF16;
    if (int rc = launch_linear_grouped(s, p)) return rc;
    profile_mark_end(s);
    note_moe_kernel("linear_wide_kernel (grouped)");
    if (a.ff_shared == 0) {
        VB200_CUDA_TRY(cudaMemsetAsync(a.y, 0, static_cast<size_t>(a.M) * a.dim * sizeof(float), s));
        return VB200_OK;
    }
    LinearParams q{};
    q.status = status;
    q.x = a.x; q.ldx = a.dim; q.w = a.w_shared_in; q.ldw = a.dim; q.out = ws + pl.shared_act; q.ldo = pad_to(a.ff_shared, 8);
    q.M = a.M; q.N = 2 * a.ff_shared; q.K = a.dim; q.epilogue = VB200_EPI_SWIGLU;
    if (int rc = launch_linear(s, q)) return rc;
    q.x = ws + pl.shared_act; q.ldx = pad_to(a.ff_shared, 8); q.w = a.w_shared_out; q.ldw = a.ld_shared; q.out = a.y; q.ldo = a.dim;
    q.N = a.dim; q.K = a.ff_shared; q.epilogue = VB200_EPI_F32;
    return launch_linear(s, q);
}

}  // namespace

MoePlan plan_moe(const vb200_moe_args& a) {
    MoePlan pl{};
    auto up = [](size_t x) { return (x + 255) / 256 * 256; };
    const size_t esz = a.dtype == VB200_F32 ? 4 : 2, M = static_cast<size_t>(a.M), pairs = M * a.top;
    size_t at = 0;
    auto take = [&](size_t bytes) { const size_t o = at; at += up(bytes); return o; };
    // sorting pays when experts are shared: token by token every pair streams an expert of its own
    pl.grouped = a.dtype == VB200_BF16 && a.form != 1 && pairs < (1u << 30) && (a.form == 2 || 4 * pairs >= 5 * static_cast<size_t>(a.experts));
    pl.max_tiles = static_cast<int>((pairs + 127) / 128) + (a.experts < static_cast<int>(pairs) ? a.experts : static_cast<int>(pairs));
    pl.logits = take(M * pad_to(a.experts, 4) * 4);
    pl.ids = take(pairs * 4);
    pl.weights = take(pairs * 4);
    if (pl.grouped) {
        pl.gather = take(pairs * 4);
        pl.row_weight = take(pairs * 4);
        pl.tiles = take(16 + static_cast<size_t>(pl.max_tiles) * 16);
        pl.sorted_x = take(pairs * a.dim * esz);
        pl.sorted_act = take(pairs * pad_to(a.ff, 8) * esz);
        pl.sorted_y = take(pairs * a.dim * esz);
        pl.shared_act = take(M * pad_to(a.ff_shared, 8) * esz);
        pl.total = at;
        return pl;
    }
    const size_t act_ld = pad_to(a.ff > a.ff_shared ? a.ff : a.ff_shared, 8);
    pl.act = take(M * (a.top + 1) * act_ld * esz);
    pl.total = at;
    return pl;
}

int launch_moe_route(cudaStream_t s, const float* logits, int ld, const float* correction, int M, int E, int top, int groups, int keep, float scale, int* ids, float* weights) {
    const size_t smem = sizeof(float) * kRouteWarps * (2 * E + groups);
    if (int rc = allow_smem(moe_route_kernel, smem)) return rc;
    return launch_pdl(moe_route_kernel, dim3(static_cast<unsigned>((M + kRouteWarps - 1) / kRouteWarps)), dim3(kRouteWarps * 32), smem, s, logits, ld, correction, M, E, top, groups, keep,
                      scale, ids, weights);
}

int launch_moe(cudaStream_t s, const vb200_moe_args& a, const MoePlan& pl, int* status) {
    uint8_t* ws = static_cast<uint8_t*>(a.workspace);
    float *logits = reinterpret_cast<float*>(ws + pl.logits), *weights = reinterpret_cast<float*>(ws + pl.weights);
    int* ids = reinterpret_cast<int*>(ws + pl.ids);
    const size_t router_smem = sizeof(float) * (static_cast<size_t>(a.dim) + 3 * a.experts + a.groups);
    if (a.M <= 32 && router_smem <= 100 * 1024) {
        auto router = [&](auto tag) -> int {
            using T = decltype(tag);
            if (int rc = allow_smem(moe_router_kernel<T>, router_smem)) return rc;
            return launch_pdl(moe_router_kernel<T>, dim3(static_cast<unsigned>(a.M)), dim3(kRouterThreads), router_smem, s, static_cast<const T*>(a.x), static_cast<const T*>(a.w_router), a.correction,
                              a.dim, a.experts, a.top, a.groups, a.keep, a.scale, ids, weights);
        };
        if (int rc = a.dtype == VB200_F32 ? router(float{}) : router(__nv_bfloat16{})) return rc;
    } else {
        if (int rc = router_logits(s, a, logits, status)) return rc;
        if (int rc = launch_moe_route(s, logits, pad_to(a.experts, 4), a.correction, a.M, a.experts, a.top, a.groups, a.keep, a.scale, ids, weights)) return rc;
    }
    if (pl.grouped) return launch_grouped(s, a, pl, ids, weights, status);
    MoeParams p{};
    p.M = a.M; p.dim = a.dim; p.ff = a.ff; p.ff_shared = a.ff_shared; p.E = a.experts; p.top = a.top; p.ld_out = a.ld_out; p.ld_shared = a.ld_shared;
    p.act_ld = pad_to(a.ff > a.ff_shared ? a.ff : a.ff_shared, 8);
    auto go = [&](auto tag) -> int {
        using T = decltype(tag);
        T* act = reinterpret_cast<T*>(ws + pl.act);
        const int widest = a.ff > a.ff_shared ? a.ff : a.ff_shared;
        const size_t smem_in = sizeof(float) * a.dim, smem_out = sizeof(float) * (static_cast<size_t>(a.top) * pad_to(a.ff, 8) + pad_to(a.ff_shared, 8));
        if (int rc = allow_smem(moe_pair_in_kernel<T>, smem_in)) return rc;
        if (int rc = allow_smem(moe_pair_out_kernel<T>, smem_out)) return rc;
        profile_mark_begin(s);
        // grid z is limited to 65535 tokens: longer prompts go in slices
        for (int m0 = 0; m0 < a.M; m0 += 65535) {
            const int n = a.M - m0 < 65535 ? a.M - m0 : 65535;
            T* act0 = act + static_cast<size_t>(m0) * (a.top + 1) * p.act_ld;
            if (int rc = launch_pdl(moe_pair_in_kernel<T>, dim3(static_cast<unsigned>((widest + kPairRows - 1) / kPairRows), static_cast<unsigned>(a.top + (a.ff_shared > 0)), static_cast<unsigned>(n)),
                                    dim3(256), smem_in, s, p, static_cast<const T*>(a.x) + static_cast<size_t>(m0) * a.dim, ids + static_cast<size_t>(m0) * a.top,
                                    static_cast<const T*>(a.w_in), static_cast<const T*>(a.w_shared_in), act0)) return rc;
            if (int rc = launch_pdl(moe_pair_out_kernel<T>, dim3(static_cast<unsigned>((a.dim + kOutRows - 1) / kOutRows), static_cast<unsigned>(n)), dim3(256), smem_out, s, p,
                                    ids + static_cast<size_t>(m0) * a.top, weights + static_cast<size_t>(m0) * a.top, static_cast<const T*>(a.w_out),
                                    static_cast<const T*>(a.w_shared_out), act0, a.y + static_cast<size_t>(m0) * a.dim)) return rc;
        }
        profile_mark_end(s);
        note_moe_kernel("moe_pair_in_kernel");
        return VB200_OK;
    };
    return a.dtype == VB200_F32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // namespace vb200
