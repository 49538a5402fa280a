// Shared pieces of the hybrid-decoder kernels (latent attention, Mamba-2, sequence operators).
#pragma once

#include "kernels.h"
#include "../../include/vesper_b200_hybrid.h"

namespace vb200 {

constexpr float kLog2e = 1.4426950408889634f;

// Launch with the programmatic-dependent-launch attribute; the kernel starts with pdl_begin().
template <typename... KArgs, typename... Args>
int launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    VB200_CUDA_TRY(cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...));
    note_launch();
    return VB200_OK;
}

// Raises a kernel's dynamic shared memory limit (a no-op below the 48 KB default).
template <typename Kernel>
int allow_smem(Kernel kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return VB200_OK;
    VB200_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
    return VB200_OK;
}

// bf16 4-D tensor map (c, h, row, batch) over strided memory (strides in elements), box [64 c][1][box_rows][1], 128-byte
// swizzle; reads past an extent return zeros.  Base and strides must be multiples of 16 bytes.
int make_map_4d(CUtensorMap* m, const void* ptr, int c, int heads, long long rows, int batch, long long head_stride, long long row_stride, long long batch_stride,
                int box_rows);                   // api_hybrid.cu
int device_sm_count();                           // api_hybrid.cu
void note_latent_kernel(const char* name);
void note_ssd_kernel(const char* name);

// ---- sequence_ops.cu ----
int launch_embed_sequence(cudaStream_t s, const vb200_embed_args& a, int* status);
int launch_residual_add(cudaStream_t s, float* h, const float* addend, const float* vec, int M, int dim, const float* scale, void* scaled_out);
int launch_norm_add(cudaStream_t s, const vb200_norm_add_args& a);
int launch_rms_norm_f32(cudaStream_t s, const float* x, const float* w, float* out, int M, int dim, int count, float eps);

// ---- latent attention ----
inline int pad_to(int x, int m) { return (x + m - 1) / m * m; }
// Split plan and workspace of a decode step: absorbed queries [B, H, qld] fp32, then per (row, head, split) the
// unnormalised latent sum [rank16], the reference maximum (log2 units) and the sum of weights.
struct LatentPlan {
    int n_max;          // keys a row can have
    int splits;
    int rank16, rot16, qld, part_ld;
    size_t q_floats, part_floats;
};
LatentPlan plan_latent(const vb200_latent_args& a);
bool latent_mma_supported(const vb200_latent_args& a);
bool latent_sm100_supported(const vb200_latent_args& a);
int launch_latent_append(cudaStream_t s, const vb200_latent_args& a);
int launch_latent_prefill_generic(cudaStream_t s, const vb200_latent_args& a);
int launch_latent_prefill_sm100(cudaStream_t s, const vb200_latent_args& a, int* status);       // latent_prefill_sm100.cu
int launch_latent_decode(cudaStream_t s, const vb200_latent_args& a, int* status);
int launch_latent_split_mma(cudaStream_t s, const vb200_latent_args& a, const LatentPlan& pl, const float* q, float* part, int* status);   // latent_decode_mma.cu

// ---- causal depthwise convolution + silu, shared by the state-space mixers (ssd_scan.cu) ----
struct ConvLaunch {
    int dtype, B, T, channels, taps;
    const void* proj; long long ldp, col;        // the channels start at column `col` of a projection row
    const float *w, *b;                          // [channels, taps], [channels]
    const int *slots, *pos;
    void* state;                                 // [slots, taps, channels], input of position p in row p mod taps
    void* out;                                   // [B*T, channels]
};
int launch_causal_conv(cudaStream_t s, const ConvLaunch& c);

// ---- Mamba-2 ----
struct SsdPlan {
    int channels, Pp;
    bool chunked;
    size_t conv_bytes, gated_bytes, chunk_bytes, total;     // conv output | gated y | chunk states
};
SsdPlan plan_ssd(const vb200_ssd_args& a);
bool ssd_chunk_supported(const vb200_ssd_args& a);
void plan_ssd_chunks(const vb200_ssd_args& a, int* slices, int* n_seg, int* seg_chunks);          // ssd_chunk.cu
int launch_ssd(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, int* status);
int launch_ssd_chunks(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, const void* xbc, void* gated, float* states, int* status);   // ssd_chunk.cu
bool ssd_walk_supported(const vb200_ssd_args& a);                                                     // ssd_walk_sm100.cu
int launch_ssd_walk(cudaStream_t s, const vb200_ssd_args& a, const SsdPlan& pl, const void* xbc, void* gated, const float* seg_state, int n_seg, int seg_chunks64, int* status);

// ---- sigmoid attention with mixed heads ----
struct SigPlan {
    bool mma;                    // tensor-core kernel for this step (q' in bf16), else CUDA cores (q' in fp32)
    int splits;                  // of a decode step
    int qld;                     // columns of a q' row: G * dim padded to 16
    size_t q_bytes, part_bytes, total;
};
SigPlan plan_sigattn(const vb200_sigattn_args& a);
int launch_sigattn(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, int* status);
bool sig_prefill_sm100_supported(const vb200_sigattn_args& a);                                                                  // sigmoid_prefill_sm100.cu
int launch_sig_prefill_sm100(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, const void* q, int* status);
bool sig_decode_mma_supported(const vb200_sigattn_args& a);                                                                     // sigmoid_decode_mma.cu
int sig_decode_ctas_per_sm(const vb200_sigattn_args& a);
int launch_sig_decode_mma(cudaStream_t s, const vb200_sigattn_args& a, const SigPlan& pl, const void* q, float* part, int* status);
void note_sigattn_kernel(const char* name);

// ---- selective scan ----
struct SelectivePlan {
    bool dt_gemm;                // step sizes by a product of their own (prompts), else inside the scan kernel
    size_t conv_bytes, xdbl_bytes, dt_bytes, total;
};
SelectivePlan plan_selective(const vb200_selective_args& a);
int launch_selective(cudaStream_t s, const vb200_selective_args& a, const SelectivePlan& pl, int* status);
void note_selective_kernel(const char* name);

// ---- mixture of experts ----
struct MoePlan {
    bool grouped;                // sorted by expert, tcgen05 products; else token by token on CUDA cores
    int max_tiles;               // 128-row tiles the sorted rows can need
    size_t logits, ids, weights, act, sorted_x, sorted_act, sorted_y, gather, row_weight, tiles, shared_act, total;      // byte offsets
};
MoePlan plan_moe(const vb200_moe_args& a);
int launch_moe(cudaStream_t s, const vb200_moe_args& a, const MoePlan& pl, int* status);
int launch_moe_route(cudaStream_t s, const float* logits, int ld, const float* correction, int M, int E, int top, int groups, int keep, float scale, int* ids, float* weights);
void note_moe_kernel(const char* name);

#ifdef __CUDACC__
// Programmatic dependent launch: let the next kernel be scheduled, then wait for the previous one's results.
__device__ __forceinline__ void pdl_begin() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
}
__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max_f(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, o));
    return v;
}
// Sum over a CTA of W warps; `part` holds W floats and may be reused after the next barrier.
template <int W>
__device__ __forceinline__ float block_sum(float v, float* part) {
    v = warp_sum_f(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < W; ++i) t += part[i];
    return t;
}
__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }
// fp32 all the way in the fp32 form; the approximate exponential and division (a few ulp) where the result becomes bf16
template <typename T> __device__ __forceinline__ float silu_for(float x) {
    if constexpr (sizeof(T) == 4) return silu_exact(x);
    else return __fdividef(x, 1.0f + __expf(-x));
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// cos / sin of position * f: the product and the reduction to one turn in fp64, the functions in fp32.
__device__ __forceinline__ float2 rope_cs(int position, double f) {
    const double turns = static_cast<double>(position) * f * 0.15915494309189533577;
    const float r = static_cast<float>((turns - rint(turns)) * 6.283185307179586476925);
    float s, c;
    sincosf(r, &s, &c);
    return make_float2(c, s);
}
// eight consecutive elements (16-byte aligned for bf16, 32 for fp32)
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = Elem<__nv_bfloat16>::unpack2(w[i]);
        v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 u;
    u.x = Elem<__nv_bfloat16>::pack2(v[0], v[1]); u.y = Elem<__nv_bfloat16>::pack2(v[2], v[3]);
    u.z = Elem<__nv_bfloat16>::pack2(v[4], v[5]); u.w = Elem<__nv_bfloat16>::pack2(v[6], v[7]);
    *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
// eight elements as loaded, to be unpacked later
template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> {
    uint4 u;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { u = __ldg(reinterpret_cast<const uint4*>(p)); }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = Elem<__nv_bfloat16>::unpack2(w[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
};
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = __ldg(reinterpret_cast<const float4*>(p)); b = __ldg(reinterpret_cast<const float4*>(p + 4)); }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
};
// x = hi + lo with both halves bf16 (16 of fp32's 24 significand bits): an fp32 operand of a bf16 tensor-core product
__device__ __forceinline__ void split_hi_lo(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = Elem<__nv_bfloat16>::pack2(x, y);
    const float2 h = Elem<__nv_bfloat16>::unpack2(hi);
    lo = Elem<__nv_bfloat16>::pack2(x - h.x, y - h.y);
}
#endif

}  // namespace vb200
