// extern "C" entry points of vesper_b200_hybrid.h: argument validation and orchestration.
#include "hybrid.cuh"

#include <cstdio>

namespace vb200 {

namespace {
thread_local const char* t_latent_kernel = "";
thread_local const char* t_ssd_kernel = "";
thread_local const char *t_sigattn_kernel = "", *t_selective_kernel = "", *t_moe_kernel = "";
bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }
bool dtype_ok(int d) { return d == VB200_F32 || d == VB200_BF16; }
}  // namespace

void note_latent_kernel(const char* name) { t_latent_kernel = name; }
void note_ssd_kernel(const char* name) { t_ssd_kernel = name; }
void note_sigattn_kernel(const char* name) { t_sigattn_kernel = name; }
void note_selective_kernel(const char* name) { t_selective_kernel = name; }
void note_moe_kernel(const char* name) { t_moe_kernel = name; }

// Streaming multiprocessors of the current device (148 where no device answers: workspace sizes on a machine without a GPU).
int device_sm_count() {
    static int cache[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) { (void)cudaGetLastError(); return 148; }
    if (cache[dev] == 0) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) { (void)cudaGetLastError(); n = 148; }
        cache[dev] = n;
    }
    return cache[dev];
}

int make_map_4d(CUtensorMap* m, const void* ptr, int c, int heads, long long rows, int batch, long long head_stride, long long row_stride, long long batch_stride,
                int box_rows) {
    using Encode = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                                CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static Encode encode = []() -> Encode {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) return nullptr;
        return reinterpret_cast<Encode>(fn);
    }();
    if (!encode) return set_detail(VB200_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
    const cuuint64_t dims[4] = {static_cast<cuuint64_t>(c), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows), static_cast<cuuint64_t>(batch)};
    const cuuint64_t strides[3] = {static_cast<cuuint64_t>(head_stride) * 2, static_cast<cuuint64_t>(row_stride) * 2, static_cast<cuuint64_t>(batch_stride) * 2};
    const cuuint32_t box[4] = {64, 1, static_cast<cuuint32_t>(box_rows), 1};
    const cuuint32_t es[4] = {1, 1, 1, 1};
    const CUresult r = encode(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        static thread_local char buf[96];
        snprintf(buf, sizeof(buf), "cuTensorMapEncodeTiled failed with CUresult %d", static_cast<int>(r));
        return set_detail(VB200_ERR_CUDA, buf);
    }
    return VB200_OK;
}

namespace {

int validate_latent(const vb200_latent_args* a, const char* who) {
    if (!a || a->struct_size != sizeof(vb200_latent_args)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_args: null or struct_size mismatch");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_latent: dtype must be bf16 or fp32");
    if (a->B <= 0 || a->T <= 0 || a->H <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->rot_dim % 2 != 0 || a->vdim <= 0 || a->rank <= 0 || a->window <= 0 || a->ring <= 0)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent: sizes must be positive and rot_dim even");
    if (a->rank > 2048 || a->rot_dim > 1024 || a->dim > 1024 || a->vdim > 1024) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_latent: rank above 2048 or a head size above 1024");
    if (a->H > 65535 || a->B > 65535) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_latent: more than 65535 heads or rows");
    if (a->start_pos < 0 || !a->pos || !a->proj || !a->c_norm || !a->cache || (a->rot_dim > 0 && !a->inv_freq)) return set_detail(VB200_ERR_INVALID_ARG, who);
    const int64_t width = static_cast<int64_t>(a->H) * (a->dim + a->rot_dim) + a->rank + a->rot_dim;
    if (a->ldp < width || a->ldc != vb200_latent_row(a->rank, a->rot_dim)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent: a row stride does not hold its row");
    if (!aligned16(a->proj) || !aligned16(a->cache)) return set_detail(VB200_ERR_ALIGNMENT, "vb200_latent: 16-byte alignment required");
    return VB200_OK;
}

}  // namespace
}  // namespace vb200

using namespace vb200;

extern "C" {

int vb200_embed_sequence(const vb200_embed_args* a) {
    if (!a || a->struct_size != sizeof(vb200_embed_args)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_embed_args: null or struct_size mismatch");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_embed_sequence: dtype must be bf16 or fp32");
    if (!a->ids || !a->table || !a->lens || !a->step_pos || !a->prev || !a->h || a->B <= 0 || a->T <= 0 || a->dim <= 0 || a->vocab <= 0)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_embed_sequence: null pointer or non-positive size");
    if (a->bigram && a->buckets <= 0) return set_detail(VB200_ERR_INVALID_ARG, "vb200_embed_sequence: a bigram table needs buckets > 0");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_embed_sequence(static_cast<cudaStream_t>(a->stream), *a, status);
}

int vb200_residual_add(int device, void* stream, float* h, const float* addend, const float* vec, int32_t M, int32_t dim,
                       const float* scale, void* scaled_out) {
    if (!h || M <= 0 || dim <= 0 || (scaled_out && !scale)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_residual_add: bad arguments");
    DeviceGuard g;
    if (int rc = g.init(device)) return rc;
    return launch_residual_add(static_cast<cudaStream_t>(stream), h, addend, vec, M, dim, scale, scaled_out);
}

int vb200_rms_norm_f32(int device, void* stream, const float* x, const float* w, float* out, int32_t M, int32_t dim, int32_t count, float eps) {
    if (!x || !w || !out || M <= 0 || dim <= 0 || count <= 0 || count > dim) return set_detail(VB200_ERR_INVALID_ARG, "vb200_rms_norm_f32: bad arguments");
    DeviceGuard g;
    if (int rc = g.init(device)) return rc;
    return launch_rms_norm_f32(static_cast<cudaStream_t>(stream), x, w, out, M, dim, count, eps);
}

int vb200_linear_f32_ex(int device, void* stream, const float* x, int64_t ldx, const float* w, int64_t ldw, const float* bias,
                        const float* addend, float* out, int64_t ldo, int32_t M, int32_t N, int32_t K, int32_t epilogue) {
    if (!x || !w || !out || M <= 0 || N <= 0 || K <= 0) return set_detail(VB200_ERR_INVALID_ARG, "vb200_linear_f32_ex: null pointer or non-positive size");
    const bool gated = epilogue == VB200_EPI_SWIGLU || epilogue == VB200_EPI_REGLU;
    if (ldx < K || ldw < K || ldo < (gated ? N / 2 : N)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_linear_f32_ex: a row stride is smaller than its row");
    if (gated && (N % 2 != 0 || addend)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_linear_f32_ex: a gated epilogue needs an even N and takes no addend");
    if (!gated && epilogue != VB200_EPI_F32 && epilogue != VB200_EPI_ADD_F32 && epilogue != VB200_EPI_RELU2)
        return set_detail(VB200_ERR_UNSUPPORTED, "vb200_linear_f32_ex: epilogue not available in fp32");
    DeviceGuard g;
    if (int rc = g.init(device)) return rc;
    return launch_linear_f32(static_cast<cudaStream_t>(stream), x, ldx, w, ldw, bias, out, ldo, M, N, K, epilogue, addend);
}

size_t vb200_latent_workspace_bytes(const vb200_latent_args* a) {
    if (!a || a->struct_size != sizeof(vb200_latent_args) || a->B <= 0 || a->H <= 0 || a->rank <= 0 || a->ring <= 0) return 0;
    const LatentPlan pl = plan_latent(*a);
    return ((pl.q_floats + 63) / 64 * 64 + pl.part_floats) * sizeof(float);
}

int vb200_latent_append(const vb200_latent_args* a) {
    if (int rc = validate_latent(a, "vb200_latent_append: null pointer or negative start_pos")) return rc;
    if (!a->ctx_latent || !aligned16(a->ctx_latent)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_append: ctx_latent must be given and 16-byte aligned");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    return launch_latent_append(static_cast<cudaStream_t>(a->stream), *a);
}

int vb200_latent_prefill(const vb200_latent_args* a) {
    if (int rc = validate_latent(a, "vb200_latent_prefill: null pointer or negative start_pos")) return rc;
    if (!a->ctx_latent || !a->ctx_kv || !a->out) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_prefill: null pointer");
    if (a->ldkv < static_cast<int64_t>(a->H) * (a->dim + a->vdim) || a->ldo < static_cast<int64_t>(a->H) * a->vdim)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_prefill: a row stride does not hold its row");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    cudaStream_t s = static_cast<cudaStream_t>(a->stream);
    profile_mark_begin(s);
    const bool tuned = latent_sm100_supported(*a);
    const int rc = tuned ? launch_latent_prefill_sm100(s, *a, status) : launch_latent_prefill_generic(s, *a);
    note_latent_kernel(tuned ? "latent_prefill_sm100_kernel" : "latent_prefill_generic_kernel");
    profile_mark_end(s);
    return rc;
}

int vb200_latent_decode(const vb200_latent_args* a) {
    if (int rc = validate_latent(a, "vb200_latent_decode: null pointer or negative start_pos")) return rc;
    if (a->T != 1) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_decode: one token per row");
    if (!a->w_uk || !a->w_uv || !a->out) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_decode: null pointer");
    if (a->ldu % 8 != 0 || a->ldu < a->rank || !aligned16(a->w_uk) || !aligned16(a->w_uv))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_latent_decode: ldu must be a multiple of 8 that holds a latent, the weights 16-byte aligned");
    if (a->ldo < static_cast<int64_t>(a->H) * a->vdim) return set_detail(VB200_ERR_INVALID_ARG, "vb200_latent_decode: ldo smaller than the output row");
    if (!a->workspace || a->workspace_bytes < vb200_latent_workspace_bytes(a)) return set_detail(VB200_ERR_WORKSPACE, "vb200_latent_decode: workspace too small");
    if (!aligned16(a->workspace)) return set_detail(VB200_ERR_ALIGNMENT, "vb200_latent_decode: workspace must be 16-byte aligned");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_latent_decode(static_cast<cudaStream_t>(a->stream), *a, status);
}

const char* vb200_last_latent_kernel(void) { return t_latent_kernel; }

static bool ssd_sizes_ok(const vb200_ssd_args* a) {
    return a && a->struct_size == sizeof(vb200_ssd_args) && a->B > 0 && a->T > 0 && a->H > 0 && a->P > 0 && a->N > 0 && a->G > 0 && a->taps > 0 && a->norm_groups > 0;
}

size_t vb200_ssd_workspace_bytes(const vb200_ssd_args* a) { return ssd_sizes_ok(a) ? plan_ssd(*a).total : 0; }

int vb200_ssd_forward(const vb200_ssd_args* a) {
    if (!ssd_sizes_ok(a)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_ssd_args: null, struct_size mismatch or non-positive size");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_ssd_forward: dtype must be bf16 or fp32");
    if (a->H % a->G != 0 || (static_cast<int64_t>(a->H) * a->P) % a->norm_groups != 0)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_ssd_forward: heads must divide into the groups, inner into the norm groups");
    if (a->taps > 32) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_ssd_forward: more than 32 convolution taps");
    if (a->B > 65535 || static_cast<int64_t>(a->B) * a->T > 65535LL * 1024) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_ssd_forward: batch too large");
    if (!a->proj || !a->conv_w || !a->conv_b || !a->dt_bias || !a->A_log || !a->D || !a->norm_w || !a->pos || !a->conv_state || !a->state || !a->out)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_ssd_forward: null pointer");
    const int64_t inner = static_cast<int64_t>(a->H) * a->P;
    if (a->ldp < 2 * inner + 2LL * a->G * a->N + a->H || a->ldo < inner) return set_detail(VB200_ERR_INVALID_ARG, "vb200_ssd_forward: a row stride does not hold its row");
    if (!aligned16(a->proj) || !aligned16(a->conv_state) || !aligned16(a->state) || !aligned16(a->workspace))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_ssd_forward: 16-byte alignment required");
    const SsdPlan pl = plan_ssd(*a);
    if (!a->workspace || a->workspace_bytes < pl.total) return set_detail(VB200_ERR_WORKSPACE, "vb200_ssd_forward: workspace too small");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_ssd(static_cast<cudaStream_t>(a->stream), *a, pl, status);
}

const char* vb200_last_ssd_kernel(void) { return t_ssd_kernel; }

int vb200_norm_add(const vb200_norm_add_args* a) {
    if (!a || a->struct_size != sizeof(vb200_norm_add_args)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_norm_add_args: null or struct_size mismatch");
    if (!a->x || !a->w || (!a->y && !a->gather) || (a->gather && (!a->rows || a->n_gather <= 0)) || a->M <= 0 || a->dim <= 0 || a->count <= 0 || a->count > a->dim)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_norm_add: bad arguments");
    if (a->dim % 4 != 0 || !aligned16(a->x) || !aligned16(a->y) || !aligned16(a->w) || !aligned16(a->rows) || !aligned16(a->scale) || !aligned16(a->copy_out))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_norm_add: dim must be a multiple of 4, pointers 16-byte aligned");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    return launch_norm_add(static_cast<cudaStream_t>(a->stream), *a);
}

static bool sigattn_sizes_ok(const vb200_sigattn_args* a) {
    return a && a->struct_size == sizeof(vb200_sigattn_args) && a->B > 0 && a->T > 0 && a->H > 0 && a->G > 0 && a->dim > 0 && a->vdim > 0 && a->cap > 0 && a->H % a->G == 0 &&
           a->n_bias > 0;
}

size_t vb200_sigattn_workspace_bytes(const vb200_sigattn_args* a) { return sigattn_sizes_ok(a) ? plan_sigattn(*a).total : 0; }

int vb200_sigattn_forward(const vb200_sigattn_args* a) {
    if (!sigattn_sizes_ok(a)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_sigattn_args: null, struct_size mismatch, non-positive size or heads not divisible by kv heads");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_sigattn_forward: dtype must be bf16 or fp32");
    if (static_cast<int64_t>(a->H) * (a->dim + a->H) > 48 * 1024 || 4LL * (static_cast<int64_t>(a->G) * a->dim + a->vdim) > 48 * 1024)
        return set_detail(VB200_ERR_UNSUPPORTED, "vb200_sigattn_forward: heads * (dim + heads) above 48 K, or kv_heads * dim + vdim above 12 K");
    if (a->B > 65535 || (static_cast<int64_t>(a->T) + 3) / 4 * a->H > 65535) {
        if (a->B > 65535 || a->dtype == VB200_F32 || a->form == 1 || !plan_sigattn(*a).mma)
            return set_detail(VB200_ERR_UNSUPPORTED, "vb200_sigattn_forward: too many rows for one call");
    }
    if (!a->proj || !a->talk || !a->bias || !a->pos || !a->k_cache || !a->v_cache || !a->out || a->start_pos < 0 || a->temp_every < 0)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_sigattn_forward: null pointer or negative position");
    if (a->value_role < 0 || a->value_role > 2 || (a->value_role > 0 && !a->first_values)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_sigattn_forward: value mixing needs first_values");
    if (a->ldp < static_cast<int64_t>(a->H) * (a->dim + 1) + static_cast<int64_t>(a->G) * (a->dim + a->vdim) || a->ldk < static_cast<int64_t>(a->G) * a->dim ||
        a->ldv < static_cast<int64_t>(a->G) * a->vdim || a->ldo < static_cast<int64_t>(a->H) * a->vdim)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_sigattn_forward: a row stride does not hold its row");
    if (a->ldk % 8 != 0 || a->ldv % 8 != 0 || !aligned16(a->k_cache) || !aligned16(a->v_cache) || !aligned16(a->workspace))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_sigattn_forward: cache rows must be multiples of 8 elements, pointers 16-byte aligned");
    const SigPlan pl = plan_sigattn(*a);
    if (!a->workspace || a->workspace_bytes < pl.total) return set_detail(VB200_ERR_WORKSPACE, "vb200_sigattn_forward: workspace too small");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_sigattn(static_cast<cudaStream_t>(a->stream), *a, pl, status);
}

const char* vb200_last_sigattn_kernel(void) { return t_sigattn_kernel; }

static bool selective_sizes_ok(const vb200_selective_args* a) {
    return a && a->struct_size == sizeof(vb200_selective_args) && a->B > 0 && a->T > 0 && a->inner > 0 && a->N > 0 && a->rank > 0 && a->taps > 0;
}

size_t vb200_selective_workspace_bytes(const vb200_selective_args* a) { return selective_sizes_ok(a) ? plan_selective(*a).total : 0; }

int vb200_selective_forward(const vb200_selective_args* a) {
    if (!selective_sizes_ok(a)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_selective_args: null, struct_size mismatch or non-positive size");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_selective_forward: dtype must be bf16 or fp32");
    if (a->inner % 8 != 0 || a->N % 8 != 0 || a->rank % 8 != 0) return set_detail(VB200_ERR_ALIGNMENT, "vb200_selective_forward: inner, N and rank must be multiples of 8");
    if (a->N > 512 || a->taps > 32 || a->rank + 2 * a->N > 6 * 1024) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_selective_forward: more than 512 states, 32 taps, or too large a rank");
    if (a->B > 65535 || static_cast<int64_t>(a->T) > 65535LL * 32) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_selective_forward: batch too large");
    if (!a->proj || !a->conv_w || !a->conv_b || !a->w_x || !a->w_dt || !a->dt_bias || !a->A || !a->D || !a->pos || !a->conv_state || !a->state || !a->out)
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_selective_forward: null pointer");
    if (a->ldp < 2LL * a->inner || a->ldo < a->inner) return set_detail(VB200_ERR_INVALID_ARG, "vb200_selective_forward: a row stride does not hold its row");
    if (a->ldp % 8 != 0 || a->ldo % 8 != 0 || !aligned16(a->proj) || !aligned16(a->w_x) || !aligned16(a->w_dt) || !aligned16(a->A) || !aligned16(a->conv_state) || !aligned16(a->state) ||
        !aligned16(a->out) || !aligned16(a->workspace))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_selective_forward: row strides must be multiples of 8, pointers 16-byte aligned");
    const SelectivePlan pl = plan_selective(*a);
    if (!a->workspace || a->workspace_bytes < pl.total) return set_detail(VB200_ERR_WORKSPACE, "vb200_selective_forward: workspace too small");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_selective(static_cast<cudaStream_t>(a->stream), *a, pl, status);
}

const char* vb200_last_selective_kernel(void) { return t_selective_kernel; }

static bool choice_ok(int32_t experts, int32_t top, int32_t groups, int32_t keep) {
    if (experts <= 0 || experts > 1024 || top <= 0 || top > experts || groups < 0) return false;
    return groups == 0 || (experts % groups == 0 && keep > 0 && keep <= groups && top <= keep * (experts / groups));
}
static bool moe_sizes_ok(const vb200_moe_args* a) {
    return a && a->struct_size == sizeof(vb200_moe_args) && a->M > 0 && a->dim > 0 && a->ff > 0 && a->ff_shared >= 0 && choice_ok(a->experts, a->top, a->groups, a->keep);
}

size_t vb200_moe_workspace_bytes(const vb200_moe_args* a) { return moe_sizes_ok(a) ? plan_moe(*a).total : 0; }
int32_t vb200_moe_rows(const vb200_moe_args* a) { return moe_sizes_ok(a) && plan_moe(*a).grouped ? a->top : 0; }
int vb200_moe_rows_of(const vb200_moe_args* a, const void** rows, const int32_t** gather) {
    if (!moe_sizes_ok(a) || !rows || !gather || !a->workspace) return set_detail(VB200_ERR_INVALID_ARG, "vb200_moe_rows_of: bad arguments");
    const MoePlan pl = plan_moe(*a);
    if (!pl.grouped) return set_detail(VB200_ERR_INVALID_ARG, "vb200_moe_rows_of: this call leaves no rows");
    *rows = static_cast<const uint8_t*>(a->workspace) + pl.sorted_y;
    *gather = reinterpret_cast<const int32_t*>(static_cast<const uint8_t*>(a->workspace) + pl.gather);
    return VB200_OK;
}

int vb200_moe_forward(const vb200_moe_args* a) {
    if (!moe_sizes_ok(a)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_moe_args: null, struct_size mismatch, or sizes that do not fit together (at most 1024 experts)");
    if (!dtype_ok(a->dtype)) return set_detail(VB200_ERR_UNSUPPORTED, "vb200_moe_forward: dtype must be bf16 or fp32");
    if (!a->x || !a->w_router || !a->w_in || !a->w_out || !a->y || (a->ff_shared > 0 && (!a->w_shared_in || !a->w_shared_out)))
        return set_detail(VB200_ERR_INVALID_ARG, "vb200_moe_forward: null pointer");
    if (a->dim % 8 != 0 || a->ld_out % 8 != 0 || a->ld_out < a->ff || (a->ff_shared > 0 && (a->ld_shared % 8 != 0 || a->ld_shared < a->ff_shared)) || !aligned16(a->x) ||
        !aligned16(a->w_router) || !aligned16(a->w_in) || !aligned16(a->w_out) || !aligned16(a->w_shared_in) || !aligned16(a->w_shared_out) || !aligned16(a->y) || !aligned16(a->workspace))
        return set_detail(VB200_ERR_ALIGNMENT, "vb200_moe_forward: dim and row strides must be multiples of 8, pointers 16-byte aligned");
    if (4LL * a->dim > 200 * 1024 || 4LL * (static_cast<int64_t>(a->top) * (a->ff + 7) + a->ff_shared + 7) > 200 * 1024)
        return set_detail(VB200_ERR_UNSUPPORTED, "vb200_moe_forward: a token's row or hidden units above 200 KB");
    const MoePlan pl = plan_moe(*a);
    if (!a->workspace || a->workspace_bytes < pl.total) return set_detail(VB200_ERR_WORKSPACE, "vb200_moe_forward: workspace too small");
    DeviceGuard g;
    if (int rc = g.init(a->device)) return rc;
    int* status = kernel_status_word();
    if (!status) return VB200_ERR_CUDA;
    return launch_moe(static_cast<cudaStream_t>(a->stream), *a, pl, status);
}

int vb200_moe_route(int device, void* stream, const float* logits, const float* correction, int32_t M, int32_t experts, int32_t top, int32_t groups, int32_t keep,
                    float scale, int32_t* ids, float* weights) {
    if (!logits || !ids || !weights || M <= 0 || !choice_ok(experts, top, groups, keep)) return set_detail(VB200_ERR_INVALID_ARG, "vb200_moe_route: bad arguments");
    DeviceGuard g;
    if (int rc = g.init(device)) return rc;
    return launch_moe_route(static_cast<cudaStream_t>(stream), logits, experts, correction, M, experts, top, groups, keep, scale, ids, weights);
}

const char* vb200_last_moe_kernel(void) { return t_moe_kernel; }

}  // extern "C"
