// Small kernels of a layer whose branches all read ONE norm's output and are added to the stream together
// (x += s0 * a + s1 * f with a gain per feature on each branch), with a layer norm (mean taken off) as that norm,
// and the elementwise half of a gated feed-forward with a choice of activation.  All arithmetic is fp32; `dtype`
// is the type of the activations (0 = float32, 1 = bfloat16).  The residual stream is float32.
#include "common.cuh"

#include <initializer_list>

// A branch output at element i of row r: an activation-dtype tensor, or fp32 partial sums added in index order.
template <typename T>
__device__ __forceinline__ float branch_at(const T* y, const float* parts, int n_parts, long long part_stride, size_t at) {
    if (parts) {
        float acc = parts[at];
        for (int s = 1; s < n_parts; ++s) acc += parts[(size_t)s * part_stride + at];
        return acc;
    }
    return to_f32<T>(y[at]);
}

// VEC consecutive elements of a branch output from element `at` on
template <typename T, int VEC>
__device__ __forceinline__ void branch_vec(const T* y, const float* parts, int n_parts, long long part_stride, size_t at, float (&out)[VEC]) {
    if (parts) {
        const Vec<float, VEC> first = load_vec<float, VEC>(parts + at);
#pragma unroll
        for (int k = 0; k < VEC; ++k) out[k] = first.v[k];
        for (int s = 1; s < n_parts; ++s) {
            const Vec<float, VEC> p = load_vec<float, VEC>(parts + (size_t)s * part_stride + at);
#pragma unroll
            for (int k = 0; k < VEC; ++k) out[k] += p.v[k];
        }
        return;
    }
    const Vec<T, VEC> v = load_vec<T, VEC>(y + at);
#pragma unroll
    for (int k = 0; k < VEC; ++k) out[k] = to_f32<T>(v.v[k]);
}

// v[k] = x[k] + (s0 * b0 + s1 * b1) for the VEC elements at `at` (column i of its row); a branch may be absent
template <typename T, int VEC>
__device__ __forceinline__ void add_branches(float (&v)[VEC], int i, size_t at, const T* y0, const float* p0, int n0, const float* s0,
                                             const T* y1, const float* p1, int n1, const float* s1, long long part_stride) {
    const bool b0 = y0 != nullptr || p0 != nullptr, b1 = y1 != nullptr || p1 != nullptr;
    if (!b0 && !b1) return;
    float add[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) add[k] = 0.f;
    if (b0) {
        float b[VEC];
        branch_vec<T, VEC>(y0, p0, n0, part_stride, at, b);
        const Vec<float, VEC> s = load_vec<float, VEC>(s0 + i);
#pragma unroll
        for (int k = 0; k < VEC; ++k) add[k] = __fmul_rn(s.v[k], b[k]);
    }
    if (b1) {
        float b[VEC];
        branch_vec<T, VEC>(y1, p1, n1, part_stride, at, b);
        const Vec<float, VEC> s = load_vec<float, VEC>(s1 + i);
#pragma unroll
        for (int k = 0; k < VEC; ++k) add[k] = __fadd_rn(add[k], __fmul_rn(s.v[k], b[k]));
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = __fadd_rn(v[k], add[k]);
}

// Vectors of four serve rows whose length is a multiple of four, if every pointer given is aligned to 16 bytes
static inline bool aligned16(std::initializer_list<const void*> ptrs) {
    uintptr_t bits = 0;
    for (const void* p : ptrs) bits |= (uintptr_t)p;
    return (bits & 15) == 0;
}

// ---------------------------------------------------------------------------
// v      = x[src] + (s0 * b0[src] + s1 * b1[src])      src = rows[r] or r; a branch may be absent
// x[src] = v                                            (update_x, without rows)
// out[r] = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * w (+ bias)      activation dtype, or fp32 when out_f32
// out2[r] = the same rows times w2                                              (out2 null: one norm only)
// One block per row; the row waits in shared memory between the passes.  The block size depends on H only, so a
// row's sums are added in the same order whatever the batch holds.
// ---------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void add_layernorm_kernel(float* x, const T* y0, const float* p0, int n0, const float* s0, const T* y1,
                                     const float* p1, int n1, const float* s1, long long part_stride, const float* w,
                                     const float* bias, const float* w2, void* out, void* out2, int out_f32, const int* rows, int H, float eps,
                                     int update_x) {
    extern __shared__ __align__(16) float row_smem[];   // [H]
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* xr = x + (size_t)src * H;
    const bool any = y0 != nullptr || p0 != nullptr || y1 != nullptr || p1 != nullptr;
    float sum = 0.f;
    for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
        Vec<float, VEC> x4 = load_vec<float, VEC>(xr + i);
        if (any) {
            add_branches<T, VEC>(x4.v, i, (size_t)src * H + i, y0, p0, n0, s0, y1, p1, n1, s1, part_stride);
            if (update_x) store_vec<float, VEC>(xr + i, x4);
        }
        store_vec<float, VEC>(row_smem + i, x4);
#pragma unroll
        for (int k = 0; k < VEC; ++k) sum += x4.v[k];
    }
    // a thread reads back what it wrote itself: the row needs no barrier of its own
    const float mean = block_sum(sum, scratch) / (float)H;
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
        const Vec<float, VEC> v = load_vec<float, VEC>(row_smem + i);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float d = v.v[k] - mean;
            ss = fmaf(d, d, ss);
        }
    }
    const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
        const Vec<float, VEC> v = load_vec<float, VEC>(row_smem + i), g = load_vec<float, VEC>(w + i);
        Vec<float, VEC> unit, o;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            unit.v[k] = __fmul_rn(v.v[k] - mean, rstd);
            o.v[k] = __fmul_rn(unit.v[k], g.v[k]);
        }
        const size_t at = (size_t)r * H + i;
        if (out2) {
            const Vec<float, VEC> g2 = load_vec<float, VEC>(w2 + i);
            Vec<T, VEC> t;
#pragma unroll
            for (int k = 0; k < VEC; ++k) t.v[k] = from_f32<T>(__fmul_rn(unit.v[k], g2.v[k]));
            store_vec<T, VEC>((T*)out2 + at, t);
        }
        if (bias) {
            const Vec<float, VEC> b = load_vec<float, VEC>(bias + i);
#pragma unroll
            for (int k = 0; k < VEC; ++k) o.v[k] = __fadd_rn(o.v[k], b.v[k]);
        }
        if (out_f32) {
            store_vec<float, VEC>((float*)out + at, o);
        } else {
            Vec<T, VEC> t;
#pragma unroll
            for (int k = 0; k < VEC; ++k) t.v[k] = from_f32<T>(o.v[k]);
            store_vec<T, VEC>((T*)out + at, t);
        }
    }
}

PYRE_API int pyre_add_layernorm(float* x, const void* y0, const float* p0, int n0, const float* s0, const void* y1,
                                const float* p1, int n1, const float* s1, long long part_stride, const float* weight,
                                const float* bias, const float* weight2, void* out, void* out2, int out_f32, const int* rows, int n_rows, int H,
                                float eps, int update_x,
                                int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (H <= 0 || (size_t)H * sizeof(float) > 48 * 1024) return PYRE_ERR_UNSUPPORTED;
    if ((y0 && p0) || (y1 && p1) || ((y0 || p0) && !s0) || ((y1 || p1) && !s1)) return PYRE_ERR_BAD_ARG;
    if ((p0 && n0 < 1) || (p1 && n1 < 1) || (out2 && !weight2)) return PYRE_ERR_BAD_ARG;
    const size_t smem = (size_t)H * sizeof(float);
    const bool vec = H % 4 == 0 && part_stride % 4 == 0 && aligned16({x, y0, p0, s0, y1, p1, s1, weight, bias, weight2, out, out2});
    // the block size depends on H only: vectors shared out evenly among at most 512 threads
    const int items = (H + 3) / 4, rounds = ceil_div(items, 512);
    const int threads = vec ? ceil_div(ceil_div(items, rounds), 32) * 32 : min(512, max(32, ((H / 4 + 31) / 32) * 32));
#define LAUNCH(T, V)                                                                                                              \
    pyre_launch(add_layernorm_kernel<T, V>, dim3(n_rows), dim3(threads), smem, stream, x, (const T*)y0, p0, n0, s0, (const T*)y1, \
                p1, n1, s1, part_stride, weight, bias, weight2, out, out2, out_f32, rows, H, eps, update_x)
    if (dtype == PYRE_BF16) { if (vec) LAUNCH(__nv_bfloat16, 4); else LAUNCH(__nv_bfloat16, 1); }
    else if (dtype == PYRE_F32) { if (vec) LAUNCH(float, 4); else LAUNCH(float, 1); }
    else return PYRE_ERR_BAD_ARG;
#undef LAUNCH
    PYRE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------------------
// out[r, i] = s0[i] * b0[r, i] + s1[i] * b1[r, i] in the activation dtype: the branches of such a layer as one
// plain tensor, for a consumer that knows nothing of them.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void scaled_sum_kernel(const T* y0, const float* p0, int n0, const float* s0, const T* y1, const float* p1,
                                  int n1, const float* s1, long long part_stride, T* out, size_t n, int H) {
    pdl_trigger();
    pdl_wait();
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    const bool b1 = y1 != nullptr || p1 != nullptr;
    for (size_t at = (size_t)blockIdx.x * blockDim.x + threadIdx.x; at < n; at += stride) {
        const int i = (int)(at % H);
        float add = __fmul_rn(s0[i], branch_at<T>(y0, p0, n0, part_stride, at));
        if (b1) add = __fadd_rn(add, __fmul_rn(s1[i], branch_at<T>(y1, p1, n1, part_stride, at)));
        out[at] = from_f32<T>(add);
    }
}

PYRE_API int pyre_scaled_sum(const void* y0, const float* p0, int n0, const float* s0, const void* y1, const float* p1,
                             int n1, const float* s1, long long part_stride, void* out, int n_rows, int H, int dtype,
                             cudaStream_t stream) {
    if (n_rows <= 0 || H <= 0) return 0;
    if ((y0 == nullptr) == (p0 == nullptr) || !s0 || (y1 && p1) || ((y1 || p1) && !s1)) return PYRE_ERR_BAD_ARG;
    const size_t n = (size_t)n_rows * H;
    const int blocks = (int)min((long long)pyre_sm_count() * 8, ceil_div_ll((long long)n, 256));
    if (dtype == PYRE_BF16)
        pyre_launch(scaled_sum_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)y0, p0, n0, s0,
                    (const __nv_bfloat16*)y1, p1, n1, s1, part_stride, (__nv_bfloat16*)out, n, H);
    else if (dtype == PYRE_F32)
        pyre_launch(scaled_sum_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)y0, p0, n0, s0, (const float*)y1,
                    p1, n1, s1, part_stride, (float*)out, n, H);
    else return PYRE_ERR_BAD_ARG;
    PYRE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------------------
// out[r, i] = act(gu[r, i]) * gu[r, I + i]: the elementwise half of a gated feed-forward whose product left
// [gates | ups] per row.  kind 0: silu, z / (1 + exp(-z)); kind 1: the tanh form of gelu,
// 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))); kind 2: relu, max(z, 0); kind 3: the clamped form
// z sigmoid(1.702 z) (u + 1) with z = min(gate, limit), u = clamp(up, -limit, limit).
// ---------------------------------------------------------------------------
__device__ __forceinline__ float gate_act(float z, int kind) {
    if (kind == 0) return z / (1.0f + expf(-z));
    if (kind == 2) return fmaxf(z, 0.f);
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return 0.5f * z * (1.0f + tanhf(u));
}

__device__ __forceinline__ float gated_pair(float z, float u, int kind, float limit) {
    if (kind == 3) {
        z = fminf(z, limit);
        return __fmul_rn(z / (1.0f + expf(-CLAMPED_GLU_SLOPE * z)), fminf(fmaxf(u, -limit), limit) + 1.0f);
    }
    return __fmul_rn(gate_act(z, kind), u);
}

// VEC neighbouring features per thread (I a multiple of VEC, pointers aligned)
template <typename T, int VEC>
__global__ void act_mul_kernel(const T* gu, T* out, size_t n_rows, int I, int kind, float limit) {
    pdl_trigger();
    pdl_wait();
    const size_t per_row = (size_t)(I / VEC), total = n_rows * per_row;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += stride) {
        const size_t r = idx / per_row;
        const int i = (int)(idx - r * per_row) * VEC;
        const T* row = gu + r * (size_t)(2 * I);
        const Vec<T, VEC> g = load_vec<T, VEC>(row + i), u = load_vec<T, VEC>(row + I + i);
        Vec<T, VEC> o;
#pragma unroll
        for (int k = 0; k < VEC; ++k) o.v[k] = from_f32<T>(gated_pair(to_f32<T>(g.v[k]), to_f32<T>(u.v[k]), kind, limit));
        store_vec<T, VEC>(out + r * (size_t)I + i, o);
    }
}

PYRE_API int pyre_act_mul(const void* gu, void* out, int n_rows, int I, int kind, float limit, int dtype, cudaStream_t stream) {
    if (n_rows <= 0 || I <= 0) return 0;
    if (kind < 0 || kind > 3 || (kind == 3 && !(limit > 0.f))) return PYRE_ERR_BAD_ARG;
    const int vec = dtype == PYRE_BF16 ? 8 : 4;
    const bool wide = I % vec == 0 && aligned16({gu, out});
    const long long total = (long long)n_rows * (wide ? I / vec : I);
    const int blocks = (int)min((long long)pyre_sm_count() * 16, ceil_div_ll(total, 256));
#define LAUNCH(T, V) pyre_launch(act_mul_kernel<T, V>, dim3(blocks), dim3(256), 0, stream, (const T*)gu, (T*)out, (size_t)n_rows, I, kind, limit)
    if (dtype == PYRE_BF16) { if (wide) LAUNCH(__nv_bfloat16, 8); else LAUNCH(__nv_bfloat16, 1); }
    else if (dtype == PYRE_F32) { if (wide) LAUNCH(float, 4); else LAUNCH(float, 1); }
    else return PYRE_ERR_BAD_ARG;
#undef LAUNCH
    PYRE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------------------
// The stream with everything pending added, as activations for a product that reads the stream itself:
//   out[i] = T( x[i] + (s0 * b0[i] + s1 * b1[i]) )        a branch may be absent
// ---------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void stream_rows_kernel(const float* x, const T* y0, const float* p0, int n0, const float* s0, const T* y1,
                                   const float* p1, int n1, const float* s1, long long part_stride, T* out, size_t n, int H) {
    pdl_trigger();
    pdl_wait();
    const size_t stride = (size_t)gridDim.x * blockDim.x * VEC;
    for (size_t at = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC; at < n; at += stride) {
        Vec<float, VEC> v = load_vec<float, VEC>(x + at);
        add_branches<T, VEC>(v.v, (int)(at % H), at, y0, p0, n0, s0, y1, p1, n1, s1, part_stride);
        Vec<T, VEC> t;
#pragma unroll
        for (int k = 0; k < VEC; ++k) t.v[k] = from_f32<T>(v.v[k]);
        store_vec<T, VEC>(out + at, t);
    }
}

PYRE_API int pyre_stream_rows(const float* x, const void* y0, const float* p0, int n0, const float* s0, const void* y1,
                              const float* p1, int n1, const float* s1, long long part_stride, void* out, int n_rows, int H,
                              int dtype, cudaStream_t stream) {
    if (n_rows <= 0 || H <= 0) return 0;
    if ((y0 && p0) || (y1 && p1) || ((y0 || p0) && !s0) || ((y1 || p1) && !s1) || (p0 && n0 < 1) || (p1 && n1 < 1)) return PYRE_ERR_BAD_ARG;
    const size_t n = (size_t)n_rows * H;
    const bool vec = H % 4 == 0 && part_stride % 4 == 0 && aligned16({x, y0, p0, s0, y1, p1, s1, out});
    const int blocks = (int)min((long long)pyre_sm_count() * 8, ceil_div_ll((long long)n, vec ? 1024 : 256));
#define LAUNCH(T, V)                                                                                                               \
    pyre_launch(stream_rows_kernel<T, V>, dim3(blocks), dim3(256), 0, stream, x, (const T*)y0, p0, n0, s0, (const T*)y1, p1, n1, s1, \
                part_stride, (T*)out, n, H)
    if (dtype == PYRE_BF16) { if (vec) LAUNCH(__nv_bfloat16, 4); else LAUNCH(__nv_bfloat16, 1); }
    else if (dtype == PYRE_F32) { if (vec) LAUNCH(float, 4); else LAUNCH(float, 1); }
    else return PYRE_ERR_BAD_ARG;
#undef LAUNCH
    PYRE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------------------
// x[i] = base[i] + sum_s parts[s * part_stride + i]: the stream set anew from a product's fp32 partial sums and a
// fixed term.
// ---------------------------------------------------------------------------
template <int VEC>
__global__ void stream_set_kernel(float* x, const float* base, const float* parts, int n_parts, long long part_stride, size_t n) {
    pdl_trigger();
    pdl_wait();
    const size_t stride = (size_t)gridDim.x * blockDim.x * VEC;
    for (size_t at = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC; at < n; at += stride) {
        Vec<float, VEC> acc = load_vec<float, VEC>(parts + at);
        for (int s = 1; s < n_parts; ++s) {
            const Vec<float, VEC> p = load_vec<float, VEC>(parts + (size_t)s * part_stride + at);
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc.v[k] += p.v[k];
        }
        const Vec<float, VEC> b = load_vec<float, VEC>(base + at);
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc.v[k] += b.v[k];
        store_vec<float, VEC>(x + at, acc);
    }
}

PYRE_API int pyre_stream_set(float* x, const float* base, const float* parts, int n_parts, long long part_stride, long long n,
                             cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!x || !base || !parts || n_parts < 1) return PYRE_ERR_BAD_ARG;
    const bool vec = n % 4 == 0 && part_stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)base | (uintptr_t)parts) & 15) == 0;
    const int blocks = (int)min((long long)pyre_sm_count() * 8, ceil_div_ll(n, vec ? 1024 : 256));
    if (vec) pyre_launch(stream_set_kernel<4>, dim3(blocks), dim3(256), 0, stream, x, base, parts, n_parts, part_stride, (size_t)n);
    else pyre_launch(stream_set_kernel<1>, dim3(blocks), dim3(256), 0, stream, x, base, parts, n_parts, part_stride, (size_t)n);
    PYRE_LAUNCH_CHECK();
    return 0;
}
