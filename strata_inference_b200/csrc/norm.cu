// RMS norm, alone and fused with the residual add around it (further down: Dynamic Tanh and the
// layer norm in the same two forms).
//
//   rms(x, g) = x * 1/sqrt(mean(x^2) + eps) * g        (statistics in f32)
//
// The gain g arrives ready-made in f32 (the norm part adds the architecture's
// offset to the stored weight once, when it is built).
// Plain counterpart: tests/plain_gemma2.py rms_norm().
// Reference formula: src/backend/cpu.rs:797-810; the order "norm of the
// sub-layer's output, then the add" is src/model/layer.rs:1163-1170,1185-1192.
#include "common.cuh"

// out[i, :] = rms(x[rows ? rows[i] : i, :], gain).  The row is held in shared
// memory (hidden floats) between the two passes.  A row of x starts every `x_stride`
// elements (the leading columns of a wider buffer are normed where it exceeds `hidden`).
template <typename Tin, typename Tout>
__global__ void rms_norm_kernel(const Tin* __restrict__ x, const int* __restrict__ rows,
                                const float* __restrict__ gain, Tout* __restrict__ out,
                                int hidden, float eps, long long x_stride) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x;
    const Tin* src = x + (size_t)(rows ? rows[i] : i) * x_stride;
    float ss = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float v = to_f32(src[c]);
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)hidden + eps);
    Tout* dst = out + (size_t)i * hidden;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        dst[c] = from_f32<Tout>(row[c] * inv * gain[c]);
}

// h[r, :] += post_gain ? rms(a[r, :], post_gain) : a[r, :]
// out[r, :] = pre_gain ? rms(h[r, :], pre_gain) : h[r, :]      (only if out)
// h is the 32-bit residual stream; a and out have the activation type.
template <typename T>
__global__ void add_rms_norm_kernel(const T* __restrict__ a, const float* __restrict__ post_gain,
                                    float post_eps, float* __restrict__ h,
                                    const float* __restrict__ pre_gain, float pre_eps,
                                    T* __restrict__ out, int hidden) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * hidden;
    float ss = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float v = to_f32(a[base + c]);
        row[c] = v;
        ss += v * v;
    }
    float inv = 1.f;
    if (post_gain) {
        ss = block_sum(ss, scratch);
        inv = 1.0f / sqrtf(ss / (float)hidden + post_eps);
    }
    float ss2 = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float add = post_gain ? row[c] * inv * post_gain[c] : row[c];
        const float v = h[base + c] + add;
        h[base + c] = v;
        row[c] = v;
        ss2 += v * v;
    }
    if (!out) return;
    float inv2 = 1.f;
    if (pre_gain) {
        ss2 = block_sum(ss2, scratch);
        inv2 = 1.0f / sqrtf(ss2 / (float)hidden + pre_eps);
    }
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        out[base + c] = from_f32<T>(pre_gain ? row[c] * inv2 * pre_gain[c] : row[c]);
}

// The same for bfloat16 activations and a hidden size in whole groups of 8: every
// access is 16 bytes wide (8 activations, 4 stream or gain values).
__global__ void add_rms_norm_bf16_kernel(const __nv_bfloat16* __restrict__ a,
                                         const float* __restrict__ post_gain, float post_eps,
                                         float* __restrict__ h, const float* __restrict__ pre_gain,
                                         float pre_eps, __nv_bfloat16* __restrict__ out, int hidden) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * hidden;
    const int groups = hidden / 8;
    float ss = 0.f;
    for (int v = threadIdx.x; v < groups; v += blockDim.x) {
        const uint4 raw = *reinterpret_cast<const uint4*>(a + base + 8 * v);
        const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float lo = __uint_as_float(w[k] << 16), hi = __uint_as_float(w[k] & 0xffff0000u);
            row[8 * v + 2 * k] = lo;
            row[8 * v + 2 * k + 1] = hi;
            ss += lo * lo + hi * hi;
        }
    }
    float inv = 1.f;
    if (post_gain) {
        ss = block_sum(ss, scratch);
        inv = 1.0f / sqrtf(ss / (float)hidden + post_eps);
    } else {
        __syncthreads();   // the next pass reads the row in another order
    }
    float ss2 = 0.f;
    for (int v = threadIdx.x; v < 2 * groups; v += blockDim.x) {   // float4 at a time
        float4 hv = *reinterpret_cast<const float4*>(h + base + 4 * v);
        float4 av = *reinterpret_cast<const float4*>(row + 4 * v);
        if (post_gain) {
            const float4 gv = *reinterpret_cast<const float4*>(post_gain + 4 * v);
            av.x *= inv * gv.x; av.y *= inv * gv.y; av.z *= inv * gv.z; av.w *= inv * gv.w;
        }
        hv.x += av.x; hv.y += av.y; hv.z += av.z; hv.w += av.w;
        *reinterpret_cast<float4*>(h + base + 4 * v) = hv;
        *reinterpret_cast<float4*>(row + 4 * v) = hv;
        ss2 += hv.x * hv.x + hv.y * hv.y + hv.z * hv.z + hv.w * hv.w;
    }
    if (!out) return;
    float inv2 = 1.f;
    if (pre_gain) {
        ss2 = block_sum(ss2, scratch);
        inv2 = 1.0f / sqrtf(ss2 / (float)hidden + pre_eps);
    } else {
        __syncthreads();   // the next pass reads the row in another order
    }
    for (int v = threadIdx.x; v < groups; v += blockDim.x) {
        uint32_t w[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int c = 8 * v + 2 * k;
            const float g0 = pre_gain ? pre_gain[c] : 1.f, g1 = pre_gain ? pre_gain[c + 1] : 1.f;
            const __nv_bfloat162 o = __floats2bfloat162_rn(row[c] * inv2 * g0,
                                                           row[c + 1] * inv2 * g1);
            w[k] = *reinterpret_cast<const uint32_t*>(&o);
        }
        *reinterpret_cast<uint4*>(out + base + 8 * v) = make_uint4(w[0], w[1], w[2], w[3]);
    }
}

// One warp per row, the row in registers, no block-wide barrier: for hidden sizes that
// are NG x 256 (lane l owns the 8-element groups l, l + 32, ...).
template <int NG>
__global__ void __launch_bounds__(128)
add_rms_norm_bf16_warp_kernel(const __nv_bfloat16* __restrict__ a, const float* __restrict__ post_gain,
                              float post_eps, float* __restrict__ h,
                              const float* __restrict__ pre_gain, float pre_eps,
                              __nv_bfloat16* __restrict__ out, int n_rows) {
    pdl_trigger();
    pdl_wait();
    constexpr int hidden = NG * 256;
    const int lane = threadIdx.x & 31;
    const int r = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (r >= n_rows) return;
    const size_t base = (size_t)r * hidden;
    float v[NG][8];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NG; ++i) {
        const uint4 raw = *reinterpret_cast<const uint4*>(a + base + 8 * (lane + 32 * i));
        const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            v[i][2 * k] = __uint_as_float(w[k] << 16);
            v[i][2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
            ss += v[i][2 * k] * v[i][2 * k] + v[i][2 * k + 1] * v[i][2 * k + 1];
        }
    }
    float inv = 1.f;
    if (post_gain) inv = 1.0f / sqrtf(warp_sum(ss) / (float)hidden + post_eps);
    float ss2 = 0.f;
#pragma unroll
    for (int i = 0; i < NG; ++i) {
        const int c = 8 * (lane + 32 * i);
        float4 h0 = *reinterpret_cast<const float4*>(h + base + c);
        float4 h1 = *reinterpret_cast<const float4*>(h + base + c + 4);
        if (post_gain) {
            const float4 g0 = *reinterpret_cast<const float4*>(post_gain + c);
            const float4 g1 = *reinterpret_cast<const float4*>(post_gain + c + 4);
            v[i][0] *= inv * g0.x; v[i][1] *= inv * g0.y; v[i][2] *= inv * g0.z; v[i][3] *= inv * g0.w;
            v[i][4] *= inv * g1.x; v[i][5] *= inv * g1.y; v[i][6] *= inv * g1.z; v[i][7] *= inv * g1.w;
        }
        h0.x += v[i][0]; h0.y += v[i][1]; h0.z += v[i][2]; h0.w += v[i][3];
        h1.x += v[i][4]; h1.y += v[i][5]; h1.z += v[i][6]; h1.w += v[i][7];
        *reinterpret_cast<float4*>(h + base + c) = h0;
        *reinterpret_cast<float4*>(h + base + c + 4) = h1;
        v[i][0] = h0.x; v[i][1] = h0.y; v[i][2] = h0.z; v[i][3] = h0.w;
        v[i][4] = h1.x; v[i][5] = h1.y; v[i][6] = h1.z; v[i][7] = h1.w;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss2 += v[i][e] * v[i][e];
    }
    if (!out) return;
    const float inv2 = pre_gain ? 1.0f / sqrtf(warp_sum(ss2) / (float)hidden + pre_eps) : 1.f;
    const float4 ones = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
    for (int i = 0; i < NG; ++i) {
        const int c = 8 * (lane + 32 * i);
        const float4 g0 = pre_gain ? *reinterpret_cast<const float4*>(pre_gain + c) : ones;
        const float4 g1 = pre_gain ? *reinterpret_cast<const float4*>(pre_gain + c + 4) : ones;
        const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
        uint32_t w[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const __nv_bfloat162 o = __floats2bfloat162_rn(v[i][2 * k] * inv2 * g[2 * k],
                                                           v[i][2 * k + 1] * inv2 * g[2 * k + 1]);
            w[k] = *reinterpret_cast<const uint32_t*>(&o);
        }
        *reinterpret_cast<uint4*>(out + base + c) = make_uint4(w[0], w[1], w[2], w[3]);
    }
}

// One block per row, one 8-element group per thread, the row in registers: every load of a
// row is issued before anything is computed (the gains even before the kernel ahead of this
// one has finished), so a row costs two block-wide sums and no pass over shared memory.
// (a, h and out are not marked __restrict__: the compiler may move a load through such a pointer
// ahead of the wait for the kernel that writes there.)
__global__ void __launch_bounds__(1024)
add_rms_norm_bf16_group_kernel(const __nv_bfloat16* a, const float* __restrict__ post_gain,
                               float post_eps, float* h, const float* __restrict__ pre_gain, float pre_eps,
                               __nv_bfloat16* out, int hidden) {
    __shared__ float scratch[33];
    pdl_trigger();
    const int c = 8 * threadIdx.x;
    const bool live = c < hidden;
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
    float4 pg0 = one, pg1 = one, qg0 = one, qg1 = one;
    if (live && post_gain) {
        pg0 = *reinterpret_cast<const float4*>(post_gain + c);
        pg1 = *reinterpret_cast<const float4*>(post_gain + c + 4);
    }
    if (live && pre_gain) {
        qg0 = *reinterpret_cast<const float4*>(pre_gain + c);
        qg1 = *reinterpret_cast<const float4*>(pre_gain + c + 4);
    }
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * hidden + c;
    uint4 raw = make_uint4(0, 0, 0, 0);
    float4 h0 = make_float4(0.f, 0.f, 0.f, 0.f), h1 = h0;
    if (live) {
        raw = *reinterpret_cast<const uint4*>(a + base);
        h0 = *reinterpret_cast<const float4*>(h + base);
        h1 = *reinterpret_cast<const float4*>(h + base + 4);
    }
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
    float v[8];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        v[2 * k] = __uint_as_float(w[k] << 16);
        v[2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
        ss += v[2 * k] * v[2 * k] + v[2 * k + 1] * v[2 * k + 1];
    }
    if (post_gain) {
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)hidden + post_eps);
        v[0] *= inv * pg0.x; v[1] *= inv * pg0.y; v[2] *= inv * pg0.z; v[3] *= inv * pg0.w;
        v[4] *= inv * pg1.x; v[5] *= inv * pg1.y; v[6] *= inv * pg1.z; v[7] *= inv * pg1.w;
    }
    h0.x += v[0]; h0.y += v[1]; h0.z += v[2]; h0.w += v[3];
    h1.x += v[4]; h1.y += v[5]; h1.z += v[6]; h1.w += v[7];
    if (live) {
        *reinterpret_cast<float4*>(h + base) = h0;
        *reinterpret_cast<float4*>(h + base + 4) = h1;
    }
    if (!out) return;
    float inv2 = 1.f;
    if (pre_gain) {
        float ss2 = h0.x * h0.x + h0.y * h0.y + h0.z * h0.z + h0.w * h0.w +
                    h1.x * h1.x + h1.y * h1.y + h1.z * h1.z + h1.w * h1.w;
        ss2 = block_sum(ss2, scratch);
        inv2 = 1.0f / sqrtf(ss2 / (float)hidden + pre_eps);
    }
    if (live) {
        const __nv_bfloat162 o0 = __floats2bfloat162_rn(h0.x * inv2 * qg0.x, h0.y * inv2 * qg0.y);
        const __nv_bfloat162 o1 = __floats2bfloat162_rn(h0.z * inv2 * qg0.z, h0.w * inv2 * qg0.w);
        const __nv_bfloat162 o2 = __floats2bfloat162_rn(h1.x * inv2 * qg1.x, h1.y * inv2 * qg1.y);
        const __nv_bfloat162 o3 = __floats2bfloat162_rn(h1.z * inv2 * qg1.z, h1.w * inv2 * qg1.w);
        *reinterpret_cast<uint4*>(out + base) =
            make_uint4(*reinterpret_cast<const uint32_t*>(&o0), *reinterpret_cast<const uint32_t*>(&o1),
                       *reinterpret_cast<const uint32_t*>(&o2), *reinterpret_cast<const uint32_t*>(&o3));
    }
}

template <int NG>
static int launch_warp_norm(const void* a, const float* post_gain, float post_eps, float* h,
                            const float* pre_gain, float pre_eps, void* out, int n_rows,
                            cudaStream_t s) {
    sib_launch_chained(add_rms_norm_bf16_warp_kernel<NG>, dim3((n_rows + 3) / 4), dim3(128), 0, s,
                       (const __nv_bfloat16*)a, post_gain, post_eps, h, pre_gain, pre_eps,
                       (__nv_bfloat16*)out, n_rows);
    return sib_check_launch("add_rms_norm");
}

#include <stdlib.h>
#include <string.h>

// SIB_NORM_KERNEL=warp keeps the warp-per-row kernel for many rows.
static int norm_kernel_mode() {
    const char* v = getenv("SIB_NORM_KERNEL");
    return (v && strcmp(v, "warp") == 0) ? 1 : 0;
}
// From this many rows on the group-per-thread kernel runs (SIB_NORM_GROUP_ROWS overrides).
// It is the faster one at every number of rows: single-token steps of the Gemma2-2B shape gain
// 5 % at batch 8 and 6 % at batch 1 over the kernel that stages the row in shared memory, the 9B
// and 27B shapes 3 % and 1 %.
static int group_rows_threshold() {
    static int t = -1;
    if (t < 0) {
        const char* v = getenv("SIB_NORM_GROUP_ROWS");
        t = v ? atoi(v) : 1;
        if (t < 1) t = 1;
    }
    return t;
}

static int norm_threads(int hidden) {
    int t = 128;
    while (t < 1024 && t * 4 < hidden) t *= 2;
    return t;
}

static const int kMaxRowBytes = 200 * 1024;

template <typename K>
static int allow_row(K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return 0;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)bytes);
    if (e != cudaSuccess) {
        sib_set_error("norm: cannot reserve %zu bytes of shared memory: %s", bytes,
                      cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

SIB_EXPORT int sib_rms_norm(const void* x, int in_dtype, const int* rows, const float* gain,
                            float eps, void* out, int out_dtype, int n_rows, int hidden,
                            long long x_stride, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0 && x_stride >= hidden, "rms_norm: rows=%d hidden=%d stride=%lld",
                n_rows, hidden, x_stride);
    const size_t smem = (size_t)hidden * sizeof(float);
    SIB_REQUIRE(smem <= (size_t)kMaxRowBytes,
                "rms_norm: hidden=%d needs %zu bytes of shared memory; at most %d are supported",
                hidden, smem, kMaxRowBytes);
    const int threads = norm_threads(hidden);
    cudaStream_t s = (cudaStream_t)stream;
#define LAUNCH(TIN, TOUT)                                                              \
    do {                                                                               \
        int rc = allow_row(rms_norm_kernel<TIN, TOUT>, smem);                          \
        if (rc) return rc;                                                             \
        sib_launch_chained(rms_norm_kernel<TIN, TOUT>, dim3(n_rows), dim3(threads), smem, s, \
                           (const TIN*)x, rows, gain, (TOUT*)out, hidden, eps, x_stride); \
    } while (0)
    if (in_dtype == SIB_F32 && out_dtype == SIB_F32) LAUNCH(float, float);
    else if (in_dtype == SIB_F32 && out_dtype == SIB_BF16) LAUNCH(float, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_F32) LAUNCH(__nv_bfloat16, float);
    else SIB_REQUIRE(false, "rms_norm: unknown element types %d -> %d", in_dtype, out_dtype);
#undef LAUNCH
    return sib_check_launch("rms_norm");
}

SIB_EXPORT int sib_add_rms_norm(const void* a, int dtype, const float* post_gain, float post_eps,
                                float* h, const float* pre_gain, float pre_eps, void* out,
                                int n_rows, int hidden, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0, "add_rms_norm: rows=%d hidden=%d", n_rows, hidden);
    SIB_REQUIRE(pre_gain == nullptr || out != nullptr, "add_rms_norm: pre_gain without out");
    const size_t smem = (size_t)hidden * sizeof(float);
    SIB_REQUIRE(smem <= (size_t)kMaxRowBytes,
                "add_rms_norm: hidden=%d needs %zu bytes of shared memory; at most %d are supported",
                hidden, smem, kMaxRowBytes);
    const int threads = norm_threads(hidden);
    if (dtype == SIB_BF16 && hidden % 8 == 0 && ((uintptr_t)a % 16) == 0 &&
        ((uintptr_t)h % 16) == 0 && ((uintptr_t)out % 16) == 0 &&
        ((uintptr_t)post_gain % 16) == 0 && ((uintptr_t)pre_gain % 16) == 0) {
        // a block per row with one 8-element group per thread, every load issued at once
        // (SIB_NORM_KERNEL=warp: for many rows a warp per row, for few the row in shared memory)
        static const int mode = norm_kernel_mode();
        if (n_rows >= group_rows_threshold() && hidden / 8 <= 1024 && mode != 1) {
            const int threads = (hidden / 8 + 31) / 32 * 32;
            sib_launch_chained(add_rms_norm_bf16_group_kernel, dim3(n_rows), dim3(threads), 0,
                               (cudaStream_t)stream, (const __nv_bfloat16*)a, post_gain, post_eps, h,
                               pre_gain, pre_eps, (__nv_bfloat16*)out, hidden);
            return sib_check_launch("add_rms_norm");
        }
        if (n_rows >= 512 && hidden % 256 == 0 && hidden / 256 <= 18) {
            cudaStream_t s = (cudaStream_t)stream;
#define NORM_CASE(NG) \
    case NG: return launch_warp_norm<NG>(a, post_gain, post_eps, h, pre_gain, pre_eps, out, n_rows, s)
            switch (hidden / 256) {
                NORM_CASE(1); NORM_CASE(2); NORM_CASE(3); NORM_CASE(4); NORM_CASE(5); NORM_CASE(6);
                NORM_CASE(7); NORM_CASE(8); NORM_CASE(9); NORM_CASE(10); NORM_CASE(11); NORM_CASE(12);
                NORM_CASE(13); NORM_CASE(14); NORM_CASE(15); NORM_CASE(16); NORM_CASE(17); NORM_CASE(18);
            }
#undef NORM_CASE
        }
        int rc = allow_row(add_rms_norm_bf16_kernel, smem);
        if (rc) return rc;
        sib_launch_chained(add_rms_norm_bf16_kernel, dim3(n_rows),
                           dim3(threads < 256 ? threads : 256), smem, (cudaStream_t)stream,
                           (const __nv_bfloat16*)a, post_gain, post_eps, h, pre_gain, pre_eps,
                           (__nv_bfloat16*)out, hidden);
        return sib_check_launch("add_rms_norm");
    }
    SIB_DISPATCH_DTYPE(dtype, {
        int rc = allow_row(add_rms_norm_kernel<T>, smem);
        if (rc) return rc;
        sib_launch_chained(add_rms_norm_kernel<T>, dim3(n_rows), dim3(threads), smem,
                           (cudaStream_t)stream, (const T*)a, post_gain, post_eps, h, pre_gain,
                           pre_eps, (T*)out, hidden);
    });
    return sib_check_launch("add_rms_norm");
}

// ---------------------------------------------------------------------------
// Dynamic Tanh: a norm without statistics, element by element
//     dyt(x) = tanh(alpha x) w + b          (alpha one number, w and b one per column)
// alone (with a row gather) and fused with the residual add around it, as the RMS norm is:
//     h[r, :] += scale * (post ? dyt_post(a[r, :]) : a[r, :])      (scale: the layer's factor
//     out[r, :] = pre ? dyt_pre(h[r, :]) : h[r, :]   (only if out)  on what it adds; 1 as a rule)
// Everything is 32-bit; alpha is read from the device (it is a stored tensor).
// Plain counterpart: tests/plain_vavupel.py dynamic_tanh().
// ---------------------------------------------------------------------------
template <typename Tin, typename Tout>
__global__ void dyt_norm_kernel(const Tin* __restrict__ x, const int* __restrict__ rows,
                                const float* __restrict__ w, const float* __restrict__ b,
                                const float* __restrict__ alpha, Tout* __restrict__ out, int hidden) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x;
    const float al = *alpha;
    const Tin* src = x + (size_t)(rows ? rows[i] : i) * hidden;
    Tout* dst = out + (size_t)i * hidden;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        dst[c] = from_f32<Tout>(tanhf(al * to_f32(src[c])) * w[c] + b[c]);
}

template <typename T>
__global__ void add_dyt_norm_kernel(const T* __restrict__ a, const float* __restrict__ post_w,
                                    const float* __restrict__ post_b, const float* __restrict__ post_alpha,
                                    float* __restrict__ h, const float* __restrict__ pre_w,
                                    const float* __restrict__ pre_b, const float* __restrict__ pre_alpha,
                                    T* __restrict__ out, int hidden, size_t total, float scale) {
    pdl_trigger();
    pdl_wait();
    const float pa = post_w ? *post_alpha : 0.f, qa = pre_w ? *pre_alpha : 0.f;
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (size_t)gridDim.x * blockDim.x) {
        const int c = (int)(idx % hidden);
        float y = to_f32(a[idx]);
        if (post_w) y = tanhf(pa * y) * post_w[c] + post_b[c];
        const float s = h[idx] + scale * y;
        h[idx] = s;
        if (out) out[idx] = from_f32<T>(pre_w ? tanhf(qa * s) * pre_w[c] + pre_b[c] : s);
    }
}

SIB_EXPORT int sib_dyt_norm(const void* x, int in_dtype, const int* rows, const float* w,
                            const float* b, const float* alpha, void* out, int out_dtype,
                            int n_rows, int hidden, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0 && w && b && alpha, "dyt_norm: rows=%d hidden=%d", n_rows, hidden);
    const int threads = hidden >= 1024 ? 256 : 128;
    cudaStream_t s = (cudaStream_t)stream;
#define LAUNCH(TIN, TOUT)                                                                         \
    sib_launch_chained(dyt_norm_kernel<TIN, TOUT>, dim3(n_rows), dim3(threads), 0, s, (const TIN*)x, \
                       rows, w, b, alpha, (TOUT*)out, hidden)
    if (in_dtype == SIB_F32 && out_dtype == SIB_F32) LAUNCH(float, float);
    else if (in_dtype == SIB_F32 && out_dtype == SIB_BF16) LAUNCH(float, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_F32) LAUNCH(__nv_bfloat16, float);
    else SIB_REQUIRE(false, "dyt_norm: unknown element types %d -> %d", in_dtype, out_dtype);
#undef LAUNCH
    return sib_check_launch("dyt_norm");
}

SIB_EXPORT int sib_add_dyt_norm(const void* a, int dtype, const float* post_w, const float* post_b,
                                const float* post_alpha, float* h, const float* pre_w,
                                const float* pre_b, const float* pre_alpha, void* out, int n_rows,
                                int hidden, float scale, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0, "add_dyt_norm: rows=%d hidden=%d", n_rows, hidden);
    SIB_REQUIRE((post_w == nullptr || (post_b && post_alpha)) && (pre_w == nullptr || (pre_b && pre_alpha && out)),
                "add_dyt_norm: a norm needs its weight, its bias and alpha (and the next one out)");
    const size_t total = (size_t)n_rows * hidden;
    const size_t want = (total + 255) / 256;
    const int blocks = (int)(want < 148 * 16 ? want : 148 * 16);
    SIB_DISPATCH_DTYPE(dtype, sib_launch_chained(add_dyt_norm_kernel<T>, dim3(blocks), dim3(256), 0,
                                                 (cudaStream_t)stream, (const T*)a, post_w, post_b,
                                                 post_alpha, h, pre_w, pre_b, pre_alpha, (T*)out,
                                                 hidden, total, scale));
    return sib_check_launch("add_dyt_norm");
}

// ---------------------------------------------------------------------------
// pair_norm_mean: the joint output of two mixers that ran side by side on the same input:
//     y = (a / rms(a) * wa + b / rms(b) * wb) / 2          (rms over the row, eps inside the root)
// One block per row; statistics and sum in 32-bit.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
pair_norm_mean_kernel(const T* __restrict__ a, const T* __restrict__ b, const float* __restrict__ wa,
                      const float* __restrict__ wb, T* __restrict__ y, int width, float eps) {
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const size_t r = blockIdx.x;
    const T* ar = a + r * width;
    const T* br = b + r * width;
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float x = to_f32(ar[c]), z = to_f32(br[c]);
        sa += x * x;
        sb += z * z;
    }
    const float ia = 1.0f / sqrtf(block_sum(sa, scratch) / (float)width + eps);
    const float ib = 1.0f / sqrtf(block_sum(sb, scratch) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x)
        y[r * width + c] = from_f32<T>(0.5f * (to_f32(ar[c]) * ia * wa[c] + to_f32(br[c]) * ib * wb[c]));
}

SIB_EXPORT int sib_pair_norm_mean(const void* a, const void* b, const float* wa, const float* wb,
                                  void* y, int dtype, int rows, int width, float eps, void* stream) {
    if (rows == 0) return 0;
    SIB_REQUIRE(rows > 0 && width > 0 && a && b && wa && wb && y, "pair_norm_mean: rows=%d width=%d",
                rows, width);
    SIB_DISPATCH_DTYPE(dtype, sib_launch_chained(pair_norm_mean_kernel<T>, dim3(rows), dim3(256), 0,
                                                 (cudaStream_t)stream, (const T*)a, (const T*)b, wa,
                                                 wb, (T*)y, width, eps));
    return sib_check_launch("pair_norm_mean");
}

// ---------------------------------------------------------------------------
// Layer norm with weight and bias, alone (with a row gather) and fused with the residual add
// around it, as the RMS norm is:
//     ln(x) = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b
//     h[r, :] += post ? ln_post(a[r, :]) : a[r, :]
//     out[r, :] = pre ? ln_pre(h[r, :]) : h[r, :]        (only if out)
// Everything is 32-bit; the mean is taken first and the variance from the deviations (two sums
// over the row, so that a large mean costs no digits).
// (What the kernel ahead writes is not marked __restrict__: the compiler may move a load through
// such a pointer ahead of the wait for that kernel.)
// Plain counterpart: tests/plain_simetar.py layer_norm().
// ---------------------------------------------------------------------------
template <typename Tin, typename Tout>
__global__ void layer_norm_kernel(const Tin* x, const int* __restrict__ rows,
                                  const float* __restrict__ w, const float* __restrict__ b,
                                  Tout* out, int hidden, float eps) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x;
    const Tin* src = x + (size_t)(rows ? rows[i] : i) * hidden;
    float sum = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float v = to_f32(src[c]);
        row[c] = v;
        sum += v;
    }
    const float mean = block_sum(sum, scratch) / (float)hidden;
    float ss = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float d = row[c] - mean;
        ss += d * d;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
    Tout* dst = out + (size_t)i * hidden;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        dst[c] = from_f32<Tout>((row[c] - mean) * inv * w[c] + b[c]);
}

struct LayerNormPair {
    const float* post_w;       // null: what is added is not normed
    const float* post_b;
    const float* pre_w;        // null: the rows of h go out as they are
    const float* pre_b;
    float post_eps, pre_eps;
};

template <typename T>
__global__ void add_layer_norm_kernel(const T* a, float* h, T* out,
                                      int hidden, LayerNormPair p) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    pdl_trigger();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * hidden;
    // (a thread only ever touches its own columns of `row`)
    auto statistics = [&](float sum, float eps, float& mean, float& inv) {
        mean = block_sum(sum, scratch) / (float)hidden;
        float ss = 0.f;
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float d = row[c] - mean;
            ss += d * d;
        }
        inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
    };
    float sum = 0.f, mean = 0.f, inv = 1.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float v = to_f32(a[base + c]);
        row[c] = v;
        sum += v;
    }
    if (p.post_w) statistics(sum, p.post_eps, mean, inv);
    sum = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        const float v = h[base + c] + (p.post_w ? (row[c] - mean) * inv * p.post_w[c] + p.post_b[c] : row[c]);
        h[base + c] = v;
        row[c] = v;
        sum += v;
    }
    if (!out) return;
    if (p.pre_w) statistics(sum, p.pre_eps, mean, inv);
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        out[base + c] = from_f32<T>(p.pre_w ? (row[c] - mean) * inv * p.pre_w[c] + p.pre_b[c] : row[c]);
}

// One block per row, one group of 8 columns per thread, the row in registers: every load is issued
// before anything is computed, weights and biases before the kernel ahead has finished.
__global__ void __launch_bounds__(1024)
add_layer_norm_bf16_kernel(const __nv_bfloat16* a, float* h, __nv_bfloat16* out, int hidden, LayerNormPair p) {
    __shared__ float scratch[33];
    pdl_trigger();
    const int c = 8 * threadIdx.x;
    const bool live = c < hidden;
    const float n = (float)hidden;
    auto load8 = [&](const float* from, float (&o)[8]) {
        const float4 lo = *reinterpret_cast<const float4*>(from), hi = *reinterpret_cast<const float4*>(from + 4);
        o[0] = lo.x; o[1] = lo.y; o[2] = lo.z; o[3] = lo.w;
        o[4] = hi.x; o[5] = hi.y; o[6] = hi.z; o[7] = hi.w;
    };
    float pw[8], pb[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) pw[e] = pb[e] = 0.f;
    if (live && p.post_w) {
        load8(p.post_w + c, pw);
        load8(p.post_b + c, pb);
    }
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * hidden + c;
    uint4 raw = make_uint4(0, 0, 0, 0);
    float s[8], v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) s[e] = 0.f;
    if (live) {
        raw = *reinterpret_cast<const uint4*>(a + base);
        load8(h + base, s);
    }
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        v[2 * k] = __uint_as_float(w[k] << 16);
        v[2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
    }
    auto statistics = [&](const float (&x)[8], float eps, float& mean, float& inv) {
        float sum = 0.f, ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) sum += x[e];           // (columns that do not exist hold zeros)
        mean = block_sum(sum, scratch) / n;
        if (live) {
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += (x[e] - mean) * (x[e] - mean);
        }
        inv = 1.0f / sqrtf(block_sum(ss, scratch) / n + eps);
    };
    float mean = 0.f, inv = 1.f;
    if (p.post_w) {
        statistics(v, p.post_eps, mean, inv);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = live ? (v[e] - mean) * inv * pw[e] + pb[e] : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) s[e] += v[e];
    if (live) {
        *reinterpret_cast<float4*>(h + base) = make_float4(s[0], s[1], s[2], s[3]);
        *reinterpret_cast<float4*>(h + base + 4) = make_float4(s[4], s[5], s[6], s[7]);
    }
    if (!out) return;
    if (p.pre_w) {
        statistics(s, p.pre_eps, mean, inv);
        if (live) {
            load8(p.pre_w + c, pw);
            load8(p.pre_b + c, pb);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) s[e] = (s[e] - mean) * inv * pw[e] + pb[e];
    }
    if (live) {
        uint32_t o[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const __nv_bfloat162 pr = __floats2bfloat162_rn(s[2 * k], s[2 * k + 1]);
            o[k] = *reinterpret_cast<const uint32_t*>(&pr);
        }
        *reinterpret_cast<uint4*>(out + base) = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

SIB_EXPORT int sib_layer_norm(const void* x, int in_dtype, const int* rows, const float* w, const float* b,
                              float eps, void* out, int out_dtype, int n_rows, int hidden, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0 && w && b, "layer_norm: rows=%d hidden=%d", n_rows, hidden);
    const size_t smem = (size_t)hidden * sizeof(float);
    SIB_REQUIRE(smem <= (size_t)kMaxRowBytes, "layer_norm: hidden=%d needs %zu bytes of shared memory; at most "
                "%d are supported", hidden, smem, kMaxRowBytes);
    const int threads = norm_threads(hidden);
    cudaStream_t s = (cudaStream_t)stream;
#define LAUNCH(TIN, TOUT)                                                                        \
    do {                                                                                         \
        int rc = allow_row(layer_norm_kernel<TIN, TOUT>, smem);                                  \
        if (rc) return rc;                                                                       \
        sib_launch_chained(layer_norm_kernel<TIN, TOUT>, dim3(n_rows), dim3(threads), smem, s,   \
                           (const TIN*)x, rows, w, b, (TOUT*)out, hidden, eps);                  \
    } while (0)
    if (in_dtype == SIB_F32 && out_dtype == SIB_F32) LAUNCH(float, float);
    else if (in_dtype == SIB_F32 && out_dtype == SIB_BF16) LAUNCH(float, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (in_dtype == SIB_BF16 && out_dtype == SIB_F32) LAUNCH(__nv_bfloat16, float);
    else SIB_REQUIRE(false, "layer_norm: unknown element types %d -> %d", in_dtype, out_dtype);
#undef LAUNCH
    return sib_check_launch("layer_norm");
}

SIB_EXPORT int sib_add_layer_norm(const void* a, int dtype, const float* post_w, const float* post_b,
                                  float post_eps, float* h, const float* pre_w, const float* pre_b,
                                  float pre_eps, void* out, int n_rows, int hidden, void* stream) {
    if (n_rows == 0) return 0;
    SIB_REQUIRE(n_rows > 0 && hidden > 0, "add_layer_norm: rows=%d hidden=%d", n_rows, hidden);
    SIB_REQUIRE((post_w != nullptr) == (post_b != nullptr) && (pre_w != nullptr) == (pre_b != nullptr) &&
                    (pre_w == nullptr || out != nullptr),
                "add_layer_norm: a norm needs its weight and its bias (and the next one out)");
    const LayerNormPair p{post_w, post_b, pre_w, pre_b, post_eps, pre_eps};
    cudaStream_t s = (cudaStream_t)stream;
    auto wide = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
    if (dtype == SIB_BF16 && hidden % 8 == 0 && hidden / 8 <= 1024 && wide(a) && wide(h) && wide(out) &&
        wide(post_w) && wide(post_b) && wide(pre_w) && wide(pre_b)) {
        sib_launch_chained(add_layer_norm_bf16_kernel, dim3(n_rows), dim3((hidden / 8 + 31) / 32 * 32), 0, s,
                           (const __nv_bfloat16*)a, h, (__nv_bfloat16*)out, hidden, p);
        return sib_check_launch("add_layer_norm");
    }
    const size_t smem = (size_t)hidden * sizeof(float);
    SIB_REQUIRE(smem <= (size_t)kMaxRowBytes, "add_layer_norm: hidden=%d needs %zu bytes of shared memory; at "
                "most %d are supported", hidden, smem, kMaxRowBytes);
    SIB_DISPATCH_DTYPE(dtype, {
        int rc = allow_row(add_layer_norm_kernel<T>, smem);
        if (rc) return rc;
        sib_launch_chained(add_layer_norm_kernel<T>, dim3(n_rows), dim3(norm_threads(hidden)), smem, s, (const T*)a,
                           h, (T*)out, hidden, p);
    });
    return sib_check_launch("add_layer_norm");
}
