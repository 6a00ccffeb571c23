// The norm on a sublayer's RESULT and the residual sum behind it, for layers of the form x <- x + norm(f(x)):
//   y = sum_p part[p][t]  (a product's result, or its split-K partial sums, added in index order)
//   x[t] += y * rsqrt(mean(y^2) + eps) * w;  lowp[t] = x[t] rounded to the compute type (optional)
// The statistics, the scaling and the sum are float.  The rounded copy is what the next sublayer reads, since it takes
// the stream as it is, un-normed: writing it here saves a kernel of its own.
// One block per row; the row of y is held in shared memory between the two passes.  Every row's sum of squares is
// added up in an order fixed by the width alone, so a row does not depend on what else the step holds.
#include <type_traits>

#include "common.cuh"

namespace bg {

template <typename TY, typename TW, typename TL>
__global__ void __launch_bounds__(256)
rmsnorm_add_kernel(float* __restrict__ x, const TY* __restrict__ y, int parts, size_t part_stride, const TW* __restrict__ w,
                   float eps, TL* __restrict__ lowp, int d) {
    extern __shared__ float row_buf[];
    __shared__ float red[32];
    pdl_launch();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * d;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = sum_parts(y + base + i, parts, part_stride);
        row_buf[i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = x[base + i] + row_buf[i] * inv * to_float(w[i]);
        x[base + i] = v;
        if (lowp) lowp[base + i] = from_float<TL>(v);
    }
}

// Float partial sums (or one float tensor) of a width that is a multiple of 4, 16-byte aligned: four features a
// thread, the parts' loads in flight together.
template <typename TW, typename TL>
__global__ void __launch_bounds__(256)
rmsnorm_add_vec4_kernel(float* __restrict__ x, const float* __restrict__ y, int parts, size_t part_stride,
                        const TW* __restrict__ w, float eps, TL* __restrict__ lowp, int d) {
    extern __shared__ float row_buf[];
    __shared__ float red[32];
    pdl_launch();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * d;
    float ss = 0.0f;
    for (int i = threadIdx.x * 4; i < d; i += blockDim.x * 4) {
        const float4 v = sum_parts4(reinterpret_cast<const float4*>(y + base + i), parts, part_stride / 4);
        *reinterpret_cast<float4*>(row_buf + i) = v;
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)d + eps);
    for (int i = threadIdx.x * 4; i < d; i += blockDim.x * 4) {
        const float4 v = *reinterpret_cast<const float4*>(row_buf + i);
        float4 o = *reinterpret_cast<const float4*>(x + base + i);
        o.x += v.x * inv * to_float(w[i]);     o.y += v.y * inv * to_float(w[i + 1]);
        o.z += v.z * inv * to_float(w[i + 2]); o.w += v.w * inv * to_float(w[i + 3]);
        *reinterpret_cast<float4*>(x + base + i) = o;
        if (lowp) {
            if constexpr (std::is_same<TL, float>::value) {
                *reinterpret_cast<float4*>(lowp + base + i) = o;
            } else {
                uint2 raw;
                __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
                h[0] = __floats2bfloat162_rn(o.x, o.y);
                h[1] = __floats2bfloat162_rn(o.z, o.w);
                *reinterpret_cast<uint2*>(lowp + base + i) = raw;
            }
        }
    }
}

// Many rows of a bfloat16 step: a warp per row, the row's values in registers (ITER chunks of eight a lane), one trip to
// memory.  The float32 path keeps ONE kernel for every number of rows, so that a row's statistics are added up in the same
// order whatever else the step holds.
template <typename TY, typename TW, int ITER>
__global__ void __launch_bounds__(256)
rmsnorm_add_warp_kernel(float* __restrict__ x, const TY* __restrict__ y, int parts, size_t part_stride, const TW* __restrict__ w,
                        float eps, __nv_bfloat16* __restrict__ lowp, int n_rows, int d) {
    pdl_launch();
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    const bool idle = warp >= n_rows;
    const size_t base = (size_t)(idle ? 0 : warp) * d;
    const int d8 = d >> 3;
    pdl_wait();
    if (idle) return;
    float v[ITER][8];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
        const int c = lane + 32 * i;
        if (c < d8) {
            load8(y + base + 8 * c, v[i]);
            for (int pp = 1; pp < parts; ++pp) {
                float u[8];
                load8(y + (size_t)pp * part_stride + base + 8 * c, u);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[i][e] += u[e];
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += v[i][e] * v[i][e];
        }
    }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)d + eps);
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
        const int c = lane + 32 * i;
        if (c < d8) {
            float xv[8], wv[8];
            load8(x + base + 8 * c, xv);
            load8(w + 8 * c, wv);
#pragma unroll
            for (int e = 0; e < 8; ++e) xv[e] += v[i][e] * inv * wv[e];
            store8(x + base + 8 * c, xv);
            if (lowp) store8(lowp + base + 8 * c, xv);
        }
    }
}

// The same behind routed experts: a token's y is the sum of the rows that its `top` chosen experts produced,
// y[t] = sum_j (weights[a] *) yp[row_of[a]], a = t * top + j, added in rank order; the sum that a kernel of its own would
// write and this one read back is formed here.  `vec`: the width is a multiple of 4 and everything 16-byte aligned.
template <typename TW, typename TL>
__global__ void __launch_bounds__(256)
rmsnorm_add_routed_kernel(float* __restrict__ x, const float* __restrict__ yp, const int* __restrict__ row_of,
                          const float* __restrict__ weights, int top, int scale, const TW* __restrict__ w, float eps,
                          TL* __restrict__ lowp, int d, int vec) {
    extern __shared__ float row_buf[];
    __shared__ float red[32];
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    const size_t base = (size_t)t * d;
    float ss = 0.0f;
    if (vec) {
        for (int i = threadIdx.x * 4; i < d; i += blockDim.x * 4) {
            float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            for (int j = 0; j < top; ++j) {
                const int a = t * top + j;
                const float4 v = *reinterpret_cast<const float4*>(yp + (size_t)row_of[a] * d + i);
                const float f = scale ? weights[a] : 1.0f;
                acc.x += f * v.x; acc.y += f * v.y; acc.z += f * v.z; acc.w += f * v.w;
            }
            *reinterpret_cast<float4*>(row_buf + i) = acc;
            ss += acc.x * acc.x + acc.y * acc.y + acc.z * acc.z + acc.w * acc.w;
        }
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) {
            float acc = 0.0f;
            for (int j = 0; j < top; ++j) {
                const int a = t * top + j;
                const float v = yp[(size_t)row_of[a] * d + i];
                acc += scale ? weights[a] * v : v;
            }
            row_buf[i] = acc;
            ss += acc * acc;
        }
    }
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = x[base + i] + row_buf[i] * inv * to_float(w[i]);
        x[base + i] = v;
        if (lowp) lowp[base + i] = from_float<TL>(v);
    }
}

template <typename TO>
__global__ void cast_rows_kernel(const float* __restrict__ x, TO* __restrict__ out, long long n) {
    pdl_launch();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_float<TO>(x[i]);
}

// What stands between two sublayers of a layer with a norm in front of each and another on its result, in one pass:
//   x[t] += rmsnorm(y[t]) * wy    (y: the sublayer's product, or its split-K partial sums)
//   x[t] += rows[t] + vec         (where a pass of a repeated run of layers begins: the embedded rows, a learned row)
//   out[t] = rmsnorm(x[t]) * w    (what the next sublayer reads)
// each where its pointer is given.  A row's sums are added up in an order fixed by the width alone.
struct NormStepParams {
    float* x;
    const void* y; int parts; size_t part_stride;
    const void* wy; float y_eps;
    const float* rows; const float* vec;
    const void* w; float eps;
    void* out;
    int n_rows, d;
};

template <typename TY, typename TW, typename TO>
__global__ void __launch_bounds__(256) norm_step_kernel(NormStepParams p) {
    extern __shared__ float row_buf[];
    __shared__ float red[32];
    pdl_launch();
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * p.d;
    float inv = 0.0f;
    if (p.y) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < p.d; i += blockDim.x) {
            const float v = sum_parts((const TY*)p.y + base + i, p.parts, p.part_stride);
            row_buf[i] = v;
            ss += v * v;
        }
        ss = block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)p.d + p.y_eps);
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < p.d; i += blockDim.x) {
        float v = p.x[base + i];
        if (p.y) v += row_buf[i] * inv * to_float(((const TW*)p.wy)[i]);
        if (p.rows) v += p.rows[base + i];
        if (p.vec) v += p.vec[i];
        p.x[base + i] = v;
        row_buf[i] = v;
        ss += v * v;
    }
    if (!p.out) return;
    ss = block_sum(ss, red);
    inv = 1.0f / sqrtf(ss / (float)p.d + p.eps);
    for (int i = threadIdx.x; i < p.d; i += blockDim.x)
        ((TO*)p.out)[base + i] = from_float<TO>(row_buf[i] * inv * to_float(((const TW*)p.w)[i]));
}

__device__ __forceinline__ float4 step_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 step_load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void step_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void step_store4(__nv_bfloat16* p, float4 v) {
    uint2 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
    h[0] = __floats2bfloat162_rn(v.x, v.y);
    h[1] = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = raw;
}

// Four columns a thread (d a multiple of 4, everything 16-byte aligned), the row in registers: ITER groups of four a thread.
template <typename TY, typename TW, typename TO, int ITER>
__global__ void __launch_bounds__(1024) norm_step_vec4_kernel(NormStepParams p) {
    __shared__ float red[32];
    pdl_launch();
    const int d4 = p.d >> 2;
    const size_t base = (size_t)blockIdx.x * p.d;
    // bfloat16 weights are asked for before the wait for the kernel ahead (no kernel of the step writes them)
    constexpr bool AHEAD = !std::is_same<TW, float>::value && ITER <= 2;
    uint2 wy_raw[AHEAD ? ITER : 1], w_raw[AHEAD ? ITER : 1];
    if constexpr (AHEAD) {
#pragma unroll
        for (int it = 0; it < ITER; ++it) {
            const int c = threadIdx.x + it * blockDim.x;
            if (c >= d4) continue;
            if (p.y) wy_raw[it] = *reinterpret_cast<const uint2*>((const TW*)p.wy + 4 * c);
            if (p.out) w_raw[it] = *reinterpret_cast<const uint2*>((const TW*)p.w + 4 * c);
        }
    }
    auto weight4 = [&](const void* w, const uint2* raw, int it, int c) {
        if constexpr (AHEAD) return step_load4(reinterpret_cast<const __nv_bfloat16*>(raw + it));
        else return step_load4((const TW*)w + 4 * c);
    };
    pdl_wait();
    float4 xv[ITER];
    float inv = 0.0f;
    {
        float4 yv[ITER];
        float ss = 0.0f;
#pragma unroll
        for (int it = 0; it < ITER; ++it) {                      // the residual and the addend are asked for together
            const int c = threadIdx.x + it * blockDim.x;
            if (c >= d4) continue;
            xv[it] = step_load4(p.x + base + 4 * c);
            if (p.y) {
                if constexpr (std::is_same<TY, float>::value)
                    yv[it] = sum_parts4(reinterpret_cast<const float4*>((const float*)p.y + base) + c, p.parts, p.part_stride / 4);
                else yv[it] = step_load4((const TY*)p.y + base + 4 * c);
                ss += yv[it].x * yv[it].x + yv[it].y * yv[it].y + yv[it].z * yv[it].z + yv[it].w * yv[it].w;
            }
        }
        if (p.y) {
            ss = block_sum(ss, red);
            inv = 1.0f / sqrtf(ss / (float)p.d + p.y_eps);
        }
#pragma unroll
        for (int it = 0; it < ITER; ++it) {
            const int c = threadIdx.x + it * blockDim.x;
            if (c >= d4) continue;
            float4 v = xv[it];
            if (p.y) {
                const float4 w = weight4(p.wy, wy_raw, it, c);
                v.x += yv[it].x * inv * w.x; v.y += yv[it].y * inv * w.y; v.z += yv[it].z * inv * w.z; v.w += yv[it].w * inv * w.w;
            }
            if (p.rows) {
                const float4 a = step_load4(p.rows + base + 4 * c);
                v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
            }
            if (p.vec) {
                const float4 a = step_load4(p.vec + 4 * c);
                v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
            }
            xv[it] = v;
            step_store4(p.x + base + 4 * c, v);
        }
    }
    if (!p.out) return;
    float ss = 0.0f;
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
        const int c = threadIdx.x + it * blockDim.x;
        if (c < d4) ss += xv[it].x * xv[it].x + xv[it].y * xv[it].y + xv[it].z * xv[it].z + xv[it].w * xv[it].w;
    }
    ss = block_sum(ss, red);
    inv = 1.0f / sqrtf(ss / (float)p.d + p.eps);
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
        const int c = threadIdx.x + it * blockDim.x;
        if (c >= d4) continue;
        const float4 w = weight4(p.w, w_raw, it, c), v = xv[it];
        step_store4((TO*)p.out + base + 4 * c, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
    }
}

}  // namespace bg

using namespace bg;

template <typename TY, typename TW, typename TL>
static int rmsnorm_add_launch(float* x, const void* y, int parts, size_t part_stride, const void* w, float eps, void* lowp,
                              int n_rows, int d, cudaStream_t stream) {
    const size_t smem = (size_t)d * sizeof(float);
    if (smem > 200 * 1024) return BG_ERR_SHAPE;
    const bool vec = std::is_same<TY, float>::value && d % 4 == 0 && part_stride % 4 == 0 && (uintptr_t)x % 16 == 0 &&
                     (uintptr_t)y % 16 == 0 && (uintptr_t)lowp % 8 == 0;
    const bool rows_in_registers = std::is_same<TL, __nv_bfloat16>::value && lowp && n_rows >= 64 && d % 8 == 0 && d <= 8 * 32 * 16 &&
                                   part_stride % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                                   (uintptr_t)lowp % 16 == 0;
    if (rows_in_registers) {
        const int iter = (d / 8 + 31) / 32;
        const unsigned blocks = (unsigned)((n_rows + 7) / 8);
#define BG_NORM_ADD_WARP(IT)                                                                                                \
        launch(rmsnorm_add_warp_kernel<TY, TW, IT>, dim3(blocks), dim3(256), 0, stream, x, (const TY*)y, parts, part_stride,     \
               (const TW*)w, eps, (__nv_bfloat16*)lowp, n_rows, d)
        if (iter <= 2) BG_NORM_ADD_WARP(2);
        else if (iter <= 4) BG_NORM_ADD_WARP(4);
        else if (iter <= 8) BG_NORM_ADD_WARP(8);
        else BG_NORM_ADD_WARP(16);
#undef BG_NORM_ADD_WARP
    } else if (vec) {
        auto kern = rmsnorm_add_vec4_kernel<TW, TL>;
        if (smem > BG_SMEM_OPT_IN) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        int threads = ((d / 4 + 31) / 32) * 32;
        threads = threads > 256 ? 256 : (threads < 32 ? 32 : threads);
        launch(kern, dim3(n_rows), dim3(threads), smem, stream, x, (const float*)y, parts, part_stride, (const TW*)w, eps,
               (TL*)lowp, d);
    } else {
        auto kern = rmsnorm_add_kernel<TY, TW, TL>;
        if (smem > BG_SMEM_OPT_IN) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch(kern, dim3(n_rows), dim3(256), smem, stream, x, (const TY*)y, parts, part_stride, (const TW*)w, eps, (TL*)lowp, d);
    }
    BG_LAUNCH_CHECK();
    return BG_OK;
}

// y is [T][d] of y_dtype or float [parts][T][d] with part_stride elements between the parts; lowp may be null.
extern "C" int bg_rmsnorm_add(float* x, const void* y, int y_dtype, int parts, long long part_stride, const void* w,
                              int w_dtype, float eps, void* lowp, int lowp_dtype, int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0) return BG_OK;
    if (parts < 1 || d <= 0) return BG_ERR_SHAPE;
    if (!lowp) lowp_dtype = BG_DTYPE_F32;
    BG_DISPATCH_DTYPE(y_dtype, TY, BG_DISPATCH_DTYPE(w_dtype, TW, BG_DISPATCH_DTYPE(lowp_dtype, TL,
        return (rmsnorm_add_launch<TY, TW, TL>(x, y, parts, (size_t)part_stride, w, eps, lowp, n_rows, d, stream)))));
    return BG_OK;
}

// x [T][d] += norm(sum over a token's `top` rows of yp [T * top][d] float) * w; lowp may be null.
extern "C" int bg_rmsnorm_add_routed(float* x, const float* yp, const int* row_of, const float* weights, int top, int scale,
                                     const void* w, int w_dtype, float eps, void* lowp, int lowp_dtype, int n_rows, int d,
                                     cudaStream_t stream) {
    if (n_rows <= 0) return BG_OK;
    if (top < 1 || d <= 0) return BG_ERR_SHAPE;
    const size_t smem = (size_t)d * sizeof(float);
    if (smem > 200 * 1024) return BG_ERR_SHAPE;
    if (!lowp) lowp_dtype = BG_DTYPE_F32;
    const int vec = d % 4 == 0 && (uintptr_t)yp % 16 == 0;
    int threads = ((d / 4 + 31) / 32) * 32;
    threads = threads > 256 ? 256 : (threads < 32 ? 32 : threads);
#define BG_ROUTED(TW, TL)                                                                                                   \
    do {                                                                                                                    \
        auto kern = rmsnorm_add_routed_kernel<TW, TL>;                                                                      \
        if (smem > BG_SMEM_OPT_IN) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
        launch(kern, dim3(n_rows), dim3(threads), smem, stream, x, yp, row_of, weights, top, scale, (const TW*)w, eps, (TL*)lowp, d, vec); \
    } while (0)
    BG_DISPATCH_DTYPE(w_dtype, TW, BG_DISPATCH_DTYPE(lowp_dtype, TL, BG_ROUTED(TW, TL)));
#undef BG_ROUTED
    BG_LAUNCH_CHECK();
    return BG_OK;
}

extern "C" int bg_cast_rows(const float* x, void* out, int out_dtype, long long n, cudaStream_t stream) {
    if (n <= 0) return BG_OK;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    BG_DISPATCH_DTYPE(out_dtype, TO, launch(cast_rows_kernel<TO>, dim3(blocks), dim3(256), 0, stream, x, (TO*)out, n));
    BG_LAUNCH_CHECK();
    return BG_OK;
}

template <typename TY, typename TW, typename TO>
static int norm_step_launch(const NormStepParams& p, bool vec, cudaStream_t stream) {
    const int d4 = p.d / 4;
    if (vec && d4 <= 4096) {
        // (the number of threads depends on the width alone: it decides the order in which a row is added up)
        int threads = (d4 + 31) / 32 * 32;
        if (threads > 1024) threads = 1024;
        if (threads > 512 && (d4 + 1) / 2 <= 512) threads = ((d4 + 1) / 2 + 31) / 32 * 32;
        const int iter = (d4 + threads - 1) / threads;
        if (iter <= 1) launch(norm_step_vec4_kernel<TY, TW, TO, 1>, dim3(p.n_rows), dim3(threads), 0, stream, p);
        else if (iter <= 2) launch(norm_step_vec4_kernel<TY, TW, TO, 2>, dim3(p.n_rows), dim3(threads), 0, stream, p);
        else launch(norm_step_vec4_kernel<TY, TW, TO, 4>, dim3(p.n_rows), dim3(threads), 0, stream, p);
        BG_LAUNCH_CHECK();
        return BG_OK;
    }
    const size_t smem = (size_t)p.d * sizeof(float);
    if (smem > 200 * 1024) return BG_ERR_SHAPE;
    auto kern = norm_step_kernel<TY, TW, TO>;
    if (smem > BG_SMEM_OPT_IN) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    launch(kern, dim3(p.n_rows), dim3(256), smem, stream, p);
    BG_LAUNCH_CHECK();
    return BG_OK;
}

// See NormStepParams.  y, rows, vec and out may be null; wy and w are of one type (w_dtype).
extern "C" int bg_norm_step(float* x, const void* y, int y_dtype, int parts, long long part_stride, const void* wy, float y_eps,
                            const float* rows, const float* vec, const void* w, int w_dtype, float eps, void* out, int out_dtype,
                            int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0 || d <= 0) return BG_OK;
    if (parts < 1 || (y && !wy) || (out && !w)) return BG_ERR_SHAPE;
    NormStepParams p;
    p.x = x; p.y = y; p.parts = parts; p.part_stride = (size_t)part_stride; p.wy = wy; p.y_eps = y_eps; p.rows = rows; p.vec = vec;
    p.w = w; p.eps = eps; p.out = out; p.n_rows = n_rows; p.d = d;
    if (!y) y_dtype = BG_DTYPE_F32;
    if (!out) out_dtype = BG_DTYPE_F32;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)wy | (uintptr_t)rows | (uintptr_t)vec | (uintptr_t)w | (uintptr_t)out;
    const bool vec4 = d % 4 == 0 && all % 16 == 0 && part_stride % 4 == 0 && (y_dtype == BG_DTYPE_F32 || parts == 1);
    BG_DISPATCH_DTYPE(y_dtype, TY, BG_DISPATCH_DTYPE(w_dtype, TW, BG_DISPATCH_DTYPE(out_dtype, TO,
        return (norm_step_launch<TY, TW, TO>(p, vec4, stream)))));
    return BG_OK;
}
