// The kernel of an arrangement whose norms stand behind the sums, on a float32 residual stream:
//     x <- w * N(alpha * x + y),  N(z) = z / sqrt(mean(z^2) + eps),  and x's rows in the run's type for the next product.
// One block per row; sum, statistic and stream are float32.  Rows of a multiple of four entries (up to 8,192) stay in registers
// between the statistic and the output (16-byte loads of the stream); other rows are written once unnormed and read back.
#include "common.cuh"

using namespace mi;

namespace {

constexpr int NT = 256;

template <typename TD, typename TR>
__global__ void __launch_bounds__(NT) sum_rmsnorm_kernel(float* __restrict__ x, const TD* __restrict__ y, const float* __restrict__ w,
                                                         TR* __restrict__ rows, int hidden, float alpha, float eps) {
    __shared__ float scratch[32];
    float* xr = x + (size_t)blockIdx.x * hidden;
    const TD* yr = y + (size_t)blockIdx.x * hidden;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += NT) {
        const float v = fmaf(alpha, xr[i], to_f32(yr[i]));
        xr[i] = v;
        ss += v * v;
    }
    const float s = rsqrtf(block_sum<NT>(ss, scratch) / hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += NT) {              // this thread's own writes of the first pass
        const float v = xr[i] * s * w[i];
        xr[i] = v;
        if (rows) rows[(size_t)blockIdx.x * hidden + i] = from_f32<TR>(v);
    }
}

template <typename TD> __device__ __forceinline__ float4 four(const TD* p) {
    if constexpr (sizeof(TD) == 4) {
        return *reinterpret_cast<const float4*>(p);
    } else {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xffff0000u));
    }
}

template <typename TD, int VPT>
__global__ void __launch_bounds__(NT) sum_rmsnorm_vec_kernel(float* __restrict__ x, const TD* __restrict__ y, const float* __restrict__ w,
                                                             __nv_bfloat16* __restrict__ rows, int hidden, float alpha, float eps) {
    __shared__ float scratch[32];
    float* xr = x + (size_t)blockIdx.x * hidden;
    const TD* yr = y + (size_t)blockIdx.x * hidden;
    const int quads = hidden >> 2;
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int q = threadIdx.x + k * NT;
        if (q < quads) {
            const float4 a = *reinterpret_cast<const float4*>(xr + 4 * q), d = four<TD>(yr + 4 * q);
            v[k] = make_float4(fmaf(alpha, a.x, d.x), fmaf(alpha, a.y, d.y), fmaf(alpha, a.z, d.z), fmaf(alpha, a.w, d.w));
            ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
        }
    }
    const float s = rsqrtf(block_sum<NT>(ss, scratch) / hidden + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int q = threadIdx.x + k * NT;
        if (q < quads) {
            const float4 wv = *reinterpret_cast<const float4*>(w + 4 * q);
            const float4 o = make_float4(v[k].x * s * wv.x, v[k].y * s * wv.y, v[k].z * s * wv.z, v[k].w * s * wv.w);
            *reinterpret_cast<float4*>(xr + 4 * q) = o;
            if (rows) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(o.x, o.y), hi = __floats2bfloat162_rn(o.z, o.w);
                uint2 r;
                r.x = *reinterpret_cast<uint32_t*>(&lo);
                r.y = *reinterpret_cast<uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(rows + (size_t)blockIdx.x * hidden + 4 * q) = r;
            }
        }
    }
}

}  // namespace

// y [n, hidden] in y_dtype; rows: null or [n, hidden] bfloat16
MI_EXPORT int mi_sum_rmsnorm(float* x, const void* y, const float* w, void* rows, int n, int hidden, float alpha, float eps, int y_dtype,
                             cudaStream_t stream) {
    if (n == 0) return 0;
    const bool vec = hidden % 4 == 0 && hidden <= 8 * 4 * NT && ((uintptr_t)x | (uintptr_t)y | (uintptr_t)w) % 16 == 0 && (uintptr_t)rows % 8 == 0;
    const int quads = hidden / 4;
#define GO(TD, VPT) sum_rmsnorm_vec_kernel<TD, VPT><<<n, NT, 0, stream>>>(x, (const TD*)y, w, (__nv_bfloat16*)rows, hidden, alpha, eps)
#define PICK(TD) do { if (quads <= NT) GO(TD, 1); else if (quads <= 2 * NT) GO(TD, 2); else if (quads <= 4 * NT) GO(TD, 4); else GO(TD, 8); } while (0)
    if (vec) { if (y_dtype == MI_BF16) PICK(__nv_bfloat16); else PICK(float); }
    else if (y_dtype == MI_BF16) sum_rmsnorm_kernel<__nv_bfloat16, __nv_bfloat16><<<n, NT, 0, stream>>>(x, (const __nv_bfloat16*)y, w, (__nv_bfloat16*)rows, hidden, alpha, eps);
    else sum_rmsnorm_kernel<float, __nv_bfloat16><<<n, NT, 0, stream>>>(x, (const float*)y, w, (__nv_bfloat16*)rows, hidden, alpha, eps);
#undef PICK
#undef GO
    return (int)cudaGetLastError();
}
