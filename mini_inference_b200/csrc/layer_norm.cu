// Layer norms (no bias) around a float32 residual stream whose sublayers stand between two of them.  ONE kernel per place:
//
//     v = x + pre + L(y) * wy          (pre: float32 rows, or none; y: a sublayer's output that is normed before it is added, or none)
//     x <- v                           (unless told to leave the stream as it is)
//     out = L(v) * w                   (w null: out = v, the stream's own rows for a product that reads them)
//
// L(z) = (z - mean) / sqrt(variance + eps), the variance being the mean of the squared deviations.  One block per row.  Sums,
// statistics and the stream are float32.  Statistics: every warp finds the mean of its own entries and their squared deviations from
// it; the block then combines the warps' means and squares (no sum of raw squares, so a large common mean costs no digits).
// Rows of a multiple of four entries (up to 8,192) stay in registers from the first load to the output; other rows are read again.
#include "common.cuh"

using namespace mi;

namespace {

constexpr int LOOP_NT = 256;

struct Moments { float mean, rstd; };

// what the warps found (mean of their entries, squared deviations from it, entries) -> the row's mean and 1 / deviation
// (scratch: a float4 per warp that no earlier call of the block has used)
template <int NW>
__device__ __forceinline__ Moments combine(float mean_w, float m2, float count, float4* scratch, int hidden, float eps) {
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = make_float4(mean_w, m2, count, 0.f);
    __syncthreads();
    const float inv = 1.f / hidden;
    float4 p[NW];
    float total = 0.f, sq = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) { p[w] = scratch[w]; total = fmaf(p[w].x, p[w].z, total); }
    const float mean = total * inv;
#pragma unroll
    for (int w = 0; w < NW; ++w) { const float d = p[w].x - mean; sq += fmaf(p[w].z * d, d, p[w].y); }
    return Moments{mean, rsqrtf(sq * inv + eps)};
}

template <typename TD> __device__ __forceinline__ float4 load4(const TD* p) {
    if constexpr (sizeof(TD) == 4) {
        return *reinterpret_cast<const float4*>(p);
    } else {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xffff0000u));
    }
}
template <typename TY> __device__ __forceinline__ void store4(TY* p, float4 v) {
    if constexpr (sizeof(TY) == 4) {
        *reinterpret_cast<float4*>(p) = v;
    } else {
        store2(p, v.x, v.y);
        store2(p + 2, v.z, v.w);
    }
}

// Mean and deviation of a row held as v[VPT] (thread t: quads t, t + NT, ..; entries beyond the row are zero and not counted)
template <int NT, int VPT>
__device__ __forceinline__ Moments row_moments(const float4 (&v)[VPT], int quads, int hidden, float eps, float4* scratch) {
    const int warp0 = threadIdx.x & ~31;
    float sum = 0.f, count = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        sum += (v[k].x + v[k].y) + (v[k].z + v[k].w);
        count += 4.f * (float)max(0, min(32, quads - warp0 - k * NT));
    }
    sum = warp_sum(sum);
    const float m = count > 0.f ? sum / count : 0.f;
    float m2 = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
        if ((int)threadIdx.x + k * NT < quads) {
            const float a = v[k].x - m, b = v[k].y - m, c = v[k].z - m, d = v[k].w - m;
            m2 += (a * a + b * b) + (c * c + d * d);
        }
    return combine<NT / 32>(m, warp_sum(m2), count, scratch, hidden, eps);
}

// NT threads a row (few for many rows, so that more rows are in flight; many for few rows), VPT quads a thread
template <typename TD, typename TY, int NT, int VPT>
__global__ void __launch_bounds__(NT) stream_layernorm_vec_kernel(float* __restrict__ x, const TD* __restrict__ y, const float* __restrict__ wy, float eps_y,
                                                                  const float* __restrict__ pre, const float* __restrict__ w, TY* __restrict__ out,
                                                                  const int* __restrict__ rows, int hidden, float eps, int keep) {
    __shared__ float4 scratch[2][NT / 32];
    const size_t r = (rows ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x) * hidden;
    const int quads = hidden >> 2;
    constexpr bool AHEAD = VPT <= 2;                          // the weights are fetched before the row, so that no wait for them follows a sum
    pdl_trigger();
    float4 v[VPT], wv[AHEAD ? VPT : 1], wyv[AHEAD ? VPT : 1];
    if constexpr (AHEAD) {
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int q = threadIdx.x + k * NT;
            wv[k] = w && q < quads ? *reinterpret_cast<const float4*>(w + 4 * q) : make_float4(1.f, 1.f, 1.f, 1.f);
            wyv[k] = y && q < quads ? *reinterpret_cast<const float4*>(wy + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    pdl_wait();
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int q = threadIdx.x + k * NT;
        v[k] = q < quads ? *reinterpret_cast<const float4*>(x + r + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (pre && q < quads) {
            const float4 a = *reinterpret_cast<const float4*>(pre + r + 4 * q);
            v[k].x += a.x; v[k].y += a.y; v[k].z += a.z; v[k].w += a.w;
        }
    }
    if (y) {
        float4 d[VPT];
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int q = threadIdx.x + k * NT;
            d[k] = q < quads ? load4<TD>(y + r + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        const Moments m = row_moments<NT, VPT>(d, quads, hidden, eps_y, scratch[0]);
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int q = threadIdx.x + k * NT;
            if (q < quads) {
                const float4 a = AHEAD ? wyv[AHEAD ? k : 0] : *reinterpret_cast<const float4*>(wy + 4 * q);
                v[k].x = fmaf((d[k].x - m.mean) * m.rstd, a.x, v[k].x); v[k].y = fmaf((d[k].y - m.mean) * m.rstd, a.y, v[k].y);
                v[k].z = fmaf((d[k].z - m.mean) * m.rstd, a.z, v[k].z); v[k].w = fmaf((d[k].w - m.mean) * m.rstd, a.w, v[k].w);
            }
        }
    }
    Moments m{0.f, 1.f};
    if (w) m = row_moments<NT, VPT>(v, quads, hidden, eps, scratch[1]);
    TY* o = out + (size_t)blockIdx.x * hidden;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int q = threadIdx.x + k * NT;
        if (q >= quads) continue;
        if (!keep) *reinterpret_cast<float4*>(x + r + 4 * q) = v[k];
        float4 a = wv[AHEAD ? k : 0];
        if (!AHEAD) a = w ? *reinterpret_cast<const float4*>(w + 4 * q) : make_float4(1.f, 1.f, 1.f, 1.f);
        store4<TY>(o + 4 * q, make_float4((v[k].x - m.mean) * m.rstd * a.x, (v[k].y - m.mean) * m.rstd * a.y, (v[k].z - m.mean) * m.rstd * a.z,
                                          (v[k].w - m.mean) * m.rstd * a.w));
    }
}

// the statistics of a row whose entry i is at(i), i over the block's threads
template <typename F> __device__ __forceinline__ Moments loop_moments(F at, int hidden, float eps, float4* scratch) {
    float sum = 0.f, count = 0.f;
    for (int i = threadIdx.x; i < hidden; i += LOOP_NT) { sum += at(i); count += 1.f; }
    sum = warp_sum(sum);
    count = warp_sum(count);
    const float m = count > 0.f ? sum / count : 0.f;
    float m2 = 0.f;
    for (int i = threadIdx.x; i < hidden; i += LOOP_NT) { const float d = at(i) - m; m2 += d * d; }
    return combine<LOOP_NT / 32>(m, warp_sum(m2), count, scratch, hidden, eps);
}

template <typename TD, typename TY>
__global__ void __launch_bounds__(LOOP_NT) stream_layernorm_kernel(float* __restrict__ x, const TD* __restrict__ y, const float* __restrict__ wy, float eps_y,
                                                              const float* __restrict__ pre, const float* __restrict__ w, TY* __restrict__ out,
                                                              const int* __restrict__ rows, int hidden, float eps, int keep) {
    __shared__ float4 scratch[2][LOOP_NT / 32];
    pdl_trigger();
    pdl_wait();
    const size_t r = (rows ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x) * hidden;
    Moments my{0.f, 0.f};
    if (y) my = loop_moments([&](int i) { return to_f32(y[r + i]); }, hidden, eps_y, scratch[0]);
    auto sum = [&](int i) {                                   // the row as it will be; x is written only after its last reading
        float v = x[r + i];
        if (pre) v += pre[r + i];
        if (y) v = fmaf((to_f32(y[r + i]) - my.mean) * my.rstd, wy[i], v);
        return v;
    };
    Moments m{0.f, 1.f};
    if (w) m = loop_moments(sum, hidden, eps, scratch[1]);
    TY* o = out + (size_t)blockIdx.x * hidden;
    for (int i = threadIdx.x; i < hidden; i += LOOP_NT) {
        const float v = sum(i);
        if (!keep) x[r + i] = v;
        o[i] = from_f32<TY>((v - m.mean) * m.rstd * (w ? w[i] : 1.f));
    }
}

}  // namespace

// x float32 [T, hidden]; y [T, hidden] in y_dtype or null; pre float32 [T, hidden] or null; out [n, hidden] in out_dtype.
// rows: output row i reads stream row rows[i]; keep != 0: x is left as it is (rows implies it).
MI_EXPORT int mi_stream_layernorm(float* x, const void* y, const float* wy, float eps_y, const float* pre, const float* w, void* out, const int* rows,
                                  int n, int hidden, float eps, int keep, int y_dtype, int out_dtype, cudaStream_t stream) {
    if (n == 0) return 0;
    if (y && !wy) return -2;
    keep = keep || rows || (!y && !pre);
    const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)wy | (uintptr_t)pre | (uintptr_t)w | (uintptr_t)out;
    const bool vec = hidden % 4 == 0 && hidden <= 8192 && all % 16 == 0;
    const int quads = hidden / 4;
#define VEC(TD, TY, NT, VPT) return (int)launch_pdl(stream_layernorm_vec_kernel<TD, TY, NT, VPT>, dim3(n), dim3(NT), 0, stream, x, (const TD*)y, wy, eps_y, pre, w, (TY*)out, rows, hidden, eps, keep)
#define GO(TD, TY) do { \
        if (!vec) return (int)launch_pdl(stream_layernorm_kernel<TD, TY>, dim3(n), dim3(LOOP_NT), 0, stream, x, (const TD*)y, wy, eps_y, pre, w, (TY*)out, rows, hidden, eps, keep); \
        if (n >= 512) { if (quads <= 128) VEC(TD, TY, 128, 1); else if (quads <= 256) VEC(TD, TY, 128, 2); else if (quads <= 512) VEC(TD, TY, 128, 4); \
                        else if (quads <= 1024) VEC(TD, TY, 256, 4); else VEC(TD, TY, 256, 8); } \
        if (quads <= 256) VEC(TD, TY, 256, 1); else if (quads <= 512) VEC(TD, TY, 256, 2); else if (quads <= 1024) VEC(TD, TY, 512, 2); \
        else VEC(TD, TY, 512, 4); } while (0)
    if (y_dtype == MI_BF16 && out_dtype == MI_BF16) GO(__nv_bfloat16, __nv_bfloat16);
    else if (y_dtype == MI_F32 && out_dtype == MI_F32) GO(float, float);
    return -1;
#undef GO
#undef VEC
}
