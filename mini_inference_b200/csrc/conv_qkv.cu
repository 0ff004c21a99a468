// Between the q | k | v product and attention, for mixers whose projections pass a short causal convolution:
//     u = p + bias;  y_t = sum_j w[:, j] u_(t - taps + 1 + j) per channel (zeros before a sequence's first position);
//     q and k: divided by the root mean square over the WHOLE projection (all heads), times a weight per channel, then the first
//     2 nf coordinates of every head turned pairwise (2i with 2i + 1; angle = position * inv_freq[i]); v as convolved.
// q goes to a tensor of its own (the projected rows are still read by the convolution of later tokens), k and v to the token's slot of
// the pages.  The inputs u of the taps - 1 positions before an entry's first token are rows of state[slot], float32 [taps - 1, C]
// (zeros for a request's first entry); the entry's newest inputs are left there: by the kernel itself in a step whose entries bring
// one token each (a channel of a slot then has one reader), by a kernel behind it otherwise.
// Convolution, norms and rotation are float32.  grid.y = 0 takes the q channels, 1 the k and v channels (KV = 0: no such block).
#include "common.cuh"
#include <math.h>

using namespace mi;

namespace {

struct ConvQkv {
    const float *bias, *q_w, *k_w, *inv_freq;
    float* state;
    long long state_stride;
    const int *positions, *slots, *token_seg, *seg_q_start, *seg_slot;
    int T, H, KV, D, V, nf, ps, shift;
    float eps;
};

// Any sizes: one block per token; the convolved channels wait in shared memory for the norm.
template <typename T>
__global__ void __launch_bounds__(256) conv_qkv_kernel(const T* __restrict__ p, int ldp, const T* __restrict__ w, int taps, T* __restrict__ q_out,
                                                       T* __restrict__ k_cache, T* __restrict__ v_cache, const ConvQkv a) {
    extern __shared__ float ysm[];
    __shared__ float scratch[32];
    const int t = blockIdx.x, seg = a.token_seg[t], qs = a.seg_q_start[seg], r = t - qs;
    const int HD = a.H * a.D, KD = a.KV * a.D, C = HD + KD + a.KV * a.V;
    const bool kv = blockIdx.y == 1;
    const int c0 = kv ? HD : 0, n = kv ? C - HD : HD, normed = kv ? KD : HD;
    float* hist = taps > 1 ? a.state + (long long)a.seg_slot[seg] * a.state_stride : nullptr;
    float* cs = ysm + n;                                        // [nf] cosines, [nf] sines
    const float pos = (float)a.positions[t];
    for (int i = threadIdx.x; i < a.nf; i += 256) sincosf(pos * a.inv_freq[i], &cs[a.nf + i], &cs[i]);
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += 256) {
        const int c = c0 + i;
        const float b = a.bias[c], own = to_f32(p[(size_t)t * ldp + c]) + b;
        float y = 0.f;
        for (int j = 0; j < taps; ++j) {
            const int off = r - (taps - 1 - j);
            const float u = j == taps - 1 ? own : off >= 0 ? to_f32(p[(size_t)(qs + off) * ldp + c]) + b : hist[(size_t)(taps - 1 + off) * C + c];
            y = fmaf(to_f32(w[(size_t)c * taps + j]), u, y);
        }
        ysm[i] = y;
        if (i < normed) ss += y * y;
        if (a.shift && taps > 1) {
            for (int j = 0; j + 2 < taps; ++j) hist[(size_t)j * C + c] = hist[(size_t)(j + 1) * C + c];
            hist[(size_t)(taps - 2) * C + c] = own;
        }
    }
    const float s = rsqrtf(block_sum<256>(ss, scratch) / normed + a.eps);
    const float* nw = kv ? a.k_w : a.q_w;
    const int slot = a.slots[t];
    const long long page = slot / a.ps, off = slot % a.ps;
    for (int i = threadIdx.x; i < n; i += 256) {
        if (i >= normed) {
            const int h = (i - normed) / a.V, d = (i - normed) % a.V;
            v_cache[((page * a.KV + h) * a.ps + off) * a.V + d] = from_f32<T>(ysm[i]);
            continue;
        }
        const int h = i / a.D, d = i % a.D;
        float v = ysm[i] * s * nw[i];
        if (d < 2 * a.nf) {
            const int o = d & 1 ? i - 1 : i + 1, f = d >> 1;
            const float other = ysm[o] * s * nw[o];
            v = d & 1 ? v * cs[f] + other * cs[a.nf + f] : v * cs[f] - other * cs[a.nf + f];
        }
        if (kv) k_cache[((page * a.KV + h) * a.ps + off) * a.D + d] = from_f32<T>(v);
        else q_out[(size_t)t * HD + i] = from_f32<T>(v);
    }
}

__device__ __forceinline__ void eight(const __nv_bfloat16* p, float (&x)[8]) { load16<__nv_bfloat16>(p, x); }
__device__ __forceinline__ void eight(const float* p, float (&x)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}
__device__ __forceinline__ void store_eight(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 o;
    __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
    for (int e = 0; e < 4; ++e) oh[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = o;
}

// bfloat16, head sizes in multiples of eight: a thread owns eight neighbouring channels (their taps in registers) of TOK neighbouring
// tokens; the TOK sums of squares are reduced together.
template <int TAPS, int TOK, int MAXT>
__global__ void __launch_bounds__(MAXT) conv_qkv_vec_kernel(const __nv_bfloat16* __restrict__ p, int ldp, const __nv_bfloat16* __restrict__ w,
                                                            __nv_bfloat16* __restrict__ q_out, __nv_bfloat16* __restrict__ k_cache,
                                                            __nv_bfloat16* __restrict__ v_cache, const ConvQkv a) {
    extern __shared__ float csm[];                              // [TOK][nf] cosines, then sines
    __shared__ float part[TOK][32];
    const int t0 = blockIdx.x * TOK, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int HD = a.H * a.D, KD = a.KV * a.D, C = HD + KD + a.KV * a.V;
    const bool kv = blockIdx.y == 1;
    const int c0 = kv ? HD : 0, n = kv ? C - HD : HD, normed = kv ? KD : HD;
    const int i0 = threadIdx.x * 8, c = c0 + i0;
    const bool live = i0 < n;
    // inside one entry, beyond its first taps: all rows that the TOK tokens read are fetched at once (no history, no look-ups between)
    constexpr int ROWS = TOK + TAPS - 1;
    const int seg0 = a.token_seg[t0];
    const bool inside = TOK > 1 && t0 + TOK <= a.T && a.token_seg[min(t0 + TOK, a.T) - 1] == seg0 && t0 - a.seg_q_start[seg0] >= TAPS - 1;
    uint4 raw[ROWS];
    if (inside && live) {
#pragma unroll
        for (int i = 0; i < ROWS; ++i) raw[i] = *reinterpret_cast<const uint4*>(p + (size_t)(t0 - (TAPS - 1) + i) * ldp + c);
    }
    for (int i = threadIdx.x; i < TOK * a.nf; i += blockDim.x) {
        const int k = i / a.nf, f = i - k * a.nf;
        sincosf((float)a.positions[min(t0 + k, a.T - 1)] * a.inv_freq[f], &csm[TOK * a.nf + i], &csm[i]);
    }
    float y[TOK][8], ss[TOK];
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
        ss[k] = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) y[k][e] = 0.f;
    }
    if (live) {
        float bias[8];
        eight(a.bias + c, bias);
        uint32_t wr[4 * TAPS];                                   // 8 TAPS bfloat16: channel e, tap j at e TAPS + j
#pragma unroll
        for (int i = 0; i < TAPS; ++i) *reinterpret_cast<uint4*>(wr + 4 * i) = *reinterpret_cast<const uint4*>(w + (size_t)c * TAPS + 8 * i);
        auto tap = [&](int e, int j) {
            const int at = e * TAPS + j;
            return __uint_as_float(at & 1 ? wr[at >> 1] & 0xffff0000u : wr[at >> 1] << 16);
        };
        if (inside) {
#pragma unroll
            for (int k = 0; k < TOK; ++k)
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {                 // the order of the general form: per token, taps ascending
                    const uint32_t q[4] = {raw[k + j].x, raw[k + j].y, raw[k + j].z, raw[k + j].w};
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const float u = __uint_as_float(e & 1 ? q[e >> 1] & 0xffff0000u : q[e >> 1] << 16) + bias[e];
                        y[k][e] = fmaf(tap(e, j), u, y[k][e]);
                    }
                }
        } else
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
            const int t = t0 + k;
            if (t >= a.T) break;
            const int seg = a.token_seg[t], qs = a.seg_q_start[seg], r = t - qs;
            float* hist = TAPS > 1 ? a.state + (long long)a.seg_slot[seg] * a.state_stride + c : nullptr;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                const int off = r - (TAPS - 1 - j);
                float u[8];
                if (off >= 0) {
                    eight(p + (size_t)(qs + off) * ldp + c, u);
#pragma unroll
                    for (int e = 0; e < 8; ++e) u[e] += bias[e];
                } else {
                    eight(hist + (size_t)(TAPS - 1 + off) * C, u);
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) y[k][e] = fmaf(tap(e, j), u[e], y[k][e]);
                if (a.shift && j > 0) {                          // single-token entries: row j of the inputs is row j - 1 of the next step's history
                    float* hw = hist + (size_t)(j - 1) * C;
                    *reinterpret_cast<float4*>(hw) = make_float4(u[0], u[1], u[2], u[3]);
                    *reinterpret_cast<float4*>(hw + 4) = make_float4(u[4], u[5], u[6], u[7]);
                }
            }
        }
        if (i0 < normed) {
#pragma unroll
            for (int k = 0; k < TOK; ++k)
#pragma unroll
                for (int e = 0; e < 8; ++e) ss[k] += y[k][e] * y[k][e];
        }
    }
#pragma unroll
    for (int k = 0; k < TOK; ++k) ss[k] = warp_sum(ss[k]);
    if (lane == 0) {
#pragma unroll
        for (int k = 0; k < TOK; ++k) part[k][warp] = ss[k];
    }
    __syncthreads();
    if (!live) return;
    const bool value = i0 >= normed;
    float nw[8];
    if (!value) eight((kv ? a.k_w : a.q_w) + i0, nw);
    const int h = value ? (i0 - normed) / a.V : i0 / a.D, d = value ? (i0 - normed) % a.V : i0 % a.D;
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
        const int t = t0 + k;
        if (t >= a.T) break;
        const int slot = kv ? a.slots[t] : 0;
        const long long row = kv ? ((long long)(slot / a.ps) * a.KV + h) * a.ps + slot % a.ps : 0;
        if (value) { store_eight(v_cache + row * a.V + d, y[k]); continue; }
        float total = 0.f;
        for (int i = 0; i < warps; ++i) total += part[k][i];
        const float s = rsqrtf(total / normed + a.eps);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[k][e] *= s * nw[e];
#pragma unroll
        for (int e = 0; e < 8; e += 2)
            if (d + e < 2 * a.nf) {
                const float co = csm[k * a.nf + ((d + e) >> 1)], si = csm[(TOK + k) * a.nf + ((d + e) >> 1)], u = y[k][e], v = y[k][e + 1];
                y[k][e] = u * co - v * si;
                y[k][e + 1] = v * co + u * si;
            }
        if (kv) store_eight(k_cache + row * a.D + d, y[k]);
        else store_eight(q_out + (size_t)t * HD + i0, y[k]);
    }
}

// state[slot][j] <- input u at (entry's end - (taps - 1) + j); a thread owns a channel and goes up in j, so an entry shorter than
// taps - 1 shifts its own rows safely.
template <typename T>
__global__ void conv_qkv_tail_kernel(const T* __restrict__ p, int ldp, const float* __restrict__ bias, float* __restrict__ state, long long state_stride,
                                     const int* __restrict__ seg_q_start, const int* __restrict__ seg_slot, int C, int taps) {
    const int seg = blockIdx.x, qs = seg_q_start[seg], n = seg_q_start[seg + 1] - qs, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    float* hist = state + (long long)seg_slot[seg] * state_stride;
    for (int j = 0; j < taps - 1; ++j) {
        const int src = n - (taps - 1) + j;
        hist[(size_t)j * C + c] = src >= 0 ? to_f32(p[(size_t)(qs + src) * ldp + c]) + bias[c] : hist[(size_t)(taps - 1 + src) * C + c];
    }
}

}  // namespace

// p [T, ldp] = q | k | v | ..; w [C, taps] in p's type, C = H D + KV (D + V); q_out [T, H D]; KV = 0: no keys and values (k_w, caches null)
MI_EXPORT int mi_conv_qkv_cache(const void* p, int ldp, const float* bias, const void* w, int taps, const float* q_w, const float* k_w, float eps,
                                const float* inv_freq, int nf, float* state, long long state_stride, void* q_out, void* k_cache, void* v_cache,
                                const int* positions, const int* slots, const int* token_seg, const int* seg_q_start, const int* seg_slot, int T_,
                                int num_segs, int H, int KV, int D, int V, int ps, int dtype, cudaStream_t stream) {
    if (T_ == 0) return 0;
    if (2 * nf > D || taps < 1 || (taps > 1 && !state) || (KV > 0 && (!k_cache || !v_cache || !k_w))) return -2;
    const int HD = H * D, KD = KV * D, C = HD + KD + KV * V, widest = HD > C - HD ? HD : C - HD;
    const int shift = T_ == num_segs ? 1 : 0;
    const ConvQkv a{bias, q_w, k_w, inv_freq, state, state_stride, positions, slots, token_seg, seg_q_start, seg_slot, T_, H, KV, D, V, nf, ps, shift, eps};
    const int ny = KV > 0 ? 2 : 1;
    const bool vec = dtype == MI_BF16 && D % 8 == 0 && (KV == 0 || V % 8 == 0) && ldp % 8 == 0 && taps <= 4 && widest <= 8192 && nf <= 512 &&
                     ((uintptr_t)p | (uintptr_t)w | (uintptr_t)bias | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)q_out | (uintptr_t)k_cache |
                      (uintptr_t)v_cache | (uintptr_t)state) % 16 == 0 && (taps == 1 || state_stride % 4 == 0);
    if (vec) {
        const int threads = (widest / 8 + 31) / 32 * 32;
#define GO(TAPS, TOK, MAXT) conv_qkv_vec_kernel<TAPS, TOK, MAXT><<<dim3((T_ + TOK - 1) / TOK, ny), threads, 2 * TOK * nf * sizeof(float), stream>>>( \
            (const __nv_bfloat16*)p, ldp, (const __nv_bfloat16*)w, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, a)
#define PICK(TAPS) do { if (T_ < 512) { if (threads <= 512) GO(TAPS, 1, 512); else GO(TAPS, 1, 1024); } \
                        else if (threads <= 512) GO(TAPS, 4, 512); else GO(TAPS, 2, 1024); } while (0)
        if (taps == 1) PICK(1); else if (taps == 2) PICK(2); else if (taps == 3) PICK(3); else PICK(4);
#undef PICK
#undef GO
    } else {
        const size_t smem = (size_t)(widest + 2 * nf) * sizeof(float);
        if (smem > 200 * 1024) return -2;
#define GO(T) do { if (smem > 48 * 1024) cudaFuncSetAttribute(conv_qkv_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
        conv_qkv_kernel<T><<<dim3(T_, ny), 256, smem, stream>>>((const T*)p, ldp, (const T*)w, taps, (T*)q_out, (T*)k_cache, (T*)v_cache, a); } while (0)
        if (dtype == MI_BF16) GO(__nv_bfloat16); else GO(float);
#undef GO
    }
    const int err = (int)cudaGetLastError();
    if (err || taps <= 1 || shift) return err;
    const dim3 tgrid(num_segs, (C + 255) / 256);
    if (dtype == MI_BF16) conv_qkv_tail_kernel<__nv_bfloat16><<<tgrid, 256, 0, stream>>>((const __nv_bfloat16*)p, ldp, bias, state, state_stride, seg_q_start, seg_slot, C, taps);
    else conv_qkv_tail_kernel<float><<<tgrid, 256, 0, stream>>>((const float*)p, ldp, bias, state, state_stride, seg_q_start, seg_slot, C, taps);
    return (int)cudaGetLastError();
}
