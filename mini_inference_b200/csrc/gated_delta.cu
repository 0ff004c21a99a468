// Gated delta rule with one decay per head and token, around the state scan of recurrent.cu:
//
//     q, k, v = silu(conv(.));  q, k <- x / sqrt(sum x^2 + unit_eps), q also * key_dim^-1/2;  beta = sigmoid(b);  f = exp(-rate softplus(a + dt_bias))
//     S <- f S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;     rows: o / rms(o) * weight * silu(gate) per head
//
// p [T, ldp] as projected: q [KV D] | k [KV D] | v [H V] (the C channels that pass the convolution) | gate [H V] | b [H] | a [H] | ..
// conv float32 [C, taps], the last tap multiplies the current token.  A request's slot holds S (float32 [H, D, V]) and behind it a ring
// of the convolution's inputs, [taps, C]: position p has row p mod taps, positions before 0 count as zeros.
//
// Prompts: delta_ready_kernel makes what the scan reads (float32 rows q | k | v | beta | f | log f), the scan runs (gated_delta_chunk.cu, or
// token by token in recurrent.cu), then delta_ring_kernel writes the entry's newest inputs into the ring.  Decode steps (every entry one token): delta_step_kernel does all of
// it in one pass over the state, one block per (entry, head).  The ring has one row more than a token looks back on, so the block that
// writes a token's inputs overwrites none that the other heads' blocks (which share a q and k head) still read.
// Everything is float32.  The decay acts on a state hundreds of times in a row, so it is made as 1 + expm1(.) where it is near one: rounded
// once, not one-sided.
#include "sm100.cuh"
#include <math.h>

using namespace mi;
using namespace mi::sm100;

namespace {

__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
// behind a convolution of bfloat16 inputs the fast exponential and quotient (a few units in the last place of float32) are as good
template <typename T> __device__ __forceinline__ float conv_silu(float x) {
    if constexpr (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-x));
    else return silu(x);
}
__device__ __forceinline__ float log_decay(float a, float dt_bias, float rate) {
    const float z = a + dt_bias;
    return -rate * (z > 20.f ? z : log1pf(expf(z)));
}
__device__ __forceinline__ float decay_of(float log_f) { return log_f > -0.7f ? 1.f + expm1f(log_f) : expf(log_f); }

// ------------------------------------------------------------------ prompts: what the scan reads
// grid (token groups of TOK, units / 4), four warps, a warp per unit: the KV q heads, the KV k heads, then the value channels in pieces of
// 32 NI, then one unit for the gates of all heads.  A lane owns the channels c0 + lane + 32 i of its unit (i < NI) with their taps in
// registers.  A group inside one entry fetches its inputs all at once; a group that crosses entries goes token by token.
template <typename T, int TAPS, int NI, int TOK>
__global__ void __launch_bounds__(128) delta_ready_kernel(const T* __restrict__ p, int ldp, const float* __restrict__ conv, const float* __restrict__ rate,
                                                          const float* __restrict__ dt_bias, const float* __restrict__ state, long long state_stride,
                                                          long long ring_off, float* __restrict__ out, int ldo, const int* __restrict__ positions,
                                                          const int* __restrict__ token_seg, const int* __restrict__ seg_q_start,
                                                          const int* __restrict__ seg_slot, int T_, int H, int KV, int D, int V, int taps_, float unit_eps,
                                                          float q_scale) {
    constexpr int W = TAPS > 0 ? TAPS : 1;                     // TAPS 0: any number of taps, read again for every token
    const int taps = TAPS > 0 ? TAPS : taps_;
    const int lane = threadIdx.x & 31, unit = blockIdx.y * 4 + (threadIdx.x >> 5);
    const int C = 2 * KV * D + H * V, pieces = (H * V + 32 * NI - 1) / (32 * NI);
    const int t0 = blockIdx.x * TOK, t1 = min(T_, t0 + TOK);
    if (unit > 2 * KV + pieces) return;
    if (unit == 2 * KV + pieces) {                             // beta, f and log f of every head
        for (int i = lane; i < (t1 - t0) * H; i += 32) {
            const int t = t0 + i / H, h = i % H;
            const T* row = p + (size_t)t * ldp + C + H * V;
            float* o = out + (size_t)t * ldo + C;
            const float lf = log_decay(to_f32(row[H + h]), dt_bias[h], rate[h]);
            o[h] = 1.f / (1.f + expf(-to_f32(row[h])));
            o[H + h] = decay_of(lf);
            o[2 * H + h] = lf;
        }
        return;
    }
    const bool head = unit < 2 * KV;
    const int c0 = head ? unit * D : 2 * KV * D + (unit - 2 * KV) * 32 * NI;
    const int n = head ? D : min(32 * NI, C - c0);
    auto finish = [&](float (&y)[NI], int t) {                 // silu, the head's unit norm, out
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) { y[i] = lane + 32 * i < n ? conv_silu<T>(y[i]) : 0.f; ss = fmaf(y[i], y[i], ss); }
        float s = 1.f;
        if (head) s = (unit < KV ? q_scale : 1.f) / sqrtf(warp_sum(ss) + unit_eps);
        float* o = out + (size_t)t * ldo + c0;
#pragma unroll
        for (int i = 0; i < NI; ++i)
            if (lane + 32 * i < n) o[lane + 32 * i] = y[i] * s;
    };
    auto input = [&](int c, int back, int t, int r, int pos, const float* ring) {      // the input `back` tokens before t
        if (back <= r) return to_f32(p[(size_t)(t - back) * ldp + c]);
        return back <= pos ? ring[(size_t)((pos - back) % taps) * C + c] : 0.f;
    };
    if (TAPS > 0 && t1 - t0 == TOK) {
        // the rows are fetched before it is known where the tokens stand in their entry; what lies before the entry is replaced then
        float w[NI][W], x[NI][TOK + W - 1];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = c0 + lane + 32 * i;
            const bool mine = lane + 32 * i < n;
#pragma unroll
            for (int j = 0; j < TOK + W - 1; ++j) x[i][j] = mine && t0 + j >= W - 1 ? to_f32(p[(size_t)(t0 + j - (W - 1)) * ldp + c]) : 0.f;
            if constexpr (W == 4) {
                const float4 t = mine ? *reinterpret_cast<const float4*>(conv + (size_t)c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
                w[i][0] = t.x; w[i][1] = t.y; w[i][2] = t.z; w[i][3] = t.w;
            } else {
#pragma unroll
                for (int j = 0; j < W; ++j) w[i][j] = mine ? conv[(size_t)c * W + j] : 0.f;
            }
        }
        const int seg0 = token_seg[t0], pos = positions[t0];
        if (token_seg[t1 - 1] == seg0) {
        const int r = t0 - seg_q_start[seg0];
        if (r < W - 1) {
            const float* ring = state + (long long)seg_slot[seg0] * state_stride + ring_off;
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j < W - 1; ++j)
                    if (W - 1 - j > r) x[i][j] = lane + 32 * i < n ? input(c0 + lane + 32 * i, W - 1 - j, t0, r, pos, ring) : 0.f;
        }
        float y[TOK][NI], ss[TOK];                              // all tokens side by side: their sums over the warp do not wait for one another
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
            ss[k] = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                float a = 0.f;
#pragma unroll
                for (int j = 0; j < W; ++j) a = fmaf(w[i][j], x[i][k + j], a);
                y[k][i] = lane + 32 * i < n ? conv_silu<T>(a) : 0.f;
                ss[k] = fmaf(y[k][i], y[k][i], ss[k]);
            }
        }
        if (head) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int k = 0; k < TOK; ++k) ss[k] += __shfl_xor_sync(0xffffffffu, ss[k], o);
        }
#pragma unroll
        for (int k = 0; k < TOK; ++k) {
            const float s = head ? (unit < KV ? q_scale : 1.f) / sqrtf(ss[k] + unit_eps) : 1.f;
            float* o = out + (size_t)(t0 + k) * ldo + c0;
#pragma unroll
            for (int i = 0; i < NI; ++i)
                if (lane + 32 * i < n) o[lane + 32 * i] = y[k][i] * s;
        }
        return;
        }
    }
    for (int t = t0; t < t1; ++t) {
        const int seg = token_seg[t], r = t - seg_q_start[seg], pos = positions[t];
        const float* ring = state + (long long)seg_slot[seg] * state_stride + ring_off;
        float y[NI];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = c0 + lane + 32 * i;
            y[i] = 0.f;
            if (lane + 32 * i < n)
                for (int j = 0; j < taps; ++j) y[i] = fmaf(conv[(size_t)c * taps + j], input(c, taps - 1 - j, t, r, pos, ring), y[i]);
        }
        finish(y, t);
    }
}

// the inputs of the entry's last min(n, taps) positions -> their ring rows; grid (entries, channel groups)
template <typename T>
__global__ void delta_ring_kernel(const T* __restrict__ p, int ldp, float* __restrict__ state, long long state_stride, long long ring_off,
                                  const int* __restrict__ positions, const int* __restrict__ seg_q_start, const int* __restrict__ seg_slot, int C, int taps) {
    const int seg = blockIdx.x, q1 = seg_q_start[seg + 1], n = q1 - seg_q_start[seg], c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    float* ring = state + (long long)seg_slot[seg] * state_stride + ring_off;
    for (int t = q1 - min(n, taps); t < q1; ++t) ring[(size_t)(positions[t] % taps) * C + c] = to_f32(p[(size_t)t * ldp + c]);
}

// ------------------------------------------------------------------ decode steps: everything in one pass over the state
// grid (entries, H).  The head's state (D V contiguous floats) comes into shared memory as one bulk copy, under which the convolution, the
// norms and the gates are made.  The copy, and the filter's sums over earlier inputs, start before the kernel ahead (which makes p) is
// done: the state and the ring were last written in the step before.  Thread (rg, cv) then owns the columns 4 cv .. of the rows rg + RG i, cv < V / 4, RG = 256 / (V / 4), in
// both passes over it (S^T k; update, read-out and the way back to memory).
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) delta_step_kernel(const T* __restrict__ p, int ldp, const float* __restrict__ conv, int taps_,
                                                         const float* __restrict__ rate, const float* __restrict__ dt_bias, float* __restrict__ state,
                                                         long long state_stride, long long ring_off, const float* __restrict__ norm, T* __restrict__ rows,
                                                         const int* __restrict__ positions, const int* __restrict__ seg_q_start,
                                                         const int* __restrict__ seg_slot, int H, int KV, int D, int V, float unit_eps, float q_scale, float eps,
                                                         int* __restrict__ error) {
    extern __shared__ __align__(128) float sm[];
    __shared__ __align__(8) uint64_t arrived;
    __shared__ float2 squares[8];
    __shared__ float outs[8], gates[2];
    const int taps = TAPS > 0 ? TAPS : taps_;
    float* Ss = sm;                                            // [D, V]
    float* qs = Ss + D * V;                                    // [D]
    float* ks = qs + D;                                        // [D]
    float* vs = ks + D;                                        // [V]: the values, then u
    float* red = qs + ((2 * D + V + 3) & ~3);                  // [RG, V]
    const int seg = blockIdx.x, h = blockIdx.y, rep = H / KV, kvh = h / rep, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* slot = state + (long long)seg_slot[seg] * state_stride;
    float* S = slot + (long long)h * D * V;
    const uint32_t bar = smem_u32(&arrived);
    pdl_trigger();
    if (tid == 0) {
        const uint32_t bytes = (uint32_t)(D * V) * 4;
        mbar_init(bar, 1);
        mbar_init_fence();
        mbar_expect_tx(bar, bytes);
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
                     :: "r"(smem_u32(Ss)), "l"(S), "r"(bytes), "r"(bar) : "memory");
    }
    const int CV = V >> 2, RG = 256 / CV, cv = tid % CV, rg = tid / CV;
    const int t = seg_q_start[seg], pos = positions[t];
    float* ring = slot + ring_off;
    const T* row = p + (size_t)t * ldp;
    const int C = 2 * KV * D + H * V;
    const int channels = 2 * D + V;                            // this head's q, k and v channels
    auto channel = [&](int i) { return i < D ? kvh * D + i : i < 2 * D ? KV * D + kvh * D + i - D : 2 * KV * D + h * V + i - 2 * D; };
    auto past = [&](int c) {                                   // the filter's sum over the inputs before this token
        float acc = 0.f;
        auto tap = [&](int j) {
            const int back = taps - 1 - j;
            if (back <= pos) acc = fmaf(conv[(size_t)c * taps + j], ring[(size_t)((pos - back) % taps) * C + c], acc);
        };
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) tap(j);
        } else {
            for (int j = 0; j + 1 < taps; ++j) tap(j);
        }
        return acc;
    };
    float early[2], last_tap[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int i = tid + 256 * k, c = i < channels ? channel(i) : 0;
        early[k] = i < channels ? past(c) : 0.f;
        last_tap[k] = conv[(size_t)c * taps + taps - 1];
    }
    pdl_wait();
    if (tid == 255) {
        gates[0] = 1.f / (1.f + expf(-to_f32(row[C + H * V + h])));
        gates[1] = decay_of(log_decay(to_f32(row[C + H * V + H + h]), dt_bias[h], rate[h]));
    }
    float sq = 0.f, sk = 0.f;
    auto finish = [&](int i, int c, float acc, float w) {
        const float own = to_f32(row[c]);
        const float y = silu(fmaf(w, own, acc));
        qs[i] = y;
        if (i < D) sq = fmaf(y, y, sq); else if (i < 2 * D) sk = fmaf(y, y, sk);
        if (taps > 1 && (i >= 2 * D || h % rep == 0)) ring[(size_t)(pos % taps) * C + c] = own;      // one writer a channel
    };
#pragma unroll
    for (int k = 0; k < 2; ++k)
        if (tid + 256 * k < channels) finish(tid + 256 * k, channel(tid + 256 * k), early[k], last_tap[k]);
    for (int i = tid + 512; i < channels; i += 256) finish(i, channel(i), past(channel(i)), conv[(size_t)channel(i) * taps + taps - 1]);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) squares[warp] = make_float2(sq, sk);
    __syncthreads();                                           // also: the barrier's word is ready for every thread
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { sq += squares[w].x; sk += squares[w].y; }
    const float beta = gates[0], f = gates[1], rq = q_scale / sqrtf(sq + unit_eps), rk = 1.f / sqrtf(sk + unit_eps);
    const bool here = mbar_wait(bar, 0);
    if (!here) atomicExch(error, 72);
    if (__syncthreads_or(!here)) return;                       // the state did not arrive: nothing of it is changed
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (rg < RG) {
#pragma unroll 8
        for (int r = rg; r < D; r += RG) {
            const float4 s = *reinterpret_cast<const float4*>(Ss + r * V + 4 * cv);
            const float kr = ks[r];
            a.x = fmaf(s.x, kr, a.x); a.y = fmaf(s.y, kr, a.y); a.z = fmaf(s.z, kr, a.z); a.w = fmaf(s.w, kr, a.w);
        }
        *reinterpret_cast<float4*>(red + rg * V + 4 * cv) = a;
    }
    __syncthreads();
    for (int c = tid; c < V; c += 256) {
        float dot = 0.f;
#pragma unroll 8
        for (int g = 0; g < RG; ++g) dot += red[g * V + c];
        vs[c] = beta * (vs[c] - f * (rk * dot));
    }
    __syncthreads();
    if (rg < RG) {
        const float4 u = *reinterpret_cast<const float4*>(vs + 4 * cv);
        const float4 ku = make_float4(rk * u.x, rk * u.y, rk * u.z, rk * u.w);
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int r = rg; r < D; r += RG) {
            float4 s = *reinterpret_cast<const float4*>(Ss + r * V + 4 * cv);
            const float kr = ks[r], qr = qs[r];
            s.x = fmaf(kr, ku.x, f * s.x); s.y = fmaf(kr, ku.y, f * s.y); s.z = fmaf(kr, ku.z, f * s.z); s.w = fmaf(kr, ku.w, f * s.w);
            o.x = fmaf(s.x, qr, o.x); o.y = fmaf(s.y, qr, o.y); o.z = fmaf(s.z, qr, o.z); o.w = fmaf(s.w, qr, o.w);
            *reinterpret_cast<float4*>(S + (size_t)r * V + 4 * cv) = s;
        }
        *reinterpret_cast<float4*>(red + rg * V + 4 * cv) = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < V; c += 256) {
        float o = 0.f;
#pragma unroll 8
        for (int g = 0; g < RG; ++g) o += red[g * V + c];
        o *= rq;
        vs[c] = o;                                             // read again below by the same thread
        ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) outs[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += outs[w];
    const float r = rsqrtf(ss / V + eps);
    for (int c = tid; c < V; c += 256)
        rows[(size_t)t * H * V + (size_t)h * V + c] = from_f32<T>(vs[c] * r * norm[c] * silu(to_f32(row[C + h * V + c])));
}

template <typename T>
int launch_ready(const T* p, int ldp, const float* conv, const float* rate, const float* dt_bias, const float* state, long long state_stride,
                 long long ring_off, float* out, int ldo, const int* positions, const int* token_seg, const int* seg_q_start, const int* seg_slot,
                 int T_, int H, int KV, int D, int V, int taps, float unit_eps, cudaStream_t stream) {
    const int NI = D <= 32 ? 1 : D <= 64 ? 2 : D <= 128 ? 4 : 8;
    const int units = 2 * KV + (H * V + 32 * NI - 1) / (32 * NI) + 1;
    const int TOK = T_ >= 512 ? 8 : T_ >= 128 ? 4 : 1;
    dim3 grid((T_ + TOK - 1) / TOK, (units + 3) / 4);
    if (grid.y > 65535) return -2;
    const float q_scale = 1.f / sqrtf((float)D);
#define GO(TAPS, N, TK) delta_ready_kernel<T, TAPS, N, TK><<<grid, 128, 0, stream>>>(p, ldp, conv, rate, dt_bias, state, state_stride, ring_off, out, ldo, \
                            positions, token_seg, seg_q_start, seg_slot, T_, H, KV, D, V, taps, unit_eps, q_scale)
#define TOKENS(TAPS, N) do { if (TOK == 8) GO(TAPS, N, 8); else if (TOK == 4) GO(TAPS, N, 4); else GO(TAPS, N, 1); } while (0)
#define CHANNELS(TAPS) do { if (NI == 1) TOKENS(TAPS, 1); else if (NI == 2) TOKENS(TAPS, 2); else if (NI == 4) TOKENS(TAPS, 4); else TOKENS(TAPS, 8); } while (0)
    if (taps == 4) CHANNELS(4); else if (taps == 3) CHANNELS(3); else if (taps == 2) CHANNELS(2); else CHANNELS(0);
#undef CHANNELS
#undef TOKENS
#undef GO
    return (int)cudaGetLastError();
}

}  // namespace

// out [T, ldo] float32 = q | k | v | beta [H] | f [H] | log f [H] (ldo may pad)
MI_EXPORT int mi_gated_delta_ready(const void* p, int ldp, const float* conv, const float* rate, const float* dt_bias, const float* state,
                                   long long state_stride, long long ring_off, float* out, int ldo, const int* positions, const int* token_seg,
                                   const int* seg_q_start, const int* seg_slot, int T_, int H, int KV, int D, int V, int taps, float unit_eps, int dtype,
                                   cudaStream_t stream) {
    if (T_ == 0) return 0;
    if (H % KV || D > 256 || taps < 1) return -2;
    if (dtype == MI_BF16)
        return launch_ready<__nv_bfloat16>((const __nv_bfloat16*)p, ldp, conv, rate, dt_bias, state, state_stride, ring_off, out, ldo, positions, token_seg,
                                           seg_q_start, seg_slot, T_, H, KV, D, V, taps, unit_eps, stream);
    return launch_ready<float>((const float*)p, ldp, conv, rate, dt_bias, state, state_stride, ring_off, out, ldo, positions, token_seg, seg_q_start, seg_slot,
                               T_, H, KV, D, V, taps, unit_eps, stream);
}

MI_EXPORT int mi_gated_delta_ring(const void* p, int ldp, float* state, long long state_stride, long long ring_off, const int* positions,
                                  const int* seg_q_start, const int* seg_slot, int num_segs, int C, int taps, int dtype, cudaStream_t stream) {
    if (num_segs == 0 || taps <= 1) return 0;
    dim3 grid(num_segs, (C + 255) / 256);
    if (grid.y > 65535) return -2;
    if (dtype == MI_BF16)
        delta_ring_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)p, ldp, state, state_stride, ring_off, positions, seg_q_start, seg_slot, C, taps);
    else
        delta_ring_kernel<float><<<grid, 256, 0, stream>>>((const float*)p, ldp, state, state_stride, ring_off, positions, seg_q_start, seg_slot, C, taps);
    return (int)cudaGetLastError();
}

// Every entry brings one token.  rows [entries, H V] in the type of p.  -2: sizes that this form does not take (V or D not a multiple of
// four, or a head's state larger than shared memory); the caller then runs the prompt form.  error: receives 72 when a head's state did
// not arrive in time (the entry is then left as it is).
MI_EXPORT int mi_gated_delta_step(const void* p, int ldp, const float* conv, int taps, const float* rate, const float* dt_bias, float* state,
                                  long long state_stride, long long ring_off, const float* norm, void* rows, const int* positions, const int* seg_q_start,
                                  const int* seg_slot, int num_segs, int H, int KV, int D, int V, float unit_eps, float eps, int* error, int dtype,
                                  cudaStream_t stream) {
    if (num_segs == 0) return 0;
    if (H % KV || H > 65535 || V % 4 || D % 2 || V > 1024 || state_stride % 4 || (uintptr_t)state % 16) return -2;
    const int RG = 256 / (V / 4);
    const size_t smem = ((size_t)D * V + ((2 * D + V + 3) & ~3) + RG * V) * sizeof(float);
    if (smem > 220 * 1024) return -2;
    const float q_scale = 1.f / sqrtf((float)D);
    dim3 grid(num_segs, H);
#define GO(T, TAPS) do { \
        static bool configured = false; \
        if (!configured) { \
            const cudaError_t e = cudaFuncSetAttribute(delta_step_kernel<T, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024); \
            if (e != cudaSuccess) return (int)e; \
            configured = true; \
        } \
        return (int)launch_pdl(delta_step_kernel<T, TAPS>, grid, dim3(256), smem, stream, (const T*)p, ldp, conv, taps, rate, dt_bias, state, state_stride, ring_off, norm, \
                               (T*)rows, positions, seg_q_start, seg_slot, H, KV, D, V, unit_eps, q_scale, eps, error); } while (0)
    if (dtype == MI_BF16) { if (taps == 4) GO(__nv_bfloat16, 4); GO(__nv_bfloat16, 0); }
    if (taps == 4) GO(float, 4);
    GO(float, 0);
#undef GO
}
