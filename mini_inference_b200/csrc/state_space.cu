// A state-space recurrence with one decay per head and token (Mamba-2), over a float32 state S [heads, N, V] in a request's slot:
//     S <- e^(A dt) S + dt B x^T,   y = S^T C + D x      (A < 0 per head; head h uses the B and C of group floor(h / (heads / groups)))
// p [T, ldp] = z | x | B | C | dt as projected (I, I, G N, G N, heads columns, I = heads V); x, B and C pass a short convolution with a
// bias and silu, dt a bias and softplus.  Decays, dt, sums and the state are float32.
//
// Prompt portions (bfloat16): ssd_chunk_kernel.  Unrolled over a chunk of 64 tokens with c_t = sum_{r <= t} A dt_r the recurrence is
//     y_t = e^(c_t) C_t^T S_0 + sum_{s <= t} e^(c_t - c_s) dt_s (C_t . B_s) x_s
//     S'  = e^(c_63) S_0 + sum_s B_s (e^(c_63 - c_s) dt_s x_s)^T
// which is three products of tensor-core shape.  A block owns one entry, one head and 32 columns of V; it walks the entry's chunks in
// order, the state's accumulators staying in registers from the first chunk to the last.  B, C and x are bfloat16 as the convolution left
// them; the float32 operands (the decayed scores, the decayed x, the state) enter as TWO bfloat16 numbers each, their rounding and what
// it leaves, so that they keep 16 mantissa bits; all sums are float32.  mma.sync: the operands of every product but the first are made in
// registers, 16 rows a warp, and the sizes are a quarter of a tcgen05 tile.
//
// Decode steps: ssd_step_kernel, one block per (entry, head): convolution, dt, state update and read-out in one pass over the state.
// gated_part_norm_kernel finishes both: (y + D x) * silu(z), divided by its root mean square in equal parts, times a weight; in a decode
// step it also moves the slot's convolution inputs up (the step kernel's blocks share them, so none of them may).
#include "common.cuh"
#include <math.h>

using namespace mi;

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;                              // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" :: "r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ float fast_exp2(float x) {              // ex2.approx: 2 ulp
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float rest(float x) { return x - __bfloat162float(__float2bfloat16_rn(x)); }      // what the rounding leaves

constexpr int Q = 64, VB = 32, CH_WARPS = 16, CH_THREADS = 32 * CH_WARPS;

// byte offset of the 16-byte piece `ch` of row `row`: rows of N entries (a multiple of 128 bytes), and rows of 32 entries (64 bytes)
template <int N> __device__ __forceinline__ uint32_t at_n(int row, int ch) { return (uint32_t)(row * N * 2 + ((ch ^ (row & 7)) << 4)); }
__device__ __forceinline__ uint32_t at_v(int row, int ch) { return (uint32_t)(row * 64 + ((ch ^ ((row >> 1) & 3)) << 4)); }

template <int N>
struct ChunkSmem {
    static constexpr int BC = Q * N * 2, X = Q * VB * 2, STAGE = 2 * BC + X, S = N * VB * 2;
    static constexpr int XW = 2 * STAGE, SH = XW + 2 * X, YP = SH + 2 * S, CUM = YP + 4 * Q * (VB + 2) * 4, TOTAL = CUM + 4 * Q * 4;
};

// grid (entries, heads, V / 32)
template <int N>
__global__ void __launch_bounds__(CH_THREADS, 1) ssd_chunk_kernel(const __nv_bfloat16* __restrict__ xbc, int ldx, const __nv_bfloat16* __restrict__ dt_in, int ld_dt,
                                                                  const float* __restrict__ dt_bias, const float* __restrict__ A, float* __restrict__ state,
                                                                  long long state_stride, float* __restrict__ out, const int* __restrict__ seg_q_start,
                                                                  const int* __restrict__ seg_slot, int H, int V, int G) {
    using L = ChunkSmem<N>;
    extern __shared__ __align__(1024) unsigned char smem[];         // rows of up to 256 bytes start on 256: pieces are chosen by XOR below
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
    float* ypart = reinterpret_cast<float*>(smem + L::YP);         // [4][Q][VB + 2]
    float* dts = reinterpret_cast<float*>(smem + L::CUM);          // [2][Q]
    float* cums = dts + 2 * Q;                                     // [2][Q], base 2
    constexpr int CHN = N / 8, KN = N / 16;                        // 16-byte pieces of a row, k-steps over the state rows
    constexpr int NTS = N == 128 ? 2 : 1;                          // the state's tiles of 8 columns a warp owns
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3, mi_ = lane >> 3;
    const int seg = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VB, grp = h / (H / G), I = H * V;
    const int qs = seg_q_start[seg], n = seg_q_start[seg + 1] - qs;
    const __nv_bfloat16* xg = xbc + (size_t)qs * ldx + (size_t)h * V + v0;
    const __nv_bfloat16* bg = xbc + (size_t)qs * ldx + I + (size_t)grp * N;
    const __nv_bfloat16* cg = bg + (size_t)G * N;
    const float rate = A[h] * LOG2E, bias = dt_bias[h];
    const int chunks = (n + Q - 1) / Q;

    auto load = [&](int chunk) {
        const uint32_t st = base + (chunk & 1) * L::STAGE;
        const int r0 = chunk * Q;
        for (int id = tid; id < Q * CHN; id += CH_THREADS) {
            const int row = id / CHN, ch = id % CHN;
            const bool ok = r0 + row < n;
            const size_t off = ok ? (size_t)(r0 + row) * ldx + ch * 8 : 0;
            cp16(st + at_n<N>(row, ch), bg + off, ok);
            cp16(st + L::BC + at_n<N>(row, ch), cg + off, ok);
        }
        if (tid < Q * 4) {                                         // the pieces of x
            const int row = tid >> 2, ch = tid & 3;
            const bool ok = r0 + row < n;
            cp16(st + 2 * L::BC + at_v(row, ch), xg + (ok ? (size_t)(r0 + row) * ldx + ch * 8 : 0), ok);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    // one warp, two tokens a lane; the raw steps are fetched a chunk before they are summed
    float raw0 = 0.f, raw1 = 0.f;
    auto fetch_dt = [&](int chunk) {
        const int t = chunk * Q + 2 * lane;
        raw0 = t < n ? __bfloat162float(dt_in[(size_t)(qs + t) * ld_dt + h]) : 0.f;
        raw1 = t + 1 < n ? __bfloat162float(dt_in[(size_t)(qs + t + 1) * ld_dt + h]) : 0.f;
    };
    auto sum_dt = [&](int chunk) {
        const int t = chunk * Q + 2 * lane;
        const float d0 = t < n ? softplus(raw0 + bias) : 0.f, d1 = t + 1 < n ? softplus(raw1 + bias) : 0.f;
        const float a0 = rate * d0, a1 = rate * d1;
        float incl = a0 + a1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        const int b = (chunk & 1) * Q + 2 * lane;
        dts[b] = d0; dts[b + 1] = d1;
        cums[b] = incl - a1; cums[b + 1] = incl;
    };

    // this warp's piece of the state: rows sn .. sn + 15, columns 8 (st0 + nt)
    const int sn = (warp & (N / 16 - 1)) * 16, st0 = warp / (N / 16) * NTS;
    float* S = state + (long long)seg_slot[seg] * state_stride + (long long)h * N * V + v0;
    float s[NTS][4];
    auto spread_state = [&]() {                                    // the state as two bfloat16 numbers each, for the next chunk's read-out
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = sn + g + 8 * half;
                const uint32_t off = at_v(row, st0 + nt) + 4 * c;
                *reinterpret_cast<uint32_t*>(smem + L::SH + off) = pack2(s[nt][2 * half], s[nt][2 * half + 1]);
                *reinterpret_cast<uint32_t*>(smem + L::SH + L::S + off) = pack2(rest(s[nt][2 * half]), rest(s[nt][2 * half + 1]));
            }
    };
    // one warp sums the steps a chunk ahead: one whose tokens have none of its quarter before them, so that it has the time
    const bool steps_warp = warp == 13;
    load(0);
    if (steps_warp) fetch_dt(0);
#pragma unroll
    for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const float2 t = *reinterpret_cast<const float2*>(S + (size_t)(sn + g + 8 * half) * V + (st0 + nt) * 8 + 2 * c);
            s[nt][2 * half] = t.x; s[nt][2 * half + 1] = t.y;
        }
    spread_state();
    if (steps_warp) { sum_dt(0); fetch_dt(1); }

    // the warp's 16 tokens, its quarter of the state rows and of the chunk's tokens (token tiles turned from quarter to quarter: late tiles have
    // more tokens before them, and a scheduler's four warps should not all own late ones)
    const int qd = warp >> 2, m0 = ((warp + qd) & 3) * 16;
    // this lane's ldmatrix rows: of C (its tokens), of B (its quarter), of a 32-column tile, of B transposed.  The 16-byte piece is XOR-ed with the
    // row, and a k-step moves it by two: one XOR with 32 times the step
    const uint32_t o_c = at_n<N>(m0 + (lane & 7) + (mi_ & 1) * 8, mi_ >> 1), o_b = at_n<N>(16 * qd + (mi_ >> 1) * 8 + (lane & 7), mi_ & 1);
    const uint32_t o_v = at_v((mi_ & 1) * 8 + (lane & 7), mi_ >> 1), o_t = at_n<N>((lane & 7) + (mi_ >> 1) * 8, (sn >> 3) + (mi_ & 1));
    for (int ck = 0; ck < chunks; ++ck) {
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                                           // the chunk, its decays and the spread state are there; the other stage is free
        if (ck + 1 < chunks) load(ck + 1);
        const uint32_t bt = base + (ck & 1) * L::STAGE, ct = bt + L::BC, xt = bt + 2 * L::BC;
        const float* dt = dts + (ck & 1) * Q;
        const float* cum = cums + (ck & 1) * Q;
        const float end = cum[Q - 1];
        {   // the decayed x of the state's update
            const int row = tid >> 3, part = tid & 7;              // four entries a thread
            const uint32_t off = at_v(row, part >> 1) + (part & 1) * 8;
            const float w = fast_exp2(end - cum[row]) * dt[row];
            const uint2 raw = *reinterpret_cast<const uint2*>(smem + (xt - base) + off);
            const float x0 = w * __uint_as_float(raw.x << 16), x1 = w * __uint_as_float(raw.x & 0xffff0000u);
            const float x2 = w * __uint_as_float(raw.y << 16), x3 = w * __uint_as_float(raw.y & 0xffff0000u);
            *reinterpret_cast<uint2*>(smem + L::XW + off) = make_uint2(pack2(x0, x1), pack2(x2, x3));
            *reinterpret_cast<uint2*>(smem + L::XW + L::X + off) = make_uint2(pack2(rest(x0), rest(x1)), pack2(rest(x2), rest(x3)));
        }
        // ---- what the state of before the chunk gives to the outputs: this warp's quarter of its rows
        float y[4][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) y[nt][0] = y[nt][1] = y[nt][2] = y[nt][3] = 0.f;
#pragma unroll
        for (int k = 0; k < KN / 4; ++k) {
            const int ks = qd * (KN / 4) + k;
            uint32_t a[4], b[4];
            ldsm4(a, (ct + o_c) ^ (32 * ks));
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
                for (int dp = 0; dp < 2; ++dp) {
                    ldsm4t(b, (base + L::SH + part * L::S + ks * 16 * 64 + o_v) ^ (32 * dp));
                    mma16816(y[2 * dp], a, b[0], b[1]);
                    mma16816(y[2 * dp + 1], a, b[2], b[3]);
                }
        }
        const float ct0 = cum[m0 + g], ct1 = cum[m0 + g + 8];
        {
            const float e0 = fast_exp2(ct0), e1 = fast_exp2(ct1);
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) { y[nt][0] *= e0; y[nt][1] *= e0; y[nt][2] *= e1; y[nt][3] *= e1; }
        }
        // ---- the chunk's own tokens: this warp's quarter of them, unless they all come after its rows
        if (16 * qd <= m0) {
            float sc[2][4];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KN; ++ks) {
                uint32_t a[4], b[4];
                ldsm4(a, (ct + o_c) ^ (32 * ks));
                ldsm4(b, (bt + o_b) ^ (32 * ks));
                mma16816(sc[0], a, b[0], b[1]);
                mma16816(sc[1], a, b[2], b[3]);
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = 16 * qd + nt * 8 + 2 * c + e;
                    const float cj = cum[j], dj = dt[j];
                    sc[nt][e] = j <= m0 + g ? sc[nt][e] * fast_exp2(ct0 - cj) * dj : 0.f;
                    sc[nt][2 + e] = j <= m0 + g + 8 ? sc[nt][2 + e] * fast_exp2(ct1 - cj) * dj : 0.f;
                }
            uint32_t pa[4], pr[4], b[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float lo = sc[q >> 1][2 * (q & 1)], hi = sc[q >> 1][2 * (q & 1) + 1];
                pa[q] = pack2(lo, hi);
                pr[q] = pack2(rest(lo), rest(hi));
            }
#pragma unroll
            for (int dp = 0; dp < 2; ++dp) {
                ldsm4t(b, (xt + qd * 16 * 64 + o_v) ^ (32 * dp));
                mma16816(y[2 * dp], pa, b[0], b[1]);
                mma16816(y[2 * dp + 1], pa, b[2], b[3]);
                mma16816(y[2 * dp], pr, b[0], b[1]);
                mma16816(y[2 * dp + 1], pr, b[2], b[3]);
            }
        }
        if (steps_warp && ck + 1 < chunks) { sum_dt(ck + 1); fetch_dt(ck + 2); }
        {
            float* yp = ypart + (qd * Q + m0 + g) * (VB + 2) + 2 * c;
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                *reinterpret_cast<float2*>(yp + nt * 8) = make_float2(y[nt][0], y[nt][1]);
                *reinterpret_cast<float2*>(yp + 8 * (VB + 2) + nt * 8) = make_float2(y[nt][2], y[nt][3]);
            }
        }
        __syncthreads();                                           // partial outputs and the decayed x are there; nobody reads the spread state any more
#pragma unroll
        for (int i = tid; i < Q * VB / 2; i += CH_THREADS) {       // the four quarters, added in order; a row's 32 columns leave together
            const int row = i / (VB / 2), col = i % (VB / 2) * 2, t = ck * Q + row;
            float2 sum = make_float2(0.f, 0.f);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 v = *reinterpret_cast<const float2*>(ypart + (q * Q + row) * (VB + 2) + col);
                sum.x += v.x; sum.y += v.y;
            }
            if (t < n) *reinterpret_cast<float2*>(out + (size_t)(qs + t) * I + (size_t)h * V + v0 + col) = sum;
        }
        // ---- the state after the chunk
        const float keep = fast_exp2(end);
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt) { s[nt][0] *= keep; s[nt][1] *= keep; s[nt][2] *= keep; s[nt][3] *= keep; }
#pragma unroll
        for (int kt = 0; kt < Q / 16; ++kt) {
            uint32_t a[4], b[4];
            ldsm4t(a, bt + kt * 16 * N * 2 + o_t);
            if constexpr (NTS == 2) {
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    ldsm4t(b, (base + L::XW + part * L::X + kt * 16 * 64 + o_v) ^ (16 * st0));
                    mma16816(s[0], a, b[0], b[1]);
                    mma16816(s[1], a, b[2], b[3]);
                }
            } else {                                               // one tile of columns: its two parts in one load
                ldsm4t(b, base + L::XW + (mi_ >> 1) * L::X + at_v(kt * 16 + (mi_ & 1) * 8 + (lane & 7), st0));
                mma16816(s[0], a, b[0], b[1]);
                mma16816(s[0], a, b[2], b[3]);
            }
        }
        if (ck + 1 < chunks) {
            spread_state();
        }
    }
#pragma unroll
    for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half)
            *reinterpret_cast<float2*>(S + (size_t)(sn + g + 8 * half) * V + (st0 + nt) * 8 + 2 * c) = make_float2(s[nt][2 * half], s[nt][2 * half + 1]);
}

// ------------------------------------------------------------------ decode step
// grid (entries, heads), every entry brings ONE token.  VEC neighbouring columns a thread; the threads of a block are cols x rows of them.
// TAPS: the convolution's taps when known (0: any number), so that a channel's inputs are fetched together.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(256) ssd_step_kernel(const T* __restrict__ p, int ldp, const float* __restrict__ conv, const float* __restrict__ conv_b, int taps,
                                                       const float* __restrict__ dt_bias, const float* __restrict__ A, const float* __restrict__ Dv,
                                                       float* __restrict__ state, long long state_stride, float* __restrict__ out,
                                                       const int* __restrict__ seg_q_start, const int* __restrict__ seg_slot, int H, int V, int N, int G) {
    extern __shared__ float sm[];
    const int seg = blockIdx.x, h = blockIdx.y, grp = h / (H / G), I = H * V, C = I + 2 * G * N;
    const size_t t = seg_q_start[seg];
    float* slot = state + (long long)seg_slot[seg] * state_stride;
    const float* hist = slot + (long long)H * N * V;               // [taps - 1, C]
    const T* row = p + t * ldp + I;
    float* xs = sm;                                                // [V] x | [N] B dt | [N] C
    float* bs = xs + V;
    float* cs = bs + N;
    float* red = cs + N;                                           // [rows, V]
    const int cols = V / VEC, rows = max(1, 256 / cols);
    const int col = threadIdx.x % cols, r0 = threadIdx.x / cols;
    float* S = slot + (long long)h * N * V;
    constexpr int U = VEC == 4 ? 8 : 4;                            // state pieces in flight a thread
    float s[U][VEC];
    auto fetch = [&](int n0, int cc) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int nn = n0 + u * rows;
            if (nn < N) {
                if constexpr (VEC == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(S + (size_t)nn * V + cc * 4);
                    s[u][0] = f.x; s[u][1] = f.y; s[u][2] = f.z; s[u][3] = f.w;
                } else {
                    s[u][0] = S[(size_t)nn * V + cc];
                }
            }
        }
    };
    if (r0 < rows) fetch(r0, col);                                 // the first pieces travel while the convolution is made
    const float dt = softplus(to_f32(p[t * ldp + I + C + h]) + dt_bias[h]);
    __shared__ float decay_s;
    // a decay near one acts on a state hundreds of times in a row: its last bit is worth an exponential in double, rounded once
    if (threadIdx.x == 255) decay_s = (float)exp((double)A[h] * (double)dt);
    for (int i = threadIdx.x; i < V + 2 * N; i += 256) {
        const int c = i < V ? h * V + i : i < V + N ? I + grp * N + (i - V) : I + G * N + grp * N + (i - V - N);
        const int nt = TAPS ? TAPS : taps;
        float a = conv_b[c];
        const float own = to_f32(row[c]);
#pragma unroll
        for (int j = 0; j + 1 < nt; ++j) a = fmaf(conv[(size_t)c * nt + j], hist[(size_t)j * C + c], a);
        a = fmaf(conv[(size_t)c * nt + nt - 1], own, a);
        a = round_to<T>(silu(a));
        sm[i] = i >= V && i < V + N ? a * dt : a;
    }
    __syncthreads();
    const float decay = decay_s;
    for (int cc = col; cc < cols; cc += 256) {
        float acc[VEC], x[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { acc[e] = 0.f; x[e] = xs[cc * VEC + e]; }
        if (r0 < rows) {
            for (int n0 = r0; n0 < N; n0 += rows * U) {
                if (n0 != r0 || cc != col) fetch(n0, cc);
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const int nn = n0 + u * rows;
                    if (nn < N) {
                        const float b = bs[nn], cv = cs[nn];
#pragma unroll
                        for (int e = 0; e < VEC; ++e) {
                            s[u][e] = fmaf(decay, s[u][e], b * x[e]);
                            acc[e] = fmaf(s[u][e], cv, acc[e]);
                        }
                        if constexpr (VEC == 4) *reinterpret_cast<float4*>(S + (size_t)nn * V + cc * 4) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
                        else S[(size_t)nn * V + cc] = s[u][0];
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) red[(size_t)r0 * V + cc * VEC + e] = acc[e];
        }
    }
    __syncthreads();
    for (int v = threadIdx.x; v < V; v += 256) {
        float y = Dv[h] * xs[v];
        for (int r = 0; r < rows; ++r) y += red[(size_t)r * V + v];
        out[t * I + (size_t)h * V + v] = y;
    }
}

// ------------------------------------------------------------------ (y + D x) * silu(z), norm in parts, weight
struct Tail { float* state; long long stride, off; const int* seg_slot; int C, taps, parts; };      // state null: nothing to move

template <typename T>
__device__ __forceinline__ void shift_inputs(const T* __restrict__ zrow, int I, const Tail& k) {
    // a step of single tokens: entry == token; the convolution's inputs x | B | C stand behind z in the token's row.  A block behind the
    // norm's parts takes blockDim.x channels.
    float* hist = k.state + (long long)k.seg_slot[blockIdx.x] * k.stride + k.off;
    const int c = ((int)blockIdx.y - k.parts) * blockDim.x + threadIdx.x;
    if (c >= k.C) return;
    const float own = to_f32(zrow[I + c]);
    for (int j = 0; j + 2 < k.taps; ++j) hist[(size_t)j * k.C + c] = hist[(size_t)(j + 1) * k.C + c];
    hist[(size_t)(k.taps - 2) * k.C + c] = own;
}

// grid (tokens, parts (+ blocks that move the inputs)).  VPT = 0: any sizes, the values made twice; else 8 VPT neighbouring values a thread, kept in registers.
template <typename T, int VPT>
__global__ void __launch_bounds__(256) gated_part_norm_kernel(const float* __restrict__ y, const T* __restrict__ x, int ldx, const float* __restrict__ Dv, int V,
                                                              const T* __restrict__ z, int ldz, const float* __restrict__ w, T* __restrict__ out, int I, int gs,
                                                              float eps, const Tail tail) {
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    const T* zr = z + t * ldz;
    if ((int)blockIdx.y >= tail.parts) { shift_inputs(zr, I, tail); return; }
    const int c0 = blockIdx.y * gs;
    const float* yr = y + t * I + c0;
    const T* xr = x ? x + t * ldx + c0 : nullptr;
    if constexpr (VPT == 0) {
        auto value = [&](int i) { return (yr[i] + (xr ? Dv[(c0 + i) / V] * to_f32(xr[i]) : 0.f)) * silu(to_f32(zr[c0 + i])); };
        float ss = 0.f;
        for (int i = threadIdx.x; i < gs; i += 256) { const float v = value(i); ss += v * v; }
        const float s = rsqrtf(block_sum<256>(ss, scratch) / gs + eps);
        for (int i = threadIdx.x; i < gs; i += 256) out[t * I + c0 + i] = from_f32<T>(value(i) * s * w[c0 + i]);
    } else {
        float v[VPT][8], ss = 0.f;
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int i = (threadIdx.x + 256 * k) * 8;
            if (i < gs) {
                float zf[8], xf[8];
                const float4 a = *reinterpret_cast<const float4*>(yr + i), b = *reinterpret_cast<const float4*>(yr + i + 4);
                v[k][0] = a.x; v[k][1] = a.y; v[k][2] = a.z; v[k][3] = a.w; v[k][4] = b.x; v[k][5] = b.y; v[k][6] = b.z; v[k][7] = b.w;
                load16<T>(zr + c0 + i, zf);
                if (xr) {
                    load16<T>(xr + i, xf);
                    const float d = Dv[(c0 + i) / V];              // V is a multiple of eight: one head
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[k][e] = fmaf(d, xf[e], v[k][e]);
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) { v[k][e] *= silu(zf[e]); ss += v[k][e] * v[k][e]; }
            }
        }
        const float s = rsqrtf(block_sum<256>(ss, scratch) / gs + eps);
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int i = (threadIdx.x + 256 * k) * 8;
            if (i < gs) {
                uint4 o;
                uint32_t* po = reinterpret_cast<uint32_t*>(&o);
                const float4 a = *reinterpret_cast<const float4*>(w + c0 + i), b = *reinterpret_cast<const float4*>(w + c0 + i + 4);
                po[0] = pack2(v[k][0] * s * a.x, v[k][1] * s * a.y); po[1] = pack2(v[k][2] * s * a.z, v[k][3] * s * a.w);
                po[2] = pack2(v[k][4] * s * b.x, v[k][5] * s * b.y); po[3] = pack2(v[k][6] * s * b.z, v[k][7] * s * b.w);
                *reinterpret_cast<uint4*>(out + t * I + c0 + i) = o;
            }
        }
    }
}

}  // namespace

// xbc [T, ldx] bfloat16 = x | B | C behind their convolution and silu; dt_in: the dt columns as projected (rows ld_dt apart); out float32
// [T, H V] = S^T C (no D x yet).  -2: a size this kernel has no form for.
MI_EXPORT int mi_ssd_chunk(const void* xbc, int ldx, const void* dt_in, int ld_dt, const float* dt_bias, const float* A, float* state, long long state_stride,
                           float* out, const int* seg_q_start, const int* seg_slot, int T_, int num_segs, int H, int V, int N, int G, cudaStream_t stream) {
    if (T_ == 0 || num_segs == 0) return 0;
    if ((N != 64 && N != 128) || V % VB || ldx % 8 || (uintptr_t)xbc % 16 || state_stride % 2 || (uintptr_t)state % 8 || (uintptr_t)out % 8 || H > 65535 ||
        H % G) return -2;
    const dim3 grid(num_segs, H, V / VB);
#define GO(NN) do { \
        static bool configured = false; \
        if (!configured) { \
            cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NN>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkSmem<NN>::TOTAL); \
            if (e != cudaSuccess) return (int)e; \
            configured = true; \
        } \
        ssd_chunk_kernel<NN><<<grid, CH_THREADS, ChunkSmem<NN>::TOTAL, stream>>>((const __nv_bfloat16*)xbc, ldx, (const __nv_bfloat16*)dt_in, ld_dt, dt_bias, A, \
            state, state_stride, out, seg_q_start, seg_slot, H, V, G); } while (0)
    if (N == 128) GO(128); else GO(64);
#undef GO
    return (int)cudaGetLastError();
}

// A step whose entries bring one token each.  p [T, ldp] = z | x | B | C | dt; out float32 [T, H V] = S^T C + D x; the convolution's inputs
// behind the state in the slot are read, not moved (mi_gated_part_norm does that).
MI_EXPORT int mi_ssd_step(const void* p, int ldp, const float* conv, const float* conv_b, int taps, const float* dt_bias, const float* A, const float* Dv,
                          float* state, long long state_stride, float* out, const int* seg_q_start, const int* seg_slot, int num_segs, int H, int V, int N, int G,
                          int dtype, cudaStream_t stream) {
    if (num_segs == 0) return 0;
    if (H > 65535 || H % G || taps < 1) return -2;
    const bool vec = V % 4 == 0 && state_stride % 4 == 0 && (uintptr_t)state % 16 == 0 && ((long long)N * V) % 4 == 0;
    const int cols = vec ? V / 4 : V, rows = cols >= 256 ? 1 : 256 / cols;
    const size_t smem = (size_t)(V + 2 * N + rows * V) * sizeof(float);
    if (smem > 48 * 1024) return -2;
    const dim3 grid(num_segs, H);
#define STEP(T, VEC, TAPS) ssd_step_kernel<T, VEC, TAPS><<<grid, 256, smem, stream>>>((const T*)p, ldp, conv, conv_b, taps, dt_bias, A, Dv, state, state_stride, out, \
                                                                                 seg_q_start, seg_slot, H, V, N, G)
#define GO(T, VEC) do { if (taps == 4) STEP(T, VEC, 4); else if (taps == 3) STEP(T, VEC, 3); else STEP(T, VEC, 0); } while (0)
    if (dtype == MI_BF16) { if (vec) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
    else { if (vec) GO(float, 4); else GO(float, 1); }
#undef STEP
#undef GO
    return (int)cudaGetLastError();
}

// y float32 [T, I]; x (rows ldx apart, null: y holds D x already), z (rows ldz apart) and out [T, I] in dtype; parts equal parts of I / parts.
// state not null (a step of single tokens, one a slot): the slots' convolution inputs, float32 [taps - 1, C] at `off`, move up by one and
// receive the C columns that stand behind z's I.
MI_EXPORT int mi_gated_part_norm(const float* y, const void* x, int ldx, const float* Dv, int V, const void* z, int ldz, const float* w, void* out, int T_, int I,
                                 int parts, float eps, float* state, long long state_stride, long long off, const int* seg_slot, int C, int taps, int dtype,
                                 cudaStream_t stream) {
    if (T_ == 0) return 0;
    if (I % parts || parts > 65535) return -2;
    const int gs = I / parts;
    const Tail tail{taps > 1 ? state : nullptr, state_stride, off, seg_slot, C, taps, parts};
    const dim3 grid(T_, parts + (tail.state ? (C + 255) / 256 : 0));
    const bool vec = dtype == MI_BF16 && gs % 8 == 0 && gs <= 8192 && I % 8 == 0 && ldz % 8 == 0 && (!x || (ldx % 8 == 0 && V % 8 == 0)) &&
                     ((uintptr_t)y | (uintptr_t)x | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out) % 16 == 0;
#define GO(T, VPT) gated_part_norm_kernel<T, VPT><<<grid, 256, 0, stream>>>(y, (const T*)x, ldx, Dv, V, (const T*)z, ldz, w, (T*)out, I, gs, eps, tail)
    if (vec) { if (gs <= 2048) GO(__nv_bfloat16, 1); else if (gs <= 4096) GO(__nv_bfloat16, 2); else GO(__nv_bfloat16, 4); }
    else if (dtype == MI_BF16) GO(__nv_bfloat16, 0);
    else GO(float, 0);
#undef GO
    return (int)cudaGetLastError();
}
