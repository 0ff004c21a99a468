// Prompts of the gated delta rule (gated_delta.cu) in chunks of 64 tokens on the tensor cores, for key and value heads of 64 or 128.
//
// Over a chunk that starts from the state S_0 [D, V], with c_t the sum of the logarithms of the decays up to token t (inclusive),
// K, Q [64, D], V [64, V] and D(x) a diagonal matrix, the recurrence S <- f S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q unrolls to
//     (I + A) U = D(beta) V - D(beta e^c) K S_0,      A_ts = beta_t e^(c_t - c_s) (k_t . k_s) for s < t, 0 otherwise
//     O  = D(e^c) Q S_0 + P U,                        P_ts = e^(c_t - c_s) (q_t . k_s) for s <= t
//     S' = e^(c_63) S_0 + (D(e^(c_63 - c)) K)^T U
// With T = (I + A)^-1, W = T D(beta e^c) K and U_0 = T D(beta) V do not depend on the state, so
//     delta_chunk_kernel   makes -W, U_0, P, D(e^c) Q, D(e^(c_63 - c)) K of every chunk and head, all at once (grid: chunks x heads)
//     delta_pass_kernel    walks an entry's chunks in order with the state in accumulators (grid: entries x heads x groups of columns):
//                          U = U_0 - W S,  O = Q' S + P U,  S = e^(c_63) S + K'^T U
// Float32 operands of a product enter as TWO bfloat16 numbers (the rounding and what it leaves) and three products (hi hi, hi lo, lo hi):
// 16 mantissa bits each, float32 sums.  Decays, their sums, the inverse and the state are float32.  An entry's last chunk is filled up with
// tokens of k = q = v = 0, beta = 0 and decay 1, which change nothing.
#include "sm100.cuh"
#include <math.h>

using namespace mi;
using namespace mi::sm100;

namespace {

constexpr int Q = 64, NTH = 256;
constexpr float LOG2E = 1.4426950408889634f;

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
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float rest(float x) { return x - __bfloat162float(__float2bfloat16_rn(x)); }
__device__ __forceinline__ float low_of(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float high_of(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
// c[t] += (ah + al) (bh_t + bl_t) without al bl_t for N neighbouring tiles of 8 columns, their two halves each as ldmatrix left them (two
// tiles a register group).  Product by product over all tiles, so that a tile's three sums do not wait for one another.
template <int N>
__device__ __forceinline__ void mma3(float (&c)[N][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[(N + 1) / 2][4], const uint32_t (&bl)[(N + 1) / 2][4]) {
#pragma unroll
    for (int t = 0; t < N; ++t) mma16816(c[t], ah, bh[t / 2][2 * (t % 2)], bh[t / 2][2 * (t % 2) + 1]);
#pragma unroll
    for (int t = 0; t < N; ++t) mma16816(c[t], ah, bl[t / 2][2 * (t % 2)], bl[t / 2][2 * (t % 2) + 1]);
#pragma unroll
    for (int t = 0; t < N; ++t) mma16816(c[t], al, bh[t / 2][2 * (t % 2)], bh[t / 2][2 * (t % 2) + 1]);
}

// byte offset of the 16-byte piece `ch` of row `row` in a tile of rows of N bfloat16 (N a multiple of 64; pieces XOR-ed with the row so that
// ldmatrix meets no bank twice), and in a tile of rows of 32 or 16 of them
template <int N> __device__ __forceinline__ uint32_t at(int row, int ch) {
    if constexpr (N >= 64) return (uint32_t)(row * N * 2 + ((ch ^ (row & 7)) << 4));
    else if constexpr (N == 32) return (uint32_t)(row * 64 + ((ch ^ ((row >> 1) & 3)) << 4));
    else return (uint32_t)(row * 32 + ((ch ^ ((row >> 2) & 1)) << 4));
}

// What delta_chunk_kernel leaves per (chunk, head), in the order and swizzle in which delta_pass_kernel copies it to shared memory
template <int D, int V> struct Work {
    static constexpr int KD = Q * D * 2, PP = Q * Q * 2;                   // bytes of one bfloat16 half
    static constexpr int WQ = 4 * KD;                                      // -W hi | lo | Q' hi | lo
    static constexpr int KP = 2 * KD + 2 * PP;                             // K' hi | lo | P hi | lo
    static constexpr int U0 = Q * V * 4;                                   // float32
    static constexpr long long BYTES = WQ + KP + U0 + 16;                  // and e^(c_63)
};

template <int D, int V> struct PrepareSmem {
    static constexpr int K = 0, QV = 2 * Q * D * 2, MAXDV = D > V ? D : V, A = QV + 2 * Q * MAXDV * 2, LDA = 68;
    static constexpr int T = A + Q * LDA * 4, GATES = T + Q * LDA * 4, TOTAL = GATES + 4 * Q * 4;
};

// rows of N floats, ld apart (rows beyond n: zeros), -> two bfloat16 tiles
// (fetch: all of a thread's pieces at once, into registers; store: what they hold)
template <int N> struct Pieces { float4 v[2 * Q * (N / 8) / NTH]; };
template <int N> __device__ __forceinline__ Pieces<N> fetch_rows(const float* __restrict__ src, int ld, int n) {
    Pieces<N> p;
#pragma unroll
    for (int i = 0; i < Q * (N / 8) / NTH; ++i) {
        const int id = threadIdx.x + i * NTH, row = id / (N / 8), ch = id % (N / 8);
        const float* s = src + (size_t)row * ld + ch * 8;
        p.v[2 * i] = row < n ? *reinterpret_cast<const float4*>(s) : make_float4(0.f, 0.f, 0.f, 0.f);
        p.v[2 * i + 1] = row < n ? *reinterpret_cast<const float4*>(s + 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    return p;
}
template <int N> __device__ __forceinline__ void store_rows(unsigned char* hi, unsigned char* lo, const Pieces<N>& p) {
#pragma unroll
    for (int i = 0; i < Q * (N / 8) / NTH; ++i) {
        const int id = threadIdx.x + i * NTH, row = id / (N / 8), ch = id % (N / 8);
        const float4 a = p.v[2 * i], b = p.v[2 * i + 1];
        *reinterpret_cast<uint4*>(hi + at<N>(row, ch)) = make_uint4(pack2(a.x, a.y), pack2(a.z, a.w), pack2(b.x, b.y), pack2(b.z, b.w));
        *reinterpret_cast<uint4*>(lo + at<N>(row, ch)) = make_uint4(pack2(rest(a.x), rest(a.y)), pack2(rest(a.z), rest(a.w)), pack2(rest(b.x), rest(b.y)), pack2(rest(b.z), rest(b.w)));
    }
}

// dst (hi | lo, the same swizzle) = scale[row] * (hi + lo)
template <int N> __device__ __forceinline__ void scale_rows(unsigned char* dst, const unsigned char* hi, const unsigned char* lo, const float* scale) {
    for (int id = threadIdx.x; id < Q * (N / 8); id += NTH) {
        const int row = id / (N / 8);
        const uint32_t off = at<N>(row, id % (N / 8));
        const uint4 h = *reinterpret_cast<const uint4*>(hi + off), l = *reinterpret_cast<const uint4*>(lo + off);
        const float s = scale[row];
        const uint32_t hw[4] = {h.x, h.y, h.z, h.w}, lw[4] = {l.x, l.y, l.z, l.w};
        uint32_t oh[4], ol[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float a = s * (low_of(hw[i]) + low_of(lw[i])), b = s * (high_of(hw[i]) + high_of(lw[i]));
            oh[i] = pack2(a, b);
            ol[i] = pack2(rest(a), rest(b));
        }
        *reinterpret_cast<uint4*>(dst + off) = make_uint4(oh[0], oh[1], oh[2], oh[3]);
        *reinterpret_cast<uint4*>(dst + Q * N * 2 + off) = make_uint4(ol[0], ol[1], ol[2], ol[3]);
    }
}

// the 16 x 32 tile (row block rb, column half ch) of X K^T, X and K split tiles of D columns
template <int D> __device__ __forceinline__ void scores(float (&s)[4][4], uint32_t xh, uint32_t xl, uint32_t kh, uint32_t kl, int rb, int ch, int lane) {
    const int m = lane >> 3;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) { s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f; }
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t ah[4], al[4], bh[2][4], bl[2][4];
        const uint32_t ao = at<D>(rb * 16 + (lane & 7) + (m & 1) * 8, ks * 2 + (m >> 1));
        ldsm4(ah, xh + ao);
        ldsm4(al, xl + ao);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            const uint32_t bo = at<D>(ch * 32 + (2 * np + (m >> 1)) * 8 + (lane & 7), ks * 2 + (m & 1));
            ldsm4(bh[np], kh + bo);
            ldsm4(bl[np], kl + bo);
        }
        mma3<4>(s, ah, al, bh, bl);
    }
}

// the rows rb * 16 .. of T D(scale) X for the N / 2 columns of half `half`; T float32 lower triangular in shared memory, X a split tile of N columns
template <int N> __device__ __forceinline__ void apply_inverse(float (&acc)[N / 64][4][4], const float* T, int lda, const float* scale, uint32_t xh, uint32_t xl,
                                                               int rb, int half, int lane) {
    const int g = lane >> 2, c = lane & 3, m = lane >> 3;
#pragma unroll
    for (int i = 0; i < N / 4; ++i) acc[i / 16][i / 4 % 4][i % 4] = 0.f;
    for (int kb = 0; kb <= rb; ++kb) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int row = rb * 16 + g + (i & 1) * 8, col = kb * 16 + 2 * c + (i >> 1) * 8;
            const float2 t = *reinterpret_cast<const float2*>(T + row * lda + col), s = *reinterpret_cast<const float2*>(scale + col);
            ah[i] = pack2(t.x * s.x, t.y * s.y);
            al[i] = pack2(rest(t.x * s.x), rest(t.y * s.y));
        }
#pragma unroll
        for (int q4 = 0; q4 < N / 64; ++q4) {                      // four tiles of 8 columns at a time
            uint32_t bh[2][4], bl[2][4];
#pragma unroll
            for (int np = 0; np < 2; ++np) {
                const uint32_t bo = at<N>(kb * 16 + (m & 1) * 8 + (lane & 7), half * (N / 16) + 4 * q4 + 2 * np + (m >> 1));
                ldsm4t(bh[np], xh + bo);
                ldsm4t(bl[np], xl + bo);
            }
            mma3<4>(acc[q4], ah, al, bh, bl);
        }
    }
}

// X += sum over k of A[i, k] T[k, j] for one 16 x 16 block (ib, jb), k-blocks kb0 .. kb1-1; thread e of 64 owns row e / 4, columns 4 (e % 4) ..
__device__ __forceinline__ float4 block_product(const float* A, const float* T, int lda, int ib, int jb, int kb0, int kb1, int e) {
    const float* a = A + (ib * 16 + (e >> 2)) * lda;
    const float* t = T + jb * 16 + (e & 3) * 4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int kb = kb0; kb < kb1; ++kb)
#pragma unroll
        for (int kk = 0; kk < 16; kk += 4) {
            const float4 av = *reinterpret_cast<const float4*>(a + kb * 16 + kk);
            const float ae[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
            for (int e4 = 0; e4 < 4; ++e4) {
                const float4 tv = *reinterpret_cast<const float4*>(t + (kb * 16 + kk + e4) * lda);
                s.x = fmaf(ae[e4], tv.x, s.x); s.y = fmaf(ae[e4], tv.y, s.y); s.z = fmaf(ae[e4], tv.z, s.z); s.w = fmaf(ae[e4], tv.w, s.w);
            }
        }
    return s;
}

// grid (chunks, heads h0 .. ).  prep rows: q [KV D] | k [KV D] | v [H V] | beta [H] | f [H] | log f [H]
template <int D, int V>
__global__ void __launch_bounds__(NTH, 2) delta_chunk_kernel(const float* __restrict__ prep, int ld, const int* __restrict__ chunks, const int* __restrict__ seg_q_start,
                                                             unsigned char* __restrict__ work, int H, int KV, int h0) {
    using L = PrepareSmem<D, V>;
    using W = Work<D, V>;
    extern __shared__ __align__(1024) unsigned char smem[];
    const uint32_t base = smem_u32(smem);
    float* A = reinterpret_cast<float*>(smem + L::A);
    float* T = reinterpret_cast<float*>(smem + L::T);
    float* beta = reinterpret_cast<float*>(smem + L::GATES);
    float* cum = beta + Q;                                         // c_t, base 2
    float* bg = cum + Q;                                           // beta e^c, then e^c
    float* tail = bg + Q;                                          // e^(c_63 - c)
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
    const int h = h0 + blockIdx.y, kvh = h / (H / KV);
    const int seg = chunks[2 * blockIdx.x], r0 = chunks[2 * blockIdx.x + 1];
    const int t0 = seg_q_start[seg] + r0, n = min(Q, seg_q_start[seg + 1] - t0);
    const float* rows = prep + (size_t)t0 * ld;
    const int C = 2 * KV * D + H * V;
    unsigned char* wq = work + ((long long)blockIdx.x * gridDim.y + blockIdx.y) * W::BYTES;
    unsigned char* kp = wq + W::WQ;
    float* u0 = reinterpret_cast<float*>(kp + W::KP);

    const Pieces<D> kp_in = fetch_rows<D>(rows + KV * D + kvh * D, ld, n), qp_in = fetch_rows<D>(rows + kvh * D, ld, n);
    for (int i = tid; i < Q * L::LDA; i += NTH) { A[i] = 0.f; T[i] = 0.f; }
    if (warp == 0) {                                               // two tokens a lane: beta, sums of the decays' logarithms
        const int i = 2 * lane;
        const float* ra = rows + (size_t)i * ld + C + h;
        const float* rb = ra + ld;
        beta[i] = i < n ? ra[0] : 0.f;
        beta[i + 1] = i + 1 < n ? rb[0] : 0.f;
        const float l0 = i < n ? ra[2 * H] * LOG2E : 0.f, l1 = i + 1 < n ? rb[2 * H] * LOG2E : 0.f;
        float incl = l0 + l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        cum[i] = incl - l1; cum[i + 1] = incl;
        const float last = __shfl_sync(0xffffffffu, incl, 31);
        bg[i] = beta[i] * exp2f(incl - l1); bg[i + 1] = beta[i + 1] * exp2f(incl);
        tail[i] = exp2f(last - (incl - l1)); tail[i + 1] = exp2f(last - incl);
        if (lane == 31) *reinterpret_cast<float*>(kp + W::KP + W::U0) = exp2f(last);
    }
    store_rows<D>(smem + L::K, smem + L::K + Q * D * 2, kp_in);
    store_rows<D>(smem + L::QV, smem + L::QV + Q * D * 2, qp_in);
    __syncthreads();
    // the six 16 x 32 tiles that reach below the diagonal: (0,0) (1,0) (2,0) (2,1) (3,0) (3,1)
    auto task_rb = [](int i) { return i < 2 ? i : i < 4 ? 2 : 3; };
    auto task_ch = [](int i) { return i == 3 || i == 5 ? 1 : 0; };
    const uint32_t kh = base + L::K, kl = kh + Q * D * 2, qh = base + L::QV, ql = qh + Q * D * 2;
    if (warp < 6) {
        float s[4][4];
        const int rb = task_rb(warp), ch = task_ch(warp);
        scores<D>(s, kh, kl, kh, kl, rb, ch, lane);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = rb * 16 + g + (e >> 1) * 8, u = ch * 32 + nt * 8 + 2 * c + (e & 1);
                if (u < t) A[t * L::LDA + u] = beta[t] * exp2f(cum[t] - cum[u]) * s[nt][e];
            }
    }
    __syncthreads();
    if (warp >= 2) {                                               // P, while two warps invert the diagonal blocks of I + A
        float s[4][4];
        const int rb = task_rb(warp - 2), ch = task_ch(warp - 2);
        scores<D>(s, qh, ql, kh, kl, rb, ch, lane);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int t = rb * 16 + g + hf * 8, u = ch * 32 + nt * 8 + 2 * c;
                const float a = u <= t ? exp2f(cum[t] - cum[u]) * s[nt][2 * hf] : 0.f, b = u + 1 <= t ? exp2f(cum[t] - cum[u + 1]) * s[nt][2 * hf + 1] : 0.f;
                const uint32_t off = 2 * W::KD + at<Q>(t, ch * 4 + nt) + 4 * c;
                *reinterpret_cast<uint32_t*>(kp + off) = pack2(a, b);
                *reinterpret_cast<uint32_t*>(kp + W::PP + off) = pack2(rest(a), rest(b));
            }
    } else {                                                       // thread (block b, column j): x_j = 1, x_i = -sum_{j <= k < i} A_ik x_k
        const int b = tid >> 4, j = tid & 15;
        const float* a = A + (b * 16) * L::LDA + b * 16;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = 0.f, s2 = 0.f;
#pragma unroll
            for (int k = 0; k < i; k += 2) {
                s = fmaf(a[i * L::LDA + k], x[k], s);
                if (k + 1 < i) s2 = fmaf(a[i * L::LDA + k + 1], x[k + 1], s2);
            }
            s += s2;
            x[i] = i < j ? 0.f : i == j ? 1.f : -s;
            T[(b * 16 + i) * L::LDA + b * 16 + j] = x[i];
        }
    }
    __syncthreads();
    // Q' = D(e^c) Q leaves; e^c stands in bg's place once beta e^c is no longer needed, so it is made from cum here
    for (int id = tid; id < Q * (D / 8); id += NTH) {
        const int row = id / (D / 8);
        const uint32_t off = at<D>(row, id % (D / 8));
        const uint4 hq = *reinterpret_cast<const uint4*>(smem + L::QV + off), lq = *reinterpret_cast<const uint4*>(smem + L::QV + Q * D * 2 + off);
        const float s = exp2f(cum[row]);
        const uint32_t hw[4] = {hq.x, hq.y, hq.z, hq.w}, lw[4] = {lq.x, lq.y, lq.z, lq.w};
        uint32_t oh[4], ol[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float a = s * (low_of(hw[i]) + low_of(lw[i])), b = s * (high_of(hw[i]) + high_of(lw[i]));
            oh[i] = pack2(a, b);
            ol[i] = pack2(rest(a), rest(b));
        }
        *reinterpret_cast<uint4*>(wq + 2 * W::KD + off) = make_uint4(oh[0], oh[1], oh[2], oh[3]);
        *reinterpret_cast<uint4*>(wq + 3 * W::KD + off) = make_uint4(ol[0], ol[1], ol[2], ol[3]);
    }
    scale_rows<D>(kp, smem + L::K, smem + L::K + Q * D * 2, tail);                 // K'
    const Pieces<V> v_in = fetch_rows<V>(rows + 2 * KV * D + h * V, ld, n);
    // the blocks of T below the diagonal, by distance d from it: T_ij = -T_ii sum_{j <= k < i} A_ik T_kj
    for (int d = 1; d < 4; ++d) {
        const int blk = tid >> 6, e = tid & 63, ib = blk + d, jb = blk;
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ib < 4) y = block_product(A, T, L::LDA, ib, jb, jb, ib, e);
        __syncthreads();
        float* at_ij = T + (ib * 16 + (e >> 2)) * L::LDA + jb * 16 + (e & 3) * 4;
        if (ib < 4) *reinterpret_cast<float4*>(at_ij) = y;
        __syncthreads();
        if (ib < 4) y = block_product(T, T, L::LDA, ib, jb, ib, ib + 1, e);       // T_ii (rows of block ib, columns ib) times what now stands at (ib, jb)
        __syncthreads();
        if (ib < 4) *reinterpret_cast<float4*>(at_ij) = make_float4(-y.x, -y.y, -y.z, -y.w);
        __syncthreads();
    }
    store_rows<V>(smem + L::QV, smem + L::QV + Q * V * 2, v_in);      // Q is no longer needed
    __syncthreads();
    const int rb = warp >> 1, half = warp & 1;
    {
        float acc[D / 64][4][4];
        apply_inverse<D>(acc, T, L::LDA, bg, kh, kl, rb, half, lane);
#pragma unroll
        for (int nt = 0; nt < D / 16; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const uint32_t off = at<D>(rb * 16 + g + hf * 8, half * (D / 16) + nt) + 4 * c;
                const float a = -acc[nt / 4][nt % 4][2 * hf], b = -acc[nt / 4][nt % 4][2 * hf + 1];
                *reinterpret_cast<uint32_t*>(wq + off) = pack2(a, b);
                *reinterpret_cast<uint32_t*>(wq + W::KD + off) = pack2(rest(a), rest(b));
            }
    }
    {
        float acc[V / 64][4][4];
        apply_inverse<V>(acc, T, L::LDA, beta, base + L::QV, base + L::QV + Q * V * 2, rb, half, lane);
#pragma unroll
        for (int nt = 0; nt < V / 16; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf)
                *reinterpret_cast<float2*>(u0 + (rb * 16 + g + hf * 8) * V + half * (V / 2) + nt * 8 + 2 * c) = make_float2(acc[nt / 4][nt % 4][2 * hf], acc[nt / 4][nt % 4][2 * hf + 1]);
    }
}

// ------------------------------------------------------------------ the pass over an entry's chunks
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
                 :: "r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

template <int D, int V, int NC> struct PassSmem {
    static constexpr int WQ = 0, KP = Work<D, V>::WQ, S = KP + Work<D, V>::KP, U = S + 2 * D * NC * 2, BAR = U + 2 * Q * NC * 2, TOTAL = BAR + 16;
};

// grid (entries, heads h0 .., V / NC), NC columns a block
template <int D, int V, int NC>
__global__ void __launch_bounds__(NTH, 1) delta_pass_kernel(const unsigned char* __restrict__ work, const int* __restrict__ chunk_start, float* __restrict__ state,
                                                            long long state_stride, float* __restrict__ out, const int* __restrict__ seg_q_start,
                                                            const int* __restrict__ seg_slot, int H, int h0, int* __restrict__ error) {
    using L = PassSmem<D, V, NC>;
    using W = Work<D, V>;
    extern __shared__ __align__(1024) unsigned char smem[];
    const uint32_t base = smem_u32(smem), bar_wq = base + L::BAR, bar_kp = bar_wq + 8;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3, m = lane >> 3;
    const int seg = blockIdx.x, h = h0 + blockIdx.y, v0 = blockIdx.z * NC;
    const int qs = seg_q_start[seg], n = seg_q_start[seg + 1] - qs, chunks = (n + Q - 1) / Q;
    const long long step = (long long)gridDim.y * W::BYTES;
    const unsigned char* first = work + (long long)chunk_start[seg] * step + (long long)blockIdx.y * W::BYTES;
    if (tid == 0) {
        mbar_init(bar_wq, 1);
        mbar_init(bar_kp, 1);
        mbar_init_fence();
    }
    __syncthreads();
    auto fetch_wq = [&](int k) {
        const unsigned char* src = first + k * step;
        mbar_expect_tx(bar_wq, W::WQ);
        for (int i = 0; i < 4; ++i) bulk_load(base + L::WQ + i * W::KD, src + i * W::KD, W::KD, bar_wq);
    };
    auto fetch_kp = [&](int k) {
        const unsigned char* src = first + k * step + W::WQ;
        mbar_expect_tx(bar_kp, W::KP);
        bulk_load(base + L::KP, src, W::KD, bar_kp);
        bulk_load(base + L::KP + W::KD, src + W::KD, W::KD, bar_kp);
        bulk_load(base + L::KP + 2 * W::KD, src + 2 * W::KD, 2 * W::PP, bar_kp);
    };
    if (tid == 0) { fetch_wq(0); fetch_kp(0); }
    bool alive = true;                                             // a wait that ran out is recorded once; no further ones follow
    auto await = [&](uint32_t bar, int k) {
        if (alive && !mbar_wait(bar, k & 1)) { alive = false; atomicExch(error, 71); }
    };

    // Of U and O a warp has either the same 16 rows and half the columns of both, or (NC = 16, where the reads of W and Q' from shared memory
    // are what counts) 16 rows and all columns of one of them: warps 0 .. 3 of U, 4 .. 7 of O.  Of the state: row block sb, columns sc0 ..
    constexpr bool ROLES = NC == 16;
    constexpr int NT = 2, SB = D / 16, SW = 8 / SB, SNT = NC / 8 / SW;      // tiles of 8 columns a warp has of U and O; of the state
    const int rb = warp & 3, nc0 = ROLES ? 0 : (warp >> 2) * (NC / 2), sb = warp % SB, sc0 = warp / SB * (NC / SW);
    const bool has_u = !ROLES || warp < 4, has_o = !ROLES || warp >= 4;
    float* S = state + (long long)seg_slot[seg] * state_stride + (long long)h * D * V + v0;
    float s[SNT][4];
    auto spread_state = [&]() {
#pragma unroll
        for (int nt = 0; nt < SNT; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const uint32_t off = at<NC>(sb * 16 + g + hf * 8, sc0 / 8 + nt) + 4 * c;
                *reinterpret_cast<uint32_t*>(smem + L::S + off) = pack2(s[nt][2 * hf], s[nt][2 * hf + 1]);
                *reinterpret_cast<uint32_t*>(smem + L::S + D * NC * 2 + off) = pack2(rest(s[nt][2 * hf]), rest(s[nt][2 * hf + 1]));
            }
    };
#pragma unroll
    for (int nt = 0; nt < SNT; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const float2 t = *reinterpret_cast<const float2*>(S + (size_t)(sb * 16 + g + hf * 8) * V + sc0 + nt * 8 + 2 * c);
            s[nt][2 * hf] = t.x;
            s[nt][2 * hf + 1] = t.y;
        }
    spread_state();
    float next_u[NT][4], next_decay = 0.f;
    auto fetch_u = [&](int k) {
        if (!has_u) { next_decay = reinterpret_cast<const float*>(first + k * step + W::WQ + W::KP)[Q * V]; return; }
        const float* u0 = reinterpret_cast<const float*>(first + k * step + W::WQ + W::KP);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const float2 t = *reinterpret_cast<const float2*>(u0 + (rb * 16 + g + hf * 8) * V + v0 + nc0 + nt * 8 + 2 * c);
                next_u[nt][2 * hf] = t.x;
                next_u[nt][2 * hf + 1] = t.y;
            }
        next_decay = u0[Q * V];
    };
    fetch_u(0);
    __syncthreads();
    for (int k = 0; k < chunks; ++k) {
        float u[NT][4], o[NT][4];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) { u[nt][e] = has_u ? next_u[nt][e] : 0.f; o[nt][e] = 0.f; }
        const float decay = next_decay;
        if (k + 1 < chunks) fetch_u(k + 1);
        await(bar_wq, k);
        const uint32_t mine = base + L::WQ + (has_u ? 0 : 2 * W::KD);
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {                      // U = U_0 - W S;  O = Q' S
            uint32_t ah[4], al[4], bh[1][4], bl[1][4];
            const uint32_t ao = at<D>(rb * 16 + (lane & 7) + (m & 1) * 8, ks * 2 + (m >> 1));
            const uint32_t bo = at<NC>(ks * 16 + (m & 1) * 8 + (lane & 7), nc0 / 8 + (m >> 1));
            ldsm4t(bh[0], base + L::S + bo);
            ldsm4t(bl[0], base + L::S + D * NC * 2 + bo);
            if constexpr (ROLES) {
                ldsm4(ah, mine + ao);
                ldsm4(al, mine + W::KD + ao);
                mma3<NT>(u, ah, al, bh, bl);                       // U, or O held in u
            } else {
                uint32_t qh[4], ql[4];
                ldsm4(ah, base + L::WQ + ao);
                ldsm4(al, base + L::WQ + W::KD + ao);
                ldsm4(qh, base + L::WQ + 2 * W::KD + ao);
                ldsm4(ql, base + L::WQ + 3 * W::KD + ao);
                mma3<NT>(u, ah, al, bh, bl);
                mma3<NT>(o, qh, ql, bh, bl);
            }
        }
        if constexpr (ROLES) {
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[nt][e] = u[nt][e];
        }
        if (has_u) {
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const uint32_t off = at<NC>(rb * 16 + g + hf * 8, nc0 / 8 + nt) + 4 * c;
                    *reinterpret_cast<uint32_t*>(smem + L::U + off) = pack2(u[nt][2 * hf], u[nt][2 * hf + 1]);
                    *reinterpret_cast<uint32_t*>(smem + L::U + Q * NC * 2 + off) = pack2(rest(u[nt][2 * hf]), rest(u[nt][2 * hf + 1]));
                }
        }
        __syncthreads();                                           // U is complete; W and Q' have been read
        if (tid == 0 && k + 1 < chunks) fetch_wq(k + 1);
        await(bar_kp, k);
#pragma unroll
        for (int nt = 0; nt < SNT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nt][e] *= decay;
#pragma unroll
        for (int kb = 0; kb < Q / 16; ++kb) {
            if (has_o && kb <= rb) {                               // O += P U
                uint32_t ph[4], pl[4], uh[1][4], ul[1][4];
                const uint32_t ao = at<Q>(rb * 16 + (lane & 7) + (m & 1) * 8, kb * 2 + (m >> 1));
                ldsm4(ph, base + L::KP + 2 * W::KD + ao);
                ldsm4(pl, base + L::KP + 2 * W::KD + W::PP + ao);
                const uint32_t bo = at<NC>(kb * 16 + (m & 1) * 8 + (lane & 7), nc0 / 8 + (m >> 1));
                ldsm4t(uh[0], base + L::U + bo);
                ldsm4t(ul[0], base + L::U + Q * NC * 2 + bo);
                mma3<NT>(o, ph, pl, uh, ul);
            }
            uint32_t ah[4], al[4], uh[(SNT + 1) / 2][4], ul[(SNT + 1) / 2][4];      // S += K'^T U
            const uint32_t ao = at<D>(kb * 16 + (m >> 1) * 8 + (lane & 7), sb * 2 + (m & 1));
            ldsm4t(ah, base + L::KP + ao);
            ldsm4t(al, base + L::KP + W::KD + ao);
#pragma unroll
            for (int np = 0; np < (SNT + 1) / 2; ++np) {
                // (one tile a warp: the upper two matrices are read all the same and left unused)
                const uint32_t bo = at<NC>(kb * 16 + (m & 1) * 8 + (lane & 7), SNT > 1 ? sc0 / 8 + 2 * np + (m >> 1) : sc0 / 8);
                ldsm4t(uh[np], base + L::U + bo);
                ldsm4t(ul[np], base + L::U + Q * NC * 2 + bo);
            }
            mma3<SNT>(s, ah, al, uh, ul);
        }
        spread_state();
        if (has_o)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int t = k * Q + rb * 16 + g + hf * 8;
                if (t < n) *reinterpret_cast<float2*>(out + (size_t)(qs + t) * H * V + (size_t)h * V + v0 + nc0 + nt * 8 + 2 * c) = make_float2(o[nt][2 * hf], o[nt][2 * hf + 1]);
            }
        __syncthreads();                                           // the state is spread; K', P and U have been read
        if (tid == 0 && k + 1 < chunks) fetch_kp(k + 1);
    }
#pragma unroll
    for (int nt = 0; nt < SNT; ++nt)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
            *reinterpret_cast<float2*>(S + (size_t)(sb * 16 + g + hf * 8) * V + sc0 + nt * 8 + 2 * c) = make_float2(s[nt][2 * hf], s[nt][2 * hf + 1]);
}

template <int D, int V>
int launch_chunks(const float* prep, int ld, const int* chunks, int num_chunks, const int* chunk_start, void* work, long long work_bytes, float* state,
                  long long state_stride, float* out, const int* seg_q_start, const int* seg_slot, int num_segs, int H, int KV, int* error, cudaStream_t stream) {
    const long long per_head = num_chunks * Work<D, V>::BYTES;
    const int heads = (int)(work_bytes / per_head < H ? work_bytes / per_head : H);
    if (heads < 1) return -2;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, PrepareSmem<D, V>::TOTAL);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_pass_kernel<D, V, 32>, cudaFuncAttributeMaxDynamicSharedMemorySize, PassSmem<D, V, 32>::TOTAL);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_pass_kernel<D, V, 16>, cudaFuncAttributeMaxDynamicSharedMemorySize, PassSmem<D, V, 16>::TOTAL);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    for (int h0 = 0; h0 < H; h0 += heads) {                        // as many heads at a time as the work space holds
        const int nh = H - h0 < heads ? H - h0 : heads;
        delta_chunk_kernel<D, V><<<dim3(num_chunks, nh), NTH, PrepareSmem<D, V>::TOTAL, stream>>>(prep, ld, chunks, seg_q_start, (unsigned char*)work, H, KV, h0);
        const bool narrow = (long long)num_segs * nh * (V / 32) < 148;      // few blocks: half the columns each
        if (narrow)
            delta_pass_kernel<D, V, 16><<<dim3(num_segs, nh, V / 16), NTH, PassSmem<D, V, 16>::TOTAL, stream>>>((const unsigned char*)work, chunk_start, state, state_stride,
                                                                                                               out, seg_q_start, seg_slot, H, h0, error);
        else
            delta_pass_kernel<D, V, 32><<<dim3(num_segs, nh, V / 32), NTH, PassSmem<D, V, 32>::TOTAL, stream>>>((const unsigned char*)work, chunk_start, state, state_stride,
                                                                                                               out, seg_q_start, seg_slot, H, h0, error);
    }
    return (int)cudaGetLastError();
}

}  // namespace

// prep [T, ld] float32 = q [KV D] | k [KV D] | v [H V] | beta [H] | f [H] | log f [H]; chunks [num_chunks, 2] = (entry, first row), an entry's
// chunks of 64 rows in order; chunk_start [entries]: the number of an entry's first chunk.  work: scratch, 16-byte aligned, of at least
// mi_delta_chunk_bytes per chunk (for one head at a time; more lets more heads run at once).  -2: sizes that have no such form.
MI_EXPORT int mi_delta_chunk_bytes(int D, int V) {
    if (D == 128 && V == 128) return (int)Work<128, 128>::BYTES;
    if (D == 128 && V == 64) return (int)Work<128, 64>::BYTES;
    if (D == 64 && V == 128) return (int)Work<64, 128>::BYTES;
    if (D == 64 && V == 64) return (int)Work<64, 64>::BYTES;
    return -2;
}

MI_EXPORT int mi_gated_delta_chunks(const float* prep, int ld, const int* chunks, int num_chunks, const int* chunk_start, void* work, long long work_bytes,
                                    float* state, long long state_stride, float* out, const int* seg_q_start, const int* seg_slot, int num_segs, int H, int KV,
                                    int D, int V, int* error, cudaStream_t stream) {
    if (num_chunks == 0) return 0;
    if (H % KV || H > 65535 || ld % 4 || state_stride % 2 || ((uintptr_t)prep | (uintptr_t)work) % 16 || (uintptr_t)state % 8) return -2;
#define GO(DD, VV) return launch_chunks<DD, VV>(prep, ld, chunks, num_chunks, chunk_start, work, work_bytes, state, state_stride, out, seg_q_start, seg_slot, num_segs, H, KV, error, stream)
    if (D == 128 && V == 128) GO(128, 128);
    if (D == 128 && V == 64) GO(128, 64);
    if (D == 64 && V == 128) GO(64, 128);
    if (D == 64 && V == 64) GO(64, 64);
#undef GO
    return -2;
}
