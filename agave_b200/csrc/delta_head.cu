// The gated delta rule with one decay per head, as a recurrent mixer's kernels.
//
// A token's row of the stacked projection is  q | k | v | a | b | g  (G d, G d, H dv, H, H and
// H dv wide).  The convolution kernel of ssm.cu has made q, k and v of it (a short causal
// convolution and silu) and the decay  g_t = exp(neg_a softplus(a + dt_bias))  per head.  Here:
// every q and k head becomes a unit vector (x / sqrt(sum x^2 + eps_unit)), q times a constant
// besides, beta = sigmoid(b), and a head's state S [d, dv] goes, query/key head h / (H / G)
// serving head h,
//
//      S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// (the read-out sees the token's own write); the head's o is divided by its root mean square
// (eps_out), multiplied by a weight [dv] and by silu or sigmoid of its gate.
//
// The recurrence runs several tokens a round.  With tokens 1..n of a round, r_i the factor that
// makes k_i a unit vector, s_i that of q_i, and  G_ij = g_(j+1) .. g_i  (G_i0 = g_1 .. g_i):
//
//      u_i = beta_i (v_i - G_i0 r_i S^T k_i - sum_(j<i) G_ij r_i r_j (k_i . k_j) u_j)
//      o_i = G_i0 s_i S^T q_i + sum_(j<=i) G_ij s_i r_j (q_i . k_j) u_j
//      S   <- G_n0 S + sum_j G_nj r_j k_j u_j^T
//
// the same sums with S as it was before the round, so a round has one pass of dot products with
// the state, whose reductions over a column's lanes do not wait for one another.  What does not
// depend on the state (the dot products among a round's k and q, the decays' products, all of it
// folded into a few numbers a token and head) is made by a launch before for all rounds at
// once; the vectors themselves stay as the convolution left them.  A round begins at the first
// token a sequence brings in the step; a decode step's rounds are one token.
//
// 32-bit throughout.  A prompt and a decoded token differ in the order of these sums alone.
#include "common.cuh"
#include "row_in.cuh"

namespace {

// tokens a round of a prompt, by the size of a key head
__host__ __device__ constexpr int head_round(int d) { return d > 32 ? 8 : 4; }
constexpr int DH_MAX_D = 512;
// numbers a token and head, whole quads
__host__ __device__ constexpr int head_coefs(int n) { return (4 + 2 * n + 3) / 4 * 4; }

struct HeadDims {
    int G, H, d, dv;
    __host__ __device__ int nq() const { return G * d; }
    __host__ __device__ int C() const { return 2 * G * d + H * dv; }
};

__device__ __forceinline__ float silu_f(float t) { return t / (1.0f + expf(-t)); }
__device__ __forceinline__ float sigmoid_f(float t) { return 1.0f / (1.0f + expf(-t)); }

// ------------------------------------------------------------- coefficients
// A warp per (round, query/key head): the dot products by lanes over d, folded so that every lane ends with a few finished sums, then a
// lane per (head, token).  Layout of a token's numbers (i its place in the round, n the round's
// last place):
//   0 beta   1 beta G_i0 r_i   2 G_i0 s_i   3 G_ni r_i
//   4 + j: beta G_ij r_i r_j (k_i . k_j) for j < i, else 0; the last of them is G_n0 instead
//   4 + N + j: G_ij s_i r_j (q_i . k_j) for j <= i, else 0
//
// Sequence b has the rounds from number cu[b] / N + b on: room for its own, ceil(len / N), and
// T / N + B in all (a number that is no sequence's round has nothing to do).
constexpr int DH_COEF_WARPS = 8;

template <int N>
__global__ void __launch_bounds__(DH_COEF_WARPS * 32)
delta_coef_kernel(const float* __restrict__ u, const float* __restrict__ decay, RowIn<float> in,
                  int b_off, HeadDims dm, int n_tokens, int B, float eps_unit, float q_mult,
                  const int* __restrict__ cu, float* __restrict__ coef) {
    pdl_wait();
    pdl_launch_next();
    constexpr int TRI = N * (N + 1) / 2, SUMS = N + 2 * TRI, M = (SUMS + 31) / 32 * 32;
    __shared__ float sums[DH_COEF_WARPS][M];       // |q_i|^2, k_i . k_j, q_i . k_j (j <= i)
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long w = (long long)blockIdx.x * DH_COEF_WARPS + warp;
    const int round = (int)(w / dm.G), grp = (int)(w - (long long)round * dm.G);
    if (round >= n_tokens / N + B) return;
    int b = 0;                                     // the last sequence that starts at or before it
    for (int hi = B - 1; b < hi;) {
        const int mid = (b + hi + 1) >> 1;
        if (cu[mid] / N + mid <= round) b = mid;
        else hi = mid - 1;
    }
    const int first = cu[b], end = cu[b + 1];
    const int t = first + (round - (first / N + b)) * N;
    if (t >= end) return;
    const int m = min(N, end - t);
    const int C = dm.C(), d = dm.d;
    const float* q0 = u + (size_t)t * C + (size_t)grp * d;
    const float* k0 = q0 + dm.nq();
    float v[M];
#pragma unroll
    for (int x = 0; x < M; ++x) v[x] = 0.f;
#pragma unroll 2
    for (int r = lane; r < d; r += 32) {
        float q[N], k[N];
#pragma unroll
        for (int i = 0; i < N; ++i) {
            q[i] = i < m ? q0[(size_t)i * C + r] : 0.f;
            k[i] = i < m ? k0[(size_t)i * C + r] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < N; ++i) {
            v[i] = fmaf(q[i], q[i], v[i]);
#pragma unroll
            for (int j = 0; j <= i; ++j) {
                const int x = N + i * (i + 1) / 2 + j;
                v[x] = fmaf(k[i], k[j], v[x]);
                v[x + TRI] = fmaf(q[i], k[j], v[x + TRI]);
            }
        }
    }
    int at = 0;
#pragma unroll
    for (int bit = 16, half = M / 2; bit >= 1; bit >>= 1, half >>= 1) {
        const bool up = lane & bit;
        if (up) at += half;
#pragma unroll
        for (int x = 0; x < half; ++x) {
            const float out = up ? v[x] : v[x + half], keep = up ? v[x + half] : v[x];
            v[x] = keep + __shfl_xor_sync(0xffffffffu, out, bit);
        }
    }
#pragma unroll
    for (int x = 0; x < M / 32; ++x) sums[warp][at + x] = v[x];
    __syncwarp();
    const float* qq = sums[warp];
    const float* kk = qq + N;
    const float* qk = kk + TRI;
    const int per = dm.H / dm.G;
    for (int e = lane; e < per * N; e += 32) {
        const int i = e % N, h = grp * per + e / N;
        if (i >= m) continue;
        float g[N];
#pragma unroll
        for (int j = 0; j < N; ++j) g[j] = j < m ? decay[((size_t)(t + j) * dm.H + h) * 2] : 1.f;
        const float beta = sigmoid_f(in.at(t + i, b_off + h));
        const int tri = i * (i + 1) / 2;
        const float ri = 1.0f / sqrtf(kk[tri + i] + eps_unit), si = q_mult / sqrtf(qq[i] + eps_unit);
        float before = 1.f, after = 1.f;                     // g_1 .. g_i, g_(i+1) .. g_n
#pragma unroll
        for (int j = 0; j < N; ++j) {
            if (j <= i) before *= g[j];
            else after *= g[j];
        }
        constexpr int NF = head_coefs(N);
        float c[NF] = {};
        c[0] = beta;
        c[1] = beta * before * ri;
        c[2] = before * si;
        c[3] = after * ri;
        float between = 1.f;                                 // g_(j+1) .. g_i
#pragma unroll
        for (int j = N - 1; j >= 0; --j) {
            if (j > i) continue;
            const float rj = 1.0f / sqrtf(kk[j * (j + 1) / 2 + j] + eps_unit);
            if (j < i) c[4 + j] = beta * between * ri * rj * kk[tri + j];
            c[4 + N + j] = between * si * rj * qk[tri + j];
            between *= g[j];
        }
        c[4 + N - 1] = before * after;
        float4* o = reinterpret_cast<float4*>(coef + ((size_t)(t + i) * dm.H + h) * NF);
#pragma unroll
        for (int x = 0; x < NF / 4; ++x)
            o[x] = make_float4(c[4 * x], c[4 * x + 1], c[4 * x + 2], c[4 * x + 3]);
    }
}

// --------------------------------------------------------------------- scan
__device__ __forceinline__ void cp_async_4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;"
                 :: "r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;"
                 :: "r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" :: "n"(N) : "memory"); }

struct HeadScanArgs {
    const float* u;            // [T, C]: q | k | v after the convolution
    const float* coef;         // [T, H, head_coefs(tokens a round)]
    float* out;                // [T, H * dv]
    float* state;              // [n_slots, stride]: S [H, dv, d] at 0
    long long stride;
    const int* slots;          // [B]; negative: padding entry
    const int* cu;             // [B + 1]
    int TCH;                   // tokens staged in shared memory at a time, a multiple of the round
    int vec;                   // rows of q and k move in 16-byte pieces
    int vec_v;                 // those of v
    int vec_s;                 // a column of S does
};

// One buffer: k and q [TCH, Dp], v [TCH, CP] (CC rounded up to 16 bytes), the coefficients.
__host__ __device__ constexpr int head_v_floats(int CC) { return (CC + 3) / 4 * 4; }
__host__ __device__ constexpr int head_buf_floats(int TCH, int Dp, int CC, int n) {
    return TCH * (2 * Dp + head_v_floats(CC) + head_coefs(n));
}

// grid (column groups, H, B).  A CTA has CC columns of one head of one sequence; L lanes hold
// NC neighbouring columns, R rows of each a lane (L * R >= d).  A lane's rows are R / 4 quads,
// quad i of lane l being rows (i L + l) 4 .. + 3: the lanes of a column read consecutive 16
// bytes of a token's row, the columns of a warp the same ones.  Tokens come TCH at a time
// through two buffers filled by asynchronous copies; rows beyond a chunk's last token are
// zeroed where a round reads them.
//
// A round's 2 N dot products of a column are summed over its lanes so that lane p of every N
// ends with those of token p (each exchange halves the sums a lane still carries), and, where
// there are more lanes, with those of some of the columns alone.  That lane forms token p's
// right-hand side, all lanes take all of them and solve for the writes, and the lane finishes
// its token's read-out.
template <int L, int R, int NC, int N>
__global__ void __launch_bounds__(128)
head_delta_scan_kernel(HeadScanArgs a, HeadDims dm) {
    pdl_wait();
    extern __shared__ __align__(16) float smem[];
    const int b = blockIdx.z;
    const int slot = a.slots[b];
    if (slot < 0) return;
    const int t0 = a.cu[b], n = a.cu[b + 1] - t0;
    if (n <= 0) return;
    const int h = blockIdx.y, grp = h / (dm.H / dm.G);
    const int d = dm.d, dv = dm.dv, C = dm.C(), nq = dm.nq();
    constexpr int Dp = L * R;
    const int CC = (int)blockDim.x / L * NC, TCH = a.TCH;
    const int l = threadIdx.x & (L - 1);
    const int jc = (int)(threadIdx.x / L) * NC;              // first of the lane's columns in the CTA
    const int j = blockIdx.x * CC + jc;
    constexpr int NF = head_coefs(N);
    const int per = head_buf_floats(TCH, Dp, CC, N), CP = head_v_floats(CC);
    // (padding rows of k and q and columns of v past dv are never copied: zero once)
    for (int i = threadIdx.x; i < 2 * per; i += blockDim.x) smem[i] = 0.f;
    __syncthreads();

    auto fetch = [&](int c0, float* base) {
        const int m = min(TCH, n - c0);
        float *sk = base, *sq = sk + TCH * Dp, *sv = sq + TCH * Dp, *sc = sv + TCH * CP;
        const float* row = a.u + (size_t)(t0 + c0) * C + (size_t)grp * d;
        if (a.vec) {
            const int Q = d / 4;
            for (int idx = threadIdx.x; idx < m * Q; idx += blockDim.x) {
                const int tt = idx / Q, c4 = (idx - tt * Q) * 4;
                const float* src = row + (size_t)tt * C + c4;
                cp_async_16(sq + tt * Dp + c4, src);
                cp_async_16(sk + tt * Dp + c4, src + nq);
            }
        } else {
            for (int idx = threadIdx.x; idx < m * d; idx += blockDim.x) {
                const int tt = idx / d, c = idx - tt * d;
                const float* src = row + (size_t)tt * C + c;
                cp_async_4(sq + tt * Dp + c, src);
                cp_async_4(sk + tt * Dp + c, src + nq);
            }
        }
        const float* vrow = a.u + (size_t)(t0 + c0) * C + 2 * nq + (size_t)h * dv + blockIdx.x * CC;
        const int vc = min(CC, dv - (int)blockIdx.x * CC);
        if (a.vec_v) {
            const int Q = vc / 4;
            for (int idx = threadIdx.x; idx < m * Q; idx += blockDim.x) {
                const int tt = idx / Q, c4 = (idx - tt * Q) * 4;
                cp_async_16(sv + tt * CP + c4, vrow + (size_t)tt * C + c4);
            }
        } else {
            for (int idx = threadIdx.x; idx < m * vc; idx += blockDim.x) {
                const int tt = idx / vc, c = idx - tt * vc;
                cp_async_4(sv + tt * CP + c, vrow + (size_t)tt * C + c);
            }
        }
        const float* crow = a.coef + ((size_t)(t0 + c0) * dm.H + h) * NF;
        for (int idx = threadIdx.x; idx < m * (NF / 4); idx += blockDim.x) {
            const int tt = idx / (NF / 4), c4 = (idx - tt * (NF / 4)) * 4;
            cp_async_16(sc + tt * NF + c4, crow + (size_t)tt * dm.H * NF + c4);
        }
        // places of the last round that no token takes: their k and their numbers are zero
        if (N > 1 && m % N != 0) {
            const int mm = (m + N - 1) / N * N - m;
            for (int idx = threadIdx.x; idx < mm * Dp; idx += blockDim.x) sk[m * Dp + idx] = 0.f;
            for (int idx = threadIdx.x; idx < mm * NF; idx += blockDim.x) sc[m * NF + idx] = 0.f;
        }
        cp_async_commit();
    };

    fetch(0, smem);
    // S as pairs of rows
    f32x2 S[NC][R / 2];
    float* srow = a.state + (size_t)slot * a.stride + ((size_t)h * dv + j) * d;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        const bool live = j + c < dv;
        const float* s = srow + (size_t)c * d;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int r = (i * L + l) * 4;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (live) {
                if (a.vec_s) {
                    if (r < d) x = *reinterpret_cast<const float4*>(s + r);
                } else {
                    if (r < d) x.x = s[r];
                    if (r + 1 < d) x.y = s[r + 1];
                    if (r + 2 < d) x.z = s[r + 2];
                    if (r + 3 < d) x.w = s[r + 3];
                }
            }
            S[c][2 * i] = pack2(x.x, x.y);
            S[c][2 * i + 1] = pack2(x.z, x.w);
        }
    }
    int cur = 0;
    for (int c0 = 0; c0 < n; c0 += TCH, cur ^= 1) {
        const int m = min(TCH, n - c0);
        const float* base = smem + (size_t)cur * per;
        const float *sk = base + l * 4, *sq = base + TCH * Dp + l * 4;
        const float *sv = base + 2 * TCH * Dp + jc, *sc = base + TCH * (2 * Dp + CP);
        // (the other buffer was read in the round before, which ended with a barrier)
        if (c0 + TCH < n) {
            fetch(c0 + TCH, smem + (size_t)(cur ^ 1) * per);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        for (int tt = 0; tt < m; tt += N) {
            // dot products of the state with the round's k and q
            f32x2 k2[N][R / 2];
            float ak[NC][N], aq[NC][N];
#pragma unroll
            for (int i = 0; i < N; ++i) {
                f32x2 ac[NC], rc[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) ac[c] = 0ull, rc[c] = 0ull;
#pragma unroll
                for (int x = 0; x < R / 4; ++x) {
                    const ulonglong2 kv = reinterpret_cast<const ulonglong2*>(sk + (tt + i) * Dp)[x * L];
                    const ulonglong2 qv = reinterpret_cast<const ulonglong2*>(sq + (tt + i) * Dp)[x * L];
                    k2[i][2 * x] = kv.x, k2[i][2 * x + 1] = kv.y;
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        ac[c] = fma2(S[c][2 * x], kv.x, ac[c]);
                        rc[c] = fma2(S[c][2 * x], qv.x, rc[c]);
                        ac[c] = fma2(S[c][2 * x + 1], kv.y, ac[c]);
                        rc[c] = fma2(S[c][2 * x + 1], qv.y, rc[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    float lo, hi;
                    unpack2(ac[c], lo, hi);
                    ak[c][i] = lo + hi;
                    unpack2(rc[c], lo, hi);
                    aq[c][i] = lo + hi;
                }
            }
            // the sums over a column's lanes, the round's writes, and its read-outs
            float w[NC][N];
            const float* cf = sc + tt * NF;                  // numbers of the round
            if constexpr (L >= N && N > 1) {
                auto fold = [&](float& keep, float& give, bool up, int bit) {
                    const float out = up ? keep : give, in = up ? give : keep;
                    keep = in + __shfl_xor_sync(0xffffffffu, out, bit);
                };
#pragma unroll
                for (int half = N / 2; half >= 1; half >>= 1)
#pragma unroll
                    for (int i = 0; i < half; ++i)
#pragma unroll
                        for (int c = 0; c < NC; ++c) {
                            fold(ak[c][i], ak[c][i + half], l & half, half);
                            fold(aq[c][i], aq[c][i + half], l & half, half);
                        }
                // lanes beyond N: each takes some of the columns, the rest of them sum
                constexpr int XB = L / N, OWN = NC >= XB ? NC / XB : 1;      // columns a lane ends with
                int own = 0;                                                 // first of them
#pragma unroll
                for (int o = N, half = NC / 2; o < L; o <<= 1, half >>= 1) {
                    if (half >= 1) {
                        const bool up = l & o;
                        if (up) own += half;
#pragma unroll
                        for (int c = 0; c < half; ++c) {
                            fold(ak[c][0], ak[c + half][0], up, o);
                            fold(aq[c][0], aq[c + half][0], up, o);
                        }
                    } else {
#pragma unroll
                        for (int c = 0; c < OWN; ++c) {
                            ak[c][0] += __shfl_xor_sync(0xffffffffu, ak[c][0], o);
                            aq[c][0] += __shfl_xor_sync(0xffffffffu, aq[c][0], o);
                        }
                    }
                }
                const int p = l & (N - 1), base = (threadIdx.x & 31) & ~(L - 1);
                const float* mine = cf + p * NF;
                const float4 m0 = *reinterpret_cast<const float4*>(mine);
                float P[N];
#pragma unroll
                for (int x = 0; x < N / 4; ++x)
                    *reinterpret_cast<float4*>(P + 4 * x) =
                        reinterpret_cast<const float4*>(mine + 4 + N)[x];
                float rhs[OWN];
#pragma unroll
                for (int c = 0; c < OWN; ++c)
                    rhs[c] = fmaf(-m0.y, ak[c][0], m0.x * sv[(tt + p) * CP + own + c]);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    // the lanes that ended with column c: bit N of the lane is the upper half
                    int who = 0;
#pragma unroll
                    for (int o = N, half = NC / 2; o < L && half >= 1; o <<= 1, half >>= 1)
                        if (c & half) who |= o;
#pragma unroll
                    for (int i = 0; i < N; ++i)
                        w[c][i] = __shfl_sync(0xffffffffu, rhs[c & (OWN - 1)], base | who | i);
                }
#pragma unroll
                for (int i = 1; i < N; ++i) {
                    float A[N];
#pragma unroll
                    for (int x = 0; x < (i + 3) / 4; ++x)
                        *reinterpret_cast<float4*>(A + 4 * x) =
                            reinterpret_cast<const float4*>(cf + i * NF + 4)[x];
#pragma unroll
                    for (int jj = 0; jj < i; ++jj)
#pragma unroll
                        for (int c = 0; c < NC; ++c) w[c][i] = fmaf(-A[jj], w[c][jj], w[c][i]);
                }
#pragma unroll
                for (int c = 0; c < OWN; ++c) {
                    float o = m0.z * aq[c][0];
#pragma unroll
                    for (int jj = 0; jj < N; ++jj) {
                        float u = w[c][jj];                  // (of column own + c)
#pragma unroll
                        for (int e = 1; e < NC / OWN; ++e)
                            if (own == e * OWN) u = w[e * OWN + c][jj];
                        o = fmaf(P[jj], u, o);
                    }
                    constexpr int TOP = NC >= XB ? L : N * NC;               // lanes that write
                    if (l < TOP && tt + p < m && j + own + c < dv)
                        a.out[((size_t)(t0 + c0 + tt + p) * dm.H + h) * dv + j + own + c] = o;
                }
            } else {
#pragma unroll
                for (int o = 1; o < L; o <<= 1)
#pragma unroll
                    for (int i = 0; i < N; ++i)
#pragma unroll
                        for (int c = 0; c < NC; ++c) {
                            ak[c][i] += __shfl_xor_sync(0xffffffffu, ak[c][i], o);
                            aq[c][i] += __shfl_xor_sync(0xffffffffu, aq[c][i], o);
                        }
#pragma unroll
                for (int i = 0; i < N; ++i)
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const float* mine = cf + i * NF;
                        float u = fmaf(-mine[1], ak[c][i], mine[0] * sv[(tt + i) * CP + c]);
#pragma unroll
                        for (int jj = 0; jj < i; ++jj) u = fmaf(-mine[4 + jj], w[c][jj], u);
                        w[c][i] = u;
                        float o = mine[2] * aq[c][i];
#pragma unroll
                        for (int jj = 0; jj <= i; ++jj) o = fmaf(mine[4 + N + jj], w[c][jj], o);
                        if ((i & (L - 1)) == l && tt + i < m && j + c < dv)
                            a.out[((size_t)(t0 + c0 + tt + i) * dm.H + h) * dv + j + c] = o;
                    }
            }
            const float total = cf[4 + N - 1];
            const f32x2 g2 = pack2(total, total);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
#pragma unroll
                for (int x = 0; x < R / 2; ++x) S[c][x] = mul2(S[c][x], g2);
#pragma unroll
                for (int i = 0; i < N; ++i) {
                    const float wu = cf[i * NF + 3] * w[c][i];
                    const f32x2 u2 = pack2(wu, wu);
#pragma unroll
                    for (int x = 0; x < R / 2; ++x) S[c][x] = fma2(k2[i][x], u2, S[c][x]);
                }
            }
        }
        __syncthreads();
    }
    pdl_launch_next();
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        if (j + c >= dv) continue;
        float* s = srow + (size_t)c * d;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int r = (i * L + l) * 4;
            float4 x;
            unpack2(S[c][2 * i], x.x, x.y);
            unpack2(S[c][2 * i + 1], x.z, x.w);
            if (a.vec_s) {
                if (r < d) *reinterpret_cast<float4*>(s + r) = x;
            } else {
                if (r < d) s[r] = x.x;
                if (r + 1 < d) s[r + 1] = x.y;
                if (r + 2 < d) s[r + 2] = x.z;
                if (r + 3 < d) s[r + 3] = x.w;
            }
        }
    }
}

// ---------------------------------------------------------------- read-out
// y[t, h, :] = o[t, h, :] / rms(o[t, h, :]) * w * act(gate[t, h, :]): a CTA a token, a warp a
// head at a time, V values a lane; the gate is columns g_off .. of the stacked projection.
template <typename T, int V>
__global__ void __launch_bounds__(1024)
head_delta_out_kernel(const float* __restrict__ o, RowIn<float> in, int g_off,
                      const float* __restrict__ w, float eps, int H, int dv, int silu,
                      const int* __restrict__ seq_index, const int* __restrict__ slots,
                      T* __restrict__ y) {
    pdl_wait();
    pdl_launch_next();
    const int t = blockIdx.x;
    const bool pad = slots[seq_index[t]] < 0;      // a padding entry's row is zeros
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (int h = warp; h < H; h += nwarps) {
        const size_t base = ((size_t)t * H + h) * dv;
        if (pad) {
            for (int i = lane; i < dv; i += 32) y[base + i] = from_f32<T>(0.f);
            continue;
        }
        // the gate's loads go out before the reduction over the head
        constexpr int KEEP = V == 4 ? 2 : 4;                 // values a lane keeps: dv <= 32 V KEEP
        float ss = 0.f, ov[KEEP][V], gv[KEEP][V];
#pragma unroll
        for (int p = 0; p < KEEP; ++p) {
            const int i = (p * 32 + lane) * V;
#pragma unroll
            for (int x = 0; x < V; ++x) ov[p][x] = 0.f, gv[p][x] = 0.f;
            if (i < dv) {
                const int c = g_off + h * dv + i;
                if constexpr (V == 4) {
                    const float4 q = *reinterpret_cast<const float4*>(o + base + i);
                    ov[p][0] = q.x, ov[p][1] = q.y, ov[p][2] = q.z, ov[p][3] = q.w;
                    const float* src = in.part ? in.part + (size_t)t * in.W + c
                                               : in.row + (size_t)t * in.ld + c;
                    float4 g = *reinterpret_cast<const float4*>(src);
                    if (in.part)
                        for (int s = 1; s < in.n_splits; ++s) {
                            const float4 e = *reinterpret_cast<const float4*>(
                                src + (size_t)s * in.split_stride);
                            g.x += e.x, g.y += e.y, g.z += e.z, g.w += e.w;
                        }
                    gv[p][0] = g.x, gv[p][1] = g.y, gv[p][2] = g.z, gv[p][3] = g.w;
                } else {
                    ov[p][0] = o[base + i];
                    gv[p][0] = in.at(t, c);
                }
#pragma unroll
                for (int x = 0; x < V; ++x) ss = fmaf(ov[p][x], ov[p][x], ss);
            }
        }
        for (int i = KEEP * 32 * V + lane; i < dv; i += 32) ss = fmaf(o[base + i], o[base + i], ss);
        ss = warp_sum(ss);
        const float r = 1.0f / sqrtf(ss / (float)dv + eps);
#pragma unroll
        for (int p = 0; p < KEEP; ++p) {
            const int i = (p * 32 + lane) * V;
            if (i < dv) {
                T out[V];
#pragma unroll
                for (int x = 0; x < V; ++x)
                    out[x] = from_f32<T>(ov[p][x] * r * w[i + x] *
                                         (silu ? silu_f(gv[p][x]) : sigmoid_f(gv[p][x])));
                if constexpr (V == 4 && sizeof(T) == 2)
                    *reinterpret_cast<uint2*>(y + base + i) = *reinterpret_cast<const uint2*>(out);
                else if constexpr (V == 4)
                    *reinterpret_cast<float4*>(y + base + i) = *reinterpret_cast<const float4*>(out);
                else
                    y[base + i] = out[0];
            }
        }
        for (int i = KEEP * 32 * V + lane; i < dv; i += 32) {
            const float g = in.at(t, g_off + h * dv + i);
            y[base + i] = from_f32<T>(o[base + i] * r * w[i] * (silu ? silu_f(g) : sigmoid_f(g)));
        }
    }
}

int check_head_dims(const HeadDims& dm) {
    AGV_REQUIRE(dm.G > 0 && dm.H > 0 && dm.d > 0 && dm.dv > 0, "head_delta: bad sizes");
    AGV_REQUIRE(dm.H % dm.G == 0, "head_delta: %d heads are not a multiple of %d query/key heads",
                dm.H, dm.G);
    AGV_REQUIRE(dm.d <= DH_MAX_D, "head_delta: key heads of %d exceed %d", dm.d, DH_MAX_D);
    return 0;
}

int head_row(RowIn<float>& in, const float* row, long long ld, const float* part, int n_splits,
             int T, int W) {
    AGV_REQUIRE((row != nullptr) != (part != nullptr), "head_delta: rows or partial sums, one of them");
    AGV_REQUIRE(!row || ld >= W, "head_delta: row stride shorter than a row");
    AGV_REQUIRE(!part || n_splits >= 1, "head_delta: no partial sums");
    in = RowIn<float>{row, ld, part, n_splits, (long long)T * W, W};
    return 0;
}

template <int L, int R, int NC, int N>
int launch_head_scan(HeadScanArgs a, const HeadDims& dm, int B, cudaStream_t stream) {
    // 128 threads a CTA where the columns allow, whole warps always
    int threads = 128;
    while (threads > 32 && threads / 2 / L * NC >= dm.dv) threads >>= 1;
    const int CC = threads / L * NC;
    a.TCH = N > 1 ? 16 : 1;
    while (a.TCH > N && 2 * head_buf_floats(a.TCH, L * R, CC, N) * sizeof(float) > 48 * 1024)
        a.TCH >>= 1;
    const size_t smem = 2 * (size_t)head_buf_floats(a.TCH, L * R, CC, N) * sizeof(float);
    a.vec_v = a.vec_v && CC % 4 == 0;
    auto kern = head_delta_scan_kernel<L, R, NC, N>;
    if (smem > 48 * 1024) {
        static bool configured = false;
        if (!configured) {
            AGV_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             100 * 1024));
            configured = true;
        }
        AGV_REQUIRE(smem <= 100 * 1024, "head_delta_scan: %d bytes of shared memory", (int)smem);
    }
    // (few CTAs, each a long dependent chain: spread over the SMs)
    agv_launch_after(kern, dim3((unsigned)((dm.dv + CC - 1) / CC), (unsigned)dm.H, (unsigned)B),
                     (unsigned)threads, smem, stream, a, dm);
    AGV_LAUNCH_OK("head_delta_scan_kernel");
    return 0;
}

}  // namespace

// Numbers a token and head (see delta_coef_kernel).
AGV_API int agv_head_delta_coefs(int several, int d) { return head_coefs(several ? head_round(d) : 1); }

// u: [T, 2 G d + H dv] 32-bit, q | k | v after the convolution; decay: [T, H, 2] 32-bit, the
// decay first; row / part: the stacked projection [T, W] 32-bit (row stride ld) or [n_splits, T,
// W] partial sums, whose columns b_off .. b_off + H are beta's logits.  several != 0: sequences
// may bring more than one token.  coef: [T, H, agv_head_delta_coefs(several, d)].
AGV_API int agv_head_delta_coef(const float* u, const float* decay, const float* row, long long ld,
                                const float* part, int n_splits, int T, int W, int b_off, int B,
                                int G, int H, int d, int dv, float eps_unit, float q_mult,
                                int several, const int* cu, float* coef, cudaStream_t stream) {
    const HeadDims dm{G, H, d, dv};
    if (int rc = check_head_dims(dm)) return rc;
    AGV_REQUIRE(T >= 0 && B >= 1 && b_off >= 0 && b_off + H <= W, "head_delta_coef: bad sizes");
    AGV_REQUIRE(agv_aligned(coef, 16), "head_delta_coef: the output must be 16-byte aligned");
    if (T == 0) return 0;
    RowIn<float> in;
    if (int rc = head_row(in, row, ld, part, n_splits, T, W)) return rc;
#define AGV_HC(N)                                                                                \
    agv_launch(delta_coef_kernel<N>,                                                            \
               (unsigned)(((long long)(T / N + B) * G + DH_COEF_WARPS - 1) / DH_COEF_WARPS),     \
               DH_COEF_WARPS * 32, 0, stream, u, decay, in, b_off, dm, T, B, eps_unit, q_mult,   \
               cu, coef)
    if (!several) AGV_HC(1);
    else if (head_round(d) == 8) AGV_HC(8);
    else AGV_HC(4);
#undef AGV_HC
    AGV_LAUNCH_OK("delta_coef_kernel");
    return 0;
}

// The recurrence over the step's tokens, sequence by sequence; u and coef as above (coef made
// with the same `several`), out [T, H * dv] 32-bit, state: S [H, dv, d] per slot at 0.
AGV_API int agv_head_delta_scan(const float* u, const float* coef, float* out, int T, int B, int G,
                                int H, int d, int dv, int several, float* state,
                                long long state_stride, const int* slots, const int* cu,
                                cudaStream_t stream) {
    const HeadDims dm{G, H, d, dv};
    if (int rc = check_head_dims(dm)) return rc;
    AGV_REQUIRE(state && state_stride >= (long long)H * dv * d,
                "head_delta_scan: the state is too small");
    AGV_REQUIRE(B <= 65535 && H <= 65535, "head_delta_scan: batch or head count exceeds the grid limit");
    AGV_REQUIRE(agv_aligned(coef, 16), "head_delta_scan: the coefficients must be 16-byte aligned");
    if (T == 0 || B == 0) return 0;
    const int C = dm.C();
    HeadScanArgs a{u, coef, out, state, state_stride, slots, cu, 0, 0, 0, 0};
    a.vec = d % 4 == 0 && C % 4 == 0 && agv_aligned(u, 16);
    a.vec_v = dv % 4 == 0 && C % 4 == 0 && (2 * dm.nq()) % 4 == 0 && agv_aligned(u, 16);
    a.vec_s = d % 4 == 0 && state_stride % 4 == 0 && agv_aligned(state, 16);
#define AGV_HS(L, R, NC, N) return launch_head_scan<L, R, NC, N>(a, dm, B, stream)
    if (!several) {
        if (d <= 16) AGV_HS(1, 16, 1, 1);
        if (d <= 32) AGV_HS(2, 16, 1, 1);
        if (d <= 64) AGV_HS(4, 16, 1, 1);
        if (d <= 128) AGV_HS(8, 16, 1, 1);
        if (d <= 256) AGV_HS(16, 16, 1, 1);
        AGV_HS(32, 16, 1, 1);
    }
    if (d <= 16) AGV_HS(1, 16, 1, 4);
    if (d <= 32) AGV_HS(4, 8, 1, 4);
    // (more columns a lane, and so fewer reads of k and q a column, where the launch has more
    // CTAs than the SMs can take at once anyway)
    if (d <= 64) {
        if ((long long)B * H * ((dv + 7) / 8) > 296) AGV_HS(16, 4, 2, 8);
        AGV_HS(16, 4, 1, 8);
    }
    if (d <= 128) {
        if ((long long)B * H * ((dv + 15) / 16) > 192) AGV_HS(16, 8, 4, 8);
        AGV_HS(16, 8, 2, 8);
    }
    if (d <= 256) AGV_HS(32, 8, 4, 8);
    AGV_HS(32, 16, 1, 8);
#undef AGV_HS
}

// o: [T, H * dv] 32-bit; the gate: columns g_off .. g_off + H dv of the stacked projection (row /
// part as above); silu != 0: times silu(gate), else sigmoid(gate); w: [dv] 32-bit; y: [T, H * dv]
// in dtype.
AGV_API int agv_head_delta_out(const float* o, const float* row, long long ld, const float* part,
                               int n_splits, int T, int W, int g_off, const float* w, float eps,
                               int H, int dv, int silu, const int* seq_index, const int* slots,
                               void* y, int dtype, cudaStream_t stream) {
    AGV_REQUIRE(T >= 0 && H > 0 && dv > 0 && g_off >= 0 && g_off + H * dv <= W,
                "head_delta_out: bad sizes");
    if (T == 0) return 0;
    RowIn<float> in;
    if (int rc = head_row(in, row, ld, part, n_splits, T, W)) return rc;
    const bool vec = dv % 4 == 0 && g_off % 4 == 0 && agv_aligned(o, 16) && agv_aligned(y, 16) &&
                     (part ? W % 4 == 0 && agv_aligned(part, 16) : ld % 4 == 0 && agv_aligned(row, 16));
    // (few rows: a warp a head at once; many: several rows to an SM)
    const int most = T <= 296 ? 1024 : 256;
    int threads = 32;
    while (threads < most && threads < 32 * H) threads *= 2;
#define AGV_HO(TT, V)                                                                            \
    agv_launch(head_delta_out_kernel<TT, V>, (unsigned)T, threads, 0, stream, o, in, g_off, w, eps, \
               H, dv, silu, seq_index, slots, (TT*)y)
    if (dtype == AGV_F32) { if (vec) AGV_HO(float, 4); else AGV_HO(float, 1); }
    else if (dtype == AGV_BF16) { if (vec) AGV_HO(__nv_bfloat16, 4); else AGV_HO(__nv_bfloat16, 1); }
    else return agv_fail(-1, "head_delta_out: unknown dtype %d", dtype);
#undef AGV_HO
    AGV_LAUNCH_OK("head_delta_out_kernel");
    return 0;
}
