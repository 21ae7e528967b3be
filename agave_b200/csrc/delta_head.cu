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
// folded into twelve numbers a token and head) is made by a launch before for all rounds at
// once; the vectors themselves stay as the convolution left them.  A round begins at the first
// token a sequence brings in the step; a decode step's rounds are one token.
//
// 32-bit throughout.  A prompt and a decoded token differ in the order of these sums alone.
#include "common.cuh"
#include "row_in.cuh"

namespace {

constexpr int DH_R = 16;           // rows of a column a lane holds
constexpr int DH_ROUND = 4;        // tokens a round of a prompt
constexpr int DH_COEF = 12;        // numbers a token and head

struct HeadDims {
    int G, H, d, dv;
    __host__ __device__ int nq() const { return G * d; }
    __host__ __device__ int C() const { return 2 * G * d + H * dv; }
};

__device__ __forceinline__ float silu_f(float t) { return t / (1.0f + expf(-t)); }
__device__ __forceinline__ float sigmoid_f(float t) { return 1.0f / (1.0f + expf(-t)); }

// ------------------------------------------------------------- coefficients
// A warp per (token, query/key head); the first token of a round works for the whole round.
// Layout of a token's numbers (i its place in the round, n the round's last place):
//   0 beta   1 beta G_i0 r_i   2..4 beta G_ij r_i r_j (k_i . k_j), j = 0..2
//   5 G_i0 s_i   6..9 G_ij s_i r_j (q_i . k_j), j = 0..3   10 G_nj r_j with j = i   11 G_n0
// (zeros where j >= i, or j > i).
template <int N>
__global__ void __launch_bounds__(256)
delta_coef_kernel(const float* __restrict__ u, const float* __restrict__ decay, RowIn<float> in,
                  int b_off, HeadDims dm, int n_tokens, float eps_unit, float q_mult,
                  const int* __restrict__ seq_index, const int* __restrict__ cu,
                  float* __restrict__ coef) {
    pdl_wait();
    pdl_launch_next();
    const int lane = threadIdx.x & 31;
    const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (w >= (long long)n_tokens * dm.G) return;
    const int t = (int)(w / dm.G), grp = (int)(w - (long long)t * dm.G);
    const int b = seq_index[t], first = cu[b], end = cu[b + 1];
    if (N > 1 && (t - first) % N != 0) return;
    const int m = min(N, end - t);
    const int C = dm.C(), d = dm.d;
    const float* q0 = u + (size_t)t * C + (size_t)grp * d;
    const float* k0 = q0 + dm.nq();
    float qq[N] = {}, kk[N][N] = {}, qk[N][N] = {};
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
            qq[i] = fmaf(q[i], q[i], qq[i]);
#pragma unroll
            for (int j = 0; j <= i; ++j) {
                kk[i][j] = fmaf(k[i], k[j], kk[i][j]);
                qk[i][j] = fmaf(q[i], k[j], qk[i][j]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
        qq[i] = warp_sum(qq[i]);
#pragma unroll
        for (int j = 0; j <= i; ++j) {
            kk[i][j] = warp_sum(kk[i][j]);
            qk[i][j] = warp_sum(qk[i][j]);
        }
    }
    float rk[N], rq[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
        rk[i] = 1.0f / sqrtf(kk[i][i] + eps_unit);
        rq[i] = q_mult / sqrtf(qq[i] + eps_unit);
    }
    const int per = dm.H / dm.G;
    for (int hh = lane; hh < per; hh += 32) {
        const int h = grp * per + hh;
        float g[N];
#pragma unroll
        for (int i = 0; i < N; ++i)
            g[i] = i < m ? decay[((size_t)(t + i) * dm.H + h) * 2] : 1.f;
        float total = 1.f;
#pragma unroll
        for (int i = 0; i < N; ++i) total *= g[i];
        float from_start = 1.f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (i >= m) break;
            from_start *= g[i];
            const float beta = sigmoid_f(in.at(t + i, b_off + h));
            float c[DH_COEF] = {};
            c[0] = beta;
            c[1] = beta * from_start * rk[i];
            c[5] = from_start * rq[i];
            float between = 1.f;                             // g_(j+1) .. g_i
#pragma unroll
            for (int j = i; j >= 0; --j) {
                if (j < i) c[2 + j] = beta * between * rk[i] * rk[j] * kk[i][j];
                c[6 + j] = between * rq[i] * rk[j] * qk[i][j];
                between *= g[j];
            }
            float after = 1.f;                               // g_(i+1) .. g_n
#pragma unroll
            for (int j = i + 1; j < N; ++j) after *= g[j];
            c[10] = after * rk[i];
            c[11] = total;
            float4* o = reinterpret_cast<float4*>(coef + ((size_t)(t + i) * dm.H + h) * DH_COEF);
            o[0] = make_float4(c[0], c[1], c[2], c[3]);
            o[1] = make_float4(c[4], c[5], c[6], c[7]);
            o[2] = make_float4(c[8], c[9], c[10], c[11]);
        }
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
    const float* coef;         // [T, H, 12]
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

// One buffer: k and q [TCH, Dp], v [TCH, CP] (CC rounded up to 16 bytes), coefficients [TCH, 12].
__host__ __device__ constexpr int head_v_floats(int CC) { return (CC + 3) / 4 * 4; }
__host__ __device__ constexpr int head_buf_floats(int TCH, int Dp, int CC) {
    return TCH * (2 * Dp + head_v_floats(CC) + DH_COEF);
}

// grid (column groups, H, B).  A CTA has CC columns of one head of one sequence; L lanes hold
// NC neighbouring columns, 16 rows of each a lane (L * 16 >= d).  A lane's rows are four quads,
// quad i of lane l being rows (i L + l) 4 .. + 3: the lanes of a column read consecutive 16
// bytes of a token's row, the columns of a warp the same ones.  Tokens come TCH at a time
// through two buffers filled by asynchronous copies; rows beyond a chunk's last token are
// zeroed where a round reads them.
template <int L, int NC, int N>
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
    constexpr int Dp = L * DH_R;
    const int CC = (int)blockDim.x / L * NC, TCH = a.TCH;
    const int l = threadIdx.x & (L - 1);
    const int jc = (int)(threadIdx.x / L) * NC;              // first of the lane's columns in the CTA
    const int j = blockIdx.x * CC + jc;
    const int per = head_buf_floats(TCH, Dp, CC), CP = head_v_floats(CC);
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
        const float* crow = a.coef + ((size_t)(t0 + c0) * dm.H + h) * DH_COEF;
        for (int idx = threadIdx.x; idx < m * (DH_COEF / 4); idx += blockDim.x) {
            const int tt = idx / (DH_COEF / 4), c4 = (idx - tt * (DH_COEF / 4)) * 4;
            cp_async_16(sc + tt * DH_COEF + c4, crow + (size_t)tt * dm.H * DH_COEF + c4);
        }
        // places of the last round that no token takes: their k and their numbers are zero
        if (N > 1 && m % N != 0) {
            const int mm = (m + N - 1) / N * N - m;
            for (int idx = threadIdx.x; idx < mm * Dp; idx += blockDim.x) sk[m * Dp + idx] = 0.f;
            for (int idx = threadIdx.x; idx < mm * DH_COEF; idx += blockDim.x)
                sc[m * DH_COEF + idx] = 0.f;
        }
        cp_async_commit();
    };

    fetch(0, smem);
    // S as pairs of rows
    f32x2 S[NC][DH_R / 2];
    float* srow = a.state + (size_t)slot * a.stride + ((size_t)h * dv + j) * d;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        const bool live = j + c < dv;
        const float* s = srow + (size_t)c * d;
#pragma unroll
        for (int i = 0; i < DH_R / 4; ++i) {
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
            f32x2 k2[N][DH_R / 2];
            float ak[NC][N], aq[NC][N];
#pragma unroll
            for (int i = 0; i < N; ++i) {
                f32x2 ac[NC], rc[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) ac[c] = 0ull, rc[c] = 0ull;
#pragma unroll
                for (int x = 0; x < DH_R / 4; ++x) {
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
#pragma unroll
            for (int o = 1; o < L; o <<= 1)
#pragma unroll
                for (int i = 0; i < N; ++i)
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        ak[c][i] += __shfl_xor_sync(0xffffffffu, ak[c][i], o);
                        aq[c][i] += __shfl_xor_sync(0xffffffffu, aq[c][i], o);
                    }
            // the round's writes one after another, and its read-outs
            float w[NC][N];
            float total = 1.f;
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const float4* cf = reinterpret_cast<const float4*>(sc + (tt + i) * DH_COEF);
                const float4 c0v = cf[0], c1v = cf[1], c2v = cf[2];
                const float A[3] = {c0v.z, c0v.w, c1v.x};
                const float P[4] = {c1v.z, c1v.w, c2v.x, c2v.y};
                if (i == 0) total = c2v.w;
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    float u = fmaf(-c0v.y, ak[c][i], c0v.x * sv[(tt + i) * CP + c]);
#pragma unroll
                    for (int jj = 0; jj < 3; ++jj)
                        if (jj < i) u = fmaf(-A[jj], w[c][jj], u);
                    w[c][i] = u;
                    float o = c1v.y * aq[c][i];
#pragma unroll
                    for (int jj = 0; jj < 4; ++jj)
                        if (jj <= i) o = fmaf(P[jj], w[c][jj], o);
                    if ((i & (L - 1)) == l && tt + i < m && j + c < dv)
                        a.out[((size_t)(t0 + c0 + tt + i) * dm.H + h) * dv + j + c] = o;
                }
            }
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const f32x2 g2 = pack2(total, total);
#pragma unroll
                for (int x = 0; x < DH_R / 2; ++x) S[c][x] = mul2(S[c][x], g2);
#pragma unroll
                for (int i = 0; i < N; ++i) {
                    const float wu = sc[(tt + i) * DH_COEF + 10] * w[c][i];
                    const f32x2 u2 = pack2(wu, wu);
#pragma unroll
                    for (int x = 0; x < DH_R / 2; ++x) S[c][x] = fma2(k2[i][x], u2, S[c][x]);
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
        for (int i = 0; i < DH_R / 4; ++i) {
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
    AGV_REQUIRE(dm.d <= 32 * DH_R, "head_delta: key heads of %d exceed %d", dm.d, 32 * DH_R);
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

template <int L, int NC, int N>
int launch_head_scan(const HeadScanArgs& a, const HeadDims& dm, int B, int threads, size_t smem,
                     cudaStream_t stream) {
    const int CC = threads / L * NC;
    // (few CTAs, each a long dependent chain: spread over the SMs)
    agv_launch_after(head_delta_scan_kernel<L, NC, N>,
                     dim3((unsigned)((dm.dv + CC - 1) / CC), (unsigned)dm.H, (unsigned)B),
                     (unsigned)threads, smem, stream, a, dm);
    AGV_LAUNCH_OK("head_delta_scan_kernel");
    return 0;
}

}  // namespace

AGV_API int agv_head_delta_coef_numel() { return DH_COEF; }

// u: [T, 2 G d + H dv] 32-bit, q | k | v after the convolution; decay: [T, H, 2] 32-bit, the
// decay first; row / part: the stacked projection [T, W] 32-bit (row stride ld) or [n_splits, T,
// W] partial sums, whose columns b_off .. b_off + H are beta's logits.  several != 0: sequences
// may bring more than one token.  coef: [T, H, 12].
AGV_API int agv_head_delta_coef(const float* u, const float* decay, const float* row, long long ld,
                                const float* part, int n_splits, int T, int W, int b_off, int G,
                                int H, int d, int dv, float eps_unit, float q_mult, int several,
                                const int* seq_index, const int* cu, float* coef,
                                cudaStream_t stream) {
    const HeadDims dm{G, H, d, dv};
    if (int rc = check_head_dims(dm)) return rc;
    AGV_REQUIRE(T >= 0 && b_off >= 0 && b_off + H <= W, "head_delta_coef: bad sizes");
    AGV_REQUIRE(agv_aligned(coef, 16), "head_delta_coef: the output must be 16-byte aligned");
    if (T == 0) return 0;
    RowIn<float> in;
    if (int rc = head_row(in, row, ld, part, n_splits, T, W)) return rc;
    const unsigned grid = (unsigned)(((long long)T * G + 7) / 8);
    if (several)
        agv_launch(delta_coef_kernel<DH_ROUND>, grid, 256, 0, stream, u, decay, in, b_off, dm, T,
                   eps_unit, q_mult, seq_index, cu, coef);
    else
        agv_launch(delta_coef_kernel<1>, grid, 256, 0, stream, u, decay, in, b_off, dm, T, eps_unit,
                   q_mult, seq_index, cu, coef);
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
    int L = 1;
    while (L * DH_R < d) L <<= 1;
    // two columns a lane where the launch still fills the GPU, 128 threads a CTA where the
    // columns allow, whole warps always
    const long long lanes = (long long)B * H * dv * L;
    const int NC = several && L > 1 && lanes >= 148LL * 4 * 32 ? 2 : 1;
    int threads = 128;
    while (threads > 32 && threads / 2 / L * NC >= dv) threads >>= 1;
    const int CC = threads / L * NC, Dp = L * DH_R;
    int TCH = several ? 16 : 1;
    while (TCH > DH_ROUND && 2 * head_buf_floats(TCH, Dp, CC) * sizeof(float) > 48 * 1024) TCH >>= 1;
    const size_t smem = 2 * (size_t)head_buf_floats(TCH, Dp, CC) * sizeof(float);
    AGV_REQUIRE(smem <= 48 * 1024, "head_delta_scan: key heads of %d need too much shared memory", d);
    const int C = dm.C();
    HeadScanArgs a{u, coef, out, state, state_stride, slots, cu, TCH, 0, 0, 0};
    a.vec = d % 4 == 0 && C % 4 == 0 && agv_aligned(u, 16);
    a.vec_v = dv % 4 == 0 && CC % 4 == 0 && C % 4 == 0 && (2 * dm.nq()) % 4 == 0 && agv_aligned(u, 16);
    a.vec_s = d % 4 == 0 && state_stride % 4 == 0 && agv_aligned(state, 16);
#define AGV_HS(LL)                                                                              \
    case LL:                                                                                    \
        if (!several) return launch_head_scan<LL, 1, 1>(a, dm, B, threads, smem, stream);       \
        if (NC == 2) return launch_head_scan<LL, 2, DH_ROUND>(a, dm, B, threads, smem, stream); \
        return launch_head_scan<LL, 1, DH_ROUND>(a, dm, B, threads, smem, stream)
    switch (L) {
        AGV_HS(1); AGV_HS(2); AGV_HS(4); AGV_HS(8); AGV_HS(16); AGV_HS(32);
    }
#undef AGV_HS
    return agv_fail(-1, "head_delta_scan: %d lanes a column", L);
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
