// Kernels of two state-space mixers, and the convolution that both begin with.
//
//  * agv_ssm_conv: from a token's row of the stacked input projection (32-bit, or 32-bit partial
//    sums over ranges of K), channels off .. off + C: a causal convolution over time, channel by
//    channel (``taps`` weights a channel, the last one the current token's; zeros before the
//    start of a sequence), a bias (or none) and silu.  The convolution's inputs of earlier steps are part
//    of the sequence's fixed-size state: a ring by position (position p in row p % (taps - 1)).
//    Beside them, columns dt_off .. + n_dt may hold one step size per head: dt = softplus(dt +
//    bias), which leaves as the pair (exp(neg_a dt), dt) a scan with one decay per head wants.
//  * agv_selective_low: the second projection's row  r | B | C : r rounded to the compute dtype
//    for its product, B and C padded for the scan's 16-byte copies.
//  * agv_selective_scan: a decay per channel and state,
//        S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n;   y_c = sum_n S[c, n] C_n + D_c u_c
//    over the step's tokens, sequence by sequence, then y * silu(z), rounded for the output
//    product.  dt_c = softplus(dt_c + bias_c).
//  * agv_ssd_out: what follows the scan with one decay per head (the matrix-state scan of
//    mlstm.cu without its normaliser): (y + D_h u) * silu(z), divided in equal parts by each
//    part's root mean square, times a weight per channel.
//
// 32-bit throughout: sums over partial products, convolution, silu, softplus, decays, states.
// Prompts and decoded tokens run the same kernels.
#include "common.cuh"
#include "row_in.cuh"

namespace {

__device__ __forceinline__ float silu_f(float t) { return t / (1.0f + expf(-t)); }
__device__ __forceinline__ float softplus_f(float t) { return t > 20.0f ? t : log1pf(expf(t)); }

// 2^x by the hardware approximation (relative error about 2^-22; below 2^-126 it gives 0).
__device__ __forceinline__ float ex2_ftz(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct StepArgs {
    float* state;              // [n_slots, stride]
    long long stride, off;     // off: where this kernel's part of the state starts
    const int* slots;          // [B]; negative: padding entry
    const int* cu;             // [B + 1] first token of each entry
    const int* seq_index;      // [T]
    const int* positions;      // [T]
    const int* lens;           // [B] lengths after the step
};

// ------------------------------------------------------------- convolution
// A thread has one channel and R consecutive tokens, whose inputs slide through registers.
// (A step's sequences start at position 0 or bring one token: the thread that overwrites a
// ring row is the one that read it.)
template <typename T, int TAPS, int R>
__global__ void __launch_bounds__(128)
ssm_conv_kernel(RowIn<float> in, int n_tokens, int off, int C, StepArgs st,
                const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out,
                T* __restrict__ rounded, int dt_off, int n_dt, const float* __restrict__ dt_bias,
                const float* __restrict__ neg_a, float* __restrict__ coef) {
    pdl_wait();
    pdl_launch_next();
    constexpr int RING = TAPS - 1, MOD = RING > 0 ? RING : 1;
    // what the tile's tokens are: position, tokens of the sequence in this step before it, slot,
    // and whether the token is among the sequence's last inputs
    __shared__ int s_pos[R], s_in[R], s_slot[R], s_keep[R];
    const int c = blockIdx.x * 128 + threadIdx.x;
    const int t0 = blockIdx.y * R;
    if (threadIdx.x < R && t0 + threadIdx.x < n_tokens) {
        const int t = t0 + threadIdx.x, e = st.seq_index[t], p = st.positions[t];
        s_pos[threadIdx.x] = p;
        s_in[threadIdx.x] = t - st.cu[e];
        s_slot[threadIdx.x] = st.slots[e];
        s_keep[threadIdx.x] = p >= st.lens[e] - RING;
    }
    __syncthreads();
    if (c >= C + n_dt) return;
    if (c >= C) {
        const int h = c - C;
        const float b = dt_bias[h], na = neg_a[h];
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int t = t0 + i;
            if (t >= n_tokens) break;
            const float dt = softplus_f(in.at(t, dt_off + h) + b);
            coef[((size_t)t * n_dt + h) * 2] = expf(na * dt);
            coef[((size_t)t * n_dt + h) * 2 + 1] = dt;
        }
        return;
    }
    float wv[TAPS], xs[R + RING];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[j] = w[(size_t)c * TAPS + j];
    const float b = bias ? bias[c] : 0.f;
    long long ld;
    if (const float* src = in.single(ld)) {                    // (all loads in flight at once)
#pragma unroll
        for (int i = 0; i < R + RING; ++i) {
            const int t = t0 - RING + i;
            xs[i] = t >= 0 && t < n_tokens ? src[(size_t)t * ld + off + c] : 0.f;
        }
    } else {
#pragma unroll
        for (int i = 0; i < R + RING; ++i) {
            const int t = t0 - RING + i;
            xs[i] = t >= 0 && t < n_tokens ? in.at(t, off + c) : 0.f;
        }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int t = t0 + i;
        if (t >= n_tokens) break;
        const int p = s_pos[i], slot = s_slot[i], before = s_in[i];
        float* ring = slot >= 0 && RING > 0 ? st.state + (size_t)slot * st.stride + st.off + c : nullptr;
        float acc = b;
#pragma unroll
        for (int k = RING; k >= 1; --k) {                      // oldest input first
            float x = 0.f;
            if (p - k >= 0) {
                if (k <= before) x = xs[RING + i - k];
                else if (ring) x = ring[(size_t)((p - k) % MOD) * C];
            }
            acc = fmaf(wv[RING - k], x, acc);
        }
        const float cur = xs[RING + i];
        const float y = silu_f(fmaf(wv[RING], cur, acc));
        out[(size_t)t * C + c] = y;
        if (rounded) rounded[(size_t)t * C + c] = from_f32<T>(y);
        if (ring && s_keep[i]) ring[(size_t)(p % MOD) * C] = cur;
    }
}

// The same for more taps than the forms above hold in registers: a thread has one channel of one
// token and reads its inputs where they lie.
template <typename T>
__global__ void __launch_bounds__(128)
ssm_conv_long_kernel(RowIn<float> in, int off, int C, int taps, StepArgs st,
                     const float* __restrict__ w, const float* __restrict__ bias,
                     float* __restrict__ out, T* __restrict__ rounded, int dt_off, int n_dt,
                     const float* __restrict__ dt_bias, const float* __restrict__ neg_a,
                     float* __restrict__ coef) {
    pdl_wait();
    pdl_launch_next();
    const int c = blockIdx.x * 128 + threadIdx.x, t = blockIdx.y, ring_rows = taps - 1;
    if (c >= C + n_dt) return;
    if (c >= C) {
        const int h = c - C;
        const float dt = softplus_f(in.at(t, dt_off + h) + dt_bias[h]);
        coef[((size_t)t * n_dt + h) * 2] = expf(neg_a[h] * dt);
        coef[((size_t)t * n_dt + h) * 2 + 1] = dt;
        return;
    }
    const int e = st.seq_index[t], p = st.positions[t], before = t - st.cu[e], slot = st.slots[e];
    float* ring = slot >= 0 ? st.state + (size_t)slot * st.stride + st.off + c : nullptr;
    const float* wc = w + (size_t)c * taps;
    float acc = bias ? bias[c] : 0.f;
    for (int k = min(ring_rows, p); k >= 1; --k) {             // oldest input first
        float x = 0.f;
        if (k <= before) x = in.at(t - k, off + c);
        else if (ring) x = ring[(size_t)((p - k) % ring_rows) * C];
        acc = fmaf(wc[ring_rows - k], x, acc);
    }
    const float cur = in.at(t, off + c);
    const float y = silu_f(fmaf(wc[ring_rows], cur, acc));
    out[(size_t)t * C + c] = y;
    if (rounded) rounded[(size_t)t * C + c] = from_f32<T>(y);
    if (ring && p >= st.lens[e] - ring_rows) ring[(size_t)(p % ring_rows) * C] = cur;
}

// ---------------------------------------------------------- selective scan
__host__ __device__ inline int ss_pad(int N) { return N <= 4 ? 4 : N <= 8 ? 8 : N <= 16 ? 16
                                                    : N <= 32 ? 32 : N <= 64 ? 64
                                                    : N <= 128 ? 128 : 256; }
constexpr int SS_MAX_N = 256;
constexpr int SS_THREADS = 128;
constexpr int SS_CH = 16;            // tokens staged in shared memory at a time

// low [T, r] = the row's first r values, rounded; bc [T, 2 Np]: B and C, each padded with zeros.
template <typename T>
__global__ void __launch_bounds__(128)
selective_low_kernel(RowIn<T> in, int r, int N, int Np, T* __restrict__ low, float* __restrict__ bc) {
    pdl_wait();
    pdl_launch_next();
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < r; i += blockDim.x) low[(size_t)t * r + i] = from_f32<T>(in.at(t, i));
    for (int i = threadIdx.x; i < 2 * Np; i += blockDim.x) {
        const int n = i < Np ? i : i - Np;
        bc[(size_t)t * 2 * Np + i] = n < N ? in.at(t, r + (i < Np ? 0 : N) + n) : 0.f;
    }
}

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

struct SelectiveArgs {
    const float* u;            // [T, inner] after convolution and silu
    const float* dt;           // [T, inner] without its bias
    const float* dt_bias;      // [inner]
    const float* bc;           // [T, 2 Np]
    const float* a2;           // [inner, N]: A * log2(e)
    const float* D;            // [inner]
    int inner, N, z_off;       // z: columns z_off .. of the stacked projection
};

// grid (channel blocks, sequences), 128 threads: 128 / L channels a CTA, L lanes a channel, NS
// states a lane.  Tokens come SS_CH at a time through two buffers filled by asynchronous copies;
// after a chunk has landed the CTA turns its step sizes into (dt, dt u) once, runs the
// recurrence (four tokens' read-outs are reduced over the lanes together), and finishes the
// chunk's outputs with the gate.  A token beyond the chunk has dt = 0 and changes nothing.
template <typename T, int NS, int L>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(SelectiveArgs a, RowIn<float> in, StepArgs st, T* __restrict__ out) {
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    constexpr int CC = SS_THREADS / L, Np = NS * L, CH = SS_CH;
    constexpr int BUF = CH * (3 * CC + 2 * Np);
    constexpr int ZN = CH * CC / SS_THREADS > 0 ? CH * CC / SS_THREADS : 1;
    float2* dd = reinterpret_cast<float2*>(sm + 2 * BUF);     // [CH][CC] (dt, dt u)
    float* ys = reinterpret_cast<float*>(dd + CH * CC);       // [CH][CC]
    const int e = blockIdx.y, slot = st.slots[e];
    const int t0 = st.cu[e], n = st.cu[e + 1] - t0;
    const int tid = threadIdx.x, l = tid % L, jc = tid / L;
    const int cb = blockIdx.x * CC, c = cb + jc;
    const bool live = c < a.inner;
    if (slot < 0) {
        for (int i = tid; i < n * CC; i += SS_THREADS)
            if (cb + i % CC < a.inner) out[(size_t)(t0 + i / CC) * a.inner + cb + i % CC] = from_f32<T>(0.f);
        pdl_launch_next();
        return;
    }
    for (int i = tid; i < 2 * BUF; i += SS_THREADS) sm[i] = 0.f;   // (what is never copied stays zero)
    __syncthreads();
    // z comes with the tokens where it is one sum, else its partial sums are added up below
    long long zld;
    const float* zrow = in.single(zld);
    if (zrow) zrow += a.z_off;
    const bool vec = a.inner % 4 == 0 && CC % 4 == 0 &&
                     (!zrow || (zld % 4 == 0 && ((uintptr_t)zrow & 15) == 0));
    auto fetch = [&](int ch) {
        float* base = sm + (ch & 1) * BUF;
        const int c0 = ch * CH, m = min(CH, n - c0);
        float *ds = base, *us = ds + CH * CC, *zs = us + CH * CC, *bs = zs + CH * CC;
        if (vec) {
            constexpr int Q = CC / 4 > 0 ? CC / 4 : 1;
            for (int i = tid; i < m * Q; i += SS_THREADS) {
                const int tt = i / Q, k = (i % Q) * 4;
                if (cb + k < a.inner) {
                    const size_t src = (size_t)(t0 + c0 + tt) * a.inner + cb + k;
                    cp_async_16(ds + tt * CC + k, a.dt + src);
                    cp_async_16(us + tt * CC + k, a.u + src);
                    if (zrow) cp_async_16(zs + tt * CC + k, zrow + (size_t)(t0 + c0 + tt) * zld + cb + k);
                }
            }
        } else {
            for (int i = tid; i < m * CC; i += SS_THREADS) {
                const int tt = i / CC, k = i % CC;
                if (cb + k < a.inner) {
                    const size_t src = (size_t)(t0 + c0 + tt) * a.inner + cb + k;
                    cp_async_4(ds + i, a.dt + src);
                    cp_async_4(us + i, a.u + src);
                    if (zrow) cp_async_4(zs + i, zrow + (size_t)(t0 + c0 + tt) * zld + cb + k);
                }
            }
        }
        for (int i = tid; i < m * (Np / 2); i += SS_THREADS)
            cp_async_16(bs + i * 4, a.bc + (size_t)(t0 + c0) * 2 * Np + i * 4);
        cp_async_commit();
    };
    fetch(0);
    float S[NS], a2[NS];
    float* srow = st.state + (size_t)slot * st.stride + st.off + (size_t)(live ? c : 0) * a.N;
#pragma unroll
    for (int s = 0; s < NS; ++s) {
        const int k = l * NS + s;
        const bool ok = live && k < a.N;
        S[s] = ok ? srow[k] : 0.f;
        a2[s] = ok ? a.a2[(size_t)c * a.N + k] : 0.f;
    }
    // outside the recurrence a thread's places of a chunk all have one channel
    const int my_c = cb + tid % CC;
    const bool mine = my_c < a.inner;
    const float my_bias = mine ? a.dt_bias[my_c] : 0.f, my_d = mine ? a.D[my_c] : 0.f;
    const int n_chunks = (n + CH - 1) / CH;
    for (int ch = 0; ch < n_chunks; ++ch) {
        const int c0 = ch * CH, m = min(CH, n - c0);
        const float* base = sm + (ch & 1) * BUF;
        const float *ds = base, *us = ds + CH * CC, *zs = us + CH * CC, *bs = zs + CH * CC;
        cp_async_wait<0>();
        __syncthreads();
        if (ch + 1 < n_chunks) fetch(ch + 1);
#pragma unroll
        for (int i = 0; i < ZN; ++i) {
            const int k = tid + i * SS_THREADS, tt = k / CC;
            float2 v = make_float2(0.f, 0.f);
            if (k < CH * CC && tt < m && mine) {
                v.x = softplus_f(ds[k] + my_bias);
                v.y = v.x * us[k];
            }
            if (k < CH * CC) dd[k] = v;
        }
        __syncthreads();
        for (int tt = 0; tt < m; tt += 4) {
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 d = dd[(tt + q) * CC + jc];
                const float* row = bs + (tt + q) * 2 * Np + l * NS;
                float B[NS], Cv[NS];
                if constexpr (NS % 4 == 0) {
#pragma unroll
                    for (int s = 0; s < NS; s += 4) {
                        const float4 x = *reinterpret_cast<const float4*>(row + s);
                        const float4 w = *reinterpret_cast<const float4*>(row + Np + s);
                        B[s] = x.x; B[s + 1] = x.y; B[s + 2] = x.z; B[s + 3] = x.w;
                        Cv[s] = w.x; Cv[s + 1] = w.y; Cv[s + 2] = w.z; Cv[s + 3] = w.w;
                    }
                } else {
                    const float2 x = *reinterpret_cast<const float2*>(row);
                    const float2 w = *reinterpret_cast<const float2*>(row + Np);
                    B[0] = x.x; B[1] = x.y; Cv[0] = w.x; Cv[1] = w.y;
                }
                float acc = 0.f;
#pragma unroll
                for (int s = 0; s < NS; ++s) {
                    S[s] = fmaf(d.y, B[s], ex2_ftz(d.x * a2[s]) * S[s]);
                    acc = fmaf(S[s], Cv[s], acc);
                }
                y[q] = acc;
            }
            // sum over the channel's lanes: each exchange halves the tokens a lane answers for
            if constexpr (L == 1) {
#pragma unroll
                for (int q = 0; q < 4; ++q) ys[(tt + q) * CC + jc] = y[q];
            } else {
                const bool up = l & 1;
                float m0 = up ? y[2] : y[0], m1 = up ? y[3] : y[1];
                m0 += __shfl_xor_sync(0xffffffffu, up ? y[0] : y[2], 1);
                m1 += __shfl_xor_sync(0xffffffffu, up ? y[1] : y[3], 1);
                if constexpr (L == 2) {
                    ys[(tt + (up ? 2 : 0)) * CC + jc] = m0;
                    ys[(tt + (up ? 3 : 1)) * CC + jc] = m1;
                } else {
                    const bool second = l & 2;
                    float v = second ? m1 : m0;
                    v += __shfl_xor_sync(0xffffffffu, second ? m0 : m1, 2);
#pragma unroll
                    for (int o = 4; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                    if (l < 4) ys[(tt + (up ? 2 : 0) + (second ? 1 : 0)) * CC + jc] = v;
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < ZN; ++i) {
            const int k = tid + i * SS_THREADS, tt = k / CC;
            if (tt < m && mine) {
                const float y = fmaf(my_d, us[k], ys[k]);
                const float z = zrow ? zs[k] : in.at(t0 + c0 + tt, a.z_off + my_c);
                out[(size_t)(t0 + c0 + tt) * a.inner + my_c] = from_f32<T>(y * silu_f(z));
            }
        }
    }
    pdl_launch_next();
    if (live) {
#pragma unroll
        for (int s = 0; s < NS; ++s)
            if (l * NS + s < a.N) srow[l * NS + s] = S[s];
    }
}

// ------------------------------------------------------ read-out of the head scan
// grid (tokens, norm groups): y = (num + D_h u) * silu(z) over its part's root mean square,
// times the weight.  V consecutive channels (of one head) a thread at a time.
template <int V>
__device__ __forceinline__ void ld_v(const float* p, float (&o)[V]) {
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        o[0] = t.x, o[1] = t.y, o[2] = t.z, o[3] = t.w;
    } else {
        o[0] = *p;
    }
}
__device__ __forceinline__ void st_v(float* p, const float (&a)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(a[0], a[1], a[2], a[3]);
}
__device__ __forceinline__ void st_v(__nv_bfloat16* p, const float (&a)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1]), hi = __floats2bfloat162_rn(a[2], a[3]);
    uint2 t;
    t.x = *reinterpret_cast<const uint32_t*>(&lo);
    t.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = t;
}
template <typename T>
__device__ __forceinline__ void st_v(T* p, const float (&a)[1]) { *p = from_f32<T>(a[0]); }

template <typename T, int V>
__global__ void __launch_bounds__(1024)
ssd_out_kernel(const float* __restrict__ num, const float* __restrict__ u, long long ldu,
               const float* __restrict__ D, RowIn<float> in, int z_off, const float* __restrict__ weight,
               float eps, int inner, int dv, T* __restrict__ y) {
    pdl_wait();
    pdl_launch_next();
    extern __shared__ __align__(16) float buf[]; // [inner / groups]
    __shared__ float red[33];
    const int t = blockIdx.x, width = inner / gridDim.y, c0 = blockIdx.y * width;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        const int c = c0 + i;
        float n[V], uu[V], z[V], v[V];
        ld_v<V>(num + (size_t)t * inner + c, n);
        ld_v<V>(u + (size_t)t * ldu + c, uu);
        const float d = D[c / dv];
        if (in.part) {
            const float* p = in.part + (size_t)t * in.W + z_off + c;
            ld_v<V>(p, z);
#pragma unroll 4
            for (int sp = 1; sp < in.n_splits; ++sp) {
                float a[V];
                ld_v<V>(p + (size_t)sp * in.split_stride, a);
#pragma unroll
                for (int k = 0; k < V; ++k) z[k] += a[k];
            }
        } else {
            ld_v<V>(in.row + (size_t)t * in.ld + z_off + c, z);
        }
#pragma unroll
        for (int k = 0; k < V; ++k) {
            v[k] = fmaf(d, uu[k], n[k]) * silu_f(z[k]);
            ss = fmaf(v[k], v[k], ss);
        }
        st_v(buf + i, v);
    }
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float)width + eps);
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V], w[V];
        ld_v<V>(buf + i, v);                     // (a thread reads what it wrote)
        ld_v<V>(weight + c0 + i, w);
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = v[k] * r * w[k];
        st_v(y + (size_t)t * inner + c0 + i, v);
    }
}

int row_of(RowIn<float>& in, const float* row, long long ld, const float* part, int n_splits, int T,
           int W) {
    AGV_REQUIRE((row != nullptr) != (part != nullptr && n_splits > 0),
                "ssm: the projection comes as rows or as partial sums");
    AGV_REQUIRE(part || ld >= W, "ssm: row stride shorter than a row");
    in = RowIn<float>{row, ld, part, n_splits, (long long)T * W, W};
    return 0;
}

constexpr int SSM_TAPS = 8;          // taps held in registers; more are read where they lie

template <typename T, int TAPS>
void launch_conv(const RowIn<float>& in, int n_tokens, int off, int C, const StepArgs& st,
                 const float* w, const float* bias, float* out, T* rounded, int dt_off, int n_dt,
                 const float* dt_bias, const float* neg_a, float* coef, cudaStream_t stream) {
    const unsigned gx = (unsigned)((C + n_dt + 127) / 128);
    if (n_tokens >= 256)
        agv_launch(ssm_conv_kernel<T, TAPS, 8>, dim3(gx, (n_tokens + 7) / 8), 128, 0, stream, in,
                   n_tokens, off, C, st, w, bias, out, rounded, dt_off, n_dt, dt_bias, neg_a, coef);
    else
        agv_launch(ssm_conv_kernel<T, TAPS, 1>, dim3(gx, n_tokens), 128, 0, stream, in, n_tokens,
                   off, C, st, w, bias, out, rounded, dt_off, n_dt, dt_bias, neg_a, coef);
}

template <typename T, int NS, int L>
int launch_selective(const SelectiveArgs& a, const RowIn<float>& in, const StepArgs& st, int B,
                     T* out, cudaStream_t stream) {
    auto kern = selective_scan_kernel<T, NS, L>;
    constexpr int CC = SS_THREADS / L;
    constexpr int smem = (2 * SS_CH * (3 * CC + 2 * NS * L) + 3 * SS_CH * CC) * (int)sizeof(float);
    static bool configured = false;
    if (smem > 48 * 1024 && !configured) {
        AGV_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        configured = true;
    }
    // (as with the other scans: few CTAs, each a long dependent chain, spread over the SMs)
    agv_launch_after(kern, dim3((a.inner + CC - 1) / CC, B), SS_THREADS, smem, stream, a, in, st, out);
    AGV_LAUNCH_OK("selective_scan_kernel");
    return 0;
}

}  // namespace

// row / part: the stacked projection [T, W] 32-bit (row stride ld) or [n_splits, T, W] partial
// sums.  conv_w [C, taps], conv_b [C] (or null) 32-bit.  out [T, C] 32-bit and, if not null, rounded [T, C]
// in dtype.  state: the ring, (taps - 1) * C values per slot from state_off on.  n_dt > 0: coef
// [T, n_dt, 2] receives (exp(neg_a dt), dt) of the columns dt_off ..
AGV_API int agv_ssm_conv(const float* row, long long ld, const float* part, int n_splits, int T,
                         int W, int off, int C, int taps, const float* conv_w, const float* conv_b,
                         float* out, void* rounded, int dtype, int dt_off, int n_dt,
                         const float* dt_bias, const float* neg_a, float* coef, float* state,
                         long long state_stride, long long state_off, const int* slots,
                         const int* cu, const int* seq_index, const int* positions, const int* lens,
                         cudaStream_t stream) {
    AGV_REQUIRE(T >= 0 && off >= 0 && C > 0 && off + C <= W && n_dt >= 0, "ssm_conv: bad sizes");
    AGV_REQUIRE(n_dt == 0 || (dt_off >= 0 && dt_off + n_dt <= W && dt_bias && neg_a && coef),
                "ssm_conv: step sizes need their columns, bias, decay and output");
    AGV_REQUIRE(taps >= 1, "ssm_conv: %d taps", taps);
    AGV_REQUIRE(T <= (taps <= SSM_TAPS ? 65535 * 8 : 65535), "ssm_conv: %d tokens exceed the grid "
                "limit", T);
    AGV_REQUIRE(taps == 1 || (state && state_stride >= state_off + (long long)(taps - 1) * C),
                "ssm_conv: the state has no room for the convolution's inputs");
    if (T == 0) return 0;
    RowIn<float> in;
    if (int rc = row_of(in, row, ld, part, n_splits, T, W)) return rc;
    const StepArgs st{state, state_stride, state_off, slots, cu, seq_index, positions, lens};
#define AGV_CONV(TT, K)                                                                          \
    case K: launch_conv<TT, K>(in, T, off, C, st, conv_w, conv_b, out, (TT*)rounded, dt_off, n_dt, \
                               dt_bias, neg_a, coef, stream); break
#define AGV_CONVS(TT)                                                                            \
    if (taps > SSM_TAPS)                                                                         \
        agv_launch(ssm_conv_long_kernel<TT>, dim3((unsigned)((C + n_dt + 127) / 128), (unsigned)T), \
                   128, 0, stream, in, off, C, taps, st, conv_w, conv_b, out, (TT*)rounded, dt_off, \
                   n_dt, dt_bias, neg_a, coef);                                                  \
    else switch (taps) {                                                                         \
        AGV_CONV(TT, 1); AGV_CONV(TT, 2); AGV_CONV(TT, 3); AGV_CONV(TT, 4);                      \
        AGV_CONV(TT, 5); AGV_CONV(TT, 6); AGV_CONV(TT, 7); AGV_CONV(TT, 8);                      \
    }
    if (dtype == AGV_F32) { AGV_CONVS(float) }
    else if (dtype == AGV_BF16) { AGV_CONVS(__nv_bfloat16) }
    else return agv_fail(-1, "ssm_conv: unknown dtype %d", dtype);
#undef AGV_CONVS
#undef AGV_CONV
    AGV_LAUNCH_OK("ssm_conv_kernel");
    return 0;
}

// States of a channel as the scan pads them.
AGV_API int agv_selective_pad(int N) {
    AGV_REQUIRE(N > 0 && N <= SS_MAX_N, "selective_scan: %d states a channel, at most %d", N, SS_MAX_N);
    return ss_pad(N);
}

// row / part: [T, r + 2 N] in dtype (row stride ld) or [n_splits, T, r + 2 N] 32-bit partial sums.
AGV_API int agv_selective_low(const void* row, long long ld, const float* part, int n_splits,
                              int dtype, int T, int r, int N, void* low, float* bc,
                              cudaStream_t stream) {
    AGV_REQUIRE(T >= 0 && r > 0 && N > 0 && N <= SS_MAX_N && (row || part), "selective_low: bad sizes");
    if (T == 0) return 0;
    const int W = r + 2 * N, Np = ss_pad(N);
    if (dtype == AGV_F32)
        agv_launch(selective_low_kernel<float>, (unsigned)T, 128, 0, stream,
                   RowIn<float>{(const float*)row, ld, part, n_splits, (long long)T * W, W}, r, N, Np,
                   (float*)low, bc);
    else if (dtype == AGV_BF16)
        agv_launch(selective_low_kernel<__nv_bfloat16>, (unsigned)T, 128, 0, stream,
                   RowIn<__nv_bfloat16>{(const __nv_bfloat16*)row, ld, part, n_splits,
                                        (long long)T * W, W}, r, N, Np, (__nv_bfloat16*)low, bc);
    else
        return agv_fail(-1, "selective_low: unknown dtype %d", dtype);
    AGV_LAUNCH_OK("selective_low_kernel");
    return 0;
}

// u, dt [T, inner], dt_bias, D [inner], bc [T, 2 Np] (agv_selective_low), a2 [inner, N] = A *
// log2(e), all 32-bit; z: columns z_off .. z_off + inner of the stacked projection (row / part as
// in agv_ssm_conv); out [T, inner] in dtype; state: S [inner, N] per slot from state_off on.
AGV_API int agv_selective_scan(const float* u, const float* dt, const float* dt_bias,
                               const float* bc, const float* a2, const float* D, const float* row,
                               long long ld, const float* part, int n_splits, int T, int W,
                               int z_off, int B, int inner, int N, void* out, int dtype,
                               float* state, long long state_stride, long long state_off,
                               const int* slots, const int* cu, cudaStream_t stream) {
    AGV_REQUIRE(T >= 0 && B >= 0 && inner > 0 && N > 0 && N <= SS_MAX_N && z_off >= 0 &&
                z_off + inner <= W, "selective_scan: bad sizes");
    AGV_REQUIRE(B <= 65535, "selective_scan: batch %d exceeds the grid limit", B);
    AGV_REQUIRE(state && state_stride >= state_off + (long long)inner * N,
                "selective_scan: the state is too small");
    AGV_REQUIRE(agv_aligned(u, 16) && agv_aligned(dt, 16) && agv_aligned(bc, 16),
                "selective_scan: operands must be 16-byte aligned");
    if (T == 0 || B == 0) return 0;
    RowIn<float> in;
    if (int rc = row_of(in, row, ld, part, n_splits, T, W)) return rc;
    const SelectiveArgs a{u, dt, dt_bias, bc, a2, D, inner, N, z_off};
    const StepArgs st{state, state_stride, state_off, slots, cu, nullptr, nullptr, nullptr};
    const int Np = ss_pad(N);
#define AGV_SS(NS, L)                                                                            \
    return dtype == AGV_F32 ? launch_selective<float, NS, L>(a, in, st, B, (float*)out, stream)  \
                            : launch_selective<__nv_bfloat16, NS, L>(a, in, st, B,               \
                                                                     (__nv_bfloat16*)out, stream)
    AGV_REQUIRE(dtype == AGV_F32 || dtype == AGV_BF16, "selective_scan: unknown dtype %d", dtype);
    switch (Np) {
        case 4: AGV_SS(2, 2);
        case 8: AGV_SS(4, 2);
        case 16: AGV_SS(4, 4);
        case 32: AGV_SS(4, 8);
        case 64: AGV_SS(8, 8);
        case 128: AGV_SS(8, 16);
        default: AGV_SS(8, 32);
    }
#undef AGV_SS
}

// num [T, inner] 32-bit (the scan's S^T C), u [T, >= inner] 32-bit with row stride ldu, D [inner /
// dv], z as above, weight [inner]; y [T, inner] in dtype.
AGV_API int agv_ssd_out(const float* num, const float* u, long long ldu, const float* D,
                        const float* row, long long ld, const float* part, int n_splits, int T,
                        int W, int z_off, const float* weight, float eps, int inner, int dv,
                        int groups, void* y, int dtype, cudaStream_t stream) {
    AGV_REQUIRE(T >= 0 && inner > 0 && dv > 0 && inner % dv == 0 && groups > 0 &&
                inner % groups == 0 && z_off >= 0 && z_off + inner <= W && ldu >= inner,
                "ssd_out: bad sizes");
    AGV_REQUIRE(groups <= 65535, "ssd_out: %d parts exceed the grid limit", groups);
    const size_t smem = (size_t)(inner / groups) * sizeof(float);
    AGV_REQUIRE(smem <= 48 * 1024, "ssd_out: parts of %d channels exceed shared memory",
                inner / groups);
    if (T == 0) return 0;
    RowIn<float> in;
    if (int rc = row_of(in, row, ld, part, n_splits, T, W)) return rc;
    const int width = inner / groups;
    const bool vec = width % 4 == 0 && dv % 4 == 0 && z_off % 4 == 0 && ldu % 4 == 0 &&
                     agv_aligned(num, 16) && agv_aligned(u, 16) && agv_aligned(weight, 16) &&
                     agv_aligned(y, 16) &&
                     (part ? W % 4 == 0 && agv_aligned(part, 16) : ld % 4 == 0 && agv_aligned(row, 16));
    const int need = vec ? width / 4 : width;
    // (few rows: all of a row's loads in one pass; many: several rows to an SM)
    const int most = (long long)T * groups <= 296 ? 1024 : 256;
    int threads = 32;
    while (threads < most && threads < need) threads *= 2;
    const dim3 grid((unsigned)T, (unsigned)groups);
#define AGV_SO(TT, V)                                                                             \
    agv_launch(ssd_out_kernel<TT, V>, grid, threads, smem, stream, num, u, ldu, D, in, z_off,     \
               weight, eps, inner, dv, (TT*)y)
    if (dtype == AGV_F32) { if (vec) AGV_SO(float, 4); else AGV_SO(float, 1); }
    else if (dtype == AGV_BF16) { if (vec) AGV_SO(__nv_bfloat16, 4); else AGV_SO(__nv_bfloat16, 1); }
    else return agv_fail(-1, "ssd_out: unknown dtype %d", dtype);
#undef AGV_SO
    AGV_LAUNCH_OK("ssd_out_kernel");
    return 0;
}
