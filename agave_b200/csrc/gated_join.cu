// How several branches of one layer join the 32-bit residual stream in one launch:
//
//     h[t] += sum_i  mult_i * g_i(t) * (sum over ranges of K of y_i[t]);      x[t] = norm(h[t]) * w
//
// with g_i(t) = sigmoid(logits[t, gate_i] + bias[gate_i]) element by element (a stacked
// projection  G_0 | G_1 | ...  of one row width each, 32-bit or 32-bit partial sums), or one.
// The branch outputs come as 32-bit partial sums or in the compute dtype; the gate, the sum and
// the RMS norm are 32-bit.  Without a stream (h null) x receives the weighted sum itself.
#include "common.cuh"
#include "row_in.cuh"

namespace {

constexpr int JOIN_TERMS = 5;

struct JoinTerm {
    const float* y32;          // [n_splits, R, H] or null
    const __nv_bfloat16* y16;  // [R, H] or null
    long long row_stride;      // H, or 0: one row for all
    long long split_stride;
    int n_splits, gate;        // gate: index of its gate, or -1
    float mult;
};
struct JoinArgs {
    JoinTerm term[JOIN_TERMS];
    int n_terms, n_gates;
    const float* gate_bias;    // [n_gates * H]
};

template <int V> struct Pack { float v[V]; };
template <int V>
__device__ __forceinline__ Pack<V> ld_pack(const float* p) {
    Pack<V> o;
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        o.v[0] = t.x, o.v[1] = t.y, o.v[2] = t.z, o.v[3] = t.w;
    } else {
        o.v[0] = *p;
    }
    return o;
}
template <int V>
__device__ __forceinline__ Pack<V> ld_pack(const __nv_bfloat16* p) {
    Pack<V> o;
    if constexpr (V == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        o.v[0] = __uint_as_float(t.x << 16), o.v[1] = __uint_as_float(t.x & 0xffff0000u);
        o.v[2] = __uint_as_float(t.y << 16), o.v[3] = __uint_as_float(t.y & 0xffff0000u);
    } else {
        o.v[0] = __bfloat162float(*p);
    }
    return o;
}
template <int V>
__device__ __forceinline__ void st_pack(float* p, const Pack<V>& a) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
    else *p = a.v[0];
}
template <int V>
__device__ __forceinline__ void st_pack(__nv_bfloat16* p, const Pack<V>& a) {
    if constexpr (V == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]);
        const __nv_bfloat162 hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
        uint2 t;
        t.x = *reinterpret_cast<const uint32_t*>(&lo);
        t.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = t;
    } else {
        *p = __float2bfloat16_rn(a.v[0]);
    }
}
// n partial sums of one place, added in order
template <int V>
__device__ __forceinline__ Pack<V> sum_splits(const float* p, int n, long long stride) {
    Pack<V> o = ld_pack<V>(p);
#pragma unroll 4
    for (int s = 1; s < n; ++s) {
        const Pack<V> t = ld_pack<V>(p + (size_t)s * stride);
#pragma unroll
        for (int k = 0; k < V; ++k) o.v[k] += t.v[k];
    }
    return o;
}

// One CTA a row; V values a thread at a time.
template <typename TX, int V>
__global__ void __launch_bounds__(1024)
gated_join_kernel(float* __restrict__ h, JoinArgs a, RowIn<float> gates,
                  const float* __restrict__ w_next, TX* __restrict__ x, int H, float eps) {
    pdl_wait();
    pdl_launch_next();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const int t = blockIdx.x;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
        Pack<V> acc;
        if (h) acc = ld_pack<V>(h + (size_t)t * H + i);
        else {
#pragma unroll
            for (int k = 0; k < V; ++k) acc.v[k] = 0.f;
        }
        Pack<V> g[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            if (j < a.n_gates) {
                const int c = j * H + i;
                g[j] = gates.part ? sum_splits<V>(gates.part + (size_t)t * gates.W + c,
                                                  gates.n_splits, gates.split_stride)
                                  : ld_pack<V>(gates.row + (size_t)t * gates.ld + c);
                const Pack<V> b = ld_pack<V>(a.gate_bias + c);
#pragma unroll
                for (int k = 0; k < V; ++k) g[j].v[k] = 1.0f / (1.0f + expf(-(g[j].v[k] + b.v[k])));
            }
        }
#pragma unroll
        for (int j = 0; j < JOIN_TERMS; ++j) {
            if (j < a.n_terms) {
                const JoinTerm& m = a.term[j];
                const Pack<V> y = m.y32 ? sum_splits<V>(m.y32 + (size_t)t * m.row_stride + i, m.n_splits,
                                                        m.split_stride)
                                        : ld_pack<V>(m.y16 + (size_t)t * m.row_stride + i);
#pragma unroll
                for (int k = 0; k < V; ++k) {
                    const float gk = m.gate < 0 ? 1.0f : m.gate == 0 ? g[0].v[k] : g[1].v[k];
                    acc.v[k] = fmaf(gk * m.mult, y.v[k], acc.v[k]);
                }
            }
        }
        if (h) st_pack<V>(h + (size_t)t * H + i, acc);
        if (w_next) {
            st_pack<V>(row + i, acc);
#pragma unroll
            for (int k = 0; k < V; ++k) ss = fmaf(acc.v[k], acc.v[k], ss);
        } else if (x) {
            st_pack<V>(x + (size_t)t * H + i, acc);
        }
    }
    if (!w_next) return;
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float)H + eps);
    for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
        Pack<V> v = ld_pack<V>(row + i);                     // (a thread reads what it wrote)
        const Pack<V> w = ld_pack<V>(w_next + i);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] = v.v[k] * r * w.v[k];
        st_pack<V>(x + (size_t)t * H + i, v);
    }
}

}  // namespace

// Terms i < n_terms (at most 5): y[i] points to [n_splits[i], R, H] 32-bit sums (dtype[i] 0) or
// [R, H] bfloat16 (dtype[i] 1), or, with n_splits[i] 0, to one row [H] that every row takes (a
// bias), times mult[i], through gate gate[i] (-1: none).  gate_row / gate_part:
// the gates' logits [R, n_gates * H] 32-bit or partial sums of them; gate_bias [n_gates * H].  h [R,
// H] or null; w_next [H] with x [R, H], or both null (or x alone: the sum as it is).
AGV_API int agv_gated_join(float* h, int R, int H, int n_terms, const void* const* y,
                           const int* dtype, const int* n_splits, const float* mult,
                           const int* gate, int n_gates, const float* gate_row, long long gate_ld,
                           const float* gate_part, int gate_splits, const float* gate_bias,
                           const float* w_next, float eps, void* x, int x_dtype,
                           cudaStream_t stream) {
    AGV_REQUIRE(R >= 0 && H > 0 && n_terms >= 1 && n_terms <= JOIN_TERMS, "gated_join: bad sizes");
    AGV_REQUIRE(n_gates >= 0 && n_gates <= 2, "gated_join: %d gates, at most 2", n_gates);
    AGV_REQUIRE(h || x, "gated_join: nowhere to write");
    AGV_REQUIRE(!w_next || x, "gated_join: a norm needs an output");
    AGV_REQUIRE(n_gates == 0 || (gate_bias && ((gate_row != nullptr) != (gate_part != nullptr))),
                "gated_join: gates need their logits and biases");
    if (R == 0) return 0;
    JoinArgs a{};
    a.n_terms = n_terms, a.n_gates = n_gates, a.gate_bias = gate_bias;
    bool vec = H % 4 == 0 && agv_aligned(h, 16) && agv_aligned(x, 16) && agv_aligned(w_next, 16) &&
               agv_aligned(gate_row, 16) && agv_aligned(gate_part, 16) && agv_aligned(gate_bias, 16) &&
               (!gate_row || gate_ld % 4 == 0);
    for (int i = 0; i < n_terms; ++i) {
        AGV_REQUIRE(y[i] && n_splits[i] >= 0 && gate[i] >= -1 && gate[i] < n_gates,
                    "gated_join: term %d is incomplete", i);
        AGV_REQUIRE(dtype[i] == AGV_F32 || (dtype[i] == AGV_BF16 && n_splits[i] <= 1),
                    "gated_join: term %d must be 32-bit sums or one bfloat16 row", i);
        JoinTerm& m = a.term[i];
        m.y32 = dtype[i] == AGV_F32 ? (const float*)y[i] : nullptr;
        m.y16 = dtype[i] == AGV_BF16 ? (const __nv_bfloat16*)y[i] : nullptr;
        m.split_stride = (long long)R * H;
        m.row_stride = n_splits[i] ? H : 0;
        m.n_splits = n_splits[i] ? n_splits[i] : 1, m.gate = gate[i], m.mult = mult[i];
        vec = vec && agv_aligned(y[i], 16);
    }
    const int W = n_gates * H;
    const RowIn<float> gates{gate_row, gate_ld, gate_part, gate_splits, (long long)R * W, W};
    const size_t smem = w_next ? (size_t)H * sizeof(float) : 0;
    AGV_REQUIRE(smem <= 200 * 1024, "gated_join: rows of %d values exceed shared memory", H);
    const int need = vec ? (H + 3) / 4 : H;
    // (few rows: one pass of all a row's loads; many: several rows to an SM)
    const int most = R <= 296 ? 1024 : 256;
    int threads = 64;
    while (threads < most && threads < need) threads *= 2;
#define AGV_JOIN(TX, V)                                                                         \
    do {                                                                                        \
        auto kern = gated_join_kernel<TX, V>;                                                   \
        if (smem > 48 * 1024)                                                                   \
            AGV_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                             (int)smem));                                       \
        agv_launch(kern, (unsigned)R, threads, smem, stream, h, a, gates, w_next, (TX*)x, H, eps); \
    } while (0)
    const int xd = x ? x_dtype : AGV_F32;
    AGV_REQUIRE(xd == AGV_F32 || xd == AGV_BF16, "gated_join: unknown dtype %d", xd);
    if (xd == AGV_F32) { if (vec) AGV_JOIN(float, 4); else AGV_JOIN(float, 1); }
    else { if (vec) AGV_JOIN(__nv_bfloat16, 4); else AGV_JOIN(__nv_bfloat16, 1); }
#undef AGV_JOIN
    AGV_LAUNCH_OK("gated_join_kernel");
    return 0;
}
