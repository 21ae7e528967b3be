// The gated activations act(g, u) of a pair of products: what a gate/up epilogue makes of the
// two finished sums.
//
//   kind 0: gelu_tanh(g) * u        kind 1: silu(g) * u
//   kind 4: with g <- min(g, limit), u <- clamp(u, -limit, limit):
//           g * sigmoid(alpha * g) * (u + 1)
// (kinds 2 and 3 are activations of a plain product, without u.)
#pragma once

enum AgvActivation {
    AGV_ACT_GELU_TANH = 0,
    AGV_ACT_SILU = 1,
    AGV_ACT_RELU2 = 2,
    AGV_ACT_GELU_ERF = 3,
    AGV_ACT_CLAMPED = 4,
};

// An activation as a kernel receives it; alpha and limit belong to AGV_ACT_CLAMPED.
struct GateAct {
    int kind;
    float alpha, limit;
};

static inline bool gate_act_ok(const GateAct& a) {
    return a.kind == AGV_ACT_GELU_TANH || a.kind == AGV_ACT_SILU ||
           (a.kind == AGV_ACT_CLAMPED && a.limit > 0.f);
}

// AGV_ACT_CLAMPED in 32-bit.
__device__ __forceinline__ float clamped_gate(float g, float u, const GateAct& a) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    return g / (1.0f + expf(-a.alpha * g)) * (u + 1.0f);
}
// The same for a result that is rounded to bfloat16.
__device__ __forceinline__ float clamped_gate_fast(float g, float u, const GateAct& a) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    return __fdividef(g, 1.0f + __expf(-a.alpha * g)) * (u + 1.0f);
}
