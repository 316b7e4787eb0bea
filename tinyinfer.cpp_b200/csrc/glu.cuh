// A sum that passes a gate, and gated activations of a feed-forward, y = act(gate, up), shared by the row-wise kernel and the
// epilogues of the experts' products.
//   GLU_SILU      silu(g) * u
//   GLU_CLAMPED   g = min(g, limit), u = clamp(u, -limit, limit), y = g * sigmoid(alpha * g) * (u + 1)
//   GLU_GELU_TANH gelu(g) * u, the tanh form of gelu
// and activations of one value, y = act(u), of feed-forwards without a gate:
//   ACT_RELU2     the square of relu(u)
#pragma once

enum { GLU_SILU = 0, GLU_CLAMPED = 1, GLU_GELU_TANH = 2 };
enum { ACT_RELU2 = 16 };          // numbers of their own, so that one argument can name either sort
__host__ __device__ constexpr bool act_is_gated(int kind) { return kind < ACT_RELU2; }

__device__ __forceinline__ float unary_activation(int kind, float u) {
    (void)kind;                   // ACT_RELU2 is the one there is
    u = fmaxf(u, 0.0f);
    return u * u;
}

// What an epilogue needs to know of the activation; kind GLU_SILU ignores the rest.
struct GluArgs { int kind; float limit, alpha; };

// A sublayer's result y on its way into the residual x: x + scale sigmoid(g) y
__device__ __forceinline__ float gated_sum(float x, float y, float g, float scale) {
    return fmaf(scale / (1.0f + expf(-g)), y, x);
}

// What an epilogue that adds to C needs to know of such a gate (gate null: C + scale y, the plain sum for scale 1).  `gate` is written by a
// kernel of the same chain, so it is no read-only data.
struct AddGate { const float* gate; int ld; const float* bias; float scale; };

__device__ __forceinline__ float add_through(const AddGate& g, float was, float y, float gate, float bias) {
    return g.gate ? gated_sum(was, y, gate + bias, g.scale) : fmaf(g.scale, y, was);
}
// four neighbouring columns (row, col .. col + 3); the gate's rows and the bias start on 16 bytes
__device__ __forceinline__ float4 add_through4(const AddGate& g, int row, int col, float4 was, float4 y) {
    if (g.gate == nullptr)
        return make_float4(fmaf(g.scale, y.x, was.x), fmaf(g.scale, y.y, was.y), fmaf(g.scale, y.z, was.z),
                           fmaf(g.scale, y.w, was.w));
    const float4 v = __ldcg(reinterpret_cast<const float4*>(g.gate + (size_t)row * g.ld + col));
    const float4 b = __ldg(reinterpret_cast<const float4*>(g.bias + col));
    return make_float4(gated_sum(was.x, y.x, v.x + b.x, g.scale), gated_sum(was.y, y.y, v.y + b.y, g.scale),
                       gated_sum(was.z, y.z, v.z + b.z, g.scale), gated_sum(was.w, y.w, v.w + b.w, g.scale));
}

// gelu(z) = z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh(float z) {
    const float inner = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
    return 0.5f * z * (1.0f + tanhf(inner));
}

__device__ __forceinline__ float glu_activation(int kind, float g, float u, float limit, float alpha) {
    if (kind == GLU_CLAMPED) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
    }
    if (kind == GLU_GELU_TANH) return gelu_tanh(g) * u;
    return g / (1.0f + expf(-g)) * u;
}
