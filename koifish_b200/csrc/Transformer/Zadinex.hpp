// Zadinex.hpp -- neurons of the Zadinex stack.  Pre-norm layers whose norm takes no statistics and whose sublayers have a scale per entry,
//     x += ls1 * mixer(n1(x)),   x += ls2 * ff(n2(x)),      n(y) = tanh(alpha y) * w + b.
// Mixers:
//   TimeMix          r, k, v, g and the decay's input each read a mix of the token and the one before it, h + (h' - h) mu_s (h' = 0 ahead of the
//                    first token); decay d = exp(-exp(W_2 tanh(W_1 m_w) + w0)) per key channel; per head o = S^T r + (r . (u * k)) v, then
//                    S <- diag(d) S + k v^T; o over its rms, times a weight, times silu(g); W_o.  State: S [heads][dim][dim] and the last h,
//                    fp32 per sequence slot.
//   BlendedAttention causal grouped-query softmax attention: rotation in halves of the first rot_dims entries of q and k, then every head of
//                    q and k over its rms (no weight); a sink term per head in the denominator; from the second blending layer on the values
//                    are (1 - l) v + l v_first, v_first = the first blending layer's values of the same token.  Cache: one row
//                    [k | blended v] per position and slot.
// Feed-forward: dense, W_d (gelu(W_g h) * (W_u h)), or routed experts (MoE, Sipazen.hpp): softmax scores over experts and pass-through
// outputs, choice by score + correction inside the best groups, weights renormalised; experts with the clamped gate; an entry of a
// pass-through output adds the sublayer's input itself.
// The residual, norms, router, recurrence (with its decay's second projection), rotation angles, scores and softmax are fp32; matmul inputs
// and cache rows are in the activation type.  The neurons use the model's HybridScratch and SeqStateCache (Sipazen.hpp, QWen3.hpp); step
// function, graphs, sampler and generation loop are Fish's own.  The reference has no counterpart (its inference path is the Qwen3 block,
// QWen.cpp:16-145).
#pragma once
#include "Fazolorn.hpp"

namespace koifish {

struct TanhNorm : GeNeuron {
    hGTensor w, b, alpha;
};
struct TimeMix : GeNeuron {
    MIXER_CARD card;
    hGTensor mu[5];  // r, k, v, g, w
    hGTensor r, k, v, g, w1, w2, w0, u, norm, o;
    StackedLinear mus;  // the five mu as rows of one table
    // mid holds the five mixed inputs, M rows each -> sub
    int cuInfer(int M, int layer);
};
struct BlendedAttention : GeNeuron {
    MIXER_CARD card;
    hGTensor q, k, v, vmix, sink, o;
    double* inv_freq = nullptr;  // device [rot_dims / 2]
    bool blend_source = false;   // the first layer that blends: its values are what the others blend with
    // u: stacked first projections, q | k | v consecutive -> sub
    int cuInfer(int M, float* u, int ldu, int layer);
};
struct GeluFF : GeNeuron {  // W_down (gelu(W_gate h) * (W_up h)), gelu in its tanh form
    MOE_CARD card;
    hGTensor gate, up, down;
    StackedLinear cat;  // gate | up
    int cuInfer(int M);  // reads hact -> sub
};
struct ZdxBlock : GeNeuron {
    TanhNorm norm1, norm2;
    hGTensor ls1, ls2;
    StackedLinear cat;  // attention: q | k | v
    std::unique_ptr<TimeMix> wkv;
    std::unique_ptr<BlendedAttention> attn;
    std::unique_ptr<GeluFF> dense;
    std::unique_ptr<MoE> moe;
};

}  // namespace koifish
