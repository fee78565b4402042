// Gadilix.hpp -- neurons of the Gadilix stack.  A layer normalises what a sublayer RETURNS:
//     x += m * norm1(attention(shift(x))),   x += m * norm2(ff(x)),      norm(y) = y / sqrt(mean(y^2) + eps) * g   with ONE number g
// and the stream starts as norm(embedding row).  shift(x)_t = x_t + s * (x_{t-1} - x_t) per entry: the mixer reads every token mixed with the
// one before it (zeros before the first), so a sequence's last x is part of its state, in every layer.
//   PooledAttention  grouped-query softmax attention, no rotation; q and k RMS-normed per head with one weight of head size each; a query at i
//                    sees the last `window` positions and, for every block of `pool` positions that ends at or before i - window, the
//                    mean key and mean value of the block, in one softmax; head h's result times sigmoid((W_g shift(x))_h).  Cache per
//                    slot: a ring of max(window, pool) + (step) - 1 rows [k | v], the blocks' mean rows behind it, the shift's tail.
//   feed-forward     routed experts (MoE, Sipazen.hpp) that a table of token ids names -- no router, weights 1 / top -- beside an ungated
//                    shared expert.  The dispatch tables of all layers hang on the token ids alone and are made once per step.
// A layer may run on another layer's tensors (LAYER_CARD::owner) with a cache and a tail of its own.  The residual, norms, shift, scores,
// softmax and the output gate's sigmoid are fp32; matmul inputs and cache rows are in the activation type.  The neurons use the model's
// HybridScratch and SeqStateCache (Sipazen.hpp, QWen3.hpp); step function, graphs, sampler and generation loop are Fish's own.  The
// reference has no counterpart (its inference path is the Qwen3 block, QWen.cpp:16-145).
#pragma once
#include "Sipazen.hpp"

namespace koifish {

struct PooledAttention : GeNeuron {
    MIXER_CARD card;
    hGTensor q, k, v, qn, kn, g, o;
    // u: stacked first projections, q | k | v consecutive from column off, gate logits at column off_g; layer: entry of the SeqStateCache -> sub
    int cuInfer(int M, float* u, int ldu, int off, int off_g, int layer);
};
struct GdxBlock : GeNeuron {
    GroupNorm norm1, norm2;  // weights of one entry
    hGTensor shift;
    StackedLinear cat;  // q | k | v | g
    std::unique_ptr<PooledAttention> attn;
    std::unique_ptr<MoE> moe;
};

}  // namespace koifish
