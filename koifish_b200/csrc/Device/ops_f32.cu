// ops_f32.cu -- the small ops of models whose residual stream, norms and routers are kept in 32-bit floats: embedding rows widened to
// fp32, grouped RMS norm (optionally of a gated input, optionally accumulated into the residual), and the router / dispatch / combine
// steps of a mixture of experts.  Outputs that feed a matmul are written in the activation type: bf16 bits, or float for a model that
// runs entirely in 32-bit.  No reference equivalent (the reference's norms are CU_rms_infer over bf16 rows, layernorm.cuh:801-859, and
// it has no expert routing on the inference path).
#include <math.h>

#include <algorithm>

#include "kf_common.cuh"

namespace {
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

__global__ void kf_embed_f32_kernel(float* __restrict__ out, float* __restrict__ out2, const uint16_t* __restrict__ table, const int32_t* __restrict__ tokens,
                                    int dim, float scale) {
    const uint16_t* row = table + (size_t)tokens[blockIdx.x] * dim;
    float* o            = out + (size_t)blockIdx.x * dim;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const float v = bf16_bits_to_f32(row[i]) * scale;
        o[i] = v;
        if (out2) out2[(size_t)blockIdx.x * dim + i] = v;
    }
}

// out[r][c] = act(in[r][c] + bias[c]) (* mul[r][c]) ; ACT 0: identity, 1: gelu (tanh form), 2: relu squared, 3: silu, 4: relu.
// OUT 0: bf16 bits, 1: float, 2: out (float) += result.
template <int ACT, int OUT>
__global__ void kf_bias_act_kernel(void* __restrict__ out, int ldo, const float* __restrict__ in, int ldi, const uint16_t* __restrict__ bias,
                                   const float* __restrict__ mul, int ldm, int cols) {
    const int r = blockIdx.y;
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < cols; c += gridDim.x * blockDim.x) {
        float v = in[(size_t)r * ldi + c] + (bias ? bf16_bits_to_f32(bias[c]) : 0.f);
        if (ACT == 1) v = gelu_tanh_f(v);
        if (ACT == 2) v = v > 0.f ? v * v : 0.f;
        if (ACT == 3) v = v * sigmoid_f(v);
        if (ACT == 4) v = fmaxf(v, 0.f);
        if (mul) v *= mul[(size_t)r * ldm + c];
        if (OUT == 0) ((uint16_t*)out)[(size_t)r * ldo + c] = f32_to_bf16_bits(v);
        else if (OUT == 1) ((float*)out)[(size_t)r * ldo + c] = v;
        else ((float*)out)[(size_t)r * ldo + c] += v;
    }
}
// out[r][c] = gelu_tanh(in[r][c]) * table[token[r]][c0 + c]   (a per-token embedding slice gating a projection), activation type out
template <typename TO>
__global__ void kf_token_gate_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ in, int ldi, const uint16_t* __restrict__ table, int ldt, int c0,
                                     const int32_t* __restrict__ tokens, int cols) {
    const int r = blockIdx.x;
    const uint16_t* e = table + (size_t)tokens[r] * ldt + c0;
    for (int c = threadIdx.x; c < cols; c += blockDim.x) {
        const float v = gelu_tanh_f(in[(size_t)r * ldi + c]) * bf16_bits_to_f32(e[c]);
        if (sizeof(TO) == 2) ((uint16_t*)out)[(size_t)r * ldo + c] = f32_to_bf16_bits(v);
        else ((float*)out)[(size_t)r * ldo + c] = v;
    }
}
// Weighted sum over the depth of a stack: hist[n_prev] = x (this layer's result) ; x = sum_{j < n_prev} w[j] * hist[j] + w[n_prev] * x.
// hist: [n_prev + 1][hist_stride] floats; n = rows * dim elements.
__global__ void kf_depth_mix_kernel(float* __restrict__ x, float* __restrict__ hist, size_t hist_stride, const uint16_t* __restrict__ w, int n_prev, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const float cur = x[i];
    hist[(size_t)n_prev * hist_stride + i] = cur;
    float s = 0.f;
    for (int j = 0; j < n_prev; j++) s = fmaf(bf16_bits_to_f32(w[j]), hist[(size_t)j * hist_stride + i], s);
    x[i] = fmaf(bf16_bits_to_f32(w[n_prev]), cur, s);
}

// One block per (row, group).  v = x * gatefn(g) (GATE 0: none, 1: sigmoid(g + gate_bias), 2: silu(g));  r = v / sqrt(mean_group(v^2) + eps) * w;
// GATE 3 / 4: the gate multiplies the normed result instead, r *= sigmoid(g) / silu(g).  w_shared 1: one weight of group size for all groups;
// 2: one number for every entry.
// ACC: res[row] += mult * r (fp32 residual stream)  else  out[row] = r in the activation type.  w_add is added to every weight in
// fp32 (1 for weights that are stored around zero).
template <int GATE, bool ACC, typename TO>
__global__ void __launch_bounds__(256) kf_group_norm_kernel(TO* __restrict__ out, int ldo, float* __restrict__ res, const float* __restrict__ x, int ldx,
                                                            const float* __restrict__ gate, int ldg, const uint16_t* __restrict__ gate_bias,
                                                            const uint16_t* __restrict__ w, const int32_t* __restrict__ row_idx, int dim, int groups,
                                                            float eps, float mult, int w_shared, float w_add, float out_mult) {
    __shared__ float red[32];
    const int r = blockIdx.x, grp = blockIdx.y, gs = dim / groups;
    const int src = row_idx ? row_idx[r] : r;
    const float* xr = x + (size_t)src * ldx + grp * gs;
    const float* gr = GATE ? gate + (size_t)src * ldg + grp * gs : nullptr;
    auto val = [&](int i) -> float {
        float v = xr[i];
        if (GATE == 1) v *= sigmoid_f(gr[i] + (gate_bias ? bf16_bits_to_f32(gate_bias[grp * gs + i]) : 0.f));
        if (GATE == 2) {
            const float z = gr[i];
            v *= z * sigmoid_f(z);
        }
        return v;
    };
    float ss = 0.f;
    for (int i = threadIdx.x; i < gs; i += blockDim.x) {
        const float v = val(i);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)gs + eps);
    for (int i = threadIdx.x; i < gs; i += blockDim.x) {
        float o = val(i) * s * (w_add + bf16_bits_to_f32(w[w_shared == 2 ? 0 : w_shared ? i : grp * gs + i]));
        if (GATE == 3) o *= sigmoid_f(gr[i]);
        if (GATE == 4) {
            const float z = gr[i];
            o *= z * sigmoid_f(z);
        }
        if (ACC) {
            float* p = res + (size_t)r * dim + grp * gs + i;
            *p       = *p + mult * o;
        } else if (sizeof(TO) == 2) {
            ((uint16_t*)out)[(size_t)r * ldo + grp * gs + i] = f32_to_bf16_bits(o * out_mult);
        } else {
            ((float*)out)[(size_t)r * ldo + grp * gs + i] = o * out_mult;
        }
    }
}

// The same for parts of at most 32 * kPartRegs entries that do not go into the residual: a warp per (row, group), its entries in registers.
constexpr int kPartRegs = 8;
template <int GATE, typename TO>
__global__ void __launch_bounds__(256) kf_part_norm_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ x, int ldx, const float* __restrict__ gate, int ldg,
                                                           const uint16_t* __restrict__ gate_bias, const uint16_t* __restrict__ w, const int32_t* __restrict__ row_idx,
                                                           int rows, int dim, int groups, float eps, int w_shared, float w_add, float out_mult) {
    const long long u = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (u >= (long long)rows * groups) return;
    const int r = (int)(u / groups), grp = (int)(u % groups), gs = dim / groups, lane = threadIdx.x & 31;
    const int src = row_idx ? row_idx[r] : r;
    const float* xr = x + (size_t)src * ldx + grp * gs;
    const float* gr = GATE ? gate + (size_t)src * ldg + grp * gs : nullptr;
    float v[kPartRegs], g[kPartRegs], wt[kPartRegs], ss = 0.f;
#pragma unroll
    for (int k = 0; k < kPartRegs; k++) {
        const int i = lane + 32 * k;
        const bool in = i < gs;
        v[k] = in ? xr[i] : 0.f, g[k] = (GATE && in) ? gr[i] : 0.f;
        wt[k] = in ? bf16_bits_to_f32(w[w_shared == 2 ? 0 : w_shared ? i : grp * gs + i]) : 0.f;
        if (GATE == 1 && in && gate_bias) g[k] += bf16_bits_to_f32(gate_bias[grp * gs + i]);
    }
#pragma unroll
    for (int k = 0; k < kPartRegs; k++) {
        if (GATE == 1) v[k] *= sigmoid_f(g[k]);
        if (GATE == 2) v[k] *= g[k] * sigmoid_f(g[k]);
        ss = fmaf(v[k], v[k], ss);
    }
    const float s = 1.0f / sqrtf(warp_sum(ss) / (float)gs + eps);
    TO* o = out + (size_t)r * ldo + grp * gs;
#pragma unroll
    for (int k = 0; k < kPartRegs; k++) {
        const int i = lane + 32 * k;
        if (i >= gs) break;
        float t = v[k] * s * (w_add + wt[k]);
        if (GATE == 3) t *= sigmoid_f(g[k]);
        if (GATE == 4) t *= g[k] * sigmoid_f(g[k]);
        if (sizeof(TO) == 2) ((uint16_t*)o)[i] = f32_to_bf16_bits(t * out_mult);
        else ((float*)o)[i] = t * out_mult;
    }
}

// Post-norm residual step of one row:  res += mult * v / sqrt(mean(v^2) + eps) * (w_add + w)  with w per entry or (w_one) one number; v is
//   SRC 0: sa * a + sb * b (b optional);   SRC 1: sum_j wgt[j] * y[entry_slot[j]] + shared (a token's experts; shared optional);
//   SRC 2: a row of a bf16 table -- then the row starts the stream: res = the normed row.
// The new residual row is also written in the activation type (what the next sublayer's matmul reads) when act is given; with `shift`
// (rows that are one token each of different sequences) that copy is x + (prev - x) * shift, prev = the row the sequence's previous token
// left in its tail (zeros at position 0), and the tail takes x.
struct PostArgs {
    float* res;
    void* act;
    const float *a, *b;
    int lda, ldb;
    float sa, sb;
    const float *y, *wgt, *shared;
    const int32_t* entry_slot;
    int top;
    const uint16_t* table;
    const int32_t* tokens;
    const uint16_t* w;
    float w_add, mult;
    int w_one, dim;
    float eps;
    const uint16_t* shift;
    float* tail;
    size_t tail_stride;
    const int32_t *pos, *slot;
    int cache;  // 1: dynamic shared memory holds the row of v, so its parts are read once
};
// V = 4: a thread takes four neighbouring entries per access (the row length and every row's address allow it), V = 1: one.
template <int V>
__device__ __forceinline__ void ldf(float (&v)[V], const float* p) {
    if (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x, v[1 % V] = t.y, v[2 % V] = t.z, v[3 % V] = t.w;
    } else {
        v[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void stf(float* p, const float (&v)[V]) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    else *p = v[0];
}
template <int V>
__device__ __forceinline__ void ldb(float (&v)[V], const uint16_t* p) {
    if (V == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        v[0] = bf16lo(t.x), v[1 % V] = bf16hi(t.x), v[2 % V] = bf16lo(t.y), v[3 % V] = bf16hi(t.y);
    } else {
        v[0] = bf16_bits_to_f32(*p);
    }
}
constexpr int kPostTop = 64;  // experts of a token whose places and weights are staged in shared memory
template <int SRC, typename TO, int V>
__global__ void kf_postnorm_kernel(PostArgs p) {
    extern __shared__ __align__(16) float sv[];
    __shared__ float red[32];
    __shared__ int s_slot[kPostTop];
    __shared__ float s_wgt[kPostTop];
    const int r = blockIdx.x;
    if (SRC == 1) {  // read once, so that the rows below are fetched side by side
        for (int j = threadIdx.x; j < min(p.top, kPostTop); j += blockDim.x)
            s_slot[j] = p.entry_slot[(size_t)r * p.top + j], s_wgt[j] = p.wgt[(size_t)r * p.top + j];
        __syncthreads();
    }
    auto val = [&](float (&v)[V], int i) {
        if (SRC == 0) {
            ldf<V>(v, p.a + (size_t)r * p.lda + i);
#pragma unroll
            for (int k = 0; k < V; k++) v[k] *= p.sa;
            if (p.b) {
                float t[V];
                ldf<V>(t, p.b + (size_t)r * p.ldb + i);
#pragma unroll
                for (int k = 0; k < V; k++) v[k] = fmaf(p.sb, t[k], v[k]);
            }
        } else if (SRC == 1) {
            float sh[V];
            if (p.shared) ldf<V>(sh, p.shared + (size_t)r * p.dim + i);
#pragma unroll
            for (int k = 0; k < V; k++) v[k] = 0.f;
            const int n = min(p.top, kPostTop);
#pragma unroll 4
            for (int j = 0; j < n; j++) {
                float t[V];
                ldf<V>(t, p.y + (size_t)s_slot[j] * p.dim + i);
#pragma unroll
                for (int k = 0; k < V; k++) v[k] = fmaf(s_wgt[j], t[k], v[k]);
            }
            for (int j = kPostTop; j < p.top; j++) {
                float t[V];
                ldf<V>(t, p.y + (size_t)p.entry_slot[(size_t)r * p.top + j] * p.dim + i);
#pragma unroll
                for (int k = 0; k < V; k++) v[k] = fmaf(p.wgt[(size_t)r * p.top + j], t[k], v[k]);
            }
            if (p.shared)
#pragma unroll
                for (int k = 0; k < V; k++) v[k] += sh[k];
        } else {
            ldb<V>(v, p.table + (size_t)p.tokens[r] * p.dim + i);
        }
    };
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < p.dim; i += blockDim.x * V) {
        float v[V];
        val(v, i);
        if (p.cache) stf<V>(sv + i, v);  // read back by the same thread
#pragma unroll
        for (int k = 0; k < V; k++) ss = fmaf(v[k], v[k], ss);
    }
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
    const float w1 = p.w_one ? p.w_add + bf16_bits_to_f32(p.w[0]) : 0.f;
    float* tail = p.shift ? p.tail + (size_t)p.slot[r] * p.tail_stride : nullptr;
    const bool first = p.shift && p.pos[r] == 0;
    for (int i = threadIdx.x * V; i < p.dim; i += blockDim.x * V) {
        float* q = p.res + (size_t)r * p.dim + i;
        float v[V], w[V], x[V];
        if (p.cache) ldf<V>(v, sv + i);
        else val(v, i);
        if (!p.w_one) ldb<V>(w, p.w + i);
        if (SRC != 2) ldf<V>(x, q);
#pragma unroll
        for (int k = 0; k < V; k++) {
            const float n = v[k] * s * (p.w_one ? w1 : p.w_add + w[k]);
            x[k] = SRC == 2 ? n : x[k] + p.mult * n;
        }
        stf<V>(q, x);
        if (p.shift) {
            float prev[V], sh[V];
            ldb<V>(sh, p.shift + i);
            ldf<V>(prev, tail + i);
            stf<V>(tail + i, x);
#pragma unroll
            for (int k = 0; k < V; k++) x[k] = fmaf((first ? 0.f : prev[k]) - x[k], sh[k], x[k]);
        }
        if (!p.act) continue;
        if (sizeof(TO) == 4) {
            stf<V>((float*)p.act + (size_t)r * p.dim + i, x);
        } else if (V == 4) {
            const uint2 o = make_uint2(pack_bf16x2(x[0], x[1 % V]), pack_bf16x2(x[2 % V], x[3 % V]));
            *reinterpret_cast<uint2*>((uint16_t*)p.act + (size_t)r * p.dim + i) = o;
        } else {
            ((uint16_t*)p.act)[(size_t)r * p.dim + i] = f32_to_bf16_bits(x[0]);
        }
    }
}
template <int SRC>
int launch_postnorm(kf_ctx* ctx, PostArgs& p, int act_f32, int rows) {
    const size_t smem = (size_t)p.dim * sizeof(float);
    p.cache = smem <= 32 * 1024 ? 1 : 0;
    const uintptr_t at = (uintptr_t)p.res | (uintptr_t)p.act | (uintptr_t)p.a | (uintptr_t)p.b | (uintptr_t)p.y | (uintptr_t)p.shared | (uintptr_t)p.tail;
    const uintptr_t at2 = (uintptr_t)p.table | (p.w_one ? 0 : (uintptr_t)p.w) | (uintptr_t)p.shift;
    const bool v4 = p.dim % 4 == 0 && p.lda % 4 == 0 && p.ldb % 4 == 0 && p.tail_stride % 4 == 0 && at % 16 == 0 && at2 % 8 == 0;
    const int threads = v4 ? std::min(rows <= 16 ? 512 : 256, std::max(64, (p.dim / 4 + 31) / 32 * 32)) : 256;
#define KF_PN(T, V) kf_postnorm_kernel<SRC, T, V><<<rows, threads, p.cache ? smem : 0, ctx->stream>>>(p)
    if (act_f32) v4 ? KF_PN(float, 4) : KF_PN(float, 1);
    else v4 ? KF_PN(uint16_t, 4) : KF_PN(uint16_t, 1);
#undef KF_PN
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// Token shift of a panel: out[t] = h[t] + (h[t-1] - h[t]) * w (w per entry), h[t-1] of a sequence's first row of this launch = its tail (zeros
// at position 0); the tail then takes the sequence's last row.  The block row of t = 0 does both, so nobody else touches the tail.
constexpr int kShiftRows = 4;
template <typename TO>
__global__ void kf_token_shift_kernel(TO* __restrict__ out, const float* __restrict__ h, int ldh, const uint16_t* __restrict__ w, float* __restrict__ tail,
                                      size_t tail_stride, const int32_t* __restrict__ pos, const int32_t* __restrict__ slot, int T, int dim) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.z;
    if (i >= dim) return;
    const float wi = bf16_bits_to_f32(w[i]);
    const int t0 = blockIdx.y * kShiftRows, t1 = min(T, t0 + kShiftRows);
    const float* hs = h + (size_t)seq * T * ldh;
    float prev;
    if (t0 == 0) {
        float* tl = tail + (size_t)slot[(size_t)seq * T] * tail_stride + i;
        prev = *tl;
        *tl  = hs[(size_t)(T - 1) * ldh + i];
    } else {
        prev = hs[(size_t)(t0 - 1) * ldh + i];
    }
    for (int t = t0; t < t1; t++) {
        const float x = hs[(size_t)t * ldh + i];
        if (pos[(size_t)seq * T + t] == 0) prev = 0.f;
        const float o = fmaf(prev - x, wi, x);
        if (sizeof(TO) == 2) ((uint16_t*)out)[((size_t)seq * T + t) * dim + i] = f32_to_bf16_bits(o);
        else ((float*)out)[((size_t)seq * T + t) * dim + i] = o;
        prev = x;
    }
}

// Pre-norm residual step of one row:  res += a + b + vec (each optional);  act_out = res / sqrt(mean(res^2) + eps) * w in the activation
// type (what the next sublayer's matmul reads; w NULL: only the sum).
template <typename TO>
__global__ void __launch_bounds__(256) kf_residual_prenorm_kernel(float* __restrict__ res, TO* __restrict__ act_out, const float* __restrict__ a, int lda,
                                                                  const float* __restrict__ b, int ldb, const uint16_t* __restrict__ vec,
                                                                  const uint16_t* __restrict__ w, int dim, float eps) {
    __shared__ float red[32];
    const int r = blockIdx.x;
    float* xr = res + (size_t)r * dim;
    float ss = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float v = xr[i];
        if (a) v += a[(size_t)r * lda + i];
        if (b) v += b[(size_t)r * ldb + i];
        if (vec) v += bf16_bits_to_f32(vec[i]);
        if (a || b || vec) xr[i] = v;
        ss = fmaf(v, v, ss);
    }
    if (!w) return;
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)dim + eps);
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {  // a thread re-reads what it wrote itself
        const float v = xr[i] * s * bf16_bits_to_f32(w[i]);
        if (sizeof(TO) == 2) ((uint16_t*)act_out)[(size_t)r * dim + i] = f32_to_bf16_bits(v);
        else ((float*)act_out)[(size_t)r * dim + i] = v;
    }
}
// ---- steps of a stack whose norm is a saturating function of each entry, n(x) = tanh(alpha x) w + b: no statistics over the row, so every
// step between two matmuls is entry by entry and any number of CTAs can share a row ------------------------------------------------------
// Residual step:  x = res + scale * v (scale per entry, or none),  out = n(x) in the activation type;  v is
//   SRC 0: a float row (NULL: nothing is added);  SRC 1: sum_j wgt[j] * y[entry_slot[j]], where an entry without a slot (-1) stands for the
//   token's row of `pass`;  SRC 2: a row of a bf16 table, which starts the stream (res = the row).
// row_idx: rows to take, res is then left alone.  mu (rows that are one token each of different sequences): instead of n(x), n_mix rows
// h + (h' - h) mu_s one plane apart, h = n(x), h' = the row the sequence's previous token left in its tail (zeros at position 0); the tail
// takes h.  `pass` may be `out`: a thread reads its own entries first.
struct DytArgs {
    float* res;
    int dim;
    const uint16_t *scale, *w, *b, *alpha;
    void* out;
    const int32_t* row_idx;
    const uint16_t* mu;
    int n_mix;
    size_t plane;
    float* tail;
    size_t tail_stride;
    const int32_t *pos, *slot;
    const float* a;
    int lda;
    const float *y, *wgt;
    const int32_t* entry_slot;
    const void* pass;
    int top;
    const uint16_t* table;
    const int32_t* tokens;
    int T;  // token mix: tokens per sequence
};
template <typename TO, int V>
__device__ __forceinline__ void st_act(TO* p, const float (&v)[V]) {
    if (sizeof(TO) == 4) {
        stf<V>((float*)p, v);
    } else if (V == 4) {
        *reinterpret_cast<uint2*>((uint16_t*)p) = make_uint2(pack_bf16x2(v[0], v[1 % V]), pack_bf16x2(v[2 % V], v[3 % V]));
    } else {
        *(uint16_t*)p = f32_to_bf16_bits(v[0]);
    }
}
template <typename TO, int V>
__device__ __forceinline__ void ld_actv(float (&v)[V], const TO* p) {
    if (sizeof(TO) == 4) ldf<V>(v, (const float*)p);
    else ldb<V>(v, (const uint16_t*)p);
}
template <int SRC, typename TO, int V>
__global__ void __launch_bounds__(128) kf_dyt_step_kernel(DytArgs p) {
    const int r = blockIdx.y, i = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= p.dim) return;
    const int src = p.row_idx ? p.row_idx[r] : r;
    float v[V], x[V], s[V], w[V], b[V], d[V], h[V];
    // everything that does not hang on the experts' places is fetched ahead of them
#pragma unroll
    for (int k = 0; k < V; k++) v[k] = 0.f, s[k] = 1.f;
    if (SRC != 2 && p.scale) ldb<V>(s, p.scale + i);
    float al = 0.f;
    if (p.w) ldb<V>(w, p.w + i), ldb<V>(b, p.b + i), al = bf16_bits_to_f32(*p.alpha);
    float* tail = p.mu ? p.tail + (size_t)p.slot[r] * p.tail_stride + i : nullptr;
    const bool first = p.mu && p.pos[r] == 0;
    if (p.mu) ldf<V>(d, tail);
    if (SRC != 2) ldf<V>(x, p.res + (size_t)src * p.dim + i);
    if (SRC == 0) {
        if (p.a) ldf<V>(v, p.a + (size_t)src * p.lda + i);
    } else if (SRC == 1) {
        const int32_t* es = p.entry_slot + (size_t)src * p.top;
        const float* wg   = p.wgt + (size_t)src * p.top;
        float own[V];
        ld_actv<TO, V>(own, (const TO*)p.pass + (size_t)src * p.dim + i);
        for (int j0 = 0; j0 < p.top; j0 += 8) {  // eight experts at a time: their places, then their rows, are fetched together
            int sl[8];
            float wj[8], t[8][V];
#pragma unroll
            for (int j = 0; j < 8; j++) sl[j] = j0 + j < p.top ? es[j0 + j] : -1, wj[j] = j0 + j < p.top ? wg[j0 + j] : 0.f;
#pragma unroll
            for (int j = 0; j < 8; j++)
                if (sl[j] >= 0) ldf<V>(t[j], p.y + (size_t)sl[j] * p.dim + i);
#pragma unroll
            for (int j = 0; j < 8; j++)
#pragma unroll
                for (int k = 0; k < V; k++) v[k] = fmaf(wj[j], sl[j] >= 0 ? t[j][k] : own[k], v[k]);
        }
    } else {
        ldb<V>(x, p.table + (size_t)p.tokens[src] * p.dim + i);
    }
    if (SRC != 2) {
#pragma unroll
        for (int k = 0; k < V; k++) x[k] = fmaf(s[k], v[k], x[k]);
    }
    if (!p.row_idx) stf<V>(p.res + (size_t)r * p.dim + i, x);
    if (!p.w) return;
#pragma unroll
    for (int k = 0; k < V; k++) h[k] = fmaf(tanhf(al * x[k]), w[k], b[k]);
    if (!p.mu) {
        st_act<TO, V>((TO*)p.out + (size_t)r * p.dim + i, h);
        return;
    }
    stf<V>(tail, h);
#pragma unroll
    for (int k = 0; k < V; k++) d[k] = (first ? 0.f : d[k]) - h[k];
    for (int q = 0; q < p.n_mix; q++) {
        float m[V], o[V];
        ldb<V>(m, p.mu + (size_t)q * p.dim + i);
#pragma unroll
        for (int k = 0; k < V; k++) o[k] = fmaf(d[k], m[k], h[k]);
        st_act<TO, V>((TO*)p.out + (size_t)q * p.plane + (size_t)r * p.dim + i, o);
    }
}
// The mixes of a panel (rows seq * T + t of the finished stream): a thread walks kShiftRows tokens of its entries and keeps the last h.  The
// block row of t = 0 reads the tail and leaves the sequence's last h there, so nobody else touches it.
template <typename TO, int V>
__global__ void __launch_bounds__(128) kf_dyt_mix_kernel(DytArgs p) {
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * V, seq = blockIdx.z, T = p.T;
    if (i >= p.dim) return;
    const int t0 = blockIdx.y * kShiftRows, t1 = min(T, t0 + kShiftRows);
    const float al = bf16_bits_to_f32(*p.alpha);
    float w[V], b[V], prev[V];
    ldb<V>(w, p.w + i), ldb<V>(b, p.b + i);
    const float* xs = p.res + (size_t)seq * T * p.dim + i;
    auto norm = [&](float (&h)[V], int t) {
        ldf<V>(h, xs + (size_t)t * p.dim);
#pragma unroll
        for (int k = 0; k < V; k++) h[k] = fmaf(tanhf(al * h[k]), w[k], b[k]);
    };
    if (t0 == 0) {
        float* tl = p.tail + (size_t)p.slot[(size_t)seq * T] * p.tail_stride + i;
        float last[V];
        ldf<V>(prev, tl);
        norm(last, T - 1);
        stf<V>(tl, last);
    } else {
        norm(prev, t0 - 1);
    }
    for (int t = t0; t < t1; t++) {
        float h[V], d[V];
        norm(h, t);
        const bool first = p.pos[(size_t)seq * T + t] == 0;
#pragma unroll
        for (int k = 0; k < V; k++) d[k] = (first ? 0.f : prev[k]) - h[k], prev[k] = h[k];
        for (int q = 0; q < p.n_mix; q++) {
            float m[V], o[V];
            ldb<V>(m, p.mu + (size_t)q * p.dim + i);
#pragma unroll
            for (int k = 0; k < V; k++) o[k] = fmaf(d[k], m[k], h[k]);
            st_act<TO, V>((TO*)p.out + (size_t)q * p.plane + ((size_t)seq * T + t) * p.dim + i, o);
        }
    }
}
bool dyt_args(DytArgs& p, const kf_dyt_step* s) {
    p.res = s->res, p.dim = s->dim, p.scale = (const uint16_t*)s->scale_bf16, p.w = (const uint16_t*)s->w_bf16, p.b = (const uint16_t*)s->b_bf16;
    p.alpha = (const uint16_t*)s->alpha_bf16, p.out = s->out, p.row_idx = s->row_idx, p.mu = (const uint16_t*)s->mu_bf16, p.n_mix = s->n_mix, p.plane = s->plane;
    p.tail = s->tail, p.tail_stride = s->tail_stride, p.pos = s->pos, p.slot = s->slot;
    if (!s->res || s->rows < 1 || s->rows > 65535 || s->dim < 1 || (s->w_bf16 && (!s->b_bf16 || !s->alpha_bf16 || !s->out))) return false;
    return !s->mu_bf16 || (s->w_bf16 && s->n_mix >= 1 && s->plane >= (size_t)s->rows * s->dim && s->tail && s->tail_stride >= (size_t)s->dim && s->pos && s->slot && !s->row_idx);
}
// four entries per access: row length and every row's address allow it
bool dyt_vec(const DytArgs& p) {
    const uintptr_t at16 = (uintptr_t)p.res | (uintptr_t)p.out | (uintptr_t)p.a | (uintptr_t)p.y | (uintptr_t)p.tail | (uintptr_t)p.pass;
    const uintptr_t at8  = (uintptr_t)p.scale | (uintptr_t)p.w | (uintptr_t)p.b | (uintptr_t)p.mu | (uintptr_t)p.table;
    return p.dim % 4 == 0 && p.lda % 4 == 0 && p.plane % 4 == 0 && p.tail_stride % 4 == 0 && at16 % 16 == 0 && at8 % 8 == 0;
}
template <int SRC>
int launch_dyt(kf_ctx* ctx, const DytArgs& p, int out_f32, int rows) {
    const int v = dyt_vec(p) ? 4 : 1;
    const dim3 grid((p.dim + 128 * v - 1) / (128 * v), rows);
#define KF_DYT(T, V) kf_dyt_step_kernel<SRC, T, V><<<grid, 128, 0, ctx->stream>>>(p)
    if (out_f32) v == 4 ? KF_DYT(float, 4) : KF_DYT(float, 1);
    else v == 4 ? KF_DYT(uint16_t, 4) : KF_DYT(uint16_t, 1);
#undef KF_DYT
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// out = g' * sigmoid(alpha * g') * (u' + shift),  g' = min(g, limit), u' = clamp(u, -limit, limit)  (limit <= 0: not clamped)
template <typename TO>
__global__ void kf_glu_clamped_kernel(TO* __restrict__ out, int ldo, const float* __restrict__ g, int ldg, const float* __restrict__ u, int ldu, int cols,
                                      float limit, float alpha, float shift) {
    const int r = blockIdx.y;
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < cols; c += gridDim.x * blockDim.x) {
        float gv = g[(size_t)r * ldg + c], uv = u[(size_t)r * ldu + c];
        if (limit > 0.f) gv = fminf(gv, limit), uv = fminf(fmaxf(uv, -limit), limit);
        const float v = gv * sigmoid_f(alpha * gv) * (uv + shift);
        if (sizeof(TO) == 2) ((uint16_t*)out)[(size_t)r * ldo + c] = f32_to_bf16_bits(v);
        else ((float*)out)[(size_t)r * ldo + c] = v;
    }
}
__global__ void kf_scale_f32_kernel(float* __restrict__ x, size_t n, float s) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] *= s;
}

__global__ void kf_f32_to_bf16_kernel(uint16_t* __restrict__ out, const float* __restrict__ in, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = f32_to_bf16_bits(in[i]);
}

// ---- mixture of experts ---------------------------------------------------------------------------------------------------
// How a token's experts are chosen and weighted.  kind 0: arg-max over logits (+ bias), weights from a softmax (the kernels' `full` flag).
// kind 1: scores s = sigmoid(logit); the choice runs over s + bias; the experts form `groups` equal contiguous groups, a group is ranked
// by the sum of its top-2 choice values and only the `keep` best groups can be chosen from; weights = scale * s of the chosen, not
// renormalised.
// kind 2: scores s = softmax(logits) over all outputs; choice over s + bias inside the `keep` best groups as in kind 1, but a group is ranked by
// its LARGEST choice value; weights = s of the chosen over (their sum + 1e-20).
// The last `pass` outputs of the router (kind 2) are no experts: an entry that goes to one takes no slot (entry_slot -1), the combination reads
// the sublayer's input for it.
struct RouteMode {
    int kind, groups, keep;
    float scale;
    int pass;
};
constexpr int kRouteGroups = 64;
// one warp routes one token in kinds 1 and 2.  taken: the token's chosen experts so far (shared or global memory, written by lane 0).
// Up to 32 * kRouteCache outputs: a lane keeps the scores and choice values of its outputs (lane, lane + 32, ...) in registers and a mask of
// those taken; more outputs: they are formed again whenever they are looked at.
constexpr int kRouteCache = 8;
__device__ __forceinline__ unsigned route_key(float v) {  // unsigned order = float order
    const unsigned u = __float_as_uint(v);
    return (u & 0x80000000u) ? ~u : u | 0x80000000u;
}
// KEEP (CACHED, top <= 32): nothing is written; lane j returns the j-th choice and its weight, every lane the mask of its own outputs taken.
struct RouteKept {
    int e;
    float w;
    unsigned picked;
};
template <bool CACHED, bool KEEP = false>
__device__ __forceinline__ RouteKept route_grouped_body(int* taken, int32_t* idx, float* __restrict__ wgt, const float* __restrict__ lg,
                                                   const uint16_t* __restrict__ bias, int E, int top, const RouteMode md, int lane) {
    const int per = E / md.groups, n = CACHED ? kRouteCache : (E + 31) / 32;
    float sc[CACHED ? kRouteCache : 1], cv[CACHED ? kRouteCache : 1];
    float mx = 0.f, inv = 1.f;
    auto shift_of = [&](int e) { return bias ? bf16_bits_to_f32(bias[e]) : 0.f; };
    if (CACHED) {
#pragma unroll
        for (int i = 0; i < kRouteCache; i++) {
            const int e = lane + 32 * i;
            sc[i] = e < E ? lg[e] : -INFINITY, cv[i] = e < E ? shift_of(e) : 0.f;
        }
    }
    if (md.kind == 2) {
        mx = -INFINITY;
        float d = 0.f;
        if (CACHED) {
#pragma unroll
            for (int i = 0; i < kRouteCache; i++) mx = fmaxf(mx, sc[i]);
            mx = warp_max(mx);
#pragma unroll
            for (int i = 0; i < kRouteCache; i++) sc[i] = 32 * i < E ? expf(sc[i] - mx) : 0.f, d += sc[i];
        } else {
            for (int e = lane; e < E; e += 32) mx = fmaxf(mx, lg[e]);
            mx = warp_max(mx);
            for (int e = lane; e < E; e += 32) d += expf(lg[e] - mx);
        }
        inv = 1.f / warp_sum(d);
    }
    if (CACHED) {
#pragma unroll
        for (int i = 0; i < kRouteCache; i++)
            if (32 * i < E) sc[i] = md.kind == 2 ? sc[i] * inv : sigmoid_f(sc[i]), cv[i] += sc[i];
    }
    auto score  = [&](int e) { return md.kind == 2 ? expf(lg[e] - mx) * inv : sigmoid_f(lg[e]); };
    auto choice = [&](int i, int e) { return CACHED ? cv[CACHED ? i : 0] : score(e) + shift_of(e); };
    unsigned long long kept = ~0ull;
    if (md.keep < md.groups) {
        kept = 0;
        // lane g & 31 keeps the rank keys of groups g and g + 32, found by all lanes together
        unsigned gs0 = 0, gs1 = 0;
        for (int g = 0; g < md.groups; g++) {
            float a = -INFINITY, b = -INFINITY;  // largest, second largest of this lane's share
#pragma unroll CACHED ? kRouteCache : 1
            for (int i = 0; i < n; i++) {
                const int e = lane + 32 * i;
                if (e < g * per || e >= (g + 1) * per) continue;
                const float v = choice(i, e);
                if (v > a) b = a, a = v;
                else if (v > b) b = v;
            }
            float rank;
            if (md.kind == 1 && per > 1) {
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
                    const float hi = fmaxf(a, oa), lo = fmaxf(fminf(a, oa), fmaxf(b, ob));
                    a = hi, b = lo;
                }
                rank = a + b;
            } else {
                rank = warp_max(a);
            }
            if (lane == (g & 31)) (g < 32 ? gs0 : gs1) = route_key(rank);
        }
        for (int r = 0; r < md.keep; r++) {
            const bool o0 = lane < md.groups && !((kept >> lane) & 1ull), o1 = lane + 32 < md.groups && !((kept >> (lane + 32)) & 1ull);
            const unsigned best = __reduce_max_sync(0xffffffffu, max(o0 ? gs0 : 0u, o1 ? gs1 : 0u));
            const unsigned at = o0 && gs0 == best ? lane : o1 && gs1 == best ? lane + 32 : 0xffffffffu;
            const unsigned bi = __reduce_min_sync(0xffffffffu, at);  // ties to the lower index
            if (bi < 64u) kept |= 1ull << bi;
        }
    }
    float sum = 0.f;
    RouteKept mine = {0, 0.f, 0u};
    unsigned used = 0;  // CACHED: this lane's outputs that are taken or closed
    if (CACHED) {
#pragma unroll
        for (int i = 0; i < kRouteCache; i++) {
            const int e = lane + 32 * i;
            if (e >= E || !((kept >> min(63, e / per)) & 1ull)) used |= 1u << i;
        }
    }
    for (int j = 0; j < top; j++) {
        unsigned bk = 0, bi = 0xffffffffu;
        float bs = 0.f;
#pragma unroll CACHED ? kRouteCache : 1
        for (int i = 0; i < n; i++) {
            const int e = lane + 32 * i;
            if (CACHED) {
                if ((used >> i) & 1u) continue;
            } else {
                if (e >= E || !((kept >> min(63, e / per)) & 1ull)) continue;
                bool was = false;
                for (int q = 0; q < j; q++) was = was || taken[q] == e;
                if (was) continue;
            }
            const unsigned k = route_key(choice(i, e));
            if (bi == 0xffffffffu || k > bk) bk = k, bi = e, bs = CACHED ? sc[CACHED ? i : 0] : 0.f;
        }
        const unsigned best = __reduce_max_sync(0xffffffffu, bk);
        const unsigned win  = __reduce_min_sync(0xffffffffu, bk == best ? bi : 0xffffffffu);
        const int w = (int)min(win, (unsigned)(E - 1));
        if (CACHED) {
            bs = __shfl_sync(0xffffffffu, bs, w & 31);
            if (lane == (w & 31)) used |= 1u << (w >> 5), mine.picked |= 1u << (w >> 5);
        } else {
            bs = score(w);
        }
        sum += bs;
        if (KEEP) {
            if (lane == j) mine.e = w, mine.w = md.kind == 2 ? bs : md.scale * bs;
            continue;
        }
        if (lane == 0) taken[j] = w, idx[j] = w, wgt[j] = md.kind == 2 ? bs : md.scale * bs;
        __syncwarp();
    }
    if (KEEP && md.kind == 2) mine.w /= sum + 1e-20f;
    if (!KEEP && md.kind == 2 && lane == 0)
        for (int j = 0; j < top; j++) wgt[j] /= sum + 1e-20f;
    return mine;
}
// One token (decoding) in kinds 1 and 2: choice and dispatch tables by ONE warp without shared memory.  Every expert holds at most one entry, so
// an entry's slot is the number of chosen experts before its own.
__global__ void __launch_bounds__(32) kf_moe_route_one_kernel(int32_t* __restrict__ idx, float* __restrict__ wgt, int32_t* __restrict__ offsets,
                                                              int32_t* __restrict__ entry_slot, int32_t* __restrict__ slot_row, int32_t* __restrict__ slot_group,
                                                              const float* __restrict__ logits, const uint16_t* __restrict__ bias, int E, int top, const RouteMode md) {
    const int lane = threadIdx.x, X = E - md.pass;
    const RouteKept r = route_grouped_body<true, true>(nullptr, nullptr, nullptr, logits, bias, E, top, md, lane);
    const bool real = lane < top && r.e < X;
    const int n = __popc(__ballot_sync(0xffffffffu, real));
    int sl = 0;
    for (int j = 0; j < top; j++) sl += __shfl_sync(0xffffffffu, r.e, j) < r.e;
    int before = 0;
#pragma unroll
    for (int i = 0; i <= kRouteCache; i++) {
        const unsigned word = i < kRouteCache ? __ballot_sync(0xffffffffu, (r.picked >> i) & 1u) : 0u;
        if (32 * i + lane <= X) offsets[32 * i + lane] = before + __popc(word & ((1u << lane) - 1));
        before += __popc(word);
    }
    if (lane >= top) return;
    idx[lane] = r.e, wgt[lane] = r.w, entry_slot[lane] = real ? sl : -1;
    if (real) slot_row[sl] = 0, slot_group[sl] = r.e;
    if (lane >= n) slot_row[lane] = 0, slot_group[lane] = -1;
}
__device__ __forceinline__ void route_grouped_warp(int* taken, int32_t* idx, float* __restrict__ wgt, const float* __restrict__ lg,
                                                   const uint16_t* __restrict__ bias, int E, int top, const RouteMode md, int lane) {
    if (E <= 32 * kRouteCache) route_grouped_body<true>(taken, idx, wgt, lg, bias, E, top, md, lane);
    else route_grouped_body<false>(taken, idx, wgt, lg, bias, E, top, md, lane);
}
// one warp per token: `top` rounds of arg-max over the E router logits (+ bias), ties to the lower index; weights = softmax over the
// chosen logits only, or (full) the chosen entries of the softmax over ALL experts, not renormalised.  All in fp32.
__global__ void __launch_bounds__(128) kf_moe_route_kernel(int32_t* __restrict__ idx, float* __restrict__ wgt, const float* __restrict__ logits, int ldl,
                                                           const uint16_t* __restrict__ bias, int M, int E, int top, int full, const RouteMode md) {
    const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (m >= M) return;
    const float* lg = logits + (size_t)m * ldl;
    if (md.kind) {
        route_grouped_warp(idx + (size_t)m * top, idx + (size_t)m * top, wgt + (size_t)m * top, lg, bias, E, top, md, lane);
        return;
    }
    float first = 0.f, den = 0.f;
    for (int j = 0; j < top; j++) {
        float best = -INFINITY;
        int bi     = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            bool taken = false;
            for (int q = 0; q < j; q++) taken = taken || idx[(size_t)m * top + q] == e;
            if (taken) continue;
            const float v = lg[e] + (bias ? bf16_bits_to_f32(bias[e]) : 0.f);
            if (v > best || (v == best && e < bi)) best = v, bi = e;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi   = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) best = ob, bi = oi;
        }
        if (j == 0) first = best;
        const float p = expf(best - first);
        den += p;
        if (lane == 0) idx[(size_t)m * top + j] = bi, wgt[(size_t)m * top + j] = p;
        __syncwarp();
    }
    if (full) {  // the denominator runs over every expert (first = the largest logit)
        float d = 0.f;
        for (int e = lane; e < E; e += 32) d += expf(lg[e] + (bias ? bf16_bits_to_f32(bias[e]) : 0.f) - first);
        den = warp_sum(d);
    }
    if (lane < top) {
        for (int j = lane; j < top; j += 32) wgt[(size_t)m * top + j] /= den;
    }
}
// The dispatch tables of a few entries by ONE block of 256 threads: entry i = (token i / top, choice i % top) goes to expert sidx[i]; thread i
// ranks its entry among the earlier ones of its expert, the lanes of warp 0 count one expert each and scan the counts.  Entries of outputs
// beyond the E experts take no slot; the slots that stay free are marked with group -1.
constexpr int kRouteSmall = 256;
__device__ __forceinline__ void dispatch_small(const int* sidx, int* srank, int n, int E, int top, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row,
                                               int32_t* slot_group) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        int r = 0;
        for (int j = 0; j < i; j++) r += sidx[j] == sidx[i];
        srank[i] = r;
    }
    __syncthreads();
    if (warp == 0) {  // offsets: lane l counts the entries of expert e0 + l, a scan over the lanes places them behind the experts before
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane;
            int c = 0;
            for (int j = 0; j < n; j++) c += sidx[j] == e && e < E;  // outputs beyond the experts take no slot
            int incl = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            if (e < E) offsets[e] = base + incl - c;
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) offsets[E] = base;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        if (i >= offsets[E]) slot_row[i] = 0, slot_group[i] = -1;
        const int e = sidx[i];
        if (e >= E) {
            entry_slot[i] = -1;
            continue;
        }
        const int sl = offsets[e] + srank[i];
        entry_slot[i] = sl, slot_row[sl] = i / top, slot_group[sl] = e;
    }
}
// few tokens (decode): routing and the dispatch tables in ONE block
__global__ void __launch_bounds__(256) kf_moe_route_small_kernel(int32_t* __restrict__ idx, float* __restrict__ wgt, int32_t* __restrict__ offsets,
                                                                 int32_t* __restrict__ entry_slot, int32_t* __restrict__ slot_row,
                                                                 int32_t* __restrict__ slot_group, const float* __restrict__ logits, int ldl,
                                                                 const uint16_t* __restrict__ bias, int M, int E, int top, int full, const RouteMode md) {
    __shared__ int sidx[kRouteSmall];
    __shared__ int srank[kRouteSmall];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = M * top;
    for (int m = warp; m < M; m += 8) {
        const float* lg = logits + (size_t)m * ldl;
        if (md.kind) {
            route_grouped_warp(sidx + m * top, idx + (size_t)m * top, wgt + (size_t)m * top, lg, bias, E, top, md, lane);
            continue;
        }
        float first = 0.f, den = 0.f;
        for (int j = 0; j < top; j++) {
            float best = -INFINITY;
            int bi     = 0x7fffffff;
            for (int e = lane; e < E; e += 32) {
                bool taken = false;
                for (int q = 0; q < j; q++) taken = taken || sidx[m * top + q] == e;
                if (taken) continue;
                const float v = lg[e] + (bias ? bf16_bits_to_f32(bias[e]) : 0.f);
                if (v > best || (v == best && e < bi)) best = v, bi = e;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ob = __shfl_xor_sync(0xffffffffu, best, o);
                const int oi   = __shfl_xor_sync(0xffffffffu, bi, o);
                if (ob > best || (ob == best && oi < bi)) best = ob, bi = oi;
            }
            if (j == 0) first = best;
            const float p = expf(best - first);
            den += p;
            if (lane == 0) sidx[m * top + j] = bi, idx[(size_t)m * top + j] = bi, wgt[(size_t)m * top + j] = p;
            __syncwarp();
        }
        if (full) {
            float d = 0.f;
            for (int e = lane; e < E; e += 32) d += expf(lg[e] + (bias ? bf16_bits_to_f32(bias[e]) : 0.f) - first);
            den = warp_sum(d);
        }
        for (int j = lane; j < top; j += 32) wgt[(size_t)m * top + j] /= den;
    }
    dispatch_small(sidx, srank, n, E - md.pass, top, offsets, entry_slot, slot_row, slot_group);
}
// one block per expert: the entries (token, choice) routed to it, ranked in entry order (ballot + popc compaction)
__device__ __forceinline__ void rank_expert(int32_t* rank, int32_t* count, const int32_t* idx, int n, int e) {
    __shared__ int wsum[8];
    __shared__ int base;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (threadIdx.x == 0) base = 0;
    __syncthreads();
    for (int i0 = 0; i0 < n; i0 += 256) {
        const int i    = i0 + threadIdx.x;
        const bool hit = i < n && idx[i] == e;
        const unsigned b = __ballot_sync(0xffffffffu, hit);
        if (lane == 0) wsum[warp] = __popc(b);
        __syncthreads();
        int before = base;
        for (int q = 0; q < warp; q++) before += wsum[q];
        if (hit) rank[i] = before + __popc(b & ((1u << lane) - 1));
        __syncthreads();
        if (threadIdx.x == 0) {
            int t = 0;
            for (int q = 0; q < 8; q++) t += wsum[q];
            base += t;
        }
        __syncthreads();
    }
    if (threadIdx.x == 0) count[e] = base;
}
__global__ void __launch_bounds__(256) kf_moe_rank_kernel(int32_t* __restrict__ rank, int32_t* __restrict__ count, const int32_t* __restrict__ idx, int n) {
    rank_expert(rank, count, idx, n, blockIdx.x);
}
// offsets = exclusive scan of the counts (one thread: E is small); then each entry learns its slot
__global__ void kf_moe_offsets_kernel(int32_t* __restrict__ offsets, const int32_t* __restrict__ count, int E) {
    if (threadIdx.x == 0 && blockIdx.x == 0) {
        int s = 0;
        for (int e = 0; e < E; e++) offsets[e] = s, s += count[e];
        offsets[E] = s;
    }
}
__global__ void kf_moe_slots_kernel(int32_t* __restrict__ entry_slot, int32_t* __restrict__ slot_row, int32_t* __restrict__ slot_group,
                                    const int32_t* __restrict__ idx, const int32_t* __restrict__ rank, const int32_t* __restrict__ offsets, int n, int top,
                                    int E) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    if (i >= offsets[E]) slot_row[i] = 0, slot_group[i] = -1;  // no entry has this slot
    const int e = idx[i];
    if (e >= E) {
        entry_slot[i] = -1;
        return;
    }
    const int s = offsets[e] + rank[i];
    entry_slot[i] = s, slot_row[s] = i / top, slot_group[s] = e;
}
// Routing from a table of token ids: row tokens[m] names the token's `top` experts, each with weight 1 / top -- no logits.  It depends on
// the token ids alone, so ONE launch fills the tables of several layers (blockIdx.y / .x picks the layer).
__device__ __forceinline__ int table_expert(const kf_table_route& r, int token, int j) {
    return (int)min((unsigned)r.table[(size_t)token * r.top + j], (unsigned)(r.experts - 1));  // ids are checked when the table is loaded
}
__global__ void __launch_bounds__(256) kf_moe_table_small_kernel(const kf_table_route* __restrict__ routes, const int32_t* __restrict__ tokens, int M) {
    __shared__ int sidx[kRouteSmall];
    __shared__ int srank[kRouteSmall];
    const kf_table_route r = routes[blockIdx.x];
    const int n = M * r.top;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const int e = table_expert(r, tokens[i / r.top], i % r.top);
        sidx[i] = e, r.idx[i] = e, r.wgt[i] = 1.f / (float)r.top;
    }
    dispatch_small(sidx, srank, n, r.experts, r.top, r.offsets, r.entry_slot, r.slot_row, r.slot_group);
}
__global__ void kf_moe_table_idx_kernel(const kf_table_route* __restrict__ routes, const int32_t* __restrict__ tokens, int M) {
    const kf_table_route r = routes[blockIdx.y];
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < M * r.top) r.idx[i] = table_expert(r, tokens[i / r.top], i % r.top), r.wgt[i] = 1.f / (float)r.top;
}
__global__ void __launch_bounds__(256) kf_moe_table_rank_kernel(const kf_table_route* __restrict__ routes, int M) {
    const kf_table_route r = routes[blockIdx.y];
    if (blockIdx.x < r.experts) rank_expert(r.work, r.work + M * r.top, r.idx, M * r.top, blockIdx.x);
}
__global__ void kf_moe_table_slots_kernel(const kf_table_route* __restrict__ routes, int M) {  // offsets: every block scans the few counts itself
    extern __shared__ int soff[];
    const kf_table_route r = routes[blockIdx.y];
    const int n = M * r.top, E = r.experts, lane = threadIdx.x & 31;
    const int32_t* count = r.work + n;
    if (threadIdx.x < 32) {
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane, c = e < E ? count[e] : 0;
            int incl = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            if (e < E) soff[e] = base + incl - c;
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
    }
    __syncthreads();
    if (blockIdx.x == 0)
        for (int e = threadIdx.x; e <= E; e += blockDim.x) r.offsets[e] = e < E ? soff[e] : n;
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int e = r.idx[i], sl = soff[e] + r.work[i];
    r.entry_slot[i] = sl, r.slot_row[sl] = i / r.top, r.slot_group[sl] = e;
}
// out[m] = sum_j wgt[m][j] * y[slot(m, j)]  (+ sigmoid(sg[m]) * shared[m]), choices added in their routing order
__global__ void kf_moe_combine_kernel(float* __restrict__ out, const float* __restrict__ y, const int32_t* __restrict__ entry_slot,
                                      const float* __restrict__ wgt, const float* __restrict__ shared, const float* __restrict__ sg, int ldsg, int dim, int top,
                                      int accumulate) {
    const int m = blockIdx.x;
    const float gate = shared ? (sg ? sigmoid_f(sg[(size_t)m * ldsg]) : 1.f) : 0.f;
    for (int d = threadIdx.x; d < dim; d += blockDim.x) {
        float s = 0.f;
        for (int j = 0; j < top; j++) s = fmaf(wgt[(size_t)m * top + j], y[(size_t)entry_slot[(size_t)m * top + j] * dim + d], s);
        if (shared) s = fmaf(gate, shared[(size_t)m * dim + d], s);
        out[(size_t)m * dim + d] = accumulate ? out[(size_t)m * dim + d] + s : s;
    }
}
}  // namespace

// out[m] = scale * W[token[m]] as floats; out2 (optional) receives a second copy
extern "C" int kf_embed_f32_scaled(kf_ctx* ctx, float* out, float* out2, const kf_tensor_desc* w, const int32_t* tokens_dev, int M, float scale) {
    if (!ctx || !out || !w || !tokens_dev) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, w->type == KF_T_BF16 && M >= 1, "bf16 table");
    kf_embed_f32_kernel<<<M, 256, 0, ctx->stream>>>(out, out2, (const uint16_t*)w->data_dev, tokens_dev, w->cols, scale);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_embed_f32(kf_ctx* ctx, float* out, const kf_tensor_desc* w, const int32_t* tokens_dev, int M) {
    return kf_embed_f32_scaled(ctx, out, nullptr, w, tokens_dev, M, 1.f);
}
// out[rows][ldo] = act(in[rows][ldi] + bias) (* mul); act 0: none, 1: gelu (tanh form), 2: relu squared, 3: silu, 4: relu; out_kind 0: bf16 bits,
// 1: float, 2: float out += result.  bias: bf16 [cols] or NULL; mul: float [rows][ldm] or NULL.
extern "C" int kf_bias_act(kf_ctx* ctx, void* out, int out_kind, int ldo, const float* in, int ldi, const void* bias_bf16, int act, const float* mul, int ldm,
                           int rows, int cols) {
    if (!ctx || !out || !in) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && cols >= 1 && act >= 0 && act <= 4 && out_kind >= 0 && out_kind <= 2, "act / out kind");
    dim3 grid(std::min(64, (cols + 255) / 256), rows);
    const uint16_t* b = (const uint16_t*)bias_bf16;
#define KF_BA(A, O) kf_bias_act_kernel<A, O><<<grid, 256, 0, ctx->stream>>>(out, ldo, in, ldi, b, mul, ldm, cols)
#define KF_BA_O(A) (out_kind == 0 ? KF_BA(A, 0) : out_kind == 1 ? KF_BA(A, 1) : KF_BA(A, 2))
    if (act == 0) KF_BA_O(0);
    else if (act == 1) KF_BA_O(1);
    else if (act == 2) KF_BA_O(2);
    else if (act == 3) KF_BA_O(3);
    else KF_BA_O(4);
#undef KF_BA_O
#undef KF_BA
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_token_gate(kf_ctx* ctx, void* out, int out_f32, int ldo, const float* in, int ldi, const void* table_bf16, int ldt, int c0,
                             const int32_t* tokens_dev, int rows, int cols) {
    if (!ctx || !out || !in || !table_bf16 || !tokens_dev) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && cols >= 1 && c0 >= 0 && c0 + cols <= ldt, "slice inside the table row");
    if (out_f32) kf_token_gate_kernel<float><<<rows, 128, 0, ctx->stream>>>((float*)out, ldo, in, ldi, (const uint16_t*)table_bf16, ldt, c0, tokens_dev, cols);
    else kf_token_gate_kernel<uint16_t><<<rows, 128, 0, ctx->stream>>>((uint16_t*)out, ldo, in, ldi, (const uint16_t*)table_bf16, ldt, c0, tokens_dev, cols);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_depth_mix(kf_ctx* ctx, float* x, float* hist, size_t hist_stride, const void* w_bf16, int n_prev, size_t n) {
    if (!ctx || !x || !hist || !w_bf16) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n_prev >= 0 && n >= 1 && hist_stride >= n, "history stride");
    kf_depth_mix_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(x, hist, hist_stride, (const uint16_t*)w_bf16, n_prev, n);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}

// gate_kind 0: none; 1: x * sigmoid(gate + gate_bias); 2: x * silu(gate).  out_kind 0: bf16 bits [rows][ldo]; 1: float [rows][ldo];
// 2: res[rows][dim] += mult * result (out is ignored).  row_idx (device, optional): source row of each output row.
// gate_kind 3 / 4: sigmoid(gate) / silu(gate) multiply the normed result; w_shared 1: the weight has dim / groups entries, used by every group; 2: it is one
// number.
// w_add: added to every weight in fp32 (1 for weights stored around zero, 0 for plain weights).  out_mult: factor on the rows written to
// out (out_kind 0 / 1), applied in fp32 before the rounding.
extern "C" int kf_group_rmsnorm_wadd(kf_ctx* ctx, void* out, int out_kind, int ldo, float* res, float mult, const float* x, int ldx, const float* gate, int ldg,
                                     const void* gate_bias_bf16, int gate_kind, const void* w_bf16, int w_shared, float w_add, float out_mult,
                                     const int32_t* row_idx, int rows, int dim, int groups, float eps) {
    if (!ctx || !x || !w_bf16) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && dim >= 1 && groups >= 1 && dim % groups == 0, "groups must divide dim");
    KF_REQUIRE(ctx, gate_kind >= 0 && gate_kind <= 4 && (gate_kind == 0 || gate) && out_kind >= 0 && out_kind <= 2 && (out_kind == 2 ? res != nullptr : out != nullptr),
               "gate / out kind");
    dim3 grid(rows, groups);
    const uint16_t *gb = (const uint16_t*)gate_bias_bf16, *w = (const uint16_t*)w_bf16;
#define KF_GN(G, A, T) kf_group_norm_kernel<G, A, T><<<grid, 256, 0, ctx->stream>>>((T*)out, ldo, res, x, ldx, gate, ldg, gb, w, row_idx, dim, groups, eps, mult, w_shared, w_add, out_mult)
    if (out_kind != 2 && groups > 1 && dim / groups <= 32 * kPartRegs) {
        const unsigned blocks = (unsigned)(((long long)rows * groups + 7) / 8);
#define KF_PART(G, T) kf_part_norm_kernel<G, T><<<blocks, 256, 0, ctx->stream>>>((T*)out, ldo, x, ldx, gate, ldg, gb, w, row_idx, rows, dim, groups, eps, w_shared, w_add, out_mult)
#define KF_PART_G(T) (gate_kind == 0 ? KF_PART(0, T) : gate_kind == 1 ? KF_PART(1, T) : gate_kind == 2 ? KF_PART(2, T) : gate_kind == 3 ? KF_PART(3, T) : KF_PART(4, T))
        if (out_kind == 1) KF_PART_G(float);
        else KF_PART_G(uint16_t);
#undef KF_PART_G
#undef KF_PART
    } else if (out_kind == 2) {
        if (gate_kind == 0) KF_GN(0, true, float);
        else if (gate_kind == 1) KF_GN(1, true, float);
        else if (gate_kind == 2) KF_GN(2, true, float);
        else if (gate_kind == 3) KF_GN(3, true, float);
        else KF_GN(4, true, float);
    } else if (out_kind == 1) {
        if (gate_kind == 0) KF_GN(0, false, float);
        else if (gate_kind == 1) KF_GN(1, false, float);
        else if (gate_kind == 2) KF_GN(2, false, float);
        else if (gate_kind == 3) KF_GN(3, false, float);
        else KF_GN(4, false, float);
    } else {
        if (gate_kind == 0) KF_GN(0, false, uint16_t);
        else if (gate_kind == 1) KF_GN(1, false, uint16_t);
        else if (gate_kind == 2) KF_GN(2, false, uint16_t);
        else if (gate_kind == 3) KF_GN(3, false, uint16_t);
        else KF_GN(4, false, uint16_t);
    }
#undef KF_GN
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_group_rmsnorm_ex(kf_ctx* ctx, void* out, int out_kind, int ldo, float* res, float mult, const float* x, int ldx, const float* gate, int ldg,
                                   const void* gate_bias_bf16, int gate_kind, const void* w_bf16, int w_shared, const int32_t* row_idx, int rows, int dim,
                                   int groups, float eps) {
    return kf_group_rmsnorm_wadd(ctx, out, out_kind, ldo, res, mult, x, ldx, gate, ldg, gate_bias_bf16, gate_kind, w_bf16, w_shared, 0.f, 1.f, row_idx, rows,
                                 dim, groups, eps);
}
extern "C" int kf_group_rmsnorm(kf_ctx* ctx, void* out, int out_kind, int ldo, float* res, float mult, const float* x, int ldx, const float* gate, int ldg,
                                const void* gate_bias_bf16, int gate_kind, const void* w_bf16, const int32_t* row_idx, int rows, int dim, int groups,
                                float eps) {
    if (gate_kind > 2) return KF_ERR_BAD_ARG;
    return kf_group_rmsnorm_ex(ctx, out, out_kind, ldo, res, mult, x, ldx, gate, ldg, gate_bias_bf16, gate_kind, w_bf16, 0, row_idx, rows, dim, groups, eps);
}
// res[rows][dim] += rmsnorm(sa * a + sb * b) * (w_add + w);  act_out (optional, [rows][dim] in the activation type) = the new res.
// b may be NULL (one branch).  The norm runs over the whole row.
extern "C" int kf_postnorm_residual(kf_ctx* ctx, float* res, void* act_out, int act_f32, const float* a, int lda, float sa, const float* b, int ldb, float sb,
                                    const void* w_bf16, float w_add, int rows, int dim, float eps) {
    return kf_postnorm_residual_ex(ctx, res, act_out, act_f32, a, lda, sa, b, ldb, sb, w_bf16, w_add, 0, 1.f, rows, dim, eps, nullptr, nullptr, 0, nullptr, nullptr);
}
static bool post_common(PostArgs& p, float* res, void* act_out, const void* w_bf16, float w_add, int w_one, float mult, int dim, float eps, const void* shift_bf16,
                        float* tail, size_t tail_stride, const int32_t* pos, const int32_t* slot) {
    p.res = res, p.act = act_out, p.w = (const uint16_t*)w_bf16, p.w_add = w_add, p.w_one = w_one, p.mult = mult, p.dim = dim, p.eps = eps;
    p.shift = (const uint16_t*)shift_bf16, p.tail = tail, p.tail_stride = tail_stride, p.pos = pos, p.slot = slot;
    return !shift_bf16 || (tail && tail_stride >= (size_t)dim && pos && slot && act_out);
}
// The general form: the sum is multiplied by `mult`, w_one 1: the norm's weight is one number.  shift_bf16 [dim] (optional; every row then is
// one token of a sequence of its own): act_out = x + (prev - x) * shift instead of x, prev = the sequence's tail [slot][tail_stride] (zeros at
// position 0), which then takes x.
extern "C" int kf_postnorm_residual_ex(kf_ctx* ctx, float* res, void* act_out, int act_f32, const float* a, int lda, float sa, const float* b, int ldb, float sb,
                                       const void* w_bf16, float w_add, int w_one, float mult, int rows, int dim, float eps, const void* shift_bf16, float* tail,
                                       size_t tail_stride, const int32_t* pos, const int32_t* slot) {
    if (!ctx || !res || !a || !w_bf16) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && dim >= 1, "shape");
    PostArgs p = {};
    KF_REQUIRE(ctx, post_common(p, res, act_out, w_bf16, w_add, w_one, mult, dim, eps, shift_bf16, tail, tail_stride, pos, slot), "a shift needs its tail, positions and slots");
    p.a = a, p.lda = lda, p.sa = sa, p.b = b, p.ldb = ldb, p.sb = sb;
    return launch_postnorm<0>(ctx, p, act_f32, rows);
}
// The same step over a token's experts: v = sum_j wgt[m][j] * y_slots[entry_slot[m][j]] (+ shared[m]); the combination never reaches memory.
extern "C" int kf_experts_postnorm_residual(kf_ctx* ctx, float* res, void* act_out, int act_f32, const float* y_slots, const int32_t* entry_slot, const float* wgt,
                                            const float* shared, int top, const void* w_bf16, float w_add, int w_one, float mult, int rows, int dim, float eps,
                                            const void* shift_bf16, float* tail, size_t tail_stride, const int32_t* pos, const int32_t* slot) {
    if (!ctx || !res || !y_slots || !entry_slot || !wgt || !w_bf16) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && dim >= 1 && top >= 1, "shape");
    PostArgs p = {};
    KF_REQUIRE(ctx, post_common(p, res, act_out, w_bf16, w_add, w_one, mult, dim, eps, shift_bf16, tail, tail_stride, pos, slot), "a shift needs its tail, positions and slots");
    p.y = y_slots, p.entry_slot = entry_slot, p.wgt = wgt, p.shared = shared, p.top = top;
    return launch_postnorm<1>(ctx, p, act_f32, rows);
}
// The start of a stream: res[m] = rmsnorm(W[token[m]]) * (w_add + w); act_out and the shift as above.
extern "C" int kf_embed_norm(kf_ctx* ctx, float* res, void* act_out, int act_f32, const kf_tensor_desc* table, const int32_t* tokens, const void* w_bf16, float w_add,
                             int w_one, int rows, float eps, const void* shift_bf16, float* tail, size_t tail_stride, const int32_t* pos, const int32_t* slot) {
    if (!ctx || !res || !table || !table->data_dev || !tokens || !w_bf16) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && table->type == KF_T_BF16 && table->cols >= 1, "bf16 table");
    PostArgs p = {};
    KF_REQUIRE(ctx, post_common(p, res, act_out, w_bf16, w_add, w_one, 1.f, table->cols, eps, shift_bf16, tail, tail_stride, pos, slot), "a shift needs its tail, positions and slots");
    p.table = (const uint16_t*)table->data_dev, p.tokens = tokens;
    return launch_postnorm<2>(ctx, p, act_f32, rows);
}
// Token shift over nseq sequences of T consecutive tokens each (rows seq * T + t of h, row stride ldh): out [nseq * T][dim] in the activation
// type = h[t] + (h[t-1] - h[t]) * w; tail [slot][tail_stride] floats hold the last row of the sequence's earlier tokens (ignored at position 0)
// and take the last row of this step.
extern "C" int kf_token_shift(kf_ctx* ctx, void* out, int out_f32, const float* h, int ldh, const void* w_bf16, float* tail, size_t tail_stride, const int32_t* pos,
                              const int32_t* slot, int nseq, int T, int dim) {
    if (!ctx || !out || !h || !w_bf16 || !tail || !pos || !slot) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, nseq >= 1 && nseq <= 65535 && T >= 1 && dim >= 1 && ldh >= dim && tail_stride >= (size_t)dim, "shape");
    dim3 grid((dim + 127) / 128, (T + kShiftRows - 1) / kShiftRows, nseq);
    if (out_f32) kf_token_shift_kernel<float><<<grid, 128, 0, ctx->stream>>>((float*)out, h, ldh, (const uint16_t*)w_bf16, tail, tail_stride, pos, slot, T, dim);
    else kf_token_shift_kernel<uint16_t><<<grid, 128, 0, ctx->stream>>>((uint16_t*)out, h, ldh, (const uint16_t*)w_bf16, tail, tail_stride, pos, slot, T, dim);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// res[rows][dim] += a + b + vec (a, b: float rows or NULL; vec: bf16 [dim] or NULL); act_out (with w_bf16) = rmsnorm(res) * w in the
// activation type.  w_bf16 NULL: the sum only.
extern "C" int kf_residual_prenorm(kf_ctx* ctx, float* res, void* act_out, int act_f32, const float* a, int lda, const float* b, int ldb, const void* vec_bf16,
                                   const void* w_bf16, int rows, int dim, float eps) {
    if (!ctx || !res || (w_bf16 && !act_out)) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && dim >= 1, "shape");
    if (!w_bf16 && !a && !b && !vec_bf16) return KF_OK;
    if (act_f32)
        kf_residual_prenorm_kernel<float><<<rows, 256, 0, ctx->stream>>>(res, (float*)act_out, a, lda, b, ldb, (const uint16_t*)vec_bf16, (const uint16_t*)w_bf16, dim, eps);
    else
        kf_residual_prenorm_kernel<uint16_t><<<rows, 256, 0, ctx->stream>>>(res, (uint16_t*)act_out, a, lda, b, ldb, (const uint16_t*)vec_bf16, (const uint16_t*)w_bf16, dim, eps);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// out[rows][ldo] (activation type) = g' * sigmoid(alpha * g') * (u' + shift) with g' = min(gate, limit), u' = clamp(up, -limit, limit); limit <= 0: no clamp
extern "C" int kf_glu_clamped(kf_ctx* ctx, void* out, int out_f32, int ldo, const float* gate, int ldg, const float* up, int ldu, int rows, int cols, float limit,
                              float alpha, float shift) {
    if (!ctx || !out || !gate || !up) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, rows >= 1 && cols >= 1, "shape");
    dim3 grid(std::min(64, (cols + 255) / 256), rows);
    if (out_f32) kf_glu_clamped_kernel<float><<<grid, 256, 0, ctx->stream>>>((float*)out, ldo, gate, ldg, up, ldu, cols, limit, alpha, shift);
    else kf_glu_clamped_kernel<uint16_t><<<grid, 256, 0, ctx->stream>>>((uint16_t*)out, ldo, gate, ldg, up, ldu, cols, limit, alpha, shift);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// Steps of a stack with the norm n(x) = tanh(alpha x) w + b (see kf_dyt_step): x = res + scale * a, out = n(x) or the token mixes of n(x).
extern "C" int kf_dyt_residual(kf_ctx* ctx, const kf_dyt_step* s, const float* a, int lda) {
    if (!ctx || !s) return KF_ERR_BAD_ARG;
    DytArgs p = {};
    KF_REQUIRE(ctx, dyt_args(p, s) && (!a || lda >= s->dim), "rows, norm, mixes");
    p.a = a, p.lda = lda;
    return launch_dyt<0>(ctx, p, s->out_f32, s->rows);
}
// The same over a token's experts: the added row is sum_j wgt[m][j] * y_slots[entry_slot[m][j]]; an entry without a slot (-1) stands for row m of
// `pass` ([rows][dim] in the activation type), which may be the buffer that out writes.
extern "C" int kf_dyt_experts(kf_ctx* ctx, const kf_dyt_step* s, const float* y_slots, const int32_t* entry_slot, const float* wgt, const void* pass, int top) {
    if (!ctx || !s || !y_slots || !entry_slot || !wgt || !pass) return KF_ERR_BAD_ARG;
    DytArgs p = {};
    KF_REQUIRE(ctx, dyt_args(p, s) && top >= 1 && !(s->row_idx && pass == s->out), "rows, norm, mixes");
    p.y = y_slots, p.entry_slot = entry_slot, p.wgt = wgt, p.pass = pass, p.top = top;
    return launch_dyt<1>(ctx, p, s->out_f32, s->rows);
}
// The start of a stream: res[m] = W[token[m]], out as above.
extern "C" int kf_dyt_embed(kf_ctx* ctx, const kf_dyt_step* s, const kf_tensor_desc* table, const int32_t* tokens) {
    if (!ctx || !s || !table || !table->data_dev || !tokens) return KF_ERR_BAD_ARG;
    DytArgs p = {};
    KF_REQUIRE(ctx, dyt_args(p, s) && !s->row_idx && table->type == KF_T_BF16 && table->cols == s->dim, "bf16 table of the stream's width");
    p.table = (const uint16_t*)table->data_dev, p.tokens = tokens;
    return launch_dyt<2>(ctx, p, s->out_f32, s->rows);
}
// The token mixes of n(res) for nseq sequences of T consecutive tokens each (res is only read; rows = nseq * T).
extern "C" int kf_dyt_token_mix(kf_ctx* ctx, const kf_dyt_step* s, int nseq, int T) {
    if (!ctx || !s) return KF_ERR_BAD_ARG;
    DytArgs p = {};
    KF_REQUIRE(ctx, dyt_args(p, s) && s->mu_bf16 && nseq >= 1 && nseq <= 65535 && T >= 1 && s->rows == nseq * T, "rows, norm, mixes");
    p.T = T;
    const int v = dyt_vec(p) ? 4 : 1;
    const dim3 grid((p.dim + 128 * v - 1) / (128 * v), (T + kShiftRows - 1) / kShiftRows, nseq);
#define KF_DYM(TY, V) kf_dyt_mix_kernel<TY, V><<<grid, 128, 0, ctx->stream>>>(p)
    if (s->out_f32) v == 4 ? KF_DYM(float, 4) : KF_DYM(float, 1);
    else v == 4 ? KF_DYM(uint16_t, 4) : KF_DYM(uint16_t, 1);
#undef KF_DYM
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_scale_f32(kf_ctx* ctx, float* x, size_t n, float s) {
    if (!ctx || !x) return KF_ERR_BAD_ARG;
    if (!n || s == 1.f) return KF_OK;
    kf_scale_f32_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(x, n, s);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_f32_to_bf16(kf_ctx* ctx, void* out_bf16, const float* in, size_t n) {
    if (!ctx || !out_bf16 || !in) return KF_ERR_BAD_ARG;
    if (!n) return KF_OK;
    kf_f32_to_bf16_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>((uint16_t*)out_bf16, in, n);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}

// Router of a mixture of experts over fp32 logits [M][ldl] (+ bf16 bias [E] or NULL): idx / wgt [M][top]; then the dispatch tables:
// offsets [E + 1], entry_slot [M * top] (where each (token, choice) sits among the expert-sorted slots), slot_row / slot_group [M * top].
// work: device int32 scratch of 2 * M * top + E entries.
// full_softmax 0: weights = softmax over the chosen logits; 1: the chosen entries of the softmax over all E experts (not renormalised).
static int moe_route_impl(kf_ctx* ctx, int32_t* idx, float* wgt, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row, int32_t* slot_group,
                          int32_t* work, const float* logits, int ldl, const void* bias_bf16, int M, int E, int top, int full_softmax, const RouteMode md) {
    if (!ctx || !idx || !wgt || !offsets || !entry_slot || !slot_row || !slot_group || !work || !logits) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, M >= 1 && E >= 1 && top >= 1 && top <= E && ldl >= E, "1 <= top <= experts");
    const int n = M * top;
    if (M == 1 && md.kind && top <= 32 && E <= 32 * kRouteCache) {
        kf_moe_route_one_kernel<<<1, 32, 0, ctx->stream>>>(idx, wgt, offsets, entry_slot, slot_row, slot_group, logits, (const uint16_t*)bias_bf16, E, top, md);
        KF_LAUNCH_CHECK(ctx);
        return KF_OK;
    }
    if (n <= kRouteSmall && (long long)E * n <= 16384) {
        kf_moe_route_small_kernel<<<1, 256, 0, ctx->stream>>>(idx, wgt, offsets, entry_slot, slot_row, slot_group, logits, ldl, (const uint16_t*)bias_bf16, M, E, top, full_softmax, md);
        KF_LAUNCH_CHECK(ctx);
        return KF_OK;
    }
    int32_t *rank = work, *count = work + n;
    kf_moe_route_kernel<<<(M + 3) / 4, 128, 0, ctx->stream>>>(idx, wgt, logits, ldl, (const uint16_t*)bias_bf16, M, E, top, full_softmax, md);
    KF_LAUNCH_CHECK(ctx);
    const int X = E - md.pass;
    kf_moe_rank_kernel<<<X, 256, 0, ctx->stream>>>(rank, count, idx, n);
    KF_LAUNCH_CHECK(ctx);
    kf_moe_offsets_kernel<<<1, 32, 0, ctx->stream>>>(offsets, count, X);
    KF_LAUNCH_CHECK(ctx);
    kf_moe_slots_kernel<<<(n + 255) / 256, 256, 0, ctx->stream>>>(entry_slot, slot_row, slot_group, idx, rank, offsets, n, top, X);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_moe_route_ex(kf_ctx* ctx, int32_t* idx, float* wgt, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row, int32_t* slot_group,
                               int32_t* work, const float* logits, int ldl, const void* bias_bf16, int M, int E, int top, int full_softmax) {
    const RouteMode md = {0, 1, 1, 1.f, 0};
    return moe_route_impl(ctx, idx, wgt, offsets, entry_slot, slot_row, slot_group, work, logits, ldl, bias_bf16, M, E, top, full_softmax, md);
}
// The same tables from sigmoid scores: the choice runs over sigmoid(logit) + choice_bias (bf16 [E] or NULL) inside the `keep` best of
// `groups` equal contiguous groups of experts (a group ranks by the sum of its top-2 choice values; groups <= 64, groups 1: no
// grouping); weights = scale * sigmoid(logit) of the chosen experts, not renormalised.  top <= keep * (E / groups).
extern "C" int kf_moe_route_grouped(kf_ctx* ctx, int32_t* idx, float* wgt, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row, int32_t* slot_group,
                                    int32_t* work, const float* logits, int ldl, const void* choice_bias_bf16, int M, int E, int top, int groups, int keep,
                                    float scale) {
    if (!ctx) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, groups >= 1 && groups <= kRouteGroups && E >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && top >= 1 && top <= keep * (E / groups),
               "groups <= 64 divide the experts; 1 <= keep <= groups; top <= keep * experts / groups");
    const RouteMode md = {1, groups, keep, scale, 0};
    return moe_route_impl(ctx, idx, wgt, offsets, entry_slot, slot_row, slot_group, work, logits, ldl, choice_bias_bf16, M, E, top, 0, md);
}
// The same tables from softmax scores over experts + pass outputs (logits [M][ldl >= experts + pass]): the choice runs over s + choice_bias
// inside the `keep` best of `groups` equal contiguous groups of the outputs (a group ranks by its largest choice value; groups <= 64);
// weights = s of the chosen over (their sum + 1e-20).  The last `pass` outputs are no experts: their entries get entry_slot -1 and no slot,
// slots that stay unused get slot_group -1.
extern "C" int kf_moe_route_softmax_grouped(kf_ctx* ctx, int32_t* idx, float* wgt, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row, int32_t* slot_group,
                                            int32_t* work, const float* logits, int ldl, const void* choice_bias_bf16, int M, int experts, int pass, int top,
                                            int groups, int keep) {
    if (!ctx) return KF_ERR_BAD_ARG;
    const int E = experts + pass;
    KF_REQUIRE(ctx, experts >= 1 && pass >= 0 && groups >= 1 && groups <= kRouteGroups && E % groups == 0 && keep >= 1 && keep <= groups && top >= 1 &&
                        top <= keep * (E / groups),
               "groups <= 64 divide the outputs; 1 <= keep <= groups; top <= keep * outputs / groups");
    const RouteMode md = {2, groups, keep, 1.f, pass};
    return moe_route_impl(ctx, idx, wgt, offsets, entry_slot, slot_row, slot_group, work, logits, ldl, choice_bias_bf16, M, E, top, 0, md);
}
extern "C" int kf_moe_route(kf_ctx* ctx, int32_t* idx, float* wgt, int32_t* offsets, int32_t* entry_slot, int32_t* slot_row, int32_t* slot_group,
                            int32_t* work, const float* logits, int ldl, const void* bias_bf16, int M, int E, int top) {
    return kf_moe_route_ex(ctx, idx, wgt, offsets, entry_slot, slot_row, slot_group, work, logits, ldl, bias_bf16, M, E, top, 0);
}
// kf_moe_route's tables for n_routes layers at once, the experts read from tables of token ids (see kf_table_route): routes_dev is a device
// array; max_experts / max_top bound the entries of all routes.  work of a route: M * top + experts ints.
extern "C" int kf_moe_route_table(kf_ctx* ctx, const kf_table_route* routes_dev, int n_routes, int max_experts, int max_top, const int32_t* tokens, int M) {
    if (!ctx || !routes_dev || !tokens) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n_routes >= 1 && n_routes <= 65535 && max_experts >= 1 && max_experts <= 8192 && max_top >= 1 && M >= 1, "shape");
    const int n = M * max_top;
    if (n <= kRouteSmall && (long long)max_experts * n <= 16384) {
        kf_moe_table_small_kernel<<<n_routes, 256, 0, ctx->stream>>>(routes_dev, tokens, M);
        KF_LAUNCH_CHECK(ctx);
        return KF_OK;
    }
    kf_moe_table_idx_kernel<<<dim3((n + 255) / 256, n_routes), 256, 0, ctx->stream>>>(routes_dev, tokens, M);
    KF_LAUNCH_CHECK(ctx);
    kf_moe_table_rank_kernel<<<dim3(max_experts, n_routes), 256, 0, ctx->stream>>>(routes_dev, M);
    KF_LAUNCH_CHECK(ctx);
    kf_moe_table_slots_kernel<<<dim3((n + 255) / 256, n_routes), 256, (size_t)max_experts * sizeof(int), ctx->stream>>>(routes_dev, M);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
// accumulate 1: out += the combination (the residual stream takes the experts' sum directly)
extern "C" int kf_moe_combine_ex(kf_ctx* ctx, float* out, const float* y_slots, const int32_t* entry_slot, const float* wgt, const float* shared,
                                 const float* shared_gate_logit, int ld_gate, int M, int dim, int top, int accumulate) {
    if (!ctx || !out || !y_slots || !entry_slot || !wgt) return KF_ERR_BAD_ARG;
    kf_moe_combine_kernel<<<M, 256, 0, ctx->stream>>>(out, y_slots, entry_slot, wgt, shared, shared_gate_logit, ld_gate, dim, top, accumulate);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
extern "C" int kf_moe_combine(kf_ctx* ctx, float* out, const float* y_slots, const int32_t* entry_slot, const float* wgt, const float* shared,
                              const float* shared_gate_logit, int ld_gate, int M, int dim, int top) {
    return kf_moe_combine_ex(ctx, out, y_slots, entry_slot, wgt, shared, shared_gate_logit, ld_gate, M, dim, top, 0);
}
