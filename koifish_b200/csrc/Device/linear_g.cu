// linear_g.cu -- matmuls of ANY shape over bf16 weights with fp32 results, for the layers whose sizes the tuned kernels of gemv.cu /
// gemm_tc.cu do not take (their K must be a multiple of 128 and their N of 16): y[m][n] = sum_k x[m][k] * W[n][k].
//   * activations x are bf16 bits (act_f32 = 0: the products are exact in fp32 and accumulate in fp32, i.e. the arithmetic of a bf16
//     tensor-core matmul) or float (act_f32 = 1: a true 32-bit matmul, FMA by FMA, no reduced-precision mode);
//   * "grouped" form for mixtures of experts: every output row (a slot) names the weight matrix it uses; slots of one expert are
//     contiguous (offsets[e] .. offsets[e+1]) and may gather their input row through src_row;
//   * DUAL form: two weight tables A, B of equal shape and y = silu(A x) * (B x), the gate / up pair of a gated feed-forward, or its clamped
//     form y = g sigmoid(alpha g) (u + shift) with g = min(A x, limit), u = clamp(B x, -limit, limit);
//   * "batch" form for a handful of rows: several weights, each with an input and an output of its own, in one launch.
// Two kernels: a warp-per-output GEMV for a handful of rows (decode: every weight row is read once, 16-byte loads when the row length
// allows) and a 64 x 64 x 32 shared-memory tile kernel for panels (mma.sync m16n8k16 for bf16 activations, FFMA for float ones).
// No reference equivalent: the reference's SLP::Forw hands every shape to cuBLASLt (src/Device/CUDA/NeuronFuse.cu:305-381).
#include <algorithm>

#include "kf_common.cuh"

namespace {

struct LinArgs {
    const uint16_t* W0;          // single weight (dense) -- or
    const uint16_t* const* Wt0;  // table of per-expert weights (grouped)
    const uint16_t* W1;          // DUAL: second weight
    const uint16_t* const* Wt1;
    const void* x;               // [rows][ldx] bf16 bits or float
    void* y;                     // [slots][ldy] float (or, DUAL with out_act, the activation type)
    const int32_t* offsets;      // grouped: [E + 1] slot ranges; nullptr: one group [0, M)
    const int32_t* src_row;      // slot -> row of x; nullptr: slot
    const int32_t* slot_group;   // GEMV form: slot -> expert; nullptr: 0
    int M, N, K, ldx, ldy;
    int out_act;                 // DUAL or act != 0: 0 = float out, 1 = bf16 out, (float activations: float out)
    int act;                     // single-weight form: 0 = none, 1 = gelu (tanh form), 2 = relu squared, 3 = tanh, applied to the result
    int glu;                     // DUAL: 0 = silu(a) * b, 1 = the clamped form
    float limit, alpha, shift;   // ... its constants (limit <= 0: not clamped)
};
__device__ __forceinline__ float lin_act(float v, int act) {
    if (act == 1) return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    if (act == 2) return v > 0.f ? v * v : 0.f;
    if (act == 3) return tanhf(v);
    return v;
}

template <typename TA>
__device__ __forceinline__ float ld_act(const TA* p);
template <>
__device__ __forceinline__ float ld_act<uint16_t>(const uint16_t* p) { return bf16_bits_to_f32(*p); }
template <>
__device__ __forceinline__ float ld_act<float>(const float* p) { return *p; }

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float lin_pair(const LinArgs& a, float g, float u) {
    if (!a.glu) return silu_f(g) * u;
    if (a.limit > 0.f) g = fminf(g, a.limit), u = fminf(fmaxf(u, -a.limit), a.limit);
    return g / (1.f + expf(-a.alpha * g)) * (u + a.shift);
}

// ------------------------------------------------------------------------------------------------------------------ GEMV (few slots)
// one warp per (slot, output n): lanes stride over k, fixed butterfly reduction -> deterministic.
template <typename TA, bool DUAL>
__global__ void __launch_bounds__(256) kf_lin_gemv_kernel(LinArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n    = blockIdx.x * 8 + warp;
    const int slot = blockIdx.y;
    if (n >= a.N) return;
    const int g   = a.slot_group ? a.slot_group[slot] : 0;
    if (g < 0) return;  // a slot that no token uses
    const int row = a.src_row ? a.src_row[slot] : slot;
    const uint16_t* w0 = (a.Wt0 ? a.Wt0[g] : a.W0) + (size_t)n * a.K;
    const uint16_t* w1 = DUAL ? (a.Wt1 ? a.Wt1[g] : a.W1) + (size_t)n * a.K : nullptr;
    const TA* x = (const TA*)a.x + (size_t)row * a.ldx;
    float s0 = 0.f, s1 = 0.f;
    const bool vec = (a.K % 8 == 0) && (a.ldx % 8 == 0) && (((uintptr_t)w0 & 15) == 0) && (((uintptr_t)x & 15) == 0) && (!DUAL || ((uintptr_t)w1 & 15) == 0);
    if (vec) {
#pragma unroll DUAL ? 2 : 4
        for (int k = lane * 8; k < a.K; k += 256) {
            const uint4 wv = *reinterpret_cast<const uint4*>(w0 + k);
            const uint32_t wq[4] = {wv.x, wv.y, wv.z, wv.w};
            float xv[8];
            if (sizeof(TA) == 2) {
                const uint4 xq4 = *reinterpret_cast<const uint4*>((const uint16_t*)x + k);
                const uint32_t xq[4] = {xq4.x, xq4.y, xq4.z, xq4.w};
#pragma unroll
                for (int j = 0; j < 4; j++) xv[2 * j] = bf16lo(xq[j]), xv[2 * j + 1] = bf16hi(xq[j]);
            } else {
                const float4 f0 = *reinterpret_cast<const float4*>((const float*)x + k), f1 = *reinterpret_cast<const float4*>((const float*)x + k + 4);
                xv[0] = f0.x, xv[1] = f0.y, xv[2] = f0.z, xv[3] = f0.w, xv[4] = f1.x, xv[5] = f1.y, xv[6] = f1.z, xv[7] = f1.w;
            }
#pragma unroll
            for (int j = 0; j < 4; j++) s0 = fmaf(bf16lo(wq[j]), xv[2 * j], s0), s0 = fmaf(bf16hi(wq[j]), xv[2 * j + 1], s0);
            if (DUAL) {
                const uint4 uv = *reinterpret_cast<const uint4*>(w1 + k);
                const uint32_t uq[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
                for (int j = 0; j < 4; j++) s1 = fmaf(bf16lo(uq[j]), xv[2 * j], s1), s1 = fmaf(bf16hi(uq[j]), xv[2 * j + 1], s1);
            }
        }
    } else {
        for (int k = lane; k < a.K; k += 32) {
            const float xv = ld_act<TA>(x + k);
            s0 = fmaf(bf16_bits_to_f32(w0[k]), xv, s0);
            if (DUAL) s1 = fmaf(bf16_bits_to_f32(w1[k]), xv, s1);
        }
    }
    s0 = warp_sum(s0);
    if (DUAL) s1 = warp_sum(s1);
    if (lane == 0) {
        const float r = DUAL ? lin_pair(a, s0, s1) : lin_act(s0, a.act);
        if ((DUAL || a.act) && a.out_act == 1)
            ((uint16_t*)a.y)[(size_t)slot * a.ldy + n] = f32_to_bf16_bits(r);
        else
            ((float*)a.y)[(size_t)slot * a.ldy + n] = r;
    }
}

// Several independent products of one reduction length, each with its own weight, input and output, for a handful of rows: a warp per
// (row, output) as above; blockIdx.x walks the outputs of all of them one after the other.
constexpr int kBatchMax = 8;
struct BatchArgs {
    const uint16_t* W[kBatchMax];
    const void* x[kBatchMax];
    float* y[kBatchMax];
    int N[kBatchMax], ldy[kBatchMax], act[kBatchMax], first[kBatchMax + 1];  // first: the block at which a product starts
    int n, K, ldx;
};
template <typename TA>
__global__ void __launch_bounds__(256) kf_lin_gemv_batch_kernel(BatchArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.y;
    int j = 0;
#pragma unroll
    for (int i = 1; i < kBatchMax; i++)
        if (i < a.n && (int)blockIdx.x >= a.first[i]) j = i;
    const int n = ((int)blockIdx.x - a.first[j]) * 8 + warp;
    if (n >= a.N[j]) return;
    const uint16_t* w = a.W[j] + (size_t)n * a.K;
    const TA* x = (const TA*)a.x[j] + (size_t)row * a.ldx;
    float s = 0.f;
    if ((a.K % 8 == 0) && (a.ldx % 8 == 0) && (((uintptr_t)w & 15) == 0) && (((uintptr_t)x & 15) == 0)) {
#pragma unroll 4
        for (int k = lane * 8; k < a.K; k += 256) {
            const uint4 wv = *reinterpret_cast<const uint4*>(w + k);
            const uint32_t wq[4] = {wv.x, wv.y, wv.z, wv.w};
            float xv[8];
            if (sizeof(TA) == 2) {
                const uint4 xq4 = *reinterpret_cast<const uint4*>((const uint16_t*)x + k);
                const uint32_t xq[4] = {xq4.x, xq4.y, xq4.z, xq4.w};
#pragma unroll
                for (int i = 0; i < 4; i++) xv[2 * i] = bf16lo(xq[i]), xv[2 * i + 1] = bf16hi(xq[i]);
            } else {
                const float4 f0 = *reinterpret_cast<const float4*>((const float*)x + k), f1 = *reinterpret_cast<const float4*>((const float*)x + k + 4);
                xv[0] = f0.x, xv[1] = f0.y, xv[2] = f0.z, xv[3] = f0.w, xv[4] = f1.x, xv[5] = f1.y, xv[6] = f1.z, xv[7] = f1.w;
            }
#pragma unroll
            for (int i = 0; i < 4; i++) s = fmaf(bf16lo(wq[i]), xv[2 * i], s), s = fmaf(bf16hi(wq[i]), xv[2 * i + 1], s);
        }
    } else {
        for (int k = lane; k < a.K; k += 32) s = fmaf(bf16_bits_to_f32(w[k]), ld_act<TA>(x + k), s);
    }
    s = warp_sum(s);
    if (lane == 0) a.y[j][(size_t)row * a.ldy[j] + n] = lin_act(s, a.act[j]);
}

// Few outputs over a long reduction for a panel of rows (a router, a low-rank projection): a warp takes kSkC outputs of kSkR rows, so a weight
// fragment serves kSkR rows and a row fragment kSkC outputs.  Row lengths are multiples of 8 and everything is 16-byte aligned.
constexpr int kSkR = 4, kSkC = 2;
template <typename TA>
__global__ void __launch_bounds__(256) kf_lin_skinny_kernel(LinArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = (blockIdx.x * 8 + warp) * kSkC, m0 = blockIdx.y * kSkR;
    if (n0 >= a.N) return;
    const uint16_t* w[kSkC];
    const TA* x[kSkR];
#pragma unroll
    for (int j = 0; j < kSkC; j++) w[j] = a.W0 + (size_t)min(n0 + j, a.N - 1) * a.K;
#pragma unroll
    for (int i = 0; i < kSkR; i++) x[i] = (const TA*)a.x + (size_t)min(m0 + i, a.M - 1) * a.ldx;
    float s[kSkR][kSkC];
#pragma unroll
    for (int i = 0; i < kSkR; i++)
#pragma unroll
        for (int j = 0; j < kSkC; j++) s[i][j] = 0.f;
#pragma unroll 2
    for (int k = lane * 8; k < a.K; k += 256) {
        float wv[kSkC][8];
#pragma unroll
        for (int j = 0; j < kSkC; j++) {
            const uint4 q = *reinterpret_cast<const uint4*>(w[j] + k);
            const uint32_t u[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
            for (int e = 0; e < 4; e++) wv[j][2 * e] = bf16lo(u[e]), wv[j][2 * e + 1] = bf16hi(u[e]);
        }
#pragma unroll
        for (int i = 0; i < kSkR; i++) {
            float xv[8];
            if (sizeof(TA) == 2) {
                const uint4 q = *reinterpret_cast<const uint4*>((const uint16_t*)x[i] + k);
                const uint32_t u[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                for (int e = 0; e < 4; e++) xv[2 * e] = bf16lo(u[e]), xv[2 * e + 1] = bf16hi(u[e]);
            } else {
                const float4 f0 = *reinterpret_cast<const float4*>((const float*)x[i] + k), f1 = *reinterpret_cast<const float4*>((const float*)x[i] + k + 4);
                xv[0] = f0.x, xv[1] = f0.y, xv[2] = f0.z, xv[3] = f0.w, xv[4] = f1.x, xv[5] = f1.y, xv[6] = f1.z, xv[7] = f1.w;
            }
#pragma unroll
            for (int j = 0; j < kSkC; j++)
#pragma unroll
                for (int e = 0; e < 8; e++) s[i][j] = fmaf(wv[j][e], xv[e], s[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < kSkR; i++)
#pragma unroll
        for (int j = 0; j < kSkC; j++) {
            const float t = warp_sum(s[i][j]);
            if (lane == 0 && m0 + i < a.M && n0 + j < a.N) {
                const float r = lin_act(t, a.act);
                if (a.act && a.out_act == 1) ((uint16_t*)a.y)[(size_t)(m0 + i) * a.ldy + n0 + j] = f32_to_bf16_bits(r);
                else ((float*)a.y)[(size_t)(m0 + i) * a.ldy + n0 + j] = r;
            }
        }
}

// ------------------------------------------------------------------------------------------------------------------ tile kernel
// 64 slots x 64 outputs per CTA, k in steps of 64 (bf16) or 32 (float); 256 threads.  Float activations: each thread a 4 x 4 block of FFMA accumulators.
// bf16 activations: 8 warps as 4 (m) x 2 (n), each warp 16 x 32 through mma.sync.m16n8k16; operands come from the same shared tiles.
// The next k step's operands are fetched into registers (16-byte loads when the row length and alignment allow, else element by
// element) while the current one is multiplied.  Every load is bounds-checked, so M, N and K are free.
constexpr int BM = 64, BN = 64;  // k step: 64 for bf16 activations (two 16-byte fetches per operand and thread in flight), 32 for float

__device__ __forceinline__ void mma_bf16_16816(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

__device__ __forceinline__ void ldsm_x4(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
// 8 consecutive k of one row: thread t fetches row t / 4, k offset (t % 4) * 8
template <typename T>
struct __align__(16) Frag8 {
    T v[8];
};
template <typename T>
__device__ __forceinline__ void fetch8(Frag8<T>& f, const T* base, size_t row_off, int k, int K, bool row_ok, bool vec) {
    if (row_ok && vec && k + 8 <= K) {
        if (sizeof(T) == 2) {
            *reinterpret_cast<uint4*>(f.v) = *reinterpret_cast<const uint4*>(base + row_off + k);
        } else {
            *reinterpret_cast<float4*>(f.v)     = *reinterpret_cast<const float4*>(base + row_off + k);
            *reinterpret_cast<float4*>(f.v + 4) = *reinterpret_cast<const float4*>(base + row_off + k + 4);
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < 8; j++) f.v[j] = (row_ok && k + j < K) ? base[row_off + k + j] : T(0);
}

// The same shapes with bf16 activations on the tensor cores: a CTA takes 16 rows and all outputs (up to 8 * NT), its 8 warps deal the k chunks of
// 32 among themselves and their sums meet in shared memory, always in the same order.  Fragments come straight from memory: a product over k
// does not mind how k is numbered, so lane (g, t) of an operand's row g loads the 8 consecutive k 8t .. 8t + 7 of a chunk in one access and
// hands them out as the k places that two m16n8k16 steps expect of it; both operands use the same numbering.
template <int NT>
__global__ void __launch_bounds__(256) kf_lin_skinny_mma_kernel(LinArgs a) {
    __shared__ __align__(16) float part[4][16][NT * 8 + 2];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, m0 = blockIdx.x * 16;
    const uint16_t* xa = (const uint16_t*)a.x + (size_t)min(m0 + g, a.M - 1) * a.ldx + 8 * t;
    const uint16_t* xb = (const uint16_t*)a.x + (size_t)min(m0 + g + 8, a.M - 1) * a.ldx + 8 * t;
    const uint16_t* w[NT];
#pragma unroll
    for (int j = 0; j < NT; j++) w[j] = a.W0 + (size_t)min(j * 8 + g, a.N - 1) * a.K + 8 * t;
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; j++) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    for (int k = warp * 32; k < a.K; k += 256) {
        const uint4 pa = *reinterpret_cast<const uint4*>(xa + k), pb = *reinterpret_cast<const uint4*>(xb + k);
        uint4 q[NT];
#pragma unroll
        for (int j = 0; j < NT; j++) q[j] = *reinterpret_cast<const uint4*>(w[j] + k);
        const uint32_t a0[4] = {pa.x, pb.x, pa.y, pb.y}, a1[4] = {pa.z, pb.z, pa.w, pb.w};
#pragma unroll
        for (int j = 0; j < NT; j++) {
            const uint32_t b0[2] = {q[j].x, q[j].y}, b1[2] = {q[j].z, q[j].w};
            mma_bf16_16816(acc[j], a0, b0);
            mma_bf16_16816(acc[j], a1, b1);
        }
    }
    auto put = [&](int slot) {
#pragma unroll
        for (int j = 0; j < NT; j++) {
            part[slot][g][j * 8 + 2 * t] = acc[j][0], part[slot][g][j * 8 + 2 * t + 1] = acc[j][1];
            part[slot][g + 8][j * 8 + 2 * t] = acc[j][2], part[slot][g + 8][j * 8 + 2 * t + 1] = acc[j][3];
        }
    };
    if (warp >= 4) put(warp - 4);
    __syncthreads();
    if (warp < 4) {
#pragma unroll
        for (int j = 0; j < NT; j++) {
            acc[j][0] += part[warp][g][j * 8 + 2 * t], acc[j][1] += part[warp][g][j * 8 + 2 * t + 1];
            acc[j][2] += part[warp][g + 8][j * 8 + 2 * t], acc[j][3] += part[warp][g + 8][j * 8 + 2 * t + 1];
        }
        put(warp);  // the places this thread has just read
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * a.N; i += blockDim.x) {
        const int r = i / a.N, n = i - r * a.N;
        if (m0 + r >= a.M) break;
        const float v = lin_act((part[0][r][n] + part[1][r][n]) + (part[2][r][n] + part[3][r][n]), a.act);
        if (a.act && a.out_act == 1) ((uint16_t*)a.y)[(size_t)(m0 + r) * a.ldy + n] = f32_to_bf16_bits(v);
        else ((float*)a.y)[(size_t)(m0 + r) * a.ldy + n] = v;
    }
}

template <typename TA, bool DUAL>
__global__ void __launch_bounds__(256) kf_lin_tile_kernel(LinArgs a) {
    const int g    = blockIdx.z;
    const int lo   = a.offsets ? a.offsets[g] : 0;
    const int hi   = a.offsets ? a.offsets[g + 1] : a.M;
    const int n0 = blockIdx.x * BN;
    // a CTA walks the slot tiles blockIdx.y, blockIdx.y + gridDim.y, ... of its group: the grid is sized for the average group, not the worst
    for (int m0 = lo + blockIdx.y * BM; m0 < hi; m0 += gridDim.y * BM) {
    const uint16_t* W0 = a.Wt0 ? a.Wt0[g] : a.W0;
    const uint16_t* W1 = DUAL ? (a.Wt1 ? a.Wt1[g] : a.W1) : nullptr;
    constexpr bool MMA = sizeof(TA) == 2;
    constexpr int BK  = MMA ? 64 : 32, NF = BK / 32;
    constexpr int LDS = BK + 8;  // row pitch in elements: 16-byte aligned rows, conflict-free fragment loads
    __shared__ __align__(16) TA sx[BM][LDS];
    __shared__ __align__(16) uint16_t sw0[BN][LDS];
    __shared__ __align__(16) uint16_t sw1[DUAL ? BN : 1][LDS];
    const int tid = threadIdx.x;
    const int lr = tid >> 2, lk = (tid & 3) * 8;  // this thread's load: row lr, k offset lk
    int xrow = -1;
    {
        const int s = m0 + lr;
        if (s < hi) xrow = a.src_row ? a.src_row[s] : s;
    }
    const bool wok = n0 + lr < a.N;
    const size_t xoff = (size_t)(xrow < 0 ? 0 : xrow) * a.ldx, woff = (size_t)(n0 + lr) * a.K;
    const bool xvec = (a.ldx % 8 == 0) && (((uintptr_t)a.x & 15) == 0) && (a.K % 8 == 0);
    const bool wvec = (a.K % 8 == 0) && (((uintptr_t)W0 & 15) == 0) && (!DUAL || ((uintptr_t)W1 & 15) == 0);
    float acc0[16], acc1[DUAL ? 16 : 1];
#pragma unroll
    for (int i = 0; i < 16; i++) acc0[i] = 0.f;
    if (DUAL)
#pragma unroll
        for (int i = 0; i < 16; i++) acc1[i] = 0.f;
    const int warp = tid >> 5, lane = tid & 31;
    const int wm = warp & 3, wn = warp >> 2;      // MMA: warp tile rows wm*16, cols wn*32
    const int tr = tid >> 4, tc = tid & 15;        // FFMA: thread rows tr*4.., cols tc*4..
    Frag8<TA> fx[NF];
    Frag8<uint16_t> fw0[NF], fw1[NF];
    auto fetch = [&](int kb) {  // fragment f covers k = kb + f * 32 + lk .. + 7
#pragma unroll
        for (int f = 0; f < NF; f++) {
            fetch8<TA>(fx[f], (const TA*)a.x, xoff, kb + f * 32 + lk, a.K, xrow >= 0, xvec);
            fetch8<uint16_t>(fw0[f], W0, woff, kb + f * 32 + lk, a.K, wok, wvec);
            if (DUAL) fetch8<uint16_t>(fw1[f], W1, woff, kb + f * 32 + lk, a.K, wok, wvec);
        }
    };
    fetch(0);
    for (int k0 = 0; k0 < a.K; k0 += BK) {
        __syncthreads();  // the previous step's fragments have been read
#pragma unroll
        for (int f = 0; f < NF; f++) {
            const int kc = f * 32 + lk;
            if (MMA) {
                *reinterpret_cast<uint4*>(&sx[lr][kc]) = *reinterpret_cast<const uint4*>(fx[f].v);
            } else {
                *reinterpret_cast<float4*>(&sx[lr][kc])     = *reinterpret_cast<const float4*>(fx[f].v);
                *reinterpret_cast<float4*>(&sx[lr][kc + 4]) = *reinterpret_cast<const float4*>(fx[f].v + 4);
            }
            *reinterpret_cast<uint4*>(&sw0[lr][kc]) = *reinterpret_cast<const uint4*>(fw0[f].v);
            if (DUAL) *reinterpret_cast<uint4*>(&sw1[lr][kc]) = *reinterpret_cast<const uint4*>(fw1[f].v);
        }
        __syncthreads();
        if (k0 + BK < a.K) fetch(k0 + BK);  // next step's operands travel while this one is multiplied
        if (MMA) {
            // fragments through ldmatrix: A = 16 rows x 16 k of this warp's slots; B = two 8-output tiles per instruction
            const uint16_t* xa = (const uint16_t*)&sx[wm * 16][0];
#pragma unroll
            for (int kk = 0; kk < BK; kk += 16) {
                uint32_t af[4];
                ldsm_x4(af, xa + (lane & 15) * LDS + kk + (lane >> 4) * 8);
#pragma unroll
                for (int j = 0; j < 4; j += 2) {
                    const int nr = wn * 32 + j * 8 + (lane & 7) + (lane >> 4) * 8, kc = kk + ((lane >> 3) & 1) * 8;
                    uint32_t bf[4];
                    ldsm_x4(bf, &sw0[nr][kc]);
                    mma_bf16_16816(&acc0[j * 4], af, bf);
                    mma_bf16_16816(&acc0[(j + 1) * 4], af, bf + 2);
                    if (DUAL) {
                        ldsm_x4(bf, &sw1[nr][kc]);
                        mma_bf16_16816(&acc1[j * 4], af, bf);
                        mma_bf16_16816(&acc1[(j + 1) * 4], af, bf + 2);
                    }
                }
            }
        } else {
            // a step's products are summed on their own and then added: the rounding error grows with K / BK + BK terms, not with K
            float p0[16], p1[DUAL ? 16 : 1];
#pragma unroll
            for (int i = 0; i < 16; i++) p0[i] = 0.f;
            if (DUAL)
#pragma unroll
                for (int i = 0; i < 16; i++) p1[DUAL ? i : 0] = 0.f;
#pragma unroll 8
            for (int k = 0; k < BK; k++) {
                float xv[4], wv[4], uv[4];
#pragma unroll
                for (int i = 0; i < 4; i++) xv[i] = ld_act<TA>(&sx[tr * 4 + i][k]);
#pragma unroll
                for (int j = 0; j < 4; j++) wv[j] = bf16_bits_to_f32(sw0[tc * 4 + j][k]);
                if (DUAL)
#pragma unroll
                    for (int j = 0; j < 4; j++) uv[j] = bf16_bits_to_f32(sw1[tc * 4 + j][k]);
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        p0[i * 4 + j] = fmaf(xv[i], wv[j], p0[i * 4 + j]);
                        if (DUAL) p1[DUAL ? i * 4 + j : 0] = fmaf(xv[i], uv[j], p1[DUAL ? i * 4 + j : 0]);
                    }
            }
#pragma unroll
            for (int i = 0; i < 16; i++) acc0[i] += p0[i];
            if (DUAL)
#pragma unroll
                for (int i = 0; i < 16; i++) acc1[DUAL ? i : 0] += p1[DUAL ? i : 0];
        }
    }
    auto store = [&](int r, int n, float v0, float v1) {
        const int s = m0 + r;
        if (s >= hi || n >= a.N) return;
        const float v = DUAL ? lin_pair(a, v0, v1) : lin_act(v0, a.act);
        if ((DUAL || a.act) && a.out_act == 1)
            ((uint16_t*)a.y)[(size_t)s * a.ldy + n] = f32_to_bf16_bits(v);
        else
            ((float*)a.y)[(size_t)s * a.ldy + n] = v;
    };
    if (MMA) {
        const int gr = lane >> 2, tg = lane & 3;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + wn * 32 + j * 8 + tg * 2, r = wm * 16 + gr;
            store(r, n, acc0[j * 4 + 0], DUAL ? acc1[j * 4 + 0] : 0.f);
            store(r, n + 1, acc0[j * 4 + 1], DUAL ? acc1[j * 4 + 1] : 0.f);
            store(r + 8, n, acc0[j * 4 + 2], DUAL ? acc1[j * 4 + 2] : 0.f);
            store(r + 8, n + 1, acc0[j * 4 + 3], DUAL ? acc1[j * 4 + 3] : 0.f);
        }
    } else {
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) store(tr * 4 + i, n0 + tc * 4 + j, acc0[i * 4 + j], DUAL ? acc1[i * 4 + j] : 0.f);
    }
    __syncthreads();  // the shared tiles are free for the next slot tile
    }
}

template <typename TA, bool DUAL>
int launch(kf_ctx* ctx, const LinArgs& a, int slots, int groups, bool gemv) {
    if (gemv) {
        dim3 grid((a.N + 7) / 8, slots);
        kf_lin_gemv_kernel<TA, DUAL><<<grid, 256, 0, ctx->stream>>>(a);
    } else {
        const int tiles = (slots + BM - 1) / BM;
        const int gy    = groups > 1 ? std::min(tiles, std::max(1, (2 * slots / groups + BM - 1) / BM)) : tiles;
        dim3 grid((a.N + BN - 1) / BN, gy, groups);
        kf_lin_tile_kernel<TA, DUAL><<<grid, 256, 0, ctx->stream>>>(a);
    }
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
int dispatch(kf_ctx* ctx, const LinArgs& a, int slots, int groups, bool gemv, bool dual, int act_f32) {
    if (act_f32) return dual ? launch<float, true>(ctx, a, slots, groups, gemv) : launch<float, false>(ctx, a, slots, groups, gemv);
    return dual ? launch<uint16_t, true>(ctx, a, slots, groups, gemv) : launch<uint16_t, false>(ctx, a, slots, groups, gemv);
}
constexpr int kGemvMaxSlots = 16;
// one weight, a panel of rows, few outputs and a long reduction: tiles would leave all but a handful of SMs idle
bool skinny_shape(const LinArgs& a) { return a.N <= 128 && a.K >= 512 && a.M > kGemvMaxSlots; }
int dispatch_one(kf_ctx* ctx, const LinArgs& a, int act_f32) {
    const bool skinny = skinny_shape(a);
    if (skinny && a.K % 8 == 0 && a.ldx % 8 == 0 && (((uintptr_t)a.W0 | (uintptr_t)a.x) & 15) == 0 && (a.M + kSkR - 1) / kSkR <= 65535) {
        if (!act_f32 && a.K % 32 == 0) {
            const int nt = (a.N + 7) / 8, blocks = (a.M + 15) / 16;
            if (nt <= 4) kf_lin_skinny_mma_kernel<4><<<blocks, 256, 0, ctx->stream>>>(a);
            else if (nt <= 8) kf_lin_skinny_mma_kernel<8><<<blocks, 256, 0, ctx->stream>>>(a);
            else if (nt <= 10) kf_lin_skinny_mma_kernel<10><<<blocks, 256, 0, ctx->stream>>>(a);
            else kf_lin_skinny_mma_kernel<16><<<blocks, 256, 0, ctx->stream>>>(a);
            KF_LAUNCH_CHECK(ctx);
            return KF_OK;
        }
        const dim3 grid((a.N + 8 * kSkC - 1) / (8 * kSkC), (a.M + kSkR - 1) / kSkR);
        if (act_f32) kf_lin_skinny_kernel<float><<<grid, 256, 0, ctx->stream>>>(a);
        else kf_lin_skinny_kernel<uint16_t><<<grid, 256, 0, ctx->stream>>>(a);
        KF_LAUNCH_CHECK(ctx);
        return KF_OK;
    }
    return dispatch(ctx, a, a.M, 1, a.M <= kGemvMaxSlots || (skinny && a.N <= 64), false, act_f32);
}
}  // namespace

extern "C" int kf_linear_g(kf_ctx* ctx, float* y, int ldy, const kf_tensor_desc* w, const void* x, int act_f32, int ldx, int M) {
    if (!ctx || !y || !w || !x) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, w->type == KF_T_BF16 && M >= 1 && w->rows >= 1 && w->cols >= 1 && ldx >= w->cols && ldy >= w->rows, "bf16 weight, ld >= extent");
    LinArgs a = {};
    a.W0 = (const uint16_t*)w->data_dev, a.x = x, a.y = y, a.M = M, a.N = w->rows, a.K = w->cols, a.ldx = ldx, a.ldy = ldy;
    // a few rows over a small weight: the warp-per-output kernel is through before the tuned ones have filled their pipelines (measured: 2.9 against
    // 5.3 us at 1024 x 1024, 4.5 against 6.0 at 2048 x 2048, even at 34 MB of weight x rows)
    const bool few = M <= kGemvMaxSlots && w->cols <= 4096 && (size_t)M * w->rows * w->cols * 2 <= ((size_t)34 << 20);
    // shapes the tuned kernels take go there (tcgen05 / TMEM panels, the HBM-rate GEMV); fp32 result through their fp32 epilogue
    if (!few && !skinny_shape(a) && !act_f32 && ldx == w->cols && ldy == w->rows && w->cols % 128 == 0 && w->rows % 16 == 0 && w->rows >= 16 && ctx->tc_min_m != 0 &&
        (((uintptr_t)w->data_dev | (uintptr_t)x | (uintptr_t)y) & 15) == 0)
        return kf_linear(ctx, y, w, x, M, KF_EPI_F32, nullptr);
    return dispatch_one(ctx, a, act_f32);
}
// y = silu(Wg x) * (Wu x), written in the activation type (bf16 bits, or float when act_f32)
extern "C" int kf_linear_g_swiglu(kf_ctx* ctx, void* y, int ldy, const kf_tensor_desc* wg, const kf_tensor_desc* wu, const void* x, int act_f32,
                                  int ldx, int M) {
    if (!ctx || !y || !wg || !wu || !x) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, wg->type == KF_T_BF16 && wu->type == KF_T_BF16 && wg->rows == wu->rows && wg->cols == wu->cols && M >= 1 && ldx >= wg->cols &&
                        ldy >= wg->rows, "gate / up: bf16, equal shapes");
    LinArgs a = {};
    a.W0 = (const uint16_t*)wg->data_dev, a.W1 = (const uint16_t*)wu->data_dev, a.x = x, a.y = y, a.M = M, a.N = wg->rows, a.K = wg->cols;
    a.ldx = ldx, a.ldy = ldy, a.out_act = act_f32 ? 0 : 1;
    return dispatch(ctx, a, M, 1, M <= kGemvMaxSlots, true, act_f32);
}
// Grouped matmul over expert-sorted slots.  w_table / w2_table: device arrays of n_groups bf16 weight pointers ([N][K] each);
// offsets: device int32 [n_groups + 1]; slot_group: device int32 [slots] (the expert of each slot); src_row: device int32 [slots] or
// NULL.  w2_table != NULL: y = silu(W x) * (W2 x) in the activation type; else y is float.  `slots` is the launch bound (tokens x top).
extern "C" int kf_linear_grouped(kf_ctx* ctx, void* y, int ldy, const void* const* w_table, const void* const* w2_table, int n_groups, int N, int K,
                                 const void* x, int act_f32, int ldx, const int32_t* offsets, const int32_t* slot_group, const int32_t* src_row,
                                 int slots) {
    if (!ctx || !y || !w_table || !x || !offsets || !slot_group) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n_groups >= 1 && N >= 1 && K >= 1 && slots >= 1 && ldx >= K && ldy >= N, "shape");
    LinArgs a = {};
    a.Wt0 = (const uint16_t* const*)w_table, a.Wt1 = (const uint16_t* const*)w2_table, a.x = x, a.y = y, a.M = slots, a.N = N, a.K = K;
    a.ldx = ldx, a.ldy = ldy, a.offsets = offsets, a.slot_group = slot_group, a.src_row = src_row, a.out_act = act_f32 ? 0 : 1;
    return dispatch(ctx, a, slots, n_groups, slots <= kGemvMaxSlots, w2_table != nullptr, act_f32);
}

// The single-weight grouped form with an activation on the result (1: gelu, tanh form; 2: relu squared), written in the activation type
// (bf16 bits, or float when act_f32): the up projection of experts that have no gate.  act 0 = kf_linear_grouped without a second table.
extern "C" int kf_linear_grouped_act(kf_ctx* ctx, void* y, int ldy, const void* const* w_table, int n_groups, int N, int K, const void* x, int act_f32, int ldx,
                                     const int32_t* offsets, const int32_t* slot_group, const int32_t* src_row, int slots, int act) {
    if (!ctx || !y || !w_table || !x || !offsets || !slot_group) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n_groups >= 1 && N >= 1 && K >= 1 && slots >= 1 && ldx >= K && ldy >= N && act >= 0 && act <= 2, "shape / act");
    LinArgs a = {};
    a.Wt0 = (const uint16_t* const*)w_table, a.x = x, a.y = y, a.M = slots, a.N = N, a.K = K;
    a.ldx = ldx, a.ldy = ldy, a.offsets = offsets, a.slot_group = slot_group, a.src_row = src_row, a.out_act = act_f32 ? 0 : 1, a.act = act;
    return dispatch(ctx, a, slots, n_groups, slots <= kGemvMaxSlots, false, act_f32);
}
// kf_linear_grouped's two-weight form with the clamped gate: y = g sigmoid(alpha g) (u + shift), g = min(W x, limit), u = clamp(W2 x, -limit,
// limit) (limit <= 0: not clamped), written in the activation type.  A slot whose slot_group is -1 is left out.
extern "C" int kf_linear_grouped_glu(kf_ctx* ctx, void* y, int ldy, const void* const* w_table, const void* const* w2_table, int n_groups, int N, int K,
                                     const void* x, int act_f32, int ldx, const int32_t* offsets, const int32_t* slot_group, const int32_t* src_row, int slots,
                                     float limit, float alpha, float shift) {
    if (!ctx || !y || !w_table || !w2_table || !x || !offsets || !slot_group) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n_groups >= 1 && N >= 1 && K >= 1 && slots >= 1 && ldx >= K && ldy >= N, "shape");
    LinArgs a = {};
    a.Wt0 = (const uint16_t* const*)w_table, a.Wt1 = (const uint16_t* const*)w2_table, a.x = x, a.y = y, a.M = slots, a.N = N, a.K = K;
    a.ldx = ldx, a.ldy = ldy, a.offsets = offsets, a.slot_group = slot_group, a.src_row = src_row, a.out_act = act_f32 ? 0 : 1;
    a.glu = 1, a.limit = limit, a.alpha = alpha, a.shift = shift;
    return dispatch(ctx, a, slots, n_groups, slots <= kGemvMaxSlots, true, act_f32);
}
// y[i][m] = act_i(W_i x[i][m]) for n <= 8 bf16 weights with the same number of columns, each with an input [M][ldx] and a float output [M][rows of
// W_i] of its own; act: 0 none, 3 tanh (host array, NULL: none).  A handful of rows: one launch; panels: one matmul per weight.
extern "C" int kf_linear_batch(kf_ctx* ctx, int n, float* const* y, const kf_tensor_desc* w, const void* const* x, const int* act, int act_f32, int ldx, int M) {
    if (!ctx || !y || !w || !x) return KF_ERR_BAD_ARG;
    KF_REQUIRE(ctx, n >= 1 && n <= kBatchMax && M >= 1, "1 .. 8 weights");
    for (int i = 0; i < n; i++) {
        KF_REQUIRE(ctx, y[i] && x[i] && w[i].type == KF_T_BF16 && w[i].rows >= 1 && w[i].cols == w[0].cols && ldx >= w[i].cols, "bf16 weights, equal columns");
        KF_REQUIRE(ctx, !act || act[i] == 0 || act[i] == 3, "act");
    }
    if (M > kGemvMaxSlots) {
        for (int i = 0; i < n; i++) {
            int rc;
            if (act && act[i]) {
                LinArgs a = {};
                a.W0 = (const uint16_t*)w[i].data_dev, a.x = x[i], a.y = y[i], a.M = M, a.N = w[i].rows, a.K = w[i].cols, a.ldx = ldx, a.ldy = w[i].rows, a.act = act[i];
                rc = dispatch_one(ctx, a, act_f32);
            } else {
                rc = kf_linear_g(ctx, y[i], w[i].rows, &w[i], x[i], act_f32, ldx, M);
            }
            if (rc) return rc;
        }
        return KF_OK;
    }
    BatchArgs a = {};
    a.n = n, a.K = w[0].cols, a.ldx = ldx;
    for (int i = 0; i < n; i++) {
        a.W[i] = (const uint16_t*)w[i].data_dev, a.x[i] = x[i], a.y[i] = y[i], a.N[i] = a.ldy[i] = w[i].rows, a.act[i] = act ? act[i] : 0;
        a.first[i + 1] = a.first[i] + (w[i].rows + 7) / 8;
    }
    const dim3 grid(a.first[n], M);
    if (act_f32) kf_lin_gemv_batch_kernel<float><<<grid, 256, 0, ctx->stream>>>(a);
    else kf_lin_gemv_batch_kernel<uint16_t><<<grid, 256, 0, ctx->stream>>>(a);
    KF_LAUNCH_CHECK(ctx);
    return KF_OK;
}
