// moe_ops.cuh -- a feed-forward made of routed experts, around the matrix kernels of dense_ops.cuh / dense_gemm.cuh:
//   moe_logits_kernel    router logits in f32 (f32 router matrix), and the logits of further rows stacked below the router's (a
//                        gate on a shared expert)
//   moe_topk_kernel      score = sigmoid(logit), or the softmax over all logits; the `top` experts with the largest
//                        score + correction[e] are chosen, their weights are score / (sum of chosen scores + 1e-20) * scale; the
//                        choice may be limited to the best `keep` of `groups` equal groups of neighbouring experts
//   moe_sort_kernel      (token, choice) pairs counted and sorted by expert: row offsets per expert, the slot of every pair,
//                        the token of every slot
//   moe_gather_kernel    the normalised rows copied into expert order (the grouped matrix kernels then see one contiguous row
//                        range per expert)
//   moe_combine_kernel   x += f(sum over the token's choices of weight * expert output), f = a tanh norm on the way into the
//                        residual (or the identity); or the sum stored for a norm that needs statistics.  Experts beyond
//                        the ones with matrices are identity experts (their output is the token's input row); a shared
//                        expert's output row can be added, times the sigmoid of one logit per token
//   moe_combine_layernorm_kernel   the same sum through a layer norm into the residual stream: one CTA per token, or a
//                        single token's columns over several CTAs of which the last one to finish applies the norm
//   moe_combine_resnorm_kernel     the same sum through an RMS norm into the residual stream (resnorm_rows_kernel's row pass)
// A one-row step needs no sorting: the one-row matrix kernel takes the chosen experts from the router's device-side list.
#pragma once
#include "dense_ops.cuh"

namespace lmrs {
namespace dense {

template <typename AT> struct MoeRouterParams {
    const AT* h; int ld;          // [T][width] normalised input (operand type), or null:
    const float* x; TanhNorm tn;  // ... the residual row, normalised here (tanh norm) and rounded to the operand type
    const float* router;          // [E][width]
    const float* correction;      // [E], added for the choice only
    int E, top, width;
    int extra;                    // further rows of `router` (behind the E) whose logits are computed with it and never chosen
    int groups, keep;             // groups > 1: E / groups neighbouring outputs form a group that scores its largest choice score;
                                  // only the `keep` best groups can be chosen from (keep * (E / groups) >= top)
    int softmax;                  // 0: score = sigmoid(logit); 1: scores = softmax over the E logits; 2: the largest logits are
                                  // chosen and the weights are the softmax over the chosen logits only (times scale)
    const float* bias;            // [E] or null: added to the router logits
    float scale;
    float* z;                     // [T][E + extra] router logits (scratch between the two kernels)
    int* idx; float* wts;         // [T][top]
};
// logits: one warp per (token, expert), so that a single token still spreads over E warps on many SMs
template <typename AT> __global__ void __launch_bounds__(128) moe_logits_kernel(const MoeRouterParams<AT> p) {
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int e = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int rows = p.E + p.extra;
    if (e >= rows) return;
    const float* w = p.router + (size_t)e * p.width;
    float a = 0.0f;
    if (p.h) {
        const AT* h = p.h + (size_t)t * p.ld;
#pragma unroll 8
        for (int c = lane; c < p.width; c += 32) a = fmaf(w[c], to_f(h[c]), a);
    } else {
        const float* x = p.x + (size_t)t * p.ld;
        const float alpha = *p.tn.alpha;
#pragma unroll 8
        for (int c = lane; c < p.width; c += 32) { AT r; from_f(r, tanhnorm_apply(p.tn, alpha, c, x[c])); a = fmaf(w[c], to_f(r), a); }
    }
    a = warp_sum(a);
    if (lane == 0) p.z[(size_t)t * rows + e] = p.bias && e < p.E ? a + p.bias[e] : a;
}
// choice: one warp per token
template <typename AT> __global__ void __launch_bounds__(32) moe_topk_kernel(const MoeRouterParams<AT> p) {
    extern __shared__ __align__(16) float mr_sm[];
    float* score = mr_sm;            // [E] sigmoid(logit)
    float* choice = score + p.E;     // [E] score + correction; -inf once chosen or when its group is out
    float* gscore = choice + p.E;    // [groups] (groups > 1)
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x;
    const float* zt = p.z + (size_t)t * (p.E + p.extra);
    float zmax = -INFINITY, zsum = 0.0f;
    if (p.softmax == 1) {
        for (int e = lane; e < p.E; e += 32) zmax = fmaxf(zmax, zt[e]);
        zmax = warp_max(zmax);
        for (int e = lane; e < p.E; e += 32) zsum += expf(zt[e] - zmax);
        zsum = warp_sum(zsum);
    }
    for (int e = lane; e < p.E; e += 32) {
        const float z = zt[e];
        const float sg = p.softmax == 2 ? z : (p.softmax == 1 ? expf(z - zmax) / zsum : 1.0f / (1.0f + expf(-z)));
        score[e] = sg;
        choice[e] = sg + (p.correction ? p.correction[e] : 0.0f);
    }
    __syncwarp();
    if (p.groups > 1) {
        const int size = p.E / p.groups;
        for (int g = lane; g < p.groups; g += 32) {
            float m = choice[g * size];
            for (int i = 1; i < size; i++) m = fmaxf(m, choice[g * size + i]);
            gscore[g] = m;
        }
        __syncwarp();
        for (int g = lane; g < p.groups; g += 32) {   // a group stays when fewer than `keep` others are better (a tie: the lower index)
            int better = 0;
            for (int o = 0; o < p.groups; o++) better += gscore[o] > gscore[g] || (gscore[o] == gscore[g] && o < g) ? 1 : 0;
            if (better >= p.keep)
                for (int i = 0; i < size; i++) choice[g * size + i] = -INFINITY;
        }
        __syncwarp();
    }
    float sum = 0.0f;
    for (int k = 0; k < p.top; k++) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < p.E; e += 32)
            if (choice[e] > best) { best = choice[e]; bi = e; }   // ascending e: the lowest index wins a tie inside a lane
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
        }
        if (bi >= p.E) bi = k;   // scores that are no numbers compare with nothing: stay inside the list
        const float sg = score[bi];
        sum += sg;
        if (lane == 0) { p.idx[(size_t)t * p.top + k] = bi; p.wts[(size_t)t * p.top + k] = sg; choice[bi] = -INFINITY; }
        __syncwarp();
    }
    if (p.softmax == 2) {   // the first choice holds the largest logit: weights exp(z_k - z_0) / sum
        __syncwarp();
        const float z0 = p.wts[(size_t)t * p.top];
        float es = 0.0f;
        for (int k = lane; k < p.top; k += 32) es += expf(p.wts[(size_t)t * p.top + k] - z0);
        es = warp_sum(es);
        for (int k = lane; k < p.top; k += 32) p.wts[(size_t)t * p.top + k] = expf(p.wts[(size_t)t * p.top + k] - z0) / es * p.scale;
        return;
    }
    const float f = p.scale / (sum + 1e-20f);
    for (int k = lane; k < p.top; k += 32) p.wts[(size_t)t * p.top + k] *= f;
}

// n = T * top pairs.  One CTA: histogram, exclusive scan, placement.  Which pair of an expert gets which of the expert's
// slots depends on the order the atomics land in; every row is computed on its own, so the results do not.
struct MoeSortParams {
    const int* idx; int n, E, top;
    int* grp;       // [E + 1]
    int* slot;      // [n]: slot of pair (t, k)
    int* row_of;    // [n]: token of a slot
};
static __global__ void __launch_bounds__(1024) moe_sort_kernel(const MoeSortParams p) {
    extern __shared__ int ms_sm[];   // [E] counts, then [E] cursors
    int* cnt = ms_sm;
    int* cur = cnt + p.E;
    pdl_launch();
    pdl_wait();
    for (int e = threadIdx.x; e < p.E; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < p.n; i += blockDim.x) atomicAdd(&cnt[p.idx[i]], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        int a = 0;
        for (int e = 0; e < p.E; e++) { p.grp[e] = a; cur[e] = a; a += cnt[e]; }
        p.grp[p.E] = a;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.n; i += blockDim.x) {
        const int s = atomicAdd(&cur[p.idx[i]], 1);
        p.slot[i] = s;
        p.row_of[s] = i / p.top;
    }
}

template <typename AT> struct MoeGatherParams {
    const AT* h; int ld; const int* row_of; AT* out; int width;
};
template <typename AT> __global__ void __launch_bounds__(128) moe_gather_kernel(const MoeGatherParams<AT> p) {
    pdl_launch();
    pdl_wait();
    const AT* src = p.h + (size_t)p.row_of[blockIdx.x] * p.ld;
    AT* dst = p.out + (size_t)blockIdx.x * p.width;
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) dst[c] = src[c];
}

struct MoeCombineParams {
    const float* y;           // [slots][width] expert outputs
    const int* slot;          // [T][top] slot of every pair, or null: pair (t, k) sits in slot t*top + k
    const float* wts;         // [T][top]
    float* x; int ldx;        // residual stream
    TanhNorm n;               // n.alpha null: x += sum;  else x += tanh(alpha * sum) * w + b
    int top, width;
    const int* idx; int n_real;        // idx set: a pair whose expert idx[t][k] >= n_real is an identity expert ...
    const float* xin; int ld_in;       // ... whose output is row t of xin
    const float* add;                  // or null: [T][width] added to the sum (a shared expert's output) ...
    const float* add_gate; int ld_gate;   // ... times sigmoid(add_gate[t * ld_gate]) when set
    float* out; int ldo;               // when set: the sum is stored here and x is left alone
};
DN_DEVINL float moe_add_gate(const MoeCombineParams& p, int t) { return p.add_gate ? 1.0f / (1.0f + expf(-p.add_gate[(size_t)t * p.ld_gate])) : 1.0f; }
// the weighted sum of one token's expert outputs at column c; ag = moe_add_gate of the token
DN_DEVINL float moe_combined(const MoeCombineParams& p, int t, int c, float ag = 1.0f) {
    float a = p.add ? ag * p.add[(size_t)t * p.width + c] : 0.0f;
    for (int k = 0; k < p.top; k++) {
        const float w = p.wts[(size_t)t * p.top + k];
        if (p.idx && p.idx[(size_t)t * p.top + k] >= p.n_real) { a = fmaf(w, p.xin[(size_t)t * p.ld_in + c], a); continue; }
        const int s = p.slot ? p.slot[(size_t)t * p.top + k] : t * p.top + k;
        a = fmaf(w, p.y[(size_t)s * p.width + c], a);
    }
    return a;
}
static __global__ void __launch_bounds__(256) moe_combine_kernel(const MoeCombineParams p) {
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    const float alpha = p.n.alpha ? *p.n.alpha : 0.0f, ag = moe_add_gate(p, t);
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.width; c += gridDim.y * blockDim.x) {
        const float a = moe_combined(p, t, c, ag);
        if (p.out) p.out[(size_t)t * p.ldo + c] = a;
        else p.x[(size_t)t * p.ldx + c] += p.n.alpha ? tanhnorm_apply(p.n, alpha, c, a) : a;
    }
}
// the same sum sent through a layer norm into the residual stream, x <- x + ls * LN(sum) w, and x again in the operand type
// to h.  The norm needs the whole row: with gridDim.y == 1 one CTA per token computes the row and holds it in registers.  A
// single token (gridDim.x == 1) may instead spread its columns over gridDim.y CTAs, which store the sums in c.out; each takes a
// ticket from *counter when its stores are done and the one that comes last applies the norm (nobody waits; that CTA puts
// the counter back to zero).
template <typename AT> struct MoeCombineNormParams {
    MoeCombineParams c;
    const float* w; const float* ls; float eps;
    AT* h; int ldh;
    unsigned int* counter;
};
template <typename AT> __global__ void __launch_bounds__(256) moe_combine_layernorm_kernel(const MoeCombineNormParams<AT> p) {
    __shared__ float red[33];
    __shared__ unsigned int last;
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    float* xr = p.c.x + (size_t)t * p.c.ldx;
    const float ag = moe_add_gate(p.c, t);
    if (gridDim.y == 1) {
        layernorm_row<AT>([&](int c) { return moe_combined(p.c, t, c, ag); }, p.c.width, p.w, p.eps, red, xr, p.ls, nullptr, p.h + (size_t)t * p.ldh);
        return;
    }
    float* row = p.c.out + (size_t)t * p.c.ldo;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.c.width; c += gridDim.y * blockDim.x) row[c] = moe_combined(p.c, t, c, ag);
    __threadfence();   // this thread's stores of the row before the ticket
    __syncthreads();
    if (threadIdx.x == 0) last = atomicAdd(p.counter, 1u) == gridDim.y - 1 ? 1u : 0u;
    __syncthreads();
    if (!last) return;
    __threadfence();
    layernorm_row<AT>([&](int c) { return __ldcg(row + c); }, p.c.width, p.w, p.eps, red, xr, p.ls, nullptr, p.h + (size_t)t * p.ldh);
    if (threadIdx.x == 0) *p.counter = 0u;
}

// the same sum sent through an RMS norm into the residual stream, x <- x + rms(sum) w, with x again in the operand type to h: one CTA
// per token (ONE: a single token, up to 1024 threads).  A thread loads its columns of several experts before it adds the first.
struct MoeRow {
    const MoeCombineParams& p;
    int t;
    float ag;
    template <int CACHE> DN_DEVINL void fill(float (&v)[CACHE]) const {
        constexpr int KU = CACHE <= 4 ? 4 : (CACHE <= 8 ? 2 : 1);   // experts in flight
#pragma unroll
        for (int i = 0; i < CACHE; i++) {
            const int c = threadIdx.x + i * blockDim.x;
            v[i] = p.add && c < p.width ? ag * p.add[(size_t)t * p.width + c] : 0.0f;
        }
        for (int k0 = 0; k0 < p.top; k0 += KU) {
            float w[KU], e[KU][CACHE];
#pragma unroll
            for (int u = 0; u < KU; u++) {
                const int k = min(k0 + u, p.top - 1);
                const size_t pair = (size_t)t * p.top + k;
                w[u] = k0 + u < p.top ? p.wts[pair] : 0.0f;
                const float* row = p.idx && p.idx[pair] >= p.n_real ? p.xin + (size_t)t * p.ld_in : p.y + (p.slot ? (size_t)p.slot[pair] : pair) * p.width;
#pragma unroll
                for (int i = 0; i < CACHE; i++) {
                    const int c = threadIdx.x + i * blockDim.x;
                    e[u][i] = c < p.width ? row[c] : 0.0f;
                }
            }
#pragma unroll
            for (int u = 0; u < KU; u++)
#pragma unroll
                for (int i = 0; i < CACHE; i++)
                    if (k0 + u < p.top) v[i] = fmaf(w[u], e[u][i], v[i]);
        }
    }
    DN_DEVINL float at(int c) const { return moe_combined(p, t, c, ag); }
};
template <typename AT> struct MoeCombineResNormParams {
    MoeCombineParams c;
    const float* w; float eps;
    AT* h; int ldh;
};
// CACHE: columns a thread holds (a row of up to CACHE * blockDim.x stays in registers)
template <typename AT, bool ONE, int CACHE> __global__ void __launch_bounds__(ONE ? 1024 : 256) moe_combine_resnorm_kernel(const MoeCombineResNormParams<AT> p) {
    __shared__ float red[33];
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    sandwich_row<AT, CACHE, ONE>(MoeRow{p.c, t, moe_add_gate(p.c, t)}, p.c.width, p.c.x + (size_t)t * p.c.ldx, p.w, p.eps, red, nullptr, nullptr, nullptr,
                                        false, p.h + (size_t)t * p.ldh, nullptr);
}

}  // namespace dense
}  // namespace lmrs
