// moe.cuh — mixture-of-experts routing: sigmoid scores, a per-expert correction that enters the choice only, optional
// groups of consecutive experts of which a few stay eligible (ranked by best + second-best choice score of the group),
// the `top` largest choice scores among the eligible, weights = the scores without correction.
#pragma once
#include "layernorm.cuh"

namespace jb {

constexpr int MOE_MAX_EXPERTS = 1024, MOE_MAX_TOP = 64;

struct MoeRoute {
    int n_experts = 0, top = 0, n_groups = 1, keep_groups = 1;
    const float* correction = nullptr;          // [n_experts] or null
};

// Prompt path: routes `rows` tokens from their logits z [rows][n_experts]; ids / wts [rows][top]; counts[e] += tokens of
// expert e (zeroed by the caller), rank [rows][top] = the token's place among its expert's tokens.
int launch_moe_topk(const float* z, const MoeRoute& r, int rows, int* ids, float* wts, int* counts, int* rank, cudaStream_t st);
// Expert-major copy of the rows: off[e] = first slot of expert e (off[n_experts] = rows * top), slots [rows][top] =
// off[ids] + rank, hp[slot] = h[row].  Strides pad8(W) elements of `kind`.
int launch_moe_permute(const void* h, void* hp, int kind, int W, const MoeRoute& r, int rows, const int* ids, const int* rank, const int* counts,
                       int* slots, int* off, cudaStream_t st);

#ifdef __CUDACC__
// One warp routes one token.  z: n_experts logits (any memory); c, s: n_experts floats of shared memory each (left holding
// the choice and plain scores); emit(k, id, weight) runs on lane 0 for k = 0 .. top-1.  Equal scores: the lower index wins.
template <class Emit>
__device__ __forceinline__ void moe_route_warp(const float* z, const MoeRoute& r, float* c, float* s, float* gs, Emit emit) {
    const int lane = threadIdx.x & 31, E = r.n_experts;
    const float NINF = -INFINITY;
    for (int e = lane; e < E; e += 32) {
        const float v = 1.0f / (1.0f + expf(-z[e]));
        s[e] = v;
        c[e] = r.correction ? v + r.correction[e] : v;
    }
    __syncwarp();
    if (r.n_groups > 1 && r.keep_groups < r.n_groups) {
        const int n = E / r.n_groups;
        for (int g = lane; g < r.n_groups; g += 32) {
            float a = NINF, b = NINF;
            for (int i = 0; i < n; ++i) {
                const float v = c[g * n + i];
                if (v > a) { b = a; a = v; } else if (v > b) b = v;
            }
            gs[g] = n > 1 ? a + b : a;
        }
        __syncwarp();
        // a group is dropped when at least keep_groups groups come before it (larger score, or equal and lower index)
        for (int g = lane; g < r.n_groups; g += 32) {
            int before = 0;
            const float v = gs[g];
            for (int o = 0; o < r.n_groups; ++o) before += gs[o] > v || (gs[o] == v && o < g);
            if (before >= r.keep_groups) for (int i = 0; i < n; ++i) c[g * n + i] = NINF;
        }
        __syncwarp();
    }
    for (int k = 0; k < r.top; ++k) {
        float best = NINF; int bi = 0x7FFFFFFF;
        for (int e = lane; e < E; e += 32) if (c[e] > best) { best = c[e]; bi = e; }
        #pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xFFFFFFFFu, best, o); const int oi = __shfl_xor_sync(0xFFFFFFFFu, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        const bool ok = bi < E;                    // no eligible expert left only for logits that are not numbers
        if (lane == 0) emit(k, ok ? bi : 0, ok ? s[bi] : 0.f);
        __syncwarp();
        if (ok && lane == 0) c[bi] = NINF;
        __syncwarp();
    }
}
#endif

}  // namespace jb
