// moe.cu — routing of prompt tokens to experts (see moe.cuh).
#include "moe.cuh"

namespace jb {

constexpr int MT_WARPS = 4;

__global__ void __launch_bounds__(MT_WARPS * 32) moe_topk_kernel(const float* z, const MoeRoute r, int rows, int* ids, float* wts, int* counts, int* rank) {
    pdl_wait();
    extern __shared__ float mt_sm[];
    const int warp = threadIdx.x >> 5, row = blockIdx.x * MT_WARPS + warp, E = r.n_experts;
    if (row >= rows) return;
    float* c = mt_sm + (size_t)warp * (2 * E + r.n_groups);
    moe_route_warp(z + (size_t)row * E, r, c, c + E, c + 2 * E, [&](int k, int id, float w) {
        const size_t o = (size_t)row * r.top + k;
        ids[o] = id; wts[o] = w;
        rank[o] = atomicAdd(&counts[id], 1);
    });
}

template <typename T>
__global__ void __launch_bounds__(128) moe_permute_kernel(const T* h, T* hp, int W, const MoeRoute r, const int* ids, const int* rank, const int* counts,
                                                          int* slots, int* off, int rows) {
    pdl_wait();
    extern __shared__ int mp_off[];                          // [n_experts + 1]
    const int row = blockIdx.x, lane = threadIdx.x & 31, E = r.n_experts;
    if (threadIdx.x < 32) {                                  // exclusive prefix sums of the counts, 32 at a time
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int v = e0 + lane < E ? counts[e0 + lane] : 0;
            int s = v;
            #pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const int u = __shfl_up_sync(0xFFFFFFFFu, s, o); if (lane >= o) s += u; }
            if (e0 + lane < E) mp_off[e0 + lane] = base + s - v;
            base += __shfl_sync(0xFFFFFFFFu, s, 31);
        }
        if (lane == 0) mp_off[E] = base;
    }
    __syncthreads();
    if (row == 0) for (int e = threadIdx.x; e <= E; e += blockDim.x) off[e] = mp_off[e];
    const int ld = pad8(W), n16 = ld * (int)sizeof(T) / 16;
    const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)row * ld);
    for (int k = 0; k < r.top; ++k) {
        const size_t o = (size_t)row * r.top + k;
        const int slot = mp_off[ids[o]] + rank[o];
        if (threadIdx.x == 0) slots[o] = slot;
        uint4* dst = reinterpret_cast<uint4*>(hp + (size_t)slot * ld);
        for (int i = threadIdx.x; i < n16; i += blockDim.x) dst[i] = src[i];
    }
}

static int check_route(const MoeRoute& r) {
    if (r.n_experts <= 0 || r.n_experts > MOE_MAX_EXPERTS || r.top <= 0 || r.top > MOE_MAX_TOP || r.n_groups <= 0 || r.n_experts % r.n_groups ||
        r.keep_groups <= 0 || r.top > (r.keep_groups < r.n_groups ? r.keep_groups : r.n_groups) * (r.n_experts / r.n_groups))
        return set_error(JB_ERR_ARG, "router: %d experts, top %d, %d groups of which %d are kept", r.n_experts, r.top, r.n_groups, r.keep_groups);
    return JB_OK;
}

int launch_moe_topk(const float* z, const MoeRoute& r, int rows, int* ids, float* wts, int* counts, int* rank, cudaStream_t st) {
    const int rc = check_route(r);
    if (rc || rows <= 0) return rc;
    JB_CUDA(launch_k(moe_topk_kernel, dim3((rows + MT_WARPS - 1) / MT_WARPS), dim3(MT_WARPS * 32),
                     (size_t)MT_WARPS * (2 * r.n_experts + r.n_groups) * sizeof(float), st, pdl_enabled(), z, r, rows, ids, wts, counts, rank));
    count_launch();
    return JB_OK;
}
int launch_moe_permute(const void* h, void* hp, int kind, int W, const MoeRoute& r, int rows, const int* ids, const int* rank, const int* counts,
                       int* slots, int* off, cudaStream_t st) {
    const int rc = check_route(r);
    if (rc || rows <= 0) return rc;
    const size_t smem = (size_t)(r.n_experts + 1) * sizeof(int);
    if (kind == EK_BF16)
        JB_CUDA(launch_k(moe_permute_kernel<__nv_bfloat16>, dim3(rows), dim3(128), smem, st, pdl_enabled(), (const __nv_bfloat16*)h, (__nv_bfloat16*)hp, W, r, ids, rank, counts, slots, off, rows));
    else
        JB_CUDA(launch_k(moe_permute_kernel<float>, dim3(rows), dim3(128), smem, st, pdl_enabled(), (const float*)h, (float*)hp, W, r, ids, rank, counts, slots, off, rows));
    count_launch();
    return JB_OK;
}

}  // namespace jb
