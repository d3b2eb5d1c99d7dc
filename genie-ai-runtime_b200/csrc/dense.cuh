// dense.cuh — products with dense weights (bf16 or fp32, row-major [out][in], rows padded to a multiple of 8 elements,
// zero-filled): the decode family for one token (dense_gemv.cu), the tensor-core product for many (dense_tc.cu, bf16) and a
// CUDA-core product in true fp32 (dense_simt.cu).
#pragma once
#include "moe.cuh"

namespace jb {

// Consecutive output rows of a product that go to one place: y[token * ld + row], fp32 or the activation type.
struct OutSeg { void* y = nullptr; long long ld = 0; int rows = 0; int f32 = 0; int at_pos = 0; };   // at_pos: decode only, y += *d_pos * ld

// ── decode: one token ──
enum GemvMode {
    GEMV_NORM = 0,       // input: the residual step of layernorm.cuh (its h); CTA 0 stores x' and, when norm.h is set, h
    GEMV_PLAIN = 1,      // input: vector x of the activation type, pad8(K) elements
    GEMV_MOE_UP = 2,     // input x; routes the token from z, then out[k][f] = silu(gate row) * up row of expert ids[k], k < top, f < M; CTA 0 stores ids and wts
    GEMV_MOE_DOWN = 3,   // input x = [top][pad8(K)]; y[row] = sum_k wts[k] * (W[ids[k]][row] . x[k])
};
struct DenseGemv {
    int mode = GEMV_PLAIN, kind = EK_BF16;
    const void* W = nullptr; const void* W_up = nullptr;
    int M = 0, K = 0;
    OutSeg seg[3]; int nseg = 1;
    float softcap = 0.f;                     // y := softcap * tanh(y / softcap), fp32 outputs
    const int* d_pos = nullptr;
    const void* x = nullptr;
    NormStep norm;
    MoeRoute route; const float* z = nullptr; int* ids = nullptr; float* wts = nullptr;
};
int launch_dense_gemv(const DenseGemv& a, cudaStream_t st);

// ── many tokens ──
// y[t][r] = sum_k W[r][k] * x[t][k].  With groups (experts): W holds n_groups matrices of M rows one after the other and
// group g multiplies token rows [off[g], off[g + 1]) (off on the device).  swiglu: W is the gate, W_up the up matrix, and
// the output is silu(gate) * up.
struct DenseGemm {
    int kind = EK_BF16;
    const void* W = nullptr; const void* W_up = nullptr;
    int M = 0, K = 0, N = 0;                 // rows (per group), inner size, token rows in all
    const void* x = nullptr;                 // [N][pad8(K)]
    OutSeg seg[3]; int nseg = 1;
    float softcap = 0.f; int swiglu = 0;
    const int* off = nullptr; int n_groups = 1;
};
int launch_dense_gemm(const DenseGemm& a, cudaStream_t st);      // bf16: tensor cores; fp32: CUDA cores
int launch_dense_gemm_tc(const DenseGemm& a, cudaStream_t st);
int launch_dense_gemm_simt(const DenseGemm& a, cudaStream_t st);

#ifdef __CUDACC__
__device__ __forceinline__ float silu_f(float g) { return g / (1.0f + expf(-g)); }
template <typename T>
__device__ __forceinline__ void store_seg(const OutSeg* seg, int nseg, float softcap, const int* d_pos, long long token, int row, float v) {
    int s = 0;
    while (s + 1 < nseg && row >= seg[s].rows) { row -= seg[s].rows; ++s; }
    if (softcap > 0.f) v = softcap * tanhf(v / softcap);
    const long long o = (token + (seg[s].at_pos ? *d_pos : 0)) * seg[s].ld + row;
    if (seg[s].f32) reinterpret_cast<float*>(seg[s].y)[o] = v;
    else            reinterpret_cast<T*>(seg[s].y)[o] = from_f32<T>(v);
}
#endif

}  // namespace jb
