// The element-wise half of what stands before a pass of a loop over layers:  x <- A x + B x0 + step  (one matrix [A | B]).
//
//   tb_pass_entry   lowp = x in the compute dtype (what the product with A reads), x <- base + step (float32; ``base`` = B x0, the
//                   same in every pass of a step, null: x itself; ``step`` a vector, null: zeros).  The product then adds into x.
#include "common.cuh"

namespace {

template <typename T, int V>
__global__ void __launch_bounds__(256) pass_entry_kernel(float* x, const float* __restrict__ base, const float* __restrict__ step, T* __restrict__ lowp, int W) {
    pdl_launch_dependents();
    struct alignas(4 * V) VF { float v[V]; };
    struct alignas(sizeof(T) * V) VT { T v[V]; };
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    VF s;
#pragma unroll
    for (int e = 0; e < V; ++e) s.v[e] = 0.f;
    if (step && i < W) s = *reinterpret_cast<const VF*>(step + i);      // a weight: no kernel writes it
    pdl_wait();
    if (i >= W) return;
    const size_t at = (size_t)blockIdx.x * W + i;
    const VF old = *reinterpret_cast<const VF*>(x + at);
    const VF b = base ? *reinterpret_cast<const VF*>(base + at) : old;
    VF r;
    VT low;
#pragma unroll
    for (int e = 0; e < V; ++e) { r.v[e] = b.v[e] + s.v[e]; stf(low.v + e, old.v[e]); }
    if (lowp) *reinterpret_cast<VT*>(lowp + at) = low;
    *reinterpret_cast<VF*>(x + at) = r;
}

template <typename T>
void launch(float* x, const float* base, const float* step, T* lowp, int rows, int W, cudaStream_t stream) {
    const bool vec = W % 4 == 0 && (((uintptr_t)x | (uintptr_t)base | (uintptr_t)step | (uintptr_t)lowp) & 15) == 0;
    const int n = vec ? W / 4 : W, threads = n >= 256 ? 256 : 64;
    dim3 grid(rows, (n + threads - 1) / threads);
    if (vec) tb_launch(pass_entry_kernel<T, 4>, grid, threads, 0, stream, x, base, step, lowp, W);
    else tb_launch(pass_entry_kernel<T, 1>, grid, threads, 0, stream, x, base, step, lowp, W);
}

}  // namespace

extern "C" int tb_pass_entry(float* x, const float* base, const float* step, void* lowp, int dtype, int rows, int W, cudaStream_t stream) {
    TB_REQUIRE(x && rows > 0 && W > 0 && (W + 63) / 64 <= 65535, "pass_entry: rows of the residual stream are wanted");
    if (!lowp || dtype == TB_F32) launch<float>(x, base, step, (float*)lowp, rows, W, stream);
    else if (dtype == TB_BF16) launch<__nv_bfloat16>(x, base, step, (__nv_bfloat16*)lowp, rows, W, stream);
    else TB_REQUIRE(false, "pass_entry: unknown dtype %d", dtype);
    TB_CHECK_LAUNCH("pass_entry");
    return 0;
}
