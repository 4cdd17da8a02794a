// Differential attention around the attention kernels: what comes between the projections and the scores, and what
// finishes the heads of a prompt that the tensor-core kernels ran.
//
// Every head has two softmax maps over the same values.  A token's projection row (float32) is
//     [q of head 0: map 1, map 2 | q of head 1 ... | k of kv head 0: map 1, map 2 | ... | v of kv head 0 | ...]
// with queries and keys of ``dim`` and values of ``vdim`` elements.  The cache keeps ONE row of ``hd`` elements per kv head
// and plane: the key row is [map 1 | map 2 | zeros] and the value row [v | zeros].  A map's query is laid out over the same
// hd elements with zeros where the other map lies, so that its product with the key row is that map's score alone: the two
// maps of a head are two query heads (2h, 2h + 1) of a kv head for every attention kernel, and a value is read once for both.
//
//   tb_pair_prep      adds the biases, RMS-norms every map's query and key over its dim (one weight each), and writes the
//                     query rows, the step's own key and value rows and the cache rows
//   tb_pair_combine   o = a_1 - lambda a_2 a head, over its root mean square, times a factor (float32 rows in)
#include "common.cuh"

struct PairPrepArgs {
    const float* in; int in_stride;         // [T][in_stride] float32: H * 2 * dim | G * 2 * dim | G * vdim  (G = 0: queries only)
    const float* bias;                      // added to the row first (null: none)
    const float* q_w; const float* k_w;     // [dim] each (null: that part is not normed)
    float eps;
    void* q_out; int q_stride;              // [T][q_stride] compute dtype: map m of head h at (2h + m) * hd
    void* kv_out; int kv_stride;            // [T][kv_stride]: G key rows, then G value rows, hd each (null: to the cache only)
    int H; int G; int dim; int vdim; int hd;
    const int* pos_of; const int* seq_of; const int* slot_of_seq;
    TbKvView cache; int append; int T;
};

namespace {

__device__ __forceinline__ void store_four(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* p, const float4& v) {
    alignas(8) __nv_bfloat16 t[4];
    stf(t, v.x); stf(t + 1, v.y); stf(t + 2, v.z); stf(t + 3, v.w);
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(t);
}

// A warp takes one piece of a token: a map of a query head, a map of a key head, or a value head.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) pair_prep_kernel(PairPrepArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int piece = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int nq = 2 * a.H, nk = 2 * a.G;
    if (piece >= nq + nk + a.G) return;
    const bool is_v = piece >= nq + nk, is_q = piece < nq;
    const int n = is_v ? a.vdim : a.dim;
    const int col = is_v ? (nq + nk) * a.dim + (piece - nq - nk) * a.vdim : piece * a.dim;
    const float* src = a.in + (size_t)t * a.in_stride + col;
    const float* bias = a.bias ? a.bias + col : nullptr;
    const float* w = is_v ? nullptr : (is_q ? a.q_w : a.k_w);
    float scale = 1.f;
    if (w) {
        float ss = 0.f;
        if (VEC) {
            for (int e = lane * 4; e < n; e += 128) {
                float4 v = *reinterpret_cast<const float4*>(src + e);
                if (bias) { const float4 c = *reinterpret_cast<const float4*>(bias + e); v.x += c.x; v.y += c.y; v.z += c.z; v.w += c.w; }
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
        } else {
            for (int e = lane; e < n; e += 32) {
                const float v = src[e] + (bias ? bias[e] : 0.f);
                ss = fmaf(v, v, ss);
            }
        }
        scale = 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps);
    }
    // where the piece's elements [0, n) go inside its row of hd elements, and which elements of the row this warp writes
    const int map = is_v ? 0 : piece & 1;
    const int at = map * a.dim, lo = is_q ? 0 : at, hi = (is_q || is_v || map) ? a.hd : a.dim;
    T* own = nullptr;
    T* page = nullptr;
    if (is_q) {
        own = (T*)a.q_out + (size_t)t * a.q_stride + (size_t)piece * a.hd;
    } else {
        const int head = is_v ? piece - nq - nk : (piece - nq) >> 1;
        if (a.kv_out) own = (T*)a.kv_out + (size_t)t * a.kv_stride + (size_t)(is_v ? a.G + head : head) * a.hd;
        if (a.append) page = (T*)a.cache.storage + (is_v ? kv_half_elems(a.cache) : 0) + kv_row_offset(a.cache, a.slot_of_seq[a.seq_of[t]], a.pos_of[t], head);
    }
    if (VEC) {
        // four neighbouring elements a lane
        for (int i = lo + lane * 4; i < hi; i += 128) {
            const int e = i - at;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (e >= 0 && e < n) {
                v = *reinterpret_cast<const float4*>(src + e);
                if (bias) { const float4 c = *reinterpret_cast<const float4*>(bias + e); v.x += c.x; v.y += c.y; v.z += c.z; v.w += c.w; }
                if (w) {
                    const float4 c = *reinterpret_cast<const float4*>(w + e);
                    v.x = v.x * scale * c.x; v.y = v.y * scale * c.y; v.z = v.z * scale * c.z; v.w = v.w * scale * c.w;
                }
            }
            if (own) store_four(own + i, v);
            if (page) store_four(page + i, v);
        }
        return;
    }
    for (int i = lo + lane; i < hi; i += 32) {
        const int e = i - at;
        float v = 0.f;
        if (e >= 0 && e < n) v = (src[e] + (bias ? bias[e] : 0.f)) * scale * (w ? w[e] : 1.f);
        if (own) stf(own + i, v);
        if (page) stf(page + i, v);
    }
}

// grid (rows, ceil(H / 4)); a warp a head: both maps' rows [hd] of one token, float32.
template <typename T>
__global__ void __launch_bounds__(128) pair_combine_kernel(const float* __restrict__ in, int in_stride, int hd, const float* __restrict__ lambda,
                                                           T* __restrict__ out, int out_stride, int H, int width, float eps, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
    if (h >= H) return;
    const float* a1 = in + (size_t)blockIdx.x * in_stride + (size_t)(2 * h) * hd;
    const float* a2 = a1 + hd;
    const float lam = *lambda;
    T* o = out + (size_t)blockIdx.x * out_stride + (size_t)h * width;
    float ss = 0.f;
    if (width <= 128 && (width & 3) == 0 && (hd & 3) == 0 && (in_stride & 3) == 0) {      // four neighbouring elements a lane, kept in registers
        float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
        if (lane * 4 < width) {
            const float4 u = reinterpret_cast<const float4*>(a1)[lane], v = reinterpret_cast<const float4*>(a2)[lane];
            d = make_float4(fmaf(-lam, v.x, u.x), fmaf(-lam, v.y, u.y), fmaf(-lam, v.z, u.z), fmaf(-lam, v.w, u.w));
        }
        ss = d.x * d.x + d.y * d.y + d.z * d.z + d.w * d.w;
        const float r = scale / sqrtf(warp_sum(ss) / (float)width + eps);
        if (lane * 4 < width) {
            alignas(16) T four[4];
            stf(four, d.x * r); stf(four + 1, d.y * r); stf(four + 2, d.z * r); stf(four + 3, d.w * r);
            if ((out_stride & 3) == 0) {
                if (sizeof(T) == 2) *reinterpret_cast<uint2*>(o + lane * 4) = *reinterpret_cast<const uint2*>(four);
                else *reinterpret_cast<uint4*>(o + lane * 4) = *reinterpret_cast<const uint4*>(four);
            } else {
                for (int i = 0; i < 4; ++i) o[lane * 4 + i] = four[i];
            }
        }
        return;
    }
    for (int e = lane; e < width; e += 32) {
        const float d = fmaf(-lam, a2[e], a1[e]);
        ss = fmaf(d, d, ss);
    }
    const float r = scale / sqrtf(warp_sum(ss) / (float)width + eps);
    for (int e = lane; e < width; e += 32) stf(o + e, fmaf(-lam, a2[e], a1[e]) * r);
}

}  // namespace

extern "C" int tb_pair_prep(const PairPrepArgs* args, int dtype, cudaStream_t stream) {
    PairPrepArgs a = *args;
    TB_REQUIRE(a.T > 0 && a.H > 0 && a.G >= 0 && a.dim > 0 && a.vdim > 0, "pair_prep: sizes must be positive");
    TB_REQUIRE(a.hd >= 2 * a.dim && a.hd >= a.vdim, "pair_prep: a row of %d elements for two maps of %d and values of %d", a.hd, a.dim, a.vdim);
    TB_REQUIRE(a.in && a.q_out && a.in_stride >= (2 * a.H + 2 * a.G) * a.dim + a.G * a.vdim, "pair_prep: the projection row is too short");
    TB_REQUIRE(a.q_stride >= 2 * a.H * a.hd && (!a.kv_out || a.kv_stride >= 2 * a.G * a.hd), "pair_prep: output rows are too short");
    TB_REQUIRE(!a.append || (a.cache.storage && a.cache.kv_heads == a.G && a.cache.head_dim == a.hd && a.cache.ring_rows == 0),
               "pair_prep: the cache view does not match the heads (a cache that keeps every key is wanted)");
    const int pieces = 2 * a.H + 3 * a.G, warps = 8;
    TB_REQUIRE((pieces + warps - 1) / warps <= 65535, "pair_prep: too many heads");
    const dim3 grid(a.T, (pieces + warps - 1) / warps);
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.hd % 4 == 0 && a.in_stride % 4 == 0 && a.q_stride % 4 == 0 && a.kv_stride % 4 == 0 &&
                     (((uintptr_t)a.in | (uintptr_t)a.bias | (uintptr_t)a.q_w | (uintptr_t)a.k_w | (uintptr_t)a.q_out | (uintptr_t)a.kv_out | (uintptr_t)a.cache.storage) & 15) == 0;
    if (dtype == TB_F32) {
        if (vec) tb_launch(pair_prep_kernel<float, true>, grid, warps * 32, 0, stream, a);
        else tb_launch(pair_prep_kernel<float, false>, grid, warps * 32, 0, stream, a);
    } else if (dtype == TB_BF16) {
        if (vec) tb_launch(pair_prep_kernel<__nv_bfloat16, true>, grid, warps * 32, 0, stream, a);
        else tb_launch(pair_prep_kernel<__nv_bfloat16, false>, grid, warps * 32, 0, stream, a);
    }
    else TB_REQUIRE(false, "pair_prep: unknown dtype %d", dtype);
    TB_CHECK_LAUNCH("pair_prep");
    return 0;
}

extern "C" int tb_pair_combine(const float* in, int in_stride, int hd, const float* lambda, void* out, int out_stride, int dtype, int rows, int H,
                               int width, float eps, float scale, cudaStream_t stream) {
    TB_REQUIRE(in && lambda && out && rows > 0 && H > 0 && width > 0 && width <= hd && (H + 3) / 4 <= 65535, "pair_combine: rows of pairs of heads are wanted");
    TB_REQUIRE(in_stride >= 2 * H * hd && out_stride >= H * width && (((uintptr_t)in | (uintptr_t)out) & 15) == 0, "pair_combine: row strides, or buffers that are not 16-byte aligned");
    const dim3 grid(rows, (H + 3) / 4);
    if (dtype == TB_F32) tb_launch(pair_combine_kernel<float>, grid, 128, 0, stream, in, in_stride, hd, lambda, (float*)out, out_stride, H, width, eps, scale);
    else if (dtype == TB_BF16) tb_launch(pair_combine_kernel<__nv_bfloat16>, grid, 128, 0, stream, in, in_stride, hd, lambda, (__nv_bfloat16*)out, out_stride, H, width, eps, scale);
    else TB_REQUIRE(false, "pair_combine: unknown dtype %d", dtype);
    TB_CHECK_LAUNCH("pair_combine");
    return 0;
}
