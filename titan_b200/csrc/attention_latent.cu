// Decode attention over a shared latent on tensor cores (bfloat16 rows of up to 1,024 elements in pages of 64).
//
// Every head of a latent-attention mixer scores the SAME cached row [latent r | rotated part | padding] and takes the row's
// latent part as its value, so up to 16 heads are the 16 rows of one mma.sync tile and a row is read once for all of them.
// One CTA per (sequence, group of 16 heads, split of the keys): a producer warp brings whole pages (64 rows, boxes of 64
// columns, 128-byte swizzled) into a ring of shared memory by TMA; per page
//     S[16 x 64] = Q . K^T       eight warps, eight keys each, over the whole row
//     softmax                    sixteen threads a head: running maximum and sum, float32; the weights go to shared memory as two
//                                bfloat16 halves (the rounded weight and what rounding left over), sixteen bits of each
//     O[16 x r] += P . V         eight warps, every eighth pair of 8-column tiles each, the page read again as V
// Partials (maximum, sum, unnormalised output) go to scratch in the layout of tb_attn_merge, which finishes (and adds a sink).
// A sequence's keys are cut by its own length and the launch's two numbers (tb_split_keys).
//
// All waits are bounded (tma.cuh); tb_attn_latent_error() reads the error word.
#include <float.h>

#include "attention_args.h"
#include "common.cuh"
#include "mma.cuh"
#include "tma.cuh"

int tb_make_map_bf16(CUtensorMap* out, const void* ptr, long long rows, long long cols, long long stride, int box_rows);

namespace {

using namespace tbtma;
using namespace tbmma;

__device__ unsigned int g_latent_error = 0;

constexpr int PAGE = 64, WARPS = 8, THREADS = (WARPS + 1) * 32, HEADS = 16;
constexpr int S_PITCH = 68, P_PITCH = 72;            // floats, bfloat16s: rows of whole 16 bytes that spread over the banks

struct LatentDecArgs {
    const __nv_bfloat16* q; int q_stride;            // [B][q_stride], head h at h * dk
    float* scratch;                                  // [B][nh][n_splits][r + 2]
    const int* table; int table_width; int ring_rows;
    const int* slot_of_seq; const int* kv_len;
    const int* early_len; int early_mode;            // lengths that were final before the step's first kernel (AttnArgs); 0: none
    int nh; int dk; int r; int boxes; int stages; int window; float scale_log2;
    int chunk; int n_splits;
};

__host__ __device__ __forceinline__ int q_pitch(int boxes) { return boxes * 64 + 8; }

// NP: pairs of 8-column output tiles a warp holds (r <= 128 * NP).
template <int NP>
__global__ void __launch_bounds__(THREADS, 1)
attn_decode_latent_kernel(const __grid_constant__ CUtensorMap map, LatentDecArgs a) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* base = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t stage_bytes = (uint32_t)a.boxes * 8192u;
    __nv_bfloat16* q_sh = (__nv_bfloat16*)(base + (size_t)a.stages * stage_bytes);      // [16][q_pitch]
    const int qp = q_pitch(a.boxes);
    float* s_sh = (float*)(q_sh + HEADS * qp);                                           // [16][S_PITCH]
    __nv_bfloat16* p_hi = (__nv_bfloat16*)(s_sh + HEADS * S_PITCH);                      // [16][P_PITCH]
    __nv_bfloat16* p_lo = p_hi + HEADS * P_PITCH;
    float* alpha_sh = (float*)(p_lo + HEADS * P_PITCH);                                  // [16]
    uint64_t* full = (uint64_t*)(alpha_sh + HEADS);
    uint64_t* empty = full + 2;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.x, h0 = blockIdx.y * HEADS, split = blockIdx.z;
    const bool early = a.early_mode != 0;
    if (!early) { pdl_launch_dependents(); pdl_wait(); }
    const int len = a.early_mode == 2 ? a.early_len[a.slot_of_seq[b]] + 1 : (early ? a.early_len[b] : a.kv_len[b]);
    const int keys = tb_split_keys(len, a.chunk, a.n_splits);
    if ((long long)split * keys >= len) return;      // uniform over the CTA; the merge skips these splits
    const int wlo = a.window > 0 ? max(0, len - a.window) : 0;
    const int lo = max(wlo, split * keys), hi = (int)min((long long)len, (long long)(split + 1) * keys);
    const int page0 = lo / PAGE, n_pages = lo < hi ? (hi - 1) / PAGE - page0 + 1 : 0;

    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; ++s) { mbar_init(full + s, 1); mbar_init(empty + s, WARPS); }
        mbar_fence_init();
    }
    __syncthreads();

    if (warp == WARPS) {                             // ---------------- producer
        if (lane == 0) {
            const int* tab = a.table + (size_t)a.slot_of_seq[b] * a.table_width;
            // before the wait for the kernels ahead: pages of older positions only, never the one whose newest row is still being written
            const int old_pages = n_pages - (hi == len && n_pages > 0 ? 1 : 0), ahead = early ? min(old_pages, a.stages) : 0;
            for (int i = 0; i < n_pages; ++i) {
                if (early && i == ahead) {
                    pdl_wait();
                    if (a.kv_len[b] != len) atomicCAS(&g_latent_error, 0u, 7u);          // the early length was not the step's
                }
                const int s = i % a.stages, round = i / a.stages;
                if (round > 0) mbar_wait(empty + s, (round - 1) & 1, &g_latent_error, 1);
                const int pos0 = (page0 + i) * PAGE;
                const int row = tab[(a.ring_rows ? pos0 % a.ring_rows : pos0) / PAGE] * PAGE;
                mbar_expect_tx(full + s, stage_bytes);
                for (int x = 0; x < a.boxes; ++x) tma_load_2d(base + (size_t)s * stage_bytes + x * 8192, &map, full + s, x * 64, row);
            }
            if (early && ahead >= n_pages) {         // everything was requested ahead: check the length all the same
                pdl_wait();
                if (a.kv_len[b] != len) atomicCAS(&g_latent_error, 0u, 7u);
            }
        }
        if (early) pdl_launch_dependents();
        return;
    }

    // ---------------- compute warps
    if (early) { pdl_wait(); pdl_launch_dependents(); }
    const int tid = threadIdx.x;                     // 0 .. 255
    {
        const int chunks = a.boxes * 8, have = a.dk / 8;
        for (int i = tid; i < HEADS * chunks; i += WARPS * 32) {
            const int row = i / chunks, c = i - row * chunks;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (c < have && h0 + row < a.nh) v = *reinterpret_cast<const uint4*>(a.q + (size_t)b * a.q_stride + (size_t)(h0 + row) * a.dk + c * 8);
            *reinterpret_cast<uint4*>(q_sh + row * qp + c * 8) = v;
        }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const int g = lane >> 2, t = lane & 3, mtx = lane >> 3, r8 = lane & 7;
    const uint32_t q_addr = smem_u32(q_sh + ((mtx & 1) * 8 + r8) * qp + (mtx >> 1) * 8);
    const uint32_t ph_addr = smem_u32(p_hi + ((mtx & 1) * 8 + r8) * P_PITCH + (mtx >> 1) * 8);
    const uint32_t pl_addr = smem_u32(p_lo + ((mtx & 1) * 8 + r8) * P_PITCH + (mtx >> 1) * 8);
    float o[NP][2][4];
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) o[j][n][0] = o[j][n][1] = o[j][n][2] = o[j][n][3] = 0.f;
    float m_run = -1e30f, l_run = 0.f;               // of row tid / 16, the same in its sixteen threads

    for (int i = 0; i < n_pages; ++i) {
        const int s = i % a.stages;
        mbar_wait(full + s, (i / a.stages) & 1, &g_latent_error, 2);
        const uint32_t page = smem_u32(base) + (uint32_t)s * stage_bytes;
        {   // S: keys 8 * warp .. + 7, two sums of every other 16 dimensions
            float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
            const int key = warp * 8 + r8;
            for (int ks = 0; ks < a.boxes * 4; ks += 2) {
                uint32_t a0, a1, a2, a3, e0, e1, e2, e3, b0, b1, b2, b3;
                ldsm_x4(q_addr + ks * 32, a0, a1, a2, a3);
                ldsm_x4(q_addr + ks * 32 + 32, e0, e1, e2, e3);
                const int dim0 = ks * 16 + mtx * 8;
                ldsm_x4(page + (dim0 >> 6) * 8192 + swz(key, (dim0 & 63) >> 3), b0, b1, b2, b3);
                mma_bf16(c0, a0, a1, a2, a3, b0, b1);
                mma_bf16(c1, e0, e1, e2, e3, b2, b3);
            }
            const int pos = (page0 + i) * PAGE + warp * 8 + 2 * t;
            const bool ok0 = pos >= lo && pos < hi, ok1 = pos + 1 >= lo && pos + 1 < hi;
            float* d0 = s_sh + g * S_PITCH + warp * 8 + 2 * t;
            *reinterpret_cast<float2*>(d0) = make_float2(ok0 ? (c0[0] + c1[0]) * a.scale_log2 : -INFINITY, ok1 ? (c0[1] + c1[1]) * a.scale_log2 : -INFINITY);
            *reinterpret_cast<float2*>(d0 + 8 * S_PITCH) = make_float2(ok0 ? (c0[2] + c1[2]) * a.scale_log2 : -INFINITY, ok1 ? (c0[3] + c1[3]) * a.scale_log2 : -INFINITY);
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        {   // softmax: thread tid takes four keys of row tid / 16
            const int row = tid >> 4, k4 = (tid & 15) * 4;
            const float4 v = *reinterpret_cast<const float4*>(s_sh + row * S_PITCH + k4);
            float mx = fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w));
#pragma unroll
            for (int w = 8; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
            const float m_new = fmaxf(m_run, mx), alpha = exp2f(m_run - m_new);
            const float p0 = exp2f(v.x - m_new), p1 = exp2f(v.y - m_new), p2 = exp2f(v.z - m_new), p3 = exp2f(v.w - m_new);
            float sum = (p0 + p1) + (p2 + p3);
#pragma unroll
            for (int w = 8; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
            l_run = l_run * alpha + sum;
            m_run = m_new;
            const uint32_t x = pack2(p0, p1), y = pack2(p2, p3);
            *reinterpret_cast<uint2*>(p_hi + row * P_PITCH + k4) = make_uint2(x, y);
            *reinterpret_cast<uint2*>(p_lo + row * P_PITCH + k4) = make_uint2(rest2(p0, p1, x), rest2(p2, p3, y));
            if ((tid & 15) == 0) alpha_sh[row] = alpha;
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        {   // O: column pairs warp, warp + 8, ...
            const float al0 = alpha_sh[g], al1 = alpha_sh[g + 8];
#pragma unroll
            for (int j = 0; j < NP; ++j)
#pragma unroll
                for (int n = 0; n < 2; ++n) { o[j][n][0] *= al0; o[j][n][1] *= al0; o[j][n][2] *= al1; o[j][n][3] *= al1; }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t x0, x1, x2, x3, y0, y1, y2, y3;
                ldsm_x4(ph_addr + kk * 32, x0, x1, x2, x3);
                ldsm_x4(pl_addr + kk * 32, y0, y1, y2, y3);
                const int key = kk * 16 + (mtx & 1) * 8 + r8;
#pragma unroll
                for (int j = 0; j < NP; ++j) {
                    const int dim0 = (warp + WARPS * j) * 16 + (mtx >> 1) * 8;
                    if ((warp + WARPS * j) * 16 >= a.r) break;                            // uniform over the warp
                    uint32_t b0, b1, b2, b3;
                    ldsm_x4_trans(page + (dim0 >> 6) * 8192 + swz(key, (dim0 & 63) >> 3), b0, b1, b2, b3);
                    mma_bf16(o[j][0], x0, x1, x2, x3, b0, b1);
                    mma_bf16(o[j][1], x0, x1, x2, x3, b2, b3);
                    mma_bf16(o[j][0], y0, y1, y2, y3, b0, b1);
                    mma_bf16(o[j][1], y0, y1, y2, y3, b2, b3);
                }
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(empty + s);
    }
    const size_t stride = a.r + 2;
    float* part = a.scratch + ((size_t)(b * a.nh + h0) * a.n_splits + split) * stride;    // of head h0; the next head n_splits * stride on
    const size_t head = (size_t)a.n_splits * stride;
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int d = (warp + WARPS * j) * 16 + n * 8 + 2 * t;
#pragma unroll
            for (int c = 0; c < 2; ++c)
                if (d + c < a.r) {
                    if (h0 + g < a.nh) part[g * head + d + c] = o[j][n][c];
                    if (h0 + g + 8 < a.nh) part[(g + 8) * head + d + c] = o[j][n][c + 2];
                }
        }
    const int row = tid >> 4;
    if ((tid & 15) == 0 && h0 + row < a.nh) {
        part[row * head + a.r] = m_run * 0.69314718055994531f;                            // the merge works with natural exponents
        part[row * head + a.r + 1] = l_run;
    }
}

size_t latent_smem(int boxes, int stages) {
    return 1024 + (size_t)stages * boxes * 8192 + (size_t)HEADS * q_pitch(boxes) * 2 + HEADS * S_PITCH * 4 + 2 * HEADS * P_PITCH * 2 + HEADS * 4 + 4 * sizeof(uint64_t);
}

template <int NP>
int launch_latent(const CUtensorMap& map, const LatentDecArgs& d, dim3 grid, cudaStream_t stream) {
    static size_t configured = 0;
    const size_t smem = latent_smem(d.boxes, d.stages);
    if (configured < smem) {
        const cudaError_t e = cudaFuncSetAttribute(attn_decode_latent_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        TB_REQUIRE(e == cudaSuccess, "attn_decode_latent: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = smem;
    }
    tb_launch(attn_decode_latent_kernel<NP>, grid, THREADS, smem, stream, map, d);
    return 0;
}

}  // namespace

extern "C" int tb_attn_merge(const AttnArgs* args, int dtype, cudaStream_t stream);

// 0 if the tensor-core kernel takes this problem (one stored row a token as key and value, no pairs, no kept tokens), else 1
// with the reason in tb_last_error().
extern "C" int tb_attn_decode_latent_check(const AttnArgs* a, int dtype) {
    TB_REQUIRE(dtype == TB_BF16, "attn_decode_latent: bfloat16 only");
    TB_REQUIRE(a->v_alias && a->nkv == 1 && a->hd_v > 0 && a->hd_v <= a->hd, "attn_decode_latent: one row a token as key and value");
    TB_REQUIRE(a->hd % 8 == 0 && a->hd <= 1024, "attn_decode_latent: rows of %d elements (a multiple of 8 up to 1024)", a->hd);
    TB_REQUIRE(a->cache.page_size == PAGE, "attn_decode_latent: pages of %d rows, not %d", PAGE, a->cache.page_size);
    TB_REQUIRE(a->q_stride % 8 == 0 && ((uintptr_t)a->q & 15) == 0 && ((uintptr_t)a->cache.storage & 15) == 0, "attn_decode_latent: queries and cache must be 16-byte aligned rows");
    TB_REQUIRE(a->chunk > 0 && a->chunk % PAGE == 0, "attn_decode_latent: the chunk %d must be a multiple of %d", a->chunk, PAGE);
    TB_REQUIRE(!(a->softcap > 0.f) && !a->rel_bias && !a->head_mix && !a->pair_lambda && !a->fused_qk && a->keep_first == 0 && !a->out_f32, "attn_decode_latent: shaped scores, pairs and kept tokens run on other kernels");
    return 0;
}

extern "C" int tb_attn_decode_latent(const AttnArgs* args, cudaStream_t stream) {
    const AttnArgs& a = *args;
    if (tb_attn_decode_latent_check(args, TB_BF16)) return 1;
    TB_REQUIRE(a.batch.B > 0 && a.cache.storage && a.scratch, "attn_decode_latent: needs sequences, a cache and scratch");
    TB_REQUIRE(a.n_splits > 0 && a.n_splits <= 65535, "attn_decode_latent: bad grid");
    TB_REQUIRE(a.cache.head_dim == a.hd && a.cache.kv_heads == 1, "attn_decode_latent: the cache view does not match the rows");
    CUtensorMap map;
    if (tb_make_map_bf16(&map, a.cache.storage, (long long)a.cache.num_pages * PAGE, a.hd, a.hd, PAGE)) return 1;
    LatentDecArgs d;
    d.q = (const __nv_bfloat16*)a.q; d.q_stride = a.q_stride; d.scratch = a.scratch;
    d.table = a.cache.table; d.table_width = a.cache.table_width; d.ring_rows = a.cache.ring_rows;
    d.slot_of_seq = a.batch.slot_of_seq; d.kv_len = a.batch.kv_len;
    d.early_len = a.early_len; d.early_mode = a.early_len ? a.early_mode : 0;
    TB_REQUIRE(d.early_mode >= 0 && d.early_mode <= 2, "attn_decode_latent: early_mode %d (0, 1 or 2)", d.early_mode);
    d.nh = a.nh; d.dk = a.hd; d.r = a.hd_v; d.boxes = (a.hd + 63) / 64; d.stages = d.boxes <= 11 ? 2 : 1;
    d.window = a.window; d.scale_log2 = a.scale * 1.4426950408889634f; d.chunk = a.chunk; d.n_splits = a.n_splits;
    const dim3 grid(a.batch.B, (a.nh + HEADS - 1) / HEADS, a.n_splits);
    TB_REQUIRE(grid.y <= 65535, "attn_decode_latent: too many heads");
    const int rc = d.r <= 128 ? launch_latent<1>(map, d, grid, stream) : (d.r <= 512 ? launch_latent<4>(map, d, grid, stream) : launch_latent<8>(map, d, grid, stream));
    if (rc) return rc;
    TB_CHECK_LAUNCH("attn_decode_latent");
    return tb_attn_merge(args, TB_BF16, stream);
}

// Reads and clears the error word of this file's kernel (0: none).  Synchronises the device.
extern "C" int tb_attn_latent_error() {
    unsigned int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_latent_error, sizeof(v)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_latent_error, &zero, sizeof(zero));
    return (int)v;
}
