// Causal grouped-query attention over the paged cache, for every head size and group.
//
//   tb_attn_prefill  queries of a ragged step; keys before the step come from the cache, keys of
//                    the step itself from the step's own K | V rows (so a ring cache can be
//                    written after attention)
//   tb_attn_decode   one query per sequence over its cached keys, cut into splits by the sequence's
//                    own length (tb_split_keys), each giving (max, sum, unnormalised output)
//   tb_attn_merge    log-sum-exp merge of the chunks in chunk order (a block per sequence and head, or, with
//                    AttnArgs.pair_lambda, per sequence and pair of heads, whose difference it finishes)
//
// One warp per (query, head): a lane scores one key per round with the whole query in shared
// memory, the warp folds 32 scores into the running softmax, then every lane accumulates its
// output dims over the 32 values.  Scores, softmax and PV are float32 with precise expf.
// A chunk's borders depend on the sequence's own length only, never on the batch.
//
// berniehans/titan: flash_attention_2_kernel (engine/engine-cuda/kernels/flash_attention_2.cu:22-106),
// paged_attention_decode_kernel, flash_decoding_split_kernel and flash_decoding_reduce_kernel
// (kernels/paged_attention.cu:6-103, 200-309, 314-369): score = q.k / sqrt(hd), keys t <= position,
// query head h reads kv head h / (nh/nkv), partials merged with exp(m_s - m_max).
#include <float.h>

#include "attention_args.h"
#include "common.cuh"

#define ATT_MAXE 8        // head_dim <= 256 (the wide instantiation: 32 values a lane, rows up to 1,024)
#define ATT_MAXE_WIDE 32
#define ATT_WARPS 4


template <typename T> __device__ __forceinline__ void load8(const T* p, float* o);
template <> __device__ __forceinline__ void load8<float>(const float* p, float* o) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float* o) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        o[2 * i] = __uint_as_float(w[i] << 16);
        o[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}

// Running softmax state of one warp: every lane holds the same m and l, and acc for dims lane + 32 j.
template <int MAXE>
struct Running {
    float m, l;
    float acc[MAXE];
};

// Width of a value row (and of an output row): the key's width unless the launch says otherwise.
__device__ __host__ __forceinline__ int value_width(const AttnArgs& a) { return a.hd_v > 0 ? a.hd_v : a.hd; }

// Folds keys [lo, hi) of one sequence into ``st``.  Keys at positions >= first_new are read from the
// step's own rows (row index first_new_row + pos - first_new), earlier ones from the cache.
template <typename T, int MAXE>
__device__ __forceinline__ void attend_range(Running<MAXE>& st, const float* qs, const AttnArgs& a, int lo, int hi,
                                             int first_new, int first_new_row, int slot, int kh, int lane) {
    const int hd = a.hd, hdv = value_width(a);
    const T* knew = (const T*)a.kv_new;
    const T* cache = (const T*)a.cache.storage;
    const size_t vhalf = (cache && !a.v_alias) ? kv_half_elems(a.cache) : 0;
    const int vnew = a.v_alias ? 0 : a.nkv * hd;
    for (int base = lo; base < hi; base += 32) {
        const int kpos = base + lane;
        const bool valid = kpos < hi;
        const T* kp = nullptr;
        const T* vp = nullptr;
        if (valid) {
            if (kpos >= first_new) {
                kp = knew + (size_t)(first_new_row + kpos - first_new) * a.kv_stride + kh * hd;
                vp = kp + vnew;
            } else {
                kp = cache + kv_row_offset(a.cache, slot, kpos, kh);
                vp = kp + vhalf;
            }
        }
        float s = -FLT_MAX;
        if (valid) {
            float dot = 0.f;
            for (int e = 0; e < hd; e += 8) {
                float kv[8];
                load8<T>(kp + e, kv);
#pragma unroll
                for (int i = 0; i < 8; ++i) dot = fmaf(qs[e + i], kv[i], dot);
            }
            s = dot * a.scale;
        }
        const float m_new = fmaxf(st.m, warp_max(s));
        const float alpha = expf(st.m - m_new);           // st.m = -FLT_MAX at the start: exp(-huge) = 0
        const float p = valid ? expf(s - m_new) : 0.f;
        st.l = st.l * alpha + warp_sum(p);
        st.m = m_new;
#pragma unroll
        for (int j = 0; j < MAXE; ++j) st.acc[j] *= alpha;
        const int n_valid = min(32, hi - base);
        for (int kk = 0; kk < n_valid; ++kk) {
            const float pk = __shfl_sync(0xffffffffu, p, kk);
            const T* v = (const T*)__shfl_sync(0xffffffffu, (unsigned long long)vp, kk);
#pragma unroll
            for (int j = 0; j < MAXE; ++j) {
                const int d = lane + 32 * j;
                if (d < hdv) st.acc[j] = fmaf(pk, ldf(v + d), st.acc[j]);
            }
        }
    }
}

template <typename T>
__device__ __forceinline__ void load_query(float* qs, const T* q, int hd, int lane) {
    for (int e = lane; e < hd; e += 32) qs[e] = ldf(q + e);
    __syncwarp();
}

// ------------------------------------------------------------------ prefill
// grid (T, ceil(nh / ATT_WARPS)); warp = one head of one query token.
template <typename T, int MAXE>
__global__ void __launch_bounds__(ATT_WARPS * 32) attn_prefill_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float q_smem[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x, h = blockIdx.y * ATT_WARPS + warp;
    if (h >= a.nh) return;                             // (the two heads of a pair leave or stay together)
    const int hd = a.hd;
    float* qs = q_smem + warp * hd;
    load_query<T>(qs, (const T*)a.q + (size_t)t * a.q_stride + h * hd, hd, lane);
    const int seq = a.batch.seq_of[t], pos = a.batch.pos_of[t];
    const int slot = a.batch.slot_of_seq[seq];
    const int first_new = a.kv_new ? a.batch.start_pos[seq] : 0x7fffffff;
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    Running<MAXE> st;
    st.m = -FLT_MAX; st.l = 0.f;
#pragma unroll
    for (int j = 0; j < MAXE; ++j) st.acc[j] = 0.f;
    if (a.keep_first > 0 && lo > 0)                    // the kept first tokens that the window has left behind
        attend_range<T, MAXE>(st, qs, a, 0, min(a.keep_first, lo), first_new, a.batch.q_start[seq], slot, h / (a.nh / a.nkv), lane);
    attend_range<T, MAXE>(st, qs, a, lo, pos + 1, first_new, a.batch.q_start[seq], slot, h / (a.nh / a.nkv), lane);
    if (a.sink) {                                     // one more term of the denominator, against the larger of the two maxima
        const float sk = a.sink[h], m_new = fmaxf(st.m, sk), alpha = expf(st.m - m_new);
        st.l = st.l * alpha + expf(sk - m_new);
#pragma unroll
        for (int j = 0; j < MAXE; ++j) st.acc[j] *= alpha;
    }
    const float inv = 1.0f / st.l;
    const int hdv = value_width(a);
    if (a.pair_lambda) {
        // heads 2p and 2p + 1 sit in neighbouring warps: the second leaves its output where its query lay, and the first
        // takes it off its own, divides by the root mean square and writes the pair's row
        if (h & 1) {
            __syncwarp();
#pragma unroll
            for (int j = 0; j < MAXE; ++j) {
                const int d = lane + 32 * j;
                if (d < hdv) qs[d] = st.acc[j] * inv;
            }
        }
        asm volatile("bar.sync %0, 64;" ::"r"(1 + (warp >> 1)) : "memory");      // the pair's two warps
        if (h & 1) return;
        const float lam = *a.pair_lambda;
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < MAXE; ++j) {
            const int d = lane + 32 * j;
            st.acc[j] = d < a.pair_width ? fmaf(-lam, qs[hd + d], st.acc[j] * inv) : 0.f;
            ss = fmaf(st.acc[j], st.acc[j], ss);
        }
        const float r = a.pair_scale / sqrtf(warp_sum(ss) / (float)a.pair_width + a.pair_eps);
        T* o = (T*)a.out + (size_t)t * a.out_stride + (h >> 1) * a.pair_width;
#pragma unroll
        for (int j = 0; j < MAXE; ++j) {
            const int d = lane + 32 * j;
            if (d < a.pair_width) stf(o + d, st.acc[j] * r);
        }
        return;
    }
    T* o = (T*)a.out + (size_t)t * a.out_stride + h * hdv;
#pragma unroll
    for (int j = 0; j < MAXE; ++j) {
        const int d = lane + 32 * j;
        if (d < hdv) stf(o + d, st.acc[j] * inv);
    }
}

// ------------------------------------------------------------------ decode, split over the keys
// grid (B, nkv, n_splits); the warps of a block take the query heads of one kv head in turn.
// Partial of (sequence b, head h, split s) at scratch[((b * nh + h) * n_splits + s) * (hd + 2)]:
// hd unnormalised outputs, then m, then l (l = 0: the split saw no key).
template <typename T, int MAXE>
__global__ void __launch_bounds__(ATT_WARPS * 32) attn_decode_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float q_smem[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int blocks_y = a.head_blocks > 0 ? a.head_blocks : a.nkv;
    const int b = blockIdx.x, kh = (int)blockIdx.y * a.nkv / blocks_y, split = blockIdx.z;
    const int hd = a.hd, hdv = value_width(a), group = a.nh / blocks_y;
    const int len = a.batch.kv_len[b];
    const int keys = tb_split_keys(len, a.chunk, a.n_splits);
    if ((long long)split * keys >= len) return;     // the merge reads ceil(len / keys) splits only
    const int pos = len - 1;
    const int slot = a.batch.slot_of_seq[b];
    const int wlo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int lo = max(wlo, split * keys), hi = min(len, (split + 1) * keys);
    // the kept first tokens that lie in this split and before the window
    const int klo = split * keys, khi = a.window > 0 ? min(min(a.keep_first, wlo), hi) : 0;
    float* qs = q_smem + warp * hd;
    for (int g = warp; g < group; g += ATT_WARPS) {
        const int h = (int)blockIdx.y * group + g;
        float* part = a.scratch + ((size_t)(b * a.nh + h) * a.n_splits + split) * (hdv + 2);
        Running<MAXE> st;
        st.m = -FLT_MAX; st.l = 0.f;
#pragma unroll
        for (int j = 0; j < MAXE; ++j) st.acc[j] = 0.f;
        if (lo < hi || klo < khi) {
            __syncwarp();
            load_query<T>(qs, (const T*)a.q + (size_t)b * a.q_stride + h * hd, hd, lane);
            if (klo < khi) attend_range<T, MAXE>(st, qs, a, klo, khi, 0x7fffffff, 0, slot, kh, lane);
            if (lo < hi) attend_range<T, MAXE>(st, qs, a, lo, hi, 0x7fffffff, 0, slot, kh, lane);
        }
#pragma unroll
        for (int j = 0; j < MAXE; ++j) {
            const int d = lane + 32 * j;
            if (d < hdv) part[d] = st.acc[j];
        }
        if (lane == 0) { part[hdv] = st.m; part[hdv + 1] = st.l; }
    }
}

// The splits of NH neighbouring heads (h0 ..) merged for output dims ``d0 + threadIdx.x + blockDim.x * j``: acc[k][j] =
// sum_s exp(m_s - m) acc_s and l[k] = sum_s exp(m_s - m) l_s (the sink's term included), both in the order of the splits.  The
// block first turns the splits' (m, l) pairs into weights, a thread a split, MERGE_TILE splits at a time; the loads of the
// sums then wait for nothing but the weights in shared memory.  Splits that saw no key (l = 0) get the weight zero.
#define MERGE_TILE 128
template <int NH, int PER>
__device__ __forceinline__ void merge_splits(const AttnArgs& a, int b, int h0, int hd, int d0, int used, int first, float (&acc)[NH][PER], float (&l)[NH]) {
    __shared__ float sm[NH][MERGE_TILE], sl[NH][MERGE_TILE], red[NH][32];
    const int stride = hd + 2, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    const float* part = a.scratch + (size_t)(b * a.nh + h0) * a.n_splits * stride;
    const size_t head = (size_t)a.n_splits * stride;
    float m[NH];
#pragma unroll
    for (int k = 0; k < NH; ++k) {
        m[k] = -FLT_MAX; l[k] = 0.f;
#pragma unroll
        for (int j = 0; j < PER; ++j) acc[k][j] = 0.f;
    }
    // the first tile's pairs stay in shared memory; the maximum runs over all of them
    for (int s = threadIdx.x; s < used - first; s += blockDim.x)
#pragma unroll
        for (int k = 0; k < NH; ++k) {
            const float* p = part + k * head + (size_t)(first + s) * stride + hd;
            const float ms = p[0], ls = p[1];
            if (ls > 0.f) m[k] = fmaxf(m[k], ms);
            if (s < MERGE_TILE) { sm[k][s] = ms; sl[k][s] = ls; }
        }
#pragma unroll
    for (int k = 0; k < NH; ++k) {
        m[k] = warp_max(m[k]);
        if (lane == 0) red[k][warp] = m[k];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < NH; ++k) {
        for (int w = 0; w < nwarp; ++w) m[k] = fmaxf(m[k], red[k][w]);
        if (a.sink) m[k] = fmaxf(m[k], a.sink[h0 + k]);
    }
    for (int s0 = 0; s0 < used - first; s0 += MERGE_TILE) {
        const int n = min(MERGE_TILE, used - first - s0);
        if (s0 > 0) __syncthreads();
        for (int s = threadIdx.x; s < n; s += blockDim.x)
#pragma unroll
            for (int k = 0; k < NH; ++k) {
                const float* p = part + k * head + (size_t)(first + s0 + s) * stride + hd;
                const float ms = s0 > 0 ? p[0] : sm[k][s], ls = s0 > 0 ? p[1] : sl[k][s];      // (a thread reads back what it wrote itself)
                const float w = ls > 0.f ? expf(ms - m[k]) : 0.f;
                sm[k][s] = w; sl[k][s] = w * ls;
            }
        __syncthreads();
        const float* p = part + (size_t)(first + s0) * stride + d0 + threadIdx.x;
#pragma unroll 8
        for (int s = 0; s < n; ++s)
#pragma unroll
            for (int k = 0; k < NH; ++k) {
                const float w = sm[k][s];
                l[k] += sl[k][s];
#pragma unroll
                for (int j = 0; j < PER; ++j)
                    if (d0 + (int)threadIdx.x + (int)blockDim.x * j < hd) acc[k][j] = fmaf(w, p[k * head + (size_t)s * stride + blockDim.x * j], acc[k][j]);
            }
    }
    if (a.sink)                                        // the sink counts once, here, not once a split
#pragma unroll
        for (int k = 0; k < NH; ++k) l[k] += expf(a.sink[h0 + k] - m[k]);
}

// grid (B, nh, ceil(value width / 128)), 128 threads: out = sum_s exp(m_s - m) acc_s / sum_s exp(m_s - m) l_s.
template <typename T>
__global__ void __launch_bounds__(128) attn_merge_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, hd = value_width(a), d = blockIdx.z * 128 + threadIdx.x;
    const int len = a.batch.kv_len[b], keys = tb_split_keys(len, a.chunk, a.n_splits);
    const int used = min(a.n_splits, (len + keys - 1) / keys);
    const int first = (a.window > 0 && a.keep_first <= 0) ? max(0, len - a.window) / keys : 0;      // splits before the window's first key hold nothing
    float acc[1][1], l[1];
    merge_splits<1, 1>(a, b, h, hd, blockIdx.z * 128, used, first, acc, l);
    float inv = 1.0f / l[0];
    if (a.head_gate) inv *= 1.0f / (1.0f + expf(-a.head_gate[(size_t)b * a.head_gate_stride + h]));      // the head's gate
    if (d < hd) stf((T*)a.out + (size_t)b * a.out_stride + h * hd + d, acc[0][0] * inv);
}

// grid (B, nh / 2), 128 threads: both maps of a pair merged, the second times lambda taken off the first, the difference
// divided by its root mean square (AttnArgs.pair_lambda).
template <typename T, int PER>
__global__ void __launch_bounds__(128) attn_merge_pair_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[33];
    const int b = blockIdx.x, p = blockIdx.y, hd = value_width(a);
    const int len = a.batch.kv_len[b], keys = tb_split_keys(len, a.chunk, a.n_splits);
    const int used = min(a.n_splits, (len + keys - 1) / keys);
    const int first = (a.window > 0 && a.keep_first <= 0) ? max(0, len - a.window) / keys : 0;
    float acc[2][PER], l[2];
    merge_splits<2, PER>(a, b, 2 * p, hd, 0, used, first, acc, l);
    const float lam = *a.pair_lambda, inv1 = 1.0f / l[0], inv2 = 1.0f / l[1];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = threadIdx.x + 128 * j;
        acc[0][j] = d < a.pair_width ? fmaf(-lam, acc[1][j] * inv2, acc[0][j] * inv1) : 0.f;
        ss = fmaf(acc[0][j], acc[0][j], ss);
    }
    const float r = a.pair_scale / sqrtf(block_sum(ss, red) / (float)a.pair_width + a.pair_eps);
    T* o = (T*)a.out + (size_t)b * a.out_stride + p * a.pair_width;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = threadIdx.x + 128 * j;
        if (d < a.pair_width) stf(o + d, acc[0][j] * r);
    }
}

static int check_common(const AttnArgs& a, const char* who) {
    TB_REQUIRE(a.nh > 0 && a.nkv > 0 && a.nh % a.nkv == 0, "%s: %d query heads are not a multiple of %d kv heads", who, a.nh, a.nkv);
    TB_REQUIRE(a.hd >= 8 && a.hd % 8 == 0 && a.hd <= 32 * ATT_MAXE_WIDE, "%s: head_dim %d must be a multiple of 8 up to %d", who, a.hd, 32 * ATT_MAXE_WIDE);
    TB_REQUIRE(a.hd_v >= 0 && a.hd_v <= 32 * ATT_MAXE_WIDE, "%s: a value row of %d elements (at most %d)", who, a.hd_v, 32 * ATT_MAXE_WIDE);
    TB_REQUIRE(!a.v_alias || value_width(a) <= a.hd, "%s: a value that is the head of its key row cannot be wider (%d) than the key (%d)", who, value_width(a), a.hd);
    TB_REQUIRE(a.q_stride % 8 == 0 && a.kv_stride % 8 == 0, "%s: row strides must be multiples of 8 elements", who);
    TB_REQUIRE(a.window >= 0 && a.keep_first >= 0, "%s: negative window or kept tokens", who);
    TB_REQUIRE(!(a.softcap > 0.f) && !a.rel_bias && !a.head_mix, "%s: capped, biased or mixed scores run on the mixed-heads kernels", who);
    TB_REQUIRE(!a.out_f32, "%s: float32 output rows are the tensor-core prompt kernels'", who);
    TB_REQUIRE(!a.pair_lambda || (a.nh % 2 == 0 && a.pair_width > 0 && a.pair_width <= value_width(a) && a.pair_eps > 0.f && !a.head_gate && !a.sink),
               "%s: pairs of heads need an even number of them (%d), a width (%d) within the value's and no gate or sink a head", who, a.nh, a.pair_width);
    TB_REQUIRE(!a.pair_lambda || value_width(a) <= a.hd, "%s: a pair's value row (%d) may not be wider than its key row (%d)", who, value_width(a), a.hd);
    TB_REQUIRE(!a.cache.storage || (a.cache.head_dim == a.hd && a.cache.kv_heads == a.nkv), "%s: the cache view does not match the heads", who);
    return 0;
}

// Rows of up to 256 elements take 8 values a lane, wider ones 32.
static bool wide_rows(const AttnArgs& a) { return a.hd > 32 * ATT_MAXE || value_width(a) > 32 * ATT_MAXE; }

#define ATT_DISPATCH(kernel, grid, threads, smem)                                                              \
    do {                                                                                                       \
        if (dtype == TB_F32) {                                                                                 \
            if (wide) tb_launch(kernel<float, ATT_MAXE_WIDE>, grid, threads, smem, stream, a);                 \
            else tb_launch(kernel<float, ATT_MAXE>, grid, threads, smem, stream, a);                           \
        } else {                                                                                               \
            if (wide) tb_launch(kernel<__nv_bfloat16, ATT_MAXE_WIDE>, grid, threads, smem, stream, a);         \
            else tb_launch(kernel<__nv_bfloat16, ATT_MAXE>, grid, threads, smem, stream, a);                   \
        }                                                                                                      \
    } while (0)

extern "C" int tb_attn_prefill(const AttnArgs* args, int dtype, cudaStream_t stream) {
    AttnArgs a = *args;
    if (check_common(a, "attn_prefill")) return 1;
    TB_REQUIRE(dtype == TB_F32 || dtype == TB_BF16, "attn_prefill: unknown dtype %d", dtype);
    TB_REQUIRE(a.batch.T > 0, "attn_prefill: no tokens");
    TB_REQUIRE(a.kv_new || a.cache.storage, "attn_prefill: neither new keys nor a cache");
    TB_REQUIRE(!a.head_gate, "attn_prefill: a gate on the heads is applied by the merge of decode splits or by the mixed-heads kernels");
    dim3 grid(a.batch.T, (a.nh + ATT_WARPS - 1) / ATT_WARPS);
    const size_t smem = (size_t)ATT_WARPS * a.hd * sizeof(float);
    const bool wide = wide_rows(a);
    ATT_DISPATCH(attn_prefill_kernel, grid, ATT_WARPS * 32, smem);
    TB_CHECK_LAUNCH("attn_prefill");
    return 0;
}

extern "C" int tb_attn_merge(const AttnArgs* args, int dtype, cudaStream_t stream) {
    AttnArgs a = *args;
    TB_REQUIRE(dtype == TB_F32 || dtype == TB_BF16, "attn_merge: unknown dtype %d", dtype);
    const int width = value_width(a);
    if (a.pair_lambda) {
        TB_REQUIRE(a.nh % 2 == 0 && a.pair_width > 0 && a.pair_width <= width && !a.head_gate && !a.sink, "attn_merge: pairs of heads do not fit");
        const dim3 grid(a.batch.B, a.nh / 2);
        if (dtype == TB_F32) {
            if (width <= 128) tb_launch(attn_merge_pair_kernel<float, 1>, grid, 128, 0, stream, a);
            else if (width <= 256) tb_launch(attn_merge_pair_kernel<float, 2>, grid, 128, 0, stream, a);
            else tb_launch(attn_merge_pair_kernel<float, 8>, grid, 128, 0, stream, a);
        } else {
            if (width <= 128) tb_launch(attn_merge_pair_kernel<__nv_bfloat16, 1>, grid, 128, 0, stream, a);
            else if (width <= 256) tb_launch(attn_merge_pair_kernel<__nv_bfloat16, 2>, grid, 128, 0, stream, a);
            else tb_launch(attn_merge_pair_kernel<__nv_bfloat16, 8>, grid, 128, 0, stream, a);
        }
    } else {
        const dim3 grid(a.batch.B, a.nh, (width + 127) / 128);
        if (dtype == TB_F32) tb_launch(attn_merge_kernel<float>, grid, 128, 0, stream, a);
        else tb_launch(attn_merge_kernel<__nv_bfloat16>, grid, 128, 0, stream, a);
    }
    TB_CHECK_LAUNCH("attn_merge");
    return 0;
}

extern "C" int tb_attn_decode(const AttnArgs* args, int dtype, cudaStream_t stream) {
    AttnArgs a = *args;
    if (check_common(a, "attn_decode")) return 1;
    TB_REQUIRE(dtype == TB_F32 || dtype == TB_BF16, "attn_decode: unknown dtype %d", dtype);
    TB_REQUIRE(a.batch.B > 0 && a.cache.storage && a.scratch, "attn_decode: needs sequences, a cache and scratch");
    TB_REQUIRE(a.chunk > 0 && a.n_splits > 0 && a.n_splits <= 65535, "attn_decode: bad split (chunk=%d splits=%d)", a.chunk, a.n_splits);
    TB_REQUIRE(a.nkv <= 65535 && a.head_blocks <= 65535, "attn_decode: too many kv heads");
    TB_REQUIRE(a.head_blocks == 0 || (a.head_blocks > 0 && a.nh % a.head_blocks == 0 && a.head_blocks % a.nkv == 0),
               "attn_decode: %d blocks for %d query heads on %d kv heads", a.head_blocks, a.nh, a.nkv);
    dim3 grid(a.batch.B, a.head_blocks > 0 ? a.head_blocks : a.nkv, a.n_splits);
    const size_t smem = (size_t)ATT_WARPS * a.hd * sizeof(float);
    const bool wide = wide_rows(a);
    ATT_DISPATCH(attn_decode_kernel, grid, ATT_WARPS * 32, smem);
    TB_CHECK_LAUNCH("attn_decode");
    return tb_attn_merge(args, dtype, stream);
}
