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

// The splits of one head in order: acc = sum_s exp(m_s - m) acc_s, returned unnormalised, with l = sum_s exp(m_s - m) l_s
// (the sink's term included).  Every thread finds the maximum and the weights' sum itself from the splits' (m, l) pairs (a
// few broadcast loads) and adds up its own output dims, so the loads of different splits do not wait for one another; splits
// that saw no key (all of them before a window's first key) are skipped.
template <int PER>
__device__ __forceinline__ float merge_splits(const AttnArgs& a, int b, int h, int hd, int used, int first, float* acc) {
    const int stride = hd + 2;
    const float* part = a.scratch + (size_t)(b * a.nh + h) * a.n_splits * stride;
    float m = -FLT_MAX;
    for (int s = first; s < used; ++s)
        if (part[s * stride + hd + 1] > 0.f) m = fmaxf(m, part[s * stride + hd]);
    const bool sunk = a.sink != nullptr;
    if (sunk) m = fmaxf(m, a.sink[h]);
    float l = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) acc[j] = 0.f;
    for (int s = first; s < used; ++s) {
        const float ls = part[s * stride + hd + 1];
        if (!(ls > 0.f)) continue;
        const float w = expf(part[s * stride + hd] - m);
        l = fmaf(w, ls, l);
        const float* p = part + (size_t)s * stride;
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int d = threadIdx.x + blockDim.x * j;
            if (d < hd) acc[j] = fmaf(w, p[d], acc[j]);
        }
    }
    if (sunk) l += expf(a.sink[h] - m);               // the sink counts once, here, not once a split
    return l;
}

// grid (B, nh), one block of up to 128 threads: out = sum_s exp(m_s - m) acc_s / sum_s exp(m_s - m) l_s.
template <typename T, int MAXE>
__global__ void attn_merge_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y, hd = value_width(a);
    const int len = a.batch.kv_len[b], keys = tb_split_keys(len, a.chunk, a.n_splits);
    const int used = min(a.n_splits, (len + keys - 1) / keys);
    const int first = (a.window > 0 && a.keep_first <= 0) ? max(0, len - a.window) / keys : 0;      // splits before the window's first key hold nothing
    constexpr int PER = (32 * MAXE + 127) / 128;
    float acc[PER];
    float inv = 1.0f / merge_splits<PER>(a, b, h, hd, used, first, acc);
    if (a.head_gate) inv *= 1.0f / (1.0f + expf(-a.head_gate[(size_t)b * a.head_gate_stride + h]));      // the head's gate
    T* o = (T*)a.out + (size_t)b * a.out_stride + h * hd;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = threadIdx.x + blockDim.x * j;
        if (d < hd) stf(o + d, acc[j] * inv);
    }
}

// grid (B, nh / 2), 128 threads: both maps of a pair merged, the second times lambda taken off the first, the difference
// divided by its root mean square (AttnArgs.pair_lambda).
template <typename T, int MAXE>
__global__ void __launch_bounds__(128) attn_merge_pair_kernel(AttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[33];
    const int b = blockIdx.x, p = blockIdx.y, hd = value_width(a);
    const int len = a.batch.kv_len[b], keys = tb_split_keys(len, a.chunk, a.n_splits);
    const int used = min(a.n_splits, (len + keys - 1) / keys);
    const int first = (a.window > 0 && a.keep_first <= 0) ? max(0, len - a.window) / keys : 0;
    constexpr int PER = (32 * MAXE + 127) / 128;
    float a1[PER], a2[PER];
    const float inv1 = 1.0f / merge_splits<PER>(a, b, 2 * p, hd, used, first, a1);
    const float inv2 = 1.0f / merge_splits<PER>(a, b, 2 * p + 1, hd, used, first, a2);
    const float lam = *a.pair_lambda;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = threadIdx.x + blockDim.x * j;
        a1[j] = d < a.pair_width ? fmaf(-lam, a2[j] * inv2, a1[j] * inv1) : 0.f;
        ss = fmaf(a1[j], a1[j], ss);
    }
    const float r = a.pair_scale / sqrtf(block_sum(ss, red) / (float)a.pair_width + a.pair_eps);
    T* o = (T*)a.out + (size_t)b * a.out_stride + p * a.pair_width;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int d = threadIdx.x + blockDim.x * j;
        if (d < a.pair_width) stf(o + d, a1[j] * r);
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
    const bool wide = wide_rows(a);
    if (a.pair_lambda) {
        TB_REQUIRE(a.nh % 2 == 0 && a.pair_width > 0 && a.pair_width <= value_width(a) && !a.head_gate && !a.sink, "attn_merge: pairs of heads do not fit");
        ATT_DISPATCH(attn_merge_pair_kernel, dim3(a.batch.B, a.nh / 2), 128, 0);
    } else {
        ATT_DISPATCH(attn_merge_kernel, dim3(a.batch.B, a.nh), 128, 0);
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
