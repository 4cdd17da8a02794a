// What lies between a fused Q | K | V projection and its attention where every projected channel passes a short causal
// convolution over time: convolution, rotation of Q and K, append to the cache, in one kernel.
//
//   u_t = the projected row of token t;   y_t[c] = sum_j taps[j][c] u_(t - n + 1 + j)[c],  j < n, zeros before the sequence's start
//   Q and K heads of y turn by their position (a whole head, or its first ``rot`` elements; either pairing); V heads pass
//
// The n - 1 projected rows before the step come from the sequence's state (float32, oldest first), and the last n - 1 rows
// of the sequence are its state afterwards.  A block takes a run of tokens of ONE sequence, at least n - 1 of them, so only
// the block with a sequence's first token of the step reads the old state; it also writes the new one, each thread for its
// own channels after it has read them.  Sums, angles and the rotation are float32.
//
//   conv_qkv_vec_kernel   up to four taps, heads of 16, 32, 64, 128 or 256: a thread owns four neighbouring channels (eight in heads of
//                         256) and slides its window over the run in registers (a row is read once, plus n - 1 rows of the run
//                         before); rotation partners, in halves, are lanes of the same warp.
//   conv_qkv_kernel       any size: a warp a head, a token at a time.
#include "common.cuh"
#include "qk_args.h"

struct ConvQkvArgs {
    const void* in; int in_stride;          // [T][in_stride]: Q heads | K heads | V heads, hd wide each
    const float* taps; int n_taps;          // [n_taps][C], C = (nh + 2 nkv) hd; the last row is the current token's
    float* state; long long state_stride;   // per slot [n_taps - 1][C]; null with one tap
    void* q_out; int q_stride;              // [T][q_stride]
    void* kv_out; int kv_stride;            // [T][kv_stride]: K heads | V heads (null: to the cache only)
    TbRotary rope;
    int nh; int nkv; int hd;
    const int* q_start; const int* start_pos; const int* kv_len; const int* slot_of_seq;
    TbKvView cache; int append;
    int zero_in;                            // steps of single tokens: the input rows are left zeroed (sums of the next step's products)
    int T; int B; int max_new;
};

namespace {

constexpr int RUN = 8, RUN_THREADS = 128;     // tokens and threads of a block of the vector kernel
constexpr int NT = 4;                       // taps of the vector kernel's window (fewer: the window's oldest rows weigh nothing)

// V neighbouring elements of a row as one access.
template <typename T, int V> struct alignas(sizeof(T) * V > 16 ? 16 : sizeof(T) * V) Raw {
    T t[V];
    __device__ __forceinline__ void load(const T* p) { *this = *reinterpret_cast<const Raw*>(p); }
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (int e = 0; e < V; ++e) t[e] = T(0.f);
    }
    __device__ __forceinline__ void get(float* o) const {
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = ldf(t + e);
    }
};
template <int V, typename T> __device__ __forceinline__ void store(T* p, const float* v) {
    Raw<T, V> r;
#pragma unroll
    for (int e = 0; e < V; ++e) stf(r.t + e, v[e]);
    *reinterpret_cast<Raw<T, V>*>(p) = r;
}

// Whether position ``pos`` goes to the cache: in a ring, a row that a later token of the step takes is not written.
__device__ __forceinline__ bool appended(const ConvQkvArgs& a, int pos, int seq) {
    return a.append && !(a.cache.ring_rows && pos < a.kv_len[seq] - a.cache.ring_rows);
}

template <typename TIn, typename TOut, int V, int TOK>
__global__ void __launch_bounds__(128, V == 4 ? 6 : 3) conv_qkv_vec_kernel(ConvQkvArgs a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float angles[];                 // [TOK][rot/2] cosines, then sines
    __shared__ long long row_off[TOK];                // element offset of the token's cache row for kv head 0; < 0: not written
    const int hd = a.hd, C = (a.nh + 2 * a.nkv) * hd, n = a.n_taps, half = a.rope.inv_freq ? a.rope.rot >> 1 : 0;
    const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * V, lane = threadIdx.x & 31;
    const bool live = c0 < C;                         // (a lane without channels still takes part in the shuffles)
    float w[NT][V];                                   // the taps depend on nothing that the kernel before makes
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const int row = j - (NT - n);
#pragma unroll
        for (int e = 0; e < V; ++e) w[j][e] = 0.f;
        if (live && row >= 0) { Raw<float, V> t; t.load(a.taps + (size_t)row * C + c0); t.get(w[j]); }
    }
    pdl_wait();
    const int seq = blockIdx.z, first = a.q_start[seq], L = a.q_start[seq + 1] - first, i0 = blockIdx.x * TOK;
    if (i0 >= L) return;
    const int n_tok = min(TOK, L - i0), slot = a.slot_of_seq[seq], pos0 = a.start_pos[seq] + i0;
    const TIn* in = (const TIn*)a.in + (size_t)first * a.in_stride + c0;
    float* state = a.state ? a.state + (size_t)slot * a.state_stride + c0 : nullptr;
    Raw<TIn, V> raw[TOK];
    float past[NT - 1][V];                            // rows i0 - 3 .. i0 - 1
#pragma unroll
    for (int j = 0; j < TOK; ++j) {
        raw[j].clear();
        if (live && j < n_tok) raw[j].load(in + (size_t)(i0 + j) * a.in_stride);
    }
#pragma unroll
    for (int k = 0; k < NT - 1; ++k) {
        const int r = i0 - (NT - 1) + k, old = n - 1 + r;      // row of the step, or (negative) of the state
#pragma unroll
        for (int e = 0; e < V; ++e) past[k][e] = 0.f;
        if (live && r >= 0) { Raw<TIn, V> t; t.load(in + (size_t)r * a.in_stride); t.get(past[k]); }
        if (live && r < 0 && old >= 0 && state) { Raw<float, V> t; t.load(state + (size_t)old * C); t.get(past[k]); }
    }
    float* cs = angles;
    float* sn = angles + TOK * half;
    for (int i = threadIdx.x; i < n_tok * half; i += blockDim.x) {
        const int j = i / half, k = i - j * half;
        float sv, cv;
        sincosf(((float)(pos0 + j) + a.rope.offset) * a.rope.inv_freq[k], &sv, &cv);
        cs[i] = cv * a.rope.magnitude; sn[i] = sv * a.rope.magnitude;
    }
    if (threadIdx.x < n_tok) row_off[threadIdx.x] = appended(a, pos0 + threadIdx.x, seq) ? (long long)kv_row_offset(a.cache, slot, pos0 + threadIdx.x, 0) : -1;
    if (i0 == 0 && state && live) {                   // the sequence's last n - 1 rows become its state
#pragma unroll
        for (int k = 0; k < NT - 1; ++k) {
            const int idx = L - (NT - 1) + k, row = k - (NT - n);
            float v[V];
            if (row >= 0 && idx >= 0) { Raw<TIn, V> t; t.load(in + (size_t)idx * a.in_stride); t.get(v); }
            // where the step brought fewer, old rows move up: row ``row + L``, which is still as it was
            if (row >= 0 && idx < 0) { Raw<float, V> t; t.load(state + (size_t)(row + L) * C); t.get(v); }
            if (row >= 0) store<V>(state + (size_t)row * C, v);
        }
    }
    if (a.zero_in && live) {                          // one token: this thread has read its channels
        float z[V];
#pragma unroll
        for (int e = 0; e < V; ++e) z[e] = 0.f;
        store<V>((TIn*)const_cast<void*>(a.in) + (size_t)first * a.in_stride + c0, z);
    }
    __syncthreads();
    const int head = c0 / hd, e0 = c0 - head * hd;
    const bool is_q = head < a.nh, is_k = !is_q && head < a.nh + a.nkv;
    const bool turns = live && (is_q || is_k) && e0 < 2 * half;
    const bool lower = e0 < half;
    const int hop = half / V, source = !turns ? lane : (lower ? lane + hop : lane - hop);
    const bool warp_turns = __any_sync(0xffffffffu, turns);
    // where this thread's channels go: a query row, or a key or value row beside the cache (if asked) and the cache's own
    TOut* beside = is_q ? (TOut*)a.q_out + (size_t)(first + i0) * a.q_stride + c0
                        : (a.kv_out ? (TOut*)a.kv_out + (size_t)(first + i0) * a.kv_stride + (c0 - a.nh * hd) : nullptr);
    const size_t beside_stride = is_q ? a.q_stride : a.kv_stride;
    TOut* cached = nullptr;
    if (!is_q && a.append)
        cached = (TOut*)a.cache.storage + e0 + (is_k ? 0 : kv_half_elems(a.cache)) + (size_t)(head - a.nh - (is_k ? 0 : a.nkv)) * a.cache.page_size * a.cache.head_dim;
    const float* trig = angles + (lower ? e0 : e0 - half);
#pragma unroll
    for (int j = 0; j < TOK; ++j) {
        float cur[V], y[V];
        raw[j].get(cur);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w[0][e], past[0][e], fmaf(w[1][e], past[1][e], fmaf(w[2][e], past[2][e], w[3][e] * cur[e])));
#pragma unroll
        for (int e = 0; e < V; ++e) { past[0][e] = past[1][e]; past[1][e] = past[2][e]; past[2][e] = cur[e]; }
        if (warp_turns) {
            float other[V];
#pragma unroll
            for (int e = 0; e < V; ++e) other[e] = __shfl_sync(0xffffffffu, y[e], source);
            if (turns && j < n_tok) {
                Raw<float, 4> c[V / 4], sv[V / 4];        // ``half`` is a multiple of V: whole 16 bytes
#pragma unroll
                for (int r = 0; r < V / 4; ++r) { c[r].load(trig + j * half + 4 * r); sv[r].load(trig + (TOK + j) * half + 4 * r); }
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = fmaf(lower ? -other[e] : other[e], sv[e / 4].t[e % 4], y[e] * c[e / 4].t[e % 4]);
            }
        }
        if (live && j < n_tok) {
            const long long off = row_off[j];
            if (beside) store<V>(beside + j * beside_stride, y);
            if (cached && off >= 0) store<V>(cached + off, y);
        }
    }
}

template <typename TIn, typename TOut>
__global__ void __launch_bounds__(128) conv_qkv_kernel(ConvQkvArgs a, int tile) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ float sm[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.y * (blockDim.x >> 5) + warp;
    const int hd = a.hd, C = (a.nh + 2 * a.nkv) * hd, n = a.n_taps, half = a.rope.inv_freq ? a.rope.rot >> 1 : 0;
    const int seq = blockIdx.z, first = a.q_start[seq], L = a.q_start[seq + 1] - first, i0 = blockIdx.x * tile;
    if (head >= a.nh + 2 * a.nkv || i0 >= L) return;
    float* y = sm + warp * (hd + 2 * half);
    float* cs = y + hd;
    float* sn = cs + half;
    const bool is_q = head < a.nh, is_k = !is_q && head < a.nh + a.nkv;
    const int slot = a.slot_of_seq[seq], col = head * hd;
    const TIn* in = (const TIn*)a.in + (size_t)first * a.in_stride + col;
    float* state = a.state ? a.state + (size_t)slot * a.state_stride + col : nullptr;
    const float* taps = a.taps + col;
    for (int i = i0; i < min(i0 + tile, L); ++i) {
        const int pos = a.start_pos[seq] + i;
        if (is_q || is_k)
            for (int k = lane; k < half; k += 32) {
                float sv, cv;
                sincosf(((float)pos + a.rope.offset) * a.rope.inv_freq[k], &sv, &cv);
                cs[k] = cv * a.rope.magnitude; sn[k] = sv * a.rope.magnitude;
            }
        for (int e = lane; e < hd; e += 32) {
            float acc = 0.f;
            for (int j = 0; j < n; ++j) {
                const int idx = i - (n - 1) + j;
                const float x = idx >= 0 ? ldf(in + (size_t)idx * a.in_stride + e) : state[(size_t)(n - 1 + idx) * C + e];
                acc = fmaf(taps[(size_t)j * C + e], x, acc);
            }
            y[e] = acc;
        }
        __syncwarp();
        const size_t t = first + i;
        TOut* out = is_q ? (TOut*)a.q_out + t * a.q_stride + col : (a.kv_out ? (TOut*)a.kv_out + t * a.kv_stride + (col - a.nh * hd) : nullptr);
        TOut* row = nullptr;
        if (!is_q && appended(a, pos, seq))
            row = (TOut*)a.cache.storage + (is_k ? kv_row_offset(a.cache, slot, pos, head - a.nh)
                                                 : kv_half_elems(a.cache) + kv_row_offset(a.cache, slot, pos, head - a.nh - a.nkv));
        for (int e = lane; e < hd; e += 32) {
            float r = y[e];
            if ((is_q || is_k) && e < 2 * half) {
                int k, partner; float sign;
                tb_rotary_pair(a.rope, e, &k, &partner, &sign);
                r = y[e] * cs[k] + sign * y[partner] * sn[k];
            }
            if (out) stf(out + e, r);
            if (row) stf(row + e, r);
        }
        __syncwarp();
    }
    if (i0 == 0 && state)                             // a lane goes from the oldest row on: every old row is read before it is written over
        for (int e = lane; e < hd; e += 32)
            for (int r = 0; r < n - 1; ++r) {
                const int idx = L - (n - 1) + r;
                state[(size_t)r * C + e] = idx >= 0 ? ldf(in + (size_t)idx * a.in_stride + e) : state[(size_t)(r + L) * C + e];
            }
    if (a.zero_in)
        for (int e = lane; e < hd; e += 32) ((TIn*)const_cast<void*>(a.in))[(size_t)first * a.in_stride + col + e] = TIn(0.f);
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

template <typename TIn, typename TOut, int V, int TOK>
void launch_vec(const ConvQkvArgs& a, int threads, cudaStream_t stream) {
    const int C = (a.nh + 2 * a.nkv) * a.hd, half = a.rope.inv_freq ? a.rope.rot >> 1 : 0;
    dim3 grid((a.max_new + TOK - 1) / TOK, (C / V + threads - 1) / threads, a.B);
    tb_launch(conv_qkv_vec_kernel<TIn, TOut, V, TOK>, grid, dim3(threads), (size_t)2 * TOK * half * sizeof(float), stream, a);
}

// A head's lanes (hd / V of them) divide a warp, and rotation partners are whole vectors apart.
bool vectors_fit(const ConvQkvArgs& a, int V) {
    const int half = a.rope.inv_freq ? a.rope.rot >> 1 : 0;
    return a.hd % V == 0 && a.hd / V <= 32 && 32 % (a.hd / V) == 0 && half % V == 0 && (half == 0 || !a.rope.adjacent);
}

template <typename TIn, typename TOut>
int launch(const ConvQkvArgs& a, bool any_size, cudaStream_t stream) {
    const int half = a.rope.inv_freq ? a.rope.rot >> 1 : 0, heads = a.nh + 2 * a.nkv;
    const bool rows = !any_size && a.n_taps <= NT && a.in_stride % 8 == 0 && a.q_stride % 8 == 0 && a.kv_stride % 8 == 0 && a.state_stride % 4 == 0 && aligned16(a.in) &&
                      aligned16(a.taps) && aligned16(a.state) && aligned16(a.q_out) && aligned16(a.kv_out) && aligned16(a.cache.storage);
    if (rows && vectors_fit(a, 4)) {
        if (a.max_new == 1) launch_vec<TIn, TOut, 4, 1>(a, 32, stream);        // single tokens: many small blocks, a warp's channels each
        else launch_vec<TIn, TOut, 4, RUN>(a, RUN_THREADS, stream);
        return 0;
    }
    if (rows && vectors_fit(a, 8)) {                                           // heads of 256
        if (a.max_new == 1) launch_vec<TIn, TOut, 8, 1>(a, 32, stream);
        else launch_vec<TIn, TOut, 8, 4>(a, 128, stream);
        return 0;
    }
    const int tile = a.n_taps - 1 > 8 ? a.n_taps - 1 : 8;
    dim3 grid((a.max_new + tile - 1) / tile, (heads + 3) / 4, a.B);
    tb_launch(conv_qkv_kernel<TIn, TOut>, grid, dim3(128), (size_t)4 * (a.hd + 2 * half) * sizeof(float), stream, a, tile);
    return 0;
}

}  // namespace

// any_size: the any-size kernel even where the vector kernel fits (tests).
extern "C" int tb_conv_qkv(const ConvQkvArgs* args, int in_dtype, int out_dtype, int any_size, cudaStream_t stream) {
    const ConvQkvArgs& a = *args;
    TB_REQUIRE(a.T > 0 && a.B > 0 && a.B <= 65535 && a.max_new > 0 && a.nh > 0 && a.nkv > 0 && a.hd > 0 && a.hd <= 1024, "conv_qkv: sizes must be positive (heads of at most 1,024, at most 65,535 sequences)");
    TB_REQUIRE(a.n_taps >= 1 && a.n_taps <= 64, "conv_qkv: %d taps (1 to 64)", a.n_taps);
    TB_REQUIRE(a.in && a.taps && a.q_out && a.q_start && a.start_pos && a.kv_len && a.slot_of_seq, "conv_qkv: missing buffers");
    TB_REQUIRE(a.n_taps == 1 || a.state, "conv_qkv: a window over time needs the sequences' states");
    TB_REQUIRE(a.in_stride >= (a.nh + 2 * a.nkv) * a.hd && a.q_stride >= a.nh * a.hd && (!a.kv_out || a.kv_stride >= 2 * a.nkv * a.hd), "conv_qkv: rows too short");
    TB_REQUIRE(a.rope.rot >= 0 && a.rope.rot <= a.hd && a.rope.rot % 2 == 0, "conv_qkv: %d rotated elements must be even and within a head of %d", a.rope.rot, a.hd);
    TB_REQUIRE(!a.append || (a.cache.storage && a.cache.kv_heads == a.nkv && a.cache.head_dim == a.hd), "conv_qkv: the cache view does not match the heads");
    TB_REQUIRE(a.append || a.kv_out, "conv_qkv: keys and values need somewhere to go");
    TB_REQUIRE(!a.zero_in || a.max_new == 1, "conv_qkv: input rows are zeroed in steps of single tokens only");
    TB_REQUIRE(a.in != a.q_out && a.in != a.kv_out, "conv_qkv: later tokens read the input rows: the output lies elsewhere");
    if (in_dtype == TB_F32 && out_dtype == TB_F32) launch<float, float>(a, any_size, stream);
    else if (in_dtype == TB_BF16 && out_dtype == TB_BF16) launch<__nv_bfloat16, __nv_bfloat16>(a, any_size, stream);
    else if (in_dtype == TB_F32 && out_dtype == TB_BF16) launch<float, __nv_bfloat16>(a, any_size, stream);
    else TB_REQUIRE(false, "conv_qkv: unsupported dtypes in=%d out=%d", in_dtype, out_dtype);
    TB_CHECK_LAUNCH("conv_qkv");
    return 0;
}
