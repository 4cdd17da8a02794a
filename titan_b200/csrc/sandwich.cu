// The element-wise work of a block whose sublayers are normed before AND after, with a token shift in front of its mixer
// and an average over depth behind it.
//
//   tb_sandwich_join   a sublayer's result y joins the residual stream:  x <- x + rms(y) * post_w,  y <- 0.  With it, each if
//                      asked: the rows of x as they were are kept (``keep``); the new rows enter the history of the rows that
//                      left earlier layers, and x becomes the weighted sum of that history (``dwa``, the new row included); the
//                      next sublayer's normed rows h = rms(x) * pre_w leave in the compute dtype; in a step of single tokens
//                      those rows are shifted on the way (below).
//   tb_shift_norm      h = g + (g' - g) * mu with g = rms(x) * w and g' the row of the same sequence's previous token: the
//                      row before inside the step, or, for a sequence's first row of the step, what the step before left in
//                      the sequence's state (zeros at its start).  The state then holds the g of the sequence's last row.
//
// Everything is float32 up to the rounding of h; one block a row (tb_shift_norm: a few neighbouring rows).  A thread owns the
// same elements of every row it works on, so what one phase stores to memory the next reads back without a barrier.
#include "common.cuh"

struct SandwichArgs {
    float* y; const float* post_w; float post_eps;      // [rows][W]
    float* x; int W; int rows;                          // [rows][W], in place
    float* keep;                                        // [rows][W] or null: x as it was
    float* hist; long long hist_stride; int n_hist;     // n_hist > 0: rows of depth j at hist + j * hist_stride, j < n_hist
    const float* dwa;                                   // [n_hist + 1]
    int store_hist;                                     // the new rows go to depth n_hist (a later layer will read them)
    const float* pre_w; float pre_eps; void* h;         // h null: no norm of the new rows
    const float* mu;                                    // null: no shift
    float* state; long long state_stride; const int* slot_of_row;      // [slots][state_stride]: the previous token's g, by slot
};

struct ShiftNormArgs {
    const float* x; int W; int rows;
    const float* w; float eps; const float* mu; void* h;
    float* state; long long state_stride;
    const int* seq_of; const int* q_start; const int* slot_of_seq;
    int rows_per_block;
};

namespace {

template <int V> struct alignas(4 * V) Vec { float v[V]; };
template <int V> __device__ __forceinline__ Vec<V> ldv(const float* p) { return *reinterpret_cast<const Vec<V>*>(p); }
template <int V> __device__ __forceinline__ void stv(float* p, const Vec<V>& v) { *reinterpret_cast<Vec<V>*>(p) = v; }
template <typename T, int V> __device__ __forceinline__ void sth(T* p, const Vec<V>& v) {
    struct alignas(sizeof(T) * V) Out { T t[V]; } o;
#pragma unroll
    for (int e = 0; e < V; ++e) stf(o.t + e, v.v[e]);
    *reinterpret_cast<Out*>(p) = o;
}
template <int V> __device__ __forceinline__ float sum_sq(const Vec<V>& v) {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s = fmaf(v.v[e], v.v[e], s);
    return s;
}

// NR > 0: a row fits NR vectors of V elements a thread, held in registers from the first read to the last write.
// NR = 0: rows of any width, read again from memory (each element by the thread that wrote it).
template <typename T, int V, int NR>
__global__ void __launch_bounds__(NR >= 4 ? 512 : 1024) sandwich_join_kernel(SandwichArgs a) {
    pdl_launch_dependents();
    __shared__ float red[33];
    const size_t t = blockIdx.x;
    const int W = a.W, step = blockDim.x * V, first = threadIdx.x * V;
    float* y = a.y + t * W;
    float* x = a.x + t * W;
    if constexpr (NR > 0) {
        Vec<V> vy[NR], vx[NR], vw[NR];
        // the weights depend on nothing that the kernel before makes: requested while the wait for it lasts
#pragma unroll
        for (int j = 0; j < NR; ++j)
            if (first + j * step < W) vw[j] = ldv<V>(a.post_w + first + j * step);
        pdl_wait();
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NR; ++j) {
            const int i = first + j * step;
            if (i < W) { vy[j] = ldv<V>(y + i); vx[j] = ldv<V>(x + i); ss += sum_sq<V>(vy[j]); }
        }
        // the history does not depend on y's norm: its sum is gathered while the block adds up
        Vec<V> av[NR];
        if (a.n_hist > 0) {
#pragma unroll
            for (int j = 0; j < NR; ++j) {
                const int i = first + j * step;
#pragma unroll
                for (int e = 0; e < V; ++e) av[j].v[e] = 0.f;
                if (i >= W) continue;
                const float* hrow = a.hist + t * W + i;
                int d = 0;
                if (a.keep == a.hist) {                      // depth 0 is being made in this launch: it is x as it was
                    const float w0 = a.dwa[0];
#pragma unroll
                    for (int e = 0; e < V; ++e) av[j].v[e] = w0 * vx[j].v[e];
                    d = 1;
                }
#pragma unroll 4
                for (; d < a.n_hist; ++d) {
                    const Vec<V> hv = ldv<V>(hrow + (size_t)d * a.hist_stride);
                    const float wd = a.dwa[d];
#pragma unroll
                    for (int e = 0; e < V; ++e) av[j].v[e] = fmaf(wd, hv.v[e], av[j].v[e]);
                }
            }
        }
        const float scale = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.post_eps);
        const float w_new = a.n_hist > 0 ? a.dwa[a.n_hist] : 0.f;
        Vec<V> zero;
#pragma unroll
        for (int e = 0; e < V; ++e) zero.v[e] = 0.f;
        ss = 0.f;
#pragma unroll
        for (int j = 0; j < NR; ++j) {
            const int i = first + j * step;
            if (i >= W) continue;
            if (a.keep) stv<V>(a.keep + t * W + i, vx[j]);
#pragma unroll
            for (int e = 0; e < V; ++e) vx[j].v[e] += vy[j].v[e] * scale * vw[j].v[e];
            if (a.n_hist > 0) {
                if (a.store_hist) stv<V>(a.hist + (size_t)a.n_hist * a.hist_stride + t * W + i, vx[j]);
#pragma unroll
                for (int e = 0; e < V; ++e) vx[j].v[e] = fmaf(w_new, vx[j].v[e], av[j].v[e]);
            }
            stv<V>(x + i, vx[j]);
            stv<V>(y + i, zero);
            ss += sum_sq<V>(vx[j]);
        }
        if (!a.h) return;
        const float pre = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.pre_eps);
        float* st = a.mu ? a.state + (size_t)a.slot_of_row[t] * a.state_stride : nullptr;
#pragma unroll
        for (int j = 0; j < NR; ++j) {
            const int i = first + j * step;
            if (i >= W) continue;
            const Vec<V> pw = ldv<V>(a.pre_w + i);
#pragma unroll
            for (int e = 0; e < V; ++e) vx[j].v[e] = vx[j].v[e] * pre * pw.v[e];
            if (st) {
                const Vec<V> before = ldv<V>(st + i), m = ldv<V>(a.mu + i);
                stv<V>(st + i, vx[j]);
#pragma unroll
                for (int e = 0; e < V; ++e) vx[j].v[e] = fmaf(before.v[e] - vx[j].v[e], m.v[e], vx[j].v[e]);
            }
            sth<T, V>((T*)a.h + t * W + i, vx[j]);
        }
    } else {
        pdl_wait();
        float ss = 0.f;
        for (int i = first; i < W; i += step) ss += sum_sq<V>(ldv<V>(y + i));
        const float scale = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.post_eps);
        ss = 0.f;
        for (int i = first; i < W; i += step) {
            const Vec<V> vy = ldv<V>(y + i), vw = ldv<V>(a.post_w + i);
            Vec<V> vx = ldv<V>(x + i);
            if (a.keep) stv<V>(a.keep + t * W + i, vx);
#pragma unroll
            for (int e = 0; e < V; ++e) vx.v[e] += vy.v[e] * scale * vw.v[e];
            if (a.n_hist > 0) {
                if (a.store_hist) stv<V>(a.hist + (size_t)a.n_hist * a.hist_stride + t * W + i, vx);
                const float w_new = a.dwa[a.n_hist];
                Vec<V> s;
#pragma unroll
                for (int e = 0; e < V; ++e) s.v[e] = 0.f;
                for (int d = 0; d < a.n_hist; ++d) {
                    const Vec<V> hv = ldv<V>(a.hist + (size_t)d * a.hist_stride + t * W + i);
                    const float wd = a.dwa[d];
#pragma unroll
                    for (int e = 0; e < V; ++e) s.v[e] = fmaf(wd, hv.v[e], s.v[e]);
                }
#pragma unroll
                for (int e = 0; e < V; ++e) vx.v[e] = fmaf(w_new, vx.v[e], s.v[e]);
            }
            stv<V>(x + i, vx);
            Vec<V> zero;
#pragma unroll
            for (int e = 0; e < V; ++e) zero.v[e] = 0.f;
            stv<V>(y + i, zero);
            ss += sum_sq<V>(vx);
        }
        if (!a.h) return;
        const float pre = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.pre_eps);
        float* st = a.mu ? a.state + (size_t)a.slot_of_row[t] * a.state_stride : nullptr;
        for (int i = first; i < W; i += step) {
            Vec<V> g = ldv<V>(x + i);
            const Vec<V> pw = ldv<V>(a.pre_w + i);
#pragma unroll
            for (int e = 0; e < V; ++e) g.v[e] = g.v[e] * pre * pw.v[e];
            if (st) {
                const Vec<V> before = ldv<V>(st + i), m = ldv<V>(a.mu + i);
                stv<V>(st + i, g);
#pragma unroll
                for (int e = 0; e < V; ++e) g.v[e] = fmaf(before.v[e] - g.v[e], m.v[e], g.v[e]);
            }
            sth<T, V>((T*)a.h + t * W + i, g);
        }
    }
}

template <int V>
__device__ __forceinline__ float row_scale(const float* x, int W, float eps, float* red) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) ss += sum_sq<V>(ldv<V>(x + i));
    return 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
}

// A block takes ``rows_per_block`` neighbouring rows; the scale of the row before comes along from one row to the next, and
// its elements are read again (from L1 or L2).
template <typename T, int V>
__global__ void __launch_bounds__(512) shift_norm_kernel(ShiftNormArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[33];
    const int W = a.W, r0 = blockIdx.x * a.rows_per_block, r1 = min(a.rows, r0 + a.rows_per_block);
    float before = 0.f;                                   // scale of row r - 1, if that row is of the same sequence
    for (int r = r0; r < r1; ++r) {
        const int seq = a.seq_of[r];
        const bool first = r == a.q_start[seq];
        const float* x = a.x + (size_t)r * W;
        if (!first && r == r0) before = row_scale<V>(x - W, W, a.eps, red);
        const float scale = row_scale<V>(x, W, a.eps, red);
        T* h = (T*)a.h + (size_t)r * W;
        if (!first) {
            for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
                const Vec<V> u = ldv<V>(x + i), p = ldv<V>(x - W + i), w = ldv<V>(a.w + i), m = ldv<V>(a.mu + i);
                Vec<V> o;
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const float g = u.v[e] * scale * w.v[e], q = p.v[e] * before * w.v[e];
                    o.v[e] = fmaf(q - g, m.v[e], g);
                }
                sth<T, V>(h + i, o);
            }
        } else {
            // this block also leaves the sequence's last row in the state, each thread after it has read what lay there
            const int last = a.q_start[seq + 1] - 1;
            const float* xl = a.x + (size_t)last * W;
            const float scale_l = last == r ? scale : row_scale<V>(xl, W, a.eps, red);
            float* st = a.state + (size_t)a.slot_of_seq[seq] * a.state_stride;
            for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
                const Vec<V> u = ldv<V>(x + i), p = ldv<V>(st + i), l = ldv<V>(xl + i), w = ldv<V>(a.w + i), m = ldv<V>(a.mu + i);
                Vec<V> o, s;
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const float g = u.v[e] * scale * w.v[e];
                    o.v[e] = fmaf(p.v[e] - g, m.v[e], g);
                    s.v[e] = l.v[e] * scale_l * w.v[e];
                }
                stv<V>(st + i, s);
                sth<T, V>(h + i, o);
            }
        }
        before = scale;
    }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }
int threads_for(int vectors) { int t = 32; while (t < vectors && t < 1024) t <<= 1; return t; }

template <typename T>
int launch_join(const SandwichArgs& a, cudaStream_t stream) {
    const bool vec = a.W % 4 == 0 && a.hist_stride % 4 == 0 && a.state_stride % 4 == 0 && aligned16(a.y) && aligned16(a.x) && aligned16(a.post_w) &&
                     aligned16(a.keep) && aligned16(a.hist) && aligned16(a.pre_w) && aligned16(a.h) && aligned16(a.mu) && aligned16(a.state);
    if (!vec) {
        tb_launch(sandwich_join_kernel<T, 1, 0>, a.rows, a.W >= 512 ? 256 : 64, 0, stream, a);
        return 0;
    }
    // a few rows: many threads a row, one vector each; many rows: two or four vectors a thread, so that more rows are in flight
    // (two where the history is read as well: its sums take registers)
    const int n4 = a.W / 4, per = a.rows <= 296 ? 1 : (n4 >= 512 && a.n_hist == 0 ? 4 : 2);
    int threads = threads_for((n4 + per - 1) / per);
    const int held = (n4 + threads - 1) / threads;
    if (held <= 1) tb_launch(sandwich_join_kernel<T, 4, 1>, a.rows, threads, 0, stream, a);
    else if (held <= 2) tb_launch(sandwich_join_kernel<T, 4, 2>, a.rows, threads, 0, stream, a);
    else if (held <= 4 && threads <= 512) tb_launch(sandwich_join_kernel<T, 4, 4>, a.rows, threads, 0, stream, a);
    else tb_launch(sandwich_join_kernel<T, 4, 0>, a.rows, threads, 0, stream, a);
    return 0;
}

template <typename T>
int launch_shift(const ShiftNormArgs& a, cudaStream_t stream) {
    const bool vec = a.W % 4 == 0 && a.state_stride % 4 == 0 && aligned16(a.x) && aligned16(a.w) && aligned16(a.mu) && aligned16(a.h) && aligned16(a.state);
    const int grid = (a.rows + a.rows_per_block - 1) / a.rows_per_block;
    const int vectors = vec ? a.W / 4 : a.W;
    int threads = threads_for((vectors + 1) / 2);
    if (threads > 512) threads = 512;
    if (vec) tb_launch(shift_norm_kernel<T, 4>, grid, threads, 0, stream, a);
    else tb_launch(shift_norm_kernel<T, 1>, grid, threads, 0, stream, a);
    return 0;
}

}  // namespace

extern "C" int tb_sandwich_join(const SandwichArgs* args, int h_dtype, cudaStream_t stream) {
    const SandwichArgs& a = *args;
    TB_REQUIRE(a.rows > 0 && a.W > 0 && a.y && a.x && a.post_w, "sandwich_join: a sublayer's rows, the residual rows and the norm's weight are wanted");
    TB_REQUIRE(a.n_hist >= 0 && (a.n_hist == 0 || (a.hist && a.dwa && a.hist_stride >= (long long)a.rows * a.W)), "sandwich_join: an average over depth needs its history and weights");
    TB_REQUIRE(!a.h || a.pre_w, "sandwich_join: normed rows are wanted without the norm's weight");
    TB_REQUIRE(!a.mu || (a.h && a.state && a.slot_of_row && a.state_stride >= a.W), "sandwich_join: a shift needs the normed rows and the sequences' states");
    if (!a.h || h_dtype == TB_F32) launch_join<float>(a, stream);
    else if (h_dtype == TB_BF16) launch_join<__nv_bfloat16>(a, stream);
    else TB_REQUIRE(false, "sandwich_join: unknown dtype %d", h_dtype);
    TB_CHECK_LAUNCH("sandwich_join");
    return 0;
}

extern "C" int tb_shift_norm(const ShiftNormArgs* args, int h_dtype, cudaStream_t stream) {
    ShiftNormArgs a = *args;
    TB_REQUIRE(a.rows > 0 && a.W > 0 && a.x && a.w && a.mu && a.h, "shift_norm: rows, the norm's weight and the shift's factors are wanted");
    TB_REQUIRE(a.state && a.state_stride >= a.W && a.seq_of && a.q_start && a.slot_of_seq, "shift_norm: the sequences' states are wanted");
    if (a.rows_per_block <= 0) a.rows_per_block = a.rows >= 592 ? 2 : 1;
    if (h_dtype == TB_F32) launch_shift<float>(a, stream);
    else if (h_dtype == TB_BF16) launch_shift<__nv_bfloat16>(a, stream);
    else TB_REQUIRE(false, "shift_norm: unknown dtype %d", h_dtype);
    TB_CHECK_LAUNCH("shift_norm");
    return 0;
}
