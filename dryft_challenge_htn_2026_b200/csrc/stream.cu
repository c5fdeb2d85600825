// Row kernels around the float32 residual stream for blocks that norm a sublayer's OUTPUT before it joins the stream and
// whose mixers read the stream mixed with the stream of the token before:
//   * embed_bigram      : h = embed[tok] * scale + table[pair row], the pair row from this token and the one before it in
//                         its sequence (the last row of the table for a sequence's first token); the last token of every
//                         sequence is per-sequence state.
//   * sublayer_add      : h_out = h + norm(d), and a = that row in the storage type, or its next norm. d is a sublayer's
//                         output (a tensor or split-K partial sums), or a scaled sum of two of them, each over its own root
//                         mean square times a weight first. norm is a layer norm (mean taken off) or an RMS norm, with a
//                         weight and, where given, a bias, or none. Without an h the stream starts anew from a vector (null:
//                         zero), the same for every row. With ``rows`` the kernel gathers and leaves h alone. It may also put the stream as
//                         it stood BEFORE the sum into the shift's state at every sequence's last row: that is the vector the
//                         mixer in front of it has read, and by now every reader of the old state is done.
//   * sublayer_add_shift: the same sum, then a = x + (x_prev - x) * share with x_prev the row of the token before (the
//                         sequence's state at the first row of a step). A block takes several consecutive rows and works
//                         the row ahead of them out once more, so h_out must not be h.
//   * stream_save       : the stream at every sequence's last row into the shift's state, where no sublayer_add follows.
// All arithmetic is float32. A block per row (or run of rows); a thread keeps its columns in registers.
#include "common.cuh"

template <typename T> struct Source {
    const T* x;              // [rows, H] in the storage type, or null
    const float* parts;      // n_parts float32 partial sums [n_parts][rows][H], or null
    int n_parts;
    size_t stride;
    const float* w;          // RMS weight of this source (null: taken as it is)
};
struct NormArgs {
    const float* w;          // null: no norm
    const float* b;          // null: no bias
    float eps;
    int center;              // 1: layer norm, 0: RMS norm
};
template <typename T> struct AddArgs {
    Source<T> s0, s1;        // s1.x and s1.parts null: one source
    float pre_eps, pre_scale;   // of the sources' RMS norms and of their sum
    NormArgs norm;
};

__device__ __forceinline__ void ld_cols(const float* p, int c, int H, bool vec, float (&v)[4]) {
    if (vec) {
        const float4 x = c < H ? *reinterpret_cast<const float4*>(p + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
        return;
    }
#pragma unroll
    for (int k = 0; k < 4; k++) v[k] = c + k < H ? p[c + k] : 0.f;
}
__device__ __forceinline__ void ld_cols(const bf16* p, int c, int H, bool vec, float (&v)[4]) {
    if (vec) {
        uint2 r = make_uint2(0u, 0u);
        if (c < H) r = *reinterpret_cast<const uint2*>(p + c);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
        v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
        return;
    }
#pragma unroll
    for (int k = 0; k < 4; k++) v[k] = c + k < H ? __bfloat162float(p[c + k]) : 0.f;
}
__device__ __forceinline__ void st_cols(float* p, int c, int H, bool vec, const float (&v)[4]) {
    if (vec) {
        if (c < H) *reinterpret_cast<float4*>(p + c) = make_float4(v[0], v[1], v[2], v[3]);
        return;
    }
#pragma unroll
    for (int k = 0; k < 4; k++)
        if (c + k < H) p[c + k] = v[k];
}
__device__ __forceinline__ void st_cols(bf16* p, int c, int H, bool vec, const float (&v)[4]) {
    if (vec) {
        if (c >= H) return;
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        uint2 o;
        o.x = *reinterpret_cast<uint32_t*>(&lo);
        o.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p + c) = o;
        return;
    }
#pragma unroll
    for (int k = 0; k < 4; k++)
        if (c + k < H) p[c + k] = __float2bfloat16_rn(v[k]);
}

// Sums over the block of two values, every thread gets both. Two buffers in turn, so one barrier a call is enough: a warp
// that comes to the call after next has seen every warp past the barrier in between.
struct BlockSums {
    float2 (*red)[32];
    int turn;
    __device__ __forceinline__ float2 operator()(float a, float b) {
        const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
        a = warp_sum(a), b = warp_sum(b);
        if (lane == 0) red[turn][w] = make_float2(a, b);
        __syncthreads();
        float2 t = make_float2(0.f, 0.f);
        for (int i = 0; i < nw; i++) {
            const float2 x = red[turn][i];
            t.x += x.x, t.y += x.y;
        }
        turn ^= 1;
        return t;
    }
};

// d <- norm(d)
template <int NV>
__device__ __forceinline__ void norm_row(float (&d)[NV][4], const NormArgs& n, int H, bool vec, BlockSums& sums) {
    float mean = 0.f;
    if (n.center) {
        float s = 0.f;
#pragma unroll
        for (int q = 0; q < NV; q++) s += (d[q][0] + d[q][1]) + (d[q][2] + d[q][3]);      // columns past H are zero
        mean = sums(s, 0.f).x / (float)H;
    }
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < NV; q++) {
        const int c = (threadIdx.x + q * blockDim.x) * 4;
#pragma unroll
        for (int k = 0; k < 4; k++) {
            d[q][k] = c + k < H ? d[q][k] - mean : 0.f;
            ss += d[q][k] * d[q][k];
        }
    }
    const float rs = 1.f / sqrtf(sums(ss, 0.f).x / (float)H + n.eps);
#pragma unroll
    for (int q = 0; q < NV; q++) {
        float w[4];
        ld_cols(n.w, (threadIdx.x + q * blockDim.x) * 4, H, vec, w);
#pragma unroll
        for (int k = 0; k < 4; k++) d[q][k] *= rs * w[k];
        if (n.b) {
            ld_cols(n.b, (threadIdx.x + q * blockDim.x) * 4, H, vec, w);
#pragma unroll
            for (int k = 0; k < 4; k++) d[q][k] += w[k];
        }
    }
}

template <typename T, int NV>
__device__ __forceinline__ void load_source(float (&d)[NV][4], const Source<T>& s, size_t row, int H, bool vec) {
#pragma unroll
    for (int q = 0; q < NV; q++) {
        const int c = (threadIdx.x + q * blockDim.x) * 4;
        if (s.x) ld_cols(s.x + row * H, c, H, vec, d[q]);
        else d[q][0] = d[q][1] = d[q][2] = d[q][3] = 0.f;
    }
    for (int k = 0; k < s.n_parts; k++)
#pragma unroll
        for (int q = 0; q < NV; q++) {
            float p[4];
            ld_cols(s.parts + (size_t)k * s.stride + row * H, (threadIdx.x + q * blockDim.x) * 4, H, vec, p);
#pragma unroll
            for (int i = 0; i < 4; i++) d[q][i] += p[i];
        }
}

// v <- h[row] + norm(delta[row]): first the loads, which wait for nothing, ...
template <typename T, int NV, bool TWO>
__device__ __forceinline__ void load_row(float (&v)[NV][4], float (&d)[NV][4], float (&e)[TWO ? NV : 1][4], const float* h, size_t row,
                                         const AddArgs<T>& a, int H, bool vec, const float* base = nullptr) {
    const float* from = h ? h + row * H : base;          // the stream, or the vector it starts anew from
#pragma unroll
    for (int q = 0; q < NV; q++) {
        if (from) ld_cols(from, (threadIdx.x + q * blockDim.x) * 4, H, vec, v[q]);
        else v[q][0] = v[q][1] = v[q][2] = v[q][3] = 0.f;
    }
    if (a.s0.x || a.s0.parts) load_source<T, NV>(d, a.s0, row, H, vec);
    if constexpr (TWO) load_source<T, NV>(e, a.s1, row, H, vec);
}
// ... then the norms and the sum
template <typename T, int NV, bool TWO>
__device__ __forceinline__ void sum_row(float (&v)[NV][4], float (&d)[NV][4], float (&e)[TWO ? NV : 1][4], const AddArgs<T>& a, int H, bool vec,
                                        BlockSums& sums) {
    if (!a.s0.x && !a.s0.parts) return;
    if (a.s0.w) {
        float sd = 0.f, se = 0.f;
#pragma unroll
        for (int q = 0; q < NV; q++)
#pragma unroll
            for (int k = 0; k < 4; k++) {
                sd += d[q][k] * d[q][k];
                if constexpr (TWO) se += e[q][k] * e[q][k];
            }
        const float2 t = sums(sd, se);
        const float rd = a.pre_scale / sqrtf(t.x / (float)H + a.pre_eps), re = a.pre_scale / sqrtf(t.y / (float)H + a.pre_eps);
#pragma unroll
        for (int q = 0; q < NV; q++) {
            const int c = (threadIdx.x + q * blockDim.x) * 4;
            float w[4];
            ld_cols(a.s0.w, c, H, vec, w);
#pragma unroll
            for (int k = 0; k < 4; k++) d[q][k] *= rd * w[k];
            if constexpr (TWO) {
                ld_cols(a.s1.w, c, H, vec, w);
#pragma unroll
                for (int k = 0; k < 4; k++) d[q][k] = fmaf(e[q][k], re * w[k], d[q][k]);
            }
        }
    }
    if (a.norm.w) norm_row<NV>(d, a.norm, H, vec, sums);
#pragma unroll
    for (int q = 0; q < NV; q++)
#pragma unroll
        for (int k = 0; k < 4; k++) v[q][k] += d[q][k];
}

template <typename T, int NV, bool TWO, int MAXT>
__global__ void __launch_bounds__(MAXT)
sublayer_add_kernel(const float* h, const float* base, float* h_out, const AddArgs<T> args, const int* rows, NormArgs next, T* a, long long lda, float* save,
                    const int* row_pos, const int* row_seq, const int* cu_q, const int* seq_slot, int H, int vec) {
    __shared__ float2 red[2][32];
    BlockSums sums{red, 0};
    pdl_wait();
    pdl_launch_dependents();
    const size_t out_row = blockIdx.x, row = rows ? (size_t)rows[out_row] : out_row;
    float v[NV][4], d[NV][4], e[TWO ? NV : 1][4];
    load_row<T, NV, TWO>(v, d, e, h, row, args, H, vec, base);
    if (save != nullptr && row_pos[row] >= 0) {
        const int s = row_seq[row];
        if (cu_q == nullptr || (int)row + 1 == cu_q[s + 1]) {
            float* to = save + (size_t)seq_slot[s] * H;
#pragma unroll
            for (int q = 0; q < NV; q++) st_cols(to, (threadIdx.x + q * blockDim.x) * 4, H, vec, v[q]);
        }
    }
    sum_row<T, NV, TWO>(v, d, e, args, H, vec, sums);
    if (h_out != nullptr) {
#pragma unroll
        for (int q = 0; q < NV; q++) st_cols(h_out + row * H, (threadIdx.x + q * blockDim.x) * 4, H, vec, v[q]);
    }
    if (a == nullptr) return;
    if (next.w) norm_row<NV>(v, next, H, vec, sums);
#pragma unroll
    for (int q = 0; q < NV; q++) st_cols(a + out_row * lda, (threadIdx.x + q * blockDim.x) * 4, H, vec, v[q]);
}

template <typename T, int NV, bool TWO, int MAXT>
__global__ void __launch_bounds__(MAXT)
sublayer_add_shift_kernel(const float* h, float* h_out, const AddArgs<T> args, const float* __restrict__ share, const float* state,
                          const int* row_pos, const int* row_seq, const int* cu_q, const int* seq_slot, int n_rows, int run,
                          T* a, int H, int vec) {
    __shared__ float2 red[2][32];
    BlockSums sums{red, 0};
    pdl_wait();
    pdl_launch_dependents();
    const int r0 = blockIdx.x * run, r1 = min(n_rows, r0 + run);
    float prev[NV][4], v[NV][4], d[NV][4], e[TWO ? NV : 1][4];
    // whether row r is the first its sequence brings (or a padding row), so that its row before is not the one above
    auto starts = [&](int r) { return row_pos[r] < 0 || cu_q == nullptr || r == cu_q[row_seq[r]]; };
    bool first = starts(r0);
    for (int r = first ? r0 : r0 - 1; r < r1; r++) {         // else the row ahead of the run is worked out once more
        load_row<T, NV, TWO>(v, d, e, h, (size_t)r, args, H, vec);
        const bool mine = r >= r0;
        if (mine && r > r0) first = starts(r);
        if (mine && first) {
            if (row_pos[r] < 0) {
#pragma unroll
                for (int q = 0; q < NV; q++) prev[q][0] = prev[q][1] = prev[q][2] = prev[q][3] = 0.f;
            } else {                                         // what the step before left
                const float* st = state + (size_t)seq_slot[row_seq[r]] * H;
#pragma unroll
                for (int q = 0; q < NV; q++) ld_cols(st, (threadIdx.x + q * blockDim.x) * 4, H, vec, prev[q]);
            }
        }
        sum_row<T, NV, TWO>(v, d, e, args, H, vec, sums);
#pragma unroll
        for (int q = 0; q < NV; q++) {
            const int c = (threadIdx.x + q * blockDim.x) * 4;
            if (mine) {
                float w[4], o[4];
                ld_cols(share, c, H, vec, w);
                if (h_out != nullptr) st_cols(h_out + (size_t)r * H, c, H, vec, v[q]);
#pragma unroll
                for (int k = 0; k < 4; k++) o[k] = fmaf(prev[q][k] - v[q][k], w[k], v[q][k]);
                st_cols(a + (size_t)r * H, c, H, vec, o);
            }
#pragma unroll
            for (int k = 0; k < 4; k++) prev[q][k] = v[q][k];
        }
    }
}

__global__ void stream_save_kernel(const float* h, float* state, const int* cu_q, const int* seq_pos0, const int* seq_slot, int H) {
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x;
    if (seq_pos0[s] < 0) return;
    const size_t row = cu_q ? (size_t)cu_q[s + 1] - 1 : (size_t)s;
    float* to = state + (size_t)seq_slot[s] * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) to[i] = h[row * H + i];
}

// The block of a sequence's first row in the step reads the state and then stores the last token the sequence brings: one
// thread does both, so nobody reads the new one.
template <typename T>
__global__ void embed_bigram_kernel(const int* tok, const T* __restrict__ embed, float scale, const T* __restrict__ table,
                                    int buckets, long long mul_prev, long long mul_cur, int* state, const int* row_pos,
                                    const int* row_seq, const int* cu_q, const int* seq_slot, int H, int V, float* h) {
    __shared__ int pair_row;
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    int t = tok[r];
    t = t < 0 ? 0 : (t >= V ? V - 1 : t);       // ids are validated on the host; never read out of bounds
    if (threadIdx.x == 0) {
        const int pos = row_pos[r];
        int row = buckets;
        if (pos >= 0) {
            const int s = row_seq[r];
            const bool first = cu_q == nullptr || r == cu_q[s];
            int* st = state + seq_slot[s];
            const int prev = first ? *st : tok[r - 1];
            if (first) *st = cu_q ? tok[cu_q[s + 1] - 1] : tok[r];
            if (pos > 0) row = (int)(((long long)prev * mul_prev + (long long)t * mul_cur) % buckets);
        }
        pair_row = row < 0 ? 0 : (row > buckets ? buckets : row);
    }
    __syncthreads();
    const T* e = embed + (size_t)t * H;
    const T* b = table + (size_t)pair_row * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) h[(size_t)r * H + i] = fmaf(to_f(e[i]), scale, to_f(b[i]));
}

// Few rows (a decode step): every column of a row at once, four a thread. Many rows: eight a thread, which leaves room for
// more blocks an SM (up to 4,096 columns; wider rows take 512 threads).
static inline int stream_threads(int H, int n_rows) {
    const int quads = (H + 3) / 4;
    if (quads > 2048) return 1024;
    if (n_rows <= 256 && quads <= 1024) return (quads + 31) / 32 * 32;
    return quads > 1024 ? 512 : ((quads + 1) / 2 + 31) / 32 * 32;
}

#define STREAM_DISPATCH(dtype, ...)                     \
    if ((dtype) == 0) { typedef float T; __VA_ARGS__; } \
    else { typedef bf16 T; __VA_ARGS__; }

template <typename T>
static AddArgs<T> make_add(const void* x0, const float* parts0, int n0, long long stride0, const float* w0, const void* x1,
                           const float* parts1, int n1, long long stride1, const float* w1, float pre_eps, float pre_scale,
                           const float* norm_w, const float* norm_b, float eps, int center) {
    AddArgs<T> a;
    a.s0 = {(const T*)x0, parts0, n0, (size_t)stride0, w0};
    a.s1 = {(const T*)x1, parts1, n1, (size_t)stride1, w1};
    a.pre_eps = pre_eps, a.pre_scale = pre_scale;
    a.norm = {norm_w, norm_b, eps, center};
    return a;
}

#define ADD_PARAMS const void *x0, const float *parts0, int n0, long long stride0, const float *w0, const void *x1,          \
                   const float *parts1, int n1, long long stride1, const float *w1, float pre_eps, float pre_scale,          \
                   const float *norm_w, const float *norm_b, float eps, int center
#define ADD_NAMES x0, parts0, n0, stride0, w0, x1, parts1, n1, stride1, w1, pre_eps, pre_scale, norm_w, norm_b, eps, center
// four columns at a time where rows, partial sums and every pointer sit on 16-byte boundaries
#define ADD_VEC (H % 4 == 0 && stride0 % 4 == 0 && stride1 % 4 == 0 &&                                                        \
                 (((uintptr_t)h | (uintptr_t)h_out | (uintptr_t)x0 | (uintptr_t)parts0 | (uintptr_t)w0 | (uintptr_t)x1 |      \
                   (uintptr_t)parts1 | (uintptr_t)w1 | (uintptr_t)norm_w | (uintptr_t)norm_b | (uintptr_t)a) % 16 == 0))

DK_EXPORT int dk_sublayer_add(int dtype, const float* h, const float* base, float* h_out, ADD_PARAMS, const int* rows, const float* next_w,
                              const float* next_b, float next_eps, int next_center, void* a, long long lda, float* save, const int* row_pos, const int* row_seq,
                              const int* cu_q, const int* seq_slot, int n_rows, int H, cudaStream_t st) {
    if (H < 1 || H > 16384) return (int)cudaErrorInvalidValue;
    const int threads = stream_threads(H, n_rows), nv = ((H + 3) / 4 + threads - 1) / threads;
    const int vec = ADD_VEC && lda % 4 == 0 && ((uintptr_t)next_w | (uintptr_t)next_b | (uintptr_t)base | (uintptr_t)save) % 16 == 0;
    const NormArgs next = {next_w, next_b, next_eps, next_center};
    const bool two = x1 != nullptr || parts1 != nullptr;
#define ADD_GO(NV, TWO, MAXT)                                                                                                       \
    STREAM_DISPATCH(dtype, return dk_launch(sublayer_add_kernel<T, NV, TWO, MAXT>, dim3(n_rows), dim3(threads), 0, st, h, base, h_out,     \
                                            make_add<T>(ADD_NAMES), rows, next, (T*)a, lda, save, row_pos, row_seq, cu_q, seq_slot, \
                                            H, vec))
#define ADD_LAUNCH(NV, MAXT)                                                                                                         \
    if (nv <= NV && threads <= MAXT) {                                                                  \
        if (two) ADD_GO(NV, true, MAXT);                                                                                             \
        ADD_GO(NV, false, MAXT);                                                                                                     \
    }
    ADD_LAUNCH(1, 1024) ADD_LAUNCH(2, 512) ADD_LAUNCH(3, 512) ADD_LAUNCH(4, 512) ADD_LAUNCH(4, 1024)
#undef ADD_LAUNCH
#undef ADD_GO
    return (int)cudaErrorInvalidValue;
}

DK_EXPORT int dk_sublayer_add_shift(int dtype, const float* h, float* h_out, ADD_PARAMS, const float* share, const float* state,
                                    const int* row_pos, const int* row_seq, const int* cu_q, const int* seq_slot, int n_rows,
                                    int run, void* a, int H, cudaStream_t st) {
    if (H < 1 || H > 16384 || run < 1 || h == h_out) return (int)cudaErrorInvalidValue;
    const int threads = stream_threads(H, n_rows), nv = ((H + 3) / 4 + threads - 1) / threads;
    const int vec = ADD_VEC && ((uintptr_t)share | (uintptr_t)state) % 16 == 0;
    const bool two = x1 != nullptr || parts1 != nullptr;
#define ADD_GO(NV, TWO, MAXT)                                                                                                       \
    STREAM_DISPATCH(dtype, return dk_launch(sublayer_add_shift_kernel<T, NV, TWO, MAXT>, dim3((n_rows + run - 1) / run),             \
                                            dim3(threads), 0, st, h, h_out, make_add<T>(ADD_NAMES), share, state, row_pos,     \
                                            row_seq, cu_q, seq_slot, n_rows, run, (T*)a, H, vec))
#define ADD_LAUNCH(NV, MAXT)                                                                                                         \
    if (nv <= NV && threads <= MAXT) {                                                                  \
        if (two) ADD_GO(NV, true, MAXT);                                                                                             \
        ADD_GO(NV, false, MAXT);                                                                                                     \
    }
    ADD_LAUNCH(1, 1024) ADD_LAUNCH(2, 512) ADD_LAUNCH(3, 512) ADD_LAUNCH(4, 512) ADD_LAUNCH(4, 1024)
#undef ADD_LAUNCH
#undef ADD_GO
    return (int)cudaErrorInvalidValue;
}

DK_EXPORT int dk_stream_save(const float* h, float* state, const int* cu_q, const int* seq_pos0, const int* seq_slot, int n_seq,
                             int H, cudaStream_t st) {
    return dk_launch(stream_save_kernel, dim3(n_seq), dim3(256), 0, st, h, state, cu_q, seq_pos0, seq_slot, H);
}

DK_EXPORT int dk_embed_bigram(int dtype, const int* tok, const void* embed, float scale, const void* table, int buckets,
                              long long mul_prev, long long mul_cur, int* state, const int* row_pos, const int* row_seq,
                              const int* cu_q, const int* seq_slot, int n_rows, int H, int V, float* h, cudaStream_t st) {
    if (buckets < 1) return (int)cudaErrorInvalidValue;
    STREAM_DISPATCH(dtype, return dk_launch(embed_bigram_kernel<T>, dim3(n_rows), dim3(H >= 512 ? 256 : 128), 0, st, tok,
                                            (const T*)embed, scale, (const T*)table, buckets, mul_prev, mul_cur, state, row_pos,
                                            row_seq, cu_q, seq_slot, H, V, h));
}
