// Matrix memory with exponential gates (the mLSTM of xLSTM): per (sequence, head) a state S [D, V], a key sum n [D] and a
// running maximum m, float32, all zero at a sequence's start (m too: not minus infinity). Per token, with the log gates
//     i = cap tanh((i_row + i_bias) / cap),   f = log sigmoid(cap tanh((f_row + f_bias) / cap)):
//     m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n <- exp(f + m - m') n + exp(i - m') k;
//     o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),
// and behind it each head's o over its root mean square, times a weight of all heads' size, times sigmoid of a gate.
// q, k, v, gate and the two gate rows are columns of one projection in the storage type; everything else is float32.
//
// Portions run in three kernels:
// (bfloat16 portions of suitable sizes go on to matrix_memory_bf16.cu behind the first of them):
//   * mm_gates: a block per (sequence, head). A token maps m to max(f + m, i); two such maps in a row are another one,
//     (f1 + f2, max(i1 + f2, i2)), so a warp's 32 running maxima come from five shuffles, and a block's from five more over its
//     warps' maps. Leaves per (token, head) what the
//     recurrence multiplies by: exp(f + m - m'), exp(i - m'), exp(-m').
//   * mm_portion: the recurrence over the portion, columns of S in registers, rows staged ahead by cp.async.
//   * mm_output: quotient, norm, weight, gate; a warp per (token, head).
// Single tokens run in one kernel (mm_step), a block per (sequence, head), one pass over the state.
// Rows of sequence s are cu_q[s] .. cu_q[s + 1]. seq_pos0[s] < 0 marks a padding row: zeros out, state untouched.
#include "common.cuh"
#include <type_traits>

#define MM_NT 16          // tokens a stage
#define MM_SMALL 1e-6f

__device__ __forceinline__ float mm_cap(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float mm_log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// ------------------------------------------------------------------------------------------------ gates of a portion
// scal [tokens, heads, 4] = (exp(f + m - m'), exp(i - m'), exp(-m'), -); the last number is n . q, from mm_portion. With
// ``chunk`` (a multiple of 32, the block's threads a multiple of it) the first number is the sum of (f + m - m') log2(e) from the
// first token of the token's chunk on.
struct MaxMap {          // m -> max(f + m, i)
    float f, i;
};
// the maps of the lanes up to this one, in order
__device__ __forceinline__ MaxMap warp_maps(MaxMap a, int lane) {
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
        const float f1 = __shfl_up_sync(0xffffffffu, a.f, d), i1 = __shfl_up_sync(0xffffffffu, a.i, d);
        if (lane >= d) {
            a.i = fmaxf(i1 + a.f, a.i);
            a.f += f1;
        }
    }
    return a;
}

template <typename T>
__global__ void __launch_bounds__(1024)
mm_gates_kernel(const T* irow, const T* frow, long long ld, const float* __restrict__ ibias, const float* __restrict__ fbias, float cap,
                float4* scal, float* m_state, const int* cu_q, const int* seq_pos0, const int* seq_slot, int nh, int chunk) {
    __shared__ MaxMap maps[32];
    __shared__ float sums[32], m_next;
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
    const int s = blockIdx.x, h = blockIdx.y;
    if (seq_pos0[s] < 0) return;
    const int r0 = cu_q[s], r1 = cu_q[s + 1];
    float* mp = m_state + (size_t)seq_slot[s] * nh + h;
    float m = *mp;
    const float ib = ibias[h], fb = fbias[h];
    float iz = 0.f, fz = 0.f;
    auto fetch = [&](int t) {
        if (t < r1) {
            iz = to_f(irow[(size_t)t * ld + h]);
            fz = to_f(frow[(size_t)t * ld + h]);
        }
    };
    fetch(r0 + tid);
    for (int t0 = r0; t0 < r1; t0 += blockDim.x) {
        const bool on = t0 + tid < r1;
        // past the end: the map that leaves m alone
        const float i = on ? mm_cap(iz + ib, cap) : -INFINITY;
        const float f = on ? mm_log_sigmoid(mm_cap(fz + fb, cap)) : 0.f;
        fetch(t0 + blockDim.x + tid);
        const MaxMap a = warp_maps({f, i}, lane);
        if (lane == 31) maps[warp] = a;
        __syncthreads();
        if (warp == 0) {
            const MaxMap all = warp_maps(lane < n_warps ? maps[lane] : MaxMap{0.f, -INFINITY}, lane);
            maps[lane] = all;
        }
        __syncthreads();
        const float ahead = warp == 0 ? m : fmaxf(maps[warp - 1].f + m, maps[warp - 1].i);        // the maximum ahead of this warp
        const float mt = fmaxf(a.f + ahead, a.i);
        float before = __shfl_up_sync(0xffffffffu, mt, 1);
        if (lane == 0) before = ahead;
        float keep = f + before - mt;
        if (chunk) {
            keep *= 1.4426950408889634f;
#pragma unroll
            for (int d = 1; d < 32; d <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, keep, d);
                if (lane >= d) keep += x;
            }
            if (lane == 31) sums[warp] = keep;
            __syncthreads();
            for (int w = warp / (chunk / 32) * (chunk / 32); w < warp; w++) keep += sums[w];
        } else {
            keep = expf(keep);
        }
        if (on) scal[(size_t)(t0 + tid) * nh + h] = make_float4(keep, expf(i - mt), expf(-mt), 0.f);
        if (tid == (int)blockDim.x - 1) m_next = mt;
        __syncthreads();              // also: maps and sums may be written again
        m = m_next;
    }
    if (tid == 0) *mp = m;
}

// --------------------------------------------------------------------------------------------- recurrence of a portion
__device__ __forceinline__ void mm_cp16(void* smem, const void* gmem) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(gmem) : "memory");
}
template <int N> __device__ __forceinline__ void mm_ld(const float* p, float (&f)[N]) {
    if (N % 4 == 0) {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(p + i);
            f[i % N] = v.x, f[(i + 1) % N] = v.y, f[(i + 2) % N] = v.z, f[(i + 3) % N] = v.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; i++) f[i] = p[i];
    }
}
template <int N> __device__ __forceinline__ void mm_ld(const bf16* p, float (&f)[N]) {
    if (N == 8) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float2 x = __bfloat1622float2(h[i]);
            f[(2 * i) % N] = x.x, f[(2 * i + 1) % N] = x.y;
        }
    } else if (N == 4) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float2 x = __bfloat1622float2(h[i]);
            f[(2 * i) % N] = x.x, f[(2 * i + 1) % N] = x.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; i++) f[i] = __bfloat162float(p[i]);
    }
}
// the VC column sums over the 32 lanes: halves are exchanged while more than one value is left, then plain sums; lane l ends
// with the sum of the column that its top log2(VC) bits spell
template <int VC> __device__ __forceinline__ float mm_fold(const float (&o)[VC], int lane) {
    float r[VC];
#pragma unroll
    for (int c = 0; c < VC; c++) r[c] = o[c];
    int bit = 16;
#pragma unroll
    for (int n = VC / 2; n >= 1; n >>= 1, bit >>= 1) {
        const bool up = lane & bit;
#pragma unroll
        for (int c = 0; c < n; c++) {
            const float mine = up ? r[n + c] : r[c], other = up ? r[c] : r[n + c];
            r[c] = mine + __shfl_xor_sync(0xffffffffu, other, bit);
        }
    }
    float x = r[0];
#pragma unroll
    for (; bit >= 1; bit >>= 1) x += __shfl_xor_sync(0xffffffffu, x, bit);
    return x;
}

// Block (sequence, head, BC value columns); a warp takes VC of them, lane l the state's rows DPL l .. DPL l + DPL - 1. The
// block of the first columns has one warp more, for n: a column whose value is one. Rows of MM_NT tokens a stage: q [D], k [D],
// (exp, exp) and the block's value columns, padded with zeros to 32 DPL rows and BC columns. vec: rows and heads lie on 16-byte
// boundaries and come by cp.async, n_stages - 1 stages ahead; otherwise element by element.
template <typename T, int DPL, int VC>
__global__ void __launch_bounds__(32 * (32 / VC + 1))
mm_portion_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld, float4* scal,
                  float* __restrict__ out, float* state, float* n_state, const int* cu_q, const int* seq_pos0, const int* seq_slot,
                  int nh, int hd, int hdv, float q_scale, int BC, int n_stages, int vec) {
    constexpr int HDK = 32 * DPL;
    constexpr int QB = MM_NT * HDK * (int)sizeof(T), SB = MM_NT * 8, VB = MM_NT * 32 * (int)sizeof(T);
    constexpr int STAGE = 2 * QB + SB + VB;
    constexpr int WRITERS = 32 / VC;
    extern __shared__ __align__(16) unsigned char mm_smem[];
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, threads = blockDim.x;
    const int s = blockIdx.x, h = blockIdx.y;
    const int col0 = blockIdx.z * BC, cols_here = min(BC, hdv - col0);
    const bool is_n = warp == BC / VC;
    const int c0 = is_n ? 0 : col0 + warp * VC;
    const bool active = is_n ? blockIdx.z == 0 : c0 < hdv;
    const int r0 = cu_q[s], r1 = cu_q[s + 1];
    const size_t ow = (size_t)nh * hdv;
    const int my_col = lane / WRITERS;
    if (seq_pos0[s] < 0) {
        if (active && !is_n && lane % WRITERS == 0 && c0 + my_col < hdv)
            for (int t = r0; t < r1; t++) out[(size_t)t * ow + (size_t)h * hdv + c0 + my_col] = 0.f;
        return;
    }
    const size_t sh = (size_t)seq_slot[s] * nh + h;
    float* S = is_n ? n_state + sh * hd : state + sh * hd * hdv + c0;
    const int pitch = is_n ? 1 : hdv, cols = active ? (is_n ? 1 : min(VC, hdv - c0)) : 0;
    float st[DPL][VC];
#pragma unroll
    for (int i = 0; i < DPL; i++)
#pragma unroll
        for (int c = 0; c < VC; c++) st[i][c] = c < cols && DPL * lane + i < hd ? S[(size_t)(DPL * lane + i) * pitch + c] : 0.f;
    // rows past the head and columns past the values stay zero in every stage
    for (int i = tid; i < n_stages * STAGE / 16; i += threads) reinterpret_cast<uint4*>(mm_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int n_chunks = (r1 - r0 + MM_NT - 1) / MM_NT;
    const int QP = hd * (int)sizeof(T) / 16, VP = cols_here * (int)sizeof(T) / 16;         // 16-byte pieces a token
    auto issue = [&](int c) {
        if (c < n_chunks) {
            unsigned char* base = mm_smem + (c % n_stages) * STAGE;
            T* sq = reinterpret_cast<T*>(base);
            T* sk = reinterpret_cast<T*>(base + QB);
            float2* ss = reinterpret_cast<float2*>(base + 2 * QB);
            T* sv = reinterpret_cast<T*>(base + 2 * QB + SB);
            const int t0 = r0 + c * MM_NT, nt = min(MM_NT, r1 - t0);
            if (vec) {
                for (int i = tid; i < nt * QP; i += threads) {
                    const int tt = i / QP, pc = i % QP * (16 / (int)sizeof(T));
                    const size_t src = (size_t)(t0 + tt) * ld + (size_t)h * hd + pc;
                    mm_cp16(sq + tt * HDK + pc, q + src);
                    mm_cp16(sk + tt * HDK + pc, k + src);
                }
                for (int i = tid; i < nt * VP; i += threads) {
                    const int tt = i / VP, pc = i % VP * (16 / (int)sizeof(T));
                    mm_cp16(sv + tt * 32 + pc, v + (size_t)(t0 + tt) * ld + (size_t)h * hdv + col0 + pc);
                }
            } else {
                for (int i = tid; i < nt * hd; i += threads) {
                    const int tt = i / hd, d = i % hd;
                    const size_t src = (size_t)(t0 + tt) * ld + (size_t)h * hd + d;
                    sq[tt * HDK + d] = q[src];
                    sk[tt * HDK + d] = k[src];
                }
                for (int i = tid; i < nt * cols_here; i += threads)
                    sv[i / cols_here * 32 + i % cols_here] = v[(size_t)(t0 + i / cols_here) * ld + (size_t)h * hdv + col0 + i % cols_here];
            }
            for (int i = tid; i < nt; i += threads) {
                const uint32_t a = (uint32_t)__cvta_generic_to_shared(ss + i);
                asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(a), "l"(scal + (size_t)(t0 + i) * nh + h) : "memory");
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int c = 0; c < n_stages - 1; c++) issue(c);
    for (int c = 0; c < n_chunks; c++) {
        issue(c + n_stages - 1);
        if (n_stages == 4) asm volatile("cp.async.wait_group 3;" ::: "memory");
        else if (n_stages == 3) asm volatile("cp.async.wait_group 2;" ::: "memory");
        else asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const unsigned char* base = mm_smem + (c % n_stages) * STAGE;
        const T* sq = reinterpret_cast<const T*>(base);
        const T* sk = reinterpret_cast<const T*>(base + QB);
        const float2* ss = reinterpret_cast<const float2*>(base + 2 * QB);
        const T* sv = reinterpret_cast<const T*>(base + 2 * QB + SB);
        const int t0 = r0 + c * MM_NT, nt = min(MM_NT, r1 - t0);
        if (active) {
            // U tokens a turn: their state updates follow one another, their folds are independent chains of shuffles
            constexpr int U = DPL * VC <= 16 ? 4 : 2;
            auto turn = [&](int tt0, auto tail_c) {
                constexpr bool TAIL = decltype(tail_c)::value;    // the stage's last turn may hold fewer than U tokens
                float o[U][VC];
#pragma unroll
                for (int u = 0; u < U; u++) {
                    const int tt = TAIL ? min(tt0 + u, nt - 1) : tt0 + u;   // past the end: the last token again, its result unused
                    float qv[DPL], kv[DPL], vv[VC];
                    mm_ld<DPL>(sq + tt * HDK + DPL * lane, qv);
                    mm_ld<DPL>(sk + tt * HDK + DPL * lane, kv);
                    const float2 g = ss[tt];
                    if (is_n) {
#pragma unroll
                        for (int cc = 0; cc < VC; cc++) vv[cc] = cc == 0 ? 1.f : 0.f;
                    } else {
                        mm_ld<VC>(sv + tt * 32 + warp * VC, vv);
                    }
                    const bool live = !TAIL || tt0 + u < nt;
#pragma unroll
                    for (int cc = 0; cc < VC; cc++) o[u][cc] = 0.f;
#pragma unroll
                    for (int i = 0; i < DPL; i++) {
                        const float qs = qv[i] * q_scale, kw = kv[i] * g.y;
#pragma unroll
                        for (int cc = 0; cc < VC; cc++) {
                            const float nx = fmaf(g.x, st[i][cc], kw * vv[cc]);
                            st[i][cc] = live ? nx : st[i][cc];
                            o[u][cc] = fmaf(nx, qs, o[u][cc]);
                        }
                    }
                }
                float r[U];
#pragma unroll
                for (int u = 0; u < U; u++) r[u] = mm_fold<VC>(o[u], lane);
#pragma unroll
                for (int u = 0; u < U; u++) {
                    if (TAIL && tt0 + u >= nt) continue;
                    const size_t t = (size_t)(t0 + tt0 + u);
                    if (is_n) {
                        if (lane == 0) scal[t * nh + h].w = r[u];
                    } else if (lane % WRITERS == 0 && c0 + my_col < hdv) {
                        out[t * ow + (size_t)h * hdv + c0 + my_col] = r[u];
                    }
                }
            };
            int tt0 = 0;
            for (; tt0 + U <= nt; tt0 += U) turn(tt0, std::false_type{});
            if (tt0 < nt) turn(tt0, std::true_type{});
        }
        __syncthreads();              // the stage is free for a later chunk
    }
#pragma unroll
    for (int i = 0; i < DPL; i++)
#pragma unroll
        for (int c = 0; c < VC; c++)
            if (c < cols && DPL * lane + i < hd) S[(size_t)(DPL * lane + i) * pitch + c] = st[i][c];
}

// ------------------------------------------------------------------------------------------------ output of a portion
// out[t, h] = rms(o / (max(|n . q|, exp(-m)) + 1e-6)) * w * sigmoid(gate) * out_scale; a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256)
mm_output_kernel(const float* __restrict__ o, const float4* __restrict__ scal, const float* __restrict__ w, float eps, const T* gate, long long ldg,
                 float out_scale, T* out, long long ldo, const int* row_pos, int n_tok, int nh, int hdv) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= (long long)n_tok * nh) return;
    const size_t t = (size_t)(item / nh);
    const int h = (int)(item % nh);
    const size_t at = t * nh * hdv + (size_t)h * hdv;
    T* dst = out + t * ldo + (size_t)h * hdv;
    if (row_pos[t] < 0) {
        for (int c = lane; c < hdv; c += 32) dst[c] = from_f<T>(0.f);
        return;
    }
    const float4 g = scal[t * nh + h];
    const float inv = 1.f / (fmaxf(fabsf(g.w), g.z) + MM_SMALL);
    float ss = 0.f;
    for (int c = lane; c < hdv; c += 32) {
        const float y = o[at + c] * inv;
        ss += y * y;
    }
    const float rs = inv * (out_scale / sqrtf(warp_sum(ss) / (float)hdv + eps));
    for (int c = lane; c < hdv; c += 32) {
        const float z = to_f(gate[t * ldg + (size_t)h * hdv + c]);
        dst[c] = from_f<T>(o[at + c] * rs * w[(size_t)h * hdv + c] / (1.f + expf(-z)));
    }
}

// -------------------------------------------------------------------------------------------------------- single tokens
// Block (row, head): gates, one pass over the state, quotient, norm, weight and gate. Thread (rg, cg): columns N cg .. N cg +
// N - 1 of the rows rg, rg + R, .. (N = 4: 16 bytes a row). Columns beyond 256 threads' worth come in further turns.
template <typename T, int N>
__global__ void __launch_bounds__(256)
mm_step_kernel(const T* q, const T* k, const T* v, const T* gate, const T* irow, const T* frow, long long ld,
               const float* __restrict__ ibias, const float* __restrict__ fbias, float cap, float* state, float* n_state, float* m_state,
               const float* __restrict__ w, float eps, float out_scale, T* out, long long ldo, const int* seq_pos0, const int* seq_slot,
               int nh, int hd, int hdv, float q_scale, int cg_pad) {
    extern __shared__ __align__(16) float mms[];
    __shared__ float red[33];
    float* sq = mms;                       // [hd]
    float* sk = sq + (hd + 3) / 4 * 4;     // [hd], times exp(i - m')
    float* so = sk + (hd + 3) / 4 * 4;     // [hdv]
    float* part = so + (hdv + 3) / 4 * 4;  // [256 * N]
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, s = blockIdx.x, h = blockIdx.y;
    T* dst = out + (size_t)s * ldo + (size_t)h * hdv;
    if (seq_pos0[s] < 0) {
        for (int c = tid; c < hdv; c += 256) dst[c] = from_f<T>(0.f);
        return;
    }
    const size_t sh = (size_t)seq_slot[s] * nh + h, row = (size_t)s * ld;
    const float m = m_state[sh];
    const float i = mm_cap(to_f(irow[row + h]) + ibias[h], cap);
    const float f = mm_log_sigmoid(mm_cap(to_f(frow[row + h]) + fbias[h], cap));
    const float mt = fmaxf(f + m, i);
    const float keep = expf(f + m - mt), write = expf(i - mt);
    float dot = 0.f;
    for (int d = tid; d < hd; d += 256) {
        const float qd = to_f(q[row + (size_t)h * hd + d]) * q_scale, kd = to_f(k[row + (size_t)h * hd + d]) * write;
        sq[d] = qd;
        sk[d] = kd;
        const float nd = fmaf(keep, n_state[sh * hd + d], kd);
        n_state[sh * hd + d] = nd;
        dot = fmaf(nd, qd, dot);
    }
    const float den = fmaxf(fabsf(block_sum(dot, red)), expf(-mt)) + MM_SMALL;      // a barrier: everybody has read m, q and k
    if (tid == 0) m_state[sh] = mt;
    const int cgs = (hdv + N - 1) / N, R = 256 / cg_pad, rg = tid / cg_pad;
    float* S = state + sh * hd * hdv;
    for (int cb = 0; cb < cgs; cb += cg_pad) {
        const int c0 = (cb + tid % cg_pad) * N;
        float acc[N];
#pragma unroll
        for (int c = 0; c < N; c++) acc[c] = 0.f;
        if (c0 < hdv) {
            float vv[N];
#pragma unroll
            for (int c = 0; c < N; c++) vv[c] = to_f(v[row + (size_t)h * hdv + c0 + c]);
#pragma unroll 8
            for (int d = rg; d < hd; d += R) {
                float x[N];
                float* p = S + (size_t)d * hdv + c0;
                if (N == 4) {
                    const float4 y = *reinterpret_cast<const float4*>(p);
                    x[0] = y.x, x[1 % N] = y.y, x[2 % N] = y.z, x[3 % N] = y.w;
                } else {
                    x[0] = *p;
                }
#pragma unroll
                for (int c = 0; c < N; c++) {
                    x[c] = fmaf(keep, x[c], sk[d] * vv[c]);
                    acc[c] = fmaf(x[c], sq[d], acc[c]);
                }
                if (N == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1 % N], x[2 % N], x[3 % N]);
                else *p = x[0];
            }
        }
#pragma unroll
        for (int c = 0; c < N; c++) part[tid * N + c] = acc[c];
        __syncthreads();
        for (int c = tid; c < cg_pad * N; c += 256) {
            float o = 0.f;
            for (int g = 0; g < R; g++) o += part[g * cg_pad * N + c];
            if (cb * N + c < hdv) so[cb * N + c] = o / den;
        }
        __syncthreads();
    }
    float ss = 0.f;
    for (int c = tid; c < hdv; c += 256) ss += so[c] * so[c];
    const float rs = out_scale / sqrtf(block_sum(ss, red) / (float)hdv + eps);
    for (int c = tid; c < hdv; c += 256) {
        const float z = to_f(gate[row + (size_t)h * hdv + c]);
        dst[c] = from_f<T>(so[c] * rs * w[(size_t)h * hdv + c] / (1.f + expf(-z)));
    }
}

DK_EXPORT int dk_mm_gates(int dtype, const void* irow, const void* frow, long long ld, const float* ibias, const float* fbias, float cap,
                          void* scal, float* m_state, const int* cu_q, const int* seq_pos0, const int* seq_slot, int n_seq, int nh,
                          int chunk, long long n_rows, cudaStream_t st) {
    if (chunk < 0 || chunk % 32 || (chunk && 256 % chunk)) return (int)cudaErrorInvalidValue;
    const dim3 grid(n_seq, nh), block(n_rows > 256LL * n_seq ? 1024 : 256);
    if (dtype == 0)
        return dk_launch(mm_gates_kernel<float>, grid, block, 0, st, (const float*)irow, (const float*)frow, ld, ibias, fbias, cap, (float4*)scal,
                         m_state, cu_q, seq_pos0, seq_slot, nh, chunk);
    return dk_launch(mm_gates_kernel<bf16>, grid, block, 0, st, (const bf16*)irow, (const bf16*)frow, ld, ibias, fbias, cap, (float4*)scal, m_state,
                     cu_q, seq_pos0, seq_slot, nh, chunk);
}

template <typename T>
static int launch_portion(const void* q, const void* k, const void* v, long long ld, void* scal, float* out, float* state, float* n_state,
                          const int* cu_q, const int* seq_pos0, const int* seq_slot, float q_scale, int n_seq, int nh, int hd, int hdv,
                          cudaStream_t st) {
    const int esz = (int)sizeof(T);
    const int vec = ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) % 16 == 0 && (ld * esz) % 16 == 0 && (hd * esz) % 16 == 0 && (hdv * esz) % 16 == 0;
    int sms = 0, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    // columns a warp and a block: coarse when the sequences and heads alone fill the schedulers, finer when not
    const long long blocks32 = (long long)n_seq * nh * ((hdv + 31) / 32), scheds = 4LL * sms;
    int VC = 8, BC = 32;
    if (blocks32 * 4 < 3 * scheds) VC = 4;
    if (blocks32 * 8 < 3 * scheds) { VC = 2; if (blocks32 < sms) BC = 16; }
    const dim3 grid(n_seq, nh, (hdv + BC - 1) / BC), block(32 * (BC / VC + 1));
#define MM_GO(D, V)                                                                                                            \
    if (hd <= 32 * D && VC == V) {                                                                                             \
        const size_t stage = (2 * MM_NT * 32 * D + MM_NT * 32) * sizeof(T) + MM_NT * 8;                                        \
        const int n_stages = stage * 4 <= 160 * 1024 ? 4 : (stage * 3 <= 160 * 1024 ? 3 : 2);                                  \
        const size_t smem = n_stages * stage;                                                                                  \
        if (smem > 48 * 1024)                                                                                                  \
            cudaFuncSetAttribute(mm_portion_kernel<T, D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
        return dk_launch(mm_portion_kernel<T, D, V>, grid, block, smem, st, (const T*)q, (const T*)k, (const T*)v, ld,         \
                         (float4*)scal, out, state, n_state, cu_q, seq_pos0, seq_slot, nh, hd, hdv, q_scale, BC, n_stages, vec); \
    }
    MM_GO(1, 8) MM_GO(2, 8) MM_GO(4, 8) MM_GO(8, 8)
    MM_GO(1, 4) MM_GO(2, 4) MM_GO(4, 4) MM_GO(8, 4)
    MM_GO(1, 2) MM_GO(2, 2) MM_GO(4, 2) MM_GO(8, 2)
#undef MM_GO
    return (int)cudaErrorInvalidValue;
}

DK_EXPORT int dk_mm_portion(int dtype, const void* q, const void* k, const void* v, long long ld, void* scal, float* out, float* state,
                            float* n_state, const int* cu_q, const int* seq_pos0, const int* seq_slot, float q_scale, int n_seq, int nh,
                            int hd, int hdv, cudaStream_t st) {
    if (hd < 1 || hd > 256 || hdv < 1) return (int)cudaErrorInvalidValue;
    if (dtype == 0)
        return launch_portion<float>(q, k, v, ld, scal, out, state, n_state, cu_q, seq_pos0, seq_slot, q_scale, n_seq, nh, hd, hdv, st);
    return launch_portion<bf16>(q, k, v, ld, scal, out, state, n_state, cu_q, seq_pos0, seq_slot, q_scale, n_seq, nh, hd, hdv, st);
}

DK_EXPORT int dk_mm_output(int dtype, const float* o, const void* scal, const float* w, float eps, const void* gate, long long ldg,
                           float out_scale, void* out, long long ldo, const int* row_pos, int n_tok, int nh, int hdv, cudaStream_t st) {
    const dim3 grid((unsigned)(((long long)n_tok * nh + 7) / 8)), block(256);
    if (dtype == 0)
        return dk_launch(mm_output_kernel<float>, grid, block, 0, st, o, (const float4*)scal, w, eps, (const float*)gate, ldg, out_scale,
                         (float*)out, ldo, row_pos, n_tok, nh, hdv);
    return dk_launch(mm_output_kernel<bf16>, grid, block, 0, st, o, (const float4*)scal, w, eps, (const bf16*)gate, ldg, out_scale, (bf16*)out,
                     ldo, row_pos, n_tok, nh, hdv);
}

template <typename T>
static int launch_mm_step(const void* q, const void* k, const void* v, const void* gate, const void* irow, const void* frow, long long ld,
                          const float* ibias, const float* fbias, float cap, float* state, float* n_state, float* m_state, const float* w,
                          float eps, float out_scale, void* out, long long ldo, const int* seq_pos0, const int* seq_slot, float q_scale,
                          int n_rows, int nh, int hd, int hdv, cudaStream_t st) {
    const int N = hdv % 4 == 0 && (uintptr_t)state % 16 == 0 ? 4 : 1;
    const int cgs = (hdv + N - 1) / N;
    int cg_pad = 1;
    while (cg_pad < cgs && cg_pad < 256) cg_pad <<= 1;
    const size_t smem = sizeof(float) * (size_t)(2 * ((hd + 3) / 4 * 4) + (hdv + 3) / 4 * 4 + 256 * N);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(n_rows, nh), block(256);
#define MM_STEP(NN)                                                                                                              \
    return dk_launch(mm_step_kernel<T, NN>, grid, block, smem, st, (const T*)q, (const T*)k, (const T*)v, (const T*)gate, (const T*)irow, \
                     (const T*)frow, ld, ibias, fbias, cap, state, n_state, m_state, w, eps, out_scale, (T*)out, ldo, seq_pos0,  \
                     seq_slot, nh, hd, hdv, q_scale, cg_pad)
    if (N == 4) MM_STEP(4);
    MM_STEP(1);
#undef MM_STEP
}

DK_EXPORT int dk_mm_step(int dtype, const void* q, const void* k, const void* v, const void* gate, const void* irow, const void* frow,
                         long long ld, const float* ibias, const float* fbias, float cap, float* state, float* n_state, float* m_state,
                         const float* w, float eps, float out_scale, void* out, long long ldo, const int* seq_pos0, const int* seq_slot,
                         float q_scale, int n_rows, int nh, int hd, int hdv, cudaStream_t st) {
    if (hd < 1 || hd > 256 || hdv < 1 || hdv > 4096) return (int)cudaErrorInvalidValue;
    if (dtype == 0)
        return launch_mm_step<float>(q, k, v, gate, irow, frow, ld, ibias, fbias, cap, state, n_state, m_state, w, eps, out_scale, out, ldo,
                                     seq_pos0, seq_slot, q_scale, n_rows, nh, hd, hdv, st);
    return launch_mm_step<bf16>(q, k, v, gate, irow, frow, ld, ibias, fbias, cap, state, n_state, m_state, w, eps, out_scale, out, ldo,
                                seq_pos0, seq_slot, q_scale, n_rows, nh, hd, hdv, st);
}
