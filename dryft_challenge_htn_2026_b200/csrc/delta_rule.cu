// The gated delta rule over a float32 state per (sequence, head), S [D, V]:
//     S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
// with unit keys and queries shared by the heads of a group, one decay g and one step size beta per head and token.
//   * delta_prepare  : what enters the recurrence, in float32, from the projection's rows: a causal convolution per channel
//                      of q, k and v (its memory, the last taps - 1 projected rows, is a per-sequence state, read only
//                      here), SiLU; q and k over sqrt(sum of squares + unit_eps) per head, q times D^(-1/2); g = exp(-exp(A)
//                      softplus(a + dt)), beta = sigmoid(b); and k . q per key head (below).
//   * delta_rule     : portions, four tokens a turn. Eight lanes share a column of the state, its rows dealt
//                      out over their registers for the whole portion; the rows q, k, v of 16 tokens at a time come through shared memory by
//                      cp.async, three chunks in turn.
//   * delta_rule_step: one token a sequence: a block per (sequence, head, 32 columns) passes once over its part of the state:
//                      with a = S^T k and b = S^T q of the state as the token finds it, u = beta (v - g a), o = g b + (k . q) u.
// Rows with position < 0 are padding: zeros out, states untouched.
#include "common.cuh"

#define DP_THREADS 256
#define DR_NT 16            // tokens a staged chunk
#define DR_STAGES 3
#define DR_COLS 16          // columns of a state a block takes

__device__ __forceinline__ float dr_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T> __device__ __forceinline__ void dr_ld4(const T* p, float (&y)[4]);
template <> __device__ __forceinline__ void dr_ld4<float>(const float* p, float (&y)[4]) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    y[0] = x.x, y[1] = x.y, y[2] = x.z, y[3] = x.w;
}
template <> __device__ __forceinline__ void dr_ld4<bf16>(const bf16* p, float (&y)[4]) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    y[0] = a.x, y[1] = a.y, y[2] = b.x, y[3] = b.y;
}

// A block per token. proj rows [q (G D) | k (G D) | v (H V)]; a_rows, b_rows: columns [H] of the same matrix (row stride ld).
// qkv [rows, 2 G D + H V] float32 out; scal [rows, 2 H + G] float32 out: g, beta, k . q.
template <typename T>
__global__ void __launch_bounds__(DP_THREADS)
delta_prepare_kernel(const T* proj, long long ld, const T* a_rows, const T* b_rows, const T* state, const T* __restrict__ wconv,
                     int taps, const float* __restrict__ a_log, const float* __restrict__ dt_bias, float unit_eps, const int* row_pos,
                     const int* row_seq, const int* seq_pos0, const int* seq_slot, float* qkv, float* scal, int H, int G, int D, int V,
                     int vec) {
    extern __shared__ __align__(16) float row[];         // [C] after convolution and SiLU
    pdl_wait();
    pdl_launch_dependents();
    const int nqk = G * D, C = 2 * nqk + H * V, t = blockIdx.x, tid = threadIdx.x;
    float* out = qkv + (size_t)t * C;
    float* sc = scal + (size_t)t * (2 * H + G);
    const int pos = row_pos[t];
    if (pos < 0) {
        for (int c = tid; c < C; c += DP_THREADS) out[c] = 0.f;
        for (int c = tid; c < 2 * H + G; c += DP_THREADS) sc[c] = 0.f;
        return;
    }
    const int s = row_seq[t], p0 = seq_pos0[s];
    const T* st = taps > 1 ? state + (size_t)seq_slot[s] * (taps - 1) * C : nullptr;
    if (vec) {
        for (int c = 4 * tid; c < C; c += 4 * DP_THREADS) {
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
            float w[4][4];
            if (taps == 4) {
#pragma unroll
                for (int e = 0; e < 4; e++) dr_ld4<T>(wconv + (size_t)(c + e) * 4, w[e]);
            }
            auto tap = [&](int j, float w0, float w1, float w2, float w3) {
                const int back = taps - 1 - j, pp = pos - back;
                float u[4];
                dr_ld4<T>(pp >= p0 ? proj + (size_t)(t - back) * ld + c : st + (size_t)(taps - 1 - (p0 - pp)) * C + c, u);
                acc[0] = fmaf(w0, u[0], acc[0]), acc[1] = fmaf(w1, u[1], acc[1]);
                acc[2] = fmaf(w2, u[2], acc[2]), acc[3] = fmaf(w3, u[3], acc[3]);
            };
            if (taps == 4) {
#pragma unroll
                for (int j = 0; j < 4; j++) tap(j, w[0][j], w[1][j], w[2][j], w[3][j]);
            } else {
                const T* wc = wconv + (size_t)c * taps;
                for (int j = 0; j < taps; j++) tap(j, to_f(wc[j]), to_f(wc[taps + j]), to_f(wc[2 * taps + j]), to_f(wc[3 * taps + j]));
            }
            float y[4];
#pragma unroll
            for (int e = 0; e < 4; e++) y[e] = acc[e] * dr_sigmoid(acc[e]);
            if (c < 2 * nqk) *reinterpret_cast<float4*>(row + c) = make_float4(y[0], y[1], y[2], y[3]);
            else *reinterpret_cast<float4*>(out + c) = make_float4(y[0], y[1], y[2], y[3]);
        }
    } else {
        for (int c = tid; c < C; c += DP_THREADS) {
            float acc = 0.f;
            for (int j = 0; j < taps; j++) {
                const int back = taps - 1 - j, pp = pos - back;
                const float u = to_f(pp >= p0 ? proj[(size_t)(t - back) * ld + c] : st[(size_t)(taps - 1 - (p0 - pp)) * C + c]);
                acc = fmaf(to_f(wconv[(size_t)c * taps + j]), u, acc);
            }
            const float y = acc * dr_sigmoid(acc);
            if (c < 2 * nqk) row[c] = y;
            else out[c] = y;
        }
    }
    for (int h = tid; h < H; h += DP_THREADS) {
        const float z = to_f(a_rows[(size_t)t * ld + h]) + dt_bias[h];
        const float dt = z > 20.f ? z : log1pf(expf(z));
        sc[h] = expf(-expf(a_log[h]) * dt);
        sc[H + h] = dr_sigmoid(to_f(b_rows[(size_t)t * ld + h]));
    }
    __syncthreads();
    const int lane = tid & 31, warp = tid >> 5;
    const float qs = 1.f / sqrtf((float)D);
    for (int g = warp; g < G; g += DP_THREADS / 32) {
        const float *q = row + g * D, *k = row + nqk + g * D;
        float sq = 0.f, sk = 0.f, kq = 0.f;
        for (int d = lane; d < D; d += 32) sq += q[d] * q[d], sk += k[d] * k[d];
        const float rq = qs / sqrtf(warp_sum(sq) + unit_eps), rk = 1.f / sqrtf(warp_sum(sk) + unit_eps);
        for (int d = lane; d < D; d += 32) {
            const float a = q[d] * rq, b = k[d] * rk;
            out[g * D + d] = a;
            out[nqk + g * D + d] = b;
            kq = fmaf(a, b, kq);
        }
        kq = warp_sum(kq);
        if (lane == 0) sc[2 * H + g] = kq;
    }
}

// two float32 multiply-adds an instruction (the halves of 64-bit registers), and their packing
__device__ __forceinline__ uint64_t dr_fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t dr_mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t dr_pack2(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 dr_unpack2(uint64_t x) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(x));
    return d;
}

__device__ __forceinline__ void dr_cp(float* smem, const float* gmem, bool wide) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
    if (wide) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(gmem) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(a), "l"(gmem) : "memory");
}

// The 16 sums a turn of four tokens needs over the lanes of a warp: halves are exchanged while more than one value is left,
// then a plain sum; lane l ends with the sum of value l / 2.
__device__ __forceinline__ float dr_fold16(float (&d)[16], int lane) {
#pragma unroll
    for (int n = 8; n >= 1; n >>= 1) {
        const bool up = lane & (2 * n);
#pragma unroll
        for (int i = 0; i < n; i++) {
            const float send = up ? d[i] : d[i + n], keep = up ? d[i + n] : d[i];
            d[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2 * n);
        }
    }
    return d[0] + __shfl_xor_sync(0xffffffffu, d[0], 1);
}

// grid (sequences, heads, ceil(V / 16)). LPC (8) lanes share a column of the state; lane i of them holds the RPL rows
// 4 i + 4 LPC j + (0 .. 3), D <= LPC RPL. Four tokens a turn: with S the state the turn finds, G_j = g_0 ..
// g_j and R_ji = g_(i+1) .. g_j (products, so that a vanishing decay is no division),
//     u_j = beta_j (v_j - G_j S^T k_j - sum_(i<j) R_ji (k_i . k_j) u_i),   o_j = G_j S^T q_j + sum_(i<=j) R_ji (k_i . q_j) u_i,
//     S <- G_3 S + sum_i R_3i k_i u_i,
// which is the token-by-token recurrence written out: the eight sums over the state's rows are taken side by side. The factors
// R_ji (k_i . k_j) and R_ji (k_i . q_j) do not depend on the column: each warp makes those of one turn of a staged chunk.
#define DR_COEF 28          // floats a turn: 6 of keys on keys, 10 of keys on queries, G, R_3, beta
template <int RPL, int LPC>
__global__ void __launch_bounds__(LPC * DR_COLS)
delta_rule_kernel(const float* qkv, const float* scal, float* out, float* state, const int* cu_q, const int* seq_pos0,
                  const int* seq_slot, int H, int G, int D, int V, int wide_qk, int wide_v) {
    constexpr int DP = LPC * RPL, NJ = RPL / 4, TURNS = DR_NT / 4, THREADS = LPC * DR_COLS;
    static_assert(TURNS <= THREADS / 32, "a warp makes the factors of one turn of a chunk");
    constexpr int STAGE = DR_NT * (2 * DP + DR_COLS + 2) + TURNS * DR_COEF;          // k, q, v columns, (g, beta), factors
    extern __shared__ __align__(16) float dr_smem[];
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DR_COLS, kh = h / (H / G);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, il = lane % LPC;
    const int col = col0 + tid / LPC;
    for (int i = tid; i < DR_STAGES * STAGE; i += THREADS) dr_smem[i] = 0.f;      // rows past D stay zero
    pdl_wait();
    pdl_launch_dependents();
    if (seq_pos0[s] < 0) return;
    const int r0 = cu_q[s], n_tok = cu_q[s + 1] - r0;
    const int C = 2 * G * D + H * V, nsc = 2 * H + G;
    const size_t ow = (size_t)H * V;
    __syncthreads();
    const int n_cols = min(DR_COLS, V - col0);
    auto fetch = [&](int c) {                     // chunk c into its stage
        float* base = dr_smem + (c % DR_STAGES) * STAGE;
        const int t0 = c * DR_NT, nt = min(DR_NT, n_tok - t0);
        const float* src = qkv + (size_t)(r0 + t0) * C + kh * D;
        constexpr int PER = DP / 4;
#pragma unroll
        for (int n = 0; n < (2 * DR_NT * PER + THREADS - 1) / THREADS; n++) {
            const int i = tid + n * THREADS;
            const int which = i / (DR_NT * PER), tt = i / PER % DR_NT, d = (i % PER) * 4;      // 0: k, 1: q
            if (which > 1 || tt >= nt || d >= D) continue;
            float* to = base + (which * DR_NT + tt) * DP + d;
            const float* from = src + (size_t)tt * C + (which ? 0 : G * D) + d;
            if (wide_qk) dr_cp(to, from, true);
            else
                for (int e = 0; e < min(4, D - d); e++) dr_cp(to + e, from + e, false);
        }
        if (tid < DR_NT * DR_COLS / 4) {
            const int tt = tid / (DR_COLS / 4), d = tid % (DR_COLS / 4) * 4;
            if (tt < nt && d < n_cols) {
                float* to = base + 2 * DR_NT * DP + tt * DR_COLS + d;
                const float* from = qkv + (size_t)(r0 + t0 + tt) * C + 2 * G * D + h * V + col0 + d;
                if (wide_v) dr_cp(to, from, true);
                else
                    for (int e = 0; e < min(4, n_cols - d); e++) dr_cp(to + e, from + e, false);
            }
        } else if (tid < DR_NT * DR_COLS / 4 + 2 * DR_NT) {
            const int i = tid - DR_NT * DR_COLS / 4, tt = i / 2, w = i % 2;
            float* to = base + DR_NT * (2 * DP + DR_COLS) + 2 * tt + w;
            if (tt < nt) dr_cp(to, scal + (size_t)(r0 + t0 + tt) * nsc + (w == 0 ? h : H + h), false);
            else *to = w == 0 ? 1.f : 0.f;         // tokens past the end: no decay and no step
        }
    };
    const int n_chunks = (n_tok + DR_NT - 1) / DR_NT;
#pragma unroll
    for (int c = 0; c < DR_STAGES - 1; c++) {
        if (c < n_chunks) fetch(c);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    const bool live = col < V;
    float* S = state + (((size_t)seq_slot[s] * H + h) * D) * V + col;
    uint64_t st[RPL / 2];                          // rows in pairs
#pragma unroll
    for (int j = 0; j < RPL / 2; j++) {
        const int d = 4 * il + 4 * LPC * (j / 2) + 2 * (j % 2);
        st[j] = dr_pack2(live && d < D ? S[(size_t)d * V] : 0.f, live && d + 1 < D ? S[(size_t)(d + 1) * V] : 0.f);
    }
    for (int c = 0; c < n_chunks; c++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DR_STAGES - 2) : "memory");
        __syncthreads();                           // chunk c is there, and every warp has left chunk c - 1
        if (c + DR_STAGES - 1 < n_chunks) fetch(c + DR_STAGES - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        float* base = dr_smem + (c % DR_STAGES) * STAGE;
        float* coefs = base + DR_NT * (2 * DP + DR_COLS + 2);
        if (warp < TURNS) {   // the factors of turn ``warp``
            float d[16];
#pragma unroll
            for (int i = 0; i < 16; i++) d[i] = 0.f;
#pragma unroll
            for (int n = 0; n < (DP + 127) / 128; n++) {
                const int at = 4 * lane + 128 * n;
                if (at < DP) {
                    float4 k[4];
#pragma unroll
                    for (int j = 0; j < 4; j++) k[j] = *reinterpret_cast<const float4*>(base + (4 * warp + j) * DP + at);
                    auto dot = [](float acc, const float4& x, const float4& y) {
                        return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, acc))));
                    };
#pragma unroll
                    for (int j = 0, n1 = 0, n2 = 6; j < 4; j++) {
                        const float4 q = *reinterpret_cast<const float4*>(base + (DR_NT + 4 * warp + j) * DP + at);
#pragma unroll
                        for (int i = 0; i < j; i++, n1++) d[n1] = dot(d[n1], k[i], k[j]);
#pragma unroll
                        for (int i = 0; i <= j; i++, n2++) d[n2] = dot(d[n2], k[i], q);
                    }
                }
            }
            const float sum = dr_fold16(d, lane);
            const float* gb = base + DR_NT * (2 * DP + DR_COLS) + 8 * warp;
            const float g[4] = {gb[0], gb[2], gb[4], gb[6]};
            const int idx = lane >> 1;
            // (j, i) of the 16 values: keys on keys (1,0) (2,0) (2,1) (3,0) (3,1) (3,2), keys on queries (0,0) (1,0) (1,1) (2,0) .. (3,3)
            const int j = (int)(0x3333222110333221ull >> (4 * idx)) & 15, i = (int)(0x3210210100210100ull >> (4 * idx)) & 15;
            float r = 1.f;
#pragma unroll
            for (int m = 1; m < 4; m++)
                if (m > i && m <= j) r *= g[m];
            float* cf = coefs + warp * DR_COEF;
            if ((lane & 1) == 0) cf[idx] = sum * r;
            if (lane < 4) {
                float up = 1.f, down = 1.f;
#pragma unroll
                for (int m = 0; m < 4; m++) {
                    if (m <= lane) up *= g[m];
                    if (m > lane) down *= g[m];
                }
                cf[16 + lane] = up, cf[20 + lane] = down, cf[24 + lane] = gb[2 * lane + 1];
            }
        }
        __syncthreads();
        const float *ks = base + 4 * il, *qs = ks + DR_NT * DP;
        const float* vs = base + 2 * DR_NT * DP + tid / LPC;
        const int nt = min(DR_NT, n_tok - c * DR_NT);
#pragma unroll 1
        for (int t0 = 0; t0 < nt; t0 += 4) {
            uint64_t a2[4] = {0, 0, 0, 0}, b2[4] = {0, 0, 0, 0};
            constexpr bool KEEP = RPL <= 16;       // the keys stay in registers for the state's update
            uint64_t kr[KEEP ? 4 : 1][KEEP ? RPL / 2 : 1];
#pragma unroll
            for (int n = 0; n < NJ; n++) {
                ulonglong2 k[4], q[4];
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    k[j] = *reinterpret_cast<const ulonglong2*>(ks + (t0 + j) * DP + 4 * LPC * n);
                    q[j] = *reinterpret_cast<const ulonglong2*>(qs + (t0 + j) * DP + 4 * LPC * n);
                }
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    a2[j] = dr_fma2(st[2 * n], k[j].x, a2[j]), b2[j] = dr_fma2(st[2 * n], q[j].x, b2[j]);
                    a2[j] = dr_fma2(st[2 * n + 1], k[j].y, a2[j]), b2[j] = dr_fma2(st[2 * n + 1], q[j].y, b2[j]);
                    if constexpr (KEEP) kr[j][2 * n] = k[j].x, kr[j][2 * n + 1] = k[j].y;
                }
            }
            float a[4], b[4];
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const float2 x = dr_unpack2(a2[j]), y = dr_unpack2(b2[j]);
                a[j] = x.x + x.y, b[j] = y.x + y.y;
            }
            float v[4];
#pragma unroll
            for (int j = 0; j < 4; j++) v[j] = vs[(t0 + j) * DR_COLS];
            float cf[DR_COEF];
#pragma unroll
            for (int i = 0; i < DR_COEF; i += 4) {
                const float4 x = *reinterpret_cast<const float4*>(coefs + (t0 / 4) * DR_COEF + i);
                cf[i] = x.x, cf[i + 1] = x.y, cf[i + 2] = x.z, cf[i + 3] = x.w;
            }
#pragma unroll
            for (int off = 1; off < LPC; off <<= 1)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    a[j] += __shfl_xor_sync(0xffffffffu, a[j], off);
                    b[j] += __shfl_xor_sync(0xffffffffu, b[j], off);
                }
            float u[4], o[4];
#pragma unroll
            for (int j = 0, n1 = 0, n2 = 6; j < 4; j++) {
                float x = v[j] - cf[16 + j] * a[j];
#pragma unroll
                for (int i = 0; i < j; i++, n1++) x = fmaf(-cf[n1], u[i], x);
                u[j] = cf[24 + j] * x;
                o[j] = cf[16 + j] * b[j];
#pragma unroll
                for (int i = 0; i <= j; i++, n2++) o[j] = fmaf(cf[n2], u[i], o[j]);
            }
            uint64_t w[4];
#pragma unroll
            for (int j = 0; j < 4; j++) w[j] = dr_pack2(cf[20 + j] * u[j], cf[20 + j] * u[j]);
            const uint64_t decay = dr_pack2(cf[19], cf[19]);
#pragma unroll
            for (int n = 0; n < RPL / 2; n++) {
                uint64_t x = dr_mul2(decay, st[n]);
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    uint64_t k;
                    if constexpr (KEEP) k = kr[j][n];
                    else k = *reinterpret_cast<const uint64_t*>(ks + (t0 + j) * DP + 4 * LPC * (n / 2) + 2 * (n % 2));
                    x = dr_fma2(k, w[j], x);
                }
                st[n] = x;
            }
            // lane j of a column stores token j
            const float mine = il == 0 ? o[0] : il == 1 ? o[1] : il == 2 ? o[2] : o[3];
            if (il < 4 && live && t0 + il < nt) out[(size_t)(r0 + c * DR_NT + t0 + il) * ow + (size_t)h * V + col] = mine;
        }
    }
    if (live) {
#pragma unroll
        for (int j = 0; j < RPL / 2; j++) {
            const int d = 4 * il + 4 * LPC * (j / 2) + 2 * (j % 2);
            const float2 x = dr_unpack2(st[j]);
            if (d < D) S[(size_t)d * V] = x.x;
            if (d + 1 < D) S[(size_t)(d + 1) * V] = x.y;
        }
    }
}

// One token a row: grid (rows, heads, ceil(V / 32)), 256 threads; thread (rg, c4): columns 4 c4 .. + 3 of the block's 32, state
// rows rg, rg + 32, .. NR: rows a thread holds, D <= 32 NR. VEC: 16-byte accesses (V a multiple of 4).
template <int NR, bool VEC>
__global__ void __launch_bounds__(256)
delta_rule_step_kernel(const float* qkv, const float* scal, float* out, float* state, const int* row_pos, const int* seq_slot, int H,
                       int G, int D, int V) {
    __shared__ float ks[256], qs[256];
    __shared__ float4 red[8][8][2];
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c4 = tid & 7, rg = tid >> 3, col = blockIdx.z * 32 + 4 * c4, kh = h / (H / G);
    const int C = 2 * G * D + H * V, nsc = 2 * H + G;
    if (row_pos[r] < 0) {
        if (rg == 0)
            for (int e = 0; e < 4; e++)
                if (col + e < V) out[(size_t)r * H * V + (size_t)h * V + col + e] = 0.f;
        return;
    }
    const float* src = qkv + (size_t)r * C;
    float* S = state + (((size_t)seq_slot[r] * H + h) * D) * V;
    float st[NR][4];
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int d = rg + 32 * i;
        if (VEC) {
            const float4 x = d < D && col < V ? *reinterpret_cast<const float4*>(S + (size_t)d * V + col) : make_float4(0.f, 0.f, 0.f, 0.f);
            st[i][0] = x.x, st[i][1] = x.y, st[i][2] = x.z, st[i][3] = x.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) st[i][e] = d < D && col + e < V ? S[(size_t)d * V + col + e] : 0.f;
        }
    }
    for (int d = tid; d < D; d += 256) qs[d] = src[kh * D + d], ks[d] = src[G * D + kh * D + d];
    const float* sc = scal + (size_t)r * nsc;
    const float g = sc[h], beta = sc[H + h], kq = sc[2 * H + kh];
    float v[4];
#pragma unroll
    for (int e = 0; e < 4; e++) v[e] = col + e < V ? src[2 * G * D + h * V + col + e] : 0.f;
    __syncthreads();
    float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int d = rg + 32 * i;
        if (d < D) {
            const float k = ks[d], q = qs[d];
#pragma unroll
            for (int e = 0; e < 4; e++) a[e] = fmaf(st[i][e], k, a[e]), b[e] = fmaf(st[i][e], q, b[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < 4; e++) {
        a[e] += __shfl_xor_sync(0xffffffffu, a[e], 8);
        b[e] += __shfl_xor_sync(0xffffffffu, b[e], 8);
        a[e] += __shfl_xor_sync(0xffffffffu, a[e], 16);
        b[e] += __shfl_xor_sync(0xffffffffu, b[e], 16);
    }
    if (lane < 8) red[warp][c4][0] = make_float4(a[0], a[1], a[2], a[3]), red[warp][c4][1] = make_float4(b[0], b[1], b[2], b[3]);
    __syncthreads();
    float4 as = red[0][c4][0], bs = red[0][c4][1];
#pragma unroll
    for (int w = 1; w < 8; w++) {
        const float4 x = red[w][c4][0], y = red[w][c4][1];
        as.x += x.x, as.y += x.y, as.z += x.z, as.w += x.w;
        bs.x += y.x, bs.y += y.y, bs.z += y.z, bs.w += y.w;
    }
    const float at[4] = {as.x, as.y, as.z, as.w}, bt[4] = {bs.x, bs.y, bs.z, bs.w};
    float u[4];
#pragma unroll
    for (int e = 0; e < 4; e++) u[e] = beta * (v[e] - g * at[e]);
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int d = rg + 32 * i;
        if (d >= D) continue;
        const float k = ks[d];
        if (VEC) {
            if (col < V)
                *reinterpret_cast<float4*>(S + (size_t)d * V + col) =
                    make_float4(fmaf(k, u[0], g * st[i][0]), fmaf(k, u[1], g * st[i][1]), fmaf(k, u[2], g * st[i][2]), fmaf(k, u[3], g * st[i][3]));
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (col + e < V) S[(size_t)d * V + col + e] = fmaf(k, u[e], g * st[i][e]);
        }
    }
    if (rg == 0)
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (col + e < V) out[(size_t)r * H * V + (size_t)h * V + col + e] = fmaf(kq, u[e], g * bt[e]);
}

DK_EXPORT int dk_delta_prepare(int dtype, const void* proj, long long ld, const void* a_rows, const void* b_rows, const void* state,
                               const void* wconv, int taps, const float* a_log, const float* dt_bias, float unit_eps,
                               const int* row_pos, const int* row_seq, const int* seq_pos0, const int* seq_slot, float* qkv,
                               float* scal, int n_tok, int H, int G, int D, int V, cudaStream_t st) {
    if (G < 1 || H % G || taps < 1 || (taps > 1 && state == nullptr)) return (int)cudaErrorInvalidValue;
    const int C = 2 * G * D + H * V;
    const size_t smem = sizeof(float) * (size_t)(2 * G * D);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const int esz = dtype == 0 ? 4 : 2;
    const int vec = C % 4 == 0 && (2 * G * D) % 4 == 0 && ld % 4 == 0 && (uintptr_t)qkv % 16 == 0 &&
                    ((uintptr_t)proj | (uintptr_t)state | (uintptr_t)wconv) % (4 * esz) == 0;
    if (dtype == 0) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(delta_prepare_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        return dk_launch(delta_prepare_kernel<float>, dim3(n_tok), dim3(DP_THREADS), smem, st, (const float*)proj, ld,
                         (const float*)a_rows, (const float*)b_rows, (const float*)state, (const float*)wconv, taps, a_log, dt_bias,
                         unit_eps, row_pos, row_seq, seq_pos0, seq_slot, qkv, scal, H, G, D, V, vec);
    }
    if (smem > 48 * 1024) cudaFuncSetAttribute(delta_prepare_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return dk_launch(delta_prepare_kernel<bf16>, dim3(n_tok), dim3(DP_THREADS), smem, st, (const bf16*)proj, ld, (const bf16*)a_rows,
                     (const bf16*)b_rows, (const bf16*)state, (const bf16*)wconv, taps, a_log, dt_bias, unit_eps, row_pos, row_seq,
                     seq_pos0, seq_slot, qkv, scal, H, G, D, V, vec);
}

DK_EXPORT int dk_delta_rule(const float* qkv, const float* scal, float* out, float* state, const int* cu_q, const int* seq_pos0,
                            const int* seq_slot, int n_seq, int H, int G, int D, int V, cudaStream_t st) {
    if (G < 1 || H % G || D < 1 || D > 256 || V < 1 || cu_q == nullptr) return (int)cudaErrorInvalidValue;
    const int C = 2 * G * D + H * V;
    const int wide_qk = D % 4 == 0 && C % 4 == 0 && (uintptr_t)qkv % 16 == 0;
    const int wide_v = wide_qk && V % 4 == 0;
    const dim3 grid(n_seq, H, (V + DR_COLS - 1) / DR_COLS);
    // Blocks that have an SM each must not share one: launched while the kernel before drains, they would pile up where it
    // leaves first. More than half of an SM's shared memory keeps them apart.
    int sms = 0, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const bool alone = (long long)grid.x * grid.y * grid.z <= sms;
#define DR_LAUNCH(R, L)                                                                                                        \
    if (D <= L * R) {                                                                                                          \
        size_t smem = sizeof(float) * DR_STAGES * (DR_NT * (2 * L * R + DR_COLS + 2) + DR_NT / 4 * DR_COEF);             \
        static bool attr = false;                                                                                              \
        if (!attr) cudaFuncSetAttribute(delta_rule_kernel<R, L>, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024);     \
        attr = true;                                                                                                           \
        if (alone && smem < 116 * 1024) smem = 116 * 1024;                                                                     \
        return dk_launch(delta_rule_kernel<R, L>, grid, dim3(L * DR_COLS), smem, st, qkv, scal, out, state, cu_q, seq_pos0,    \
                         seq_slot, H, G, D, V, wide_qk, wide_v);                                                               \
    }
    DR_LAUNCH(4, 8) DR_LAUNCH(8, 8) DR_LAUNCH(16, 8) DR_LAUNCH(32, 8)
#undef DR_LAUNCH
    return (int)cudaErrorInvalidValue;
}

DK_EXPORT int dk_delta_rule_step(const float* qkv, const float* scal, float* out, float* state, const int* row_pos,
                                 const int* seq_slot, int n_rows, int H, int G, int D, int V, cudaStream_t st) {
    if (G < 1 || H % G || D < 1 || D > 256 || V < 1) return (int)cudaErrorInvalidValue;
    const bool vec = V % 4 == 0 && (uintptr_t)state % 16 == 0;
    const dim3 grid(n_rows, H, (V + 31) / 32), block(256);
#define DS_LAUNCH(R)                                                                                                           \
    if (D <= 32 * R)                                                                                                           \
        return vec ? dk_launch(delta_rule_step_kernel<R, true>, grid, block, 0, st, qkv, scal, out, state, row_pos, seq_slot, H, G, D, V) \
                   : dk_launch(delta_rule_step_kernel<R, false>, grid, block, 0, st, qkv, scal, out, state, row_pos, seq_slot, H, G, D, V);
    DS_LAUNCH(1) DS_LAUNCH(2) DS_LAUNCH(4) DS_LAUNCH(8)
#undef DS_LAUNCH
    return (int)cudaErrorInvalidValue;
}
