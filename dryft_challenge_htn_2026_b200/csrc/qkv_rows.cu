// What stands between an attention mixer's fused projection and its cache, and behind its attention, for mixers without a
// convolution or biases (short_conv.cu has those):
//   * qkv_rows: rows [q heads | k heads | v heads] of a projection -> q rows for the attention, k and v heads at each token's
//     place in the paged stores. q and k: an RMS norm, with a weight or without, over all heads at once before the
//     rotation (norm_mode 3, weights of the whole projection's size), per head before it (1) or per head behind it (2);
//     a rotation of the first rot_dims coordinates, halves (i with i + rot_dims / 2) or neighbouring pairs (2i with 2i + 1),
//     by tables [positions, rot_dims / 2]. v: a rotation over the whole value head by tables of its own. Rows may also be
//     [q heads | k heads]: the values are then the keys as projected, before norm and rotation.
//   * turn_back_gate: per head the attention's output turned back by the token's position (the same tables, the sine
//     negated), times sigmoid of one gate number per head, times a constant.
// Norms, rotations and gates are float32 whatever the storage type. Rows with position < 0 are padding.
#include "common.cuh"

#define QR_WARPS 8

// four consecutive numbers of a head; vec: they lie on their natural boundary and the head is a multiple of four
template <typename T> __device__ __forceinline__ void ld_four(const T* p, int d, int size, bool vec, float (&y)[4]);
template <> __device__ __forceinline__ void ld_four<float>(const float* p, int d, int size, bool vec, float (&y)[4]) {
    if (vec) {
        const float4 x = d < size ? *reinterpret_cast<const float4*>(p + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        y[0] = x.x, y[1] = x.y, y[2] = x.z, y[3] = x.w;
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; e++) y[e] = d + e < size ? p[d + e] : 0.f;
}
template <> __device__ __forceinline__ void ld_four<bf16>(const bf16* p, int d, int size, bool vec, float (&y)[4]) {
    if (vec) {
        uint2 r = make_uint2(0u, 0u);
        if (d < size) r = *reinterpret_cast<const uint2*>(p + d);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
        y[0] = a.x, y[1] = a.y, y[2] = b.x, y[3] = b.y;
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; e++) y[e] = d + e < size ? __bfloat162float(p[d + e]) : 0.f;
}
__device__ __forceinline__ void st_four(float* p, int d, int size, bool vec, const float (&y)[4]) {
    if (vec) {
        if (d < size) *reinterpret_cast<float4*>(p + d) = make_float4(y[0], y[1], y[2], y[3]);
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; e++)
        if (d + e < size) p[d + e] = y[e];
}
__device__ __forceinline__ void st_four(bf16* p, int d, int size, bool vec, const float (&y)[4]) {
    if (vec) {
        if (d >= size) return;
        __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
        uint2 o;
        o.x = *reinterpret_cast<uint32_t*>(&lo);
        o.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p + d) = o;
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; e++)
        if (d + e < size) p[d + e] = __float2bfloat16_rn(y[e]);
}

// A lane's angles of a rotation over the first ``dims`` coordinates: its coordinates are 4 lane + 128 i + e. Pairs: the
// angle of coordinate d is d / 2; halves: d below dims / 2, d - dims / 2 from there. Past the rotation: the identity.
template <int NI>
struct Angles {
    float c[NI][4], s[NI][4];
    __device__ __forceinline__ void load(const float* cosv, const float* sinv, int pos, int dims, int pairs) {
        const int lane = threadIdx.x & 31, half = dims / 2;
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int d = 4 * lane + 128 * i + e, j = pairs ? d / 2 : d < half ? d : d - half;
                const bool on = d < dims;
                c[i][e] = on ? cosv[(size_t)pos * half + j] : 1.f;
                s[i][e] = on ? sinv[(size_t)pos * half + j] : 0.f;
            }
    }
};

// y[i] holds coordinates 4 lane + 128 i .. + 3 of a head. Pairs turn inside a lane; halves meet their partner by a shuffle
// where half the rotation is a multiple of four inside the first 128 coordinates, else through the warp's own shared memory.
template <int NI>
__device__ __forceinline__ void rotate_head(float (&y)[NI][4], float* ys, const Angles<NI>& a, int dims, int pairs) {
    const int lane = threadIdx.x & 31, half = dims / 2;
    if (pairs) {
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const float u = y[i][e], v = y[i][e + 1];
                y[i][e] = u * a.c[i][e] - v * a.s[i][e];
                y[i][e + 1] = v * a.c[i][e] + u * a.s[i][e];
            }
        return;
    }
    if (NI == 1 && half % 4 == 0) {
        const bool low = 4 * lane < half;
        const int from = low ? lane + half / 4 : lane - half / 4;
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const float other = __shfl_sync(0xffffffffu, y[0][e], from & 31);
            y[0][e] = low ? y[0][e] * a.c[0][e] - other * a.s[0][e] : y[0][e] * a.c[0][e] + other * a.s[0][e];
        }
        return;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) ys[4 * lane + 128 * i + e] = y[i][e];
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int d = 4 * lane + 128 * i + e;
            if (d < dims) y[i][e] = d < half ? y[i][e] * a.c[i][e] - ys[d + half] * a.s[i][e] : y[i][e] * a.c[i][e] + ys[d - half] * a.s[i][e];
        }
}

// A block per token (and part of its heads); a warp takes up to HPW heads at a time, all of them asked for before any is
// used. NI: 1 for heads up to 128, 2 up to 256.
template <typename T, int NI, int HPW>
__global__ void __launch_bounds__(32 * QR_WARPS)
qkv_rows_kernel(const T* proj, long long ld, T* q_out, long long ldq, int norm_mode, const float* __restrict__ qn,
                const float* __restrict__ kn, float eps, const float* __restrict__ cosv, const float* __restrict__ sinv,
                int rot_dims, int pairs, const float* __restrict__ vcos, const float* __restrict__ vsin, int v_pairs,
                const int* row_pos, const int* row_seq, int nh, int nkv, int hd, int hdv, T* k_store, T* v_store,
                const int* page_table, int pt_stride, int kv_same, int vec) {
    __shared__ float ys_all[QR_WARPS][128 * NI];
    __shared__ float2 sums[QR_WARPS];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x;
    const int nq = nh * hd, nk = nkv * hd, heads = nh + 2 * nkv;
    pdl_wait();
    pdl_launch_dependents();
    const T* row = proj + (size_t)t * ld;
    float y[HPW][NI][4];
    auto load = [&](int head0) {
#pragma unroll
        for (int n = 0; n < HPW; n++) {
            const int head = head0 + n * gridDim.y * QR_WARPS;
            const bool is_v = head >= nh + nkv;
            const T* src = row + (is_v ? nq + (kv_same ? 0 : nk) + (head - nh - nkv) * hdv : head * hd);
#pragma unroll
            for (int i = 0; i < NI; i++) ld_four<T>(src, 4 * lane + 128 * i, head >= heads ? 0 : is_v ? hdv : hd, vec, y[n][i]);
        }
    };
    const int first = blockIdx.y * QR_WARPS + warp;
    load(first);
    const int pos = row_pos[t];
    if (pos < 0) return;
    Angles<NI> ang, vang;
    if (rot_dims > 0) ang.load(cosv, sinv, pos, rot_dims, pairs);
    if (vcos != nullptr) vang.load(vcos, vsin, pos, hdv, v_pairs);
    float rq = 1.f, rk = 1.f;
    if (norm_mode == 3) {                          // all of q, and all of k, over their root mean squares
        float sq = 0.f, sk = 0.f;
        if (gridDim.y == 1 && heads <= HPW * QR_WARPS) {        // every head of the row is here already
#pragma unroll
            for (int n = 0; n < HPW; n++) {
                const int head = first + n * QR_WARPS;
                float ss = 0.f;
#pragma unroll
                for (int i = 0; i < NI; i++) ss += (y[n][i][0] * y[n][i][0] + y[n][i][1] * y[n][i][1]) + (y[n][i][2] * y[n][i][2] + y[n][i][3] * y[n][i][3]);
                if (head < nh) sq += ss;
                else if (head < nh + nkv) sk += ss;
            }
        } else {
            for (int d = 4 * threadIdx.x; d < nq; d += 4 * 32 * QR_WARPS) {
                float x[4];
                ld_four<T>(row, d, nq, vec, x);
                sq += (x[0] * x[0] + x[1] * x[1]) + (x[2] * x[2] + x[3] * x[3]);
            }
            for (int d = 4 * threadIdx.x; d < nk; d += 4 * 32 * QR_WARPS) {
                float x[4];
                ld_four<T>(row + nq, d, nk, vec, x);
                sk += (x[0] * x[0] + x[1] * x[1]) + (x[2] * x[2] + x[3] * x[3]);
            }
        }
        sq = warp_sum(sq), sk = warp_sum(sk);
        if (lane == 0) sums[warp] = make_float2(sq, sk);
        __syncthreads();
        sq = sk = 0.f;
#pragma unroll
        for (int i = 0; i < QR_WARPS; i++) sq += sums[i].x, sk += sums[i].y;
        rq = 1.f / sqrtf(sq / (float)nq + eps);
        rk = 1.f / sqrtf(sk / (float)nk + eps);
    }
    const int page = k_store != nullptr ? page_table[(size_t)row_seq[t] * pt_stride + pos / DK_PAGE] : -1;
    float* ys = ys_all[warp];
    for (int head0 = first;;) {
#pragma unroll
        for (int n = 0; n < HPW; n++) {
            const int head = head0 + n * gridDim.y * QR_WARPS;
            if (head >= heads) break;
            const bool is_q = head < nh, is_v = head >= nh + nkv;
            if (!is_q && page < 0) continue;       // another layer's cache: only the queries are wanted
            if (is_v) {
                if (vcos != nullptr) rotate_head<NI>(y[n], ys, vang, hdv, v_pairs);
            } else {
                const float* w = is_q ? qn : kn;
                auto scale = [&](float r, int w0) {
#pragma unroll
                    for (int i = 0; i < NI; i++) {
                        float ww[4] = {1.f, 1.f, 1.f, 1.f};
                        if (w) ld_four<float>(w + w0, 4 * lane + 128 * i, hd, hd % 4 == 0, ww);
#pragma unroll
                        for (int e = 0; e < 4; e++) y[n][i][e] *= r * ww[e];
                    }
                };
                auto norm_head = [&]() {
                    float ss = 0.f;
#pragma unroll
                    for (int i = 0; i < NI; i++)
#pragma unroll
                        for (int e = 0; e < 4; e++) ss += y[n][i][e] * y[n][i][e];          // coordinates past the head are zero
                    scale(1.f / sqrtf(warp_sum(ss) / (float)hd + eps), 0);
                };
                if (norm_mode == 3) scale(is_q ? rq : rk, (is_q ? head : head - nh) * hd);
                if (norm_mode == 1) norm_head();
                if (rot_dims > 0) rotate_head<NI>(y[n], ys, ang, rot_dims, pairs);
                if (norm_mode == 2) norm_head();
            }
            T* dst = is_q ? q_out + (size_t)t * ldq + head * hd
                          : is_v ? v_store + kv_offset(page, nkv, head - nh - nkv, pos % DK_PAGE, hdv)
                                 : k_store + kv_offset(page, nkv, head - nh, pos % DK_PAGE, hd);
#pragma unroll
            for (int i = 0; i < NI; i++) st_four(dst, 4 * lane + 128 * i, is_v ? hdv : hd, vec, y[n][i]);
        }
        head0 += HPW * gridDim.y * QR_WARPS;
        if (head0 >= heads) break;
        load(head0);
    }
}

// A thread per (token, head, N pairs). N = 4: the pairs' numbers are two runs of four on their natural boundaries; N = 1: any.
template <typename T, int N, bool PAIRS>
__global__ void turn_back_gate_kernel(const T* o, long long ldi, T* out, long long ldo, const T* gate, long long ldg,
                                      const float* __restrict__ cosv, const float* __restrict__ sinv, float out_scale,
                                      const int* row_pos, long long items, int nh, int hdv) {
    pdl_wait();
    pdl_launch_dependents();
    const long long item = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (item >= items) return;
    const int half = hdv / 2, per = half / N;
    const int m0 = (int)(item % per) * N, h = (int)(item / per % nh);
    const size_t t = (size_t)(item / per / nh);
    const int pos = max(row_pos[t], 0);
    float f = out_scale;
    if (gate != nullptr) f /= 1.f + expf(-to_f(gate[t * ldg + h]));
    const T* src = o + t * ldi + (size_t)h * hdv;
    T* dst = out + t * ldo + (size_t)h * hdv;
    // the two runs of N numbers: first and second members of the pairs (halves), or the pairs side by side (pairs)
    const int a0 = PAIRS ? 2 * m0 : m0, b0 = PAIRS ? 2 * m0 + N : m0 + half;
    float x[2 * N];
    if (N == 4) {
        float u[4], v[4];
        ld_four<T>(src, a0, hdv, true, u);
        ld_four<T>(src, b0, hdv, true, v);
#pragma unroll
        for (int e = 0; e < N; e++) x[e] = u[e & 3], x[N + e] = v[e & 3];
    } else {
        x[0] = to_f(src[a0]), x[1] = to_f(src[b0]);
    }
    if (cosv != nullptr) {
#pragma unroll
        for (int e = 0; e < N; e++) {
            const float c = cosv[(size_t)pos * half + m0 + e], s = -sinv[(size_t)pos * half + m0 + e];
            const int iu = PAIRS ? 2 * e : e, iv = PAIRS ? 2 * e + 1 : N + e;
            const float u = x[iu], v = x[iv];
            x[iu] = u * c - v * s;
            x[iv] = v * c + u * s;
        }
    }
    if (N == 4) {
        float u[4], v[4];
#pragma unroll
        for (int e = 0; e < N; e++) u[e & 3] = x[e] * f, v[e & 3] = x[N + e] * f;
        st_four(dst, a0, hdv, true, u);
        st_four(dst, b0, hdv, true, v);
    } else {
        dst[a0] = from_f<T>(x[0] * f), dst[b0] = from_f<T>(x[1] * f);
    }
}

DK_EXPORT int dk_qkv_rows(int dtype, const void* proj, long long ld, void* q_out, long long ldq, int norm_mode, const float* qn,
                          const float* kn, float eps, const float* cosv, const float* sinv, int rot_dims, int pairs,
                          const float* vcos, const float* vsin, int v_pairs, const int* row_pos, const int* row_seq, int n_tok,
                          int nh, int nkv, int hd, int hdv, void* k_store, void* v_store, const int* page_table, int pt_stride,
                          int kv_same, cudaStream_t st) {
    if (hd < 1 || hd > 256 || hdv < 1 || hdv > 256 || rot_dims > hd || rot_dims % 2 || (vcos != nullptr && hdv % 2) ||
        norm_mode < 0 || norm_mode > 3 || (kv_same && hd != hdv))
        return (int)cudaErrorInvalidValue;
    const int esz = dtype == 0 ? 4 : 2;
    const int vec = hd % 4 == 0 && hdv % 4 == 0 && ld % 4 == 0 && ldq % 4 == 0 &&
                    ((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_store | (uintptr_t)v_store) % (4 * esz) == 0;
    // the heads of a row in one block where its norm spans them all, else dealt out so that few rows still fill the SMs
    const int groups = (nh + 2 * nkv + QR_WARPS - 1) / QR_WARPS;
    int split = 1;
    if (norm_mode != 3) split = n_tok < 512 ? groups : (groups + 2) / 3;
    else if (n_tok <= 64) split = min(groups, 4);       // every block takes the sums anew: a short row read again
    const int per = (groups + split - 1) / split;       // heads a warp
    const dim3 grid(n_tok, split), block(32 * QR_WARPS);
#define QR_LAUNCH(T, NI, HPW)                                                                                                \
    return dk_launch(qkv_rows_kernel<T, NI, HPW>, grid, block, 0, st, (const T*)proj, ld, (T*)q_out, ldq, norm_mode, qn, kn, eps, \
                     cosv, sinv, rot_dims, pairs, vcos, vsin, v_pairs, row_pos, row_seq, nh, nkv, hd, hdv, (T*)k_store,      \
                     (T*)v_store, page_table, pt_stride, kv_same, vec)
    const bool small = hd <= 128 && hdv <= 128;
    if (dtype == 0) {
        if (small) QR_LAUNCH(float, 1, 3);
        QR_LAUNCH(float, 2, 2);
    }
    if (small && per <= 1) QR_LAUNCH(bf16, 1, 1);
    if (small && per <= 3) QR_LAUNCH(bf16, 1, 3);
    if (small) QR_LAUNCH(bf16, 1, 6);
    QR_LAUNCH(bf16, 2, 2);
#undef QR_LAUNCH
}

DK_EXPORT int dk_turn_back_gate(int dtype, const void* o, long long ldi, void* out, long long ldo, const void* gate, long long ldg,
                                const float* cosv, const float* sinv, int pairs, float out_scale, const int* row_pos, int n_tok,
                                int nh, int hdv, cudaStream_t st) {
    if (hdv < 2 || hdv % 2) return (int)cudaErrorInvalidValue;
    const int esz = dtype == 0 ? 4 : 2;
    const bool four = hdv % 8 == 0 && ldi % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)o | (uintptr_t)out) % (4 * esz) == 0;
    const long long items = (long long)n_tok * nh * (hdv / 2 / (four ? 4 : 1));
    const dim3 grid((unsigned)((items + 255) / 256)), block(256);
#define TB_LAUNCH(T, N)                                                                                                     \
    return pairs ? dk_launch(turn_back_gate_kernel<T, N, true>, grid, block, 0, st, (const T*)o, ldi, (T*)out, ldo, (const T*)gate, \
                             ldg, cosv, sinv, out_scale, row_pos, items, nh, hdv)                                           \
                 : dk_launch(turn_back_gate_kernel<T, N, false>, grid, block, 0, st, (const T*)o, ldi, (T*)out, ldo, (const T*)gate, \
                             ldg, cosv, sinv, out_scale, row_pos, items, nh, hdv)
    if (dtype == 0) {
        if (four) TB_LAUNCH(float, 4);
        TB_LAUNCH(float, 1);
    }
    if (four) TB_LAUNCH(bf16, 4);
    TB_LAUNCH(bf16, 1);
#undef TB_LAUNCH
}
