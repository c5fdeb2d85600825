// The matrix memory with exponential gates (see matrix_memory.cu for the recurrence and its token-by-token form) for portions of
// many tokens in bfloat16 storage, in chunks of 256 tokens that run side by side. Built per pair of head sizes with -DHD=<key
// size, multiple of 16 up to 128> -DHDV=<value size, multiple of 16 up to 128>.
//
// mm_gates leaves per token L_t = sum of log2 of the factors the state is multiplied by, from its chunk's first token to t, and
// w_t = exp(i_t - m_t). With S_0, n_0 the states ahead of a chunk of n tokens,
//     S^T q_t = 2^L_t S_0^T q_t + sum_{s <= t} 2^(L_t - L_s) w_s (k_s . q_t) v_s,     S_n = 2^L_n S_0 + sum_s 2^(L_n - L_s) w_s k_s v_s^T,
// and the same for n with one in place of v: n rides along as a value column of ones.
//   * mm_chunk_states : every chunk's own sum [HD, HDV | n], a block per (chunk, head).
//   * mm_chunk_scan   : S_n of one chunk after the other, a thread per four state elements; leaves every chunk's S_0 as a high and
//                       a low bfloat16 plane.
//   * mm_chunk_outputs: 128 tokens of a chunk and a head a block: q S_0, the weighted scores inside the chunk times v, then
//                       the quotient, the norm over the head's values, weight and gate.
// All products are mma.sync with float32 sums. q, k, v are bfloat16 as projected; what is float32 (weighted keys, weighted scores,
// the state) enters as a high and a low bfloat16 half, two products, so it counts with 16 bits of mantissa.
#include "attention_mma.cuh"

#ifndef HDV
#error "compile with -DHDV=<value size>"
#endif
static_assert(HD <= 128 && HDV % 16 == 0 && HDV >= 16 && HDV <= 128, "key and value sizes in steps of 16 up to 128");

constexpr int MM_CHUNK = 256;           // tokens a chunk
constexpr int MM_TILE = 64;             // keys a stage
constexpr int MM_ROWS = 128;            // queries a block of mm_chunk_outputs
constexpr int VS = HDV + 8;             // row stride of staged values, and of a chunk's state (its last 8 columns: n, then zeros)
constexpr int NT = HDV / 8;             // value columns in tiles of 8; tile NT holds n

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t (&r)[2], const bf16* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}
// x0, x1 as bfloat16 pairs: the rounded values and what rounding left
__device__ __forceinline__ void split_pair(float x0, float x1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x0, x1);
    const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
    lo = pack_bf16(x0 - h.x, x1 - h.y);
}
// rows of a tile: n of them from memory, zeros behind
__device__ __forceinline__ void stage_rows(bf16* dst, int stride, const bf16* src, long long ld, int rows, int n, int width) {
    const int cpr = width / 8;
    for (int i = threadIdx.x; i < rows * cpr; i += blockDim.x) {
        const int r = i / cpr, c = i % cpr * 8;
        if (r < n) cp_async16(dst + r * stride + c, src + (size_t)r * ld + c);
        else *reinterpret_cast<uint4*>(dst + r * stride + c) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// chunks [n_chunks][4] = (sequence, first row of the chunk in the step, its rows, its number within the sequence)
constexpr int ST_WARPS = HD / 16;
__global__ void __launch_bounds__(32 * ST_WARPS)
mm_chunk_states_kernel(const bf16* k, const bf16* v, long long ld, const float4* scal, const int4* chunks, float* u, int nh) {
    extern __shared__ __align__(16) bf16 mmc_smem[];
    constexpr int STAGE = MM_TILE * (KSTR + VS);
    float* wt = reinterpret_cast<float*>(mmc_smem + 2 * STAGE);        // [MM_CHUNK]
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int4 ch = chunks[blockIdx.x];
    const int h = blockIdx.y, r0 = ch.y, n = ch.z;
    auto issue = [&](int st) {
        const int s0 = st * MM_TILE;
        if (s0 < n) {
            bf16* base = mmc_smem + (st & 1) * STAGE;
            stage_rows(base, KSTR, k + (size_t)(r0 + s0) * ld + (size_t)h * HD, ld, MM_TILE, n - s0, HD);
            stage_rows(base + MM_TILE * KSTR, VS, v + (size_t)(r0 + s0) * ld + (size_t)h * HDV, ld, MM_TILE, n - s0, HDV);
        }
        cp_async_commit();
    };
    issue(0);
    const float ln = scal[(size_t)(r0 + n - 1) * nh + h].x;
    for (int i = tid; i < MM_CHUNK; i += blockDim.x) {
        float w = 0.f;
        if (i < n) {
            const float4 x = scal[(size_t)(r0 + i) * nh + h];
            w = ex2(ln - x.x) * x.y;
        }
        wt[i] = w;
    }
    float acc[NT + 1][4];
#pragma unroll
    for (int i = 0; i <= NT; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const uint32_t one = g == 0 ? 0x3f803f80u : 0u;                      // the value column of ones, in tile NT
    const int n_st = (n + MM_TILE - 1) / MM_TILE;
    for (int st = 0; st < n_st; st++) {
        cp_async_wait<0>();
        __syncthreads();
        issue(st + 1);
        const bf16* Ks = mmc_smem + (st & 1) * STAGE;
        const bf16* Vt = Ks + MM_TILE * KSTR;
#pragma unroll
        for (int kk = 0; kk < MM_TILE / 16; kk++) {
            uint32_t a[4], ah[4], al[4];
            ldsm_a_transposed(a, Ks, kk * 16, warp * 16);
            const float2 w0 = *reinterpret_cast<const float2*>(wt + st * MM_TILE + kk * 16 + 2 * t);
            const float2 w1 = *reinterpret_cast<const float2*>(wt + st * MM_TILE + kk * 16 + 8 + 2 * t);
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[r]));
                split_pair(x.x * (r < 2 ? w0.x : w1.x), x.y * (r < 2 ? w0.y : w1.y), ah[r], al[r]);
            }
#pragma unroll
            for (int dp = 0; dp < HDV / 16; dp++) {
                uint32_t b[4];
                ldsm_x4_trans(b, Vt + (kk * 16 + (lane & 15)) * VS + dp * 16 + 8 * (lane >> 4));
                mma16816(acc[2 * dp], ah, b[0], b[1]);
                mma16816(acc[2 * dp + 1], ah, b[2], b[3]);
                mma16816(acc[2 * dp], al, b[0], b[1]);
                mma16816(acc[2 * dp + 1], al, b[2], b[3]);
            }
            mma16816(acc[NT], ah, one, one);
            mma16816(acc[NT], al, one, one);
        }
    }
    float* to = u + ((size_t)blockIdx.x * nh + h) * HD * VS;
#pragma unroll
    for (int i = 0; i <= NT; i++)
#pragma unroll
        for (int r = 0; r < 2; r++)
            *reinterpret_cast<float2*>(to + (size_t)(warp * 16 + g + 8 * r) * VS + i * 8 + 2 * t) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
}

// A thread: four columns of a row of [HD, HDV | n]. firsts [n_seq][4] = (first chunk, chunks, -, -). planes [chunk][head][2][HD][VS].
__global__ void __launch_bounds__(256)
mm_chunk_scan_kernel(const float* __restrict__ u, bf16* planes, const float4* __restrict__ scal, const int4* firsts, const int4* __restrict__ chunks,
                     float* state, float* n_state, const int* seq_slot, int nh) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int QUADS = HD * VS / 4;
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= QUADS) return;
    const int h = blockIdx.y, s = blockIdx.z;
    const int d = i / (VS / 4), c = i % (VS / 4) * 4;
    const size_t sh = (size_t)seq_slot[s] * nh + h;
    float* S = state + (sh * HD + d) * HDV + c;
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < HDV) {
        const float4 y = *reinterpret_cast<const float4*>(S);
        x[0] = y.x, x[1] = y.y, x[2] = y.z, x[3] = y.w;
    } else if (c == HDV) {
        x[0] = n_state[sh * HD + d];
    }
    const int c0 = firsts[s].x, nc = firsts[s].y;
#pragma unroll 4
    for (int k = 0; k < nc; k++) {
        const size_t at = (size_t)(c0 + k) * nh + h;
        const int4 ch = chunks[c0 + k];
        const float keep = ex2(scal[(size_t)(ch.y + ch.z - 1) * nh + h].x);
        const float4 y = *reinterpret_cast<const float4*>(u + at * HD * VS + (size_t)d * VS + c);
        uint32_t hi[2], lo[2];
        split_pair(x[0], x[1], hi[0], lo[0]);
        split_pair(x[2], x[3], hi[1], lo[1]);
        bf16* p = planes + at * 2 * HD * VS + (size_t)d * VS + c;
        *reinterpret_cast<uint2*>(p) = make_uint2(hi[0], hi[1]);
        *reinterpret_cast<uint2*>(p + HD * VS) = make_uint2(lo[0], lo[1]);
        x[0] = fmaf(keep, x[0], y.x), x[1] = fmaf(keep, x[1], y.y), x[2] = fmaf(keep, x[2], y.z), x[3] = fmaf(keep, x[3], y.w);
    }
    if (c < HDV) *reinterpret_cast<float4*>(S) = make_float4(x[0], x[1], x[2], x[3]);
    else if (c == HDV) n_state[sh * HD + d] = x[0];
}

// Block (128 tokens of a chunk, head); a warp 16 of the tokens. The stages: the state's planes by 64 rows, then keys and values by
// 64 tokens up to the block's last token; two in turn.
constexpr int SLAB = HD < 64 ? HD : 64, N_SLABS = (HD + 63) / 64;
constexpr int OUT_STAGE = (2 * SLAB * VS > MM_TILE * (KSTR + VS)) ? 2 * SLAB * VS : MM_TILE * (KSTR + VS);
__global__ void __launch_bounds__(256, 2)
mm_chunk_outputs_kernel(const bf16* q, const bf16* k, const bf16* v, const bf16* gate, long long ld, const float4* scal, const int4* chunks,
                        const bf16* planes, const float* __restrict__ w, float eps, float q_scale, float out_scale, bf16* out, long long ldo,
                        int nh) {
    extern __shared__ __align__(16) bf16 mmc_smem[];
    bf16* Qs = mmc_smem;                                                 // [MM_ROWS][KSTR]
    bf16* ring = Qs + MM_ROWS * KSTR;                                    // [2][OUT_STAGE]
    float2* lw = reinterpret_cast<float2*>(ring + 2 * OUT_STAGE);        // [MM_CHUNK] (L, w)
    pdl_wait();
    pdl_launch_dependents();
    constexpr int SUBS = MM_CHUNK / MM_ROWS;
    const int chunk = blockIdx.x / SUBS, row0 = blockIdx.x % SUBS * MM_ROWS;      // rows counted from the chunk's first
    const int4 ch = chunks[chunk];
    const int h = blockIdx.y, r0 = ch.y, n = ch.z;
    if (row0 >= n) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int last = min(n, row0 + MM_ROWS), n_keys = (last + MM_TILE - 1) / MM_TILE, n_st = N_SLABS + n_keys;
    const bf16* P = planes + ((size_t)chunk * nh + h) * 2 * HD * VS;
    auto issue = [&](int st) {
        bf16* base = ring + (st & 1) * OUT_STAGE;
        if (st < N_SLABS) {
            const int rows = min(SLAB, HD - st * SLAB), pieces = rows * VS / 8;       // a slab of a plane is one run of memory
            for (int i = tid; i < 2 * pieces; i += 256) {
                const int pl = i / pieces, x = i % pieces * 8;
                cp_async16(base + pl * SLAB * VS + x, P + (size_t)pl * HD * VS + (size_t)st * SLAB * VS + x);
            }
        } else if (st < n_st) {
            const int s0 = (st - N_SLABS) * MM_TILE;
            stage_rows(base, KSTR, k + (size_t)(r0 + s0) * ld + (size_t)h * HD, ld, MM_TILE, n - s0, HD);
            stage_rows(base + MM_TILE * KSTR, VS, v + (size_t)(r0 + s0) * ld + (size_t)h * HDV, ld, MM_TILE, n - s0, HDV);
        }
        cp_async_commit();
    };
    stage_rows(Qs, KSTR, q + (size_t)(r0 + row0) * ld + (size_t)h * HD, ld, MM_ROWS, n - row0, HD);
    issue(0);
    for (int i = tid; i < MM_CHUNK; i += 256) {
        float2 x = make_float2(0.f, 0.f);
        if (i < last) {
            const float4 y = scal[(size_t)(r0 + i) * nh + h];
            x = make_float2(y.x, y.y * q_scale);
        }
        lw[i] = x;
    }
    float acc[NT + 1][4];
#pragma unroll
    for (int i = 0; i <= NT; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const uint32_t one = g == 0 ? 0x3f803f80u : 0u;
    const int wrow = row0 + warp * 16;                                   // the warp's first row
    float L[2];
    for (int st = 0; st < n_st; st++) {
        cp_async_wait<0>();
        __syncthreads();
        issue(st + 1);
        const bf16* base = ring + (st & 1) * OUT_STAGE;
        if (wrow >= n) continue;
        if (st < N_SLABS) {
            const int rows = min(SLAB, HD - st * SLAB);
#pragma unroll
            for (int ks = 0; ks < SLAB / 16; ks++) {
                if (ks * 16 >= rows) break;
                uint32_t a[4];
                ldsm_x4(a, Qs + (warp * 16 + (lane & 15)) * KSTR + st * SLAB + ks * 16 + 8 * (lane >> 4));
#pragma unroll
                for (int pl = 0; pl < 2; pl++) {
                    const bf16* Sp = base + pl * SLAB * VS + (ks * 16 + (lane & 15)) * VS;
#pragma unroll
                    for (int dp = 0; dp < HDV / 16; dp++) {
                        uint32_t b[4];
                        ldsm_x4_trans(b, Sp + dp * 16 + 8 * (lane >> 4));
                        mma16816(acc[2 * dp], a, b[0], b[1]);
                        mma16816(acc[2 * dp + 1], a, b[2], b[3]);
                    }
                    uint32_t b2[2];
                    ldsm_x2_trans(b2, Sp + HDV);
                    mma16816(acc[NT], a, b2[0], b2[1]);
                }
            }
            if (st == N_SLABS - 1) {
                L[0] = lw[wrow + g].x, L[1] = lw[wrow + g + 8].x;
                const float f0 = ex2(L[0]) * q_scale, f1 = ex2(L[1]) * q_scale;
#pragma unroll
                for (int i = 0; i <= NT; i++) acc[i][0] *= f0, acc[i][1] *= f0, acc[i][2] *= f1, acc[i][3] *= f1;
            }
            continue;
        }
        const bf16* Vt = base + MM_TILE * KSTR;
        const int s0 = (st - N_SLABS) * MM_TILE;
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int j0 = s0 + half * 32;
            if (j0 > wrow + 15) break;
            float sc[4][4];
#pragma unroll
            for (int i = 0; i < 4; i++) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
            const int j4 = lane >> 3;
#pragma unroll
            for (int ks = 0; ks < HD / 16; ks++) {
                uint32_t a[4];
                ldsm_x4(a, Qs + (warp * 16 + (lane & 15)) * KSTR + ks * 16 + 8 * (lane >> 4));
#pragma unroll
                for (int np = 0; np < 2; np++) {
                    uint32_t b[4];
                    ldsm_x4(b, base + (half * 32 + np * 16 + (lane & 7) + 8 * (j4 >> 1)) * KSTR + ks * 16 + 8 * (j4 & 1));
                    mma16816(sc[2 * np], a, b[0], b[1]);
                    mma16816(sc[2 * np + 1], a, b[2], b[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < 4; nt++) {
                const int j = j0 + nt * 8 + 2 * t;
                const float4 x = *reinterpret_cast<const float4*>(lw + j);           // (L, w) of keys j and j + 1
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    const int i = wrow + g + 8 * (c >> 1);
                    const float f = ex2(L[c >> 1] - (c & 1 ? x.z : x.x)) * (c & 1 ? x.w : x.y);
                    sc[nt][c] = j + (c & 1) <= i ? sc[nt][c] * f : 0.f;
                }
            }
#pragma unroll
            for (int kk = 0; kk < 2; kk++) {
                uint32_t ah[4], al[4];
                split_pair(sc[2 * kk][0], sc[2 * kk][1], ah[0], al[0]);
                split_pair(sc[2 * kk][2], sc[2 * kk][3], ah[1], al[1]);
                split_pair(sc[2 * kk + 1][0], sc[2 * kk + 1][1], ah[2], al[2]);
                split_pair(sc[2 * kk + 1][2], sc[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
                for (int dp = 0; dp < HDV / 16; dp++) {
                    uint32_t b[4];
                    ldsm_x4_trans(b, Vt + (half * 32 + kk * 16 + (lane & 15)) * VS + dp * 16 + 8 * (lane >> 4));
                    mma16816(acc[2 * dp], ah, b[0], b[1]);
                    mma16816(acc[2 * dp + 1], ah, b[2], b[3]);
                    mma16816(acc[2 * dp], al, b[0], b[1]);
                    mma16816(acc[2 * dp + 1], al, b[2], b[3]);
                }
                mma16816(acc[NT], ah, one, one);
                mma16816(acc[NT], al, one, one);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int i = wrow + g + 8 * r;
        const float nq = __shfl_sync(0xffffffffu, acc[NT][2 * r], lane & ~3);          // column 0 of the last tile: n . q
        const size_t row = (size_t)(r0 + min(i, n - 1));
        const float inv = 1.f / (fmaxf(fabsf(nq), scal[row * nh + h].z) + 1e-6f);
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < NT; c++) {
            const float y0 = acc[c][2 * r] * inv, y1 = acc[c][2 * r + 1] * inv;
            ss += y0 * y0 + y1 * y1;
        }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        const float rs = inv * (out_scale / sqrtf(ss / (float)HDV + eps));
        if (i >= n) continue;
#pragma unroll
        for (int c = 0; c < NT; c++) {
            const size_t at = (size_t)h * HDV + c * 8 + 2 * t;
            const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + row * ld + at));
            const float2 ww = *reinterpret_cast<const float2*>(w + at);
            *reinterpret_cast<uint32_t*>(out + row * ldo + at) = pack_bf16(acc[c][2 * r] * rs * ww.x / (1.f + __expf(-z.x)),
                                                                           acc[c][2 * r + 1] * rs * ww.y / (1.f + __expf(-z.y)));
        }
    }
}

// u float32 [n_chunks, nh, HD, VS] and planes bfloat16 [n_chunks, nh, 2, HD, VS]: scratch. plan [n_seq + n_chunks][4].
DK_EXPORT int dk_mm_chunks(const void* q, const void* k, const void* v, const void* gate, long long ld, const void* scal, const int* plan,
                           int n_seq, int n_chunks, float* u, void* planes, float* state, float* n_state, const int* seq_slot,
                           const float* w, float eps, float q_scale, float out_scale, void* out, long long ldo, int nh, cudaStream_t st) {
    if (ld % 8 || ldo % 2 || ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)plan) % 16 ||
        ((uintptr_t)gate | (uintptr_t)out) % 4 || (uintptr_t)w % 8)
        return (int)cudaErrorInvalidValue;
    constexpr size_t s_smem = sizeof(bf16) * 2 * MM_TILE * (KSTR + VS) + sizeof(float) * MM_CHUNK;
    constexpr size_t o_smem = sizeof(bf16) * (MM_ROWS * KSTR + 2 * OUT_STAGE) + sizeof(float2) * MM_CHUNK;
    static bool attr = false;
    if (!attr) {
        cudaError_t e = cudaFuncSetAttribute(mm_chunk_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_smem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(mm_chunk_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)o_smem);
        if (e != cudaSuccess) return (int)e;
        attr = true;
    }
    const int4* firsts = reinterpret_cast<const int4*>(plan);
    const int4* chunks = firsts + n_seq;
    int e = dk_launch(mm_chunk_states_kernel, dim3(n_chunks, nh), dim3(32 * ST_WARPS), s_smem, st, (const bf16*)k, (const bf16*)v, ld,
                      (const float4*)scal, chunks, u, nh);
    if (e) return e;
    e = dk_launch(mm_chunk_scan_kernel, dim3((HD * VS / 4 + 255) / 256, nh, n_seq), dim3(256), 0, st, u, (bf16*)planes, (const float4*)scal, firsts,
                  chunks, state, n_state, seq_slot, nh);
    if (e) return e;
    return dk_launch(mm_chunk_outputs_kernel, dim3(n_chunks * (MM_CHUNK / MM_ROWS), nh), dim3(256), o_smem, st, (const bf16*)q, (const bf16*)k,
                     (const bf16*)v, (const bf16*)gate, ld, (const float4*)scal, chunks, (const bf16*)planes, w, eps, q_scale, out_scale,
                     (bf16*)out, ldo, nh);
}
