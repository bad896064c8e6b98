// Linear recurrences over a matrix state per head, chunk by chunk, on the tensor cores (mma.sync): what the recurrences with
// different weights have in common.  A chunk is up to C tokens of one request that do not cross a multiple of C of the
// request's positions.  q, k and v are rounded to bfloat16; everything else stays 32-bit: the scores are float32 accumulators,
// and an operand that carries a weight or the state (the weighted scores, the weighted values, the chunk's start state) goes
// into its product as three bfloat16 terms whose sum is the float32 value to its last bits.
// What weighs a pair of tokens, a token in the chunk's end state and a token's share of the start state is the includer's.
#pragma once
#include "common.cuh"

namespace {

__device__ __forceinline__ float ret_in(float x, int silu) { return silu ? x / (1.0f + expf(-x)) : x; }
__device__ __forceinline__ float4 ret_in4(float4 x, int silu) {
    return make_float4(ret_in(x.x, silu), ret_in(x.y, silu), ret_in(x.z, silu), ret_in(x.w, silu));
}


constexpr int C = 64;

__host__ __device__ inline int pad4(int x) { return (x + 3) & ~3; }

// Which chunk is CTA ``index``: request b, first row t, tokens n, position of the first token; false beyond the last.
struct ChunkRef { int b, t, n, pos; };
__device__ inline bool find_chunk(const int* __restrict__ q_start, const int* __restrict__ pos_start, int num_requests, int index,
                                  ChunkRef& c) {
    for (int b = 0; b < num_requests; ++b) {
        const int t0 = q_start[b], len = q_start[b + 1] - t0;
        if (len <= 0) continue;
        const int pos0 = pos_start[b];
        const int first = pos0 / C, count = (pos0 + len - 1) / C - first + 1;
        if (index < count) {
            const int lo = max(pos0, (first + index) * C), hi = min(pos0 + len, (first + index + 1) * C);
            c.b = b; c.pos = lo; c.t = t0 + (lo - pos0); c.n = hi - lo;
            return true;
        }
        index -= count;
    }
    return false;
}


constexpr int MT = 256;                  // eight warps
constexpr int SCOLS = 64;                // state columns a CTA of the finish kernel works on

__host__ __device__ inline int pad16(int x) { return (x + 15) & ~15; }
__device__ __forceinline__ uint32_t ret_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ret_ldsm(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(ret_smem(p)));
}
__device__ __forceinline__ void ret_ldsm_t(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(ret_smem(p)));
}
__device__ __forceinline__ void ret_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// x and y as three bfloat16 terms each (a pair a register): 8 + 8 + 8 bits of significand
__device__ __forceinline__ void split3(float x, float y, uint32_t& t1, uint32_t& t2, uint32_t& t3) {
    const float x1 = __bfloat162float(__float2bfloat16_rn(x)), y1 = __bfloat162float(__float2bfloat16_rn(y));
    const float xr = x - x1, yr = y - y1;
    const float x2 = __bfloat162float(__float2bfloat16_rn(xr)), y2 = __bfloat162float(__float2bfloat16_rn(yr));
    t1 = pack_bf16(x1, y1);
    t2 = pack_bf16(x2, y2);
    t3 = pack_bf16(xr - x2, yr - y2);
}

constexpr int LOADS = 8;

// four neighbouring floats of which ``left`` (0 or less: none) are there, zeros for the rest
__device__ __forceinline__ float4 load_four(const float* s, int left, bool vec) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (left >= 4 && vec) return __ldcg(reinterpret_cast<const float4*>(s));
    if (left > 0) x.x = __ldcg(s);
    if (left > 1) x.y = __ldcg(s + 1);
    if (left > 2) x.z = __ldcg(s + 2);
    if (left > 3) x.w = __ldcg(s + 3);
    return x;
}

// C rows of ``width`` float32 columns (rows from n on and columns up to wP are zeros) -> bfloat16 rows of ``stride``
__device__ __forceinline__ void load_rounded(bf16* dst, int stride, const float* __restrict__ src, int ld, int n, int width,
                                             int wP, int silu) {
    const int w4 = wP >> 2;
    const bool vec = ((width | ld) & 3) == 0 && ((uintptr_t)src & 15) == 0;
    for (int e0 = threadIdx.x; e0 < C * w4; e0 += MT * LOADS) {
        float4 x[LOADS];                 // a thread's loads are in flight together
#pragma unroll
        for (int u = 0; u < LOADS; ++u) {
            const int e = e0 + u * MT, i = e / w4, c = (e % w4) << 2;
            x[u] = load_four(src + (size_t)i * ld + c, (i < n && c < width) ? width - c : 0, vec);
        }
#pragma unroll
        for (int u = 0; u < LOADS; ++u) {
            const int e = e0 + u * MT, i = e / w4, c = (e % w4) << 2;
            if (e >= C * w4) continue;
            x[u] = ret_in4(x[u], silu);  // (a silu of zero is zero)
            uint2 v;
            v.x = pack_bf16(x[u].x, x[u].y);
            v.y = pack_bf16(x[u].z, x[u].w);
            *reinterpret_cast<uint2*>(dst + i * stride + c) = v;
        }
    }
}

// The local part of a chunk of n tokens whose q, k and v are the rows at ``q``, ``k``, ``v`` (leading dimensions behind them):
//   orow_i = sum_(j<=i) weights.pair(i, j) (q_i . k_j) v_j   (rows o_ld apart),   Uc = sum_j weights.tail(j) k_j v_j^T
// and, for weights that ask for them (SUMS), weights.row_sum(i, sum_j weights.pair(i, j) (q_i . k_j)).  The rounded k rows
// stay in shared memory at local_keys().  A chunk's weights are ready in shared memory when this is called.
static inline size_t local_mma_smem(int d, int dv) {
    return sizeof(bf16) * ((size_t)2 * C * (pad16(d) + 8) + (size_t)C * (pad16(dv) + 8));
}
__device__ __forceinline__ bf16* local_keys(unsigned char* smraw, int d) { return (bf16*)smraw + C * (pad16(d) + 8); }

template <class W>
__device__ __forceinline__ void chunk_local_mma(unsigned char* smraw, const float* __restrict__ q, int q_ld,
                                                const float* __restrict__ k, int k_ld, const float* __restrict__ v, int v_ld,
                                                int silu, int n, int d, int dv, const W& weights, float* __restrict__ orow,
                                                int o_ld, float* __restrict__ Uc) {
    const int dP = pad16(d), vP = pad16(dv), ks = dP + 8, vs = vP + 8;
    bf16* Qs = (bf16*)smraw;             // [C][ks]
    bf16* Ks = local_keys(smraw, d);     // [C][ks]
    bf16* Vs = Ks + C * ks;              // [C][vs]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    load_rounded(Qs, ks, q, q_ld, n, d, dP, silu);
    load_rounded(Ks, ks, k, k_ld, n, d, dP, silu);
    load_rounded(Vs, vs, v, v_ld, n, dv, vP, silu);
    __syncthreads();
    {   // a warp: 16 rows of the chunk (all their scores) and half of the value columns
        const int rg = warp & 3, cg = warp >> 2;
        float s[8][4];
#pragma unroll
        for (int t = 0; t < 8; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
        for (int kk = 0; kk < dP; kk += 16) {
            uint32_t a[4], b[4];
            ret_ldsm(a, Qs + (rg * 16 + (lane & 15)) * ks + kk + (lane >> 4) * 8);
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                if (t > rg) continue;                    // keys behind every row of the warp
                ret_ldsm(b, Ks + (t * 16 + (lane & 7) + (lane >> 4) * 8) * ks + kk + ((lane >> 3) & 1) * 8);
                ret_mma(s[2 * t], a, b[0], b[1]);
                ret_mma(s[2 * t + 1], a, b[2], b[3]);
            }
        }
        const int i0 = rg * 16 + (lane >> 2), i1 = i0 + 8;
        float sum0 = 0.f, sum1 = 0.f;
        uint32_t a3[4][3][4];                            // the weighted scores as A operands: [16 keys][term][register]
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            if ((t >> 1) > rg) continue;                 // (their terms are not used either)
            const int j = t * 8 + 2 * (lane & 3);
            auto weigh = [&](float x, int i, int jj) { return (jj <= i && jj < n) ? x * weights.pair(i, jj) : 0.f; };
            uint32_t (&r)[3][4] = a3[t >> 1];
            const int hi = (t & 1) * 2;
            const float w00 = weigh(s[t][0], i0, j), w01 = weigh(s[t][1], i0, j + 1);
            const float w10 = weigh(s[t][2], i1, j), w11 = weigh(s[t][3], i1, j + 1);
            split3(w00, w01, r[0][hi], r[1][hi], r[2][hi]);
            split3(w10, w11, r[0][hi + 1], r[1][hi + 1], r[2][hi + 1]);
            if (W::SUMS) { sum0 += w00 + w01; sum1 += w10 + w11; }
        }
        if (W::SUMS) {                                   // the rows' sums: four threads hold a row's keys
            sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1); sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
            sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1); sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
            if (cg == 0 && (lane & 3) == 0) {
                if (i0 < n) weights.row_sum(i0, sum0);
                if (i1 < n) weights.row_sum(i1, sum1);
            }
        }
        const int blocks = vP >> 4, half = (blocks + 1) >> 1;
        const bool out2 = ((dv | o_ld) & 1) == 0 && ((uintptr_t)orow & 7) == 0;
        const int b_lo = cg ? half : 0, b_hi = cg ? blocks : half;
        for (int b0 = b_lo; b0 < b_hi; b0 += 4) {
            float o[8][4];
#pragma unroll
            for (int t = 0; t < 8; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[t][e] = 0.f;
#pragma unroll
            for (int k2 = 0; k2 < 4; ++k2) {
                if (k2 > rg) continue;
#pragma unroll
                for (int bb = 0; bb < 4; ++bb) {
                    if (b0 + bb >= b_hi) continue;
                    uint32_t b[4];
                    ret_ldsm_t(b, Vs + (k2 * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + (b0 + bb) * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int s3 = 2; s3 >= 0; --s3) {    // the small terms first
                        ret_mma(o[2 * bb], a3[k2][s3], b[0], b[1]);
                        ret_mma(o[2 * bb + 1], a3[k2][s3], b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int t = 0; t < 8; ++t) {
                const int col = b0 * 16 + t * 8 + 2 * (lane & 3);
                if (b0 + (t >> 1) >= b_hi) continue;
                if (out2 && col < dv) {
                    if (i0 < n) *reinterpret_cast<float2*>(orow + (size_t)i0 * o_ld + col) = make_float2(o[t][0], o[t][1]);
                    if (i1 < n) *reinterpret_cast<float2*>(orow + (size_t)i1 * o_ld + col) = make_float2(o[t][2], o[t][3]);
                    continue;
                }
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    if (col + e < dv) {
                        if (i0 < n) orow[(size_t)i0 * o_ld + col + e] = o[t][e];
                        if (i1 < n) orow[(size_t)i1 * o_ld + col + e] = o[t][2 + e];
                    }
            }
        }
    }
    // U: a warp takes 16 rows of the state at a time
    for (int m0 = warp * 16; m0 < dP; m0 += 128) {
        for (int n0 = 0; n0 < vP; n0 += 128) {
            float u[16][4];
#pragma unroll
            for (int t = 0; t < 16; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) u[t][e] = 0.f;
            for (int k0 = 0; k0 < C && k0 < n; k0 += 16) {
                uint32_t a[4];
                ret_ldsm_t(a, Ks + (k0 + (lane & 7) + (lane >> 4) * 8) * ks + m0 + ((lane >> 3) & 1) * 8);
                uint32_t a3[3][4];                       // the keys times weights.tail(j) in three terms
                const int j = k0 + 2 * (lane & 3);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const int jj = j + (r >> 1) * 8;
                    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[r]));
                    split3(jj < n ? x.x * weights.tail(jj) : 0.f, jj + 1 < n ? x.y * weights.tail(jj + 1) : 0.f, a3[0][r], a3[1][r], a3[2][r]);
                }
#pragma unroll
                for (int t = 0; t < 8; ++t) {
                    if (n0 + t * 16 >= vP) continue;
                    uint32_t b[4];
                    ret_ldsm_t(b, Vs + (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + n0 + t * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int s3 = 2; s3 >= 0; --s3) {    // the small terms first
                        ret_mma(u[2 * t], a3[s3], b[0], b[1]);
                        ret_mma(u[2 * t + 1], a3[s3], b[2], b[3]);
                    }
                }
            }
            const int r0 = m0 + (lane >> 2), r1 = r0 + 8;
            const bool pairs = (dv & 1) == 0;
#pragma unroll
            for (int t = 0; t < 16; ++t) {
                const int col = n0 + t * 8 + 2 * (lane & 3);
                if (col >= dv) continue;
                if (pairs) {
                    if (r0 < d) *reinterpret_cast<float2*>(Uc + (size_t)r0 * dv + col) = make_float2(u[t][0], u[t][1]);
                    if (r1 < d) *reinterpret_cast<float2*>(Uc + (size_t)r1 * dv + col) = make_float2(u[t][2], u[t][3]);
                } else {
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        if (col + e < dv) {
                            if (r0 < d) Uc[(size_t)r0 * dv + col + e] = u[t][e];
                            if (r1 < d) Uc[(size_t)r1 * dv + col + e] = u[t][2 + e];
                        }
                }
            }
        }
    }
}


// The start state's part, SCOLS value columns from n0 on: orow_i = weights.join(i, (Sc^T q_i), orow_i).  A warp takes eight
// columns of the state Sc [d, dv] and all rows of the chunk: every element of the state is loaded once, straight into the
// registers of the product's B operand (three bfloat16 terms), ahead of the queries where d reaches no further than
// FINISH_ROWS.  Two steps, between which the includer may use the rounded queries in shared memory:
constexpr int FINISH_ROWS = 64, FK = FINISH_ROWS / 16;
static inline size_t finish_mma_smem(int d) { return sizeof(bf16) * (size_t)C * (pad16(d) + 8); }

struct FinishRegs { float s[FK][4]; float local[4][4]; };

__device__ __forceinline__ void finish_load_state(FinishRegs& f, const float* __restrict__ Sc, int d, int dv, int col, int r0) {
    const int kb = 2 * (threadIdx.x & 3);
#pragma unroll
    for (int kk = 0; kk < FK; ++kk)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = r0 + kk * 16 + kb + (e & 1) + (e >> 1) * 8;
            f.s[kk][e] = (r < d && col < dv) ? __ldcg(Sc + (size_t)r * dv + col) : 0.f;
        }
}

__device__ __forceinline__ void chunk_finish_load(FinishRegs& f, unsigned char* smraw, const float* __restrict__ q, int q_ld, int silu,
                                                  int n, int d, int dv, int n0, const float* __restrict__ Sc,
                                                  const float* __restrict__ orow, int o_ld) {
    const int dP = pad16(d), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    finish_load_state(f, Sc, d, dv, n0 + warp * 8 + (lane >> 2), 0);
    const int col = n0 + warp * 8 + 2 * (lane & 3);
    const bool two = ((dv | o_ld) & 1) == 0 && ((uintptr_t)orow & 7) == 0;
#pragma unroll
    for (int rg = 0; rg < 4; ++rg)
#pragma unroll
        for (int hi = 0; hi < 2; ++hi) {                 // (the local part is asked for ahead of the products)
            const int i = rg * 16 + (lane >> 2) + hi * 8;
            const float* p = orow + (size_t)i * o_ld + col;
            float2 x = make_float2(0.f, 0.f);
            if (i < n && two && col < dv) x = __ldcg(reinterpret_cast<const float2*>(p));
            else if (i < n) { if (col < dv) x.x = __ldcg(p); if (col + 1 < dv) x.y = __ldcg(p + 1); }
            f.local[rg][2 * hi] = x.x; f.local[rg][2 * hi + 1] = x.y;
        }
    load_rounded((bf16*)smraw, dP + 8, q, q_ld, n, d, dP, silu);
    __syncthreads();
}

template <class W>
__device__ __forceinline__ void chunk_finish_mma(FinishRegs& f, const unsigned char* smraw, int n, int d, int dv, int n0,
                                                 const float* __restrict__ Sc, const W& weights, float* __restrict__ orow, int o_ld) {
    const int dP = pad16(d), ks = dP + 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bf16* Qs = (const bf16*)smraw;
    float o[4][4];
#pragma unroll
    for (int rg = 0; rg < 4; ++rg)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[rg][e] = 0.f;
    for (int r0 = 0; r0 < dP; r0 += FINISH_ROWS) {
        if (r0 > 0) finish_load_state(f, Sc, d, dv, n0 + warp * 8 + (lane >> 2), r0);
#pragma unroll
        for (int kk = 0; kk < FK; ++kk) {
            if (r0 + kk * 16 >= dP) continue;
            uint32_t t0[3], t1[3];
            split3(f.s[kk][0], f.s[kk][1], t0[0], t0[1], t0[2]);
            split3(f.s[kk][2], f.s[kk][3], t1[0], t1[1], t1[2]);
#pragma unroll
            for (int rg = 0; rg < 4; ++rg) {
                uint32_t a[4];
                ret_ldsm(a, Qs + (rg * 16 + (lane & 15)) * ks + r0 + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int s3 = 2; s3 >= 0; --s3) ret_mma(o[rg], a, t0[s3], t1[s3]);          // the small terms first
            }
        }
    }
    const int col = n0 + warp * 8 + 2 * (lane & 3);
    const bool two = ((dv | o_ld) & 1) == 0 && ((uintptr_t)orow & 7) == 0;
#pragma unroll
    for (int rg = 0; rg < 4; ++rg)
#pragma unroll
        for (int hi = 0; hi < 2; ++hi) {
            const int i = rg * 16 + (lane >> 2) + hi * 8;
            if (i >= n) continue;
            float* p = orow + (size_t)i * o_ld + col;
            const float x = weights.join(i, o[rg][2 * hi], f.local[rg][2 * hi]), y = weights.join(i, o[rg][2 * hi + 1], f.local[rg][2 * hi + 1]);
            if (two && col < dv) *reinterpret_cast<float2*>(p) = make_float2(x, y);
            else { if (col < dv) p[0] = x; if (col + 1 < dv) p[1] = y; }
        }
}

}  // namespace
