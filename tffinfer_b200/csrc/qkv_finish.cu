// What lies between a mixer's merged projection and its token mixing, for mixers whose rotation is not the
// table-driven whole-head rotate-half one of elementwise.cu: one warp per (token, head) of the projection row
//   proj[t] = [q (nq*d) | k (nkv*d) | v (nkv*dv) | ... ]      float32 accumulators or the activation type
// * q and k: the first rot_dims dimensions of a head are rotated by the token's position, the rest pass.  The angle
//   of pair i is float(position) * freq[i] (one float32 product; freq is an array of rot_dims/2 frequencies, so any
//   rescaling of them is the caller's), cos and sin are multiplied by ``magnitude``.  Pairs are (2i, 2i+1)
//   (interleaved) or (i, i + rot_dims/2) (halves).  k is then multiplied by k_scale.
// * ``bias`` (float32, laid out like the row's q | k | v columns, or null) is added to q, k and v ahead of everything else;
//   with ``unit_eps`` > 0 every q and k head is divided, after the rotation, by its root mean square
//   sqrt(mean(x^2) + unit_eps) (an RMS norm without a weight).
// * q goes to q_out [T, nq*d]; k to the token's slot of the paged cache or, without a cache, to k_out [T, nkv*d].
// * v: value mixing across layers.  v_mode 0: as it is.  1: the layer is the source, its values are also kept,
//   unrounded, in v_share [T, nkv*dv] float32.  2: v <- (1 - lambda) v + lambda v_share[t], lambda a float32 scalar on
//   the device.  The (mixed) v goes to the token's slot of the cache; without a cache v is left where it is.
// * head gates: gate_out[t, h] = sigmoid(proj[t, gate_off + h]) for the nq query heads, when gate_out is given.
// With ``clear_input`` every element of the row that the kernel has consumed is set to zero behind the read (q, k,
// the gates, and v where there is a cache to take it): the row is then an accumulator buffer that the next split
// product adds into.
// The cache is [pages, layers, 2, kv heads, page, dc] with dc >= max(d, dv): keys use the first d elements of a
// slot, values the first dv.
// Everything is computed in float32; only the stores round.
#include "common.cuh"

namespace {

template <typename TIN, typename TQ, typename TC>
__global__ void __launch_bounds__(128)
qkv_finish_kernel(TIN* __restrict__ proj, int clear_input, int ld, TQ* __restrict__ q_out, float* __restrict__ k_out,
                  const float* __restrict__ freq, int rot_dims, float magnitude, int interleaved, float k_scale,
                  const int* __restrict__ positions, const int* __restrict__ tok_req,
                  const int* __restrict__ block_table, int table_width,
                  TC* __restrict__ cache, KvLayout L, int layer, int dc,
                  int v_mode, float* __restrict__ v_share, const float* __restrict__ lambda,
                  int gate_off, float* __restrict__ gate_out,
                  int nq, int nkv, int d, int dv, const float* __restrict__ bias, float unit_eps) {
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.y;
    const int head = blockIdx.x * 4 + warp;
    const int heads = nq + 2 * nkv + (gate_out ? 1 : 0);
    if (head >= heads) return;
    const int pos = positions[t];
    pdl_wait();
    TIN* row = proj + (size_t)t * ld;
    const TIN zero = from_f32<TIN>(0.f);
    if (head == nq + 2 * nkv) {                                   // the head gates of this token
        for (int h = lane; h < nq; h += 32) {
            const float g = to_f32<TIN>(row[gate_off + h]);
            if (clear_input) row[gate_off + h] = zero;
            gate_out[(size_t)t * nq + h] = 1.0f / (1.0f + expf(-g));
        }
        return;
    }
    const bool is_q = head < nq, is_k = !is_q && head < nq + nkv;
    TC* slot = nullptr;
    if (!is_q && cache != nullptr) {
        const int kvh = is_k ? head - nq : head - nq - nkv;
        const int page = block_table[(size_t)tok_req[t] * table_width + pos / L.page_size];
        if (page < 0) return;                                     // no page: the host never schedules this
        slot = cache + (size_t)page * L.page_stride + (size_t)layer * L.layer_stride + (is_k ? 0 : L.kv_stride) +
               (size_t)kvh * L.head_stride + (size_t)(pos % L.page_size) * dc;
    }
    if (!is_q && !is_k) {                                         // a value head
        const int kvh = head - nq - nkv;
        TIN* src = row + (size_t)(nq + nkv) * d + (size_t)kvh * dv;
        const float* vb = bias ? bias + (size_t)(nq + nkv) * d + (size_t)kvh * dv : nullptr;
        if (!slot && v_mode != 1) return;                         // nobody takes the values here: they stay in the row
        float* share = v_share ? v_share + (size_t)t * nkv * dv + (size_t)kvh * dv : nullptr;
        const float lam = v_mode == 2 ? *lambda : 0.f;
        for (int i = lane; i < dv; i += 32) {
            float v = to_f32<TIN>(src[i]) + (vb ? vb[i] : 0.f);
            if (clear_input && slot) src[i] = zero;
            if (v_mode == 1) share[i] = v;
            else if (v_mode == 2) v = (1.0f - lam) * v + lam * share[i];
            if (slot) slot[i] = from_f32<TC>(v);
        }
        return;
    }
    TIN* src = row + (size_t)head * d;                            // q heads, then k heads, all of size d
    const float* hb = bias ? bias + (size_t)head * d : nullptr;
    const int half = rot_dims >> 1;
    float ks = is_q ? 1.f : k_scale;
    if (unit_eps > 0.f) {                                         // the head's mean square behind the rotation, first
        float ss = 0.f;
        for (int i = lane; i < half; i += 32) {
            const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
            const float a = to_f32<TIN>(src[ia]) + (hb ? hb[ia] : 0.f), b = to_f32<TIN>(src[ib]) + (hb ? hb[ib] : 0.f);
            float s, c;
            sincosf((float)pos * freq[i], &s, &c);
            s *= magnitude; c *= magnitude;
            const float ra = a * c - b * s, rb = b * c + a * s;
            ss = fmaf(ra, ra, ss); ss = fmaf(rb, rb, ss);
        }
        for (int i = 2 * half + lane; i < d; i += 32) {
            const float a = to_f32<TIN>(src[i]) + (hb ? hb[i] : 0.f);
            ss = fmaf(a, a, ss);
        }
        ss = warp_sum(ss);
        ks *= rsqrtf(ss / (float)d + unit_eps);
    }
    for (int i = lane; i < half; i += 32) {
        const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
        const float a = to_f32<TIN>(src[ia]) + (hb ? hb[ia] : 0.f), b = to_f32<TIN>(src[ib]) + (hb ? hb[ib] : 0.f);
        if (clear_input) { src[ia] = zero; src[ib] = zero; }      // this lane alone reads these two
        float s, c;
        sincosf((float)pos * freq[i], &s, &c);
        s *= magnitude; c *= magnitude;
        const float ra = (a * c - b * s) * ks, rb = (b * c + a * s) * ks;
        if (is_q) {
            q_out[(size_t)t * nq * d + (size_t)head * d + ia] = from_f32<TQ>(ra);
            q_out[(size_t)t * nq * d + (size_t)head * d + ib] = from_f32<TQ>(rb);
        } else if (slot) {
            slot[ia] = from_f32<TC>(ra); slot[ib] = from_f32<TC>(rb);
        } else {
            k_out[(size_t)t * nkv * d + (size_t)(head - nq) * d + ia] = ra;
            k_out[(size_t)t * nkv * d + (size_t)(head - nq) * d + ib] = rb;
        }
    }
    for (int i = 2 * half + lane; i < d; i += 32) {
        const float a = (to_f32<TIN>(src[i]) + (hb ? hb[i] : 0.f)) * ks;
        if (clear_input) src[i] = zero;
        if (is_q) q_out[(size_t)t * nq * d + (size_t)head * d + i] = from_f32<TQ>(a);
        else if (slot) slot[i] = from_f32<TC>(a);
        else k_out[(size_t)t * nkv * d + (size_t)(head - nq) * d + i] = a;
    }
}

// The form for attentions that norm their heads: row = [q (nq*d) | k (nkv*d) | v (nkv*dv)] of float32 accumulators, a warp per
// (token, head), the head in registers, so that the row is read once and everything asked for together:
//   u = row + bias;   q and k: u / rms(u) * norm weight (rms over the head's d elements with ``eps``, weights [d] shared by
//   heads; null: no norm), then turned as above;   v: u of the value columns or, with ``v_is_k`` (no such columns), the key's u
// Cosines and sines of the token are made once a block, ahead of the wait for the kernel before.
constexpr int QF_WARPS = 8, QF_MOST_D = 512;

// Heads of at most 128 elements in groups of four: a lane holds four neighbouring elements (16-byte accesses), a pair's other
// member comes from the lane half/4 away.  A block takes a token, its warps heads in turn.
template <typename TQ>
__global__ void __launch_bounds__(QF_WARPS * 32)
qk_finish4_kernel(float* __restrict__ proj, int clear_input, int ld, TQ* __restrict__ q_out, const float* __restrict__ qw,
                  const float* __restrict__ kw, float eps, const float* __restrict__ bias, int v_is_k,
                  const float* __restrict__ freq, int rot_dims, float magnitude,
                  const int* __restrict__ positions, const int* __restrict__ tok_req, const int* __restrict__ block_table,
                  int table_width, TQ* __restrict__ cache, KvLayout L, int layer, int dc, int nq, int nkv, int d) {
    __shared__ float4 cs[16], sn[16];
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.y, half = rot_dims >> 1, h4 = half >> 2, pos = positions[t], d4 = d >> 2;
    if (threadIdx.x < half) {
        float s, c;
        sincosf((float)pos * freq[threadIdx.x], &s, &c);
        reinterpret_cast<float*>(sn)[threadIdx.x] = s * magnitude; reinterpret_cast<float*>(cs)[threadIdx.x] = c * magnitude;
    }
    const int page = block_table[(size_t)tok_req[t] * table_width + pos / L.page_size];
    TQ* slots = cache + (size_t)page * L.page_stride + (size_t)layer * L.layer_stride + (size_t)(pos % L.page_size) * dc;
    const bool on = lane < d4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), one = make_float4(1.f, 1.f, 1.f, 1.f);
    const float4 wq = on && qw ? reinterpret_cast<const float4*>(qw)[lane] : one;
    const float4 wk = on && kw ? reinterpret_cast<const float4*>(kw)[lane] : one;
    __syncthreads();
    const bool turned = lane < 2 * h4, first = lane < h4;
    const float4 c4 = turned ? cs[first ? lane : lane - h4] : one, s4 = turned ? sn[first ? lane : lane - h4] : zero;
    const int partner = first ? lane + h4 : lane - h4;
    const int heads = nq + nkv;
    pdl_wait();
    float4* row = reinterpret_cast<float4*>(proj + (size_t)t * ld);
    auto store = [](TQ* p, float4 v) {
        if constexpr (sizeof(TQ) == 2) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            uint2 u;
            u.x = *reinterpret_cast<uint32_t*>(&lo); u.y = *reinterpret_cast<uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(p) = u;
        } else {
            *reinterpret_cast<float4*>(p) = v;
        }
    };
    constexpr int N = 4;                                          // heads of a warp in flight
    for (int h0 = blockIdx.x * QF_WARPS + warp; h0 < heads; h0 += N * gridDim.x * QF_WARPS) {
        float4 u[N];
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int head = h0 + n * gridDim.x * QF_WARPS;
            u[n] = on && head < heads ? __ldcg(row + head * d4 + lane) : zero;
        }
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int head = h0 + n * gridDim.x * QF_WARPS;
            if (head >= heads) continue;                          // (the same for the whole warp)
            if (on && bias) {
                const float4 b = reinterpret_cast<const float4*>(bias)[head * d4 + lane];
                u[n].x += b.x; u[n].y += b.y; u[n].z += b.z; u[n].w += b.w;
            }
            if (on && clear_input) row[head * d4 + lane] = zero;
            const bool is_q = head < nq;
            float4 v = u[n];
            if (qw) {
                const float ss = warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w);
                const float rs = rsqrtf(ss / (float)d + eps);
                const float4 w = is_q ? wq : wk;
                v = make_float4(v.x * rs * w.x, v.y * rs * w.y, v.z * rs * w.z, v.w * rs * w.w);
            }
            float4 o;                                             // (every lane takes part in the exchange)
            o.x = __shfl_sync(0xffffffffu, v.x, partner & 31); o.y = __shfl_sync(0xffffffffu, v.y, partner & 31);
            o.z = __shfl_sync(0xffffffffu, v.z, partner & 31); o.w = __shfl_sync(0xffffffffu, v.w, partner & 31);
            if (turned) {
                const float sg = first ? -1.f : 1.f;
                v = make_float4(v.x * c4.x + sg * o.x * s4.x, v.y * c4.y + sg * o.y * s4.y, v.z * c4.z + sg * o.z * s4.z,
                                v.w * c4.w + sg * o.w * s4.w);
            }
            if (!on) continue;
            if (is_q) { store(q_out + ((size_t)t * nq + head) * d + 4 * lane, v); continue; }
            if (page < 0) continue;                               // no page: the host never schedules this
            TQ* slot = slots + (size_t)(head - nq) * L.head_stride;
            store(slot + 4 * lane, v);
            if (v_is_k) store(slot + L.kv_stride + 4 * lane, u[n]);
        }
    }
    if (v_is_k || page < 0) return;
    for (int g = blockIdx.x * QF_WARPS + warp; g < nkv; g += gridDim.x * QF_WARPS) {          // values of their own, of d elements
        if (!on) continue;
        float4 u = __ldcg(row + (heads + g) * d4 + lane);
        if (bias) {
            const float4 b = reinterpret_cast<const float4*>(bias)[(heads + g) * d4 + lane];
            u.x += b.x; u.y += b.y; u.z += b.z; u.w += b.w;
        }
        if (clear_input) row[(heads + g) * d4 + lane] = zero;
        store(slots + (size_t)g * L.head_stride + L.kv_stride + 4 * lane, u);
    }
}

template <typename TQ, int RJ>        // RJ: registers an element array takes, d <= 32 * RJ
__global__ void __launch_bounds__(QF_WARPS * 32)
qk_finish_kernel(float* __restrict__ proj, int clear_input, int ld, TQ* __restrict__ q_out, const float* __restrict__ qw,
                 const float* __restrict__ kw, float eps, const float* __restrict__ bias, int v_is_k,
                 const float* __restrict__ freq, int rot_dims, float magnitude, int interleaved,
                 const int* __restrict__ positions, const int* __restrict__ tok_req, const int* __restrict__ block_table,
                 int table_width, TQ* __restrict__ cache, KvLayout L, int layer, int dc, int nq, int nkv, int d, int dv) {
    __shared__ float cs[QF_MOST_D / 2], sn[QF_MOST_D / 2];
    constexpr int PJ = (RJ + 1) / 2;
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.y, head = blockIdx.x * QF_WARPS + warp;
    const int half = rot_dims >> 1, pos = positions[t];
    for (int i = threadIdx.x; i < half; i += QF_WARPS * 32) {
        float s, c;
        sincosf((float)pos * freq[i], &s, &c);
        sn[i] = s * magnitude; cs[i] = c * magnitude;
    }
    __syncthreads();
    const bool is_q = head < nq, is_k = !is_q && head < nq + nkv;
    TQ* slot = nullptr;                                           // the head's key slot (a value lies kv_stride further)
    if (!is_q && head < nq + (v_is_k ? nkv : 2 * nkv)) {
        const int page = block_table[(size_t)tok_req[t] * table_width + pos / L.page_size];
        if (page >= 0)                                            // no page: the host never schedules this
            slot = cache + (size_t)page * L.page_stride + (size_t)layer * L.layer_stride +
                   (size_t)(is_k ? head - nq : head - nq - nkv) * L.head_stride + (size_t)(pos % L.page_size) * dc;
    }
    pdl_wait();
    if (!is_q && !slot) return;
    float* row = proj + (size_t)t * ld;
    if (!is_q && !is_k) {                                         // a value head
        const int col = (nq + nkv) * d + (head - nq - nkv) * dv;
        for (int i = lane; i < dv; i += 32) {
            const float v = __ldcg(row + col + i) + (bias ? bias[col + i] : 0.f);
            if (clear_input) row[col + i] = 0.f;
            slot[L.kv_stride + i] = from_f32<TQ>(v);
        }
        return;
    }
    float* src = row + (size_t)head * d;
    const float* hb = bias ? bias + (size_t)head * d : nullptr;
    const float* hw = is_q ? qw : kw;
    float a[PJ], b[PJ], c[RJ];                                    // the turned pairs and the elements that pass
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
        const int i = lane + 32 * j, ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
        a[j] = i < half ? __ldcg(src + ia) + (hb ? hb[ia] : 0.f) : 0.f;
        b[j] = i < half ? __ldcg(src + ib) + (hb ? hb[ib] : 0.f) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < RJ; ++j) {
        const int i = 2 * half + lane + 32 * j;
        c[j] = i < d ? __ldcg(src + i) + (hb ? hb[i] : 0.f) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < PJ; ++j) { ss = fmaf(a[j], a[j], ss); ss = fmaf(b[j], b[j], ss); }
#pragma unroll
    for (int j = 0; j < RJ; ++j) ss = fmaf(c[j], c[j], ss);
    float rs = 1.f;
    if (hw) rs = rsqrtf(warp_sum(ss) / (float)d + eps);
    TQ* dst = is_q ? q_out + (size_t)t * nq * d + (size_t)head * d : slot;
    TQ* val = !is_q && v_is_k ? slot + L.kv_stride : nullptr;
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
        const int i = lane + 32 * j, ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
        if (i >= half) continue;
        if (clear_input) { src[ia] = 0.f; src[ib] = 0.f; }
        if (val) { val[ia] = from_f32<TQ>(a[j]); val[ib] = from_f32<TQ>(b[j]); }
        const float u = hw ? a[j] * rs * hw[ia] : a[j], v = hw ? b[j] * rs * hw[ib] : b[j];
        dst[ia] = from_f32<TQ>(u * cs[i] - v * sn[i]);
        dst[ib] = from_f32<TQ>(v * cs[i] + u * sn[i]);
    }
#pragma unroll
    for (int j = 0; j < RJ; ++j) {
        const int i = 2 * half + lane + 32 * j;
        if (i >= d) continue;
        if (clear_input) src[i] = 0.f;
        if (val) val[i] = from_f32<TQ>(c[j]);
        dst[i] = from_f32<TQ>(hw ? c[j] * rs * hw[i] : c[j]);
    }
}

}  // namespace

// proj float32 [num_tokens, ld]; q_out and the cache have q_dt (0 float32, 1 bfloat16); qw, kw float32 [d] or both null;
// bias float32 over the row's columns or null; v_is_k: the row has no value columns, dv = d.
TFF_API int tff_qk_finish(
    float* proj, int clear_input, int ld, void* q_out, int q_dt, const float* qw, const float* kw, float eps, const float* bias,
    int v_is_k, const float* freq, int rot_dims, float magnitude, int interleaved, const int* positions, const int* tok_req,
    const int* block_table, int table_width, void* cache, int cache_layers, int layer, int page_size, int dc,
    int num_tokens, int nq, int nkv, int d, int dv, cudaStream_t stream) {
    if (num_tokens <= 0) return TFF_OK;
    if (!proj || !q_out || !cache || !block_table || !positions || !tok_req || nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0 ||
        rot_dims < 0 || rot_dims > d || (rot_dims & 1) || (rot_dims > 0 && !freq) || page_size <= 0 || dc < d || dc < dv ||
        (v_is_k && dv != d) || (qw != nullptr) != (kw != nullptr) || (qw && !(eps > 0.f)))
        return TFF_ERR_BAD_ARGUMENT;
    if (d > QF_MOST_D || num_tokens > 65535) return TFF_ERR_UNSUPPORTED;
    const KvLayout L = make_kv_layout(cache_layers, nkv, page_size, dc);
    const int heads = nq + (v_is_k ? nkv : 2 * nkv);
    const dim3 grid((heads + QF_WARPS - 1) / QF_WARPS, num_tokens);
    const int elt = q_dt == 1 ? 2 : 4;
    if (d <= 128 && d % 4 == 0 && dv == d && rot_dims % 8 == 0 && !interleaved && ld % 4 == 0 && dc % 4 == 0 &&
        (((uintptr_t)proj | (uintptr_t)bias | (uintptr_t)qw | (uintptr_t)kw) & 15) == 0 &&
        (((uintptr_t)q_out | (uintptr_t)cache) & (4 * elt - 1)) == 0) {
        const dim3 grid4(num_tokens > 256 ? 1 : (nq + nkv + QF_WARPS - 1) / QF_WARPS, num_tokens);
#define TFF_QF4(TQ)                                                                                                   \
        return tff_launch_pdl(qk_finish4_kernel<TQ>, grid4, dim3(QF_WARPS * 32), 0, stream, proj, clear_input, ld, (TQ*)q_out, \
                              qw, kw, eps, bias, v_is_k, freq, rot_dims, magnitude, positions, tok_req, block_table,  \
                              table_width, (TQ*)cache, L, layer, dc, nq, nkv, d)
        if (q_dt == 1) TFF_QF4(bf16);
        TFF_QF4(float);
#undef TFF_QF4
    }
#define TFF_QF(TQ, RJ)                                                                                                \
    return tff_launch_pdl(qk_finish_kernel<TQ, RJ>, grid, dim3(QF_WARPS * 32), 0, stream, proj, clear_input, ld, (TQ*)q_out, \
                          qw, kw, eps, bias, v_is_k, freq, rot_dims, magnitude, interleaved, positions, tok_req,      \
                          block_table, table_width, (TQ*)cache, L, layer, dc, nq, nkv, d, dv)
    if (q_dt == 1) { if (d <= 128) TFF_QF(bf16, 4); TFF_QF(bf16, 16); }
    if (d <= 128) TFF_QF(float, 4);
    TFF_QF(float, 16);
#undef TFF_QF
}

// in_dt, q_dt, cache_dt: 0 = float32, 1 = bfloat16.  bias: float32 [nq*d + nkv*d + nkv*dv] or null; unit_eps: 0 = no norm.  q_out has q_dt; the cache cache_dt; k_out and v_share are float32.
TFF_API int tff_qkv_finish(
    void* proj, int in_dt, int clear_input, int ld, void* q_out, int q_dt, float* k_out,
    const float* freq, int rot_dims, float magnitude, int interleaved, float k_scale,
    const int* positions, const int* tok_req, const int* block_table, int table_width,
    void* cache, int cache_dt, int cache_layers, int layer, int page_size, int dc,
    int v_mode, float* v_share, const float* lambda, int gate_off, float* gate_out,
    int num_tokens, int nq, int nkv, int d, int dv, const float* bias, float unit_eps, cudaStream_t stream) {
    if (num_tokens <= 0) return TFF_OK;
    if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || rot_dims < 0 || rot_dims > d || (rot_dims & 1) || !proj || !q_out)
        return TFF_ERR_BAD_ARGUMENT;
    if (rot_dims > 0 && !freq) return TFF_ERR_BAD_ARGUMENT;
    if (cache && (!block_table || page_size <= 0 || dc < d || dc < dv)) return TFF_ERR_BAD_ARGUMENT;
    if (!cache && !k_out) return TFF_ERR_BAD_ARGUMENT;
    if ((v_mode == 1 || v_mode == 2) && !v_share) return TFF_ERR_BAD_ARGUMENT;
    if (v_mode == 2 && !lambda) return TFF_ERR_BAD_ARGUMENT;
    if (v_mode < 0 || v_mode > 2) return TFF_ERR_BAD_ARGUMENT;
    if (gate_out && gate_off < 0) return TFF_ERR_BAD_ARGUMENT;
    const KvLayout L = make_kv_layout(cache_layers, nkv, page_size > 0 ? page_size : 1, dc > 0 ? dc : 1);
    const int heads = nq + 2 * nkv + (gate_out ? 1 : 0);
    dim3 grid((heads + 3) / 4, num_tokens);
#define TFF_FIN(TIN, TQ, TC)                                                                                       \
    return tff_launch_pdl(qkv_finish_kernel<TIN, TQ, TC>, grid, dim3(128), 0, stream, (TIN*)proj, clear_input, ld, (TQ*)q_out, \
                          k_out, freq, rot_dims, magnitude, interleaved, k_scale, positions, tok_req, block_table,   \
                          table_width, (TC*)cache, L, layer, dc, v_mode, v_share, lambda, gate_off, gate_out, nq,     \
                          nkv, d, dv, bias, unit_eps)
    if (in_dt == 0 && q_dt == 0 && cache_dt == 0) TFF_FIN(float, float, float);
    if (in_dt == 0 && q_dt == 1 && cache_dt == 1) TFF_FIN(float, bf16, bf16);
    if (in_dt == 0 && q_dt == 0 && cache_dt == 1) TFF_FIN(float, float, bf16);
    if (in_dt == 1 && q_dt == 1 && cache_dt == 1) TFF_FIN(bf16, bf16, bf16);
#undef TFF_FIN
    return TFF_ERR_BAD_ARGUMENT;
}
