// The norm and the gate behind a recurrence or a linear attention: RMS norms over groups of columns of float32 rows, a
// weight, and a gate read from columns of other float32 rows (the mixer's merged projection).
#include "common.cuh"

namespace {

// out[t, out_off + c] = out_scale * y[c], c over ``width`` columns in groups of ``gs``:
//   gate_first 0:  y = o / rms_group(o) * w[c % wlen] * f(g[c])
//   gate_first 1:  u = o * f(g[c]),  y = u / rms_group(u) * w[c % wlen]
// with f silu (gate_act 0) or the sigmoid (1).
// o float32 [T, width]; g the columns g_off .. of the float32 rows ``gate`` (ld g_ld).  A warp works on a group at a time
// (WIDE false: blockIdx.y picks eight groups of a token) or, for groups of 512 columns and more, a whole block (WIDE
// true: blockIdx.y is the group); either way a group's sum of squares is added in an order that gs alone fixes.  With
// ``clear_lo`` < ``clear_hi`` those columns of the token's row of ``gate`` are set to zero
// (an accumulator buffer that the next split product adds into): a gate by the
// thread that has read it for the last time, the columns beside the gate's by the token's blocks in turn (the kernels
// ahead have read those).
__device__ __forceinline__ float norm_gate(float z, int act) {
    return (act == 0 ? z : 1.f) / (1.f + expf(-z));
}

constexpr int KEEP = 16;        // elements a thread keeps in registers

template <typename TO, bool WIDE>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ o, int width, int gs, float* __restrict__ gate, int g_ld, int g_off,
                  const float* __restrict__ w, int wlen, float eps, int gate_first, int gate_act, int clear_lo, int clear_hi,
                  TO* __restrict__ out, int out_ld, int out_off, float out_scale) {
    __shared__ float red[32];
    pdl_launch_dependents();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* orow = o + (size_t)t * width;
    float* grow = gate + (size_t)t * g_ld + g_off;
    TO* dst = out + (size_t)t * out_ld + out_off;
    const int g = WIDE ? blockIdx.y : blockIdx.y * 8 + warp;
    const int first = WIDE ? threadIdx.x : lane, step = WIDE ? 256 : 32;
    pdl_wait();
    for (int c = clear_lo + blockIdx.y * 256 + threadIdx.x; c < clear_hi; c += gridDim.y * 256)
        if (c < g_off || c >= g_off + width) gate[(size_t)t * g_ld + c] = 0.f;
    if (!WIDE && g >= width / gs) return;
    const int c0 = g * gs;
    float ss = 0.f;
    if (gs <= step * KEEP) {                     // the group's values and gates stay in registers, all loads in flight together
        float u[KEEP], z[KEEP];
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            const int i = first + k * step;
            u[k] = i < gs ? __ldcg(orow + c0 + i) : 0.f;
            z[k] = i < gs ? __ldcg(grow + c0 + i) : 0.f;
        }
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            if (first + k * step >= gs) continue;
            z[k] = norm_gate(z[k], gate_act);
            if (gate_first) u[k] *= z[k];
            ss = fmaf(u[k], u[k], ss);
        }
        ss = WIDE ? block_sum<256>(ss, red) : warp_sum(ss);
        const float inv = rsqrtf(ss / (float)gs + eps);
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            const int i = first + k * step, c = c0 + i;
            if (i >= gs) continue;
            if (g_off + c >= clear_lo && g_off + c < clear_hi) grow[c] = 0.f;
            const float y = (u[k] * inv) * w[c % wlen];
            dst[c] = from_f32<TO>((gate_first ? y : y * z[k]) * out_scale);
        }
        return;
    }
    for (int c = c0 + first; c < c0 + gs; c += step) {
        float u = __ldcg(orow + c);
        if (gate_first) u *= norm_gate(__ldcg(grow + c), gate_act);
        ss = fmaf(u, u, ss);
    }
    ss = WIDE ? block_sum<256>(ss, red) : warp_sum(ss);
    const float inv = rsqrtf(ss / (float)gs + eps);
    for (int c = c0 + first; c < c0 + gs; c += step) {
        const float sg = norm_gate(__ldcg(grow + c), gate_act);
        if (g_off + c >= clear_lo && g_off + c < clear_hi) grow[c] = 0.f;
        float y = __ldcg(orow + c);
        y = gate_first ? (y * sg) * inv * w[c % wlen] : (y * inv) * w[c % wlen] * sg;
        dst[c] = from_f32<TO>(y * out_scale);
    }
}

// Narrow groups in whole fours: a lane holds G4 times four neighbouring elements (16-byte accesses), a warp a group.
template <typename TO, int G4>
__global__ void __launch_bounds__(256)
gated_norm4_kernel(const float* __restrict__ o, int width, int gs, float* __restrict__ gate, int g_ld, int g_off,
                   const float* __restrict__ w, int wlen, float eps, int gate_first, int gate_act, int clear_lo, int clear_hi,
                   TO* __restrict__ out, int out_ld, int out_off, float out_scale) {
    pdl_launch_dependents();
    const int t = blockIdx.x, lane = threadIdx.x & 31, g = blockIdx.y * 8 + (threadIdx.x >> 5), n4 = gs >> 2;
    float* grow = gate + (size_t)t * g_ld;
    pdl_wait();
    for (int c = clear_lo + blockIdx.y * 256 + threadIdx.x; c < clear_hi; c += gridDim.y * 256)
        if (c < g_off || c >= g_off + width) grow[c] = 0.f;
    if (g >= width / gs) return;
    const float4* o4 = reinterpret_cast<const float4*>(o + (size_t)t * width + g * gs);
    float4* z4 = reinterpret_cast<float4*>(grow + g_off + g * gs);
    float u[G4][4], z[G4][4];
#pragma unroll
    for (int k = 0; k < G4; ++k) {
        const int i = lane + 32 * k;
        const float4 a = i < n4 ? __ldcg(o4 + i) : make_float4(0.f, 0.f, 0.f, 0.f), b = i < n4 ? __ldcg(z4 + i) : a;
        u[k][0] = a.x; u[k][1] = a.y; u[k][2] = a.z; u[k][3] = a.w;
        z[k][0] = b.x; z[k][1] = b.y; z[k][2] = b.z; z[k][3] = b.w;
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < G4; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            z[k][e] = norm_gate(z[k][e], gate_act);
            if (gate_first) u[k][e] *= z[k][e];
            ss = fmaf(u[k][e], u[k][e], ss);             // (elements beyond the group are zeros)
        }
    const float inv = rsqrtf(warp_sum(ss) / (float)gs + eps);
#pragma unroll
    for (int k = 0; k < G4; ++k) {
        const int i = lane + 32 * k, c = g * gs + 4 * i;
        if (i >= n4) continue;
        if (g_off + c >= clear_lo && g_off + c < clear_hi) z4[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 ww = *reinterpret_cast<const float4*>(w + c % wlen);
        const float wv[4] = {ww.x, ww.y, ww.z, ww.w};
        float r[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float y = (u[k][e] * inv) * wv[e];
            r[e] = (gate_first ? y : y * z[k][e]) * out_scale;
        }
        TO* dst = out + (size_t)t * out_ld + out_off + c;
        if constexpr (sizeof(TO) == 2) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
            uint2 v;
            v.x = *reinterpret_cast<uint32_t*>(&lo); v.y = *reinterpret_cast<uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(dst) = v;
        } else {
            *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
        }
    }
}

}  // namespace

// out_dt: 0 = float32, 1 = bfloat16.
TFF_API int tff_gated_norm(const float* o, int width, int gs, float* gate, int g_ld, int g_off, const float* w, int wlen,
                           float eps, int gate_first, int gate_act, void* out, int out_dt, int out_ld, int out_off,
                           float out_scale, int clear, int clear_lo, int clear_hi, int num_tokens, cudaStream_t stream) {
    if (num_tokens <= 0) return TFF_OK;
    if (!o || !gate || !w || !out || width <= 0 || gs <= 0 || width % gs || wlen <= 0 || !(eps > 0.f) ||
        (gate_act != 0 && gate_act != 1) ||
        (clear && (clear_lo < 0 || clear_hi > g_ld || clear_lo > clear_hi)))
        return TFF_ERR_BAD_ARGUMENT;
    const bool wide = gs >= 512;
    const dim3 grid(num_tokens, wide ? width / gs : (width / gs + 7) / 8);
    int st;
    if (!clear) clear_lo = clear_hi = 0;
    const int elt = out_dt == 1 ? 2 : 4;
    if (!wide && gs % 4 == 0 && wlen % 4 == 0 && g_ld % 4 == 0 && g_off % 4 == 0 && out_ld % 4 == 0 && out_off % 4 == 0 &&
        clear_lo % 4 == 0 && clear_hi % 4 == 0 && (((uintptr_t)o | (uintptr_t)gate | (uintptr_t)w) & 15) == 0 &&
        ((uintptr_t)out & (4 * elt - 1)) == 0) {
#define TFF_GN4(TO, G4)                                                                                               \
        return tff_launch_pdl(gated_norm4_kernel<TO, G4>, grid, dim3(256), 0, stream, o, width, gs, gate, g_ld, g_off, w, wlen, \
                              eps, gate_first, gate_act, clear_lo, clear_hi, (TO*)out, out_ld, out_off, out_scale)
        if (out_dt == 1) { if (gs <= 128) TFF_GN4(bf16, 1); TFF_GN4(bf16, 4); }
        if (gs <= 128) TFF_GN4(float, 1);
        TFF_GN4(float, 4);
#undef TFF_GN4
    }
#define TFF_GN(TO, WIDE)                                                                                              \
    st = tff_launch_pdl(gated_norm_kernel<TO, WIDE>, grid, dim3(256), 0, stream, o, width, gs, gate, g_ld,            \
                        g_off, w, wlen, eps, gate_first, gate_act, clear_lo, clear_hi, (TO*)out, out_ld, out_off, out_scale)
    if (out_dt == 1) { if (wide) TFF_GN(bf16, true); else TFF_GN(bf16, false); }
    else { if (wide) TFF_GN(float, true); else TFF_GN(float, false); }
#undef TFF_GN
    return st;
}
