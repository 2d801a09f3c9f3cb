// Scalar activations and the sums of a row norm, shared by the kernels of layered models.
#pragma once
#include <cuda_bf16.h>

#include "layered_kernels.h"

namespace tlb {

// __fdividef: two units in the last place, without the branch of the full division; a divisor near overflow gives zero, the limit
__device__ __forceinline__ float sigmoidf(float x) { return __fdividef(1.f, 1.f + expf(-x)); }
__device__ __forceinline__ float siluf(float x) { return __fdividef(x, 1.f + expf(-x)); }
// Both gated activations are z sigmoid(z (a + b z^2)): SiLU with a = 1, b = 0; the tanh form of GELU, z / 2 (1 + tanh(c)) = z sigmoid(2 c).
struct GluConst { float a, b; };
__host__ __device__ inline GluConst glu_const(int act)
{
    const float root = 2.f * 0.79788456080286535588f;        // 2 sqrt(2 / pi)
    return act == GLU_SILU ? GluConst{1.f, 0.f} : GluConst{root, 0.044715f * root};
}
__device__ __forceinline__ float glu_act(const GluConst &c, float z, float up) { return __fdividef(z, 1.f + expf(-z * fmaf(c.b * z, z, c.a))) * up; }
// value that enters a gated recurrence without a normaliser: positive, continuous, slope one above zero
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoidf(u); }

// Inverse root mean square of each of `groups` equal consecutive parts of a row of n values, value(e) giving element e.  All
// threads of the block call; values must be visible to the block.  part: max(warps, groups) floats, inv: groups floats, shared.
constexpr int kMaxNormGroups = 256;
template <typename F>
__device__ __forceinline__ void group_inv_rms(F value, int n, int groups, float eps, float *part, float *inv)
{
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = max(1, warps / groups), len = n / groups;           // warps that share a part
    for (int u = warp; u < groups * per; u += warps) {
        const int g = u / per, s = u - g * per;
        const int beg = g * len + (int)((long long)len * s / per), end = g * len + (int)((long long)len * (s + 1) / per);
        float ss = 0.f;
#pragma unroll 4
        for (int e = beg + lane; e < end; e += 32) { const float v = value(e); ss += v * v; }
#pragma unroll
        for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) part[u] = ss;
    }
    __syncthreads();
    for (int g = threadIdx.x; g < groups; g += blockDim.x) {
        float ss = 0.f;
        for (int s = 0; s < per; s++) ss += part[g * per + s];
        inv[g] = 1.f / sqrtf(ss / (float)len + eps);
    }
    __syncthreads();
}

// part of element e (below 2^22) when a part has 1 / inv_len elements
__device__ __forceinline__ int group_of(int e, float inv_len) { return (int)(((float)e + 0.5f) * inv_len); }

// Chooses the experts of one token; all threads of the block call.  Scores are sigmoids of the logits; with several groups only
// the `keep` groups whose two best scores sum highest take part (ties: the lower index).  sel / weight [top] and the scratch
// (route_scratch_floats) are shared memory.
__host__ __device__ inline int route_scratch_floats(const RouteDesc &r) { return r.experts + 2 * r.groups; }
__device__ __forceinline__ void route_token(const float *logits, const RouteDesc &r, float *scratch, int *sel, float *weight)
{
    const int tid = threadIdx.x, nt = blockDim.x, per = r.experts / r.groups;
    float *s = scratch, *gs = s + r.experts, *kept = gs + r.groups;
    for (int e = tid; e < r.experts; e += nt) s[e] = sigmoidf(__ldcg(logits + e));
    for (int i = tid; i < r.top; i += nt) sel[i] = 0;
    __syncthreads();
    for (int g = tid; g < r.groups; g += nt) {
        float a = 0.f, b = 0.f;                     // scores are positive
        for (int e = g * per; e < (g + 1) * per; e++) {
            const float v = s[e];
            if (v > a) { b = a; a = v; } else if (v > b) b = v;
        }
        gs[g] = a + b;
    }
    __syncthreads();
    for (int g = tid; g < r.groups; g += nt) {
        int rank = 0;
        for (int o = 0; o < r.groups; o++) rank += gs[o] > gs[g] || (gs[o] == gs[g] && o < g);
        kept[g] = rank < r.keep ? 1.f : 0.f;
    }
    __syncthreads();
    for (int e = tid; e < r.experts; e += nt) {
        if (kept[e / per] == 0.f) continue;
        int rank = 0;
        for (int g = 0; g < r.groups; g++) {
            if (kept[g] == 0.f) continue;
            for (int o = g * per; o < (g + 1) * per; o++) rank += s[o] > s[e] || (s[o] == s[e] && o < e);
        }
        if (rank < r.top) sel[rank] = e;
    }
    __syncthreads();
    float sum = 0.f;
    for (int i = 0; i < r.top; i++) sum += s[sel[i]];
    for (int i = tid; i < r.top; i += nt) weight[i] = s[sel[i]] / (sum + 1e-20f) * r.scale;
    __syncthreads();
}

__device__ __forceinline__ void store_actv(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_actv(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_actv4(float *p, float a, float b, float c, float d) { *reinterpret_cast<float4 *>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store_actv4(__nv_bfloat16 *p, float a, float b, float c, float d)
{
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
}

}  // namespace tlb
