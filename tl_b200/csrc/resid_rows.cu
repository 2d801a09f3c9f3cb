// The residual step of designs that norm what a sublayer adds, over rows: gate, norm in groups, addition and the next sublayer's norm
// in one pass; the sum over a token's experts comes in front where the sublayer is a mixture.
#include <algorithm>

#include "act.cuh"
#include "layered_kernels.h"

namespace tlb {

namespace {

struct ResidNormParams {
    float *x;
    int width, groups;
    float offset, eps;
    const float *y, *gate;
    int ld_gate;
    const float *post_w, *norm_w;
    int ldo;
    MoeRows moe;
};

template <typename TA>
__global__ void __launch_bounds__(256) resid_norm_rows_kernel(const ResidNormParams p, TA *__restrict__ out)
{
    extern __shared__ __align__(16) float row[];
    __shared__ float part[kMaxNormGroups], inv[kMaxNormGroups];
    __shared__ int s_slot[kMaxTop];
    __shared__ float s_w[kMaxTop];
    const int tid = threadIdx.x, W = p.width, len = W / p.groups;
    const float inv_len = 1.f / (float)len;
    const size_t t = blockIdx.x;
    float *x = p.x + t * W;
    const bool v4 = W % 4 == 0 && len % 4 == 0;
    auto at = [&](int e) { return row[e]; };
    if (p.y || p.moe.part) {
        const float *gate = p.gate ? p.gate + t * p.ld_gate : nullptr;
        auto gated = [&](float v, int e) { return gate ? v * sigmoidf(gate[e]) : v; };
        if (p.moe.part) {
            const MoeRows &m = p.moe;
            for (int i = tid; i < m.top; i += 256) { s_slot[i] = m.slot[t * m.top + i]; s_w[i] = m.weight[t * m.top + i]; }
            __syncthreads();
            const float sw = m.shared_gate ? sigmoidf(m.shared_gate[t * m.ld_shared_gate]) : 1.f;
            if (v4) {
                for (int e = tid * 4; e < W; e += 1024) {
                    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
                    for (int i = 0; i < m.top; i++) {
                        const float4 q = *reinterpret_cast<const float4 *>(m.part + (size_t)s_slot[i] * W + e);
                        const float w = s_w[i];
                        a.x = fmaf(w, q.x, a.x); a.y = fmaf(w, q.y, a.y); a.z = fmaf(w, q.z, a.z); a.w = fmaf(w, q.w, a.w);
                    }
                    if (m.shared) {
                        const float4 q = *reinterpret_cast<const float4 *>(m.shared + t * W + e);
                        a.x = fmaf(sw, q.x, a.x); a.y = fmaf(sw, q.y, a.y); a.z = fmaf(sw, q.z, a.z); a.w = fmaf(sw, q.w, a.w);
                    }
                    *reinterpret_cast<float4 *>(row + e) = make_float4(gated(a.x, e), gated(a.y, e + 1), gated(a.z, e + 2), gated(a.w, e + 3));
                }
            } else {
                for (int e = tid; e < W; e += 256) {
                    float a = 0.f;
                    for (int i = 0; i < m.top; i++) a = fmaf(s_w[i], m.part[(size_t)s_slot[i] * W + e], a);
                    if (m.shared) a = fmaf(sw, m.shared[t * W + e], a);
                    row[e] = gated(a, e);
                }
            }
        } else if (v4) {
            for (int e = tid * 4; e < W; e += 1024) {
                const float4 q = *reinterpret_cast<const float4 *>(p.y + t * W + e);
                *reinterpret_cast<float4 *>(row + e) = make_float4(gated(q.x, e), gated(q.y, e + 1), gated(q.z, e + 2), gated(q.w, e + 3));
            }
        } else {
            for (int e = tid; e < W; e += 256) row[e] = gated(p.y[t * W + e], e);
        }
        __syncthreads();
        group_inv_rms(at, W, p.groups, p.eps, part, inv);
        if (v4) {
            for (int e = tid * 4; e < W; e += 1024) {
                const float f = inv[group_of(e, inv_len)];
                const float4 a = *reinterpret_cast<const float4 *>(row + e), w = *reinterpret_cast<const float4 *>(p.post_w + e);
                float4 v = *reinterpret_cast<const float4 *>(x + e);
                v.x += a.x * f * (w.x + p.offset); v.y += a.y * f * (w.y + p.offset); v.z += a.z * f * (w.z + p.offset); v.w += a.w * f * (w.w + p.offset);
                *reinterpret_cast<float4 *>(x + e) = v;
                *reinterpret_cast<float4 *>(row + e) = v;
            }
        } else {
            for (int e = tid; e < W; e += 256) x[e] = row[e] = x[e] + row[e] * inv[group_of(e, inv_len)] * (p.post_w[e] + p.offset);
        }
    } else {
        for (int e = tid; e < W; e += 256) row[e] = x[e];
    }
    if (!p.norm_w) return;
    __syncthreads();
    group_inv_rms(at, W, p.groups, p.eps, part, inv);
    TA *o = out + t * p.ldo;
    if (v4 && p.ldo % 4 == 0) {
        for (int e = tid * 4; e < W; e += 1024) {
            const float f = inv[group_of(e, inv_len)];
            const float4 a = *reinterpret_cast<const float4 *>(row + e), w = *reinterpret_cast<const float4 *>(p.norm_w + e);
            store_actv4(o + e, a.x * f * (w.x + p.offset), a.y * f * (w.y + p.offset), a.z * f * (w.z + p.offset), a.w * f * (w.w + p.offset));
        }
    } else {
        for (int e = tid; e < W; e += 256) store_actv(o + e, row[e] * inv[group_of(e, inv_len)] * (p.norm_w[e] + p.offset));
    }
}

tlb_status launched(const char *what)
{
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return cuda_fail(e, what);
    count_launch();
    return TLB_OK;
}

template <typename TA>
tlb_status run_resid(const ResidNormParams &p, int T, void *out)
{
    const size_t smem = (size_t)p.width * sizeof(float);
    static size_t allowed = 40 << 10;
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(resid_norm_rows_kernel<TA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    resid_norm_rows_kernel<TA><<<T, 256, smem, ctx()->stream>>>(p, (TA *)out);
    return launched("residual norm launch");
}

}  // namespace

tlb_status launch_resid_norm_rows(const ResidNormJob &j, bool f32)
{
    ResidNormParams p = {};
    p.x = j.x; p.width = j.width; p.groups = j.groups; p.offset = j.offset; p.eps = j.eps;
    p.y = j.y; p.gate = j.gate; p.ld_gate = j.ld_gate; p.post_w = j.post_w; p.norm_w = j.norm_w; p.ldo = j.ldo;
    if (j.moe) p.moe = *j.moe;
    return f32 ? run_resid<float>(p, j.T, j.out) : run_resid<__nv_bfloat16>(p, j.T, j.out);
}

}  // namespace tlb
