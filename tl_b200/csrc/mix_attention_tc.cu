// Prompt attention with window, distance bias and sink over an f16 cache on the tensor cores (mma.sync m16n8k16, f32
// accumulation): one CTA per (64 queries, head), each warp 16 queries; tiles of 64 cache rows by cp.async, one ahead; only tiles
// that hold a key some query of the CTA sees are visited.  Scores and weights stay in 32 bits: the second product takes a
// weight as two f16 terms (value and remainder, 22 bits together), so nothing rounds it to 16 bits on its way to V.
// The bias is a table by distance; a tile needs 127 consecutive entries of it, staged beside the keys.
#include <algorithm>

#include "act.cuh"
#include "layered_kernels.h"
#include "qmv_common.cuh"

namespace tlb {

namespace {

constexpr int kQ = 64, kK = 64, kThreads = 128;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ uint32_t pack_h2(float a, float b)
{
    const __half2 h = __floats2half2_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&h);
}
// the part of (a, b) that the f16 pair h does not hold
__device__ __forceinline__ uint32_t rest_h2(float a, float b, uint32_t h)
{
    const float2 f = h2_to_f2(h);
    return pack_h2(a - f.x, b - f.y);
}
__device__ __forceinline__ float clamp_h(float v) { return fminf(fmaxf(v, -65504.f), 65504.f); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ float exp2_approx(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// halves of shared memory: two buffers of a K and a V tile, the queries; then the bias entries of two tiles
template <int P> constexpr size_t attn_smem() { return (size_t)(4 * kK + kQ) * (P + 8) * 2 + 2 * 128 * sizeof(float); }

template <int P>     // head sizes padded to P
__global__ void __launch_bounds__(kThreads, P <= 128 ? 2 : 1)
mix_attn_tc_kernel(const MixAttn a, int seq, int T, int pos0, __nv_bfloat16 *__restrict__ out, int ldo)
{
    constexpr int RS = P + 8;
    extern __shared__ __align__(16) __half at_smem[];
    __half *sQ = at_smem + 4 * kK * RS;
    float *s_bias = reinterpret_cast<float *>(sQ + kQ * RS);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
    const int h = blockIdx.y, kvh = h / (a.H / a.KVH);
    const int qtile = (int)(gridDim.x - 1 - blockIdx.x), qb = qtile * kQ, q0 = qb + warp * 16;
    const __half *kc = reinterpret_cast<const __half *>(a.kcache) + (size_t)seq * a.seq_stride_k + (size_t)kvh * a.max_seq * a.ldk;
    const __half *vc = reinterpret_cast<const __half *>(a.vcache) + (size_t)seq * a.seq_stride_v + (size_t)kvh * a.max_seq * a.ldv;

    // padding columns stay zero
    for (int i = tid; i < (4 * kK + kQ) * RS / 8; i += kThreads) reinterpret_cast<uint4 *>(at_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    for (int i = tid; i < kQ * a.D; i += kThreads) {
        const int r = i / a.D, d = i - r * a.D;
        if (qb + r < T) sQ[r * RS + d] = __float2half_rn(clamp_h(a.proj[(size_t)(qb + r) * a.ldp + (size_t)h * a.D + d]));
    }
    const int last_q = min(qb + kQ, T) - 1;
    const int t_end = (pos0 + last_q) / kK + 1, t_begin = max(0, pos0 + qb - a.window + 1) / kK;
    auto tile_async = [&](int t) {
        __half *ks = at_smem + (size_t)(t & 1) * 2 * kK * RS, *vs = ks + kK * RS;
        constexpr int CW = P <= 128 ? 16 : 32;               // threads per row
        const int ch = tid % CW;
        for (int key = tid / CW; key < kK; key += kThreads / CW) {
            const size_t row = min(t * kK + key, a.max_seq - 1);
            if (ch * 8 < a.ldk) cp_async16(smem_u32(ks + key * RS + ch * 8), kc + row * a.ldk + ch * 8);
            if (ch * 8 < a.ldv) cp_async16(smem_u32(vs + key * RS + ch * 8), vc + row * a.ldv + ch * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        // entry i: distance (first query of the CTA) - (last key of the tile) + i
        const int dist = pos0 + qb - (t * kK + kK - 1) + tid;
        s_bias[(t & 1) * 128 + tid] = a.bias ? kLog2e * a.bias[(size_t)h * a.bias_n + min(max(dist, 0), a.bias_n - 1)] : 0.f;
    };
    tile_async(t_begin);
    __syncthreads();
    // queries as A operands, 16 x P; for wide heads they are read again per tile
    constexpr bool kQRegs = P <= 128;
    uint32_t qa[kQRegs ? P / 16 : 1][4];
    const uint32_t q_addr = smem_u32(sQ + (warp * 16 + (lane & 15)) * RS + (lane >> 4) * 8);
    if constexpr (kQRegs) {
#pragma unroll
        for (int ks = 0; ks < P / 16; ks++) ldmatrix_x4(q_addr + ks * 32, qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
    }
    float o[P / 8][4];
#pragma unroll
    for (int i = 0; i < P / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float sink = a.sink ? a.sink[h] * kLog2e : -INFINITY;
    float mrow[2] = {sink, sink}, lrow[2];
    lrow[0] = lrow[1] = a.sink && c == 0 ? 1.f : 0.f;
    const float scale2 = a.scale * kLog2e;
    const int pq[2] = {pos0 + q0 + g, pos0 + q0 + g + 8};

    for (int t = t_begin; t < t_end; t++) {
        const int key0 = t * kK;
        const __half *Ks = at_smem + (size_t)(t & 1) * 2 * kK * RS, *Vs = Ks + kK * RS;
        if (t + 1 < t_end) {
            tile_async(t + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        float s[kK / 8][4];
#pragma unroll
        for (int nb = 0; nb < kK / 8; nb++) s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < P / 16; ks += 2) {
            uint32_t q2[2][4];
            if constexpr (kQRegs) {
#pragma unroll
                for (int i = 0; i < 4; i++) { q2[0][i] = qa[ks][i]; q2[1][i] = qa[ks + 1][i]; }
            } else {
                ldmatrix_x4(q_addr + ks * 32, q2[0][0], q2[0][1], q2[0][2], q2[0][3]);
                ldmatrix_x4(q_addr + ks * 32 + 32, q2[1][0], q2[1][1], q2[1][2], q2[1][3]);
            }
#pragma unroll
            for (int n4 = 0; n4 < kK / 8; n4 += 4) {           // four independent accumulators between two uses of one
                uint32_t kb[4][4];
#pragma unroll
                for (int i = 0; i < 4; i++)
                    ldmatrix_x4(smem_u32(Ks + ((n4 + i) * 8 + (lane & 7)) * RS + (lane >> 3) * 8 + ks * 16), kb[i][0], kb[i][1], kb[i][2], kb[i][3]);
#pragma unroll
                for (int i = 0; i < 4; i++) hmma16816(s[n4 + i], q2[0][0], q2[0][1], q2[0][2], q2[0][3], kb[i][0], kb[i][1]);
#pragma unroll
                for (int i = 0; i < 4; i++) hmma16816(s[n4 + i], q2[1][0], q2[1][1], q2[1][2], q2[1][3], kb[i][2], kb[i][3]);
            }
        }
        // inside = every key of the tile is seen by every query of the warp
        const bool inside = key0 + kK - 1 <= pos0 + q0 && key0 > pos0 + q0 + 15 - a.window;
        const float *bt = s_bias + (t & 1) * 128 + warp * 16 + g + (kK - 1) - 2 * c;       // minus 8 nb + e of the key, plus 8 for row 1
#pragma unroll
        for (int nb = 0; nb < kK / 8; nb++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[nb][e] = fmaf(s[nb][e], scale2, -bt[8 * (e >> 1) - 8 * nb - (e & 1)]);
        if (!inside) {
#pragma unroll
            for (int nb = 0; nb < kK / 8; nb++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int key = key0 + nb * 8 + 2 * c + (e & 1);
                    if (key > pq[e >> 1] || key <= pq[e >> 1] - a.window) s[nb][e] = -INFINITY;
                }
        }
        float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nb = 0; nb < kK / 8; nb++) {
            tmax[0] = fmaxf(tmax[0], fmaxf(s[nb][0], s[nb][1]));
            tmax[1] = fmaxf(tmax[1], fmaxf(s[nb][2], s[nb][3]));
        }
        float corr[2], mref[2];
#pragma unroll
        for (int r = 0; r < 2; r++) {
            tmax[r] = fmaxf(tmax[r], __shfl_xor_sync(0xffffffffu, tmax[r], 1));
            tmax[r] = fmaxf(tmax[r], __shfl_xor_sync(0xffffffffu, tmax[r], 2));
            const float mn = fmaxf(mrow[r], tmax[r]);
            mref[r] = mn == -INFINITY ? 0.f : mn;               // no key seen so far: every weight is zero
            corr[r] = exp2_approx(mrow[r] - mref[r]);
            mrow[r] = mn;
        }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
            lrow[0] *= corr[0]; lrow[1] *= corr[1];
#pragma unroll
            for (int nb = 0; nb < P / 8; nb++) {
                o[nb][0] *= corr[0]; o[nb][1] *= corr[0];
                o[nb][2] *= corr[1]; o[nb][3] *= corr[1];
            }
        }
#pragma unroll
        for (int ks = 0; ks < kK / 16; ks++) {
            // weights of 16 keys, as values and remainders
            uint32_t ph[4], pl[4];
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    const float e0 = exp2_approx(s[2 * ks + i][2 * r] - mref[r]), e1 = exp2_approx(s[2 * ks + i][2 * r + 1] - mref[r]);
                    lrow[r] += e0 + e1;
                    ph[2 * i + r] = pack_h2(e0, e1);
                    pl[2 * i + r] = rest_h2(e0, e1, ph[2 * i + r]);
                }
#pragma unroll
            for (int nb = 0; nb < P / 8; nb += 4) {
                uint32_t vb[2][4];
#pragma unroll
                for (int i = 0; i < 2; i++)
                    ldmatrix_x4_trans(smem_u32(Vs + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RS + (nb + 2 * i) * 8 + (lane >> 4) * 8), vb[i][0], vb[i][1], vb[i][2], vb[i][3]);
#pragma unroll
                for (int i = 0; i < 4; i++) hmma16816(o[nb + i], ph[0], ph[1], ph[2], ph[3], vb[i >> 1][2 * (i & 1)], vb[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
                for (int i = 0; i < 4; i++) hmma16816(o[nb + i], pl[0], pl[1], pl[2], pl[3], vb[i >> 1][2 * (i & 1)], vb[i >> 1][2 * (i & 1) + 1]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 1);
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 2);
        const int row = q0 + g + 8 * r;
        if (row >= T) continue;
        const float inv = 1.f / lrow[r];
        __nv_bfloat16 *dst = out + (size_t)row * ldo + (size_t)h * a.DV;
#pragma unroll
        for (int nb = 0; nb < P / 8; nb++) {
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int d = nb * 8 + 2 * c + e;
                if (d >= a.DV) continue;
                float v = o[nb][2 * r + e] * inv;
                if (a.gate) v *= sigmoidf(a.gate[(size_t)row * a.ld_gate + (size_t)h * a.DV + d]);
                dst[d] = __float2bfloat16_rn(v);
            }
        }
    }
}

template <int P>
tlb_status run(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo)
{
    static bool set = false;
    if (!set) {
        TLB_CUDA(cudaFuncSetAttribute(mix_attn_tc_kernel<P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)attn_smem<P>()));
        set = true;
    }
    mix_attn_tc_kernel<P><<<dim3((T + kQ - 1) / kQ, a.H), kThreads, attn_smem<P>(), ctx()->stream>>>(a, seq, T, pos0, (__nv_bfloat16 *)out, ldo);
    TLB_CUDA(cudaGetLastError());
    count_launch();
    return TLB_OK;
}

}  // namespace

bool mix_attn_prefill_tc_supported(int D, int DV) { return D >= 1 && D <= 256 && DV >= 1 && DV <= 256; }

tlb_status launch_mix_attn_prefill_tc(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo)
{
    const int p = std::max(a.D, a.DV);
    if (p <= 32) return run<32>(a, seq, T, pos0, out, ldo);
    if (p <= 64) return run<64>(a, seq, T, pos0, out, ldo);
    if (p <= 96) return run<96>(a, seq, T, pos0, out, ldo);
    if (p <= 128) return run<128>(a, seq, T, pos0, out, ldo);
    if (p <= 192) return run<192>(a, seq, T, pos0, out, ldo);
    return run<256>(a, seq, T, pos0, out, ldo);
}

}  // namespace tlb
