// Linear layers on bf16 weights, and the row kernels around them (embedding, RMS norm, PolyNorm).
//
//   dense_matvec_kernel   one activation row (decode): streams the weight once, f32 activation and accumulation.  The prologue
//                         makes the activation in shared memory - RMS norm, PolyNorm (its three root mean squares), an embedding
//                         row, the residual step of a gated and normed sublayer, a router's choice - and the finish adds the
//                         scaled result to the residual or turns gate and up into one activation.
//   dense_gemm_tc_kernel  many rows, 16-bit operands: tcgen05.mma, both tiles by TMA, f32 accumulator in tensor memory; also over
//                         row tiles of several stacked weights (experts).
//   dense_gemm_f32_kernel many rows, f32 activations: plain f32 multiply-adds (no tensor core rounds the operands).
#include <algorithm>

#include "act.cuh"
#include "layered_kernels.h"
#include "tc05.cuh"

namespace tlb {

namespace {

__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }
__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// ================================================================ one row
constexpr int kMvThreads = 256, kMvWarps = kMvThreads / 32, kMvRows = 4, kMvChunk = 256;

struct DenseMvParams {
    const __nv_bfloat16 *w;
    int n, k, ld, nch;                 // nch: chunks of 256 columns
    const float *bias;
    const float *x;
    const __nv_bfloat16 *emb;
    int emb_ld;
    const int *token;
    float *x_out;
    const float *norm_w;
    float norm_offset, eps;
    const float *poly;
    float *out;
    const float *resid_scale;
    int tiles;
    float softcap;
    int groups;
    const float *y, *y_gate, *post_w;
    float *h_out;
    float *act_out;
    int glu, ldx;
    GluConst act;
    RouteDesc route;
    const float *logits;
    int *sel;
    float *weight;
    const __nv_bfloat16 *shared_w;
    int shared_k, shared_ld, seg_nch;      // seg_nch: chunks of one expert
    const float *shared_x, *shared_gate;
};

// Shared position of activation element e: inside a chunk of 256 the first four of every eight come first, so that a lane's
// eight (two 16-byte reads) are read without bank conflicts.
__device__ __forceinline__ int xs_at(int e) { return (e & ~255) + ((e & 4) << 5) + ((e & 255) >> 3) * 4 + (e & 3); }

template <int NV>
__device__ __forceinline__ void block_sums(float (&v)[NV], float *red)
{
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        v[i] = warp_sum(v[i]);
        if (lane == 0) red[warp * NV + i] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NV; i++) {
        float s = 0.f;
        for (int w = 0; w < (int)(blockDim.x >> 5); w++) s += red[w * NV + i];
        v[i] = s;
    }
}

// WK warps share a row group's columns (chunk c belongs to warp c % WK); 8 / WK row groups of four rows per tile.
template <int PRO, int WK>
__global__ void __launch_bounds__(kMvThreads, 4) dense_matvec_kernel(const DenseMvParams p)
{
    constexpr int GROUPS = kMvWarps / WK, TILE = GROUPS * kMvRows;
    constexpr bool GNORM = PRO == DPRO_GNORM, EXPERT = PRO == DPRO_EXPERT, EXPERTS = PRO == DPRO_EXPERTS;
    extern __shared__ __align__(16) float xs[];
    __shared__ float red[GNORM ? 2 * kMaxNormGroups : kMvWarps * 3];
    __shared__ float fold[2][GROUPS][WK][kMvRows];
    __shared__ int s_sel[EXPERT ? kMaxTop : 1];
    __shared__ float s_weight[EXPERT || EXPERTS ? kMaxTop + 1 : 1];
    __shared__ const __nv_bfloat16 *s_base[EXPERTS ? kMaxTop + 1 : 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wk = warp % WK, wg = warp / WK;

    // what the first tile reads does not depend on the launch before: ask L2 for it before waiting
    if (!EXPERT) {
        const int r0 = blockIdx.x * TILE + wg * kMvRows;
        const __nv_bfloat16 *w0 = EXPERTS ? p.shared_w : p.w;         // which experts' rows is not known yet
        const int ld = EXPERTS ? p.shared_ld : p.ld, nch = EXPERTS ? (p.shared_ld + kMvChunk - 1) / kMvChunk : p.nch;
        for (int r = 0; r < kMvRows && w0; r++) {
            const int row = min(r0 + r, p.n - 1);
            const __nv_bfloat16 *src = w0 + (size_t)row * ld;
            for (int c = wk + (lane >> 2) * WK; c < nch; c += 8 * WK) {
                const int e = c * kMvChunk + (lane & 3) * 64;
                if (e < ld) asm volatile("prefetch.global.L2 [%0];" ::"l"(src + e));
            }
        }
    }
    if (GNORM) {
        for (int e = tid * 32; e < p.k; e += kMvThreads * 32) {
            asm volatile("prefetch.global.L2 [%0];" ::"l"(p.norm_w + e));
            if (p.post_w) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.post_w + e));
        }
    }
    pdl_wait();
    pdl_launch_dependents();

    const int kp = p.nch * kMvChunk;
    const __nv_bfloat16 *wbase = p.w;
    float *actp = p.act_out;
    if (PRO == DPRO_PLAIN || EXPERT) {
        for (int e = tid; e < kp; e += kMvThreads) xs[xs_at(e)] = e < p.k ? __ldcg(p.x + e) : 0.f;
        if (EXPERT) {
            route_token(p.logits, p.route, xs + kp, s_sel, s_weight);
            const int slot = blockIdx.y;
            wbase += (size_t)s_sel[slot] * p.n * p.ld;
            actp += (size_t)slot * (p.n / 2);
            if (blockIdx.x == 0 && slot == 0)
                for (int i = tid; i < p.route.top; i += kMvThreads) { p.sel[i] = s_sel[i]; p.weight[i] = s_weight[i]; }
        }
    } else if (PRO == DPRO_NORM) {
        const __nv_bfloat16 *er = p.emb ? p.emb + (size_t)*p.token * p.emb_ld : nullptr;
        float ss[1] = {0.f};
        for (int e = tid; e < p.k; e += kMvThreads) {
            const float v = er ? __bfloat162float(er[e]) : __ldcg(p.x + e);
            xs[xs_at(e)] = v;
            ss[0] += v * v;
            if (er && blockIdx.x == 0) p.x_out[e] = v;
        }
        block_sums(ss, red);
        const float inv = 1.f / sqrtf(ss[0] / (float)p.k + p.eps);
        for (int e = tid; e < kp; e += kMvThreads) {
            float *s = xs + xs_at(e);
            *s = e < p.k ? *s * inv * (p.norm_w[e] + p.norm_offset) : 0.f;
        }
    } else if (GNORM) {
        const __nv_bfloat16 *er = p.emb ? p.emb + (size_t)*p.token * p.emb_ld : nullptr;
        float *inv = red + kMaxNormGroups;
        auto at = [&](int e) { return xs[xs_at(e)]; };
        const float inv_len = (float)p.groups / (float)p.k;
        auto scaled = [&](float4 v, float4 w, int e) {
            return make_float4(v.x * inv[group_of(e, inv_len)] * (w.x + p.norm_offset), v.y * inv[group_of(e + 1, inv_len)] * (w.y + p.norm_offset),
                               v.z * inv[group_of(e + 2, inv_len)] * (w.z + p.norm_offset), v.w * inv[group_of(e + 3, inv_len)] * (w.w + p.norm_offset));
        };
        constexpr int NV = 4;
        if (!er && p.k % 4 == 0 && p.k <= NV * 4 * kMvThreads && (reinterpret_cast<uintptr_t>(p.y_gate) & 15) == 0) {
            // 16 elements per thread: every load of the rows is on its way before the first is used
            float4 v[NV], x[NV];
            auto ld4 = [&](const float *src, int e) { return e < p.k ? __ldcg(reinterpret_cast<const float4 *>(src + e)) : make_float4(0.f, 0.f, 0.f, 0.f); };
            auto slot = [&](int e) { return reinterpret_cast<float4 *>(xs + xs_at(e)); };
            if (p.y) {
                float4 g[NV];
#pragma unroll
                for (int i = 0; i < NV; i++) v[i] = ld4(p.y, (tid + i * kMvThreads) * 4);
#pragma unroll
                for (int i = 0; i < NV; i++) g[i] = p.y_gate ? ld4(p.y_gate, (tid + i * kMvThreads) * 4) : make_float4(INFINITY, INFINITY, INFINITY, INFINITY);
#pragma unroll
                for (int i = 0; i < NV; i++) x[i] = ld4(p.x, (tid + i * kMvThreads) * 4);
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    const int e = (tid + i * kMvThreads) * 4;
                    v[i].x *= sigmoidf(g[i].x); v[i].y *= sigmoidf(g[i].y); v[i].z *= sigmoidf(g[i].z); v[i].w *= sigmoidf(g[i].w);
                    if (e < p.k) *slot(e) = v[i];
                }
                __syncthreads();
                group_inv_rms(at, p.k, p.groups, p.eps, red, inv);
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    const int e = (tid + i * kMvThreads) * 4;
                    if (e < p.k) {
                        const float4 a = scaled(*slot(e), *reinterpret_cast<const float4 *>(p.post_w + e), e);
                        x[i].x += a.x; x[i].y += a.y; x[i].z += a.z; x[i].w += a.w;
                        *slot(e) = x[i];
                        if (blockIdx.x == 0) *reinterpret_cast<float4 *>(p.x_out + e) = x[i];
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < NV; i++) x[i] = ld4(p.x, (tid + i * kMvThreads) * 4);
#pragma unroll
                for (int i = 0; i < NV; i++)
                    if ((tid + i * kMvThreads) * 4 < p.k) *slot((tid + i * kMvThreads) * 4) = x[i];
            }
            __syncthreads();
            group_inv_rms(at, p.k, p.groups, p.eps, red, inv);
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int e = (tid + i * kMvThreads) * 4;
                if (e >= kp) continue;
                const float4 a = e < p.k ? scaled(x[i], *reinterpret_cast<const float4 *>(p.norm_w + e), e) : make_float4(0.f, 0.f, 0.f, 0.f);
                *slot(e) = a;
                if (p.h_out && blockIdx.x == 0 && e < p.k) *reinterpret_cast<float4 *>(p.h_out + e) = a;
            }
        } else {
        if (p.y) {
            for (int e = tid; e < p.k; e += kMvThreads) {
                const float v = __ldcg(p.y + e);
                xs[xs_at(e)] = p.y_gate ? v * sigmoidf(__ldcg(p.y_gate + e)) : v;
            }
            __syncthreads();
            group_inv_rms(at, p.k, p.groups, p.eps, red, inv);
            for (int e = tid; e < p.k; e += kMvThreads) {
                float *s = xs + xs_at(e);
                const float v = __ldcg(p.x + e) + *s * inv[group_of(e, inv_len)] * (p.post_w[e] + p.norm_offset);
                *s = v;
                if (blockIdx.x == 0) p.x_out[e] = v;
            }
        } else {
            for (int e = tid; e < p.k; e += kMvThreads) {
                const float v = er ? __bfloat162float(er[e]) : __ldcg(p.x + e);
                xs[xs_at(e)] = v;
                if (er && blockIdx.x == 0) p.x_out[e] = v;
            }
        }
        __syncthreads();
        group_inv_rms(at, p.k, p.groups, p.eps, red, inv);
        for (int e = tid; e < kp; e += kMvThreads) {
            float *s = xs + xs_at(e);
            *s = e < p.k ? *s * inv[group_of(e, inv_len)] * (p.norm_w[e] + p.norm_offset) : 0.f;
            if (p.h_out && blockIdx.x == 0 && e < p.k) p.h_out[e] = *s;
        }
        }
    } else if (EXPERTS) {
        const int top = p.route.top, seg = p.seg_nch * kMvChunk, first = top * seg;
        for (int s = tid; s <= top; s += kMvThreads) {
            s_weight[s] = s < top ? __ldcg(p.weight + s) : (p.shared_gate ? sigmoidf(__ldcg(p.shared_gate)) : 1.f);
            s_base[s] = s < top ? p.w + (size_t)__ldcg(p.sel + s) * p.n * p.ld : p.shared_w;
        }
        __syncthreads();
        for (int s = 0; s < top; s++) {
            const float w = s_weight[s];
            const float *x = p.x + (size_t)s * p.ldx;
#pragma unroll 8
            for (int e = tid; e < seg; e += kMvThreads) xs[s * seg + xs_at(e)] = e < p.k ? w * __ldcg(x + e) : 0.f;
        }
        const float w = s_weight[top];
#pragma unroll 8
        for (int e = tid; e < kp - first; e += kMvThreads) xs[first + xs_at(e)] = e < p.shared_k ? w * __ldcg(p.shared_x + e) : 0.f;
    } else {
        float ss[3] = {0.f, 0.f, 0.f};
        for (int e = tid; e < p.k; e += kMvThreads) {
            const float v = __ldcg(p.x + e), v2 = v * v;
            xs[xs_at(e)] = v;
            ss[0] += v2; ss[1] += v2 * v2; ss[2] += v2 * v2 * v2;
        }
        block_sums(ss, red);
        const float inv_n = 1.f / (float)p.k;
        const float a = p.poly[0] / sqrtf(ss[0] * inv_n + p.eps), b = p.poly[1] / sqrtf(ss[1] * inv_n + p.eps),
                    c = p.poly[2] / sqrtf(ss[2] * inv_n + p.eps), d = p.poly[3];
        for (int e = tid; e < kp; e += kMvThreads) {
            float *s = xs + xs_at(e);
            const float z = *s;
            *s = e < p.k ? z * (a + z * (b + z * c)) + d : 0.f;
        }
    }
    __syncthreads();

    int flip = 0;
    for (int tile = blockIdx.x; tile < p.tiles; tile += gridDim.x, flip ^= 1) {
        const int r0 = tile * TILE + wg * kMvRows;
        const uint4 *rows[kMvRows];
#pragma unroll
        for (int r = 0; r < kMvRows; r++) rows[r] = reinterpret_cast<const uint4 *>(wbase + (size_t)min(r0 + r, p.n - 1) * p.ld) + lane;
        float acc[kMvRows] = {0.f, 0.f, 0.f, 0.f};
        auto load = [&](int c, uint4 (&v)[kMvRows]) {
            if constexpr (EXPERTS) {
                const int seg = min(c / p.seg_nch, p.route.top), col = (c - seg * p.seg_nch) * kMvChunk + lane * 8, ld = seg < p.route.top ? p.ld : p.shared_ld;
                const bool in = c < p.nch && col < ld;
#pragma unroll
                for (int r = 0; r < kMvRows; r++)
                    v[r] = in ? __ldcs(reinterpret_cast<const uint4 *>(s_base[seg] + (size_t)min(r0 + r, p.n - 1) * ld + col)) : make_uint4(0u, 0u, 0u, 0u);
            } else {
                const bool in = c < p.nch && c * kMvChunk + lane * 8 < p.ld;
#pragma unroll
                for (int r = 0; r < kMvRows; r++) v[r] = in ? __ldcs(rows[r] + c * (kMvChunk / 8)) : make_uint4(0u, 0u, 0u, 0u);
            }
        };
        auto mul = [&](int c, const uint4 (&v)[kMvRows]) {
            if (c >= p.nch) return;
            const float4 xa = *reinterpret_cast<const float4 *>(xs + c * kMvChunk + lane * 4);
            const float4 xb = *reinterpret_cast<const float4 *>(xs + c * kMvChunk + 128 + lane * 4);
#pragma unroll
            for (int r = 0; r < kMvRows; r++) {
                float s = acc[r];
                s = fmaf(bf_lo(v[r].x), xa.x, s); s = fmaf(bf_hi(v[r].x), xa.y, s);
                s = fmaf(bf_lo(v[r].y), xa.z, s); s = fmaf(bf_hi(v[r].y), xa.w, s);
                s = fmaf(bf_lo(v[r].z), xb.x, s); s = fmaf(bf_hi(v[r].z), xb.y, s);
                s = fmaf(bf_lo(v[r].w), xb.z, s); s = fmaf(bf_hi(v[r].w), xb.w, s);
                acc[r] = s;
            }
        };
        for (int c = wk; c < p.nch; c += 2 * WK) {
            uint4 va[kMvRows], vb[kMvRows];
            load(c, va);
            load(c + WK, vb);
            mul(c, va);
            mul(c + WK, vb);
        }
#pragma unroll
        for (int r = 0; r < kMvRows; r++) acc[r] = warp_sum(acc[r]);
        float y = lane == 0 ? acc[0] : (lane == 1 ? acc[1] : (lane == 2 ? acc[2] : acc[3]));
        if (WK > 1) {
            if (lane < kMvRows) fold[flip][wg][wk][lane] = y;
            __syncthreads();
            if (wk == 0 && lane < kMvRows) {
                y = 0.f;
#pragma unroll
                for (int i = 0; i < WK; i++) y += fold[flip][wg][i][lane];
            }
        }
        if (wk == 0) {
            const int row = r0 + lane;
            const bool in = lane < kMvRows && row < p.n;
            if (in && p.bias) y += p.bias[row];
            if (r0 < p.glu) {                                  // two gates and their ups
                const float up = __shfl_down_sync(0xffffffffu, y, 2);
                if (lane < 2) actp[(r0 >> 1) + lane] = glu_act(p.act, y, up);
            } else if (in) {
                if (p.softcap > 0.f) y = p.softcap * tanhf(y / p.softcap);
                float *o = p.out + (row - p.glu);
                if (p.resid_scale) *o = __ldcg(o) + p.resid_scale[row] * y;
                else *o = y;
            }
        }
    }
}

// ================================================================ many rows, tensor cores
constexpr int kTcRows = 128, kTcK = 64, kTcThreads = 192;
constexpr uint32_t kTcWBytes = kTcRows * kTcK * 2;

struct DenseTcParams {
    float *out;
    const float *bias, *resid_scale;
    int n, T, ldo, nt, kt, stages;
    uint32_t tmem_cols;
    int *err;
    float softcap;
    int per;
    size_t block_stride;
    __half *out_h, *out_t;
    const int4 *tiles;
    int glu, ld_act;
    GluConst act;
    __nv_bfloat16 *act_out;
    uint32_t type_bits;                    // operand types in the instruction descriptor
};

// One CTA: 128 weight rows (lanes of the accumulator) x nt tokens (its columns).  Warps 0-3 write out (a warp's 32 lanes are 32
// consecutive output features of one token: coalesced), warp 4 lane 0 issues TMA, warp 5 lane 0 the MMAs.  Every wait is bounded.
__global__ void __launch_bounds__(kTcThreads, 2)
dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap xmap, const DenseTcParams p)
{
    extern __shared__ uint8_t tc_smem[];
    __shared__ int abort_word;
    __shared__ uint32_t tmem_slot;
    volatile int *abort_flag = &abort_word;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t base = (smem_u32(tc_smem) + 1023u) & ~1023u;
    const uint32_t xbytes = (uint32_t)p.nt * (kTcK * 2), stage = kTcWBytes + xbytes;
    const uint32_t bars = base + (uint32_t)p.stages * stage;
    const uint32_t full = bars, empty = bars + 8u * p.stages, done = bars + 16u * p.stages;
    const int n0 = blockIdx.y * kTcRows;
    int t0 = blockIdx.x * p.nt, t_end = p.T, wrow0 = n0;
    if (p.tiles) {                         // rows of one of several stacked weights
        const int4 tile = p.tiles[blockIdx.x];
        if (tile.z <= 0) return;
        t0 = tile.y; t_end = tile.y + tile.z; wrow0 = tile.x * p.n + n0;
    }

    if (tid == 0) {
        abort_word = 0;
        for (int i = 0; i < p.stages; i++) { mbar_init(full + 8 * i, 1); mbar_init(empty + 8 * i, 1); }
        mbar_init(done, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;

    if (warp < 4) {
        if (mbar_wait(done, 0, abort_flag, p.err, 61)) {
            tc_fence_after();
            const int row = n0 + warp * 32 + lane;
            const bool in = row < p.n;
            const float bias = in && p.bias ? p.bias[row] : 0.f, rs = in && p.resid_scale ? p.resid_scale[row] : 0.f;
            const int col = row - p.glu;
            const size_t place = (size_t)(col / p.per) * p.block_stride + col % p.per;
            if (p.out_t) t_end = (t_end + 127) / 128 * 128;        // rows past T came as zeros
            for (int c0 = 0; c0 < p.nt && t0 + c0 < t_end; c0 += 32) {
                uint32_t v[32];
                tmem_ld32(tmem + ((uint32_t)(warp * 32) << 16) + (uint32_t)c0, v);
                tmem_wait_ld();
                if (n0 + warp * 32 < p.glu) {
                    // lanes (0, 1), (2, 3) of four hold gates and ups of two units: the former take tokens 0 .. 15, the latter 16 .. 31
                    const bool hi = lane & 2;
                    const float theirs = __shfl_xor_sync(0xffffffffu, bias, 2);
                    const GluConst act = p.act;
                    __nv_bfloat16 *da = p.act_out + (size_t)(t0 + c0) * p.ld_act + (row >> 2) * 2 + (row & 1);
#pragma unroll
                    for (int i = 0; i < 16; i++) {
                        const float other = __uint_as_float(__shfl_xor_sync(0xffffffffu, hi ? v[i] : v[i + 16], 2)) + theirs;
                        const float own = __uint_as_float(hi ? v[i + 16] : v[i]) + bias;
                        const int t = hi ? i + 16 : i;
                        const float y = glu_act(act, hi ? other : own, hi ? own : other);
                        if (row < p.glu && t0 + c0 + t < t_end) da[(size_t)t * p.ld_act] = __float2bfloat16_rn(y);
                    }
                }
                if (!in || row < p.glu) continue;
                if (p.out_t) {
                    __half *dt = p.out_t + (size_t)(col / p.per) * p.block_stride + (size_t)(col % p.per) * p.ldo + t0 + c0;
#pragma unroll
                    for (int i = 0; i < 32; i += 8) {
                        uint32_t w[4];
#pragma unroll
                        for (int k = 0; k < 4; k++) {
                            const __half2 h = __floats2half2_rn(fminf(fmaxf(__uint_as_float(v[i + 2 * k]), -65504.f), 65504.f), fminf(fmaxf(__uint_as_float(v[i + 2 * k + 1]), -65504.f), 65504.f));
                            w[k] = *reinterpret_cast<const uint32_t *>(&h);
                        }
                        *reinterpret_cast<uint4 *>(dt + i) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                    continue;
                }
                float *dst = p.out + (size_t)(t0 + c0) * p.ldo + place;
                const int m = min(32, t_end - t0 - c0);
                if (p.out_h) {
                    __half *dh = p.out_h + (size_t)(t0 + c0) * p.ldo + place;
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (i < m) dh[(size_t)i * p.ldo] = __float2half_rn(fminf(fmaxf(__uint_as_float(v[i]) + bias, -65504.f), 65504.f));
                } else if (p.softcap > 0.f) {
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (i < m) dst[(size_t)i * p.ldo] = p.softcap * tanhf((__uint_as_float(v[i]) + bias) / p.softcap);
                } else if (p.resid_scale) {
                    float r[32];
#pragma unroll
                    for (int i = 0; i < 32; i++) r[i] = i < m ? dst[(size_t)i * p.ldo] : 0.f;
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (i < m) dst[(size_t)i * p.ldo] = fmaf(rs, __uint_as_float(v[i]), r[i]);
                } else {
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (i < m) dst[(size_t)i * p.ldo] = __uint_as_float(v[i]) + bias;
                }
            }
        }
    } else if (warp == 4) {
        if (lane == 0) {
            int issued = 0;
            for (int k = 0; k < p.kt; k++) {
                const int s = k % p.stages;
                if (k >= p.stages && !mbar_wait(empty + 8 * s, (uint32_t)(k / p.stages - 1) & 1u, abort_flag, p.err, 62)) break;
                mbar_expect_tx(full + 8 * s, stage);
                tma_load_2d(base + (uint32_t)s * stage, &wmap, k * kTcK, wrow0, full + 8 * s);
                tma_load_2d(base + (uint32_t)s * stage + kTcWBytes, &xmap, k * kTcK, t0, full + 8 * s);
                issued = k + 1;
            }
            if (*abort_flag)
                for (int k = max(0, issued - p.stages); k < issued; k++) mbar_wait_drain(full + 8 * (k % p.stages), (uint32_t)(k / p.stages) & 1u);
        }
    } else if (lane == 0) {
        // f32 accumulator, operands of one 16-bit type, both K-major, M 128, N nt
        const int cols = p.tiles ? (t_end - t0 + 15) / 16 * 16 : p.nt;       // a tile that is not full multiplies fewer columns
        const uint32_t idesc = (1u << 4) | p.type_bits | ((uint32_t)(cols >> 3) << 17) | ((uint32_t)(kTcRows >> 4) << 24);
        for (int k = 0; k < p.kt; k++) {
            const int s = k % p.stages;
            if (!mbar_wait(full + 8 * s, (uint32_t)(k / p.stages) & 1u, abort_flag, p.err, 63)) break;
            tc_fence_after();
            const uint64_t wd = smem_desc_sw128(base + (uint32_t)s * stage), xd = smem_desc_sw128(base + (uint32_t)s * stage + kTcWBytes);
#pragma unroll
            for (int j = 0; j < 4; j++) umma_f16_ss(tmem, wd + 2u * j, xd + 2u * j, idesc, (k | j) != 0);
            umma_commit(empty + 8 * s);
        }
        umma_commit(done);                       // also after an abort: MMAs in flight end before the tensor memory is freed
        if (*abort_flag) mbar_wait_drain(done, 0);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        __syncwarp();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
    }
}

// ================================================================ many rows, f32 operands
struct DenseF32Params {
    const __nv_bfloat16 *w;
    int n, k, ld;
    const float *bias, *x, *resid_scale;
    int ldx, T, ldo;
    float *out;
    float softcap;
    int per;
    size_t block_stride;
    const int4 *tiles;
    int glu, ld_act;
    GluConst act;
    float *act_out;
};
constexpr int kSgT = kF32GemmRows, kSgN = 64, kSgK = 16;

__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const DenseF32Params p)
{
    __shared__ float sx[kSgK][kSgT + 4], sw[kSgK][kSgN + 4];
    const int tid = threadIdx.x, n0 = blockIdx.y * kSgN;
    const int tn = tid & 15, tt = tid >> 4;
    int t0 = blockIdx.x * kSgT, t_end = p.T;
    const __nv_bfloat16 *w = p.w;
    if (p.tiles) {
        const int4 tile = p.tiles[blockIdx.x];
        if (tile.z <= 0) return;
        t0 = tile.y; t_end = tile.y + tile.z; w += (size_t)tile.x * p.n * p.ld;
    }
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.k; k0 += kSgK) {
        for (int i = tid; i < kSgT * kSgK; i += 256) {
            const int r = i / kSgK, c = i % kSgK;
            sx[c][r] = t0 + r < t_end && k0 + c < p.k ? p.x[(size_t)(t0 + r) * p.ldx + k0 + c] : 0.f;
            sw[c][r] = n0 + r < p.n && k0 + c < p.k ? __bfloat162float(w[(size_t)(n0 + r) * p.ld + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < kSgK; c++) {
            const float4 a = *reinterpret_cast<const float4 *>(&sx[c][tt * 4]), b = *reinterpret_cast<const float4 *>(&sw[c][tn * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
    if (n0 + tn * 4 < p.glu) {                 // this thread's four columns: two gates and their ups
        const int n = n0 + tn * 4;
        float b[4];
#pragma unroll
        for (int j = 0; j < 4; j++) b[j] = p.bias ? p.bias[n + j] : 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int t = t0 + tt * 4 + i;
            if (t >= t_end) continue;
#pragma unroll
            for (int j = 0; j < 2; j++) p.act_out[(size_t)t * p.ld_act + n / 2 + j] = glu_act(p.act, acc[i][j] + b[j], acc[i][j + 2] + b[j + 2]);
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int t = t0 + tt * 4 + i, n = n0 + tn * 4 + j, col = n - p.glu;
            if (t >= t_end || n >= p.n) continue;
            float *o = p.out + (size_t)t * p.ldo + (size_t)(col / p.per) * p.block_stride + col % p.per;
            if (p.resid_scale) { *o = fmaf(p.resid_scale[n], acc[i][j], *o); continue; }
            const float y = acc[i][j] + (p.bias ? p.bias[n] : 0.f);
            *o = p.softcap > 0.f ? p.softcap * tanhf(y / p.softcap) : y;
        }
}

// ================================================================ rows
__device__ __forceinline__ void store_act(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_act(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ void store_act4(float *p, float a, float b, float c, float d) { *reinterpret_cast<float4 *>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store_act4(__nv_bfloat16 *p, float a, float b, float c, float d)
{
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
}

template <typename TA>
__global__ void __launch_bounds__(256) norm_rows_kernel(const float *__restrict__ x, int width, int ldx, const float *__restrict__ w, float offset, float eps,
                                                        TA *__restrict__ out, int ld)
{
    __shared__ float red[8];
    const float *row = x + (size_t)blockIdx.x * ldx;
    TA *o = out + (size_t)blockIdx.x * ld;
    float ss[1] = {0.f};
    if (width % 4 == 0 && ldx % 4 == 0 && width <= 256 * 4 * 8) {       // the row stays in registers: one pass over memory
        float4 v[8];
        const int n4 = width / 4;
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = threadIdx.x + k * 256;
            v[k] = i < n4 ? reinterpret_cast<const float4 *>(row)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
            ss[0] += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
        }
        block_sums(ss, red);
        const float inv = 1.f / sqrtf(ss[0] / (float)width + eps);
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = threadIdx.x + k * 256;
            if (i < n4) {
                const float4 g = reinterpret_cast<const float4 *>(w)[i];
                store_act4(o + 4 * i, v[k].x * inv * (g.x + offset), v[k].y * inv * (g.y + offset), v[k].z * inv * (g.z + offset), v[k].w * inv * (g.w + offset));
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < width; i += 256) ss[0] += row[i] * row[i];
    block_sums(ss, red);
    const float inv = 1.f / sqrtf(ss[0] / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256) store_act(o + i, row[i] * inv * (w[i] + offset));
}

template <typename TA>
__global__ void __launch_bounds__(512) poly_rows_kernel(const float *__restrict__ z, int ff, int ldz, const float *__restrict__ coef, float eps,
                                                        TA *__restrict__ out, int ld)
{
    __shared__ float red[16 * 3];
    const float *row = z + (size_t)blockIdx.x * ldz;
    TA *o = out + (size_t)blockIdx.x * ld;
    const float inv_n = 1.f / (float)ff;
    float ss[3] = {0.f, 0.f, 0.f};
    auto add = [&](float v) {
        const float v2 = v * v;
        ss[0] += v2; ss[1] += v2 * v2; ss[2] += v2 * v2 * v2;
    };
    if (ff % 4 == 0 && ff <= 512 * 4 * 8) {              // the row stays in registers
        float4 v[8];
        const int n4 = ff / 4;
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = threadIdx.x + k * 512;
            v[k] = i < n4 ? reinterpret_cast<const float4 *>(row)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < 8; k++) { add(v[k].x); add(v[k].y); add(v[k].z); add(v[k].w); }
        block_sums(ss, red);
        const float a = coef[0] / sqrtf(ss[0] * inv_n + eps), b = coef[1] / sqrtf(ss[1] * inv_n + eps), c = coef[2] / sqrtf(ss[2] * inv_n + eps), d = coef[3];
        auto act = [&](float x) { return x * (a + x * (b + x * c)) + d; };
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = threadIdx.x + k * 512;
            if (i < n4) store_act4(o + 4 * i, act(v[k].x), act(v[k].y), act(v[k].z), act(v[k].w));
        }
        return;
    }
    for (int i = threadIdx.x; i < ff; i += 512) add(row[i]);
    block_sums(ss, red);
    const float a = coef[0] / sqrtf(ss[0] * inv_n + eps), b = coef[1] / sqrtf(ss[1] * inv_n + eps), c = coef[2] / sqrtf(ss[2] * inv_n + eps), d = coef[3];
    for (int i = threadIdx.x; i < ff; i += 512) store_act(o + i, row[i] * (a + row[i] * (b + row[i] * c)) + d);
}

__global__ void embed_bf16_kernel(const int *__restrict__ tokens, const __nv_bfloat16 *__restrict__ table, int width, int ld, float *__restrict__ x)
{
    const __nv_bfloat16 *src = table + (size_t)tokens[blockIdx.x] * ld;
    if (width % 8 == 0) {
        float4 *dst = reinterpret_cast<float4 *>(x + (size_t)blockIdx.x * width);
        for (int i = threadIdx.x; i < width / 8; i += blockDim.x) {
            const uint4 v = reinterpret_cast<const uint4 *>(src)[i];
            dst[2 * i] = make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y));
            dst[2 * i + 1] = make_float4(bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w));
        }
        return;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) x[(size_t)blockIdx.x * width + i] = __bfloat162float(src[i]);
}

__global__ void gather_rows_kernel(const float *__restrict__ x, int width, const int *__restrict__ idx, float *__restrict__ out)
{
    const float *src = x + (size_t)idx[blockIdx.x] * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) out[(size_t)blockIdx.x * width + i] = src[i];
}

__global__ void pack_rows_kernel(const __nv_bfloat16 *__restrict__ src, int k, __nv_bfloat16 *__restrict__ dst, int ld)
{
    for (int i = threadIdx.x; i < k; i += blockDim.x) dst[(size_t)blockIdx.x * ld + i] = src[(size_t)blockIdx.x * k + i];
}

__global__ void pack_glu_rows_kernel(const __nv_bfloat16 *__restrict__ src, int k, __nv_bfloat16 *__restrict__ dst, int ld)
{
    const int i = blockIdx.x;
    for (int e = threadIdx.x; e < k; e += blockDim.x) dst[(size_t)((i >> 1) * 4 + (i & 1)) * ld + e] = src[(size_t)i * k + e];
}

__global__ void pack_rows_f16_kernel(const __nv_bfloat16 *__restrict__ src, int k, __half *__restrict__ dst, int ld)
{
    for (int i = threadIdx.x; i < ld; i += blockDim.x)
        dst[(size_t)blockIdx.x * ld + i] = i < k ? __float2half_rn(fminf(fmaxf(__bfloat162float(src[(size_t)blockIdx.x * k + i]), -65504.f), 65504.f)) : __float2half_rn(0.f);
}

tlb_status launched(const char *what)
{
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return cuda_fail(e, what);
    count_launch();
    return TLB_OK;
}

template <int PRO, int WK>
tlb_status run_matvec(const DenseMvParams &p, bool pdl)
{
    Context *c = ctx();
    const size_t smem = ((size_t)p.nch * kMvChunk + (PRO == DPRO_EXPERT ? route_scratch_floats(p.route) : 0)) * sizeof(float);
    static size_t allowed = 40 << 10;      // with the static part, under the 48 KB that need no asking
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(dense_matvec_kernel<PRO, WK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    const int per_sm = std::max(1, std::min(4, (int)(((size_t)220 << 10) / (smem + 2048))));
    const int slots = PRO == DPRO_EXPERT ? p.route.top : 1, grid = std::min(p.tiles, std::max(1, c->sm_count * per_sm / slots));
    TLB_CUDA(launch_chained(dense_matvec_kernel<PRO, WK>, dim3(grid, slots), dim3(kMvThreads), smem, pdl, p));
    count_launch();
    return TLB_OK;
}

template <int PRO>
tlb_status pick_matvec(DenseMvParams p, bool pdl)
{
    // the fewest warps per row group that still give every SM two tiles
    int wk = 1;
    auto tiles = [&](int w) { return (p.n + kMvWarps / w * kMvRows - 1) / (kMvWarps / w * kMvRows); };
    const int slots = PRO == DPRO_EXPERT ? p.route.top : 1;
    while (wk < 8 && tiles(wk) * slots < 2 * ctx()->sm_count && wk * 2 <= p.nch) wk *= 2;
    p.tiles = tiles(wk);
    switch (wk) {
    case 1: return run_matvec<PRO, 1>(p, pdl);
    case 2: return run_matvec<PRO, 2>(p, pdl);
    case 4: return run_matvec<PRO, 4>(p, pdl);
    default: return run_matvec<PRO, 8>(p, pdl);
    }
}

}  // namespace

bool dense_matvec_supported(int k) { return k >= 1 && k <= 48 * 1024; }

bool experts_matvec_supported(const RouteDesc &r, int ff, int shared_ff)
{
    const int nch = r.top * ((ff + kMvChunk - 1) / kMvChunk) + (shared_ff + kMvChunk - 1) / kMvChunk;
    return r.top >= 1 && r.top <= kMaxTop && r.experts <= kMaxExperts && nch <= 48 * 1024 / kMvChunk;
}

tlb_status launch_dense_matvec(const DenseMatvecJob &j)
{
    if (!ctx()) return TLB_ERR_DEVICE;
    if (!dense_matvec_supported(j.w.k)) return fail(TLB_ERR_SHAPE, "a linear layer over %d inputs does not fit the matvec's shared memory", j.w.k);
    DenseMvParams p = {};
    p.w = j.w.w; p.n = j.w.n; p.k = j.w.k; p.ld = j.w.ld; p.nch = (j.w.ld + kMvChunk - 1) / kMvChunk;
    p.bias = j.w.bias; p.x = j.x; p.emb = j.emb; p.emb_ld = act_ld(j.w.k); p.token = j.token; p.x_out = j.x_out;
    p.norm_w = j.norm_w; p.norm_offset = j.norm_offset; p.eps = j.eps; p.poly = j.poly; p.out = j.out; p.resid_scale = j.resid_scale;
    p.softcap = j.softcap; p.groups = j.groups; p.y = j.y; p.y_gate = j.y_gate; p.post_w = j.post_w; p.h_out = j.h_out;
    p.glu = j.w.glu; p.act = glu_const(j.w.glu_act); p.act_out = j.act_out; p.ldx = j.ldx;
    p.route = j.route; p.logits = j.logits; p.sel = j.sel; p.weight = j.weight;
    if (j.pro == DPRO_EXPERTS) {
        p.seg_nch = p.nch;
        p.shared_w = j.shared.w; p.shared_k = j.shared.k; p.shared_ld = j.shared.ld; p.shared_x = j.shared_x; p.shared_gate = j.shared_gate;
        p.nch = j.route.top * p.seg_nch + (j.shared.ld + kMvChunk - 1) / kMvChunk;
        return pick_matvec<DPRO_EXPERTS>(p, j.pdl);
    }
    if (j.pro == DPRO_GNORM) return pick_matvec<DPRO_GNORM>(p, j.pdl);
    if (j.pro == DPRO_EXPERT) return pick_matvec<DPRO_EXPERT>(p, j.pdl);
    if (j.pro == DPRO_NORM) return pick_matvec<DPRO_NORM>(p, j.pdl);
    if (j.pro == DPRO_POLY) return pick_matvec<DPRO_POLY>(p, j.pdl);
    return pick_matvec<DPRO_PLAIN>(p, j.pdl);
}

tlb_status launch_dense_gemm(const DenseGemmJob &j, bool f32)
{
    Context *c = ctx();
    if (!c) return TLB_ERR_DEVICE;
    if (j.T < 1) return TLB_OK;
    const int per = j.per > 0 ? j.per : j.w.n;
    if (f32) {
        DenseF32Params p;
        p.softcap = j.softcap; p.per = per; p.block_stride = j.block_stride; p.tiles = j.tiles;
        p.glu = j.w.glu; p.act = glu_const(j.w.glu_act); p.ld_act = j.ld_act; p.act_out = (float *)j.act_out;
        p.w = j.w.w; p.n = j.w.n; p.k = j.w.k; p.ld = j.w.ld; p.bias = j.w.bias; p.x = (const float *)j.x; p.resid_scale = j.resid_scale;
        p.ldx = j.ldx; p.T = j.T; p.ldo = j.ldo; p.out = j.out;
        dense_gemm_f32_kernel<<<dim3(j.tiles ? j.n_tiles : (j.T + kSgT - 1) / kSgT, (j.w.n + kSgN - 1) / kSgN), 256, 0, c->stream>>>(p);
        return launched("f32 GEMM launch");
    }
    DenseTcParams p;
    p.out = j.out; p.bias = j.w.bias; p.resid_scale = j.resid_scale; p.n = j.w.n; p.T = j.T; p.ldo = j.ldo;
    p.softcap = j.softcap; p.per = per; p.block_stride = j.block_stride; p.out_h = j.out_h; p.out_t = j.out_t; p.tiles = j.tiles;
    p.glu = j.w.glu; p.act = glu_const(j.w.glu_act); p.ld_act = j.ld_act; p.act_out = (__nv_bfloat16 *)j.act_out;
    p.type_bits = j.w.f16 ? 0u : (1u << 7) | (1u << 10);
    p.kt = (j.w.k + kTcK - 1) / kTcK;
    // short sums, gated activations and experts' tiles: two CTAs share an SM, one's epilogue under the other's products
    const bool pair = p.kt <= 16 || j.w.glu || j.tiles;
    p.nt = j.tiles ? j.tile_rows : (j.out_t ? 128 : std::min(pair ? 128 : 256, (j.T + 31) / 32 * 32));
    p.tmem_cols = 32;
    while (p.tmem_cols < (uint32_t)p.nt) p.tmem_cols *= 2;
    const size_t stage = kTcWBytes + (size_t)p.nt * kTcK * 2;
    p.stages = (int)std::min<size_t>(8, ((size_t)(pair ? 104 : 216) << 10) / stage);
    p.err = c->err_flag;
    CUtensorMap wmap, xmap;
    const CUtensorMapDataType type = j.w.f16 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    if (!encode_f16_map(&wmap, j.w.w, (uint64_t)j.w.k, (uint64_t)j.w.n * j.n_weights, (uint64_t)j.w.ld * 2, kTcK, kTcRows, type) ||
        !encode_f16_map(&xmap, j.x, (uint64_t)j.w.k, (uint64_t)j.T, (uint64_t)j.ldx * 2, kTcK, (uint32_t)p.nt, type))
        return fail(TLB_ERR_DEVICE, "GEMM: cuTensorMapEncodeTiled failed or is not available");
    const size_t smem = (size_t)p.stages * stage + 16 * p.stages + 8 + 1024;
    static size_t allowed = 0;
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(dense_gemm_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    dense_gemm_tc_kernel<<<dim3(j.tiles ? j.n_tiles : (j.T + p.nt - 1) / p.nt, (j.w.n + kTcRows - 1) / kTcRows), kTcThreads, smem, c->stream>>>(wmap, xmap, p);
    return launched("GEMM launch");
}

tlb_status launch_norm_rows(const float *x, int T, int width, int ldx, const float *w, float offset, float eps, void *out, int ld, bool f32)
{
    if (f32) norm_rows_kernel<<<T, 256, 0, ctx()->stream>>>(x, width, ldx, w, offset, eps, (float *)out, ld);
    else norm_rows_kernel<<<T, 256, 0, ctx()->stream>>>(x, width, ldx, w, offset, eps, (__nv_bfloat16 *)out, ld);
    return launched("norm launch");
}

tlb_status launch_poly_rows(const float *z, int T, int ff, int ldz, const float *coef, float eps, void *out, int ld, bool f32)
{
    if (f32) poly_rows_kernel<<<T, 512, 0, ctx()->stream>>>(z, ff, ldz, coef, eps, (float *)out, ld);
    else poly_rows_kernel<<<T, 512, 0, ctx()->stream>>>(z, ff, ldz, coef, eps, (__nv_bfloat16 *)out, ld);
    return launched("PolyNorm launch");
}

tlb_status launch_embed_bf16(const int *tokens, const __nv_bfloat16 *table, int width, int ld, float *x, int T)
{
    embed_bf16_kernel<<<T, 256, 0, ctx()->stream>>>(tokens, table, width, ld, x);
    return launched("embedding launch");
}

tlb_status launch_gather_rows(const float *x, int width, const int *idx, int n, float *out)
{
    gather_rows_kernel<<<n, 256, 0, ctx()->stream>>>(x, width, idx, out);
    return launched("gather launch");
}

tlb_status launch_pack_rows(const __nv_bfloat16 *src, int n, int k, __nv_bfloat16 *dst, int ld, int col0)
{
    pack_rows_kernel<<<n, 256, 0, ctx()->stream>>>(src, k, dst + col0, ld);
    return launched("weight packing launch");
}

tlb_status launch_pack_glu_rows(const __nv_bfloat16 *src, int ff, int k, __nv_bfloat16 *dst, int ld, bool up)
{
    pack_glu_rows_kernel<<<ff, 256, 0, ctx()->stream>>>(src, k, dst + (up ? (size_t)2 * ld : 0), ld);
    return launched("weight packing launch");
}

tlb_status launch_pack_rows_f16(const __nv_bfloat16 *src, int n, int k, void *dst, int ld)
{
    pack_rows_f16_kernel<<<n, 256, 0, ctx()->stream>>>(src, k, (__half *)dst, ld);
    return launched("weight packing launch");
}

}  // namespace tlb
