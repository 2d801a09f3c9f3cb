// Latent attention: per token the cache holds a normed latent of R values and one rotated key part of RD values shared by all
// heads; the keys and values of a head are W_uk c and W_uv c.
//
// Rows of queries (one new token per sequence, or a short portion of a prompt) never form keys or values: a head's score is
// (W_uk^T q) . c + q_rot . k_rot, and W_uv is applied to the weighted sum of latents.
//   latent_query_kernel      rotation, W_uk^T q per head; the new tokens' cache rows
//   latent_attn_tc_kernel    16 heads x a range of keys per CTA on mma.sync, all heads reading one tile of latents; running softmax
//   latent_attn_f32_kernel   the same for 32-bit caches, plain multiply-adds
//   latent_value_kernel      merges the key ranges of a head, applies W_uv and the output gate
// Long portions expand the visible latents to keys and values (two GEMMs over cache rows) and take the prompt attention.
// Scores, softmax weights (two f16 terms, value and remainder, on the tensor cores) and sums are 32-bit.
#include <algorithm>
#include <vector>

#include "act.cuh"
#include "layered_kernels.h"
#include "qmv_common.cuh"

namespace tlb {

namespace {

constexpr int kThreads = 256, kWarps = 8, kKeys = 64, kHeads = 16, kMaxSplits = 64;
constexpr int kMaxLatentF32 = 2048;
constexpr int kMaxExpandedHead = 256;

__device__ __forceinline__ void store_c(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_c(__half *p, float v) { *p = __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t addr, uint32_t &r0, uint32_t &r1)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3)
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }
__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Element i of a rotated part: pairs of neighbours among the first `rot`.
__device__ __forceinline__ float turned(const float *x, int i, int rot, const float *c, const float *s)
{
    const float v = __ldcg(x + i);
    if (i >= rot) return v;
    const float o = __ldcg(x + (i ^ 1)), cs = c[i >> 1], sn = s[i >> 1];
    return i & 1 ? v * cs + o * sn : v * cs - o * sn;
}

// The key range of a query at position pos, cut into at most max_split runs of whole 64-key tiles.
struct Cut { int first, n, per, used; };
__device__ __forceinline__ Cut cut_keys(int pos, int window, int max_split)
{
    Cut c;
    c.n = min(pos + 1, window);
    c.first = pos + 1 - c.n;
    const int tiles = (c.n + kKeys - 1) / kKeys;
    c.per = (tiles + max_split - 1) / max_split;
    c.used = (tiles + c.per - 1) / c.per;
    return c;
}
// floats of one (row, split, head) of the partial results: weighted latents, then maximum and sum of exponentials
__host__ __device__ inline int part_row(int R) { return (R + 3) / 4 * 4 + 4; }

__device__ __forceinline__ int row_pos(const MixLatentRows &j, int i) { return j.pos ? __ldcg(j.pos + i) : j.pos0 + i; }
__device__ __forceinline__ int row_rope(const MixLatentRows &j, int i) { return j.rope_pos ? __ldcg(j.rope_pos + i) : j.rope0 + i * j.rope_step; }

// the new token's cache row; all threads of the block call
template <typename CT>
__device__ __forceinline__ void append_row(const MixLatent &m, int seq, int pos, int rope, const float *kv, float *part, float *inv)
{
    group_inv_rms([&](int e) { return __ldcg(kv + e); }, m.R, 1, m.eps, part, inv);
    CT *dst = reinterpret_cast<CT *>(m.cache) + (size_t)seq * m.seq_stride + (size_t)pos * m.ld;
    const size_t tab = (size_t)rope * (m.rot / 2);
    for (int e = threadIdx.x; e < m.R; e += blockDim.x) store_c(dst + e, __ldcg(kv + e) * inv[0] * m.c_norm[e]);
    for (int i = threadIdx.x; i < m.RD; i += blockDim.x) store_c(dst + m.R + i, turned(kv + m.R, i, m.rot, m.rot_cos + tab, m.rot_sin + tab));
}

// ================================================================ queries into the latent space
// Grid (chunks of 8 * tc latent columns, heads + 1, tiles of RT rows); the last y appends.  A thread owns 8 columns for every dg-th
// dimension of the head.
template <typename CT, int RT>
__global__ void __launch_bounds__(kThreads) latent_query_kernel(const MixLatentRows j, int tc)
{
    extern __shared__ __align__(16) float smem[];           // [RT][D] queries, [dg][RT][8 tc] sums
    const MixLatent &m = j.m;
    const int tid = threadIdx.x, h = blockIdx.y, row0 = blockIdx.z * RT, nr = min(RT, j.rows - row0), dg = kThreads / tc;
    const int col = (blockIdx.x * tc + tid % tc) * 8, d0 = tid / tc;
    const __nv_bfloat16 *w = m.uk.w + (size_t)h * m.D * m.uk.ld + col;
    if (h < m.H && col < m.uk.ld)
        for (int d = d0; d < m.D; d += dg) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + (size_t)d * m.uk.ld));
    pdl_wait();
    pdl_launch_dependents();
    if (h == m.H) {
        __shared__ float part[kWarps], inv[1];
        if (blockIdx.x == 0)
            for (int i = 0; i < nr; i++) {
                append_row<CT>(m, j.seq0 + (row0 + i) * j.seq_step, row_pos(j, row0 + i), row_rope(j, row0 + i), m.kv + (size_t)(row0 + i) * m.ldkv, part, inv);
                __syncthreads();
            }
        return;
    }
    float *sq = smem, *sred = smem + (RT * m.D + 3) / 4 * 4;
    const int hd = m.D + m.RD;
    for (int i = tid; i < nr * m.D; i += kThreads) sq[i] = __ldcg(m.q + (size_t)(row0 + i / m.D) * m.ldq + (size_t)h * hd + i % m.D);
    __syncthreads();
    float acc[RT][8] = {};
    if (col < m.uk.ld) {
#pragma unroll 4
        for (int d = d0; d < m.D; d += dg) {
            const uint4 v = *reinterpret_cast<const uint4 *>(w + (size_t)d * m.uk.ld);
            const float f[8] = {bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y), bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w)};
#pragma unroll
            for (int r = 0; r < RT; r++) {
                const float q = r < nr ? sq[r * m.D + d] : 0.f;
#pragma unroll
                for (int e = 0; e < 8; e++) acc[r][e] = fmaf(q, f[e], acc[r][e]);
            }
        }
    }
    const int width = tc * 8;
#pragma unroll
    for (int r = 0; r < RT; r++)
#pragma unroll
        for (int e = 0; e < 8; e += 4)
            *reinterpret_cast<float4 *>(sred + ((size_t)d0 * RT + r) * width + (tid % tc) * 8 + e) = make_float4(acc[r][e], acc[r][e + 1], acc[r][e + 2], acc[r][e + 3]);
    __syncthreads();
    for (int i = tid; i < nr * width; i += kThreads) {
        const int r = i / width, c = i - r * width, gc = blockIdx.x * width + c;
        if (gc >= m.R) continue;
        float s = 0.f;
        for (int g = 0; g < dg; g++) s += sred[((size_t)g * RT + r) * width + c];
        store_c(reinterpret_cast<CT *>(j.qa) + ((size_t)(row0 + r) * m.H + h) * m.ld + gc, s);
    }
    if (blockIdx.x == 0) {
        const int tail = m.ld - m.R;
        for (int i = tid; i < nr * tail; i += kThreads) {
            const int r = i / tail, e = i - r * tail;
            const size_t tab = (size_t)row_rope(j, row0 + r) * (m.rot / 2);
            const float v = e < m.RD ? turned(m.q + (size_t)(row0 + r) * m.ldq + (size_t)h * hd + m.D, e, m.rot, m.rot_cos + tab, m.rot_sin + tab) : 0.f;
            store_c(reinterpret_cast<CT *>(j.qa) + ((size_t)(row0 + r) * m.H + h) * m.ld + m.R + e, v);
        }
    }
}

// ================================================================ scores and weighted latents, f16 cache
// Grid (splits, groups of 16 heads, rows).  PW: 16-column pairs of n-blocks a warp owns (R <= 128 PW).
template <int PW>
__global__ void __launch_bounds__(kThreads) latent_attn_tc_kernel(const MixLatentRows j, int max_split)
{
    extern __shared__ __align__(16) uint8_t at_smem[];
    const MixLatent &m = j.m;
    const int LQ = m.ld + 8;                                 // 16-byte rows an odd number of them apart: conflict-free ldmatrix
    __half *sQ = reinterpret_cast<__half *>(at_smem), *sC = sQ + kHeads * LQ;
    float *sS = reinterpret_cast<float *>(sC + kKeys * LQ);
    __half *sPh = reinterpret_cast<__half *>(sS + kHeads * (kKeys + 4)), *sPl = sPh + kHeads * (kKeys + 8);
    float *s_m = reinterpret_cast<float *>(sPl + kHeads * (kKeys + 8)), *s_l = s_m + kHeads, *s_corr = s_l + kHeads;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * kHeads, row = blockIdx.z, nh = min(kHeads, m.H - h0);
    // the position was complete before the launch in front of this one started; of the cache only L2 is asked ahead of the wait
    const int pos = row_pos(j, row);
    const Cut cut = cut_keys(pos, m.window, max_split);
    if (split >= cut.used) { pdl_wait(); pdl_launch_dependents(); return; }
    const int key0 = cut.first + split * cut.per * kKeys, key_end = min(pos + 1, key0 + cut.per * kKeys);
    const __half *cache = reinterpret_cast<const __half *>(m.cache) + (size_t)(j.seq0 + row * j.seq_step) * m.seq_stride;
    {
        const char *p = reinterpret_cast<const char *>(cache + (size_t)key0 * m.ld);
        const size_t bytes = (size_t)min(kKeys, key_end - key0) * m.ld * 2;
        for (size_t i = (size_t)tid * 128; i < bytes; i += kThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(p + i));
    }
    pdl_wait();
    pdl_launch_dependents();
    const int vecs = m.ld / 8;
    const __half *qa = reinterpret_cast<const __half *>(j.qa) + ((size_t)row * m.H + h0) * m.ld;
    for (int i = tid; i < kHeads * vecs; i += kThreads) {
        const int h = i / vecs, v = i - h * vecs;
        if (h < nh) cp_async16(smem_u32(sQ + h * LQ + v * 8), qa + (size_t)h * m.ld + v * 8);
        else *reinterpret_cast<uint4 *>(sQ + h * LQ + v * 8) = make_uint4(0u, 0u, 0u, 0u);
    }
    auto tile_async = [&](int k0) {
        for (int i = tid; i < kKeys * vecs; i += kThreads) {
            const int k = i / vecs, v = i - k * vecs;
            cp_async16(smem_u32(sC + k * LQ + v * 8), cache + (size_t)min(k0 + k, pos) * m.ld + v * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    tile_async(key0);
    if (tid < kHeads) { s_m[tid] = -INFINITY; s_l[tid] = 0.f; }
    const int pairs = (m.R + 15) / 16;
    float o[PW][2][4] = {};
    const uint32_t qaddr = smem_u32(sQ + (lane & 15) * LQ + (lane >> 4) * 8);
    const uint32_t kaddr = smem_u32(sC + (warp * 8 + (lane & 7)) * LQ + ((lane >> 3) & 3) * 8);
    const uint32_t paddr = (uint32_t)((lane & 15) * (kKeys + 8) + (lane >> 4) * 8) * 2;
    const uint32_t ph0 = smem_u32(sPh) + paddr, pl0 = smem_u32(sPl) + paddr;
    for (int k0 = key0; k0 < key_end; k0 += kKeys) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        {   // scores of 16 heads x this warp's 8 keys
            float s[2][4] = {};
            int ks = 0;
            for (; ks + 32 <= m.ld; ks += 32) {
                uint32_t a[2][4], b[4];
                ldmatrix_x4(qaddr + ks * 2, a[0][0], a[0][1], a[0][2], a[0][3]);
                ldmatrix_x4(qaddr + ks * 2 + 32, a[1][0], a[1][1], a[1][2], a[1][3]);
                ldmatrix_x4(kaddr + ks * 2, b[0], b[1], b[2], b[3]);
                hmma16816(s[0], a[0][0], a[0][1], a[0][2], a[0][3], b[0], b[1]);
                hmma16816(s[1], a[1][0], a[1][1], a[1][2], a[1][3], b[2], b[3]);
            }
            if (ks < m.ld) {                                   // ld is a multiple of 16
                uint32_t a[4], b[2];
                ldmatrix_x4(qaddr + ks * 2, a[0], a[1], a[2], a[3]);
                ldmatrix_x2(smem_u32(sC + (warp * 8 + (lane & 7)) * LQ + ((lane >> 3) & 1) * 8 + ks), b[0], b[1]);
                hmma16816(s[0], a[0], a[1], a[2], a[3], b[0], b[1]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int k = warp * 8 + 2 * c + (e & 1);
                sS[(g + 8 * (e >> 1)) * (kKeys + 4) + k] = k0 + k < key_end ? (s[0][e] + s[1][e]) * m.scale : -INFINITY;
            }
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < 2; r++) {                          // two heads per warp
            const int h = warp * 2 + r;
            const float a = sS[h * (kKeys + 4) + lane], b = sS[h * (kKeys + 4) + 32 + lane];
            float mx = fmaxf(a, b);
#pragma unroll
            for (int d = 16; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float old = s_m[h], mn = fmaxf(old, mx);     // the first key of every tile is visible: finite
            const float ea = expf(a - mn), eb = expf(b - mn), sum = warp_sum(ea + eb);
            const __half ha = __float2half_rn(ea), hb = __float2half_rn(eb);
            sPh[h * (kKeys + 8) + lane] = ha;
            sPh[h * (kKeys + 8) + 32 + lane] = hb;
            sPl[h * (kKeys + 8) + lane] = __float2half_rn(ea - __half2float(ha));
            sPl[h * (kKeys + 8) + 32 + lane] = __float2half_rn(eb - __half2float(hb));
            __syncwarp();
            if (lane == 0) {
                const float corr = expf(old - mn);
                s_corr[h] = corr;
                s_m[h] = mn;
                s_l[h] = s_l[h] * corr + sum;
            }
        }
        __syncthreads();
        const float c0 = s_corr[g], c1 = s_corr[g + 8];
#pragma unroll
        for (int i = 0; i < PW; i++)
#pragma unroll
            for (int n = 0; n < 2; n++) { o[i][n][0] *= c0; o[i][n][1] *= c0; o[i][n][2] *= c1; o[i][n][3] *= c1; }
#pragma unroll
        for (int ks = 0; ks < kKeys / 16; ks++) {
            uint32_t ph[4], pl[4];
            ldmatrix_x4(ph0 + ks * 32, ph[0], ph[1], ph[2], ph[3]);
            ldmatrix_x4(pl0 + ks * 32, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
            for (int i = 0; i < PW; i++) {
                const int pr = warp + i * kWarps;
                if (pr < pairs) {
                    uint32_t v[4];
                    ldmatrix_x4_trans(smem_u32(sC + (ks * 16 + (lane & 15)) * LQ + pr * 16 + (lane >> 4) * 8), v[0], v[1], v[2], v[3]);
                    hmma16816(o[i][0], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
                    hmma16816(o[i][1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
                    hmma16816(o[i][0], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
                    hmma16816(o[i][1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
                }
            }
        }
        __syncthreads();
        if (k0 + kKeys < key_end) tile_async(k0 + kKeys);
    }
    const int prow = part_row(m.R);
    float *part = j.partial + (((size_t)row * max_split + split) * m.H + h0) * prow;
#pragma unroll
    for (int i = 0; i < PW; i++) {
        const int pr = warp + i * kWarps;
        if (pr >= pairs) continue;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int h = g + 8 * (e >> 1), col = pr * 16 + n * 8 + 2 * c + (e & 1);
                if (h < nh && col < m.R) part[(size_t)h * prow + col] = o[i][n][e];
            }
    }
    if (tid < nh) { part[(size_t)tid * prow + prow - 4] = s_m[tid]; part[(size_t)tid * prow + prow - 3] = s_l[tid]; }
}

// ================================================================ the same in 32 bits: grid (splits, heads, rows)
__global__ void __launch_bounds__(kThreads) latent_attn_f32_kernel(const MixLatentRows j, int max_split)
{
    extern __shared__ __align__(16) float sq[];              // [ld]
    __shared__ float sw[kKeys], s_corr;
    const MixLatent &m = j.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, split = blockIdx.x, h = blockIdx.y, row = blockIdx.z;
    const int pos = row_pos(j, row);
    const Cut cut = cut_keys(pos, m.window, max_split);
    pdl_wait();
    pdl_launch_dependents();
    if (split >= cut.used) return;
    const int key0 = cut.first + split * cut.per * kKeys, key_end = min(pos + 1, key0 + cut.per * kKeys);
    const float *cache = reinterpret_cast<const float *>(m.cache) + (size_t)(j.seq0 + row * j.seq_step) * m.seq_stride;
    const float *qa = reinterpret_cast<const float *>(j.qa) + ((size_t)row * m.H + h) * m.ld;
    for (int i = tid; i < m.ld; i += kThreads) sq[i] = __ldcg(qa + i);
    __syncthreads();
    constexpr int NA = kMaxLatentF32 / kThreads;
    float o[NA] = {}, mx = -INFINITY, l = 0.f;               // mx, l: warp 0
    for (int k0 = key0; k0 < key_end; k0 += kKeys) {
        const int nk = min(kKeys, key_end - k0);
        for (int k = warp; k < nk; k += kWarps) {
            const float *kr = cache + (size_t)(k0 + k) * m.ld;
            float s = 0.f;
            for (int i = lane * 4; i < m.ld; i += 128) {
                const float4 a = *reinterpret_cast<const float4 *>(sq + i), b = __ldcg(reinterpret_cast<const float4 *>(kr + i));
                s = fmaf(a.x, b.x, s); s = fmaf(a.y, b.y, s); s = fmaf(a.z, b.z, s); s = fmaf(a.w, b.w, s);
            }
            s = warp_sum(s);
            if (lane == 0) sw[k] = s * m.scale;
        }
        __syncthreads();
        if (warp == 0) {
            const float a = lane < nk ? sw[lane] : -INFINITY, b = lane + 32 < nk ? sw[lane + 32] : -INFINITY;
            float mn = fmaxf(a, b);
            for (int d = 16; d; d >>= 1) mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, d));
            mn = fmaxf(mn, mx);
            const float ea = expf(a - mn), eb = expf(b - mn), corr = expf(mx - mn);
            sw[lane] = ea; sw[lane + 32] = eb;
            l = l * corr + warp_sum(ea + eb);
            mx = mn;
            if (lane == 0) s_corr = corr;
        }
        __syncthreads();
        const float corr = s_corr;
#pragma unroll
        for (int i = 0; i < NA; i++) {
            const int col = tid + i * kThreads;
            if (col < m.R) {
                float a = o[i] * corr;
                for (int k = 0; k < nk; k++) a = fmaf(sw[k], __ldcg(cache + (size_t)(k0 + k) * m.ld + col), a);
                o[i] = a;
            }
        }
        __syncthreads();
    }
    const int prow = part_row(m.R);
    float *part = j.partial + (((size_t)row * max_split + split) * m.H + h) * prow;
#pragma unroll
    for (int i = 0; i < NA; i++)
        if (tid + i * kThreads < m.R) part[tid + i * kThreads] = o[i];
    if (tid == 0) { part[prow - 4] = mx; part[prow - 3] = l; }
}

// ================================================================ merge, values, gate: grid (slices of 32 outputs, heads, rows)
template <typename TO>
__global__ void __launch_bounds__(kThreads) latent_value_kernel(const MixLatentRows j, int max_split)
{
    extern __shared__ __align__(16) float so[];              // [ldv] merged latents, then [groups][items] float4
    __shared__ float s_f[kMaxSplits];
    const MixLatent &m = j.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, row = blockIdx.z;
    const int j0 = blockIdx.x * 32 + warp * 4, nv = m.uv.ld / 8;
    const __nv_bfloat16 *w[4];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        w[r] = m.uv.w + ((size_t)h * m.DV + min(j0 + r, m.DV - 1)) * m.uv.ld;
        for (int e = 512 + lane * 64; e < m.uv.ld; e += 32 * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(w[r] + e));
    }
    const Cut cut = cut_keys(row_pos(j, row), m.window, max_split);
    uint4 pre[4][2];                                         // the weights' first 512 columns, ahead of the wait
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int i = 0; i < 2; i++) pre[r][i] = lane + 32 * i < nv ? *reinterpret_cast<const uint4 *>(w[r] + (lane + 32 * i) * 8) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    pdl_launch_dependents();
    const int prow = part_row(m.R);
    const size_t step = (size_t)m.H * prow;
    const float *part = j.partial + ((size_t)row * max_split * m.H + h) * prow;
    if (warp == 0) {
        float ml[2], ll[2], mx = -INFINITY, den = 0.f;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int s = lane + 32 * i;
            ml[i] = s < cut.used ? __ldcg(part + s * step + prow - 4) : -INFINITY;
            ll[i] = s < cut.used ? __ldcg(part + s * step + prow - 3) : 0.f;
            mx = fmaxf(mx, ml[i]);
        }
        for (int d = 16; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
#pragma unroll
        for (int i = 0; i < 2; i++) { ml[i] = expf(ml[i] - mx); den += ml[i] * ll[i]; }
        den = warp_sum(den);
#pragma unroll
        for (int i = 0; i < 2; i++) s_f[lane + 32 * i] = ml[i] / den;
    }
    __syncthreads();
    const int items = (prow - 4) / 4, groups = max(1, kThreads / items);
    float4 *sp = reinterpret_cast<float4 *>(so + (m.uv.ld + 3) / 4 * 4);
    for (int i0 = 0; i0 < items; i0 += kThreads) {
        const int gr = groups > 1 ? tid / items : 0, it = groups > 1 ? tid % items : i0 + tid;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (gr < groups && it < items) {
#pragma unroll 8
            for (int s = gr; s < cut.used; s += groups) {
                const float4 x = __ldcg(reinterpret_cast<const float4 *>(part + s * step) + it);
                const float f = s_f[s];
                a.x = fmaf(f, x.x, a.x); a.y = fmaf(f, x.y, a.y); a.z = fmaf(f, x.z, a.z); a.w = fmaf(f, x.w, a.w);
            }
            if (groups > 1) sp[gr * items + it] = a;
            else *reinterpret_cast<float4 *>(so + it * 4) = a;
        }
    }
    __syncthreads();
    if (groups > 1) {
        for (int it = tid; it < items; it += kThreads) {
            float4 a = sp[it];
            for (int gr = 1; gr < groups; gr++) {
                const float4 x = sp[gr * items + it];
                a.x += x.x; a.y += x.y; a.z += x.z; a.w += x.w;
            }
            *reinterpret_cast<float4 *>(so + it * 4) = a;
        }
        __syncthreads();
    }
    for (int e = m.R + tid; e < (m.uv.ld + 3) / 4 * 4; e += kThreads) so[e] = 0.f;       // the weight's padding meets zeros
    __syncthreads();
    float acc[4] = {};
    auto mul = [&](int v, const uint4 (&x)[4]) {
        const float4 a = *reinterpret_cast<const float4 *>(so + v * 8), b = *reinterpret_cast<const float4 *>(so + v * 8 + 4);
#pragma unroll
        for (int r = 0; r < 4; r++) {
            float s = acc[r];
            s = fmaf(bf_lo(x[r].x), a.x, s); s = fmaf(bf_hi(x[r].x), a.y, s);
            s = fmaf(bf_lo(x[r].y), a.z, s); s = fmaf(bf_hi(x[r].y), a.w, s);
            s = fmaf(bf_lo(x[r].z), b.x, s); s = fmaf(bf_hi(x[r].z), b.y, s);
            s = fmaf(bf_lo(x[r].w), b.z, s); s = fmaf(bf_hi(x[r].w), b.w, s);
            acc[r] = s;
        }
    };
#pragma unroll
    for (int i = 0; i < 2; i++)
        if (lane + 32 * i < nv) {
            const uint4 x[4] = {pre[0][i], pre[1][i], pre[2][i], pre[3][i]};
            mul(lane + 32 * i, x);
        }
    for (int v = lane + 64; v < nv; v += 32) {
        uint4 x[4];
#pragma unroll
        for (int r = 0; r < 4; r++) x[r] = *reinterpret_cast<const uint4 *>(w[r] + v * 8);
        mul(v, x);
    }
#pragma unroll
    for (int r = 0; r < 4; r++) acc[r] = warp_sum(acc[r]);
    const float y = lane == 0 ? acc[0] : (lane == 1 ? acc[1] : (lane == 2 ? acc[2] : acc[3]));
    const int col = h * m.DV + j0 + lane;
    if (lane < 4 && j0 + lane < m.DV) {
        const float gate = m.gate ? sigmoidf(__ldcg(m.gate + (size_t)row * m.ld_gate + col)) : 1.f;
        store_actv(reinterpret_cast<TO *>(j.out) + (size_t)row * j.ldo + col, y * gate);
    }
}

// ================================================================ long portions
// rotates the queries of a token in place (or, with QD, into f16 rows whose heads are padded to QD) and appends its cache row
template <typename CT, int QD>
__global__ void __launch_bounds__(kThreads) latent_prep_kernel(const MixLatent m, int seq, int pos0, int rope0, int rope_step, __half *__restrict__ q16)
{
    constexpr int kPairs = QD ? QD / 2 : 1;
    __shared__ float part[kWarps], inv[1];
    const int t = blockIdx.x, rope = rope0 + t * rope_step, half = m.rot / 2, hd = m.D + m.RD;
    const float *c = m.rot_cos + (size_t)rope * half, *s = m.rot_sin + (size_t)rope * half;
    float *q = m.q + (size_t)t * m.ldq;
    if (QD) {
        __half2 *dst = reinterpret_cast<__half2 *>(q16 + (size_t)t * m.H * QD);
        auto clamp = [](float v) { return fminf(fmaxf(v, -65504.f), 65504.f); };
        if (m.D % 2 == 0 && m.RD % 2 == 0 && m.ldq % 2 == 0 && (reinterpret_cast<uintptr_t>(m.q) & 7) == 0) {
#pragma unroll 4
            for (int i = threadIdx.x; i < m.H * kPairs; i += kThreads) {
                const int h = i / kPairs, d = (i - h * kPairs) * 2, r = d - m.D;
                float2 v = d < hd ? __ldcg(reinterpret_cast<const float2 *>(q + (size_t)h * hd + d)) : make_float2(0.f, 0.f);
                if (r >= 0 && r < m.rot) {
                    const float cs = c[r >> 1], sn = s[r >> 1];
                    v = make_float2(v.x * cs - v.y * sn, v.y * cs + v.x * sn);
                }
                dst[i] = __floats2half2_rn(clamp(v.x), clamp(v.y));
            }
        } else {
            auto value = [&](const float *x, int d) { return d < m.D ? __ldcg(x + d) : (d < hd ? turned(x + m.D, d - m.D, m.rot, c, s) : 0.f); };
            for (int i = threadIdx.x; i < m.H * kPairs; i += kThreads) {
                const int h = i / kPairs, d = (i - h * kPairs) * 2;
                const float *x = q + (size_t)h * hd;
                dst[i] = __floats2half2_rn(clamp(value(x, d)), clamp(value(x, d + 1)));
            }
        }
    } else {
        for (int i = threadIdx.x; i < m.H * half; i += kThreads) {
            const int h = i / half, k = i - h * half;
            float *x = q + (size_t)h * hd + m.D + 2 * k;
            const float u = x[0], v = x[1];
            x[0] = u * c[k] - v * s[k];
            x[1] = v * c[k] + u * s[k];
        }
    }
    append_row<CT>(m, seq, pos0 + t, rope, m.kv + (size_t)t * m.ldkv, part, inv);
}

// the rotated part of every key beside each head's expanded one, and zeros up to the pitch
template <typename CT>
__global__ void __launch_bounds__(kThreads) latent_rot_kernel(const MixLatent m, const CT *__restrict__ cache, CT *__restrict__ keys, int n_keys, int ldk)
{
    const int key = blockIdx.x, tail = ldk - m.D;
    const CT *src = cache + (size_t)key * m.ld + m.R;
    constexpr int VE = 16 / sizeof(CT);
    if (m.D % VE == 0 && m.R % VE == 0 && m.RD % VE == 0) {
        const int nv = tail / VE;
        for (int i = threadIdx.x; i < m.H * nv; i += kThreads) {
            const int h = i / nv, v = i - h * nv;
            *reinterpret_cast<uint4 *>(keys + ((size_t)h * n_keys + key) * ldk + m.D + v * VE) =
                v * VE < m.RD ? *reinterpret_cast<const uint4 *>(src + v * VE) : make_uint4(0u, 0u, 0u, 0u);
        }
        return;
    }
    for (int i = threadIdx.x; i < m.H * tail; i += kThreads) {
        const int h = i / tail, e = i - h * tail;
        keys[((size_t)h * n_keys + key) * ldk + m.D + e] = e < m.RD ? src[e] : (CT)0.f;
    }
}

int max_splits(const MixLatent &m, int rows, bool f32)
{
    const int tiles = (std::min(m.window, m.max_seq) + kKeys - 1) / kKeys, per_row = f32 ? m.H : (m.H + kHeads - 1) / kHeads;
    return std::max(1, std::min(std::min(tiles, kMaxSplits), 2 * ctx()->sm_count / std::max(1, rows * per_row)));
}

size_t attn_tc_smem(const MixLatent &m)
{
    return (size_t)(kHeads + kKeys) * (m.ld + 8) * 2 + (size_t)kHeads * (kKeys + 4) * 4 + (size_t)2 * kHeads * (kKeys + 8) * 2 + 3 * kHeads * 4;
}

template <int PW>
tlb_status run_attn_tc(const MixLatentRows &j, int splits)
{
    const size_t smem = attn_tc_smem(j.m);
    static size_t allowed = 40 << 10;      // with the static part, under the 48 KB that need no asking
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(latent_attn_tc_kernel<PW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    TLB_CUDA(launch_chained(latent_attn_tc_kernel<PW>, dim3(splits, (j.m.H + kHeads - 1) / kHeads, j.rows), dim3(kThreads), smem, j.pdl, j, splits));
    count_launch();
    return TLB_OK;
}

template <typename CT, int RT>
tlb_status run_query(const MixLatentRows &j)
{
    const MixLatent &m = j.m;
    // few rows: narrow column chunks, so that a thread has all its weights in flight at once
    const int vecs = m.uk.ld / 8, tiles = (j.rows + RT - 1) / RT;
    int tc = 8;
    while (tc < 64 && tc < vecs && (vecs / tc) * m.H * tiles > 4 * ctx()->sm_count) tc *= 2;
    const size_t smem = ((size_t)(RT * m.D + 3) / 4 * 4 + (size_t)kThreads * RT * 8) * sizeof(float);
    static size_t allowed = 40 << 10;      // with the static part, under the 48 KB that need no asking
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(latent_query_kernel<CT, RT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    TLB_CUDA(launch_chained(latent_query_kernel<CT, RT>, dim3((vecs + tc - 1) / tc, m.H + 1, tiles), dim3(kThreads), smem, j.pdl, j, tc));
    count_launch();
    return TLB_OK;
}

template <typename TO>
tlb_status run_value(const MixLatentRows &j, int splits)
{
    const MixLatent &m = j.m;
    const int items = (part_row(m.R) - 4) / 4, groups = std::max(1, kThreads / items);
    const size_t smem = ((size_t)(m.uv.ld + 3) / 4 * 4 + (groups > 1 ? (size_t)groups * items * 4 : 0)) * sizeof(float);
    TLB_CUDA(launch_chained(latent_value_kernel<TO>, dim3((m.DV + 31) / 32, m.H, j.rows), dim3(kThreads), smem, j.pdl, j, splits));
    count_launch();
    return TLB_OK;
}

}  // namespace

int latent_ld(int R, int RD) { return (R + RD + 15) / 16 * 16; }

bool latent_supported(const MixLatent &m, bool f32)
{
    if (m.D < 1 || m.D > 4096 || m.H < 1 || m.H > 1024 || m.DV < 1 || m.DV > 4096) return false;
    return f32 ? m.R <= kMaxLatentF32 && m.ld <= 8192 : m.R <= 1024 && attn_tc_smem(m) <= ctx()->smem_optin;
}

size_t latent_partial_floats(const MixLatent &m, int rows)
{
    return (size_t)rows * std::max(max_splits(m, rows, false), max_splits(m, rows, true)) * m.H * part_row(m.R);
}

bool latent_expands(const MixLatent &m, int T)
{
    if (m.D + m.RD > kMaxExpandedHead || m.DV > kMaxExpandedHead) return false;
    // Expanding a key costs R (D + DV) products per head, once; attending it as a latent 2 R - D - DV more per query.
    const int even = (int)((int64_t)m.R * (m.D + m.DV) / std::max(1, 2 * m.R - m.D - m.DV) / 4);
    return T >= std::min(64, std::max(8, even));
}

tlb_status launch_latent_rows(const MixLatentRows &j)
{
    if (!ctx()) return TLB_ERR_DEVICE;
    if (j.rows < 1) return TLB_OK;
    const int splits = max_splits(j.m, j.rows, j.f32);
    if (j.f32) {
        TLB_TRY(j.rows == 1 ? (run_query<float, 1>(j)) : (run_query<float, 4>(j)));
        TLB_CUDA(launch_chained(latent_attn_f32_kernel, dim3(splits, j.m.H, j.rows), dim3(kThreads), (size_t)j.m.ld * sizeof(float), j.pdl, j, splits));
        count_launch();
    } else {
        TLB_TRY(j.rows == 1 ? (run_query<__half, 1>(j)) : (run_query<__half, 4>(j)));
        if (j.m.R <= 128) TLB_TRY(run_attn_tc<1>(j, splits));
        else if (j.m.R <= 256) TLB_TRY(run_attn_tc<2>(j, splits));
        else if (j.m.R <= 512) TLB_TRY(run_attn_tc<4>(j, splits));
        else TLB_TRY(run_attn_tc<8>(j, splits));
    }
    return j.out_f32 ? run_value<float>(j, splits) : run_value<__nv_bfloat16>(j, splits);
}

tlb_status launch_latent_prompt(const MixLatent &m, int seq, int T, int pos0, int rope0, int rope_step, void *out, int ldo, bool f32)
{
    Context *c = ctx();
    if (!c) return TLB_ERR_DEVICE;
    const size_t es = f32 ? 4 : 2;
    // the latents some query sees, from a tile border of the prompt attention on, as keys and values per head
    const int key_first = std::max(0, pos0 - m.window + 1) / 128 * 128, n_keys = pos0 + T - key_first;
    const int hd = m.D + m.RD, ldk = act_ld(hd), ldv = act_ld(m.DV), qd = mix_attn_tc5_qd(hd), vt_ld = (n_keys + 127) / 128 * 128;
    // the tcgen05 kernel takes f16 queries and V^T, which the kernels here write at once
    const bool tc5 = !f32 && mix_attn_prefill_tc5_supported(hd, m.DV, T);
    std::vector<Storage *> held;
    auto done = [&](tlb_status st) { for (Storage *s : held) storage_release(s); return st; };
    auto get = [&](size_t bytes) -> void * {
        Storage *s = storage_alloc(bytes);
        if (!s) return nullptr;
        held.push_back(s);
        return s->ptr;
    };
    void *keys = get((size_t)m.H * n_keys * ldk * es), *vals = get((size_t)m.H * (tc5 ? (size_t)128 * vt_ld : (size_t)n_keys * ldv) * es);
    __half *q16 = tc5 ? (__half *)get((size_t)T * m.H * qd * 2) : nullptr;
    if (!keys || !vals || (tc5 && !q16)) return done(TLB_ERR_ALLOC);
    if (f32) latent_prep_kernel<float, 0><<<T, kThreads, 0, c->stream>>>(m, seq, pos0, rope0, rope_step, nullptr);
    else if (!tc5) latent_prep_kernel<__half, 0><<<T, kThreads, 0, c->stream>>>(m, seq, pos0, rope0, rope_step, nullptr);
    else if (qd == 128) latent_prep_kernel<__half, 128><<<T, kThreads, 0, c->stream>>>(m, seq, pos0, rope0, rope_step, q16);
    else latent_prep_kernel<__half, 192><<<T, kThreads, 0, c->stream>>>(m, seq, pos0, rope0, rope_step, q16);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return done(cuda_fail(e, "latent preparation launch"));
    const char *cache = (const char *)m.cache + ((size_t)seq * m.seq_stride + (size_t)key_first * m.ld) * es;
    DenseGemmJob j;
    j.x = cache; j.ldx = m.ld; j.T = n_keys;
    j.w = f32 ? m.uk : m.uk16; j.per = m.D; j.ldo = ldk; j.block_stride = (size_t)n_keys * ldk;
    (f32 ? (void *&)j.out : (void *&)j.out_h) = keys;
    tlb_status st = launch_dense_gemm(j, f32);
    if (st != TLB_OK) return done(st);
    j.out = nullptr; j.out_h = nullptr;
    j.w = f32 ? m.uv : m.uv16; j.per = m.DV;
    if (tc5) { j.out_t = (__half *)vals; j.ldo = vt_ld; j.block_stride = (size_t)128 * vt_ld; }
    else { (f32 ? (void *&)j.out : (void *&)j.out_h) = vals; j.ldo = ldv; j.block_stride = (size_t)n_keys * ldv; }
    st = launch_dense_gemm(j, f32);
    if (st != TLB_OK) return done(st);
    if (f32) latent_rot_kernel<float><<<n_keys, kThreads, 0, c->stream>>>(m, (const float *)cache, (float *)keys, n_keys, ldk);
    else latent_rot_kernel<__half><<<n_keys, kThreads, 0, c->stream>>>(m, (const __half *)cache, (__half *)keys, n_keys, ldk);
    e = cudaGetLastError();
    if (e != cudaSuccess) return done(cuda_fail(e, "latent expansion launch"));
    count_launch(2);
    MixAttn a = {};
    a.H = a.KVH = m.H; a.D = hd; a.DV = m.DV; a.ldk = ldk; a.ldv = ldv; a.max_seq = n_keys; a.window = m.window; a.scale = m.scale;
    a.bias_n = 1;
    a.kcache = keys; a.vcache = vals; a.proj = m.q; a.ldp = m.ldq; a.gate = m.gate; a.ld_gate = m.ld_gate;
    if (tc5) { a.q16 = q16; a.vt = (const __half *)vals; a.vt_ld = vt_ld; }
    return done(launch_mix_attn_prompt(a, 0, T, pos0 - key_first, out, ldo, f32));
}

}  // namespace tlb
