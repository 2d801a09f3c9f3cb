// Linear recurrences with a matrix state per head, in 32-bit floats throughout.
//   retention       S <- decay S + k v^T;                                        o = S^T q
//   general delta   S <- diag(w) S - (a u)(u^T S) + k v^T,  u = k / |k|;         o = S^T r
// The state's value channels (columns) never mix, so a column lives in the registers of a few lanes - each some
// of its key channels - from the first token of a launch to the last: a prompt is scanned token by token as decoding would do it,
// whatever its length or the place where it was cut.
// State in memory: [sequence][head][value channel][key channel padded to a multiple of 32].
// Around the scan: what enters it is prepared per token and head (rotation and scale; decay, removal vector), what leaves it is
// divided by its root mean square per head and gated.  Decoding does all of it in one launch.
#include <algorithm>

#include "layered_kernels.h"
#include "qmv_common.cuh"

namespace tlb {

namespace {

constexpr int kScanThreads = 256, kScanTok = 16;      // consuming threads (a warp more fetches), tokens per chunk
constexpr int kStepThreads = 512, kStepCols = kStepThreads / 8;
constexpr float kUnitEps = 1e-6f;             // inside the root of the unit key

using f2 = unsigned long long;                // two floats for the packed multiply-adds
__device__ __forceinline__ f2 pack2(float a, float b) { f2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ float sum2(f2 a) { float x, y; asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a)); return x + y; }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) { f2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ f2 mul2(f2 a, f2 b) { f2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ f2 add2(f2 a, f2 b) { f2 d; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }

__device__ __forceinline__ void store_act(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_act(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_act4(float *p, float a, float b, float c, float d) { *reinterpret_cast<float4 *>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void store_act4(__nv_bfloat16 *p, float a, float b, float c, float d)
{
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float lanes8_sum(float v)
{
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
}
__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ void lds_f2x2(const float *p, f2 &a, f2 &b)
{
    const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(p);
    a = v.x; b = v.y;
}

// 2 NC pairs of a column's key channels: pair 2 c, 2 c + 1 = channels 32 c + 4 l .. + 3
template <int NC>
struct Column {
    f2 s[2 * NC];
    __device__ __forceinline__ void zero()
    {
#pragma unroll
        for (int i = 0; i < 2 * NC; i++) s[i] = 0ull;
    }
    __device__ __forceinline__ void load(const float *p, int l)
    {
#pragma unroll
        for (int c = 0; c < NC; c++) {
            const ulonglong2 v = __ldcg(reinterpret_cast<const ulonglong2 *>(p + 32 * c + 4 * l));
            s[2 * c] = v.x; s[2 * c + 1] = v.y;
        }
    }
    __device__ __forceinline__ void store(float *p, int l) const
    {
#pragma unroll
        for (int c = 0; c < NC; c++) *reinterpret_cast<ulonglong2 *>(p + 32 * c + 4 * l) = make_ulonglong2(s[2 * c], s[2 * c + 1]);
    }
    __device__ __forceinline__ float dot(const float *vec, int l) const      // this lane's share
    {
        f2 a = 0ull, b = 0ull;
#pragma unroll
        for (int c = 0; c < NC; c++) {
            f2 x, y;
            lds_f2x2(vec + 32 * c + 4 * l, x, y);
            a = fma2(x, s[2 * c], a);
            b = fma2(y, s[2 * c + 1], b);
        }
        return sum2(add2(a, b));
    }
    // s <- decay * s + k v, and this lane's share of q . s
    __device__ __forceinline__ float retain(const float *q, const float *k, f2 decay, float v, int l)
    {
        const f2 vv = pack2(v, v);
        f2 a = 0ull, b = 0ull;
#pragma unroll
        for (int c = 0; c < NC; c++) {
            f2 x, y;
            lds_f2x2(k + 32 * c + 4 * l, x, y);
            s[2 * c] = fma2(decay, s[2 * c], mul2(x, vv));
            s[2 * c + 1] = fma2(decay, s[2 * c + 1], mul2(y, vv));
            lds_f2x2(q + 32 * c + 4 * l, x, y);
            a = fma2(x, s[2 * c], a);
            b = fma2(y, s[2 * c + 1], b);
        }
        return sum2(add2(a, b));
    }
    // s <- w s - rem (k . s) + k v, and this lane's share of r . s; rem = a k / (k . k + eps)
    __device__ __forceinline__ float delta(const float *r, const float *k, const float *w, const float *rem, float v, int l)
    {
        const float ks = -lanes8_sum(dot(k, l));
        const f2 vv = pack2(v, v), kk = pack2(ks, ks);
        f2 a = 0ull, b = 0ull;
#pragma unroll
        for (int c = 0; c < NC; c++) {
            f2 k0, k1, w0, w1, e0, e1, r0, r1;
            lds_f2x2(k + 32 * c + 4 * l, k0, k1);
            lds_f2x2(w + 32 * c + 4 * l, w0, w1);
            lds_f2x2(rem + 32 * c + 4 * l, e0, e1);
            lds_f2x2(r + 32 * c + 4 * l, r0, r1);
            s[2 * c] = fma2(w0, s[2 * c], fma2(e0, kk, mul2(k0, vv)));
            s[2 * c + 1] = fma2(w1, s[2 * c + 1], fma2(e1, kk, mul2(k1, vv)));
            a = fma2(r0, s[2 * c], a);
            b = fma2(r1, s[2 * c + 1], b);
        }
        return sum2(add2(a, b));
    }
};

// ================================================================ scan of a prompt
// A group of L lanes owns CB columns; lane l of it holds key channels 4 (i L + l) .. + 3 for i < N4 of each, so a vector read from
// shared memory (16 bytes per lane, without bank conflicts) serves CB columns.  The outputs of L / CB tokens are summed over the
// lanes together: every lane ends up with one of them.
// General delta: u^T S of the next token is taken from the state BEFORE this token's update,
//   k'^T S_t = (k' w)^T S_(t-1) - (k' . rem) (k^T S_(t-1)) + (k' . k) v,
// so its reduction over the lanes overlaps this token's update instead of standing in front of the next one.
template <int NC> struct ScanShape {
    static constexpr int DP = 32 * NC, L = NC % 4 == 0 ? 32 : NC % 2 ? 8 : 16, N4 = DP / (4 * L), CB = N4 <= 4 ? 4 : 2, TB = L / CB;
    static constexpr int COLS = kScanThreads / L * CB;       // columns per CTA
};

struct ScanParams {
    int H, D, DV, T;
    const float *q, *k, *v, *w, *rem;         // row 0, head 0 of each; rows `ld*` apart, heads D (v: DV) apart
    int ldq, ldk, ldv, ldw, ldr;
    const float2 *look;                       // general delta: [H][look_ld] (k' . rem, k' . k) of the next token's key
    int look_ld;                              // >= T rounded up to a chunk
    int *err;
    const float *decay;
    float *state;                             // [H][DV][32 NC]
    int from_zero;
    float *o;                                 // [T][H * DV]
};

__device__ __forceinline__ void cp_async4(void *dst, const void *src)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
// N values per lane (N a power of two): afterwards lane l of every N consecutive lanes holds the sum over those N lanes of value
// l, with N - 1 shuffles.
template <int N>
__device__ __forceinline__ float scatter_sum(const float (&y)[N], int l)
{
    if constexpr (N == 1) {
        return y[0];
    } else {
        float a[N / 2];
        const bool up = l & (N / 2);
#pragma unroll
        for (int i = 0; i < N / 2; i++) a[i] = (up ? y[i + N / 2] : y[i]) + __shfl_xor_sync(0xffffffffu, up ? y[i] : y[i + N / 2], N / 2);
        return scatter_sum<N / 2>(a, l);
    }
}
// sums of N values over L lanes, in every lane
template <int N, int L>
__device__ __forceinline__ void all_sum(float (&y)[N], int lane)
{
    float s = scatter_sum<N>(y, lane);
#pragma unroll
    for (int o = N; o < L; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
#pragma unroll
    for (int c = 0; c < N; c++) y[c] = __shfl_sync(0xffffffffu, s, (lane & ~(N - 1)) | c);
}

template <int NC, bool DELTA>
__global__ void __launch_bounds__(kScanThreads + 32) scan_kernel(const ScanParams p)
{
    using S = ScanShape<NC>;
    constexpr int DP = S::DP, L = S::L, N4 = S::N4, CB = S::CB, TB = S::TB, COLS = S::COLS, NP = 2 * N4;
    constexpr int NV = DELTA ? 4 : 2, ROW = NV * DP + COLS, BUF = kScanTok * ROW + DP + 2 * kScanTok;     // k has one row more than the chunk
    extern __shared__ __align__(16) float scan_smem[];       // [2][BUF]: rows of q, k, (w, rem), value channels; one more key; look-ahead products
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = lane % L, h = blockIdx.y, c0 = blockIdx.x * COLS, col = tid / L * CB;
    __shared__ __align__(8) unsigned long long full_bar[2];
    __shared__ int abort_word;
    volatile int *abort_flag = &abort_word;
    for (int i = tid; i < 2 * BUF; i += kScanThreads + 32) scan_smem[i] = 0.f;
    if (tid == 0) {
        abort_word = 0;
        mbar_init(smem_u32(full_bar), 1);
        mbar_init(smem_u32(full_bar + 1), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");     // the zeros above before bulk copies into the same rows
    __syncthreads();
    const float *src[4] = {p.q + (size_t)h * p.D, p.k + (size_t)h * p.D, DELTA ? p.w + (size_t)h * p.D : nullptr, DELTA ? p.rem + (size_t)h * p.D : nullptr};
    const int lds[4] = {p.ldq, p.ldk, p.ldw, p.ldr};
    const int nv = min(COLS, p.DV - c0);
    const float *vsrc = p.v + (size_t)h * p.DV + c0;
    // rows that start and end on 16 bytes come as bulk copies, others element by element
    bool wide = p.D % 4 == 0 && nv % 4 == 0 && p.ldv % 4 == 0 && (reinterpret_cast<uintptr_t>(vsrc) & 15) == 0;
#pragma unroll
    for (int i = 0; i < NV; i++) wide = wide && lds[i] % 4 == 0 && (reinterpret_cast<uintptr_t>(src[i]) & 15) == 0;
    if (warp == kScanThreads / 32) {
        // ------------------------------------------------ the fetching warp: a chunk ahead of the others
        auto fetch = [&](int t0, int b) {
            float *buf = scan_smem + b * BUF;
            const int nt = min(kScanTok, p.T - t0), nk = DELTA ? min(kScanTok + 1, p.T - t0) : nt;     // the key behind the chunk comes too
            const uint32_t bar = smem_u32(full_bar + b);
            const float2 *look = DELTA ? p.look + (size_t)h * p.look_ld + t0 : nullptr;
            if (wide) {
                if (lane == 0) mbar_expect_tx(bar, (uint32_t)(((NV - 1) * nt + nk) * p.D * 4 + nt * nv * 4 + (DELTA ? kScanTok * 8 : 0)));
                __syncwarp();
                for (int i = lane; i < NV * kScanTok + 1; i += 32) {
                    const bool extra = i == NV * kScanTok;
                    const int j = extra ? 1 : i / kScanTok, t = extra ? kScanTok : i % kScanTok;
                    if (t >= (j == 1 ? nk : nt)) continue;
                    const float *s = j == 0 ? src[0] : (j == 1 ? src[1] : (j == 2 ? src[2] : src[3]));
                    const int ld = j == 0 ? lds[0] : (j == 1 ? lds[1] : (j == 2 ? lds[2] : lds[3]));
                    bulk_g2s(smem_u32(extra ? buf + kScanTok * ROW : buf + t * ROW + j * DP), s + (size_t)(t0 + t) * ld, (uint32_t)p.D * 4, bar);
                }
                if (lane < nt) bulk_g2s(smem_u32(buf + lane * ROW + NV * DP), vsrc + (size_t)(t0 + lane) * p.ldv, (uint32_t)nv * 4, bar);
                if (DELTA && lane == 0) bulk_g2s(smem_u32(buf + kScanTok * ROW + DP), look, kScanTok * 8, bar);
            } else {
                for (int i = 0; i < NV; i++)
                    for (int t = 0; t < (i == 1 ? nk : nt); t++) {
                        float *dst = t == kScanTok ? buf + kScanTok * ROW : buf + t * ROW + i * DP;
                        for (int d = lane; d < p.D; d += 32) cp_async4(dst + d, src[i] + (size_t)(t0 + t) * lds[i] + d);
                    }
                for (int t = 0; t < nt; t++)
                    for (int d = lane; d < nv; d += 32) cp_async4(buf + t * ROW + NV * DP + d, vsrc + (size_t)(t0 + t) * p.ldv + d);
                if (DELTA && lane < 2 * kScanTok) cp_async4(buf + kScanTok * ROW + DP + lane, reinterpret_cast<const float *>(look) + lane);
                asm volatile("cp.async.wait_all;" ::: "memory");
                __syncwarp();
                if (lane == 0) mbar_arrive(bar);
            }
        };
        fetch(0, 0);
        for (int t0 = 0, c = 0; t0 < p.T; t0 += kScanTok, c++) {
            // buffer (c + 1) & 1 was left by the barrier that ended chunk c - 1
            if (t0 + kScanTok < p.T) fetch(t0 + kScanTok, (c + 1) & 1);
            __syncthreads();
        }
        // nothing is in flight any more unless a consumer gave up: its copies land before the block ends
        if (*abort_flag) { mbar_wait_drain(smem_u32(full_bar), 0); mbar_wait_drain(smem_u32(full_bar + 1), 0); }
        return;
    }
    auto vec = [&](const float *row, f2 (&x)[NP]) {
#pragma unroll
        for (int i = 0; i < N4; i++) lds_f2x2(row + 4 * (i * L + l), x[2 * i], x[2 * i + 1]);
    };
    f2 st[CB][NP];
#pragma unroll
    for (int c = 0; c < CB; c++) {
        const int gc = c0 + col + c;
        const float *sp = p.state + ((size_t)h * p.DV + gc) * DP;
#pragma unroll
        for (int i = 0; i < N4; i++) {
            ulonglong2 x = make_ulonglong2(0ull, 0ull);
            if (gc < p.DV && !p.from_zero) x = __ldcg(reinterpret_cast<const ulonglong2 *>(sp + 4 * (i * L + l)));
            st[c][2 * i] = x.x; st[c][2 * i + 1] = x.y;
        }
    }
    const f2 decay = DELTA ? 0ull : pack2(p.decay[h], p.decay[h]);
    const size_t ldo = (size_t)p.H * p.DV;
    float *o = p.o + (size_t)h * p.DV + c0 + col;
    auto dot = [&](const f2 (&x)[NP], const f2 (&s)[NP]) {
        f2 a = mul2(x[0], s[0]), b = mul2(x[1], s[1]);
#pragma unroll
        for (int i = 2; i < NP; i += 2) { a = fma2(x[i], s[i], a); b = fma2(x[i + 1], s[i + 1], b); }
        return sum2(add2(a, b));
    };
    f2 kc[NP];                    // general delta: this token's key, and k^T S of it per column
    float ks[CB];
    // one token: the state moves on, y = this lane's share of the outputs
    auto token = [&](const float *r, const float *knext, const float2 *look, float *y) {
        float v[CB];
        if constexpr (CB == 4) {
            const float4 x = *reinterpret_cast<const float4 *>(r + NV * DP + col);
            v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
        } else {
#pragma unroll
            for (int c = 0; c < CB; c++) v[c] = r[NV * DP + col + c];
        }
        f2 q[NP];
        if (DELTA) {
            const float2 lk = *look;
            f2 kn[NP], w[NP], x[NP];
            vec(knext, kn);
            vec(r + 2 * DP, w);
            float d[CB];
#pragma unroll
            for (int i = 0; i < NP; i++) x[i] = mul2(kn[i], w[i]);
#pragma unroll
            for (int c = 0; c < CB; c++) d[c] = dot(x, st[c]);
            all_sum<CB, L>(d, lane);
            vec(r + 3 * DP, x);
            vec(r, q);
#pragma unroll
            for (int c = 0; c < CB; c++) {
                const f2 vv = pack2(v[c], v[c]), kk = pack2(-ks[c], -ks[c]);
#pragma unroll
                for (int i = 0; i < NP; i++) st[c][i] = fma2(w[i], st[c][i], fma2(x[i], kk, mul2(kc[i], vv)));
                y[c] = dot(q, st[c]);
                ks[c] = d[c] - lk.x * ks[c] + lk.y * v[c];
            }
#pragma unroll
            for (int i = 0; i < NP; i++) kc[i] = kn[i];
        } else {
            f2 k[NP];
            vec(r + DP, k);
            vec(r, q);
#pragma unroll
            for (int c = 0; c < CB; c++) {
                const f2 vv = pack2(v[c], v[c]);
#pragma unroll
                for (int i = 0; i < NP; i++) st[c][i] = fma2(decay, st[c][i], mul2(k[i], vv));
                y[c] = dot(q, st[c]);
            }
        }
    };
    for (int t0 = 0, ch = 0; t0 < p.T; t0 += kScanTok, ch++) {
        const float *buf = scan_smem + (ch & 1) * BUF;
        mbar_wait(smem_u32(full_bar + (ch & 1)), (uint32_t)(ch >> 1) & 1u, abort_flag, p.err, 71);
        const int nt = min(kScanTok, p.T - t0);
        if (DELTA && t0 == 0) {
            vec(buf + DP, kc);
#pragma unroll
            for (int c = 0; c < CB; c++) ks[c] = dot(kc, st[c]);
            all_sum<CB, L>(ks, lane);
        }
        auto next_key = [&](int t) { return t + 1 < kScanTok ? buf + (t + 1) * ROW + DP : buf + kScanTok * ROW; };   // past the last token: anything, unused
        const float2 *look = reinterpret_cast<const float2 *>(buf + kScanTok * ROW + DP);
        int t = 0;
        for (; t + TB <= nt; t += TB) {
            float y[TB * CB];
#pragma unroll
            for (int i = 0; i < TB; i++) token(buf + (t + i) * ROW, next_key(t + i), look + t + i, y + i * CB);
            const float sum = scatter_sum<TB * CB>(y, l);
            const int yt = l / CB, yc = l % CB;
            if (c0 + col + yc < p.DV) o[(size_t)(t0 + t + yt) * ldo + yc] = sum;
        }
        for (; t < nt; t++) {
            float y[CB];
            token(buf + t * ROW, next_key(t), look + t, y);
            all_sum<CB, L>(y, lane);
#pragma unroll
            for (int c = 0; c < CB; c++)
                if (l == c && c0 + col + c < p.DV) o[(size_t)(t0 + t) * ldo + c] = y[c];
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < CB; c++) {
        const int gc = c0 + col + c;
        float *sp = p.state + ((size_t)h * p.DV + gc) * DP;
        if (gc < p.DV) {
#pragma unroll
            for (int i = 0; i < N4; i++) *reinterpret_cast<ulonglong2 *>(sp + 4 * (i * L + l)) = make_ulonglong2(st[c][2 * i], st[c][2 * i + 1]);
        }
    }
}

// ---- what enters the scan
// q and k of one token: rotate the leading dims (rotate-half pairs), scale k
__global__ void retention_prep_kernel(const MixRecur m, int rope0, int rope_step, float kscale)
{
    const int half = m.rot / 2;
    float *row = m.proj + (size_t)blockIdx.x * m.ldp;
    const size_t tab = (size_t)(rope0 + (int)blockIdx.x * rope_step) * half;
    for (int i = threadIdx.x; i < m.H * m.D; i += blockDim.x) {
        const int h = i / m.D, d = i - h * m.D;
        float *q = row + (size_t)h * m.D, *k = q + (size_t)m.H * m.D;
        if (d < half) {
            const float c = m.rot_cos[tab + d], s = m.rot_sin[tab + d];
            const float qu = q[d], qv = q[d + half], ku = k[d], kv = k[d + half];
            q[d] = qu * c - qv * s;
            q[d + half] = qv * c + qu * s;
            k[d] = (ku * c - kv * s) * kscale;
            k[d + half] = (kv * c + ku * s) * kscale;
        } else if (d >= m.rot) {
            k[d] *= kscale;
        }
    }
}

// one warp per (token, head): decay <- exp(-exp(-1/2) sigmoid(decay + w0)), a <- sigmoid(a) k / (k . k + eps), and the two products
// with the next token's key that the scan looks ahead with.  The bias of a is in already.
__global__ void __launch_bounds__(256) delta_prep_kernel(const MixRecur m, int T, float *__restrict__ decay, float2 *__restrict__ look, int look_ld)
{
    const int lane = threadIdx.x & 31;
    const int64_t u = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (u >= (int64_t)T * m.H) return;
    const int t = (int)(u / m.H), h = (int)(u % m.H), HD = m.H * m.D;
    float *row = m.proj + (size_t)t * m.ldp;
    const float *k = row + HD + (size_t)h * m.D;
    float *a = row + 4 * (size_t)HD + (size_t)h * m.D, *dc = decay + (size_t)t * HD + (size_t)h * m.D;
    const float *w0 = m.w0 + (size_t)h * m.D;
    float ss = 0.f;
    for (int d = lane; d < m.D; d += 32) ss += k[d] * k[d];
    ss = 1.f / (warp_sum(ss) + kUnitEps);
    const float rate = expf(-0.5f);
    const float *kn = t + 1 < T ? k + m.ldp : k;
    float kr = 0.f, kk = 0.f;
    auto one = [&](float &dv, float &av, float kv, float nv, float wv) {
        dv = expf(-rate * sigmoid_f(dv + wv));
        av = sigmoid_f(av) * kv * ss;
        kr += nv * av;
        kk += nv * kv;
    };
    if (m.D % 4 == 0) {           // rows and heads then start on 16 bytes
        for (int d = lane * 4; d < m.D; d += 128) {
            float4 dv = *reinterpret_cast<float4 *>(dc + d), av = *reinterpret_cast<float4 *>(a + d);
            const float4 kv = *reinterpret_cast<const float4 *>(k + d), nv = *reinterpret_cast<const float4 *>(kn + d), wv = *reinterpret_cast<const float4 *>(w0 + d);
            one(dv.x, av.x, kv.x, nv.x, wv.x); one(dv.y, av.y, kv.y, nv.y, wv.y); one(dv.z, av.z, kv.z, nv.z, wv.z); one(dv.w, av.w, kv.w, nv.w, wv.w);
            *reinterpret_cast<float4 *>(dc + d) = dv;
            *reinterpret_cast<float4 *>(a + d) = av;
        }
    } else {
        for (int d = lane; d < m.D; d += 32) {
            float dv = dc[d], av = a[d];
            one(dv, av, k[d], kn[d], w0[d]);
            dc[d] = dv; a[d] = av;
        }
    }
    kr = warp_sum(kr);
    kk = warp_sum(kk);
    if (lane == 0) look[(size_t)h * look_ld + t] = make_float2(kr, kk);
}

__device__ __forceinline__ float gate_value(bool delta, float y, float g, float nw) { return delta ? y * nw * sigmoid_f(g) : y * (g * sigmoid_f(g)); }

// ---- what leaves it: one warp per (token, head)
template <typename TO>
__global__ void __launch_bounds__(256) recur_post_kernel(const MixRecur m, int T, const float *__restrict__ o, int g_col, TO *__restrict__ out, int ldo)
{
    const int lane = threadIdx.x & 31;
    const int64_t u = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (u >= (int64_t)T * m.H) return;
    const int t = (int)(u / m.H), h = (int)(u % m.H);
    const float *y = o + ((size_t)t * m.H + h) * m.DV, *g = m.proj + (size_t)t * m.ldp + g_col + (size_t)h * m.DV;
    float ss = 0.f;
    if (m.DV % 4 == 0 && m.DV <= 256 && g_col % 4 == 0 && ldo % 4 == 0) {
        float4 v[2], gv[2];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int d = lane * 4 + i * 128;
            v[i] = gv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (d < m.DV) { v[i] = *reinterpret_cast<const float4 *>(y + d); gv[i] = *reinterpret_cast<const float4 *>(g + d); }
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)m.DV + m.eps);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int d = lane * 4 + i * 128;
            if (d >= m.DV) continue;
            float4 nw = make_float4(1.f, 1.f, 1.f, 1.f);
            const bool delta = m.norm_w != nullptr;
            if (delta) nw = *reinterpret_cast<const float4 *>(m.norm_w + h * m.DV + d);
            store_act4(out + (size_t)t * ldo + (size_t)h * m.DV + d, gate_value(delta, v[i].x * inv, gv[i].x, nw.x), gate_value(delta, v[i].y * inv, gv[i].y, nw.y),
                       gate_value(delta, v[i].z * inv, gv[i].z, nw.z), gate_value(delta, v[i].w * inv, gv[i].w, nw.w));
        }
        return;
    }
    for (int d = lane; d < m.DV; d += 32) ss += y[d] * y[d];
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)m.DV + m.eps);
    for (int d = lane; d < m.DV; d += 32)
        store_act(out + (size_t)t * ldo + (size_t)h * m.DV + d, gate_value(m.norm_w != nullptr, y[d] * inv, g[d], m.norm_w ? m.norm_w[h * m.DV + d] : 1.f));
}

template <typename TA>
__global__ void tanh_split_kernel(const float *__restrict__ x, int rank, int ldx, TA *__restrict__ out, int ldh)
{
    const float *row = x + (size_t)blockIdx.x * ldx;
    TA *o = out + (size_t)blockIdx.x * 2 * ldh;
    for (int i = threadIdx.x; i < ldh; i += blockDim.x) {
        const float v = i < rank ? tanhf(row[i]) : 0.f;
        if constexpr (sizeof(TA) == 2) {
            const __nv_bfloat16 hi = __float2bfloat16_rn(v);
            o[i] = hi;
            o[ldh + i] = __float2bfloat16_rn(v - __bfloat162float(hi));
        } else {
            o[i] = v;
            o[ldh + i] = 0.f;
        }
    }
}

// ================================================================ one token per sequence, everything in one launch
template <int NC, bool DELTA, typename TO>
__global__ void __launch_bounds__(kStepThreads) recur_step_kernel(const MixRecurDecode j)
{
    constexpr int DP = 32 * NC;
    __shared__ __align__(16) float s_q[DP], s_k[DP], s_w[DP], s_rem[DP];
    __shared__ float red[kStepThreads / 32];
    extern __shared__ float step_smem[];                     // [DV] output, [rank] tanh of the decay's first step
    const MixRecur &m = j.m;
    float *s_o = step_smem, *s_t = s_o + m.DV;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = tid & 7, h = blockIdx.x, b = blockIdx.y;
    float *state = m.state + (size_t)b * m.seq_stride + (size_t)h * m.DV * DP;
    // The state was left by a launch of an earlier step and the position by that step's end, both complete before the launch
    // in front of this one started: they may be read before the wait.
    const int pos = __ldcg(j.pos + b);
    Column<NC> S;
    int col = tid >> 3;
    if (pos > 0 && col < m.DV) S.load(state + (size_t)col * DP, l);
    else S.zero();
    if (DELTA) {                                             // weights: on their way while the launch in front finishes
        const char *w2 = reinterpret_cast<const char *>(m.w2.w + (size_t)h * m.D * m.w2.ld);
        for (size_t i = (size_t)tid * 128; i < (size_t)m.D * m.w2.ld * 2; i += kStepThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(w2 + i));
    }
    pdl_wait();
    pdl_launch_dependents();
    const int HD = m.H * m.D;
    const float *row = m.proj + (size_t)b * m.ldp, *rq = row + (size_t)h * m.D, *rk = rq + HD, *rv = row + 2 * HD + (size_t)h * m.DV;
    const float *rg = row + (DELTA ? 3 * HD + (size_t)h * m.D : 2 * HD + (size_t)m.H * m.DV + (size_t)h * m.DV);
    f2 decay = 0ull;
    if (DELTA) {
        const float *ra = row + 4 * (size_t)HD + (size_t)h * m.D, *rw = row + 5 * (size_t)HD;
        float ss = 0.f;
        for (int d = tid; d < DP; d += kStepThreads) {
            const float k = d < m.D ? __ldcg(rk + d) : 0.f;
            s_q[d] = d < m.D ? __ldcg(rq + d) : 0.f;
            s_k[d] = k;
            s_rem[d] = d < m.D ? sigmoid_f(__ldcg(ra + d)) * k : 0.f;
            s_w[d] = 0.f;
            ss += k * k;
        }
        for (int i = tid; i < m.rank; i += kStepThreads) s_t[i] = tanhf(__ldcg(rw + i));
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < kStepThreads / 32; i++) ss += red[i];
        const float inv = 1.f / (ss + kUnitEps), rate = expf(-0.5f);
        for (int d = tid; d < m.D; d += kStepThreads) s_rem[d] *= inv;
        constexpr int NR = 8;                                // rows in flight per warp
        for (int d0 = warp * NR; d0 < m.D; d0 += kStepThreads / 32 * NR) {
            float s[NR] = {};
            for (int i = lane; i < m.rank; i += 32) {
                const __nv_bfloat16 *wr = m.w2.w + (size_t)(h * m.D + d0) * m.w2.ld + i;
                float w[NR];
#pragma unroll
                for (int r = 0; r < NR; r++) w[r] = __bfloat162float(wr[(size_t)min(r, m.D - 1 - d0) * m.w2.ld]);
#pragma unroll
                for (int r = 0; r < NR; r++) s[r] = fmaf(w[r], s_t[i], s[r]);
            }
            float mine = scatter_sum<NR>(s, lane);           // lane r of every eight: row d0 + r over those eight lanes
            mine += __shfl_xor_sync(0xffffffffu, mine, 8);
            mine += __shfl_xor_sync(0xffffffffu, mine, 16);
            if (lane < NR && d0 + lane < m.D) s_w[d0 + lane] = expf(-rate * sigmoid_f(mine + m.w0[h * m.D + d0 + lane]));
        }
    } else {
        const int half = m.rot / 2;
        const float ks = 1.f / sqrtf((float)m.D);
        const size_t tab = (size_t)__ldcg(j.rope_pos + b) * half;
        for (int d = tid; d < DP; d += kStepThreads) {
            float q = 0.f, k = 0.f;
            if (d < m.D) {
                q = __ldcg(rq + d); k = __ldcg(rk + d);
                if (d < m.rot) {
                    const bool up = d < half;
                    const int i = up ? d : d - half;
                    const float c = m.rot_cos[tab + i], s = up ? -m.rot_sin[tab + i] : m.rot_sin[tab + i];
                    const int o = up ? d + half : d - half;
                    q = q * c + __ldcg(rq + o) * s;
                    k = k * c + __ldcg(rk + o) * s;
                }
                k *= ks;
            }
            s_q[d] = q; s_k[d] = k;
        }
        decay = pack2(m.decay[h], m.decay[h]);
    }
    __syncthreads();
    for (; col - (lane >> 3) < m.DV; col += kStepCols) {       // whole warps stay in: the reductions shuffle
        const bool live = col < m.DV;
        if (col >= kStepCols) {
            if (pos > 0 && live) S.load(state + (size_t)col * DP, l);
            else S.zero();
        }
        const float v = live ? __ldcg(rv + col) : 0.f;
        const float y = lanes8_sum(DELTA ? S.delta(s_q, s_k, s_w, s_rem, v, l) : S.retain(s_q, s_k, decay, v, l));
        if (live) {
            S.store(state + (size_t)col * DP, l);
            if (l == 0) s_o[col] = y;
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < m.DV; d += kStepThreads) ss += s_o[d] * s_o[d];
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; i++) ss += red[i];
    const float inv = 1.f / sqrtf(ss / (float)m.DV + m.eps);
    TO *out = reinterpret_cast<TO *>(j.out) + (size_t)b * j.ldo + (size_t)h * m.DV;
    for (int d = tid; d < m.DV; d += kStepThreads) store_act(out + d, gate_value(DELTA, s_o[d] * inv, __ldcg(rg + d), DELTA ? m.norm_w[h * m.DV + d] : 1.f));
}

template <int NC, bool DELTA>
tlb_status scan_nc(const ScanParams &p)
{
    constexpr int COLS = ScanShape<NC>::COLS, ROW = (DELTA ? 4 : 2) * 32 * NC + COLS;
    const size_t smem = (size_t)2 * (kScanTok * ROW + 32 * NC + 2 * kScanTok) * sizeof(float);
    static bool set = false;
    if (!set) {
        TLB_CUDA(cudaFuncSetAttribute(scan_kernel<NC, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set = true;
    }
    scan_kernel<NC, DELTA><<<dim3((p.DV + COLS - 1) / COLS, p.H), kScanThreads + 32, smem, ctx()->stream>>>(p);
    TLB_CUDA(cudaGetLastError());
    count_launch();
    return TLB_OK;
}

template <bool DELTA>
tlb_status run_scan(const ScanParams &p, int nc)
{
    switch (nc) {
    case 1: return scan_nc<1, DELTA>(p);
    case 2: return scan_nc<2, DELTA>(p);
    case 3: return scan_nc<3, DELTA>(p);
    case 4: return scan_nc<4, DELTA>(p);
    case 5: return scan_nc<5, DELTA>(p);
    case 6: return scan_nc<6, DELTA>(p);
    case 7: return scan_nc<7, DELTA>(p);
    case 8: return scan_nc<8, DELTA>(p);
    }
    return fail(TLB_ERR_SHAPE, "recurrent mixer: head size %d", p.D);
}

template <int NC, bool DELTA>
tlb_status step_nc(const MixRecurDecode &j)
{
    const size_t smem = (size_t)(j.m.DV + j.m.rank) * sizeof(float);
    if (smem > (40u << 10)) return fail(TLB_ERR_SHAPE, "recurrent mixer: %d value channels and rank %d do not fit shared memory", j.m.DV, j.m.rank);
    const dim3 grid(j.m.H, j.batch);
    if (j.out_f32) TLB_CUDA(launch_chained(recur_step_kernel<NC, DELTA, float>, grid, dim3(kStepThreads), smem, j.pdl, j));
    else TLB_CUDA(launch_chained(recur_step_kernel<NC, DELTA, __nv_bfloat16>, grid, dim3(kStepThreads), smem, j.pdl, j));
    count_launch();
    return TLB_OK;
}

template <bool DELTA>
tlb_status run_step(const MixRecurDecode &j)
{
    switch (j.m.ld / 32) {
    case 1: return step_nc<1, DELTA>(j);
    case 2: return step_nc<2, DELTA>(j);
    case 3: return step_nc<3, DELTA>(j);
    case 4: return step_nc<4, DELTA>(j);
    case 5: return step_nc<5, DELTA>(j);
    case 6: return step_nc<6, DELTA>(j);
    case 7: return step_nc<7, DELTA>(j);
    case 8: return step_nc<8, DELTA>(j);
    }
    return fail(TLB_ERR_SHAPE, "recurrent mixer: head size %d", j.m.D);
}

tlb_status post(const MixRecur &m, int T, const float *o, int g_col, void *out, int ldo, bool f32)
{
    const unsigned grid = (unsigned)(((int64_t)T * m.H + 7) / 8);
    if (f32) recur_post_kernel<<<grid, 256, 0, ctx()->stream>>>(m, T, o, g_col, (float *)out, ldo);
    else recur_post_kernel<<<grid, 256, 0, ctx()->stream>>>(m, T, o, g_col, (__nv_bfloat16 *)out, ldo);
    TLB_CUDA(cudaGetLastError());
    count_launch();
    return TLB_OK;
}

}  // namespace

int scan_look_ld(int T) { return (T + kScanTok - 1) / kScanTok * kScanTok; }
bool mix_recur_supported(int D, int DV) { return D >= 1 && D <= 256 && DV >= 1 && DV <= 4096; }
int mix_recur_ld(int D) { return (D + 31) / 32 * 32; }

tlb_status launch_retention_decode(const MixRecurDecode &j) { return run_step<false>(j); }
tlb_status launch_delta_decode(const MixRecurDecode &j) { return run_step<true>(j); }

tlb_status launch_retention_prefill(const MixRecur &m, int seq, int T, int pos0, int rope0, int rope_step, float *o, void *out, int ldo, bool f32)
{
    const int HD = m.H * m.D;
    retention_prep_kernel<<<T, 256, 0, ctx()->stream>>>(m, rope0, rope_step, 1.f / sqrtf((float)m.D));
    TLB_CUDA(cudaGetLastError());
    count_launch();
    ScanParams p = {};
    p.H = m.H; p.D = m.D; p.DV = m.DV; p.T = T;
    p.q = m.proj; p.k = m.proj + HD; p.v = m.proj + 2 * HD;
    p.ldq = p.ldk = p.ldv = m.ldp;
    p.decay = m.decay;
    p.state = m.state + (size_t)seq * m.seq_stride;
    p.from_zero = pos0 == 0;
    p.o = o;
    p.err = ctx()->err_flag;
    TLB_TRY(run_scan<false>(p, m.ld / 32));
    return post(m, T, o, 2 * HD + m.H * m.DV, out, ldo, f32);
}

tlb_status launch_delta_prefill(const MixRecur &m, int seq, int T, int pos0, float *decay, float2 *look, float *o, void *out, int ldo, bool f32)
{
    const int HD = m.H * m.D;
    delta_prep_kernel<<<(unsigned)(((int64_t)T * m.H + 7) / 8), 256, 0, ctx()->stream>>>(m, T, decay, look, scan_look_ld(T));
    TLB_CUDA(cudaGetLastError());
    count_launch();
    ScanParams p = {};
    p.H = m.H; p.D = m.D; p.DV = m.DV; p.T = T;
    p.q = m.proj; p.k = m.proj + HD; p.v = m.proj + 2 * HD; p.w = decay; p.rem = m.proj + 4 * (size_t)HD;
    p.ldq = p.ldk = p.ldv = p.ldr = m.ldp;
    p.ldw = HD;
    p.look = look; p.look_ld = scan_look_ld(T);
    p.state = m.state + (size_t)seq * m.seq_stride;
    p.from_zero = pos0 == 0;
    p.o = o;
    p.err = ctx()->err_flag;
    TLB_TRY(run_scan<true>(p, m.ld / 32));
    return post(m, T, o, 3 * HD, out, ldo, f32);
}

tlb_status launch_tanh_split(const float *x, int T, int rank, int ldx, void *out, int ldh, bool f32)
{
    if (f32) tanh_split_kernel<<<T, 128, 0, ctx()->stream>>>(x, rank, ldx, (float *)out, ldh);
    else tanh_split_kernel<<<T, 128, 0, ctx()->stream>>>(x, rank, ldx, (__nv_bfloat16 *)out, ldh);
    TLB_CUDA(cudaGetLastError());
    count_launch();
    return TLB_OK;
}

}  // namespace tlb
