// Mixture of experts over many rows: every token's choice, the rows grouped by expert, and the list of row tiles the grouped GEMM
// walks (dense_linear.cu).  One token at a time chooses inside its matvec launches instead (DPRO_EXPERT, DPRO_EXPERTS).
#include <algorithm>

#include "act.cuh"
#include "layered_kernels.h"

namespace tlb {

namespace {

__global__ void __launch_bounds__(128) route_rows_kernel(const RouteDesc r, const float *__restrict__ logits, int ldl, int *__restrict__ sel, float *__restrict__ weight,
                                                         int *__restrict__ place, int *__restrict__ count)
{
    extern __shared__ float scratch[];
    __shared__ int s_sel[kMaxTop];
    __shared__ float s_w[kMaxTop];
    const size_t t = blockIdx.x;
    route_token(logits + t * ldl, r, scratch, s_sel, s_w);
    for (int i = threadIdx.x; i < r.top; i += 128) {
        sel[t * r.top + i] = s_sel[i];
        weight[t * r.top + i] = s_w[i];
        place[t * r.top + i] = atomicAdd(count + s_sel[i], 1);      // any order: a row's result does not depend on its place
    }
}

// first row of every expert and the tiles; one CTA
__global__ void __launch_bounds__(256) moe_tiles_kernel(int experts, int *__restrict__ count, int tile_rows, int4 *__restrict__ tiles, int max_tiles)
{
    extern __shared__ int s_first[];                       // [experts + 1] counts, then first rows; [experts + 1] tiles
    int *s_tile = s_first + experts + 1;
    for (int e = threadIdx.x; e < experts; e += 256) s_first[e] = count[e];
    __syncthreads();
    if (threadIdx.x == 0) {
        int row = 0, tile = 0;
        for (int e = 0; e < experts; e++) {
            const int n = s_first[e];
            s_first[e] = row; s_tile[e] = tile;
            row += n;
            tile += (n + tile_rows - 1) / tile_rows;
        }
        s_first[experts] = row; s_tile[experts] = tile;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < experts; e += 256) {
        const int n = s_first[e + 1] - s_first[e];
        count[experts + e] = s_first[e];
        for (int i = 0; i * tile_rows < n && s_tile[e] + i < max_tiles; i++)
            tiles[s_tile[e] + i] = make_int4(e, s_first[e] + i * tile_rows, min(tile_rows, n - i * tile_rows), 0);
    }
    for (int i = s_tile[experts] + threadIdx.x; i < max_tiles; i += 256) tiles[i] = make_int4(0, 0, 0, 0);
}

// one CTA per (token, choice): the row moves to its place, which becomes an index over all experts' rows
__global__ void __launch_bounds__(128) moe_gather_kernel(int top, const int *__restrict__ sel, int *__restrict__ place, const int *__restrict__ first,
                                                         const char *__restrict__ act, size_t row_bytes, char *__restrict__ out)
{
    const int i = blockIdx.x, t = i / top;
    const int dst = first[sel[i]] + place[i];
    const uint4 *s = reinterpret_cast<const uint4 *>(act + (size_t)t * row_bytes);
    uint4 *d = reinterpret_cast<uint4 *>(out + (size_t)dst * row_bytes);
    for (size_t k = threadIdx.x; k < row_bytes / 16; k += 128) d[k] = s[k];
    __syncthreads();
    if (threadIdx.x == 0) place[i] = dst;
}

tlb_status launched(const char *what)
{
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return cuda_fail(e, what);
    count_launch();
    return TLB_OK;
}

}  // namespace

int moe_tile_rows(const RouteDesc &r, int T, bool f32)
{
    if (f32) return kF32GemmRows;
    const int mean = (int)((int64_t)T * r.top / r.experts);
    return std::min(128, std::max(32, (mean + mean / 4 + 31) / 32 * 32));
}

int moe_max_tiles(const RouteDesc &r, int T, bool f32)
{
    const int64_t rows = (int64_t)T * r.top;
    return (int)(std::min<int64_t>(r.experts, rows) + rows / moe_tile_rows(r, T, f32));
}

tlb_status launch_moe_plan(const RouteDesc &r, const float *logits, int ldl, int T, const MoePlan &p, bool f32)
{
    TLB_CUDA(cudaMemsetAsync(p.count, 0, (size_t)r.experts * sizeof(int), ctx()->stream));
    route_rows_kernel<<<T, 128, route_scratch_floats(r) * sizeof(float), ctx()->stream>>>(r, logits, ldl, p.sel, p.weight, p.place, p.count);
    TLB_TRY(launched("router launch"));
    moe_tiles_kernel<<<1, 256, (size_t)2 * (r.experts + 1) * sizeof(int), ctx()->stream>>>(r.experts, p.count, moe_tile_rows(r, T, f32), p.tiles, moe_max_tiles(r, T, f32));
    return launched("expert tiles launch");
}

tlb_status launch_moe_gather(const RouteDesc &r, const MoePlan &p, const void *act, int T, int ld, void *out, bool f32)
{
    moe_gather_kernel<<<T * r.top, 128, 0, ctx()->stream>>>(r.top, p.sel, p.place, p.count + r.experts, (const char *)act, (size_t)ld * (f32 ? 4 : 2), (char *)out);
    return launched("expert gather launch");
}

}  // namespace tlb
