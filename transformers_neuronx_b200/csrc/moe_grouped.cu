// Routed experts on the tensor cores: the (token, chosen expert) pairs are sorted by expert into a layout in which every
// expert's rows begin at a multiple of the tile (128 rows where experts get many rows; 16, 32 or 64 where they get few),
// so that each tile belongs to one expert and the two products of an expert run as grouped tensor-core products
// (gemm_tc.cu: tnx_gemm_tc_grouped, tnx_gemm_tc_grouped_few).  The kernels of this file are what lies around those products:
//
//   moe_plan_kernel      one block: counts per expert, every expert's first row, the expert of every tile (-1 beyond
//                        the last used tile), and the row of every pair.  Which row of its expert's segment a pair
//                        gets depends on the order in which threads arrive; a row's result does not depend on where it sits
//   moe_gather_kernel    x[row(pair)] = weight * h[token]  (or h[token] when the weight multiplies the output), 16-bit
//   moe_act_kernel       y = g * sigmoid(alpha g) * (u + up_shift), g and u clamped, from the gate/up product's output
//                        (moe_act_relu2_kernel: y = relu(u)^2 for experts without a gate)
//   moe_combine_kernel   out[token] (+)= sum over the token's pairs, in the order of the choice, of the down product's rows
//                        (a pair whose expert is the token itself takes no row: weight * h[token])
//
// Nothing is read on the host: the sizes of the buffers follow from the numbers of tokens and experts alone (at most
// pairs / tile + experts tiles), so a step can be captured in a CUDA graph.
#include "common.cuh"

namespace {
constexpr int MAX_EXPERTS = 1024;
constexpr int IDENTITY = -2;      // of a pair's expert, and then of its row: the token itself (-1: a padded row)

__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int* __restrict__ ids, int n_pairs, int n_experts, int max_tiles, int TILE, int* __restrict__ group_of_tile,
                int* __restrict__ row_of_pair) {
    __shared__ int count[MAX_EXPERTS], first[MAX_EXPERTS], cursor[MAX_EXPERTS], used_tiles;
    pdl_launch_dependents();
    pdl_wait();
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) { count[e] = 0; cursor[e] = 0; }
    __syncthreads();
    const int lane = threadIdx.x & 31;
    // the lanes of a warp that hold pairs of the same expert count them together
    for (int i0 = 0; i0 < n_pairs; i0 += blockDim.x) {
        const int i = i0 + threadIdx.x, e = i < n_pairs ? ids[i] : -1;
        const unsigned same = __match_any_sync(0xffffffffu, e);
        if (e >= 0 && lane == __ffs(same) - 1) atomicAdd(&count[e], __popc(same));
    }
    __syncthreads();
    if (threadIdx.x < 32) {                            // every expert's first tile: a running sum, 32 experts at a time
        int before = 0;
        for (int e0 = 0; e0 < n_experts; e0 += 32) {
            const int e = e0 + lane, t = e < n_experts ? (count[e] + TILE - 1) / TILE : 0;
            int upto = t;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, upto, o); if (lane >= o) upto += v; }
            if (e < n_experts) first[e] = (before + upto - t) * TILE;
            before += __shfl_sync(0xffffffffu, upto, 31);
        }
        if (lane == 0) used_tiles = before;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n_experts; e += blockDim.x) {
        const int tile = first[e] / TILE, t = (count[e] + TILE - 1) / TILE;
        for (int j = 0; j < t && tile + j < max_tiles; ++j) group_of_tile[tile + j] = e;
    }
    for (int tile = used_tiles + threadIdx.x; tile < max_tiles; tile += blockDim.x) group_of_tile[tile] = -1;
    for (int i0 = 0; i0 < n_pairs; i0 += blockDim.x) {
        const int i = i0 + threadIdx.x, e = i < n_pairs ? ids[i] : -1;
        const unsigned same = __match_any_sync(0xffffffffu, e);
        const int leader = __ffs(same) - 1;
        int base = 0;
        if (e >= 0 && lane == leader) base = first[e] + atomicAdd(&cursor[e], __popc(same));
        base = __shfl_sync(0xffffffffu, base, leader);
        if (i < n_pairs) row_of_pair[i] = e >= 0 ? base + __popc(same & ((1u << lane) - 1u)) : e;
    }
}

__global__ void __launch_bounds__(128)
moe_gather_kernel(const h16* __restrict__ h, int ld, const float* __restrict__ weights, const int* __restrict__ row_of_pair,
                  h16* __restrict__ x, int W, int top, int weight_on_input) {
    pdl_launch_dependents();
    pdl_wait();
    const int pair = blockIdx.x, row = row_of_pair[pair];
    if (row < 0) return;
    const float wt = weight_on_input ? weights[pair] : 1.f;
    const h16* src = h + (size_t)(pair / top) * ld;
    h16* dst = x + (size_t)row * W;
    if (W % 8 == 0 && ld % 8 == 0 && !(((uintptr_t)h | (uintptr_t)x) & 15)) {
        for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
            uint4 raw = *(const uint4*)(src + c);
            h16x2* v = (h16x2*)&raw;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = h16x2_to_float2(v[i]);
                v[i] = floats_to_h16x2(f.x * wt, f.y * wt);
            }
            *(uint4*)(dst + c) = raw;
        }
    } else {
        for (int c = threadIdx.x; c < W; c += blockDim.x) dst[c] = float_to_h16(h16_to_float(src[c]) * wt);
    }
}

__global__ void __launch_bounds__(256)
moe_act_kernel(const h16* __restrict__ gu, h16* __restrict__ y, const int* __restrict__ group_of_tile, int TILE, int F,
               float gate_max, float up_min, float up_max, float alpha, float up_shift) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x;
    if (group_of_tile[row / TILE] < 0) return;
    const h16* g = gu + (size_t)row * 2 * F;
    const h16* u = g + F;
    if (F % 8 == 0 && !(((uintptr_t)gu | (uintptr_t)y) & 15)) {
        for (int c = threadIdx.x * 8; c < F; c += blockDim.x * 8) {
            Vec8<h16> gv, uv;
            float gf[8], uf[8];
            gv.load(g + c); uv.load(u + c);
            gv.get(gf); uv.get(uf);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float g0 = fminf(gf[i], gate_max), u0 = fminf(fmaxf(uf[i], up_min), up_max);
                gf[i] = __fdividef(g0, 1.f + __expf(-alpha * g0)) * (u0 + up_shift);      // rounded to 16 bits below
            }
            gv.set(gf);
            gv.store(y + (size_t)row * F + c);
        }
        return;
    }
    for (int c = threadIdx.x * 2; c < F; c += blockDim.x * 2) {
        if (c + 1 < F && F % 2 == 0) {
            const float2 gf = h16x2_to_float2(*(const h16x2*)(g + c)), uf = h16x2_to_float2(*(const h16x2*)(u + c));
            const float g0 = fminf(gf.x, gate_max), g1 = fminf(gf.y, gate_max);
            const float u0 = fminf(fmaxf(uf.x, up_min), up_max), u1 = fminf(fmaxf(uf.y, up_min), up_max);
            *(h16x2*)(y + (size_t)row * F + c) = floats_to_h16x2(g0 / (1.f + expf(-alpha * g0)) * (u0 + up_shift),
                                                                 g1 / (1.f + expf(-alpha * g1)) * (u1 + up_shift));
        } else {
            for (int i = c; i < min(c + 2, F); ++i) {
                const float g0 = fminf(h16_to_float(g[i]), gate_max);
                const float u0 = fminf(fmaxf(h16_to_float(u[i]), up_min), up_max);
                y[(size_t)row * F + i] = float_to_h16(g0 / (1.f + expf(-alpha * g0)) * (u0 + up_shift));
            }
        }
    }
}

// Experts without a gate: y = relu(u)^2 from the up product's output [rows, F].
__global__ void __launch_bounds__(256)
moe_act_relu2_kernel(const h16* __restrict__ u, h16* __restrict__ y, const int* __restrict__ group_of_tile, int TILE, int F) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x;
    if (group_of_tile[row / TILE] < 0) return;
    const h16* src = u + (size_t)row * F;
    h16* dst = y + (size_t)row * F;
    if (F % 2 == 0) {
        for (int c = threadIdx.x * 2; c < F; c += blockDim.x * 2) {
            const float2 f = h16x2_to_float2(*(const h16x2*)(src + c));
            const float a = fmaxf(f.x, 0.f), b = fmaxf(f.y, 0.f);
            *(h16x2*)(dst + c) = floats_to_h16x2(a * a, b * b);
        }
    } else {
        for (int c = threadIdx.x; c < F; c += blockDim.x) {
            const float a = fmaxf(h16_to_float(src[c]), 0.f);
            dst[c] = float_to_h16(a * a);
        }
    }
}

__global__ void __launch_bounds__(256)
moe_combine_kernel(const float* __restrict__ rows, const h16* __restrict__ h, int ld, const int* __restrict__ row_of_pair,
                   const float* __restrict__ weights, float* out, int W, int top, int accumulate, int weight_on_input) {
    pdl_launch_dependents();
    pdl_wait();
    const int n = blockIdx.x;
    if (row_of_pair[(size_t)n * top] == -1) return;               // a padded row of a captured step
    if (W % 4 == 0 && ld % 4 == 0 && !(((uintptr_t)rows | (uintptr_t)out) & 15) && !((uintptr_t)h & 7)) {
        // four columns a thread, the rows of four choices asked for together
        for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < W; c += gridDim.y * blockDim.x * 4) {
            const float4 before = accumulate ? *(const float4*)(out + (size_t)n * W + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int j0 = 0; j0 < top; j0 += 4) {
                float4 v[4];
                float wt[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
                    wt[u] = 0.f;
                    if (j0 + u >= top) continue;
                    const int row = row_of_pair[(size_t)n * top + j0 + u];
                    const bool self = row == IDENTITY;
                    wt[u] = weight_on_input && !self ? 1.f : weights[(size_t)n * top + j0 + u];
                    if (self) {
                        const h16x2* src = (const h16x2*)(h + (size_t)n * ld + c);
                        const float2 a = h16x2_to_float2(src[0]), b = h16x2_to_float2(src[1]);
                        v[u] = make_float4(a.x, a.y, b.x, b.y);
                    } else {
                        v[u] = *(const float4*)(rows + (size_t)row * W + c);
                    }
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    s.x = fmaf(v[u].x, wt[u], s.x); s.y = fmaf(v[u].y, wt[u], s.y);
                    s.z = fmaf(v[u].z, wt[u], s.z); s.w = fmaf(v[u].w, wt[u], s.w);
                }
            }
            *(float4*)(out + (size_t)n * W + c) = make_float4(before.x + s.x, before.y + s.y, before.z + s.z, before.w + s.w);
        }
        return;
    }
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < W; c += gridDim.y * blockDim.x) {
        float s = 0.f;
        for (int j = 0; j < top; ++j) {
            const int row = row_of_pair[(size_t)n * top + j];
            const bool self = row == IDENTITY;
            const float v = self ? h16_to_float(h[(size_t)n * ld + c]) : rows[(size_t)row * W + c];
            s += weight_on_input && !self ? v : v * weights[(size_t)n * top + j];
        }
        float* dst = out + (size_t)n * W + c;
        *dst = accumulate ? *dst + s : s;
    }
}
}  // namespace

// The most tiles that n_pairs pairs spread over n_experts experts can take.
TNX_EXPORT int tnx_moe_grouped_max_tiles(int n_pairs, int n_experts, int tile) {
    return n_pairs / tile + (n_pairs < n_experts ? n_pairs : n_experts);
}

TNX_EXPORT int tnx_moe_plan(const int* ids, int n_pairs, int n_experts, int max_tiles, int tile, int* group_of_tile,
                            int* row_of_pair, cudaStream_t stream) {
    if (n_pairs <= 0) return 0;
    if (n_experts <= 0 || n_experts > MAX_EXPERTS || tile <= 0 || max_tiles < tnx_moe_grouped_max_tiles(n_pairs, n_experts, tile))
        return TNX_ERR_BAD_ARG;
    return tnx_launch_in_order(moe_plan_kernel, dim3(1), dim3(1024), 0, stream, ids, n_pairs, n_experts, max_tiles, tile,
                               group_of_tile, row_of_pair);
}

TNX_EXPORT int tnx_moe_gather(const void* h, int ld, const float* weights, const int* row_of_pair, void* x, int n_pairs, int W,
                              int top, int weight_on_input, cudaStream_t stream) {
    if (n_pairs <= 0) return 0;
    return tnx_launch_in_order(moe_gather_kernel, dim3(n_pairs), dim3(128), 0, stream, (const h16*)h, ld, weights, row_of_pair,
                               (h16*)x, W, top, weight_on_input);
}

TNX_EXPORT int tnx_moe_act(const void* gu, void* y, const int* group_of_tile, int tile, int rows, int F, float gate_max,
                           float up_min, float up_max, float alpha, float up_shift, int form, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (form == 1)
        return tnx_launch_in_order(moe_act_relu2_kernel, dim3(rows), dim3(F >= 512 ? 256 : 128), 0, stream, (const h16*)gu,
                                   (h16*)y, group_of_tile, tile, F);
    return tnx_launch_in_order(moe_act_kernel, dim3(rows), dim3(F >= 512 ? 256 : 128), 0, stream, (const h16*)gu, (h16*)y,
                               group_of_tile, tile, F, gate_max, up_min, up_max, alpha, up_shift);
}

TNX_EXPORT int tnx_moe_combine(const float* rows, const void* h, int ld, const int* row_of_pair, const float* weights, float* out, int N, int W, int top,
                               int accumulate, int weight_on_input, cudaStream_t stream) {
    if (N <= 0) return 0;
    // few tokens: a slice of the width a block, so that the loads of a row are asked for together
    return tnx_launch_in_order(moe_combine_kernel, dim3(N, N >= 256 ? 1 : (W + 511) / 512), dim3(N >= 256 && W >= 1024 ? 256 : 128), 0, stream, rows, (const h16*)h, ld, row_of_pair, weights, out, W, top,
                               accumulate, weight_on_input);
}
