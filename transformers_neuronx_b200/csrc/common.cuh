// Helpers shared by every kernel file of the engine.  Each .cu file is built into a shared
// library of its own with plain C entry points (no torch headers): the Python side loads it with
// ctypes, passes device pointers and the current CUDA stream, and checks the returned code.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define TNX_EXPORT extern "C" __attribute__((visibility("default")))

// Entry points return 0 on success, a CUDA error code (>0) if a launch failed, or a negative
// code of their own for an argument they refuse.
#define TNX_ERR_BAD_ARG (-1)
#define TNX_ERR_UNSUPPORTED (-2)
#define TNX_ERR_TIMEOUT (-3)

static inline int tnx_launch_status() {
    cudaError_t e = cudaGetLastError();
    return (int)e;
}

// The 16-bit floating type of this build.  Every library is compiled once with bfloat16 as `h16` and,
// when a model asks for it, once more with TNX_F16 defined, where `h16` is IEEE half precision
// (float16): the same kernels, other conversions, other operand formats of the tensor-core instructions.
// An entry point's `*_h16` flags say "this tensor holds h16" (0: 32-bit floats).
#ifdef TNX_F16
typedef __half h16;
typedef __half2 h16x2;
#define TNX_H16_NAME "float16"
__device__ __forceinline__ float h16_to_float(h16 v) { return __half2float(v); }
__device__ __forceinline__ h16 float_to_h16(float v) { return __float2half_rn(v); }
__device__ __forceinline__ float2 h16x2_to_float2(h16x2 v) { return __half22float2(v); }
__device__ __forceinline__ h16x2 floats_to_h16x2(float a, float b) { return __floats2half2_rn(a, b); }
#else
typedef __nv_bfloat16 h16;
typedef __nv_bfloat162 h16x2;
#define TNX_H16_NAME "bfloat16"
__device__ __forceinline__ float h16_to_float(h16 v) { return __bfloat162float(v); }
__device__ __forceinline__ h16 float_to_h16(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float2 h16x2_to_float2(h16x2 v) { return __bfloat1622float2(v); }
__device__ __forceinline__ h16x2 floats_to_h16x2(float a, float b) { return __floats2bfloat162_rn(a, b); }
#endif
// 1 when this library was built with float16 as its 16-bit type, 0 for bfloat16.
TNX_EXPORT int tnx_h16_is_float16() {
#ifdef TNX_F16
    return 1;
#else
    return 0;
#endif
}

// Programmatic dependent launch.  The matrix products and LayerNorm are launched with the attribute that
// lets a kernel start while the kernel before it in the stream is still running (tnx_launch_ex with
// early = 1); the other kernels are launched in stream order (tnx_launch_in_order).  The rules every kernel
// keeps, so that either launch is right for it: it calls pdl_launch_dependents() at its start (the next kernel
// may begin its own set-up and prefetch data that no kernel writes, i.e. weights), and it calls pdl_wait()
// before it reads anything a preceding kernel wrote and before it writes anything at all.  pdl_wait() returns
// when the preceding kernel has completed and its writes are visible; since every kernel waits before
// it finishes, completion is transitive along the stream.  (In a kernel launched in stream order the wait
// returns at once; its call of pdl_launch_dependents() still lets a following kernel with the attribute in.)
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

// early != 0: the kernel may start before the kernel ahead of it has finished (it must keep the
// rules above).  early == 0: an ordinary launch, after the kernel ahead of it.
template <typename... KArgs, typename... Args>
static inline int tnx_launch_ex(int early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = early ? 1 : 0;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
    if (e != cudaSuccess) { cudaGetLastError(); return (int)e; }
    return 0;
}
// The same with the thread blocks grouped into clusters of `cluster` (which must divide the grid).
template <typename... KArgs, typename... Args>
static inline int tnx_launch_cluster(int early, dim3 cluster, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                     cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cluster.x; attr[0].val.clusterDim.y = cluster.y; attr[0].val.clusterDim.z = cluster.z;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = early ? 2 : 1;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
    if (e != cudaSuccess) { cudaGetLastError(); return (int)e; }
    return 0;
}
template <typename... KArgs, typename... Args>
static inline int tnx_launch_in_order(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                 Args... args) {
    return tnx_launch_ex(0, kernel, grid, block, smem, stream, args...);
}

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(h16 v) { return h16_to_float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ h16 from_float<h16>(float v) { return float_to_h16(v); }

// Activations that a product's epilogue applies to (sum + bias), by code: the names of
// src/transformers_neuronx/activations.py (relu :43-48, gelu_new :17-41 with its tanh form, sigmoid
// :66-67, silu :70-72) plus the exact (erf) gelu and the square of relu.  The code travels to the kernel as a number, so
// another activation is one more case here and one more name in kernels/ops.py.
#define TNX_ACT_NONE 0
#define TNX_ACT_RELU 1
#define TNX_ACT_GELU_NEW 2
#define TNX_ACT_SILU 3
#define TNX_ACT_SIGMOID 4
#define TNX_ACT_GELU 5
#define TNX_ACT_RELU2 6
#define TNX_ACT_COUNT 7
// The cheap cases are inline; everything else is one call into a function that is compiled once.
// (With every case expanded inline, the epilogues of the tensor-core products, which apply the
// activation to several accumulators per loop turn, grew so much that a 2,048-token prefill of the
// 6.7B sizes took 32 ms instead of 26: also for the products that use no activation at all.)
__device__ __noinline__ float apply_activation_other(float v, int act) {
    switch (act) {
        case TNX_ACT_GELU_NEW: return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
        case TNX_ACT_SILU: return v / (1.f + expf(-v));
        case TNX_ACT_SIGMOID: return 1.f / (1.f + expf(-v));
        case TNX_ACT_GELU: return 0.5f * v * (1.f + erff(v * 0.7071067811865476f));
        default: return v;
    }
}
// The tanh form of gelu for epilogues that round to 16 bits anyway and meet it by the million: 0.5 (1 + tanh u) is
// 1 / (1 + e^(-2u)), a handful of instructions that stay inline.
__device__ __forceinline__ float gelu_new_fast(float v) {
    const float u2 = fmaxf(1.5957691216057308f * (v + 0.044715f * v * v * v), -80.f);
    return __fdividef(v, 1.f + __expf(-u2));
}
// Eight neighbouring channels as one 16-byte access (two for floats), and as floats.
template <typename T> struct Vec8;
template <> struct Vec8<h16> {
    uint4 raw;
    __device__ __forceinline__ void load(const h16* p) { raw = *(const uint4*)p; }
    __device__ __forceinline__ void store(h16* p) const { *(uint4*)p = raw; }
    __device__ __forceinline__ void zero() { raw = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        const h16x2* h = (const h16x2*)&raw;
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = h16x2_to_float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
    }
    __device__ __forceinline__ void set(const float (&v)[8]) {
        h16x2* h = (h16x2*)&raw;
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = floats_to_h16x2(v[2 * i], v[2 * i + 1]);
    }
};
template <> struct Vec8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = *(const float4*)p; b = *(const float4*)(p + 4); }
    __device__ __forceinline__ void store(float* p) const { *(float4*)p = a; *(float4*)(p + 4) = b; }
    __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    __device__ __forceinline__ void set(const float (&v)[8]) {
        a = make_float4(v[0], v[1], v[2], v[3]); b = make_float4(v[4], v[5], v[6], v[7]);
    }
};

__device__ __forceinline__ float apply_activation(float v, int act) {
    if (act == TNX_ACT_NONE) return v;
    if (act == TNX_ACT_RELU) return fmaxf(v, 0.f);
    if (act == TNX_ACT_RELU2) { const float r = fmaxf(v, 0.f); return r * r; }
    return apply_activation_other(v, act);
}

// Which earlier keys a query reads, as one number (the `window` argument of the attention entry points):
//   0: every key up to its own position;  w > 0: the last w of them (a sliding window);
//   c < 0: those of its own block of -c positions, blocks counted from position 0 of the sequence (a chunked mask).
// The first key a query at position `pos` reads; it never decreases as pos grows.
__host__ __device__ __forceinline__ int first_visible_key(int pos, int mask) {
    if (mask > 0) return pos - mask + 1 > 0 ? pos - mask + 1 : 0;
    if (mask < 0) return pos / (-mask) * (-mask);
    return 0;
}

// With a sliding window the first `keep` positions may stay visible to every later query (keep 0: not): a query at `pos`
// then reads key j <= pos where j >= first_visible_key(pos, mask) or j < keep.  A kernel that walks the keys in blocks of
// a fixed size takes the blocks of the first positions, then jumps to the block of the first key behind the gap.
struct BlockWalk {
    int kept, first;             // blocks 0 .. kept - 1, then first, first + 1, ...
    __host__ __device__ __forceinline__ int at(int i) const { return i < kept ? i : first + i - kept; }
    // how many blocks lie on the walk up to and with block `last` (last >= first), and the place of block b >= first on it
    __host__ __device__ __forceinline__ int count(int last) const { return kept + last - first + 1; }
    __host__ __device__ __forceinline__ int place(int b) const { return kept + b - first; }
};
__host__ __device__ __forceinline__ BlockWalk walk_blocks(int first_key, int keep, int block) {
    const int fb = first_key / block, kb = keep > 0 ? (keep + block - 1) / block : 0;
    BlockWalk w;
    if (keep > 0 && kb >= fb) { w.kept = 0; w.first = 0; }        // no block between them: all from the start
    else { w.kept = kb; w.first = fb; }
    return w;
}

// A distance bias that is taken off the scores of head h: mul[h] * ln(1 + rate[h] * (i - j)) (mul null: none).
struct DistanceBias {
    const float* mul;
    const float* rate;
};
// One more key for every query and head, of a fixed score and without a value: the softmax's denominator gains exp(score).
// A kernel starts its running (maximum, sum) at (score, 1) instead of (-inf, 0); kernels that split a row's keys do so in
// one of the parts.
struct SoftmaxSink {
    int on;
    float score;
};
__device__ __forceinline__ float log2_approx(float x) {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a thread block; `scratch` holds at least 32 floats of shared memory.  Every thread
// receives the result.  The order of the additions is fixed by the block size alone.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : 0.f;
    r = warp_sum(r);
    return r;
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : -INFINITY;
    r = warp_max(r);
    return r;
}
