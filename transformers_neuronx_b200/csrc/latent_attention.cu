// What lies around the paged attention kernels for an attention whose keys and values are expanded per head from one
// low-rank latent c per position, plus one rotated key part shared by all heads:
//     k_h = [W_uk,h c | r],  v_h = W_uv,h c,  score = scale * (q_plain,h . W_uk,h c + q_rot,h . r)
// Only c and r are kept per position, as ONE key/value head of `D` dims a position: the key row is [c | r | 0], the
// value row [c | 0].  The expansion moves to the queries' side: q'_h = [W_uk,h^T q_plain,h | q_rot,h | 0], whose product
// with the key row is the score above, and the attention's output per head, sum_j p_j c_j, goes through W_uv,h afterwards.
//
// tnx_latent_prep, one thread block per token at position p: from the output of the two down projections
//   (columns: rq of the queries' latent, rkv of the keys'/values' latent, dr of the rotated key part)
//     c_q = x / sqrt(mean(x^2) + eps) * wq  -> cq_out (the input of the queries' up projection)
//     c   = x / sqrt(mean(x^2) + eps) * wkv -> key row and value row
//     r turned by p (pairs (2i, 2i + 1) when interleaved, else (i, i + dr/2); angle p * inv_freq[i]) -> key row
// tnx_headwise_product: out[n, h, :n_out] = sum_k in[n, h, k] * W[h, k, :]  for every token n and head h, 32-bit sums
//   (W stored [heads, K, n_out]); a block takes 64 outputs of one head and up to 8 tokens, so a head's matrix is read once
//   per 8 tokens; its eight warps share the K rows (two neighbouring outputs a lane) and add their sums up in a fixed order.
//   With rot_dims > 0 it also carries the head's rotated part over: in[n, h, K .. K + rot_dims) turned by the token's
//   position to out[n, h, n_out .. n_out + rot_dims), and zeroes the head's padding up to pad_to.  do_product = 0: only
//   that (the product was done elsewhere).
#include "common.cuh"

namespace {

template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ proj, int ld, int col0, const int* __restrict__ token_request,
                   const int* __restrict__ positions, const float* __restrict__ wq, const float* __restrict__ wkv,
                   float eps, const float* __restrict__ inv_freq, int interleaved, T* __restrict__ cq_out,
                   T* __restrict__ k_out, T* __restrict__ v_out, int rq, int rkv, int dr, int D) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int n = blockIdx.x;
    if (token_request[n] < 0) return;                  // a padded row of a captured step
    const float pos = (float)positions[n];
    const T* row = proj + (size_t)n * ld + col0;
    float sq = 0.f, sc = 0.f;
    for (int i = threadIdx.x; i < rq; i += blockDim.x) { const float x = to_float(row[i]); sq = fmaf(x, x, sq); }
    for (int i = threadIdx.x; i < rkv; i += blockDim.x) { const float x = to_float(row[rq + i]); sc = fmaf(x, x, sc); }
    const float rinv_q = 1.0f / sqrtf(block_sum(sq, scratch) / (float)rq + eps);
    const float rinv_c = 1.0f / sqrtf(block_sum(sc, scratch) / (float)rkv + eps);
    for (int i = threadIdx.x; i < rq; i += blockDim.x) {
        float x = to_float(row[i]) * rinv_q;
        if (wq) x *= wq[i];
        cq_out[(size_t)n * rq + i] = from_float<T>(x);
    }
    T* kd = k_out + (size_t)n * D;
    T* vd = v_out + (size_t)n * D;
    for (int i = threadIdx.x; i < rkv; i += blockDim.x) {
        float x = to_float(row[rq + i]) * rinv_c;
        if (wkv) x *= wkv[i];
        kd[i] = vd[i] = from_float<T>(x);
    }
    const T* rr = row + rq + rkv;
    for (int i = threadIdx.x; i < dr / 2; i += blockDim.x) {
        const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + dr / 2;
        float sn, cs;
        sincosf(pos * inv_freq[i], &sn, &cs);
        const float u = to_float(rr[ia]), v = to_float(rr[ib]);
        kd[rkv + ia] = from_float<T>(u * cs - v * sn);
        kd[rkv + ib] = from_float<T>(v * cs + u * sn);
    }
    for (int i = rkv + dr + threadIdx.x; i < D; i += blockDim.x) kd[i] = from_float<T>(0.f);
    for (int i = rkv + threadIdx.x; i < D; i += blockDim.x) vd[i] = from_float<T>(0.f);
}

constexpr int HP_TOKENS = 8, HP_WARPS = 8, HP_COLS = 64, HP_AHEAD = 8;

// Two neighbouring outputs of a row of W.
__device__ __forceinline__ float2 load2(const h16* p) { return h16x2_to_float2(*(const h16x2*)p); }
__device__ __forceinline__ float2 load2(const float* p) { return *(const float2*)p; }

template <typename T>
__global__ void __launch_bounds__(HP_WARPS * 32)
headwise_product_kernel(const T* __restrict__ in, int in_ld, int in_head, const T* __restrict__ W, T* __restrict__ out,
                        int out_ld, int out_head, const int* __restrict__ token_request, const int* __restrict__ positions,
                        const float* __restrict__ inv_freq, int rot_dims, int interleaved, int pad_to, int do_product,
                        int N, int K, int n_out) {
    extern __shared__ __align__(16) float xs[];        // [K][HP_TOKENS], then (same place) the warps' sums [WARPS][TOKENS][COLS]
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, n0 = blockIdx.y * HP_TOKENS, c0 = blockIdx.z * HP_COLS;
    const int nt = min(HP_TOKENS, N - n0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (do_product) {
        for (int e = threadIdx.x; e < HP_TOKENS * K; e += blockDim.x) {
            const int t = e / K, kk = e - t * K;
            xs[kk * HP_TOKENS + t] = t < nt && token_request[n0 + t] >= 0 ? to_float(in[(size_t)(n0 + t) * in_ld + (size_t)h * in_head + kk]) : 0.f;
        }
        __syncthreads();
        const T* Wh = W + (size_t)h * K * n_out;
        const int c = c0 + 2 * lane;
        const bool pair = n_out % 2 == 0;              // then both outputs exist or neither, and a load of two is aligned
        float acc[HP_TOKENS][2];
#pragma unroll
        for (int t = 0; t < HP_TOKENS; ++t) acc[t][0] = acc[t][1] = 0.f;
        for (int k0 = warp; k0 < K; k0 += HP_WARPS * HP_AHEAD) {
            float2 w[HP_AHEAD];
#pragma unroll
            for (int u = 0; u < HP_AHEAD; ++u) {       // all loads before the first use
                const int kk = k0 + u * HP_WARPS;
                const T* src = Wh + (size_t)kk * n_out + c;
                w[u] = make_float2(0.f, 0.f);
                if (kk < K && c < n_out) {
                    if (pair) w[u] = load2(src);
                    else { w[u].x = to_float(src[0]); if (c + 1 < n_out) w[u].y = to_float(src[1]); }
                }
            }
#pragma unroll
            for (int u = 0; u < HP_AHEAD; ++u) {
                const int kk = k0 + u * HP_WARPS;
                if (kk < K) {
                    const float4 a = *(const float4*)(xs + kk * HP_TOKENS), b = *(const float4*)(xs + kk * HP_TOKENS + 4);
                    const float xv[HP_TOKENS] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
                    for (int t = 0; t < HP_TOKENS; ++t) { acc[t][0] = fmaf(xv[t], w[u].x, acc[t][0]); acc[t][1] = fmaf(xv[t], w[u].y, acc[t][1]); }
                }
            }
        }
        __syncthreads();                               // the inputs are done with: their place takes the sums
#pragma unroll
        for (int t = 0; t < HP_TOKENS; ++t)
            *(float2*)(xs + (warp * HP_TOKENS + t) * HP_COLS + 2 * lane) = make_float2(acc[t][0], acc[t][1]);
        __syncthreads();
        for (int e = threadIdx.x; e < nt * HP_COLS; e += blockDim.x) {
            const int t = e / HP_COLS, cc = e % HP_COLS;
            if (c0 + cc >= n_out || token_request[n0 + t] < 0) continue;
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < HP_WARPS; ++w) s += xs[(w * HP_TOKENS + t) * HP_COLS + cc];
            out[(size_t)(n0 + t) * out_ld + (size_t)h * out_head + c0 + cc] = from_float<T>(s);
        }
    }
    if (blockIdx.z != 0) return;
    if (pad_to <= n_out) return;
    const int half = rot_dims / 2, pad = pad_to - n_out - rot_dims;
    for (int e = threadIdx.x; e < nt * (half + pad); e += blockDim.x) {
        const int t = e / (half + pad), i = e % (half + pad), n = n0 + t;
        if (token_request[n] < 0) continue;
        T* dst = out + (size_t)n * out_ld + (size_t)h * out_head + n_out;
        if (i < half) {
            const T* src = in + (size_t)n * in_ld + (size_t)h * in_head + K;
            const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
            float sn, cs;
            sincosf((float)positions[n] * inv_freq[i], &sn, &cs);
            const float u = to_float(src[ia]), v = to_float(src[ib]);
            dst[ia] = from_float<T>(u * cs - v * sn);
            dst[ib] = from_float<T>(v * cs + u * sn);
        } else {
            dst[rot_dims + i - half] = from_float<T>(0.f);
        }
    }
}

}  // namespace

TNX_EXPORT int tnx_latent_prep(const void* proj, int ld, int col0, const int* token_request, const int* positions,
                               const float* wq, const float* wkv, float eps, const float* inv_freq, int interleaved,
                               void* cq_out, void* k_out, void* v_out, int n_tokens, int rq, int rkv, int dr, int D,
                               int is_h16, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rq <= 0 || rkv <= 0 || dr < 0 || dr % 2 || D < rkv + dr || (dr && !inv_freq)) return TNX_ERR_BAD_ARG;
    if (is_h16)
        return tnx_launch_in_order(latent_prep_kernel<h16>, dim3(n_tokens), dim3(128), 0, stream, (const h16*)proj, ld, col0,
                                   token_request, positions, wq, wkv, eps, inv_freq, interleaved, (h16*)cq_out,
                                   (h16*)k_out, (h16*)v_out, rq, rkv, dr, D);
    return tnx_launch_in_order(latent_prep_kernel<float>, dim3(n_tokens), dim3(128), 0, stream, (const float*)proj, ld, col0,
                               token_request, positions, wq, wkv, eps, inv_freq, interleaved, (float*)cq_out,
                               (float*)k_out, (float*)v_out, rq, rkv, dr, D);
}

TNX_EXPORT int tnx_headwise_product(const void* in, int in_ld, int in_head, const void* W, void* out, int out_ld,
                                    int out_head, const int* token_request, const int* positions, const float* inv_freq,
                                    int rot_dims, int interleaved, int pad_to, int do_product, int n_tokens, int n_heads,
                                    int K, int n_out, int is_h16, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n_heads <= 0 || K <= 0 || n_out <= 0 || rot_dims < 0 || rot_dims % 2 || (rot_dims && (!inv_freq || !positions)) ||
        (pad_to > n_out && pad_to < n_out + rot_dims) || (pad_to <= n_out && rot_dims) || (do_product && !W))
        return TNX_ERR_BAD_ARG;
    const size_t smem = do_product ? (size_t)HP_TOKENS * (K > HP_WARPS * HP_COLS ? K : HP_WARPS * HP_COLS) * sizeof(float) : 0;
    if (smem > 200 * 1024) return TNX_ERR_UNSUPPORTED;
    const dim3 grid(n_heads, (n_tokens + HP_TOKENS - 1) / HP_TOKENS, do_product ? (n_out + HP_COLS - 1) / HP_COLS : 1);
#define HPROD(T)                                                                                                         \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            cudaFuncSetAttribute(headwise_product_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        return tnx_launch_in_order(headwise_product_kernel<T>, grid, dim3(HP_WARPS * 32), smem, stream, (const T*)in, in_ld, in_head, \
                                   (const T*)W, (T*)out, out_ld, out_head, token_request, positions, inv_freq, rot_dims, \
                                   interleaved, pad_to, do_product, n_tokens, K, n_out);                                 \
    } while (0)
    if (is_h16) HPROD(h16);
    HPROD(float);
#undef HPROD
}
