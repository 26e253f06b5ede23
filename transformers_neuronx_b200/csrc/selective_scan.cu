// A selective state-space recurrence with a decay per channel and state ("selective scan").  Per channel c and state n:
//     dt_c = softplus(dt_raw_c + dt_bias_c)
//     S[c, n] <- 2^(decay_log2[c, n] dt_c) S[c, n] + dt_c x_c B_n          (S: 32-bit, kept per request between steps)
//     out_c = (sum_n S[c, n] C_n + skip_c x_c) * act(z_c)
// with decay_log2 = -exp(A_log) log2(e); B and C of a token are shared by all channels.
//
// tnx_causal_conv: one short causal convolution per channel over a request's tokens, with bias and activation,
//     y_t[c] = act(bias[c] + sum_j w[j, c] u_(t - taps + 1 + j)[c])       (zeros before position 0; the past comes from
//                                             this step's rows or from the request's state [slots, taps - 1, channels])
//   in the projection's type.  A request with one row shifts its state here; requests with several rows are brought up
//   to date by the convolution library's state kernel afterwards.
// tnx_selective_scan: a thread block owns CH channels of one request and walks the request's tokens of this step in
//   order.  A channel's states are spread over L adjacent lanes, SPT neighbouring states a lane, in registers; the decay,
//   the write and the read of a token are SPT independent chains a lane, and only one multiply-add per state links a
//   token to the next.  A stage of ST tokens lies in shared memory as what the walk needs (dt after its softplus, dt x, x, B, C
//   in 32-bit), the next stage's numbers travel in registers meanwhile.  The lanes' partial sums of y go through shared memory
//   and are added up, gated and stored once a stage, so that the walk itself meets no rendezvous.
//   A step of single tokens runs the same kernel with stages of one token: the state is streamed through once.
#include "common.cuh"

namespace {
constexpr int MAX_TAPS = 8;
constexpr int THREADS = 128;

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <typename T>
struct ConvArgs {
    const T* proj; int ld, col0;
    const float* w; const float* b; int taps;     // [taps, C], [C] or null
    T* state;                                     // [slots, taps - 1, C]
    const int* token_request; const int* positions; const int* q_start; const int* q_len; const int* state_slots;
    int act;
    T* out; int C;
};

template <typename T>
__global__ void __launch_bounds__(256) causal_conv_kernel(const ConvArgs<T> p) {
    pdl_launch_dependents();
    pdl_wait();
    const int n = blockIdx.x;
    const int req = p.token_request[n];
    if (req < 0) return;                              // a padded row of a captured step
    const int pos = p.positions[n], idx = n - p.q_start[req], slot = p.state_slots[req];
    const bool alone = p.q_len[req] == 1;
    const int keep = p.taps - 1, C = p.C;
    const T* row = p.proj + (size_t)n * p.ld + p.col0;
    T* st = (keep > 0 && slot >= 0) ? p.state + (size_t)slot * keep * C : nullptr;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        float s = p.b ? p.b[c] : 0.f;
        for (int b = keep; b >= 0; --b) {             // oldest first
            float v = 0.f;
            if (pos - b >= 0) {
                if (idx - b >= 0) v = to_float(row[c - (ptrdiff_t)b * p.ld]);
                else if (st) v = to_float(st[(size_t)(keep + idx - b) * C + c]);
            }
            s = fmaf(p.w[(size_t)(keep - b) * C + c], v, s);
            // a request's single row moves its past on: what is b back now is b + 1 back for the next token (the place
            // written here was read one round ago)
            if (alone && st && b < keep) st[(size_t)(keep - 1 - b) * C + c] = from_float<T>(v);
        }
        p.out[(size_t)n * C + c] = from_float<T>(apply_activation(s, p.act));
    }
}

// The same with eight channels a thread (16-byte accesses; sizes and addresses in multiples of eight channels).
template <typename T>
__global__ void __launch_bounds__(256) causal_conv_vec_kernel(const ConvArgs<T> p) {
    pdl_launch_dependents();
    pdl_wait();
    const int n = blockIdx.x;
    const int req = p.token_request[n];
    if (req < 0) return;
    const int pos = p.positions[n], idx = n - p.q_start[req], slot = p.state_slots[req];
    const bool alone = p.q_len[req] == 1;
    const int keep = p.taps - 1, C = p.C;
    const T* row = p.proj + (size_t)n * p.ld + p.col0;
    T* st = (keep > 0 && slot >= 0) ? p.state + (size_t)slot * keep * C : nullptr;
    for (int c = 8 * (blockIdx.y * blockDim.x + threadIdx.x); c < C; c += 8 * gridDim.y * blockDim.x) {
        float s[8];
        if (p.b) { Vec8<float> b; b.load(p.b + c); b.get(s); }
        else {
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i] = 0.f;
        }
        for (int b = keep; b >= 0; --b) {
            const T* src = row + c;                   // the value b positions back: this step's rows, the state, or zero
            if (b > 0) {
                if (pos - b < 0) src = nullptr;
                else if (idx - b >= 0) src = row + c - (ptrdiff_t)b * p.ld;
                else src = st ? st + (size_t)(keep + idx - b) * C + c : nullptr;
            }
            Vec8<T> x;
            if (src) x.load(src); else x.zero();
            Vec8<float> w;
            w.load(p.w + (size_t)(keep - b) * C + c);
            float xv[8], wv[8];
            x.get(xv);
            w.get(wv);
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i] = fmaf(wv[i], xv[i], s[i]);
            if (alone && st && b < keep) x.store(st + (size_t)(keep - 1 - b) * C + c);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i] = apply_activation(s[i], p.act);
        Vec8<T> y;
        y.set(s);
        y.store(p.out + (size_t)n * C + c);
    }
}

template <typename T>
struct ScanArgs {
    const T* x; int x_ld;
    const float* dt;                               // [N, C]
    const T* low; int low_ld, b_off, c_off;
    const float* decay_log2;                       // [C, Ns]
    const float* dt_bias; const float* skip;       // [C], skip or null
    const T* z; int z_ld;
    float* state;                                  // [slots, C, Ns]
    const int* q_start; const int* q_len; const int* state_slots;
    int act;
    T* out; int out_ld;
    int C, Ns;
};

// L lanes a channel, SPT states a lane (L * SPT >= Ns), ST tokens a stage.
template <typename T, int L, int SPT, int ST>
__global__ void __launch_bounds__(THREADS) selective_scan_kernel(const ScanArgs<T> p) {
    constexpr int CH = THREADS / L;                // channels of the block
    constexpr int NP = L * SPT;                    // padded states
    constexpr int XN = (ST * CH + THREADS - 1) / THREADS, BN = (ST * NP + THREADS - 1) / THREADS;
    __shared__ __align__(16) float dts[2][ST][CH], dtx[2][ST][CH], xs[2][ST][CH];
    __shared__ __align__(16) float bs[2][ST][NP], cs[2][ST][NP];
    __shared__ float part[ST][THREADS + 1];
    pdl_launch_dependents();
    pdl_wait();
    const int req = blockIdx.y;
    const int len = p.q_len[req];
    if (len <= 0) return;                          // a padded request of a captured step
    const int slot = p.state_slots[req];
    if (slot < 0) return;
    const int first = p.q_start[req];
    const int c0 = blockIdx.x * CH;
    const int ch = threadIdx.x / L, l = threadIdx.x % L;
    const int c = c0 + ch, n0 = l * SPT;
    const bool mine = c < p.C;
    const int C = p.C, Ns = p.Ns;

    // a stage's numbers on their way: asked for before the stage in front of it is walked
    float r_dt[XN], r_x[XN], r_b[BN], r_c[BN];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < XN; ++i) {
            const int e = threadIdx.x + i * THREADS, t = e / CH, cc = c0 + e % CH;
            r_dt[i] = 0.f; r_x[i] = 0.f;
            if (e < ST * CH && t0 + t < len && cc < C) {
                const size_t row = (size_t)(first + t0 + t);
                r_dt[i] = p.dt[row * C + cc] + p.dt_bias[cc];
                r_x[i] = to_float(p.x[row * p.x_ld + cc]);
            }
        }
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int e = threadIdx.x + i * THREADS, t = e / NP, n = e % NP;
            r_b[i] = 0.f; r_c[i] = 0.f;
            if (e < ST * NP && t0 + t < len && n < Ns) {
                const T* row = p.low + (size_t)(first + t0 + t) * p.low_ld;
                r_b[i] = to_float(row[p.b_off + n]);
                r_c[i] = to_float(row[p.c_off + n]);
            }
        }
    };
    auto stage = [&](int s) {
#pragma unroll
        for (int i = 0; i < XN; ++i) {
            const int e = threadIdx.x + i * THREADS;
            if (e < ST * CH) {
                const float dt = softplus_f(r_dt[i]);
                (&dts[s][0][0])[e] = dt;
                (&dtx[s][0][0])[e] = dt * r_x[i];
                (&xs[s][0][0])[e] = r_x[i];
            }
        }
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int e = threadIdx.x + i * THREADS;
            if (e < ST * NP) { (&bs[s][0][0])[e] = r_b[i]; (&cs[s][0][0])[e] = r_c[i]; }
        }
    };

    float S[SPT], a2[SPT];
    float* st = p.state + ((size_t)slot * C + (mine ? c : 0)) * Ns;
    const float* ar = p.decay_log2 + (size_t)(mine ? c : 0) * Ns;
    const bool vec = SPT % 4 == 0 && Ns % 4 == 0;
    fetch(0);
    if (vec) {
#pragma unroll
        for (int m = 0; m < SPT / 4; ++m) {
            const bool in = mine && n0 + 4 * m < Ns;
            const float4 s4 = in ? *(const float4*)(st + n0 + 4 * m) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 a4 = in ? *(const float4*)(ar + n0 + 4 * m) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[4 * m] = s4.x; S[4 * m + 1] = s4.y; S[4 * m + 2] = s4.z; S[4 * m + 3] = s4.w;
            a2[4 * m] = a4.x; a2[4 * m + 1] = a4.y; a2[4 * m + 2] = a4.z; a2[4 * m + 3] = a4.w;
        }
    } else {
#pragma unroll
        for (int m = 0; m < SPT; ++m) {
            const bool in = mine && n0 + m < Ns;
            S[m] = in ? st[n0 + m] : 0.f;
            a2[m] = in ? ar[n0 + m] : 0.f;
        }
    }
    stage(0);
    __syncthreads();
    int s = 0;
    for (int t0 = 0; t0 < len; t0 += ST, s ^= 1) {
        const int nt = min(ST, len - t0);
        const bool more = t0 + ST < len;
        if (more) fetch(t0 + ST);
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const float dt = dts[s][t][ch], wx = dtx[s][t][ch];
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int m = 0; m < SPT; ++m) {
                S[m] = fmaf(exp2f(a2[m] * dt), S[m], wx * bs[s][t][n0 + m]);
                if (m & 1) y1 = fmaf(S[m], cs[s][t][n0 + m], y1); else y0 = fmaf(S[m], cs[s][t][n0 + m], y0);
            }
            part[t][threadIdx.x] = y0 + y1;
        }
        if (more) stage(s ^ 1);                    // nobody reads the other stage: its walk ended before the last rendezvous
        __syncthreads();
#pragma unroll
        for (int i = 0; i < XN; ++i) {
            const int e = threadIdx.x + i * THREADS, t = e / CH, k = e % CH, cc = c0 + k;
            if (e < ST * CH && t < nt && cc < C) {
                float y = 0.f;
#pragma unroll
                for (int j = 0; j < L; ++j) y += part[t][k * L + j];
                if (p.skip) y = fmaf(p.skip[cc], xs[s][t][k], y);
                const size_t row = (size_t)(first + t0 + t);
                y *= apply_activation(to_float(p.z[row * p.z_ld + cc]), p.act);
                p.out[row * p.out_ld + cc] = from_float<T>(y);
            }
        }
        __syncthreads();                           // the partial sums and this stage have been read
    }
    if (!mine) return;
    if (vec) {
#pragma unroll
        for (int m = 0; m < SPT / 4; ++m)
            if (n0 + 4 * m < Ns) *(float4*)(st + n0 + 4 * m) = make_float4(S[4 * m], S[4 * m + 1], S[4 * m + 2], S[4 * m + 3]);
    } else {
#pragma unroll
        for (int m = 0; m < SPT; ++m)
            if (n0 + m < Ns) st[n0 + m] = S[m];
    }
}

template <typename T, int L, int SPT>
int launch_scan(const ScanArgs<T>& p, int n_requests, int most_tokens, cudaStream_t stream) {
    constexpr int CH = THREADS / L;
    constexpr int ST = L >= 2 && L <= 8 ? 16 : 8;  // shared memory stays below 48 KB
    const dim3 grid((p.C + CH - 1) / CH, n_requests);
    if (most_tokens == 1) return tnx_launch_in_order(selective_scan_kernel<T, L, SPT, 1>, grid, dim3(THREADS), 0, stream, p);
    return tnx_launch_in_order(selective_scan_kernel<T, L, SPT, ST>, grid, dim3(THREADS), 0, stream, p);
}

template <typename T>
int scan_by_state(const ScanArgs<T>& p, int n_requests, int most_tokens, cudaStream_t stream) {
    if (p.Ns <= 4) return launch_scan<T, 1, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 8) return launch_scan<T, 2, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 16) return launch_scan<T, 4, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 32) return launch_scan<T, 8, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 64) return launch_scan<T, 16, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 128) return launch_scan<T, 32, 4>(p, n_requests, most_tokens, stream);
    if (p.Ns <= 256) return launch_scan<T, 32, 8>(p, n_requests, most_tokens, stream);
    return TNX_ERR_UNSUPPORTED;
}

template <typename T>
int conv_launch(const ConvArgs<T>& p, int N, cudaStream_t stream) {
    const bool vec = p.C % 8 == 0 && p.ld % 8 == 0 && p.col0 % 8 == 0 &&
                     !(((uintptr_t)p.proj | (uintptr_t)p.w | (uintptr_t)p.b | (uintptr_t)p.state | (uintptr_t)p.out) & 15);
    // a prompt's tokens: one block a token; the few tokens of a decode step: a token's channels over several blocks
    const int units = vec ? p.C / 8 : p.C;
    const int threads = units >= 256 ? 256 : (units >= 128 ? 128 : 64);
    int ny = 1;
    if (N < 256) { ny = (units + threads - 1) / threads; if (ny > 16) ny = 16; }
    if (vec) return tnx_launch_in_order(causal_conv_vec_kernel<T>, dim3(N, ny), dim3(threads), 0, stream, p);
    return tnx_launch_in_order(causal_conv_kernel<T>, dim3(N, ny), dim3(threads), 0, stream, p);
}
}  // namespace

TNX_EXPORT int tnx_causal_conv(const void* proj, int ld, int col0, const float* w, const float* b, int taps, void* state,
                               const int* token_request, const int* positions, const int* q_start, const int* q_len,
                               const int* state_slots, int act, void* out, int N, int C, int is_h16, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (C <= 0 || taps < 1 || taps > MAX_TAPS || !w || act < 0 || act >= TNX_ACT_COUNT || (taps > 1 && !state)) return TNX_ERR_BAD_ARG;
    if (is_h16)
        return conv_launch(ConvArgs<h16>{(const h16*)proj, ld, col0, w, b, taps, (h16*)state, token_request, positions, q_start,
                                         q_len, state_slots, act, (h16*)out, C}, N, stream);
    return conv_launch(ConvArgs<float>{(const float*)proj, ld, col0, w, b, taps, (float*)state, token_request, positions, q_start,
                                       q_len, state_slots, act, (float*)out, C}, N, stream);
}

// most_tokens: an upper bound of the requests' rows (1 for a step of single tokens).
TNX_EXPORT int tnx_selective_scan(const void* x, int x_ld, const float* dt, const void* low, int low_ld, int b_off, int c_off,
                                  const float* decay_log2, const float* dt_bias, const float* skip, const void* z, int z_ld,
                                  float* state, const int* q_start, const int* q_len, const int* state_slots, int act, void* out,
                                  int out_ld, int n_requests, int C, int Ns, int most_tokens, int is_h16, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (C <= 0 || Ns <= 0 || n_requests > 65535 || most_tokens <= 0 || act < 0 || act >= TNX_ACT_COUNT || !dt_bias || !decay_log2 ||
        (((uintptr_t)state | (uintptr_t)decay_log2) & 15))
        return TNX_ERR_BAD_ARG;
    if (is_h16)
        return scan_by_state(ScanArgs<h16>{(const h16*)x, x_ld, dt, (const h16*)low, low_ld, b_off, c_off, decay_log2, dt_bias, skip,
                                           (const h16*)z, z_ld, state, q_start, q_len, state_slots, act, (h16*)out, out_ld, C, Ns},
                             n_requests, most_tokens, stream);
    return scan_by_state(ScanArgs<float>{(const float*)x, x_ld, dt, (const float*)low, low_ld, b_off, c_off, decay_log2, dt_bias,
                                         skip, (const float*)z, z_ld, state, q_start, q_len, state_slots, act, (float*)out, out_ld, C,
                                         Ns},
                         n_requests, most_tokens, stream);
}
