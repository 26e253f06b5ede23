// A selective state-space recurrence with a decay per channel and state ("selective scan").  Per channel c and state n:
//     dt_c <- softplus(dt_c)
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
//   token to the next.  A stage of ST tokens lies in shared memory as what the walk needs (dt and dt x, four tokens of a channel
//   side by side; B and C), all 32-bit; the next stage's numbers travel in registers meanwhile.  Four tokens at a time, the lanes
//   of a channel add up their partial sums of y by exchanging halves, so that each lane ends up with whole sums of its own;
//   these go through shared memory once to the threads that gate and store them while the next stage is walked (one
//   rendezvous a stage).
//   A step of single tokens has a kernel of its own: the state is streamed through once, no shared memory.
#include "common.cuh"

namespace {
constexpr int MAX_TAPS = 8;
constexpr int THREADS = 128;

// softplus(x) = max(x, 0) + ln(1 + e), e = exp(-|x|), and ln(1 + e) = 2 artanh(r), r = e / (2 + e) <= 1/3, by its power series
// r + r^3/3 + r^5/5 + ...: exact to a few units of the last place for tiny e as well, and without a branch, so that a
// thread's several step sizes are formed together.
__device__ __forceinline__ float softplus_f(float x) {
    const float e = __expf(-fabsf(x)), r = __fdividef(e, 2.f + e), q = r * r;
    float t = 1.f / 15.f;
    t = fmaf(t, q, 1.f / 13.f); t = fmaf(t, q, 1.f / 11.f); t = fmaf(t, q, 1.f / 9.f);
    t = fmaf(t, q, 1.f / 7.f); t = fmaf(t, q, 1.f / 5.f); t = fmaf(t, q, 1.f / 3.f);
    return fmaxf(x, 0.f) + 2.f * fmaf(t * q, r, r);
}
__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// the activation the design uses inline, any other by the common function
__device__ __forceinline__ float act_inline(float v, int act) {
    return act == TNX_ACT_SILU ? __fdividef(v, 1.f + __expf(-v)) : apply_activation(v, act);
}

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
        p.out[(size_t)n * C + c] = from_float<T>(act_inline(s, p.act));
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
        for (int i = 0; i < 8; ++i) s[i] = act_inline(s[i], p.act);
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
    const float* skip;                             // [C] or null
    const T* z; int z_ld;
    float* state;                                  // [slots, C, Ns]
    const int* q_start; const int* q_len; const int* state_slots;
    int act;
    T* out; int out_ld;
    int C, Ns;
};

// Adds the four tokens' partial sums up over the L lanes of a channel.  With four or more lanes, lane l ends up with the
// whole sum of token l % 4 in y[0]; with two, of tokens 2 (l % 2) and the next in y[0], y[1]; with one they are whole.
template <int L>
__device__ __forceinline__ void sum_over_lanes(float (&y)[4], int l) {
    if constexpr (L >= 4) {
        // lanes that differ in bit 1 exchange pairs of tokens, then lanes that differ in bit 0 single ones
        const bool up2 = l & 2, up1 = l & 1;
        const float s0 = up2 ? y[0] : y[2], s1 = up2 ? y[1] : y[3];
        const float k0 = (up2 ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, s0, 2);
        const float k1 = (up2 ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, s1, 2);
        y[0] = (up1 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, up1 ? k0 : k1, 1);
#pragma unroll
        for (int o = 4; o < L; o <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
    } else if constexpr (L == 2) {
        const bool up = l & 1;
        const float s0 = up ? y[0] : y[2], s1 = up ? y[1] : y[3];
        y[0] = (up ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, s0, 1);
        y[1] = (up ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, s1, 1);
    }
}

// A lane's states (SPT neighbouring numbers from n0 on of a row of Ns) from and to memory.
template <int SPT>
__device__ __forceinline__ void load_states(const float* row, int n0, int Ns, bool mine, float (&v)[SPT]) {
    if (SPT % 4 == 0 && Ns % 4 == 0) {
#pragma unroll
        for (int m = 0; m < SPT / 4; ++m) {
            const float4 a = mine && n0 + 4 * m < Ns ? *(const float4*)(row + n0 + 4 * m) : make_float4(0.f, 0.f, 0.f, 0.f);
            v[4 * m] = a.x; v[4 * m + 1] = a.y; v[4 * m + 2] = a.z; v[4 * m + 3] = a.w;
        }
    } else {
#pragma unroll
        for (int m = 0; m < SPT; ++m) v[m] = mine && n0 + m < Ns ? row[n0 + m] : 0.f;
    }
}
template <int SPT>
__device__ __forceinline__ void store_states(float* row, int n0, int Ns, const float (&v)[SPT]) {
    if (SPT % 4 == 0 && Ns % 4 == 0) {
#pragma unroll
        for (int m = 0; m < SPT / 4; ++m)
            if (n0 + 4 * m < Ns) *(float4*)(row + n0 + 4 * m) = make_float4(v[4 * m], v[4 * m + 1], v[4 * m + 2], v[4 * m + 3]);
    } else {
#pragma unroll
        for (int m = 0; m < SPT; ++m)
            if (n0 + m < Ns) row[n0 + m] = v[m];
    }
}

// L lanes a channel, SPT states a lane (L * SPT >= Ns), ST tokens a stage.
template <typename T, int L, int SPT, int ST>
__global__ void __launch_bounds__(THREADS) selective_scan_kernel(const ScanArgs<T> p) {
    constexpr int CH = THREADS / L;                // channels of the block
    constexpr int NP = L * SPT;                    // padded states
    constexpr int TP = ST + 4;                     // a channel's tokens of a stage, padded: no bank met twice
    constexpr int XN = (ST * CH + THREADS - 1) / THREADS, BN = (ST * NP + THREADS - 1) / THREADS;
    __shared__ __align__(16) float dts[2][CH][TP], dtx[2][CH][TP];
    __shared__ __align__(16) float bs[2][ST][NP], cs[2][ST][NP];
    __shared__ float ys[2][CH][ST + 1];
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

    // A stage's numbers on their way, asked for before the stage in front of it is walked and kept as they are stored: every
    // load is issued (rows and columns that do not exist read the last ones that do) before the first one is waited for.
    // A thread has the channel ck of every STEP-th token; x and z stay with it, since it gates and stores that channel.
    constexpr int STEP = THREADS / CH;
    static_assert(ST % 4 == 0, "tokens are walked four at a time");
    const int ck = threadIdx.x % CH, tk = threadIdx.x / CH;
    const bool have = c0 + ck < C;
    const int cg = have ? c0 + ck : C - 1;
    const float skip = p.skip ? p.skip[cg] : 0.f;
    float r_dt[XN];
    T r_x[XN], r_z[XN], r_b[BN], r_c[BN];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < XN; ++i) {
            const size_t row = (size_t)(first + min(t0 + tk + i * STEP, len - 1));
            r_dt[i] = p.dt[row * C + cg];
            r_x[i] = p.x[row * p.x_ld + cg];
            r_z[i] = p.z[row * p.z_ld + cg];
        }
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int e = threadIdx.x + i * THREADS, t = e / NP, n = min(e % NP, Ns - 1);
            const T* row = p.low + (size_t)(first + min(t0 + t, len - 1)) * p.low_ld;
            r_b[i] = row[p.b_off + n];
            r_c[i] = row[p.c_off + n];
        }
    };
    // (tokens behind the request's last one are staged with a step size of zero, which leaves the state as it is)
    auto stage = [&](int s, int t0) {
#pragma unroll
        for (int i = 0; i < XN; ++i) {
            const int t = tk + i * STEP;
            const float dt = t0 + t < len ? softplus_f(r_dt[i]) : 0.f;
            if (XN * STEP == ST || t < ST) {
                dts[s][ck][t] = dt;
                dtx[s][ck][t] = dt * to_float(r_x[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < BN; ++i) {
            const int e = threadIdx.x + i * THREADS;
            if (BN * THREADS == ST * NP || e < ST * NP) {
                const bool in = e % NP < Ns;
                (&bs[s][0][0])[e] = in ? to_float(r_b[i]) : 0.f;
                (&cs[s][0][0])[e] = in ? to_float(r_c[i]) : 0.f;
            }
        }
    };

    float S[SPT], a2[SPT];
    float* st = p.state + ((size_t)slot * C + (mine ? c : 0)) * Ns;
    fetch(0);
    load_states<SPT>(st, n0, Ns, mine, S);
    load_states<SPT>(p.decay_log2 + (size_t)(mine ? c : 0) * Ns, n0, Ns, mine, a2);
    stage(0, 0);
    __syncthreads();
    int s = 0;
    for (int t0 = 0; t0 < len; t0 += ST, s ^= 1) {
        const int nt = min(ST, len - t0);
        T x_now[XN], z_now[XN];
#pragma unroll
        for (int i = 0; i < XN; ++i) { x_now[i] = r_x[i]; z_now[i] = r_z[i]; }
        const bool more = t0 + ST < len;
        if (more) fetch(t0 + ST);
#pragma unroll 2
        for (int t = 0; t < nt; t += 4) {
            const float4 d4 = *(const float4*)&dts[s][ch][t], w4 = *(const float4*)&dtx[s][ch][t];
            const float d[4] = {d4.x, d4.y, d4.z, d4.w}, w[4] = {w4.x, w4.y, w4.z, w4.w};
            float y[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                float bv[SPT], cv[SPT];
                if constexpr (SPT % 4 == 0) {
#pragma unroll
                    for (int m = 0; m < SPT / 4; ++m) {
                        *(float4*)(bv + 4 * m) = *(const float4*)&bs[s][t + u][n0 + 4 * m];
                        *(float4*)(cv + 4 * m) = *(const float4*)&cs[s][t + u][n0 + 4 * m];
                    }
                } else {
#pragma unroll
                    for (int m = 0; m < SPT / 2; ++m) {
                        *(float2*)(bv + 2 * m) = *(const float2*)&bs[s][t + u][n0 + 2 * m];
                        *(float2*)(cv + 2 * m) = *(const float2*)&cs[s][t + u][n0 + 2 * m];
                    }
                }
                float y0 = 0.f, y1 = 0.f;
#pragma unroll
                for (int m = 0; m < SPT; ++m) {
                    S[m] = fmaf(exp2_approx(a2[m] * d[u]), S[m], w[u] * bv[m]);
                    if (m & 1) y1 = fmaf(S[m], cv[m], y1); else y0 = fmaf(S[m], cv[m], y0);
                }
                y[u] = y0 + y1;
            }
            sum_over_lanes<L>(y, l);
            if constexpr (L >= 4) { if (l < 4) ys[s][ch][t + l] = y[0]; }
            else if constexpr (L == 2) { ys[s][ch][t + 2 * l] = y[0]; ys[s][ch][t + 2 * l + 1] = y[1]; }
            else {
#pragma unroll
                for (int u = 0; u < 4; ++u) ys[s][ch][t + u] = y[u];
            }
        }
        // The other stage is free: its walk ended before the last rendezvous.  Behind this one, this stage's sums are
        // complete; they are read while other warps walk on, which write the other stage's sums.
        if (more) stage(s ^ 1, t0 + ST);
        __syncthreads();
        if (have) {
#pragma unroll
            for (int i = 0; i < XN; ++i) {
                const int t = tk + i * STEP;
                if (XN * STEP != ST && t >= ST) break;
                const float y = fmaf(skip, to_float(x_now[i]), ys[s][ck][t]) * act_inline(to_float(z_now[i]), p.act);
                if (t < nt) p.out[(size_t)(first + t0 + t) * p.out_ld + cg] = from_float<T>(y);
            }
        }
    }
    if (mine) store_states<SPT>(st, n0, Ns, S);
}

// Steps of single tokens: a thread has SPT states of a channel of one request, a channel's L lanes side by side.
template <typename T, int L, int SPT>
__global__ void __launch_bounds__(THREADS) selective_step_kernel(const ScanArgs<T> p) {
    constexpr int CH = THREADS / L;
    pdl_launch_dependents();
    pdl_wait();
    const int req = blockIdx.y;
    const int len = p.q_len[req], slot = p.state_slots[req];
    const size_t n = p.q_start[req];
    if (len <= 0 || slot < 0) return;              // a padded request of a captured step
    const int l = threadIdx.x % L, c = blockIdx.x * CH + threadIdx.x / L, n0 = l * SPT;
    const int C = p.C, Ns = p.Ns;
    const bool mine = c < C;                       // a whole group of lanes
    const int cc = mine ? c : 0;
    float S[SPT], a2[SPT];
    float* st = p.state + ((size_t)slot * C + cc) * Ns;
    load_states<SPT>(st, n0, Ns, mine, S);
    load_states<SPT>(p.decay_log2 + (size_t)cc * Ns, n0, Ns, mine, a2);
    const float d = softplus_f(p.dt[n * C + cc]), x = to_float(p.x[n * p.x_ld + cc]), z = to_float(p.z[n * p.z_ld + cc]);
    const T* low = p.low + n * p.low_ld;
    const float w = d * x;
    float y = 0.f;
#pragma unroll
    for (int m = 0; m < SPT; ++m) {
        const bool in = n0 + m < Ns;
        const float b = in ? to_float(low[p.b_off + n0 + m]) : 0.f, cv = in ? to_float(low[p.c_off + n0 + m]) : 0.f;
        S[m] = fmaf(exp2_approx(a2[m] * d), S[m], w * b);
        y = fmaf(S[m], cv, y);
    }
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!mine) return;
    store_states<SPT>(st, n0, Ns, S);
    if (l) return;
    if (p.skip) y = fmaf(p.skip[c], x, y);
    p.out[n * p.out_ld + c] = from_float<T>(y * act_inline(z, p.act));
}

template <typename T, int L, int SPT>
int launch_scan(const ScanArgs<T>& p, int n_requests, int most_tokens, cudaStream_t stream) {
    constexpr int CH = THREADS / L;
    constexpr int ST = L * SPT > 128 ? 8 : (L >= 16 ? 16 : (L >= 4 ? 32 : 8));       // shared memory stays below 48 KB
    const dim3 grid((p.C + CH - 1) / CH, n_requests);
    if (most_tokens == 1) return tnx_launch_in_order(selective_step_kernel<T, L, SPT>, grid, dim3(THREADS), 0, stream, p);
    return tnx_launch_in_order(selective_scan_kernel<T, L, SPT, ST>, grid, dim3(THREADS), 0, stream, p);
}

int g_force_states = 0;

template <typename T>
int scan_by_state(const ScanArgs<T>& p, int n_requests, int most_tokens, cudaStream_t stream) {
    // Two states a lane make twice the warps of half the work a token: faster where four leave the SMs fewer than two blocks
    // each (one, for states above 16).  Measured, 2,048 tokens over a state of 16: 2,048 channels 219 us with four and 160
    // with two states a lane, 4,096 channels 221 and 178, 8,192 channels 254 and 239; four requests of 512 tokens of 4,096
    // channels 98 and 101; 4,096 channels over a state of 32 210 and 223.
    static int sms = 0;
    if (!sms) { int dev = 0; cudaGetDevice(&dev); cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev); if (sms <= 0) sms = 1; }
    const long long lanes = (long long)p.C * ((p.Ns + 3) / 4) * n_requests;
    const int spt = g_force_states ? g_force_states : (lanes < (p.Ns <= 16 ? 2LL : 1LL) * sms * THREADS ? 2 : 4);
    if (most_tokens > 1 && spt == 2) {
        if (p.Ns <= 8) return launch_scan<T, 4, 2>(p, n_requests, most_tokens, stream);
        if (p.Ns <= 16) return launch_scan<T, 8, 2>(p, n_requests, most_tokens, stream);
        if (p.Ns <= 32) return launch_scan<T, 16, 2>(p, n_requests, most_tokens, stream);
    }
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
                                  const float* decay_log2, const float* skip, const void* z, int z_ld,
                                  float* state, const int* q_start, const int* q_len, const int* state_slots, int act, void* out,
                                  int out_ld, int n_requests, int C, int Ns, int most_tokens, int is_h16, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (C <= 0 || Ns <= 0 || n_requests > 65535 || most_tokens <= 0 || act < 0 || act >= TNX_ACT_COUNT || !decay_log2 ||
        (((uintptr_t)state | (uintptr_t)decay_log2) & 15))
        return TNX_ERR_BAD_ARG;
    if (is_h16)
        return scan_by_state(ScanArgs<h16>{(const h16*)x, x_ld, dt, (const h16*)low, low_ld, b_off, c_off, decay_log2, skip,
                                           (const h16*)z, z_ld, state, q_start, q_len, state_slots, act, (h16*)out, out_ld, C, Ns},
                             n_requests, most_tokens, stream);
    return scan_by_state(ScanArgs<float>{(const float*)x, x_ld, dt, (const float*)low, low_ld, b_off, c_off, decay_log2,
                                         skip, (const float*)z, z_ld, state, q_start, q_len, state_slots, act, (float*)out, out_ld, C,
                                         Ns},
                         n_requests, most_tokens, stream);
}

// A measurement hook: the states a lane keeps (0: the kernel's own choice; 2 or 4).
TNX_EXPORT int tnx_selective_scan_force(int states) {
    if (states != 0 && states != 2 && states != 4) return TNX_ERR_BAD_ARG;
    g_force_states = states;
    return 0;
}
