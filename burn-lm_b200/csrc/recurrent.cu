// Recurrent mixers over the packed tokens of a step: the short causal convolution with its carried inputs, the
// state-space scan (a scalar decay per head), the selective scan (a decay per channel and state), the gated delta rule (a decay per key channel, an error-correcting
// write), and the group-wise RMS norm with a gate that follows either.  Everything here is fp32.
//
// What a sequence carries lives in a fixed-size block per cache slot, twice: a step that starts at position p reads
// copy (p & 1) and writes copy ((p + n) & 1) for its n new tokens.  A single-token step therefore never overwrites
// what it read, and running it again (a warm-up before a captured graph, a step enqueued ahead and then forgotten)
// gives the same result.  A step that starts at position 0 reads zeros whatever the block holds.
//
// A scan block owns (sequence, head, some value columns): 256 threads = columns x row groups; thread (col, rg) keeps rows
// rg, rg + RG, rg + 2 RG, ... of its column in registers.  A sum over rows is a thread's partial sum and then shuffles
// over the row groups (adjacent lanes): the same order whatever the step's size or batch.  RG = 8 (32 columns a block).
// More lanes a column were measured and left out.  RG = 32 (a warp a column, four times the warps): a 2,048-token scan of
// 64 heads x 128 rows x 64 lanes 0.97 against 0.86 ms, 64 single tokens 0.117 against 0.067 ms.  RG = 16: that scan 0.86
// against 0.79 ms (with the unrolled loop), the delta rule of 16 heads x 128 x 128 1.15 against 1.34 ms (its 64 blocks
// become 128), single tokens 0.089 against 0.072 and 0.069 against 0.050 ms: every block stages the same rows of B and C
// (or k, q and the decays) for fewer columns.  The state is stored as [head][row / RG][column][row % RG], which is the
// order in which a warp holds it, so RG belongs to a model's state and cannot change from step to step.  Fewer columns a
// block (16, in blocks of 128 threads, where a single sequence's 64 blocks would become 128) made the delta rule's prompt
// scan slower as well, 1.86 against 1.38 ms: the staging of a chunk is shared by fewer threads.
#include "common.cuh"

BLM_API const char* blm_recurrent_last_error() { return g_blm_error; }

constexpr int kMaxTaps = 16;
constexpr int kScanThreads = 256;
constexpr int kChunk = 32;         // tokens staged in shared memory at a time

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_r(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// ---------------------------------------------------------------------------------------------
// causal convolution per channel over time; act 1: then silu; act 2: the token's own input is added (y = x + conv(x))
//   x [N, x_stride] (channels at x_col0 ..), taps [C, K] (the last column is the current token's), bias [C] or null
//   carried inputs: hist [K - 1][C] per copy, hist[m] = the input at position start - (K - 1) + m
// ---------------------------------------------------------------------------------------------
__global__ void conv_kernel(const float* __restrict__ x, long long x_stride, int x_col0, int channels,
                            const float* __restrict__ taps, const float* __restrict__ bias, int K, int act,
                            float* __restrict__ out, long long out_stride, int out_col0,
                            const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens,
                            const int* __restrict__ slot_of_seq, const int* __restrict__ start_pos,
                            float* __restrict__ state, long long slot_stride, long long copy_stride, long long hist_off,
                            int carry_here, __nv_bfloat16* __restrict__ out_bf, long long out_bf_stride) {
    const int n = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    float* o = out + (size_t)n * out_stride + out_col0 + c;
    const int seq = token_seq[n];
    if (seq < 0) {           // a row of no sequence
        *o = 0.f;
        if (out_bf) out_bf[(size_t)n * out_bf_stride + c] = __float2bfloat16(0.f);
        return;
    }
    const int i = n - cu_seqlens[seq];
    const int start = start_pos[seq];
    float* both = state + (size_t)slot_of_seq[seq] * slot_stride + hist_off;
    const float* hist = both + (size_t)(start & 1) * copy_stride;
    float acc = bias ? bias[c] : 0.f;
    for (int j = K - 1; j >= 0; --j) {          // the oldest input first
        const int back = i - j;                   // index among the step's rows of this sequence
        float v;
        if (back >= 0) v = x[(size_t)(n - j) * x_stride + x_col0 + c];
        else if (start + back < 0) v = 0.f;
        else v = hist[(size_t)(K - 1 + back) * channels + c];
        acc += taps[(size_t)c * K + (K - 1 - j)] * v;
    }
    if (act == 2) acc += x[(size_t)n * x_stride + x_col0 + c];      // the input itself joins what the taps give
    const float res = act == 1 ? silu_f(acc) : acc;
    *o = res;
    if (out_bf) out_bf[(size_t)n * out_bf_stride + c] = __float2bfloat16(res);
    if (carry_here) {        // every sequence brings one token: its thread also moves the carried inputs on, into the other copy
        float* fresh = both + (size_t)((start + 1) & 1) * copy_stride;
        for (int m = 0; m < K - 1; ++m) {
            const int p = start + 1 - (K - 1) + m;          // the position whose input goes to place m
            fresh[(size_t)m * channels + c] = p < 0 ? 0.f : (p == start ? x[(size_t)n * x_stride + x_col0 + c] : hist[(size_t)(m + 1) * channels + c]);
        }
    }
}

__global__ void conv_carry_kernel(const float* __restrict__ x, long long x_stride, int x_col0, int channels, int K,
                                  const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                                  const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride,
                                  long long copy_stride, long long hist_off) {
    const int seq = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int first = cu_seqlens[seq];
    const int n_new = cu_seqlens[seq + 1] - first;
    if (n_new <= 0) return;      // an empty sequence (padding of a captured step)
    const int start = start_pos[seq];
    float* base = state + (size_t)slot_of_seq[seq] * slot_stride + hist_off;
    const float* old = base + (size_t)(start & 1) * copy_stride;
    float* fresh = base + (size_t)((start + n_new) & 1) * copy_stride;
    float keep[kMaxTaps];
#pragma unroll
    for (int m = 0; m < kMaxTaps - 1; ++m) {
        if (m < K - 1) {
            const int p = start + n_new - (K - 1) + m;      // the position whose input goes to place m
            float v;
            if (p < 0) v = 0.f;
            else if (p >= start) v = x[(size_t)(first + (p - start)) * x_stride + x_col0 + c];
            else v = old[(size_t)(K - 1 + (p - start)) * channels + c];
            keep[m] = v;
        }
    }
#pragma unroll
    for (int m = 0; m < kMaxTaps - 1; ++m)
        if (m < K - 1) fresh[(size_t)m * channels + c] = keep[m];
}

// The same for portions and up to four taps: a thread owns a channel and kConvRows rows after one another, the taps in
// registers and the inputs behind the current one in a sliding window (an input is read once a thread, not once a tap).
constexpr int kConvRows = 16;
template <int K>
__global__ void conv_rows_kernel(const float* __restrict__ x, long long x_stride, int x_col0, int channels, const float* __restrict__ taps,
                                 const float* __restrict__ bias, int act, float* __restrict__ out, long long out_stride, int out_col0,
                                 const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                                 const int* __restrict__ start_pos, const float* __restrict__ state, long long slot_stride,
                                 long long copy_stride, long long hist_off, __nv_bfloat16* __restrict__ out_bf, long long out_bf_stride,
                                 int n_tokens) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int first = blockIdx.y * kConvRows, last = min(n_tokens, first + kConvRows);
    float w[K], past[K];                        // past[j]: the input j tokens back (past[0]: the current one)
#pragma unroll
    for (int j = 0; j < K; ++j) w[j] = taps[(size_t)c * K + (K - 1 - j)];
    const float b = bias ? bias[c] : 0.f;
    int held = -1;                              // the sequence the window belongs to
    const float* in = x + x_col0 + c;
    const int seq0 = token_seq[first];
    if (last - first == kConvRows && seq0 >= 0 && token_seq[last - 1] == seq0 && first - cu_seqlens[seq0] >= K - 1) {
        // all rows and what lies behind them are one sequence's rows of this step: every load at once
        float v[kConvRows + K - 1];
#pragma unroll
        for (int i = 0; i < kConvRows + K - 1; ++i) v[i] = in[(size_t)(first - (K - 1) + i) * x_stride];
#pragma unroll
        for (int i = 0; i < kConvRows; ++i) {
            float acc = b;
#pragma unroll
            for (int j = K - 1; j >= 0; --j) acc += w[j] * v[i + K - 1 - j];
            if (act == 2) acc += v[i + K - 1];
            const float res = act == 1 ? silu_f(acc) : acc;
            out[(size_t)(first + i) * out_stride + out_col0 + c] = res;
            if (out_bf) out_bf[(size_t)(first + i) * out_bf_stride + c] = __float2bfloat16(res);
        }
        return;
    }
#pragma unroll 4
    for (int n = first; n < last; ++n) {
        const int seq = token_seq[n];
        float res = 0.f;
        if (seq >= 0) {
            if (seq != held) {                  // the window's inputs before this row: the step's, the carried ones, or zeros
                held = seq;
                const int i = n - cu_seqlens[seq], start = start_pos[seq];
                const float* hist = state + (size_t)slot_of_seq[seq] * slot_stride + hist_off + (size_t)(start & 1) * copy_stride;
#pragma unroll
                for (int j = 1; j < K; ++j) {
                    const int back = i - j;
                    past[j - 1] = back >= 0 ? in[(size_t)(n - j) * x_stride] : (start + back < 0 ? 0.f : hist[(size_t)(K - 1 + back) * channels + c]);
                }
            }
#pragma unroll
            for (int j = K - 1; j > 0; --j) past[j] = past[j - 1];
            past[0] = in[(size_t)n * x_stride];
            float acc = b;
#pragma unroll
            for (int j = K - 1; j >= 0; --j) acc += w[j] * past[j];
            if (act == 2) acc += past[0];
            res = act == 1 ? silu_f(acc) : acc;
        }
        out[(size_t)n * out_stride + out_col0 + c] = res;
        if (out_bf) out_bf[(size_t)n * out_bf_stride + c] = __float2bfloat16(res);
    }
}

BLM_API int blm_causal_conv(const float* x, long long x_stride, int x_col0, int channels, const float* taps, const float* bias,
                            int K, int act, float* out, long long out_stride, int out_col0, const int* token_seq,
                            const int* cu_seqlens, const int* slot_of_seq, const int* start_pos, int n_tokens, int n_seqs,
                            float* state, long long slot_stride, long long copy_stride, long long hist_off,
                            int single_tokens, void* out_bf, long long out_bf_stride, cudaStream_t stream) {
    // out_bf (may be null): the result once more as bfloat16 [N, out_bf_stride], channel c in column c
    if (n_tokens == 0) return BLM_OK;
    BLM_REQUIRE(channels > 0 && K >= 1 && K <= kMaxTaps, "causal_conv: %d taps; this kernel takes 1 to %d", K, kMaxTaps);
    BLM_REQUIRE(n_tokens <= 65535 && n_seqs <= 65535, "causal_conv: a step of %d rows; this kernel takes 65,535", n_tokens);
    const int threads = 128;
    if (!single_tokens && K >= 2 && K <= 4 && n_tokens >= 4 * kConvRows) {
        dim3 tiles((channels + threads - 1) / threads, (n_tokens + kConvRows - 1) / kConvRows);
        auto kern = K == 2 ? conv_rows_kernel<2> : (K == 3 ? conv_rows_kernel<3> : conv_rows_kernel<4>);
        kern<<<tiles, threads, 0, stream>>>(x, x_stride, x_col0, channels, taps, bias, act, out, out_stride, out_col0, token_seq, cu_seqlens,
                                            slot_of_seq, start_pos, state, slot_stride, copy_stride, hist_off, (__nv_bfloat16*)out_bf,
                                            out_bf_stride, n_tokens);
    } else {
        dim3 grid((channels + threads - 1) / threads, n_tokens);
        conv_kernel<<<grid, threads, 0, stream>>>(x, x_stride, x_col0, channels, taps, bias, K, act, out, out_stride, out_col0,
                                                  token_seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride,
                                                  hist_off, single_tokens && K > 1 ? 1 : 0, (__nv_bfloat16*)out_bf, out_bf_stride);
    }
    int rc = blm_check_launch("causal_conv");
    if (rc != BLM_OK || K == 1 || single_tokens) return rc;
    dim3 grid2((channels + threads - 1) / threads, n_seqs);
    conv_carry_kernel<<<grid2, threads, 0, stream>>>(x, x_stride, x_col0, channels, K, cu_seqlens, slot_of_seq, start_pos, state,
                                                     slot_stride, copy_stride, hist_off);
    return blm_check_launch("causal_conv (carry)");
}

// ---------------------------------------------------------------------------------------------
// the scans
// ---------------------------------------------------------------------------------------------
struct ScanSeq {
    int first, n_new, start;
    const float* read;     // nullptr: the state is zero
    float* write;
};

__device__ __forceinline__ ScanSeq scan_seq(int seq, const int* cu_seqlens, const int* slot_of_seq, const int* start_pos,
                                            float* state, long long slot_stride, long long copy_stride, long long off) {
    ScanSeq s;
    s.first = cu_seqlens[seq];
    s.n_new = cu_seqlens[seq + 1] - s.first;
    s.start = start_pos[seq];
    float* base = state + (size_t)slot_of_seq[seq < 0 ? 0 : seq] * slot_stride + off;
    s.read = s.start > 0 ? base + (size_t)(s.start & 1) * copy_stride : nullptr;
    s.write = base + (size_t)((s.start + s.n_new) & 1) * copy_stride;
    return s;
}

template <int RG, typename V>
__device__ __forceinline__ V group_sum(V v) {       // over the row groups of a column (adjacent lanes)
#pragma unroll
    for (int o = 1; o < RG; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// State-space scan.  Per head h (group g = h / (heads / groups)), S [N x dv]:
//     S <- exp(-exp(A_log_h) dt) S + dt B x^T;   y = S^T C + D_h x,    dt = softplus(dt_raw + dt_bias_h)
// xbc [T, *]: x at x_col0 + h dv, B at b_col0 + g N, C at c_col0 + g N;  dt_raw [T, *] at dt_col0 + h.
// AT: the type the state is held and summed in inside a step.  float: the serving path.  double: the 32-bit path, where a
// head whose decay is close to 1 sums a thousand tokens into a state many times larger than its read-out (S^T C cancels),
// and float sums alone put 1e-5 of the row's largest value on it; the carried state is rounded to float either way.
template <int RN, int RG, typename AT>
__global__ void __launch_bounds__(kScanThreads)
    ssm_scan_kernel(const float* __restrict__ xbc, long long xbc_stride, int x_col0, int b_col0, int c_col0,
                    const float* __restrict__ dt_raw, long long dt_stride, int dt_col0, const float* __restrict__ dt_bias,
                    const float* __restrict__ A_log, const float* __restrict__ D, float* __restrict__ y, long long y_stride,
                    int heads, int groups, int N, int dv, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                    const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride, long long copy_stride,
                    long long state_off) {
    constexpr int NP = RN * RG, kCols = kScanThreads / RG, kRowGroups = RG;
    extern __shared__ __align__(16) float sm[];
    float* Bs = sm;                         // [kChunk][NP]
    float* Cs = Bs + kChunk * NP;           // [kChunk][NP]
    float* xs = Cs + kChunk * NP;           // [kChunk][kCols]
    AT* dts = reinterpret_cast<AT*>(xs + kChunk * kCols);       // [kChunk]  (an even number of floats lies before it)
    AT* decs = dts + kChunk;                                    // [kChunk]
    const int seq = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kCols;
    const ScanSeq sq = scan_seq(seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
    if (sq.n_new <= 0) return;
    const int tid = threadIdx.x, col = tid / kRowGroups, rg = tid % kRowGroups;
    const int g = h / (heads / groups);
    const bool live = col0 + col < dv;
    const size_t head_off = (size_t)h * RN * dv * kRowGroups;
    AT s[RN];
#pragma unroll
    for (int r = 0; r < RN; ++r)
        s[r] = (sq.read && live) ? (AT)sq.read[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] : (AT)0;
    const float a = -expf(A_log[h]);
    const float bias = dt_bias[h], skip = D[h];
    for (int c0 = 0; c0 < sq.n_new; c0 += kChunk) {
        const int nt = min(kChunk, sq.n_new - c0);
        __syncthreads();
        for (int e = tid; e < nt * NP; e += blockDim.x) {
            const int t = e / NP, n = e % NP;
            const float* row = xbc + (size_t)(sq.first + c0 + t) * xbc_stride;
            Bs[e] = n < N ? row[b_col0 + g * N + n] : 0.f;
            Cs[e] = n < N ? row[c_col0 + g * N + n] : 0.f;
        }
        for (int e = tid; e < nt * kCols; e += blockDim.x) {
            const int t = e / kCols, p = e % kCols;
            xs[e] = col0 + p < dv ? xbc[(size_t)(sq.first + c0 + t) * xbc_stride + x_col0 + h * dv + col0 + p] : 0.f;
        }
        for (int t = tid; t < nt; t += blockDim.x) {
            const float dt = softplus_r(dt_raw[(size_t)(sq.first + c0 + t) * dt_stride + dt_col0 + h] + bias);
            dts[t] = (AT)dt;
            if (sizeof(AT) == 8) decs[t] = (AT)exp((double)a * (double)dt);
            else decs[t] = (AT)expf(a * dt);
        }
        __syncthreads();
        // (tokens unrolled: a token's shuffles and store wait for nothing the next token's multiply-adds need; the sum over
        // a thread's rows in four partial sums, so that no chain of dependent additions is longer than RN / 4)
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const AT dec = decs[t], dt = dts[t], xv = (AT)xs[t * kCols + col];
            const float* b = Bs + t * NP + rg;
            const float* c = Cs + t * NP + rg;
            AT part[4] = {0, 0, 0, 0};
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                s[r] = dec * s[r] + (dt * (AT)b[r * kRowGroups]) * xv;
                part[r & 3] += s[r] * (AT)c[r * kRowGroups];
            }
            AT acc = (part[0] + part[1]) + (part[2] + part[3]);
            acc = group_sum<RG>(acc);
            if (rg == 0 && live) y[(size_t)(sq.first + c0 + t) * y_stride + h * dv + col0 + col] = (float)(acc + (AT)skip * xv);
        }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < RN; ++r) sq.write[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] = (float)s[r];
    }
}

// Gated delta rule.  Per head h (query/key head c = h / (heads / qk_heads)), S [dk x dv]:
//     S <- g[:, None] S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// with k, q made unit vectors (x / sqrt(sum x^2 + 1e-6)), q also times dk^(-1/2), beta = sigmoid(b_raw),
// g = exp(-exp(A_log_h) softplus(a_raw + dt_bias)) per head and key channel.
template <int RN, int RG>
__global__ void __launch_bounds__(kScanThreads)
    delta_scan_kernel(const float* __restrict__ q, long long q_stride, int q_col0, const float* __restrict__ k, long long k_stride,
                      int k_col0, const float* __restrict__ v, long long v_stride, int v_col0, const float* __restrict__ b_raw,
                      long long b_stride, int b_col0, const float* __restrict__ a_raw, long long a_stride, int a_col0,
                      const float* __restrict__ dt_bias, const float* __restrict__ A_log, float* __restrict__ o, long long o_stride,
                      int heads, int qk_heads, int dk, int dv, const int* __restrict__ cu_seqlens,
                      const int* __restrict__ slot_of_seq, const int* __restrict__ start_pos, float* __restrict__ state,
                      long long slot_stride, long long copy_stride, long long state_off) {
    constexpr int NP = RN * RG, kCols = kScanThreads / RG, kRowGroups = RG;
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                          // [kChunk][NP]
    float* qs = ks + kChunk * NP;            // [kChunk][NP]
    float* gs = qs + kChunk * NP;            // [kChunk][NP]
    float* vs = gs + kChunk * NP;            // [kChunk][kCols]
    float* betas = vs + kChunk * kCols;      // [kChunk]
    const int seq = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kCols;
    const ScanSeq sq = scan_seq(seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
    if (sq.n_new <= 0) return;
    const int tid = threadIdx.x, col = tid / kRowGroups, rg = tid % kRowGroups;
    const int lane = tid & 31, warp = tid >> 5;
    const int c = h / (heads / qk_heads);
    const bool live = col0 + col < dv;
    const size_t head_off = (size_t)h * RN * dv * kRowGroups;
    float s[RN];
#pragma unroll
    for (int r = 0; r < RN; ++r)
        s[r] = (sq.read && live) ? sq.read[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] : 0.f;
    const float a = -expf(A_log[h]);
    const float q_scale = 1.0f / sqrtf((float)dk);
    for (int c0 = 0; c0 < sq.n_new; c0 += kChunk) {
        const int nt = min(kChunk, sq.n_new - c0);
        __syncthreads();
        for (int e = tid; e < nt * NP; e += blockDim.x) {
            const int t = e / NP, n = e % NP;
            const size_t row = (size_t)(sq.first + c0 + t);
            ks[e] = n < dk ? k[row * k_stride + k_col0 + c * dk + n] : 0.f;
            qs[e] = n < dk ? q[row * q_stride + q_col0 + c * dk + n] : 0.f;
            gs[e] = n < dk ? expf(a * softplus_r(a_raw[row * a_stride + a_col0 + h * dk + n] + dt_bias[h * dk + n])) : 1.f;
        }
        for (int e = tid; e < nt * kCols; e += blockDim.x) {
            const int t = e / kCols, p = e % kCols;
            vs[e] = col0 + p < dv ? v[(size_t)(sq.first + c0 + t) * v_stride + v_col0 + h * dv + col0 + p] : 0.f;
        }
        for (int t = tid; t < nt; t += blockDim.x)
            betas[t] = sigmoid_f(b_raw[(size_t)(sq.first + c0 + t) * b_stride + b_col0 + h]);
        __syncthreads();
        for (int t = warp; t < nt; t += blockDim.x / 32) {       // unit vectors: a warp per token
            float sk = 0.f, sqq = 0.f;
            for (int n = lane; n < NP; n += 32) {
                sk += ks[t * NP + n] * ks[t * NP + n];
                sqq += qs[t * NP + n] * qs[t * NP + n];
            }
            sk = warp_sum(sk);
            sqq = warp_sum(sqq);
            const float ik = 1.0f / sqrtf(sk + 1e-6f), iq = q_scale / sqrtf(sqq + 1e-6f);
            for (int n = lane; n < NP; n += 32) {
                ks[t * NP + n] *= ik;
                qs[t * NP + n] *= iq;
            }
        }
        __syncthreads();
#pragma unroll 2
        for (int t = 0; t < nt; ++t) {
            const float beta = betas[t], vv = vs[t * kCols + col];
            const float* kk = ks + t * NP + rg;
            const float* qq = qs + t * NP + rg;
            const float* gg = gs + t * NP + rg;
            float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                s[r] *= gg[r * kRowGroups];
                part[r & 3] += s[r] * kk[r * kRowGroups];
            }
            float acc = (part[0] + part[1]) + (part[2] + part[3]);
            acc = group_sum<RG>(acc);
            const float u = beta * (vv - acc);
            float outp[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                s[r] += kk[r * kRowGroups] * u;
                outp[r & 3] += s[r] * qq[r * kRowGroups];
            }
            float out = (outp[0] + outp[1]) + (outp[2] + outp[3]);
            out = group_sum<RG>(out);
            if (rg == 0 && live) o[(size_t)(sq.first + c0 + t) * o_stride + h * dv + col0 + col] = out;
        }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < RN; ++r) sq.write[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] = s[r];
    }
}


// ---------------------------------------------------------------------------------------------
// token shift: every one of S mixes of a token's input with the input of the token before it,
//     out[s][n] = x[n] + (x[n - 1] - x[n]) * mu[s]        (zeros before a sequence's first token)
// x float32 [N, x_stride]; mu float32 [S][C]; out [S][N][C].  The last input of every sequence is carried in `state`
// at hist_off, [C] per copy, as the convolution carries its inputs (it is the carried input of a convolution of two taps).
// ---------------------------------------------------------------------------------------------
template <typename TO>
__global__ void shift_mix_kernel(const float* __restrict__ x, long long x_stride, int channels, const float* __restrict__ mu, int S,
                                 TO* __restrict__ out, long long set_stride, const int* __restrict__ token_seq,
                                 const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                                 const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride,
                                 long long copy_stride, long long hist_off, int carry_here) {
    const int n = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int seq = token_seq[n];
    if (seq < 0) {           // a row of no sequence
        for (int s = 0; s < S; ++s) out[(size_t)s * set_stride + (size_t)n * channels + c] = from_f32<TO>(0.f);
        return;
    }
    const int i = n - cu_seqlens[seq];
    const int start = start_pos[seq];
    float* both = state + (size_t)slot_of_seq[seq] * slot_stride + hist_off;
    const float cur = x[(size_t)n * x_stride + c];
    float prev;
    if (i > 0) prev = x[(size_t)(n - 1) * x_stride + c];
    else if (start == 0) prev = 0.f;
    else prev = both[(size_t)(start & 1) * copy_stride + c];
    const float diff = prev - cur;
    for (int s = 0; s < S; ++s)
        out[(size_t)s * set_stride + (size_t)n * channels + c] = from_f32<TO>(fmaf(diff, mu[(size_t)s * channels + c], cur));
    if (carry_here) both[(size_t)((start + 1) & 1) * copy_stride + c] = cur;
}

BLM_API int blm_shift_mix(const float* x, long long x_stride, int channels, const float* mu, int n_mixes, void* out, int out_dtype,
                          const int* token_seq, const int* cu_seqlens, const int* slot_of_seq, const int* start_pos, int n_tokens,
                          int n_seqs, float* state, long long slot_stride, long long copy_stride, long long hist_off,
                          int single_tokens, cudaStream_t stream) {
    if (n_tokens == 0) return BLM_OK;
    BLM_REQUIRE(channels > 0 && n_mixes > 0, "shift_mix: bad sizes");
    BLM_REQUIRE(n_tokens <= 65535 && n_seqs <= 65535, "shift_mix: a step of %d rows; this kernel takes 65,535", n_tokens);
    const int threads = 128;
    dim3 grid((channels + threads - 1) / threads, n_tokens);
    const long long set_stride = (long long)n_tokens * channels;
    if (out_dtype == BLM_F32)
        shift_mix_kernel<float><<<grid, threads, 0, stream>>>(x, x_stride, channels, mu, n_mixes, (float*)out, set_stride, token_seq,
                                                              cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride,
                                                              hist_off, single_tokens ? 1 : 0);
    else if (out_dtype == BLM_BF16)
        shift_mix_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>(x, x_stride, channels, mu, n_mixes, (__nv_bfloat16*)out, set_stride,
                                                                      token_seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride,
                                                                      copy_stride, hist_off, single_tokens ? 1 : 0);
    else
        return blm_fail(BLM_BAD_ARGUMENT, "shift_mix: out dtype %d", out_dtype);
    int rc = blm_check_launch("shift_mix");
    if (rc != BLM_OK || single_tokens) return rc;
    dim3 grid2((channels + threads - 1) / threads, n_seqs);
    conv_carry_kernel<<<grid2, threads, 0, stream>>>(x, x_stride, 0, channels, 2, cu_seqlens, slot_of_seq, start_pos, state,
                                                     slot_stride, copy_stride, hist_off);
    return blm_check_launch("shift_mix (carry)");
}

// Linear attention with a decay per key channel.  Per head h, S [dk x dv]:
//     read first (a bonus u for the current token):   o = (S + diag(u) k v^T)^T q;   S <- diag(w) S + k v^T
//     read last:                                       S <- diag(w) S + k v^T;        o = S^T q
// What the raw inputs mean is the kind:
//     kDecayExpExp       w = exp(-exp(a + bias)),  q and k as they come            (bias [H dk]: the decays' base)
//     kDecayLowerBound   w = low + (1 - low) sigmoid(a + bias),  k = 1 - w,  q = silu(q)     (extra [H dk]: low)
// `extra` is the bonus u [H dk] when the state is read first.  AT as in the state-space scan: double holds the state and
// the sums over its rows in float64 inside a step (the 32-bit path).
constexpr int kDecayExpExp = 0, kDecayLowerBound = 1;

template <int RN, int RG, bool READ_FIRST, typename AT>
__global__ void __launch_bounds__(kScanThreads)
    decay_scan_kernel(const float* __restrict__ q, long long q_stride, int q_col0, const float* __restrict__ k, long long k_stride,
                      int k_col0, const float* __restrict__ v, long long v_stride, int v_col0, const float* __restrict__ a_raw,
                      long long a_stride, int a_col0, const float* __restrict__ bias, const float* __restrict__ extra,
                      float* __restrict__ o, long long o_stride, int heads, int dk, int dv, int kind,
                      const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq, const int* __restrict__ start_pos,
                      float* __restrict__ state, long long slot_stride, long long copy_stride, long long state_off) {
    constexpr int NP = RN * RG, kCols = kScanThreads / RG, kRowGroups = RG;
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                          // [kChunk][NP]
    float* qs = ks + kChunk * NP;            // [kChunk][NP]
    float* ws = qs + kChunk * NP;            // [kChunk][NP]
    float* vs = ws + kChunk * NP;            // [kChunk][kCols]
    const int seq = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kCols;
    const ScanSeq sq = scan_seq(seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
    if (sq.n_new <= 0) return;
    const int tid = threadIdx.x, col = tid / kRowGroups, rg = tid % kRowGroups;
    const bool live = col0 + col < dv;
    const size_t head_off = (size_t)h * RN * dv * kRowGroups;
    AT s[RN];
    float ub[RN];
#pragma unroll
    for (int r = 0; r < RN; ++r) {
        s[r] = (sq.read && live) ? (AT)sq.read[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] : (AT)0;
        const int n = r * kRowGroups + rg;
        ub[r] = (READ_FIRST && extra && n < dk) ? extra[h * dk + n] : 0.f;
    }
    for (int c0 = 0; c0 < sq.n_new; c0 += kChunk) {
        const int nt = min(kChunk, sq.n_new - c0);
        __syncthreads();
        for (int e = tid; e < nt * NP; e += blockDim.x) {
            const int t = e / NP, n = e % NP;
            const size_t row = (size_t)(sq.first + c0 + t);
            float kk = 0.f, qq = 0.f, w = 1.f;
            if (n < dk) {
                const float a = a_raw[row * a_stride + a_col0 + h * dk + n] + bias[h * dk + n];
                qq = q[row * q_stride + q_col0 + h * dk + n];
                if (kind == kDecayExpExp) {
                    w = expf(-expf(a));
                    kk = k[row * k_stride + k_col0 + h * dk + n];
                } else {
                    const float low = extra[h * dk + n];
                    w = low + (1.0f - low) * sigmoid_f(a);
                    kk = 1.0f - w;
                    qq = silu_f(qq);
                }
            }
            ks[e] = kk;
            qs[e] = qq;
            ws[e] = w;
        }
        for (int e = tid; e < nt * kCols; e += blockDim.x) {
            const int t = e / kCols, p = e % kCols;
            vs[e] = col0 + p < dv ? v[(size_t)(sq.first + c0 + t) * v_stride + v_col0 + h * dv + col0 + p] : 0.f;
        }
        __syncthreads();
#pragma unroll 2
        for (int t = 0; t < nt; ++t) {
            const AT vv = (AT)vs[t * kCols + col];
            const float* kk = ks + t * NP + rg;
            const float* qq = qs + t * NP + rg;
            const float* ww = ws + t * NP + rg;
            AT part[4] = {0, 0, 0, 0};
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                const AT kv = (AT)kk[r * kRowGroups] * vv;
                if (READ_FIRST) {
                    part[r & 3] += (s[r] + (AT)ub[r] * kv) * (AT)qq[r * kRowGroups];
                    s[r] = (AT)ww[r * kRowGroups] * s[r] + kv;
                } else {
                    s[r] = (AT)ww[r * kRowGroups] * s[r] + kv;
                    part[r & 3] += s[r] * (AT)qq[r * kRowGroups];
                }
            }
            AT acc = (part[0] + part[1]) + (part[2] + part[3]);
            acc = group_sum<RG>(acc);
            if (rg == 0 && live) o[(size_t)(sq.first + c0 + t) * o_stride + h * dv + col0 + col] = (float)acc;
        }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < RN; ++r) sq.write[head_off + ((size_t)r * dv + col0 + col) * kRowGroups + rg] = (float)s[r];
    }
}

static int row_groups(int) { return 8; }
static int rows_per_thread(int n) {       // the smallest instance that holds n rows: row groups x RN
    for (int rn : {1, 2, 4, 8, 16, 32})
        if (rn * row_groups(n) >= n) return rn;
    return 0;
}

template <typename Kern>
static int allow_smem(Kern k, size_t smem, const char* what) {
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return blm_fail(BLM_CUDA_ERROR, "%s: %s", what, cudaGetErrorString(e));
    }
    return BLM_OK;
}

BLM_API int blm_ssm_scan(const float* xbc, long long xbc_stride, int x_col0, int b_col0, int c_col0, const float* dt_raw,
                         long long dt_stride, int dt_col0, const float* dt_bias, const float* A_log, const float* D, float* y,
                         long long y_stride, int heads, int groups, int N, int dv, const int* cu_seqlens, const int* slot_of_seq,
                         const int* start_pos, int n_seqs, float* state, long long slot_stride, long long copy_stride,
                         long long state_off, int wide_sums, cudaStream_t stream) {
    if (n_seqs == 0) return BLM_OK;
    const int rn = rows_per_thread(N);
    BLM_REQUIRE(rn > 0, "ssm_scan: a state of %d rows; this kernel takes up to %d", N, 32 * 8);
    BLM_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && dv > 0, "ssm_scan: bad head counts");
    BLM_REQUIRE(heads <= 65535 && dv <= 65535 * 8, "ssm_scan: too many heads");
    const int rg = row_groups(N), cols = kScanThreads / rg;
    dim3 grid(n_seqs, heads, (dv + cols - 1) / cols);
    const size_t smem = ((size_t)2 * kChunk * rn * rg + kChunk * cols) * sizeof(float) + 2 * kChunk * sizeof(double);
#define SSM_ARGS xbc, xbc_stride, x_col0, b_col0, c_col0, dt_raw, dt_stride, dt_col0, dt_bias, A_log, D, y, y_stride, heads, groups, N, dv, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off
#define BLM_SCAN(RN, RG)                                                                                 \
    if (rn == RN && rg == RG && wide_sums) {                                                             \
        int rc = allow_smem(ssm_scan_kernel<RN, RG, double>, smem, "ssm_scan_kernel");                   \
        if (rc != BLM_OK) return rc;                                                                     \
        ssm_scan_kernel<RN, RG, double><<<grid, kScanThreads, smem, stream>>>(SSM_ARGS);                 \
    }                                                                                                    \
    if (rn == RN && rg == RG && !wide_sums) {                                                            \
        int rc = allow_smem(ssm_scan_kernel<RN, RG, float>, smem, "ssm_scan_kernel");                    \
        if (rc != BLM_OK) return rc;                                                                     \
        ssm_scan_kernel<RN, RG, float><<<grid, kScanThreads, smem, stream>>>(xbc, xbc_stride, x_col0, b_col0, c_col0, dt_raw, dt_stride, dt_col0, dt_bias, A_log, D, y, y_stride, heads, groups, N, dv, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off); \
    }
    BLM_SCAN(1, 8) BLM_SCAN(2, 8) BLM_SCAN(4, 8) BLM_SCAN(8, 8) BLM_SCAN(16, 8) BLM_SCAN(32, 8)
#undef BLM_SCAN
#undef SSM_ARGS
    return blm_check_launch("ssm_scan");
}

BLM_API int blm_delta_scan(const float* q, long long q_stride, int q_col0, const float* k, long long k_stride, int k_col0,
                           const float* v, long long v_stride, int v_col0, const float* b_raw, long long b_stride, int b_col0,
                           const float* a_raw, long long a_stride, int a_col0, const float* dt_bias, const float* A_log, float* o,
                           long long o_stride, int heads, int qk_heads, int dk, int dv, const int* cu_seqlens,
                           const int* slot_of_seq, const int* start_pos, int n_seqs, float* state, long long slot_stride,
                           long long copy_stride, long long state_off, cudaStream_t stream) {
    if (n_seqs == 0) return BLM_OK;
    const int rn = rows_per_thread(dk);
    BLM_REQUIRE(rn > 0, "delta_scan: keys of %d lanes; this kernel takes up to %d", dk, 32 * 8);
    BLM_REQUIRE(heads > 0 && qk_heads > 0 && heads % qk_heads == 0 && dv > 0, "delta_scan: bad head counts");
    BLM_REQUIRE(heads <= 65535 && dv <= 65535 * 8, "delta_scan: too many heads");
    const int rg = row_groups(dk), cols = kScanThreads / rg;
    dim3 grid(n_seqs, heads, (dv + cols - 1) / cols);
    const size_t smem = ((size_t)3 * kChunk * rn * rg + kChunk * cols + 2 * kChunk) * sizeof(float);
#define BLM_SCAN(RN, RG)                                                                                 \
    if (rn == RN && rg == RG) {                                                                          \
        int rc = allow_smem(delta_scan_kernel<RN, RG>, smem, "delta_scan_kernel");                                   \
        if (rc != BLM_OK) return rc;                                                                     \
        delta_scan_kernel<RN, RG><<<grid, kScanThreads, smem, stream>>>(q, q_stride, q_col0, k, k_stride, k_col0, v, v_stride, v_col0, b_raw, b_stride, b_col0, a_raw, a_stride, a_col0, dt_bias, A_log, o, o_stride, heads, qk_heads, dk, dv, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off); \
    }
    BLM_SCAN(1, 8) BLM_SCAN(2, 8) BLM_SCAN(4, 8) BLM_SCAN(8, 8) BLM_SCAN(16, 8) BLM_SCAN(32, 8)
#undef BLM_SCAN
    return blm_check_launch("delta_scan");
}

BLM_API int blm_decay_scan(const float* q, long long q_stride, int q_col0, const float* k, long long k_stride, int k_col0,
                           const float* v, long long v_stride, int v_col0, const float* a_raw, long long a_stride, int a_col0,
                           const float* bias, const float* extra, float* o, long long o_stride, int heads, int dk, int dv, int kind,
                           int read_first, const int* cu_seqlens, const int* slot_of_seq, const int* start_pos, int n_seqs,
                           float* state, long long slot_stride, long long copy_stride, long long state_off, int wide_sums,
                           cudaStream_t stream) {
    if (n_seqs == 0) return BLM_OK;
    const int rn = rows_per_thread(dk);
    BLM_REQUIRE(rn > 0, "decay_scan: keys of %d lanes; this kernel takes up to %d", dk, 32 * 8);
    BLM_REQUIRE(heads > 0 && dv > 0 && heads <= 65535 && dv <= 65535 * 8, "decay_scan: bad head counts");
    BLM_REQUIRE(kind == kDecayExpExp || kind == kDecayLowerBound, "decay_scan: kind %d", kind);
    BLM_REQUIRE(kind != kDecayExpExp || k != nullptr, "decay_scan: this kind reads its keys");
    BLM_REQUIRE(kind != kDecayLowerBound || (extra != nullptr && !read_first), "decay_scan: a lower bound, and the state read last");
    const int rg = row_groups(dk), cols = kScanThreads / rg;
    dim3 grid(n_seqs, heads, (dv + cols - 1) / cols);
    const size_t smem = ((size_t)3 * kChunk * rn * rg + kChunk * cols) * sizeof(float);
#define DECAY_ARGS q, q_stride, q_col0, k, k_stride, k_col0, v, v_stride, v_col0, a_raw, a_stride, a_col0, bias, extra, o, o_stride, heads, dk, dv, kind, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off
#define BLM_ONE(RN, RG, FIRST, AT)                                                                       \
    {                                                                                                    \
        int rc = allow_smem(decay_scan_kernel<RN, RG, FIRST, AT>, smem, "decay_scan_kernel");            \
        if (rc != BLM_OK) return rc;                                                                     \
        decay_scan_kernel<RN, RG, FIRST, AT><<<grid, kScanThreads, smem, stream>>>(DECAY_ARGS);          \
    }
#define BLM_SCAN(RN, RG)                                                                                 \
    if (rn == RN && rg == RG) {                                                                          \
        if (read_first && wide_sums) BLM_ONE(RN, RG, true, double)                                       \
        else if (read_first) BLM_ONE(RN, RG, true, float)                                                \
        else if (wide_sums) BLM_ONE(RN, RG, false, double)                                               \
        else BLM_ONE(RN, RG, false, float)                                                               \
    }
    BLM_SCAN(1, 8) BLM_SCAN(2, 8) BLM_SCAN(4, 8) BLM_SCAN(8, 8) BLM_SCAN(16, 8) BLM_SCAN(32, 8)
#undef BLM_SCAN
#undef BLM_ONE
#undef DECAY_ARGS
    return blm_check_launch("decay_scan");
}

// ---------------------------------------------------------------------------------------------
// RMS norm over groups of a row's lanes, with a gate
//   mode 0 (gate first):  u = y silu(gate);  out = u / sqrt(mean_group(u^2) + eps) * w[lane % period]
//   mode 1 (gate last):   out = y / sqrt(mean_group(y^2) + eps) * w[lane % period] * sigmoid(gate)
//   mode 2 (silu last):   out = y / sqrt(mean_group(y^2) + eps) * w[lane % period] * silu(gate)
//   mode 3 (no gate):     out = y / sqrt(mean_group(y^2) + eps) * w[lane % period]            (gate may be null)
// A warp per (row, group).  Rows of no sequence hold zeros and give zeros.
// ---------------------------------------------------------------------------------------------
template <typename TA>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, long long y_stride, const float* __restrict__ gate,
                                        long long gate_stride, int gate_col0, const float* __restrict__ w, int period,
                                        int group, int n_groups, int mode, float eps, TA* __restrict__ out, long long out_stride) {
    const int n = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const float* yr = y + (size_t)n * y_stride;
    const float* gr = gate ? gate + (size_t)n * gate_stride + gate_col0 : nullptr;
    TA* orow = out + (size_t)n * out_stride;
    for (int g = warp; g < n_groups; g += n_warps) {
        const int lo = g * group;
        float ss = 0.f;
        for (int i = lane; i < group; i += 32) {
            float u = yr[lo + i];
            if (mode == 0) u *= silu_f(gr[lo + i]);
            ss += u * u;
        }
        ss = warp_sum(ss);
        const float inv = 1.0f / sqrtf(ss / (float)group + eps);
        for (int i = lane; i < group; i += 32) {
            float u = yr[lo + i];
            const float gv = gr ? gr[lo + i] : 0.f;
            if (mode == 0) u = u * silu_f(gv) * inv * w[(lo + i) % period];
            else if (mode == 1) u = u * inv * w[(lo + i) % period] * sigmoid_f(gv);
            else if (mode == 2) u = u * inv * w[(lo + i) % period] * silu_f(gv);
            else u = u * inv * w[(lo + i) % period];
            orow[lo + i] = from_f32<TA>(u);
        }
    }
}

BLM_API int blm_gated_group_norm(const float* y, long long y_stride, const float* gate, long long gate_stride, int gate_col0,
                                 const float* w, int period, int group, int n_groups, int mode, float eps, void* out,
                                 int out_dtype, long long out_stride, int n, cudaStream_t stream) {
    if (n == 0) return BLM_OK;
    BLM_REQUIRE(group > 0 && n_groups > 0 && period > 0 && mode >= 0 && mode <= 3 && (gate != nullptr || mode == 3),
                "gated_group_norm: bad sizes or mode");
    const int threads = n_groups >= 8 ? 256 : 32 * n_groups;
    if (out_dtype == BLM_F32)
        gated_group_norm_kernel<float><<<n, threads, 0, stream>>>(y, y_stride, gate, gate_stride, gate_col0, w, period, group,
                                                                  n_groups, mode, eps, (float*)out, out_stride);
    else if (out_dtype == BLM_BF16)
        gated_group_norm_kernel<__nv_bfloat16><<<n, threads, 0, stream>>>(y, y_stride, gate, gate_stride, gate_col0, w, period,
                                                                          group, n_groups, mode, eps, (__nv_bfloat16*)out, out_stride);
    else
        return blm_fail(BLM_BAD_ARGUMENT, "gated_group_norm: out dtype %d", out_dtype);
    return blm_check_launch("gated_group_norm");
}

// ---------------------------------------------------------------------------------------------
// Selective scan (Mamba).  Per channel c and state n:
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B[n],   y_c = sum_n S[c, n] C[n] + D_c x_c,
//     out_c = scale y_c silu(z_c),   dt_c = softplus(dt_raw_c + dt_bias_c),   A = -exp(A_log)
// x float32 [T, *] (after convolution and silu), B and C columns of low [T, *], z columns of another row.  dt_raw is given
// [T, C], or (dt_w) formed here from the first `rank` columns of low and dt_w [C, rank]: for single tokens, where a product
// of its own would be a launch for a few kilobytes.  A block owns (sequence, kSelThreads / kSelLanes channels); kSelLanes lanes
// share a channel, RN neighbouring states each in registers.  The state is stored as [channel][state].  Three kernels:
//   selective_scan_kernel   portions, bfloat16 results: chunks of kChunk tokens; four warps walk the tokens and eight serve
//                           them (rows through cp.async, what is made of them, results out), a chunk apart, so that the
//                           walk waits for nothing but its own arithmetic; a lane leaves its share of a token's sum in
//                           shared memory, so nothing is shuffled on the way.  The exponentials are exp2 by the special
//                           function unit with A scaled by log2 e: at 16 states a channel 32 of its cycles a token and warp.
//   selective_step_kernel   one token a sequence, bfloat16 results: nothing staged but the latents the step sizes are made of.
//   selective_exact_kernel  the 32-bit path, any portion: state and sums in float64 inside a step.
// ---------------------------------------------------------------------------------------------
constexpr int kSelThreads = 128, kSelLanes = 4, kSelChannels = kSelThreads / kSelLanes;

struct SelArgs {
    const float* x; long long x_stride;
    const float* low; long long low_stride; int b_col0, c_col0;
    const float* dt_raw; long long dt_stride;
    const void* dt_w; int dt_w_bf16, rank;
    const float* dt_bias; const float* A_log; const float* D;
    const float* rates;      // A log2 e = -exp(A_log) log2 e, for the kernels that take exp2 of it
    const float* z; long long z_stride;
    void* out; long long out_stride; float scale;
    int channels, n_states;
};

template <int RN>
__global__ void __launch_bounds__(kSelThreads)
    selective_exact_kernel(SelArgs a, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                          const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride, long long copy_stride,
                          long long state_off) {
    typedef double AT;
    typedef float TO;
    constexpr int NP = RN * kSelLanes, CH = kSelChannels;
    __shared__ __align__(16) float Bs[kChunk][NP], Cs[kChunk][NP];
    __shared__ float dts[kChunk][CH], xs[kChunk][CH], ys[kChunk][CH];
    const int seq = blockIdx.x, c0 = blockIdx.y * CH;
    const ScanSeq sq = scan_seq(seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
    if (sq.n_new <= 0) return;
    const int tid = threadIdx.x, ch = tid / kSelLanes, g = tid % kSelLanes;
    const int c = c0 + ch, n0 = g * RN;
    const bool live = c < a.channels;
    AT s[RN], A[RN];
#pragma unroll
    for (int r = 0; r < RN; ++r) {
        const bool in = live && n0 + r < a.n_states;
        const size_t at = (size_t)c * a.n_states + n0 + r;
        s[r] = in && sq.read ? (AT)sq.read[at] : (AT)0;
        A[r] = in ? -exp((double)a.A_log[at]) : 0.0;
    }
    for (int t0 = 0; t0 < sq.n_new; t0 += kChunk) {
        const int nt = min(kChunk, sq.n_new - t0);
        const size_t row0 = (size_t)(sq.first + t0);
        __syncthreads();
        for (int e = tid; e < nt * NP; e += kSelThreads) {
            const int t = e / NP, n = e % NP;
            const float* low = a.low + (row0 + t) * a.low_stride;
            Bs[t][n] = n < a.n_states ? low[a.b_col0 + n] : 0.f;
            Cs[t][n] = n < a.n_states ? low[a.c_col0 + n] : 0.f;
        }
        for (int e = tid; e < nt * CH; e += kSelThreads) {
            const int t = e / CH, k = e % CH, cc = c0 + k;
            float dt = 0.f, x = 0.f;
            if (cc < a.channels) {
                x = a.x[(row0 + t) * a.x_stride + cc];
                float raw = a.dt_bias[cc];
                if (a.dt_w != nullptr) {
                    const float* low = a.low + (row0 + t) * a.low_stride;
                    float sum = 0.f;
                    if (a.dt_w_bf16) {
                        const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.dt_w) + (size_t)cc * a.rank;
#pragma unroll 8
                        for (int k2 = 0; k2 < a.rank; ++k2) sum = fmaf(__bfloat162float(w[k2]), low[k2], sum);
                    } else {
                        const float* w = reinterpret_cast<const float*>(a.dt_w) + (size_t)cc * a.rank;
#pragma unroll 8
                        for (int k2 = 0; k2 < a.rank; ++k2) sum = fmaf(w[k2], low[k2], sum);
                    }
                    raw += sum;
                } else {
                    raw += a.dt_raw[(row0 + t) * a.dt_stride + cc];
                }
                dt = softplus_r(raw);
            }
            dts[t][k] = dt;
            xs[t][k] = x;
        }
        __syncthreads();
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const AT dt = (AT)dts[t][ch], dx = dt * (AT)xs[t][ch];
            AT part[2] = {0, 0};
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                s[r] = exp(dt * A[r]) * s[r] + dx * (AT)Bs[t][n0 + r];
                part[r & 1] += s[r] * (AT)Cs[t][n0 + r];
            }
            const AT y = group_sum<kSelLanes>(part[0] + part[1]);
            if (g == 0) ys[t][ch] = (float)(y + (AT)(live ? a.D[c] : 0.f) * (AT)xs[t][ch]);
        }
        __syncthreads();
        for (int e = tid; e < nt * CH; e += kSelThreads) {
            const int t = e / CH, k = e % CH, cc = c0 + k;
            if (cc < a.channels) {
                const float z = a.z[(row0 + t) * a.z_stride + cc];
                reinterpret_cast<TO*>(a.out)[(row0 + t) * a.out_stride + cc] = from_f32<TO>(a.scale * ys[t][k] * silu_f(z));
            }
        }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < RN; ++r)
            if (n0 + r < a.n_states) sq.write[(size_t)c * a.n_states + n0 + r] = (float)s[r];
    }
}

__device__ __forceinline__ float ex2_approx(float x) {       // x <= 0 here: no overflow, and what underflows is zero
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
template <int BYTES>
__device__ __forceinline__ void copy_async(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "n"(BYTES) : "memory");
}

// states n0 .. n0 + RN of one row of B or C (shared memory): the widest loads RN allows
template <int RN>
__device__ __forceinline__ void load_states(float (&v)[RN], const float* p) {
    if (RN % 4 == 0) {
#pragma unroll
        for (int r = 0; r < RN; r += 4) {
            const float4 q = *reinterpret_cast<const float4*>(p + r);
            v[r] = q.x; v[r + 1] = q.y; v[r + 2] = q.z; v[r + 3] = q.w;
        }
    } else {
#pragma unroll
        for (int r = 0; r < RN; r += 2) {
            const float2 q = *reinterpret_cast<const float2*>(p + r);
            v[r] = q.x; v[r + 1] = q.y;
        }
    }
}

// Threads that serve the four scanning warps of a block.  Measured, one prompt of 2,048 tokens and eight of 512: 4,096
// channels of 16 states with 128 threads 156 and 194 us, with 256 112 and 163; 8,192 channels 205 and 365, 179 and 314;
// 4,096 channels of 64 states 455 and 818, 375 and 674.
#ifndef BLM_SEL_SERVE
#define BLM_SEL_SERVE 256
#endif
constexpr int kSelServe = BLM_SEL_SERVE, kSelBlock = kSelThreads + kSelServe;      // the portions' kernel: four warps scan, the others serve them

template <int RN>
struct SelSmem {
    static constexpr int NP = RN * kSelLanes, CH = kSelChannels;
    float B[3][kChunk][NP], C[3][kChunk][NP];                                    // on their way, landed, read by the scan
    float x[2][kChunk][CH], dt[2][kChunk][CH], z[2][kChunk][CH];                 // raw rows: on their way, landed
    float2 made[2][kChunk][CH];                                                  // (dt, dt x)
    float2 after[2][kChunk][CH];                                                 // (D x, scale silu(z)): what the results meet on their way out
    float4 y[2][kChunk][CH];                                                     // a channel's four lanes' sums
};

// Chunk c of the sequence passes through the block in four turns, a barrier after each:
//   turn c - 1  the serving warps ask for its rows;      turn c      they make (dt, dt x) and (D x, scale silu(z)) of them;
//   turn c + 1  the scanning warps walk its tokens;      turn c + 2  the serving warps write its results out.
template <int RN>
__global__ void __launch_bounds__(kSelBlock)
    selective_scan_kernel(SelArgs a, int rows16, int low16, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                          const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride, long long copy_stride,
                          long long state_off) {
    // rows16, low16: the rows of x, dt and z (of low) can be copied 16 bytes at a time
    constexpr int NP = RN * kSelLanes, CH = kSelChannels;
    extern __shared__ __align__(16) unsigned char sel_raw[];
    SelSmem<RN>& sm = *reinterpret_cast<SelSmem<RN>*>(sel_raw);
    const int seq = blockIdx.x, c0 = blockIdx.y * CH;
    const ScanSeq sq = scan_seq(seq, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
    if (sq.n_new <= 0) return;
    // places no copy writes stay zero: states beyond n_states, channels beyond the last, rows beyond the last token
    for (int e = threadIdx.x; e < (int)(sizeof(SelSmem<RN>) / sizeof(float)); e += kSelBlock) reinterpret_cast<float*>(&sm)[e] = 0.f;
    __syncthreads();
    const int n_chunks = (sq.n_new + kChunk - 1) / kChunk;
    auto turn_over = [] { asm volatile("bar.sync 2, %0;\n" ::"n"(kSelBlock) : "memory"); };     // both halves of the block, each from its own loop
    if (threadIdx.x < kSelThreads) {
        // ---------------- the scan: a channel's state in four lanes ----------------
        const int ch = threadIdx.x / kSelLanes, g = threadIdx.x % kSelLanes, c = c0 + ch, n0 = g * RN;
        const bool live = c < a.channels;
        float s[RN], A[RN];
#pragma unroll
        for (int r = 0; r < RN; ++r) {
            const bool in = live && n0 + r < a.n_states;
            const size_t at = (size_t)c * a.n_states + n0 + r;
            s[r] = in && sq.read ? sq.read[at] : 0.f;
            A[r] = in ? a.rates[at] : 0.f;
        }
        for (int turn = 0; turn < n_chunks + 2; ++turn) {
            const int k = turn - 1;                     // the chunk this turn walks
            if (k >= 0 && k < n_chunks) {
                // (rows beyond the last token, up to a multiple of four, meet a step size of zero: nothing changes)
                const int nt = min(kChunk, sq.n_new - k * kChunk);
                const float2* made = &sm.made[k & 1][0][ch];
                const float* Bs = &sm.B[k % 3][0][n0];
                const float* Cs = &sm.C[k % 3][0][n0];
                float* y = reinterpret_cast<float*>(&sm.y[k & 1][0][ch]) + g;
                constexpr int U = RN <= 8 ? 4 : 1;      // tokens whose operands are fetched together, ahead of the ones worked on
                float2 d[U];
                float b[U][RN], cc[U][RN];
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    d[u] = made[u * CH];
                    load_states<RN>(b[u], Bs + u * NP);
                    load_states<RN>(cc[u], Cs + u * NP);
                }
                for (int t = 0; t < nt; t += U) {
                    float2 dn[U];
                    float bn[U][RN], cn[U][RN];
                    const int tn = min(t + U, kChunk - U);      // (the last turn's fetch is not used)
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        dn[u] = made[(tn + u) * CH];
                        load_states<RN>(bn[u], Bs + (tn + u) * NP);
                        load_states<RN>(cn[u], Cs + (tn + u) * NP);
                    }
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        float p0 = 0.f, p1 = 0.f;
#pragma unroll
                        for (int r = 0; r < RN; ++r) {
                            s[r] = fmaf(ex2_approx(d[u].x * A[r]), s[r], d[u].y * b[u][r]);
                            if (r & 1) p1 = fmaf(s[r], cc[u][r], p1);
                            else p0 = fmaf(s[r], cc[u][r], p0);
                        }
                        y[(size_t)(t + u) * CH * kSelLanes] = p0 + p1;
                    }
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        d[u] = dn[u];
#pragma unroll
                        for (int r = 0; r < RN; ++r) {
                            b[u][r] = bn[u][r];
                            cc[u][r] = cn[u][r];
                        }
                    }
                }
            }
            turn_over();
        }
        if (live) {
#pragma unroll
            for (int r = 0; r < RN; ++r)
                if (n0 + r < a.n_states) sq.write[(size_t)c * a.n_states + n0 + r] = s[r];
        }
        return;
    }
    // ---------------- the serving warps: a thread always has the same column of the rows ----------------
    const int tid = threadIdx.x - kSelThreads, col = tid % CH, row_of = tid / CH;
    const bool mine = c0 + col < a.channels;
    const float bias = mine ? a.dt_bias[c0 + col] : 0.f, skip = mine ? a.D[c0 + col] : 0.f;
    auto fetch = [&](int k) {                           // the rows of chunk k
        const int t0 = k * kChunk, nt = min(kChunk, sq.n_new - t0), buf = k & 1, low_buf = k % 3;
        const size_t row0 = (size_t)(sq.first + t0);
        if (rows16) {
            constexpr int V = CH / 4;
            for (int e = tid; e < nt * V; e += kSelServe) {
                const int t = e / V, kk = (e % V) * 4;
                if (c0 + kk < a.channels) {             // channels is a multiple of 4
                    copy_async<16>(&sm.x[buf][t][kk], a.x + (row0 + t) * a.x_stride + c0 + kk);
                    copy_async<16>(&sm.dt[buf][t][kk], a.dt_raw + (row0 + t) * a.dt_stride + c0 + kk);
                    copy_async<16>(&sm.z[buf][t][kk], a.z + (row0 + t) * a.z_stride + c0 + kk);
                }
            }
        } else {
            for (int t = row_of; t < nt; t += kSelServe / CH)
                if (mine) {
                    copy_async<4>(&sm.x[buf][t][col], a.x + (row0 + t) * a.x_stride + c0 + col);
                    copy_async<4>(&sm.dt[buf][t][col], a.dt_raw + (row0 + t) * a.dt_stride + c0 + col);
                    copy_async<4>(&sm.z[buf][t][col], a.z + (row0 + t) * a.z_stride + c0 + col);
                }
        }
        if (low16) {
            constexpr int V = NP / 4;
            for (int e = tid; e < nt * V; e += kSelServe) {
                const int t = e / V, n = (e % V) * 4;
                if (n < a.n_states) {                   // n_states is a multiple of 4
                    const float* low = a.low + (row0 + t) * a.low_stride;
                    copy_async<16>(&sm.B[low_buf][t][n], low + a.b_col0 + n);
                    copy_async<16>(&sm.C[low_buf][t][n], low + a.c_col0 + n);
                }
            }
        } else {
            for (int e = tid; e < nt * NP; e += kSelServe) {
                const int t = e / NP, n = e % NP;
                if (n < a.n_states) {
                    const float* low = a.low + (row0 + t) * a.low_stride;
                    copy_async<4>(&sm.B[low_buf][t][n], low + a.b_col0 + n);
                    copy_async<4>(&sm.C[low_buf][t][n], low + a.c_col0 + n);
                }
            }
        }
    };
    fetch(0);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
    constexpr int kPasses = kChunk * CH / kSelServe;
    static_assert(kSelServe % CH == 0 && kChunk * CH % kSelServe == 0, "every serving thread has one column and as many rows");
    for (int turn = 0; turn < n_chunks + 2; ++turn) {
        if (turn >= 2 && mine) {                        // chunk turn - 2 goes out
            const int k = turn - 2, nt = min(kChunk, sq.n_new - k * kChunk);
            __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(sq.first + k * kChunk) * a.out_stride + c0 + col;
#pragma unroll
            for (int i = 0; i < kPasses; ++i) {
                const int t = row_of + i * (kSelServe / CH);
                const float4 y = sm.y[k & 1][t][col];
                const float2 f = sm.after[k & 1][t][col];
                if (t < nt) out[(size_t)t * a.out_stride] = __float2bfloat16_rn(((y.x + y.y) + (y.z + y.w) + f.x) * f.y);
            }
        }
        if (turn < n_chunks) {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
            // every serving thread's copies have landed when all of them have waited
            asm volatile("bar.sync 1, %0;\n" ::"n"(kSelServe) : "memory");
            const int k = turn, nt = min(kChunk, sq.n_new - k * kChunk), buf = k & 1;
            if (turn + 1 < n_chunks) fetch(turn + 1);
            asm volatile("cp.async.commit_group;\n" ::: "memory");
#pragma unroll
            for (int i = 0; i < kPasses; ++i) {
                const int t = row_of + i * (kSelServe / CH);
                const float x = sm.x[buf][t][col], z = sm.z[buf][t][col];
                const float dt = t < nt ? softplus_r(sm.dt[buf][t][col] + bias) : 0.f;
                sm.made[buf][t][col] = make_float2(dt, t < nt ? dt * x : 0.f);
                // (the chunk two before this one has gone out: the same thread read its place above)
                sm.after[buf][t][col] = make_float2(skip * x, a.scale * __fdividef(z, 1.0f + __expf(-z)));
            }
        }
        turn_over();
    }
}

// How many sequences a block of the single tokens' kernel takes (a channel's constants are read once for them).  Measured in a
// captured graph, 64 sequences, 4,096 and 8,192 channels of 16 states: one sequence 12.4 and 23.0 us, two 12.1 and 21.9, four
// 13.8 and 25.3; with the step sizes formed inside, 8 sequences: 4.6 and 10.3 us, 5.1 and 8.5, 6.4 and 10.0.
#ifndef BLM_STEP_SEQS
#define BLM_STEP_SEQS 2
#endif
constexpr int kStepSeqs = BLM_STEP_SEQS;

template <int RN>
__global__ void __launch_bounds__(kSelThreads)
    selective_step_kernel(SelArgs a, int n_seqs, int vec8, int vec4, const int* __restrict__ cu_seqlens, const int* __restrict__ slot_of_seq,
                          const int* __restrict__ start_pos, float* __restrict__ state, long long slot_stride, long long copy_stride,
                          long long state_off) {
    // vec8: rows of dt_w are bfloat16 and can be read 16 bytes at a time; vec4: so can a thread's states, rates, B and C
    extern __shared__ __align__(16) unsigned char sel_raw[];
    float* lat = reinterpret_cast<float*>(sel_raw);      // [kStepSeqs][rank]
    const int seq0 = blockIdx.x * kStepSeqs, many = min(kStepSeqs, n_seqs - seq0);
    const int tid = threadIdx.x, ch = tid / kSelLanes, g = tid % kSelLanes, n0 = g * RN;
    const int c = min(blockIdx.y * kSelChannels + ch, a.channels - 1);      // (lanes beyond the last channel work on it too and write nothing)
    const bool live = blockIdx.y * kSelChannels + ch < a.channels;
    auto get = [&](float (&v)[RN], const float* p) {     // this thread's states' numbers from a row of n_states
        if (vec4 && RN % 4 == 0) {
#pragma unroll
            for (int r = 0; r < RN; r += 4) {
                const float4 q = *reinterpret_cast<const float4*>(p + n0 + r);
                v[r] = q.x; v[r + 1] = q.y; v[r + 2] = q.z; v[r + 3] = q.w;
            }
        } else {
#pragma unroll
            for (int r = 0; r < RN; ++r) v[r] = n0 + r < a.n_states ? p[n0 + r] : 0.f;
        }
    };
    float A[RN], s[kStepSeqs][RN], x[kStepSeqs], z[kStepSeqs], raw[kStepSeqs];
    float* write[kStepSeqs];
    get(A, a.rates + (size_t)c * a.n_states);
    if (a.dt_w != nullptr) {
        for (int k = tid; k < many * a.rank; k += kSelThreads) {
            const int q = k / a.rank, row = cu_seqlens[seq0 + q];
            lat[k] = cu_seqlens[seq0 + q + 1] > row ? a.low[(size_t)row * a.low_stride + k % a.rank] : 0.f;
        }
        __syncthreads();
    }
#pragma unroll
    for (int q = 0; q < kStepSeqs; ++q) {
        write[q] = nullptr;
        raw[q] = x[q] = z[q] = 0.f;
        if (q < many) {
            const ScanSeq sq = scan_seq(seq0 + q, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
            if (sq.n_new > 0) {
                const size_t row = (size_t)sq.first;
                write[q] = sq.write + (size_t)c * a.n_states;
                if (sq.read) get(s[q], sq.read + (size_t)c * a.n_states);
                else
#pragma unroll
                    for (int r = 0; r < RN; ++r) s[q][r] = 0.f;
                x[q] = a.x[row * a.x_stride + c];
                z[q] = a.z[row * a.z_stride + c];
                if (a.dt_w == nullptr) raw[q] = a.dt_raw[row * a.dt_stride + c];
            }
        }
    }
    if (a.dt_w != nullptr) {
        if (vec8) {
            const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.dt_w) + (size_t)c * a.rank;
#pragma unroll 4
            for (int k = g * 8; k < a.rank; k += 8 * kSelLanes) {
                const uint4 v = *reinterpret_cast<const uint4*>(w + k);
                const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 f = __bfloat1622float2(p[e]);
#pragma unroll
                    for (int q = 0; q < kStepSeqs; ++q)
                        if (q < many) raw[q] = fmaf(f.x, lat[q * a.rank + k + 2 * e], fmaf(f.y, lat[q * a.rank + k + 2 * e + 1], raw[q]));
                }
            }
        } else {
            for (int k = g; k < a.rank; k += kSelLanes) {
                const float w = a.dt_w_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.dt_w)[(size_t)c * a.rank + k])
                                            : reinterpret_cast<const float*>(a.dt_w)[(size_t)c * a.rank + k];
#pragma unroll
                for (int q = 0; q < kStepSeqs; ++q)
                    if (q < many) raw[q] = fmaf(w, lat[q * a.rank + k], raw[q]);
            }
        }
#pragma unroll
        for (int q = 0; q < kStepSeqs; ++q) raw[q] = group_sum<kSelLanes>(raw[q]);
    }
    const float bias = a.dt_bias[c], skip = a.D[c];
#pragma unroll
    for (int q = 0; q < kStepSeqs; ++q) {
        if (q >= many || write[q] == nullptr) continue;      // (the same for the whole block)
        const size_t row = (size_t)cu_seqlens[seq0 + q];
        const float* low = a.low + row * a.low_stride;
        float b[RN], cc[RN];
        get(b, low + a.b_col0);
        get(cc, low + a.c_col0);
        const float dt = softplus_r(raw[q] + bias), dx = dt * x[q];
        float y = 0.f;
#pragma unroll
        for (int r = 0; r < RN; ++r) {
            s[q][r] = fmaf(ex2_approx(A[r] * dt), s[q][r], dx * b[r]);
            y = fmaf(s[q][r], cc[r], y);
        }
        y = group_sum<kSelLanes>(y);
        if (!live) continue;
        if (vec4 && RN % 4 == 0) {
#pragma unroll
            for (int r = 0; r < RN; r += 4) *reinterpret_cast<float4*>(write[q] + n0 + r) = make_float4(s[q][r], s[q][r + 1], s[q][r + 2], s[q][r + 3]);
        } else {
#pragma unroll
            for (int r = 0; r < RN; ++r)
                if (n0 + r < a.n_states) write[q][n0 + r] = s[q][r];
        }
        if (g == 0) reinterpret_cast<__nv_bfloat16*>(a.out)[row * a.out_stride + c] = __float2bfloat16_rn(a.scale * (y + skip * x[q]) * silu_f(z[q]));
    }
}

static bool aligned16(const void* p, long long stride) { return ((size_t)p & 15) == 0 && stride % 4 == 0; }

template <int RN>
static int launch_selective(const SelArgs& a, int exact, int single, int n_seqs, const int* cu_seqlens, const int* slot_of_seq, const int* start_pos,
                            float* state, long long slot_stride, long long copy_stride, long long state_off, cudaStream_t stream) {
    const dim3 grid(n_seqs, (a.channels + kSelChannels - 1) / kSelChannels);
    if (exact) {
        selective_exact_kernel<RN><<<grid, kSelThreads, 0, stream>>>(a, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride, state_off);
        return blm_check_launch("selective_scan (exact)");
    }
    if (single) {
        const int vec8 = a.dt_w != nullptr && a.dt_w_bf16 && a.rank % 8 == 0 && ((size_t)a.dt_w & 15) == 0;
        const size_t smem = a.dt_w != nullptr ? (size_t)kStepSeqs * a.rank * sizeof(float) : 0;
        BLM_REQUIRE(smem <= 48 * 1024, "selective_scan: step sizes made of %d numbers", a.rank);
        const int vec4 = a.n_states == RN * kSelLanes && aligned16(a.low, a.low_stride) && a.b_col0 % 4 == 0 && a.c_col0 % 4 == 0 &&
                         aligned16(state, slot_stride) && copy_stride % 4 == 0 && state_off % 4 == 0 && ((size_t)a.rates & 15) == 0;
        const dim3 tiles((n_seqs + kStepSeqs - 1) / kStepSeqs, grid.y);
        selective_step_kernel<RN><<<tiles, kSelThreads, smem, stream>>>(a, n_seqs, vec8, vec4, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, copy_stride,
                                                                       state_off);
        return blm_check_launch("selective_scan (single tokens)");
    }
    BLM_REQUIRE(a.dt_raw != nullptr, "selective_scan: portions bring their step sizes");
    const int rows16 = a.channels % 4 == 0 && aligned16(a.x, a.x_stride) && aligned16(a.dt_raw, a.dt_stride) && aligned16(a.z, a.z_stride);
    const int low16 = a.n_states % 4 == 0 && aligned16(a.low, a.low_stride) && a.b_col0 % 4 == 0 && a.c_col0 % 4 == 0;
    const int rc = allow_smem(selective_scan_kernel<RN>, sizeof(SelSmem<RN>), "selective_scan");
    if (rc != BLM_OK) return rc;
    selective_scan_kernel<RN><<<grid, kSelBlock, sizeof(SelSmem<RN>), stream>>>(a, rows16, low16, cu_seqlens, slot_of_seq, start_pos, state,
                                                                                  slot_stride, copy_stride, state_off);
    return blm_check_launch("selective_scan");
}

BLM_API int blm_selective_scan(const float* x, long long x_stride, const float* low, long long low_stride, int b_col0, int c_col0,
                               const float* dt_raw, long long dt_stride, const void* dt_w, int dt_w_dtype, int rank, const float* dt_bias,
                               const float* A_log, const float* rates, const float* D, const float* z, long long z_stride, void* out, int out_dtype,
                               long long out_stride, float scale, int channels, int n_states, const int* cu_seqlens, const int* slot_of_seq,
                               const int* start_pos, int n_seqs, int single_tokens, float* state, long long slot_stride,
                               long long copy_stride, long long state_off, cudaStream_t stream) {
    // dt_raw [T, dt_stride], or null and dt_w [channels, rank] (the step sizes' projection of low's first columns; single tokens
    // and the 32-bit path only).  single_tokens: every sequence brings one token.
    // out float32: the 32-bit path (sums in float64).  Rows of no sequence are left as they are.
    if (n_seqs == 0) return BLM_OK;
    BLM_REQUIRE(channels > 0 && n_states > 0 && n_seqs > 0, "selective_scan: bad sizes");
    BLM_REQUIRE((dt_raw == nullptr) != (dt_w == nullptr) && (dt_w == nullptr || rank > 0), "selective_scan: give step sizes or their projection");
    BLM_REQUIRE((channels + kSelChannels - 1) / kSelChannels <= 65535, "selective_scan: %d channels", channels);
    SelArgs a;
    a.x = x; a.x_stride = x_stride; a.low = low; a.low_stride = low_stride; a.b_col0 = b_col0; a.c_col0 = c_col0;
    a.dt_raw = dt_raw; a.dt_stride = dt_stride; a.dt_w = dt_w; a.dt_w_bf16 = dt_w_dtype == BLM_BF16; a.rank = rank;
    a.dt_bias = dt_bias; a.A_log = A_log; a.rates = rates; a.D = D; a.z = z; a.z_stride = z_stride;
    a.out = out; a.out_stride = out_stride; a.scale = scale; a.channels = channels; a.n_states = n_states;
    BLM_REQUIRE(out_dtype == BLM_F32 || out_dtype == BLM_BF16, "selective_scan: out dtype %d", out_dtype);
    BLM_REQUIRE(out_dtype == BLM_F32 || rates != nullptr, "selective_scan: no rates");
#define BLM_SEL(RN)                                                                                                                      \
    if (n_states <= RN * kSelLanes)                                                                                                      \
        return launch_selective<RN>(a, out_dtype == BLM_F32, single_tokens, n_seqs, cu_seqlens, slot_of_seq, start_pos, state, slot_stride, \
                                    copy_stride, state_off, stream);
    BLM_SEL(2) BLM_SEL(4) BLM_SEL(6) BLM_SEL(8) BLM_SEL(16) BLM_SEL(32)
#undef BLM_SEL
    return blm_fail(BLM_BAD_ARGUMENT, "selective_scan: %d states a channel; this kernel takes up to %d", n_states, 32 * kSelLanes);
}

// out[n, d] = src[n, col0 + d] in out's type: some columns of a wider fp32 row as a product's operand
template <typename TO>
__global__ void take_cols_kernel(const float* __restrict__ src, long long stride, int col0, TO* __restrict__ out, int width, int total) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) out[i] = from_f32<TO>(src[(size_t)(i / width) * stride + col0 + i % width]);
}

BLM_API int blm_take_cols(const float* src, long long stride, int col0, void* out, int out_dtype, int n_rows, int width, cudaStream_t stream) {
    if (n_rows == 0) return BLM_OK;
    BLM_REQUIRE(width > 0 && col0 >= 0 && (long long)n_rows * width < (1ll << 31), "take_cols: bad sizes");
    const int total = n_rows * width;
    if (out_dtype == BLM_F32) take_cols_kernel<float><<<(total + 255) / 256, 256, 0, stream>>>(src, stride, col0, (float*)out, width, total);
    else if (out_dtype == BLM_BF16)
        take_cols_kernel<__nv_bfloat16><<<(total + 255) / 256, 256, 0, stream>>>(src, stride, col0, (__nv_bfloat16*)out, width, total);
    else return blm_fail(BLM_BAD_ARGUMENT, "take_cols: out dtype %d", out_dtype);
    return blm_check_launch("take_cols");
}
