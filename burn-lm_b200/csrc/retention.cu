// Retention over the packed tokens of a step.  Per head, with a decay a of its own,
//   S_t = a S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out = o / sqrt(mean(o^2) + eps) * silu(g)      (S: dk x dv)
// with q and k turned by their position and k scaled first.  A row of the projection holds [q | k | v | g], float32.
//
// What a sequence carries is S of every head, float32 [head][dk][dv], twice (see recurrent.cu): a step that starts at position p
// reads copy (p & 1) and writes copy ((p + n) & 1) for its n new tokens; one that starts at position 0 reads zeros.
//
// Three forms, which share that state:
//   the scan: tokens in order, S and the sums over its rows in float64 inside a step; it serves the 32-bit path and head sizes
//     the others do not take, and leaves o for a kernel that norms and gates it;
//   the single token: a block a (token, head) reads S once, writes it once, and finishes the row (norm, gate);
//   chunks of 64 tokens: (1) what every chunk adds to S by itself, sum_t a^(last - t) k_t v_t^T; (2) S in front of every chunk,
//     from these in order; (3) a chunk's outputs, o_t = a^(t + 1) S^T q_t + sum_(s <= t) a^(t - s) (q_t . k_s) v_s, normed and
//     gated.  All chunks of a sequence run side by side in (1) and (3).  Products on the tensor cores with float32 sums, bfloat16
//     operands; operands that carry a decay or are S itself go in as two bfloat16 numbers, high part and rest (16 bits).
#include "common.cuh"

BLM_API const char* blm_retention_last_error() { return g_blm_error; }

constexpr int kC = 64;             // tokens of a chunk

// The step's projection and how its queries and keys turn: lanes (i, i + rot / 2) of the first `rot` by position * freq[i].
struct RetIn {
    const float* proj;
    long long stride;
    int heads, dk, dv;
    float k_scale;
    const double* freq;
    int rot;
    const float2* table;           // [table_len][rot / 2] (cosine, sine), or null
    int table_len;
    const float* powers;           // [heads][kC + 1]: the decay to the power m
};
struct RetSeq {
    const int* cu_seqlens;
    const int* slot_of_seq;
    const int* start_pos;
    int n_seqs;
    float* state;
    long long slot_stride, copy_stride, offset;
    __device__ __forceinline__ float* copy(int seq, int pos) const {
        return state + (size_t)slot_of_seq[seq] * slot_stride + (size_t)(pos & 1) * copy_stride + offset;
    }
};

// (a call of its own: inlined, it would cost every kernel its registers)
__device__ __noinline__ float2 ret_angle(double angle) {
    double sn, cs;
    sincos(angle, &sn, &cs);
    return make_float2((float)cs, (float)sn);
}
__device__ __forceinline__ float2 ret_turn(const RetIn& in, int pos, int i) {
    if (pos < in.table_len) return in.table[(size_t)pos * (in.rot >> 1) + i];
    return ret_angle((double)pos * in.freq[i]);
}
// (cosine, sine) of pairs i .. i + 3, i a multiple of 4
__device__ __forceinline__ void ret_turn4(const RetIn& in, int pos, int i, float4& lo, float4& hi) {
    if (pos < in.table_len) {
        const float4* t = reinterpret_cast<const float4*>(in.table + (size_t)pos * (in.rot >> 1) + i);
        lo = __ldg(t);
        hi = __ldg(t + 1);
        return;
    }
    float2 a = ret_angle((double)pos * in.freq[i]), b = ret_angle((double)pos * in.freq[i + 1]);
    lo = make_float4(a.x, a.y, b.x, b.y);
    a = ret_angle((double)pos * in.freq[i + 2]);
    b = ret_angle((double)pos * in.freq[i + 3]);
    hi = make_float4(a.x, a.y, b.x, b.y);
}
// lanes d .. d + 3 of the first half (a) and of the second (b), turned together
__device__ __forceinline__ void ret_turn_pairs(float4& a, float4& b, const float4& lo, const float4& hi) {
    const float4 u = a, v = b;
    a = make_float4(u.x * lo.x - v.x * lo.y, u.y * lo.z - v.y * lo.w, u.z * hi.x - v.z * hi.y, u.w * hi.z - v.w * hi.w);
    b = make_float4(v.x * lo.x + u.x * lo.y, v.y * lo.z + u.y * lo.w, v.z * hi.x + u.z * hi.y, v.w * hi.z + u.w * hi.w);
}
// lane d of a head's query or key (`src`: the head's first lane), turned
__device__ __forceinline__ float ret_lane(const RetIn& in, const float* src, int pos, int d) {
    if (d >= in.rot) return src[d];
    const int half = in.rot >> 1;
    if (d < half) {
        const float2 t = ret_turn(in, pos, d);
        return src[d] * t.x - src[d + half] * t.y;
    }
    const float2 t = ret_turn(in, pos, d - half);
    return src[d] * t.x + src[d - half] * t.y;
}
// lanes d .. d + 3, d a multiple of 4; `vec`: rows and halves allow 16-byte loads
__device__ __forceinline__ void ret_lanes4(const RetIn& in, const float* src, int pos, int d, bool vec, float (&v)[4]) {
    if (!vec) {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = d + e < in.dk ? ret_lane(in, src, pos, d + e) : 0.f;
        return;
    }
    const float4 a = *reinterpret_cast<const float4*>(src + d);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    if (d >= in.rot) return;
    const int half = in.rot >> 1;
    const bool first = d < half;
    const float4 b = *reinterpret_cast<const float4*>(src + (first ? d + half : d - half));
    const float o[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 t = ret_turn(in, pos, (first ? d : d - half) + e);
        v[e] = first ? v[e] * t.x - o[e] * t.y : v[e] * t.x + o[e] * t.y;
    }
}
static bool ret_vec(const RetIn& in) {
    return in.dk % 4 == 0 && in.dv % 4 == 0 && in.rot % 8 == 0 && in.stride % 4 == 0 && ((size_t)in.proj & 15) == 0;
}
__device__ __forceinline__ float ret_silu(float z) { return z / (1.0f + expf(-z)); }

// ---------------------------------------------------------------------------------------------
// the scan: a block per (32 value lanes, head, sequence); thread (column, row group) keeps rows rg, rg + 8, ... of its column
// ---------------------------------------------------------------------------------------------
constexpr int kScanTokens = 32;    // tokens staged in shared memory at a time

template <int RN>
__global__ void __launch_bounds__(256) retention_scan_kernel(RetIn in, RetSeq sq, float* __restrict__ o, long long o_stride) {
    extern __shared__ float sm[];
    float* qs = sm;                                    // [kScanTokens][dk]
    float* ks = qs + kScanTokens * in.dk;
    float* vs = ks + kScanTokens * in.dk;              // [kScanTokens][32]
    const int head = blockIdx.y, seq = blockIdx.z, col0 = blockIdx.x * 32;
    const int rg = threadIdx.x & 7, col = threadIdx.x >> 3, dk = in.dk, dv = in.dv;
    const int t0 = sq.cu_seqlens[seq], len = sq.cu_seqlens[seq + 1] - t0;
    if (len <= 0) return;
    const int start = sq.start_pos[seq];
    const bool mine = col0 + col < dv;
    const float* from = sq.copy(seq, start) + (size_t)head * dk * dv + col0 + col;
    double S[RN];
#pragma unroll
    for (int r = 0; r < RN; ++r) {
        const int row = rg + 8 * r;
        S[r] = mine && row < dk && start > 0 ? (double)from[(size_t)row * dv] : 0.0;
    }
    const double decay = (double)in.powers[(size_t)head * (kC + 1) + 1];
    const int hq = head * dk, hk = in.heads * dk + hq, hv = 2 * in.heads * dk + head * dv + col0;
    for (int c0 = 0; c0 < len; c0 += kScanTokens) {
        const int m = min(kScanTokens, len - c0);
        __syncthreads();
        for (int idx = threadIdx.x; idx < m * dk; idx += 256) {
            const int t = idx / dk, d = idx % dk, pos = start + c0 + t;
            const float* row = in.proj + (size_t)(t0 + c0 + t) * in.stride;
            qs[idx] = ret_lane(in, row + hq, pos, d);
            ks[idx] = ret_lane(in, row + hk, pos, d) * in.k_scale;
        }
        for (int idx = threadIdx.x; idx < m * 32; idx += 256) {
            const int t = idx >> 5, c = idx & 31;
            vs[idx] = col0 + c < dv ? in.proj[(size_t)(t0 + c0 + t) * in.stride + hv + c] : 0.f;
        }
        __syncthreads();
        for (int t = 0; t < m; ++t) {
            const double v = (double)vs[t * 32 + col];
            double acc = 0.0;
#pragma unroll
            for (int r = 0; r < RN; ++r) {
                const int row = rg + 8 * r;
                if (row < dk) {
                    S[r] = decay * S[r] + (double)ks[t * dk + row] * v;
                    acc += S[r] * (double)qs[t * dk + row];
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (rg == 0 && mine) o[(size_t)(t0 + c0 + t) * o_stride + (size_t)head * dv + col0 + col] = (float)acc;
        }
    }
    float* to = sq.copy(seq, start + len) + (size_t)head * dk * dv + col0 + col;
#pragma unroll
    for (int r = 0; r < RN; ++r) {
        const int row = rg + 8 * r;
        if (mine && row < dk) to[(size_t)row * dv] = (float)S[r];
    }
}

// ---------------------------------------------------------------------------------------------
// the single token: a block per (head, token).  Thread (row group, column group) takes N value lanes of rows rg, rg + n_rg, ...
// ---------------------------------------------------------------------------------------------
constexpr int kStepThreads = 256;

// kAhead: rows a thread asks for before it works on the first
template <typename TO, int N, int kAhead>
__global__ void __launch_bounds__(kStepThreads, kAhead > 4 ? 3 : 4) retention_step_kernel(RetIn in, RetSeq sq, const int* __restrict__ token_seq,
                                                                      const int* __restrict__ token_pos, float eps, TO* __restrict__ out,
                                                                      long long out_stride, int vec) {
    extern __shared__ __align__(16) float sm[];
    const int dk = in.dk, dv = in.dv, head = blockIdx.x, tid = threadIdx.x;
    float* qs = sm;                                    // [dk]
    float* ks = qs + ((dk + 3) & ~3);
    float* red = ks + ((dk + 3) & ~3);                 // [36], then [n_rg][dv] partial sums
    float* part = red + 36;
    const size_t n = blockIdx.y;
    TO* orow = out + n * out_stride + (size_t)head * dv;
    const int seq = token_seq[n];
    if (seq < 0) {                                     // a row of no sequence
        for (int d = tid; d < dv; d += kStepThreads) orow[d] = from_f32<TO>(0.f);
        return;
    }
    const int pos = token_pos[n], groups = dv / N, n_rg = kStepThreads / groups;
    const int cg = tid % groups, rg = tid / groups, c = cg * N;
    const bool works = rg < n_rg;
    const float* from = sq.copy(seq, pos) + (size_t)head * dk * dv + c;
    float* to = sq.copy(seq, pos + 1) + (size_t)head * dk * dv + c;
    float S[kAhead][N];
    auto fetch = [&](int row0) {
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int row = row0 + a * n_rg;
            if (works && row < dk && pos > 0) {
                if (N == 4) {
                    const float4 v = *reinterpret_cast<const float4*>(from + (size_t)row * dv);
                    S[a][0] = v.x; S[a][1 % N] = v.y; S[a][2 % N] = v.z; S[a][3 % N] = v.w;
                } else {
                    S[a][0] = from[(size_t)row * dv];
                }
            } else {
#pragma unroll
                for (int e = 0; e < N; ++e) S[a][e] = 0.f;
            }
        }
    };
    fetch(rg);                                         // the state is on its way while the token's row is prepared
    const float* row_p = in.proj + n * in.stride;
    const int quads = (dk + 3) / 4;
    for (int i = tid; i < 2 * quads; i += kStepThreads) {
        const bool is_k = i >= quads;
        const int d = (is_k ? i - quads : i) * 4;
        float v[4];
        ret_lanes4(in, row_p + (is_k ? in.heads * dk : 0) + head * dk, pos, d, vec, v);
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (d + e < dk) (is_k ? ks : qs)[d + e] = is_k ? v[e] * in.k_scale : v[e];
    }
    const float decay = in.powers[(size_t)head * (kC + 1) + 1];
    float v[N], acc[N];
#pragma unroll
    for (int e = 0; e < N; ++e) {
        v[e] = works ? row_p[2 * in.heads * dk + head * dv + c + e] : 0.f;
        acc[e] = 0.f;
    }
    __syncthreads();
    for (int row0 = rg; row0 < dk && works; row0 += kAhead * n_rg) {
        if (row0 != rg) fetch(row0);
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int row = row0 + a * n_rg;
            if (row >= dk) break;
            const float kk = ks[row], qq = qs[row];
#pragma unroll
            for (int e = 0; e < N; ++e) {
                S[a][e] = fmaf(decay, S[a][e], kk * v[e]);
                acc[e] = fmaf(qq, S[a][e], acc[e]);
            }
            if (N == 4) *reinterpret_cast<float4*>(to + (size_t)row * dv) = make_float4(S[a][0], S[a][1 % N], S[a][2 % N], S[a][3 % N]);
            else to[(size_t)row * dv] = S[a][0];
        }
    }
    if (works) {
#pragma unroll
        for (int e = 0; e < N; ++e) part[(size_t)rg * dv + c + e] = acc[e];
    }
    __syncthreads();
    // the row groups' sums in order, then the norm over the head's lanes and the gate
    float ss = 0.f;
    for (int d = tid; d < dv; d += kStepThreads) {
        float s = 0.f;
        for (int r = 0; r < n_rg; ++r) s += part[(size_t)r * dv + d];
        part[d] = s;                                   // (only this thread reads or writes column d from here on)
        ss += s * s;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + eps);
    const float* gate = row_p + 2 * in.heads * dk + in.heads * dv + head * dv;
    for (int d = tid; d < dv; d += kStepThreads) orow[d] = from_f32<TO>(part[d] * inv * ret_silu(gate[d]));
}

// ---------------------------------------------------------------------------------------------
// chunks
// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ unsigned ret_smem(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ret_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ret_ldsm(uint32_t (&r)[4], unsigned a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ret_ldsm_t(uint32_t (&r)[4], unsigned a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ uint32_t ret_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// two numbers as bfloat16 pairs: the rounded ones, and what the rounding left (rounded again)
__device__ __forceinline__ void ret_split(float a, float b, uint32_t& hi, uint32_t& rest) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    rest = ret_pack(a - f.x, b - f.y);
}
__device__ __forceinline__ void ret_put4(__nv_bfloat16* dst, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(dst) = make_uint2(ret_pack(v[0], v[1]), ret_pack(v[2], v[3]));
}

// Which chunk a block has: sequence, first token of the chunk in the sequence, tokens, and whether there is one.
struct RetChunk {
    int seq, t0, rows, first_row, start;
    bool found;
};
__device__ __forceinline__ RetChunk ret_find(const RetSeq& sq, int block, int* shared3) {
    if (threadIdx.x == 0) {
        int t = block;
        shared3[0] = -1;
        for (int s = 0; s < sq.n_seqs; ++s) {
            const int len = sq.cu_seqlens[s + 1] - sq.cu_seqlens[s], tiles = (len + kC - 1) / kC;
            if (t < tiles) {
                shared3[0] = s;
                shared3[1] = t * kC;
                shared3[2] = len;
                break;
            }
            t -= tiles;
        }
    }
    __syncthreads();
    RetChunk c;
    c.seq = shared3[0];
    c.found = c.seq >= 0;
    if (!c.found) return c;
    c.t0 = shared3[1];
    c.rows = min(kC, shared3[2] - c.t0);
    c.first_row = sq.cu_seqlens[c.seq] + c.t0;
    c.start = sq.start_pos[c.seq] + c.t0;
    return c;
}

// How a block's threads share out [rows][per] items: thread (ty, tx) takes item tx of rows ty, ty + step, ...
struct RetShare {
    int tx, ty, step;
    bool works;
    __device__ __forceinline__ explicit RetShare(int per) {
        tx = threadIdx.x % per;
        ty = threadIdx.x / per;
        step = blockDim.x / per;
        works = ty < step;
    }
};
__device__ __forceinline__ float4 ret_zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ void ret_put4(__nv_bfloat16* dst, const float4& v) {
    *reinterpret_cast<uint2*>(dst) = make_uint2(ret_pack(v.x, v.y), ret_pack(v.z, v.w));
}
__device__ __forceinline__ void ret_split4(__nv_bfloat16* hi, __nv_bfloat16* rest, const float4& v) {
    uint32_t h0, h1, r0, r1;
    ret_split(v.x, v.y, h0, r0);
    ret_split(v.z, v.w, h1, r1);
    *reinterpret_cast<uint2*>(hi) = make_uint2(h0, h1);
    *reinterpret_cast<uint2*>(rest) = make_uint2(r0, r1);
}

// a head's values of a chunk as bfloat16 [kC][vstride], zeros beyond its tokens and lanes
__device__ __forceinline__ void ret_stage_values(const RetIn& in, const RetChunk& c, int head, __nv_bfloat16* vs, int vstride, int cols, bool vec) {
    const float* src = in.proj + (size_t)c.first_row * in.stride + 2 * in.heads * in.dk + head * in.dv;
    if (vec) {
        const RetShare sh(cols / 4);
        const int d = sh.tx * 4;
        for (int t = sh.ty; t < kC && sh.works; t += 4 * sh.step) {
            float4 v[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int r = t + u * sh.step;
                v[u] = r < c.rows && d < in.dv ? __ldg(reinterpret_cast<const float4*>(src + (size_t)r * in.stride + d)) : ret_zero4();
            }
#pragma unroll
            for (int u = 0; u < 4; ++u)
                if (t + u * sh.step < kC) ret_put4(vs + (t + u * sh.step) * vstride + d, v[u]);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < kC * cols; idx += blockDim.x) {
        const int t = idx / cols, d = idx % cols;
        vs[t * vstride + d] = __float2bfloat16_rn(t < c.rows && d < in.dv ? src[(size_t)t * in.stride + d] : 0.f);
    }
}

// a head's turned keys (and queries, where QUERIES) of a chunk: put(is_query, token, first of four lanes, values), every token of
// kC and every four lanes of dkp, zeros beyond the chunk's tokens and the head's lanes.  Keys come times k_scale.
template <bool QUERIES, typename Put>
__device__ __forceinline__ void ret_stage_rows(const RetIn& in, const RetChunk& c, int head, int dkp, bool vec, Put put) {
    const float* kp = in.proj + (size_t)c.first_row * in.stride + (in.heads + head) * in.dk;
    const float* qp = in.proj + (size_t)c.first_row * in.stride + head * in.dk;
    if (vec) {
        // an item: four lanes of the first half with their partners in the second, or four lanes that pass
        const int half = in.rot >> 1, pairs = half / 4, per = pairs + (dkp - in.rot) / 4;
        const RetShare sh(per);
        const bool turns = sh.tx < pairs;
        const int d = turns ? sh.tx * 4 : in.rot + (sh.tx - pairs) * 4;
        for (int t0 = sh.ty; t0 < kC && sh.works; t0 += 2 * sh.step) {
            float4 k[2][2], q[2][2], lo[2], hi[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int t = t0 + u * sh.step;
                const bool there = t < c.rows && d < in.dk;
                const size_t at = (size_t)t * in.stride + d;
                k[u][0] = there ? __ldg(reinterpret_cast<const float4*>(kp + at)) : ret_zero4();
                k[u][1] = there && turns ? __ldg(reinterpret_cast<const float4*>(kp + at + half)) : ret_zero4();
                if (QUERIES) {
                    q[u][0] = there ? __ldg(reinterpret_cast<const float4*>(qp + at)) : ret_zero4();
                    q[u][1] = there && turns ? __ldg(reinterpret_cast<const float4*>(qp + at + half)) : ret_zero4();
                }
                if (there && turns) ret_turn4(in, c.start + t, d, lo[u], hi[u]);
                else lo[u] = hi[u] = make_float4(1.f, 0.f, 1.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int t = t0 + u * sh.step;
                if (t >= kC) continue;
                if (turns) ret_turn_pairs(k[u][0], k[u][1], lo[u], hi[u]);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (e == 1 && !turns) continue;
                    float4& v = k[u][e];
                    v.x *= in.k_scale; v.y *= in.k_scale; v.z *= in.k_scale; v.w *= in.k_scale;
                    put(false, t, d + e * half, v);
                }
                if (QUERIES) {
                    if (turns) ret_turn_pairs(q[u][0], q[u][1], lo[u], hi[u]);
                    put(true, t, d, q[u][0]);
                    if (turns) put(true, t, d + half, q[u][1]);
                }
            }
        }
        return;
    }
    const int quads = dkp / 4;
    for (int idx = threadIdx.x; idx < (QUERIES ? 2 : 1) * kC * quads; idx += blockDim.x) {
        const bool is_q = idx >= kC * quads;
        const int i = is_q ? idx - kC * quads : idx, t = i / quads, d = (i % quads) * 4;
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (t < c.rows && d < in.dk) ret_lanes4(in, (is_q ? qp : kp) + (size_t)t * in.stride, c.start + t, d, false, v);
        const float w = is_q ? 1.f : in.k_scale;
        put(is_q, t, d, make_float4(v[0] * w, v[1] * w, v[2] * w, v[3] * w));
    }
}

// rows s0 .. s0 + m - 1 of S as high parts and rests [m][vstride], zeros beyond its rows and columns
__device__ __forceinline__ void ret_stage_state(const RetIn& in, const float* S, int s0, int m, __nv_bfloat16* sh, __nv_bfloat16* sr, int vstride, int cols,
                                                bool vec) {
    const RetShare share(cols / 4);
    const int d = share.tx * 4;
    for (int r0 = share.ty; r0 < m && share.works; r0 += 4 * share.step) {
        float4 v[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = r0 + u * share.step;
            v[u] = ret_zero4();
            if (r >= m || s0 + r >= in.dk || d >= in.dv) continue;
            const float* src = S + (size_t)(s0 + r) * in.dv + d;
            if (vec) {
                v[u] = __ldg(reinterpret_cast<const float4*>(src));
            } else {
                v[u].x = src[0];
                if (d + 1 < in.dv) v[u].y = src[1];
                if (d + 2 < in.dv) v[u].z = src[2];
                if (d + 3 < in.dv) v[u].w = src[3];
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = r0 + u * share.step;
            if (r < m) ret_split4(sh + r * vstride + d, sr + r * vstride + d, v[u]);
        }
    }
}

// (1) what a chunk adds to S by itself: kv [chunk][head][dk][dv]
__global__ void __launch_bounds__(256) retention_chunk_add_kernel(RetIn in, RetSeq sq, float* __restrict__ kv, int vec) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int found[3];
    const RetChunk c = ret_find(sq, blockIdx.x, found);
    if (!c.found) return;
    const int head = blockIdx.y, dk = in.dk, dv = in.dv;
    const int dkp = (dk + 15) & ~15, kstride = dkp + 8, cols = (dv + 63) & ~63, vstride = cols + 8;
    __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [kC][kstride] a^(last - t) k_t: high parts
    __nv_bfloat16* kr = kh + kC * kstride;                               // ... and rests
    __nv_bfloat16* vs = kr + kC * kstride;                               // [kC][vstride]
    const float* powers = in.powers + (size_t)head * (kC + 1);
    ret_stage_rows<false>(in, c, head, dkp, vec, [&](bool, int t, int d, float4 v) {
        const float w = t < c.rows ? powers[c.rows - 1 - t] : 0.f;
        v.x *= w; v.y *= w; v.z *= w; v.w *= w;
        ret_split4(kh + t * kstride + d, kr + t * kstride + d, v);
    });
    ret_stage_values(in, c, head, vs, vstride, cols, vec);
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int lrow = lane & 7, lmat = lane >> 3, quad = lane >> 2, pair = (lane & 3) * 2;
    float* dst = kv + ((size_t)blockIdx.x * in.heads + head) * dk * dv;
    // a unit: 16 rows of S by 32 of its columns
    const int units = (dkp / 16) * (cols / 32);
    const bool two = dv % 2 == 0;
    for (int u = warp; u < units; u += n_warps) {
        const int m0 = (u % (dkp / 16)) * 16, n0 = (u / (dkp / 16)) * 32;
        float acc[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        // A: the keys read transposed (rows of S by tokens)
        const unsigned ao = (unsigned)((((lmat >> 1) * 8 + lrow) * kstride + m0 + (lmat & 1) * 8) * 2);
        const unsigned bo = ret_smem(vs) + (unsigned)((((lmat & 1) * 8 + lrow) * vstride + n0 + (lmat >> 1) * 8) * 2);
#pragma unroll
        for (int kk = 0; kk < kC; kk += 16) {
            uint32_t ah[4], ar[4], b[4];
            ret_ldsm_t(ah, ret_smem(kh) + ao + kk * kstride * 2);
            ret_ldsm_t(ar, ret_smem(kr) + ao + kk * kstride * 2);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                ret_ldsm_t(b, bo + (kk * vstride + 16 * j) * 2);
                ret_mma(acc[2 * j], ah, b[0], b[1]);
                ret_mma(acc[2 * j + 1], ah, b[2], b[3]);
                ret_mma(acc[2 * j], ar, b[0], b[1]);
                ret_mma(acc[2 * j + 1], ar, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = m0 + quad + 8 * half, col = n0 + 8 * j + pair;
                if (row >= dk || col >= dv) continue;
                float* p = dst + (size_t)row * dv + col;
                if (two) {
                    *reinterpret_cast<float2*>(p) = make_float2(acc[j][2 * half], acc[j][2 * half + 1]);
                } else {
                    p[0] = acc[j][2 * half];
                    if (col + 1 < dv) p[1] = acc[j][2 * half + 1];
                }
            }
    }
}

// (2) S in front of every chunk, in place of what the chunk adds; S behind the last one goes to the sequence's state
__global__ void __launch_bounds__(256) retention_carry_kernel(RetIn in, RetSeq sq, float* __restrict__ kv) {
    const int head = blockIdx.y, seq = blockIdx.z;
    const size_t size = (size_t)in.dk * in.dv, at = (size_t)blockIdx.x * 256 + threadIdx.x;
    const int len = sq.cu_seqlens[seq + 1] - sq.cu_seqlens[seq];
    if (at >= size || len <= 0) return;
    int first = 0;                                     // the sequence's first chunk
    for (int s = 0; s < seq; ++s) first += (sq.cu_seqlens[s + 1] - sq.cu_seqlens[s] + kC - 1) / kC;
    const int start = sq.start_pos[seq], n_chunks = (len + kC - 1) / kC;
    float S = start > 0 ? sq.copy(seq, start)[(size_t)head * size + at] : 0.f;
    const float* powers = in.powers + (size_t)head * (kC + 1);
    const float full = powers[kC], last = powers[len - (n_chunks - 1) * kC];
    const size_t step = (size_t)in.heads * size;
    float* p = kv + (size_t)first * step + (size_t)head * size + at;
    constexpr int kRead = 16;                          // chunks read ahead of their turn
    for (int c0 = 0; c0 < n_chunks; c0 += kRead) {
        float add[kRead];
#pragma unroll
        for (int a = 0; a < kRead; ++a)
            if (c0 + a < n_chunks) add[a] = p[(size_t)(c0 + a) * step];
#pragma unroll
        for (int a = 0; a < kRead; ++a)
            if (c0 + a < n_chunks) {
                p[(size_t)(c0 + a) * step] = S;
                S = fmaf(c0 + a == n_chunks - 1 ? last : full, S, add[a]);
            }
    }
    sq.copy(seq, start + len)[(size_t)head * size + at] = S;
}

// (3) a chunk's rows: four warps of 16 rows each for every 8 NV value lanes.  slice: rows of S in shared memory at a time.
template <int WARPS, int NV>
__global__ void __launch_bounds__(32 * WARPS, NV == 4 ? 32 / WARPS : 1) retention_chunk_out_kernel(RetIn in, RetSeq sq, const float* __restrict__ kv, int slice, float eps,
                                                                   __nv_bfloat16* __restrict__ out, long long out_stride, int n_tokens, int vec) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ int found[3];
    __shared__ float pw[kC + 1];
    __shared__ float ssq[8][kC];
    const RetChunk c = ret_find(sq, blockIdx.x, found);
    const int head = blockIdx.y, dk = in.dk, dv = in.dv, tid = threadIdx.x;
    if (!c.found) {                                    // rows after the last sequence (padding up to a captured step's size) get zeros
        const int end = sq.cu_seqlens[sq.n_seqs];
        for (int idx = tid; idx < (n_tokens - end) * dv; idx += blockDim.x)
            out[(size_t)(end + idx / dv) * out_stride + (size_t)head * dv + idx % dv] = __float2bfloat16_rn(0.f);
        return;
    }
    const int dkp = (dk + 15) & ~15, kstride = dkp + 8, cols = (dv + 63) & ~63, vstride = cols + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [kC][kstride]
    __nv_bfloat16* ks = qs + kC * kstride;                               // [kC][kstride]
    __nv_bfloat16* vs = ks + kC * kstride;                               // [kC][vstride]
    __nv_bfloat16* sh = vs + kC * vstride;                               // [slice][vstride] S: high parts
    __nv_bfloat16* sr = sh + slice * vstride;                            // ... and rests
    const float* S = kv + ((size_t)blockIdx.x * in.heads + head) * dk * dv;
    ret_stage_rows<true>(in, c, head, dkp, vec, [&](bool is_q, int t, int d, const float4& v) { ret_put4((is_q ? qs : ks) + t * kstride + d, v); });
    ret_stage_values(in, c, head, vs, vstride, cols, vec);
    if (c.start > 0) ret_stage_state(in, S, 0, min(slice, dkp), sh, sr, vstride, cols, vec);      // (else S is zero)
    for (int i = tid; i <= kC; i += blockDim.x) pw[i] = in.powers[(size_t)head * (kC + 1) + i];
    const int lane = tid & 31, warp = tid >> 5, wr = warp & 3, wc = warp >> 2;
    const int lrow = lane & 7, lmat = lane >> 3, quad = lane >> 2, pair = (lane & 3) * 2;
    const int r0 = wr * 16 + quad, r1 = r0 + 8;        // this thread's two rows of the chunk
    float acc[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const unsigned qa = ret_smem(qs) + (unsigned)(((wr * 16 + lrow + (lmat & 1) * 8) * kstride + (lmat >> 1) * 8) * 2);
    const unsigned vo = (unsigned)((((lmat & 1) * 8 + lrow) * vstride + wc * 8 * NV + (lmat >> 1) * 8) * 2);
    __syncthreads();
    if (c.start > 0) {
        for (int s0 = 0; s0 < dkp; s0 += slice) {
            const int m = min(slice, dkp - s0);
            if (s0 > 0) {
                __syncthreads();
                ret_stage_state(in, S, s0, m, sh, sr, vstride, cols, vec);
                __syncthreads();
            }
            for (int kk = 0; kk < m; kk += 16) {
                uint32_t a[4], b[4];
                ret_ldsm(a, qa + (s0 + kk) * 2);
#pragma unroll
                for (int j = 0; j < NV / 2; ++j) {
                    ret_ldsm_t(b, ret_smem(sh) + vo + (kk * vstride + 16 * j) * 2);
                    ret_mma(acc[2 * j], a, b[0], b[1]);
                    ret_mma(acc[2 * j + 1], a, b[2], b[3]);
                    ret_ldsm_t(b, ret_smem(sr) + vo + (kk * vstride + 16 * j) * 2);
                    ret_mma(acc[2 * j], a, b[0], b[1]);
                    ret_mma(acc[2 * j + 1], a, b[2], b[3]);
                }
            }
        }
        const float w0 = pw[r0 + 1], w1 = pw[r1 + 1];
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            acc[j][0] *= w0; acc[j][1] *= w0;
            acc[j][2] *= w1; acc[j][3] *= w1;
        }
    }
    // the chunk's own tokens, 16 keys at a time: (q_t . k_s) a^(t - s), then times the values; keys behind every row of the warp
    // are passed by
    const unsigned ka = ret_smem(ks) + (unsigned)(((lrow + (lmat >> 1) * 8) * kstride + (lmat & 1) * 8) * 2);
#pragma unroll 1
    for (int j16 = 0; j16 <= wr; ++j16) {
        float s[2][4];
        s[0][0] = s[0][1] = s[0][2] = s[0][3] = s[1][0] = s[1][1] = s[1][2] = s[1][3] = 0.f;
        for (int kk = 0; kk < dkp; kk += 16) {
            uint32_t a[4], b[4];
            ret_ldsm(a, qa + kk * 2);
            ret_ldsm(b, ka + (16 * j16 * kstride + kk) * 2);
            ret_mma(s[0], a, b[0], b[1]);
            ret_mma(s[1], a, b[2], b[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int back = (e < 2 ? r0 : r1) - (16 * j16 + 8 * j + pair + (e & 1));
                s[j][e] = back >= 0 ? s[j][e] * pw[back] : 0.f;
            }
        uint32_t ah[4], ar[4], b[4];
        ret_split(s[0][0], s[0][1], ah[0], ar[0]);
        ret_split(s[0][2], s[0][3], ah[1], ar[1]);
        ret_split(s[1][0], s[1][1], ah[2], ar[2]);
        ret_split(s[1][2], s[1][3], ah[3], ar[3]);
#pragma unroll
        for (int j = 0; j < NV / 2; ++j) {
            ret_ldsm_t(b, ret_smem(vs) + vo + (16 * j16 * vstride + 16 * j) * 2);
            ret_mma(acc[2 * j], ah, b[0], b[1]);
            ret_mma(acc[2 * j + 1], ah, b[2], b[3]);
            ret_mma(acc[2 * j], ar, b[0], b[1]);
            ret_mma(acc[2 * j + 1], ar, b[2], b[3]);
        }
    }
    // the norm over the head's lanes: this warp's of them, then the other warps' of the same rows
    float q0 = 0.f, q1 = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        q0 += acc[j][0] * acc[j][0] + acc[j][1] * acc[j][1];
        q1 += acc[j][2] * acc[j][2] + acc[j][3] * acc[j][3];
    }
    q0 += __shfl_xor_sync(0xffffffffu, q0, 1);
    q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
    q1 += __shfl_xor_sync(0xffffffffu, q1, 1);
    q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
    if (pair == 0) {
        ssq[wc][r0] = q0;
        ssq[wc][r1] = q1;
    }
    __syncthreads();
    const int n_wc = WARPS / 4;
    const bool two = dv % 2 == 0 && out_stride % 2 == 0 && ((size_t)out & 3) == 0 && vec;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = half ? r1 : r0;
        if (r >= c.rows) continue;
        float ss = 0.f;
        for (int w = 0; w < n_wc; ++w) ss += ssq[w][r];
        const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
        const float* gate = in.proj + (size_t)(c.first_row + r) * in.stride + 2 * in.heads * dk + (in.heads + head) * dv;
        __nv_bfloat16* o = out + (size_t)(c.first_row + r) * out_stride + (size_t)head * dv;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int d = wc * 8 * NV + 8 * j + pair;
            if (d >= dv) continue;
            const float x0 = acc[j][2 * half] * inv, x1 = acc[j][2 * half + 1] * inv;
            if (two) {
                const float2 g = *reinterpret_cast<const float2*>(gate + d);
                *reinterpret_cast<uint32_t*>(o + d) = ret_pack(x0 * ret_silu(g.x), x1 * ret_silu(g.y));
            } else {
                o[d] = __float2bfloat16_rn(x0 * ret_silu(gate[d]));
                if (d + 1 < dv) o[d + 1] = __float2bfloat16_rn(x1 * ret_silu(gate[d + 1]));
            }
        }
    }
}

// ---------------------------------------------------------------------------------------------
// entry points
// ---------------------------------------------------------------------------------------------
static size_t chunk_smem(int dk, int dv, int slice) {
    const int kstride = ((dk + 15) & ~15) + 8, vstride = ((dv + 63) & ~63) + 8;
    return ((size_t)2 * kC * kstride + (size_t)kC * vstride + (size_t)2 * slice * vstride) * sizeof(__nv_bfloat16);
}
// rows of S that fit beside a chunk's tokens, 0 when the chunk kernels do not take the head size
static int chunk_slice(int dk, int dv) {
    if (dk > 256 || dv > 512) return 0;
    const int dkp = (dk + 15) & ~15;
    for (int slice = dkp < 64 ? dkp : 64; slice >= 16; slice -= 16)
        if (chunk_smem(dk, dv, slice) <= 220 * 1024) return slice;
    return 0;
}
BLM_API int blm_retention_chunks_take(int dk, int dv) { return chunk_slice(dk, dv) > 0; }
BLM_API int blm_retention_step_takes(int dk, int dv) { return dk <= 2048 && (dv % 4 == 0 ? dv <= 4 * kStepThreads : dv <= kStepThreads); }
BLM_API int blm_retention_power_row() { return kC + 1; }
BLM_API int blm_retention_chunks(int n_tokens, int n_seqs) { return (n_tokens + kC - 1) / kC + n_seqs; }

#define RET_ARGS                                                                                                                          \
    const float *proj, long long stride, int heads, int dk, int dv, float k_scale, const double *freq, int rot, const float *table,      \
        int table_len, const float *powers, const int *cu_seqlens, const int *slot_of_seq, const int *start_pos, int n_seqs, float *state, \
        long long slot_stride, long long copy_stride, long long offset
#define RET_CHECK(what)                                                                                                                   \
    BLM_REQUIRE(heads > 0 && heads <= 65535 && dk > 0 && dv > 0 && n_seqs >= 0 && n_seqs <= 65535, what ": bad sizes");                  \
    BLM_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dk && (rot == 0 || freq != nullptr), what ": %d turning lanes of %d", rot, dk);       \
    BLM_REQUIRE(stride >= (long long)heads * (2 * dk + 2 * dv) && powers != nullptr && state != nullptr, what ": rows of %lld", stride); \
    const RetIn in{proj, stride, heads, dk, dv, k_scale, freq, rot, (const float2*)table, table ? table_len : 0, powers};                \
    const RetSeq sq{cu_seqlens, slot_of_seq, start_pos, n_seqs, state, slot_stride, copy_stride, offset};                                \
    const int vec = ret_vec(in) && (((size_t)state | (size_t)table) & 15) == 0 && slot_stride % 4 == 0 && copy_stride % 4 == 0 && offset % 4 == 0

// o [N, heads * dv] float32, not normed yet; rows of no sequence are left alone
BLM_API int blm_retention_scan(RET_ARGS, float* o, long long o_stride, cudaStream_t stream) {
    if (n_seqs == 0) return BLM_OK;
    RET_CHECK("retention_scan");
    (void)vec;
    BLM_REQUIRE(dk <= 512 && dv <= 65535, "retention_scan: keys of %d lanes; at most 512", dk);
    const size_t smem = (size_t)kScanTokens * (2 * dk + 32) * sizeof(float);
    const dim3 grid((dv + 31) / 32, heads, n_seqs);
    auto launch = [&](auto kernel) -> int {
        if (smem > 48 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return blm_fail(BLM_CUDA_ERROR, "retention_scan: %s", cudaGetErrorString(e));
        }
        kernel<<<grid, 256, smem, stream>>>(in, sq, o, o_stride);
        return blm_check_launch("retention_scan");
    };
    if (dk <= 16) return launch(retention_scan_kernel<2>);
    if (dk <= 32) return launch(retention_scan_kernel<4>);
    if (dk <= 64) return launch(retention_scan_kernel<8>);
    if (dk <= 128) return launch(retention_scan_kernel<16>);
    if (dk <= 256) return launch(retention_scan_kernel<32>);
    return launch(retention_scan_kernel<64>);
}

// out [N, heads * dv] (rows of out_stride), finished; every sequence brings one token
BLM_API int blm_retention_step(RET_ARGS, const int* token_seq, const int* token_pos, int n_tokens, float eps, void* out, int out_dtype,
                               long long out_stride, cudaStream_t stream) {
    if (n_tokens == 0) return BLM_OK;
    RET_CHECK("retention_step");
    BLM_REQUIRE(blm_retention_step_takes(dk, dv) && n_tokens <= 65535, "retention_step: %d tokens, heads of %d and %d lanes", n_tokens, dk, dv);
    const int n = vec ? 4 : 1;
    BLM_REQUIRE(dv / n <= kStepThreads, "retention_step: values of %d lanes", dv);
    const size_t smem = ((size_t)2 * ((dk + 3) & ~3) + 36 + (size_t)(kStepThreads / (dv / n)) * dv) * sizeof(float);
    const dim3 grid(heads, n_tokens);
    const bool few = dk <= 4 * (kStepThreads / (dv / n));
#define RET_STEP_OF(TO, N, A) retention_step_kernel<TO, N, A><<<grid, kStepThreads, smem, stream>>>(in, sq, token_seq, token_pos, eps, (TO*)out, out_stride, vec)
#define RET_STEP(TO, N) do { if (few) RET_STEP_OF(TO, N, 4); else RET_STEP_OF(TO, N, 8); } while (0)
    if (out_dtype == BLM_BF16) {
        if (vec) RET_STEP(__nv_bfloat16, 4); else RET_STEP(__nv_bfloat16, 1);
    } else if (out_dtype == BLM_F32) {
        if (vec) RET_STEP(float, 4); else RET_STEP(float, 1);
    } else {
        return blm_fail(BLM_BAD_ARGUMENT, "retention_step: dtype %d", out_dtype);
    }
#undef RET_STEP
#undef RET_STEP_OF
    return blm_check_launch("retention_step");
}

// out bfloat16 as above, any number of tokens a sequence; kv: float32 scratch [blm_retention_chunks(...)][heads][dk][dv]
BLM_API int blm_retention_portions(RET_ARGS, int n_tokens, float eps, float* kv, void* out, long long out_stride, cudaStream_t stream) {
    if (n_tokens == 0) return BLM_OK;
    RET_CHECK("retention_portions");
    const int slice = chunk_slice(dk, dv), chunks = blm_retention_chunks(n_tokens, n_seqs);
    BLM_REQUIRE(slice > 0 && kv != nullptr && ((size_t)kv & 15) == 0, "retention_portions: heads of %d and %d lanes", dk, dv);
    const size_t smem1 = ((size_t)2 * kC * (((dk + 15) & ~15) + 8) + (size_t)kC * (((dv + 63) & ~63) + 8)) * sizeof(__nv_bfloat16);
    const size_t smem3 = chunk_smem(dk, dv, slice);
    static size_t allowed1 = 48 * 1024;
    if (smem1 > allowed1) {
        cudaError_t e = cudaFuncSetAttribute(retention_chunk_add_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return blm_fail(BLM_CUDA_ERROR, "retention_portions: %s", cudaGetErrorString(e));
        allowed1 = smem1;
    }
    const dim3 grid(chunks, heads);
    retention_chunk_add_kernel<<<grid, 256, smem1, stream>>>(in, sq, kv, vec);
    const size_t size = (size_t)dk * dv;
    retention_carry_kernel<<<dim3((unsigned)((size + 255) / 256), heads, n_seqs), 256, 0, stream>>>(in, sq, kv);
    auto rows = [&](auto kernel, int threads) -> int {
        if (smem3 > 48 * 1024) {
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
            if (e != cudaSuccess) return blm_fail(BLM_CUDA_ERROR, "retention_portions: %s", cudaGetErrorString(e));
        }
        kernel<<<grid, threads, smem3, stream>>>(in, sq, kv, slice, eps, (__nv_bfloat16*)out, out_stride, n_tokens, vec);
        return blm_check_launch("retention_portions");
    };
    if (dv <= 64) return rows(retention_chunk_out_kernel<8, 4>, 256);
    if (dv <= 128) return rows(retention_chunk_out_kernel<16, 4>, 512);
    if (dv <= 256) return rows(retention_chunk_out_kernel<16, 8>, 512);
    return rows(retention_chunk_out_kernel<32, 8>, 1024);
}
