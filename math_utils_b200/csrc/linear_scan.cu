// Recurrent mixers with a matrix state S [dk][dv] per head that is written without being read first:
//     S <- decay S + take k v^T,   o = scale * S^T q,
// and the gates they take.  Everything float32.
//
// mu_linear_scan   per (sequence, head, a few columns of S), the step's tokens in order.  The decay is one number per
//                  head (with a `take` beside it) or one per head and key channel (gated linear attention).  With a
//                  normalizer the state has one more column, n <- decay n + take k, whose read-out n . q goes to an
//                  array of its own (the matrix memory of xLSTM).  Gates that are the same for every token (lightning
//                  attention's constant decays) are read with a token stride of zero; with `silu_rows` keys, queries and
//                  values pass silu once they are staged.  State of a slot, from state_offset on:
//                  [ S: heads x dv x dk (a head's S column after column) | n: heads x dk ].
//                  Four columns live in the registers of up to 32 lanes, two entries to a 64-bit register; a key, a
//                  query and a decay read from shared memory serve four columns.  Nothing waits for a token's
//                  read-out, so the lanes keep their partial sums of as many (token, column) pairs as there are lanes
//                  and add them crosswise: 31 exchanges for 8 tokens of 4 columns over 32 lanes, after which every lane
//                  holds one finished sum.  Keys, queries, decays and values of 16 tokens at a time are copied to
//                  shared memory asynchronously, the next 16 on their way meanwhile.  The order of every sum is fixed
//                  by dk alone: a token's result does not depend on how the sequence was cut into steps or on the batch.
// mu_exp_gates     the exponential gates of such a memory: i = cap tanh((i_raw + i_bias) / cap),
//                  f = log sigmoid(cap tanh((f_raw + f_bias) / cap)), a running maximum m <- max(f + m, i) that starts
//                  at zero and stays with the sequence's state; per token and head (decay, take, floor) =
//                  (exp(f + m_before - m), exp(i - m), exp(-m)).  m enters S, n and the floor alike, so which
//                  maximum is kept changes no result; it is found for 256 tokens at a time by a scan.
// mu_low_rank      out[t][c] = fn( sum_r W[c][r] low[t][r] + bias[c] ): the second of a projection's two matrices, for
//                  one or two such projections in one launch, with what follows it:
//                  (bfloat16 weights and many tokens: tensor cores; few tokens: eight lanes an output; else one
//                  running sum per output over r.)
//                  fn 0: nothing;  1: sigmoid(z)^power;  2: exp(-exp(A_log[c / per_head]) softplus(z));  3: softplus(z).
#include "common.cuh"

#include <math.h>

namespace mu {

constexpr int LS_THREADS = 128;
constexpr int LS_PER = 4;         // columns of S whose entries a lane holds
constexpr int LS_CHUNK = 16;      // tokens staged at a time
constexpr int LS_MAX_DK = 256;

// Columns a block takes: LANES lanes share four columns.
__host__ __device__ constexpr int ls_columns(int lanes) { return LS_PER * LS_THREADS / lanes; }
// Floats of one staged chunk: keys, queries (and the channels' decays), values, (decay, take, floor, -).
__host__ __device__ constexpr int ls_chunk_floats(int dkp, int cols, bool per_channel) {
    return LS_CHUNK * ((per_channel ? 3 : 2) * dkp + cols + 4);
}

__device__ __forceinline__ float ls_silu(float z) { return z / (1.0f + expf(-z)); }

// LANES lanes hold four columns of S, R entries of each a lane (a multiple of 4; dk <= LANES R), dealt to the lanes
// four entries at a time: what a lane reads of a staged key, query and decay serves its four columns.  LANES and R
// follow from dk alone.  VEC: every row, slice and state column starts on a 16-byte boundary.
template <int R, int LANES, bool VEC, bool PER_CHANNEL>
__global__ void __launch_bounds__(LS_THREADS)
linear_scan_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                   const float* __restrict__ decay, int n_heads, int dk, int dv, float scale,
                   const int* __restrict__ seq_first, const int* __restrict__ seq_slots, float* __restrict__ state,
                   long long state_stride, long long state_offset, float* __restrict__ out, long long ldo,
                   float* __restrict__ norm_out, long long gate_stride, int silu_rows) {
    constexpr int DKP = LANES * R, Q = R / 4, COLS = ls_columns(LANES), BUF = ls_chunk_floats(DKP, COLS, PER_CHANNEL);
    constexpr int GROUP = LANES / LS_PER;                    // tokens whose read-outs are summed together
    extern __shared__ __align__(16) float ls_smem[];
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, c0 = LS_PER * (tid / LANES), l = tid % LANES;
    for (int i = tid; i < 2 * BUF; i += LS_THREADS) ls_smem[i] = 0.0f;   // the padding past dk and dv stays zero
    pdl_wait();
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    float* const slot = state + (long long)seq_slots[s] * state_stride + state_offset;
    // the columns of this lane: a value entry each, or (column dv, where asked for) the normalizer, whose value is one
    auto column = [&](int c) {
        const int j = col0 + c0 + c;
        return slot + (j == dv ? (long long)n_heads * dv + h : (long long)h * dv + j) * dk;
    };
    const int n_live = min(LS_PER, dv + (norm_out ? 1 : 0) - col0 - c0);         // (may be negative)
    const int norm_at = norm_out ? dv - col0 - c0 : LS_PER;                      // which of the four is the normalizer
    float2x S[LS_PER][2 * Q];
#pragma unroll
    for (int c = 0; c < LS_PER; ++c)
#pragma unroll
        for (int i = 0; i < Q; ++i) {
            const int d = 4 * (l + LANES * i);
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (c < n_live) {
                const float* mine = column(c);
                if (VEC) {
                    if (d < dk) x = *reinterpret_cast<const float4*>(mine + d);
                } else {
                    if (d < dk) x.x = mine[d];
                    if (d + 1 < dk) x.y = mine[d + 1];
                    if (d + 2 < dk) x.z = mine[d + 2];
                    if (d + 3 < dk) x.w = mine[d + 3];
                }
            }
            S[c][2 * i] = pair_of_floats(x.x, x.y);
            S[c][2 * i + 1] = pair_of_floats(x.z, x.w);
        }
    // stages the chunk that starts at the sequence's li0-th token of this step into buffer `b`
    auto stage = [&](int li0, int b) {
        float* ks = ls_smem + b * BUF;
        float* qs = ks + LS_CHUNK * DKP;
        float* gs = qs + LS_CHUNK * DKP;
        float* vs = gs + (PER_CHANNEL ? LS_CHUNK * DKP : 0);
        float* sc = vs + LS_CHUNK * COLS;
        const int n = min(LS_CHUNK, count - li0);
        const long long t0 = first + li0;
        if (VEC) {
            const int per = dk / 4;
            for (int i = tid; i < n * per; i += LS_THREADS) {
                const int tok = i / per, d = 4 * (i % per);
                const long long at = (t0 + tok) * ld + (long long)h * dk + d;
                copy_async16(ks + tok * DKP + d, k + at);
                copy_async16(qs + tok * DKP + d, q + at);
                if (PER_CHANNEL) copy_async16(gs + tok * DKP + d, decay + ((t0 + tok) * n_heads + h) * dk + d);
            }
            for (int i = tid; i < n * (COLS / 4); i += LS_THREADS) {
                const int tok = i / (COLS / 4), cc = 4 * (i % (COLS / 4));
                if (col0 + cc < dv) copy_async16(vs + tok * COLS + cc, v + (t0 + tok) * ld + (long long)h * dv + col0 + cc);
            }
        } else {
            for (int i = tid; i < n * dk; i += LS_THREADS) {
                const int tok = i / dk, d = i % dk;
                const long long at = (t0 + tok) * ld + (long long)h * dk + d;
                copy_async4(ks + tok * DKP + d, k + at);
                copy_async4(qs + tok * DKP + d, q + at);
                if (PER_CHANNEL) copy_async4(gs + tok * DKP + d, decay + ((t0 + tok) * n_heads + h) * dk + d);
            }
            for (int i = tid; i < n * COLS; i += LS_THREADS) {
                const int tok = i / COLS, cc = i % COLS;
                if (col0 + cc < dv) copy_async4(vs + tok * COLS + cc, v + (t0 + tok) * ld + (long long)h * dv + col0 + cc);
            }
        }
        if (!PER_CHANNEL)
            for (int tok = tid; tok < n; tok += LS_THREADS) copy_async16(sc + tok * 4, decay + (t0 + tok) * gate_stride + 4 * h);
        copy_async_commit();
    };
    __syncthreads();                                         // the zeros are down before the first copies land
    if (count > 0) stage(0, 0);
    int b = 0;
    for (int li0 = 0; li0 < count; li0 += LS_CHUNK, b ^= 1) {
        const int n = min(LS_CHUNK, count - li0);
        if (li0 + LS_CHUNK < count) {
            stage(li0 + LS_CHUNK, b ^ 1);
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        if (silu_rows) {                                     // (zeros stay zeros)
            float* rows = ls_smem + b * BUF;
            for (int i = tid; i < n * DKP; i += LS_THREADS) {
                rows[i] = ls_silu(rows[i]);
                rows[LS_CHUNK * DKP + i] = ls_silu(rows[LS_CHUNK * DKP + i]);
            }
            float* values = rows + (PER_CHANNEL ? 3 : 2) * LS_CHUNK * DKP;
            for (int i = tid; i < n * COLS; i += LS_THREADS) values[i] = ls_silu(values[i]);
            __syncthreads();
        }
        const float* ks = ls_smem + b * BUF;
        const float* qs = ks + LS_CHUNK * DKP;
        const float* gs = qs + LS_CHUNK * DKP;
        const float* vs = gs + (PER_CHANNEL ? LS_CHUNK * DKP : 0);
        const float* sc = vs + LS_CHUNK * COLS;
        // One token: S = g S + k v for the lane's entries, and the lane's share of each column's S . q into `sum`.
        auto step = [&](int tok, float* sum) {
            float4 v4 = *reinterpret_cast<const float4*>(vs + tok * COLS + c0);
            float value[LS_PER] = {v4.x, v4.y, v4.z, v4.w};
            float2x fade = 0;
            if (!PER_CHANNEL) {
                const float2 gate = *reinterpret_cast<const float2*>(sc + tok * 4);      // decay, take
                fade = pair_of_floats(gate.x, gate.x);
#pragma unroll
                for (int c = 0; c < LS_PER; ++c) value[c] = (c == norm_at ? 1.0f : value[c]) * gate.y;
            }
            float2x a[LS_PER] = {0, 0, 0, 0};                                            // (two zeros each)
#pragma unroll
            for (int i = 0; i < Q; ++i) {
                const int at = tok * DKP + 4 * (l + LANES * i);
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(ks + at);
                const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(qs + at);
                ulonglong2 gg = make_ulonglong2(fade, fade);
                if (PER_CHANNEL) gg = *reinterpret_cast<const ulonglong2*>(gs + at);
#pragma unroll
                for (int c = 0; c < LS_PER; ++c) {
                    const float2x v2 = pair_of_floats(value[c], value[c]);
                    S[c][2 * i] = pair_fma(kk.x, v2, pair_mul(gg.x, S[c][2 * i]));
                    S[c][2 * i + 1] = pair_fma(kk.y, v2, pair_mul(gg.y, S[c][2 * i + 1]));
                    a[c] = pair_fma(S[c][2 * i], qq.x, a[c]);
                    a[c] = pair_fma(S[c][2 * i + 1], qq.y, a[c]);
                }
            }
#pragma unroll
            for (int c = 0; c < LS_PER; ++c) {
                const float2 x = floats_of_pair(a[c]);
                sum[c] = x.x + x.y;
            }
        };
        for (int t0 = 0; t0 < n; t0 += GROUP) {
            float acc[LANES];                                // token t0 + i, column c at [4 i + c]
            const int left = n - t0;
            if (left >= GROUP) {                             // a whole group: no branch between the tokens
#pragma unroll
                for (int i = 0; i < GROUP; ++i) step(t0 + i, acc + LS_PER * i);
            } else {
#pragma unroll
                for (int i = 0; i < GROUP; ++i) {
#pragma unroll
                    for (int c = 0; c < LS_PER; ++c) acc[LS_PER * i + c] = 0.0f;
                    if (i < left) step(t0 + i, acc + LS_PER * i);
                }
            }
#pragma unroll
            for (int width = LANES / 2; width >= 1; width >>= 1) {
#pragma unroll
                for (int i = 0; i < width; ++i) {
                    const bool upper = (l & width) != 0;
                    const float send = upper ? acc[i] : acc[i + width];
                    const float keep = upper ? acc[i + width] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, width);
                }
            }
            const int tok = l / LS_PER, c = l % LS_PER;      // what this lane's sum is of
            if (tok < left && c < n_live) {
                const long long t = first + li0 + t0 + tok;
                if (c == norm_at) norm_out[t * n_heads + h] = scale * acc[0];
                else out[t * ldo + (long long)h * dv + col0 + c0 + c] = scale * acc[0];
            }
        }
        __syncthreads();                                     // this buffer is free for the chunk after the next
    }
    pdl_trigger();                                           // (only now: see the delta scan)
#pragma unroll
    for (int c = 0; c < LS_PER; ++c)
#pragma unroll
        for (int i = 0; i < Q; ++i) {
            const int d = 4 * (l + LANES * i);
            const float2 lo = floats_of_pair(S[c][2 * i]), hi = floats_of_pair(S[c][2 * i + 1]);
            if (c >= n_live) continue;
            float* mine = column(c);
            if (VEC) {
                if (d < dk) *reinterpret_cast<float4*>(mine + d) = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
                if (d < dk) mine[d] = lo.x;
                if (d + 1 < dk) mine[d + 1] = lo.y;
                if (d + 2 < dk) mine[d + 2] = hi.x;
                if (d + 3 < dk) mine[d + 3] = hi.y;
            }
        }
}

// One block per (sequence, head); a thread a token of the chunk.  What a run of tokens does to m is a pair (F, M):
// m -> max(F + m, M); two runs in a row are (F1 + F2, max(M1 + F2, M2)).
__global__ void __launch_bounds__(256)
exp_gates_kernel(const float* __restrict__ i_raw, const float* __restrict__ f_raw, long long ld,
                 const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap, int n_heads,
                 const int* __restrict__ seq_first, const int* __restrict__ seq_slots, float* __restrict__ state,
                 long long state_stride, long long m_offset, float4* __restrict__ gates) {
    __shared__ float run_f[8], run_m[8], last_m[8];
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    if (count <= 0) return;
    float* kept = state + (long long)seq_slots[s] * state_stride + m_offset + h;
    float carry = *kept;
    const float ib = i_bias[h], fb = f_bias[h];
    for (int li0 = 0; li0 < count; li0 += blockDim.x) {
        const bool in = li0 + tid < count;
        const long long t = first + li0 + tid;
        float i = -INFINITY, f = 0.0f;                       // a token that is not there leaves m as it is
        if (in) {
            i = cap * tanhf((i_raw[t * ld + h] + ib) / cap);
            f = -softplus(-cap * tanhf((f_raw[t * ld + h] + fb) / cap));
        }
        float F = f, M = i;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) {
                M = fmaxf(pm + F, M);
                F += pf;
            }
        }
        if (lane == 31) {
            run_f[warp] = F;
            run_m[warp] = M;
        }
        __syncthreads();
        float before = carry;                                // m as this warp's first token finds it
        for (int w = 0; w < warp; ++w) before = fmaxf(run_f[w] + before, run_m[w]);
        const float m = fmaxf(F + before, M);
        float prev = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) prev = before;
        if (in) gates[t * n_heads + h] = make_float4(expf(f + prev - m), expf(i - m), expf(-m), 0.0f);
        if (lane == 31) last_m[warp] = m;
        __syncthreads();
        carry = last_m[warps - 1];
    }
    if (tid == 0) *kept = carry;
}

constexpr int LR_CHANNELS = 128, LR_THREADS = 64, LR_TOK = 16;           // a thread takes two channels
struct LowRankPart {
    const void* w;            // [n][ldw], the first `rank` entries of a row
    const float* bias;        // [n] or null
    const float* a_log;       // fn 2: one per `per_head` channels
    float* out;               // [T][n]
    long long ldw;
    int col, rank, n, fn, per_head;
    float power;
};

__device__ __forceinline__ float low_rank_fn(float z, const LowRankPart& p, float rate) {
    if (p.fn == 1) return expf(-p.power * softplus(-z));
    if (p.fn == 2) return expf(-rate * softplus(z));
    if (p.fn == 3) return softplus(z);
    return z;
}

template <int N, typename T> __device__ __forceinline__ void load_weights(float (&x)[N], const T* p, int n) {
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = i < n ? to_float(p[i]) : 0.0f;
}

// A block: 16 tokens x 128 channels of one of the parts.  The tokens' low-rank rows are staged in shared memory; a
// thread keeps eight weights of each of its two channels and runs over the tokens.  One running sum per output over r
// in order, whatever shares its block.
template <typename TW>
__global__ void __launch_bounds__(LR_THREADS)
low_rank_kernel(const float* __restrict__ low, long long ldl, int n_tokens, LowRankPart p0, LowRankPart p1, int blocks0) {
    extern __shared__ __align__(16) float lr_smem[];         // [LR_TOK][rank padded to 8]
    pdl_trigger();
    const bool second = (int)blockIdx.y >= blocks0;
    const LowRankPart p = second ? p1 : p0;
    const int c0 = ((int)blockIdx.y - (second ? blocks0 : 0)) * LR_CHANNELS + threadIdx.x, c1 = c0 + LR_THREADS;
    const int t0 = blockIdx.x * LR_TOK, nt = min(LR_TOK, n_tokens - t0);
    const int rp = (p.rank + 7) & ~7;
    pdl_wait();
    for (int i = threadIdx.x; i < LR_TOK * rp; i += LR_THREADS) {
        const int t = i / rp, r = i % rp;
        lr_smem[i] = t < nt && r < p.rank ? low[(long long)(t0 + t) * ldl + p.col + r] : 0.0f;
    }
    __syncthreads();
    const TW* w0 = reinterpret_cast<const TW*>(p.w) + (long long)min(c0, p.n - 1) * p.ldw;
    const TW* w1 = reinterpret_cast<const TW*>(p.w) + (long long)min(c1, p.n - 1) * p.ldw;
    float a0[LR_TOK], a1[LR_TOK];
#pragma unroll
    for (int t = 0; t < LR_TOK; ++t) a0[t] = a1[t] = 0.0f;
    const bool vec = sizeof(TW) == 2 && p.ldw % 8 == 0 && ((uintptr_t)p.w & 15) == 0;
    for (int r = 0; r < p.rank; r += 8) {
        float x0[8], x1[8];
        if (vec && r + 8 <= p.rank) {
            const uint4 u0 = *reinterpret_cast<const uint4*>(w0 + r), u1 = *reinterpret_cast<const uint4*>(w1 + r);
            const __nv_bfloat162* b0 = reinterpret_cast<const __nv_bfloat162*>(&u0);
            const __nv_bfloat162* b1 = reinterpret_cast<const __nv_bfloat162*>(&u1);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f0 = __bfloat1622float2(b0[i]), f1 = __bfloat1622float2(b1[i]);
                x0[2 * i] = f0.x, x0[2 * i + 1] = f0.y, x1[2 * i] = f1.x, x1[2 * i + 1] = f1.y;
            }
        } else {
            load_weights<8>(x0, w0 + r, p.rank - r);
            load_weights<8>(x1, w1 + r, p.rank - r);
        }
#pragma unroll
        for (int t = 0; t < LR_TOK; ++t) {
            const float4 y = *reinterpret_cast<const float4*>(lr_smem + t * rp + r);
            const float4 z = *reinterpret_cast<const float4*>(lr_smem + t * rp + r + 4);
            a0[t] = fmaf(x0[0], y.x, a0[t]), a1[t] = fmaf(x1[0], y.x, a1[t]);
            a0[t] = fmaf(x0[1], y.y, a0[t]), a1[t] = fmaf(x1[1], y.y, a1[t]);
            a0[t] = fmaf(x0[2], y.z, a0[t]), a1[t] = fmaf(x1[2], y.z, a1[t]);
            a0[t] = fmaf(x0[3], y.w, a0[t]), a1[t] = fmaf(x1[3], y.w, a1[t]);
            a0[t] = fmaf(x0[4], z.x, a0[t]), a1[t] = fmaf(x1[4], z.x, a1[t]);
            a0[t] = fmaf(x0[5], z.y, a0[t]), a1[t] = fmaf(x1[5], z.y, a1[t]);
            a0[t] = fmaf(x0[6], z.z, a0[t]), a1[t] = fmaf(x1[6], z.z, a1[t]);
            a0[t] = fmaf(x0[7], z.w, a0[t]), a1[t] = fmaf(x1[7], z.w, a1[t]);
        }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int c = half ? c1 : c0;
        if (c >= p.n) continue;
        const float bias = p.bias ? p.bias[c] : 0.0f;
        const float rate = p.fn == 2 ? expf(p.a_log[c / p.per_head]) : 0.0f;
#pragma unroll
        for (int t = 0; t < LR_TOK; ++t) {
            if (t >= nt) break;
            p.out[(long long)(t0 + t) * p.n + c] = low_rank_fn((half ? a1[t] : a0[t]) + bias, p, rate);
        }
    }
}

// The same for a few tokens (single-token steps above all): eight lanes share a channel and take its weights eight
// entries at a time in turn, so that a row's weights are on their way at once; the lanes' sums meet by shuffles, and
// lane i finishes token i of the block's four.
constexpr int LF_TOK = 4, LF_THREADS = 128, LF_CHANNELS = LF_THREADS / 8;

template <typename TW>
__global__ void __launch_bounds__(LF_THREADS)
low_rank_few_kernel(const float* __restrict__ low, long long ldl, int n_tokens, LowRankPart p0, LowRankPart p1, int blocks0) {
    pdl_trigger();
    const bool second = (int)blockIdx.y >= blocks0;
    const LowRankPart p = second ? p1 : p0;
    const int lane = threadIdx.x & 7, c = ((int)blockIdx.y - (second ? blocks0 : 0)) * LF_CHANNELS + (threadIdx.x >> 3);
    const int t0 = blockIdx.x * LF_TOK, nt = min(LF_TOK, n_tokens - t0);
    const TW* w = reinterpret_cast<const TW*>(p.w) + (long long)min(c, p.n - 1) * p.ldw;
    const bool vec = sizeof(TW) == 2 && p.ldw % 8 == 0 && ((uintptr_t)p.w & 15) == 0;
    const bool wide = ldl % 4 == 0 && p.col % 4 == 0 && ((uintptr_t)low & 15) == 0;
    float acc[LF_TOK] = {};
    bool ready = false;
#pragma unroll 2
    for (int r = 8 * lane; r < p.rank; r += 64) {
        float x[8];
        if (vec && r + 8 <= p.rank) {
            const uint4 u = *reinterpret_cast<const uint4*>(w + r);
            const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = __bfloat1622float2(b[i]);
                x[2 * i] = f.x, x[2 * i + 1] = f.y;
            }
        } else {
            load_weights<8>(x, w + r, p.rank - r);
        }
        if (!ready) {                                        // the weights are asked for before the rows are there
            pdl_wait();
            ready = true;
        }
#pragma unroll
        for (int t = 0; t < LF_TOK; ++t) {
            if (t >= nt) break;
            const float* y = low + (long long)(t0 + t) * ldl + p.col + r;
            if (wide && r + 8 <= p.rank) {
                const float4 a = *reinterpret_cast<const float4*>(y), b = *reinterpret_cast<const float4*>(y + 4);
                acc[t] = fmaf(x[0], a.x, fmaf(x[1], a.y, fmaf(x[2], a.z, fmaf(x[3], a.w, acc[t]))));
                acc[t] = fmaf(x[4], b.x, fmaf(x[5], b.y, fmaf(x[6], b.z, fmaf(x[7], b.w, acc[t]))));
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    if (r + i < p.rank) acc[t] = fmaf(x[i], y[i], acc[t]);
            }
        }
    }
    if (!ready) pdl_wait();
#pragma unroll
    for (int t = 0; t < LF_TOK; ++t)
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], o);
    const float z = lane == 0 ? acc[0] : lane == 1 ? acc[1] : lane == 2 ? acc[2] : acc[3];
    if (lane >= nt || c >= p.n) return;
    const float rate = p.fn == 2 ? expf(p.a_log[c / p.per_head]) : 0.0f;
    p.out[(long long)(t0 + lane) * p.n + c] = low_rank_fn(z + (p.bias ? p.bias[c] : 0.0f), p, rate);
}

// The same on tensor cores for steps of many tokens with bfloat16 weights: a block takes 64 tokens x 128 channels of one
// part, a warp 16 tokens x 64 channels.  The tokens' rows enter as two bfloat16 terms (rounded, and what the rounding left), so a
// product keeps 16 bits of the row and all of the weight; float32 accumulators.  rank: a multiple of 16.
// The decays for the tensor-core kernel (bfloat16 models): softplus with the fast exponential and logarithm, a series
// where e^-|z| is small (its next term is 3e-9), so that a decay is off by a few of its own roundings; the exact
// functions cost several times the product.
__device__ __forceinline__ float low_rank_fn_fast(float z, const LowRankPart& p, float rate) {
    if (p.fn == 0) return z;
    const float y = p.fn == 1 ? -z : z, e = __expf(-fabsf(y));
    const float tail = e < 0.01f ? e * fmaf(e, fmaf(e, 1.0f / 3.0f, -0.5f), 1.0f) : __logf(1.0f + e);
    if (p.fn == 3) return fmaxf(y, 0.0f) + tail;
    return __expf(-(p.fn == 1 ? p.power : rate) * (fmaxf(y, 0.0f) + tail));
}

constexpr int LM_TOK = 64, LM_CH = 128, LM_PAD = 8, LM_THREADS = 256;

__device__ __forceinline__ void lm_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lm_ldmatrix(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}

__global__ void __launch_bounds__(LM_THREADS)
low_rank_mma_kernel(const float* __restrict__ low, long long ldl, int n_tokens, LowRankPart p0, LowRankPart p1, int blocks0) {
    extern __shared__ __align__(16) unsigned char lm_raw[];  // weights [128][pitch], rows' two terms [64][pitch] each
    pdl_trigger();
    const bool second = (int)blockIdx.y >= blocks0;
    const LowRankPart p = second ? p1 : p0;
    const int c0 = ((int)blockIdx.y - (second ? blocks0 : 0)) * LM_CH, t0 = blockIdx.x * LM_TOK;
    const int pitch = p.rank + LM_PAD;
    __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(lm_raw);
    __nv_bfloat16* hi = ws + LM_CH * pitch;
    __nv_bfloat16* lo = hi + LM_TOK * pitch;
    const int tid = threadIdx.x, warp = (tid >> 5) & 3, half0 = (tid >> 7) * (LM_CH / 2);
    const int lane = tid & 31, gid = lane >> 2, tig = lane & 3;
    // sixteen threads a row, sixteen rows at a time
    const int row0 = tid >> 4, piece0 = tid & 15;
    for (int c = 8 * piece0; c < p.rank; c += 128) {         // (the weights: nothing in flight writes them)
#pragma unroll
        for (int r = row0; r < LM_CH; r += LM_THREADS / 16) {
            const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.w) + (long long)min(c0 + r, p.n - 1) * p.ldw + c;
            *reinterpret_cast<uint4*>(ws + r * pitch + c) = *reinterpret_cast<const uint4*>(src);
        }
    }
    pdl_wait();
    const bool wide = ldl % 4 == 0 && p.col % 4 == 0 && ((uintptr_t)low & 15) == 0;
    for (int c = 4 * piece0; c < p.rank; c += 64) {
#pragma unroll
        for (int r = row0; r < LM_TOK; r += LM_THREADS / 16) {
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (t0 + r < n_tokens) {
                const float* src = low + (long long)(t0 + r) * ldl + p.col + c;
                x = wide ? *reinterpret_cast<const float4*>(src) : make_float4(src[0], src[1], src[2], src[3]);
            }
            const __nv_bfloat162 h0 = __floats2bfloat162_rn(x.x, x.y), h1 = __floats2bfloat162_rn(x.z, x.w);
            __nv_bfloat162* hp = reinterpret_cast<__nv_bfloat162*>(hi + r * pitch + c);
            __nv_bfloat162* lp = reinterpret_cast<__nv_bfloat162*>(lo + r * pitch + c);
            hp[0] = h0, hp[1] = h1;
            lp[0] = __floats2bfloat162_rn(x.x - __low2float(h0), x.y - __high2float(h0));
            lp[1] = __floats2bfloat162_rn(x.z - __low2float(h1), x.w - __high2float(h1));
        }
    }
    __syncthreads();
    float acc[LM_CH / 16][4] = {};
    for (int kk = 0; kk < p.rank; kk += 16) {
        uint32_t ah[4], al[4], bf[4];
        const int arow = (warp * 16 + (lane & 15)) * pitch + kk + (lane >> 4) * 8;
        lm_ldmatrix(ah, hi + arow);
        lm_ldmatrix(al, lo + arow);
#pragma unroll
        for (int j = 0; j < LM_CH / 16; j += 2) {
            lm_ldmatrix(bf, ws + (half0 + j * 8 + (lane & 7) + (lane >> 4) * 8) * pitch + kk + ((lane >> 3) & 1) * 8);
            lm_mma(acc[j], ah, bf[0], bf[1]);
            lm_mma(acc[j], al, bf[0], bf[1]);
            lm_mma(acc[j + 1], ah, bf[2], bf[3]);
            lm_mma(acc[j + 1], al, bf[2], bf[3]);
        }
    }
#pragma unroll
    for (int j = 0; j < LM_CH / 16; ++j) {
        const int c = c0 + half0 + j * 8 + tig * 2;          // this thread's two channels
        if (c >= p.n) continue;
        const bool two = c + 1 < p.n;
        const int d = two ? c + 1 : c;
        const float bias0 = p.bias ? p.bias[c] : 0.0f, bias1 = p.bias ? p.bias[d] : 0.0f;
        const float rate0 = p.fn == 2 ? expf(p.a_log[c / p.per_head]) : 0.0f;
        const float rate1 = p.fn == 2 ? expf(p.a_log[d / p.per_head]) : 0.0f;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = t0 + warp * 16 + gid + 8 * half;
            if (t >= n_tokens) continue;
            const float y0 = low_rank_fn_fast(acc[j][2 * half] + bias0, p, rate0);
            const float y1 = low_rank_fn_fast(acc[j][2 * half + 1] + bias1, p, rate1);
            float* dst = p.out + (long long)t * p.n + c;
            if (two && p.n % 2 == 0) {
                *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
            } else {
                dst[0] = y0;
                if (two) dst[1] = y1;
            }
        }
    }
}

}  // namespace mu

// The largest key size the scan takes.
MU_EXPORT int mu_linear_scan_max_dk() { return mu::LS_MAX_DK; }

// q, k [T][heads * dk], v [T][heads * dv]: float32 slices of rows `ld` apart.  per_channel: decay is [T][heads * dk];
// else [T][heads][4] = (decay, take, -, -), a token's gates `gate_stride` floats after the one's before (0: the same for all).  norm_out (may be null; not with per_channel): [T][heads].  long_steps:
// many tokens a sequence; the launch then waits for an empty device.
MU_EXPORT int mu_linear_scan(const float* q, const float* k, const float* v, long long ld, const float* decay,
                             int per_channel, int n_seqs, int n_heads, int dk, int dv, float scale,
                             const int* seq_first, const int* seq_slots, float* state, long long state_stride,
                             long long state_offset, float* out, long long ldo, float* norm_out, int long_steps,
                             void* stream, long long gate_stride, int silu_rows) {
    if (n_seqs <= 0) return MU_OK;
    if (!q || !k || !v || !decay || !seq_first || !seq_slots || !state || !out || n_heads <= 0 || dk <= 0 || dv <= 0)
        return MU_ERR_BAD_ARGUMENT;
    if (dk > mu::LS_MAX_DK) return MU_ERR_UNSUPPORTED_SIZE;
    if (!per_channel && (((uintptr_t)decay & 15) || gate_stride % 4)) return MU_ERR_ALIGNMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const int cols = dv + (norm_out ? 1 : 0);
    const bool vec = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0 &&
                     (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (per_channel ? (uintptr_t)decay : 0)) & 15) == 0;
#define MU_LINEAR_SCAN_V(R, LANES, V, PC)                                                                             \
    do {                                                                                                              \
        const size_t smem = 2 * sizeof(float) * mu::ls_chunk_floats(LANES * R, mu::ls_columns(LANES), PC);            \
        const dim3 grid(n_seqs, n_heads, (cols + mu::ls_columns(LANES) - 1) / mu::ls_columns(LANES));                 \
        const dim3 block(mu::LS_THREADS);                                                                             \
        auto kernel = mu::linear_scan_kernel<R, LANES, V, PC>;                                                        \
        if (!mu::allow_shared((const void*)kernel, smem)) return MU_ERR_LAUNCH;                                       \
        mu::prefer_shared_memory((const void*)kernel);                                                                \
        if (long_steps)                                                                                               \
            return mu::launch_after(kernel, grid, block, smem, s, q, k, v, ld, decay, n_heads, dk, dv, scale,         \
                                    seq_first, seq_slots, state, state_stride, state_offset, out, ldo, norm_out,      \
                                    gate_stride, silu_rows);                                                          \
        return mu::launch_pdl(kernel, grid, block, smem, s, 1, q, k, v, ld, decay, n_heads, dk, dv, scale, seq_first, \
                              seq_slots, state, state_stride, state_offset, out, ldo, norm_out, gate_stride,          \
                              silu_rows);                                                                             \
    } while (0)
#define MU_LINEAR_SCAN(R, LANES)                                                                                      \
    do {                                                                                                              \
        if (vec && per_channel) MU_LINEAR_SCAN_V(R, LANES, true, true);                                               \
        if (per_channel) MU_LINEAR_SCAN_V(R, LANES, false, true);                                                     \
        if (vec) MU_LINEAR_SCAN_V(R, LANES, true, false);                                                             \
        MU_LINEAR_SCAN_V(R, LANES, false, false);                                                                     \
    } while (0)
    if (dk <= 32) MU_LINEAR_SCAN(4, 8);
    if (dk <= 64) MU_LINEAR_SCAN(4, 16);
    if (dk <= 128) MU_LINEAR_SCAN(4, 32);
    MU_LINEAR_SCAN(8, 32);
#undef MU_LINEAR_SCAN
#undef MU_LINEAR_SCAN_V
}

// i_raw, f_raw: [T][heads] float32 slices of rows `ld` apart; gates: [T][heads][4] = (decay, take, floor, 0).
MU_EXPORT int mu_exp_gates(const float* i_raw, const float* f_raw, long long ld, const float* i_bias,
                           const float* f_bias, float cap, int n_tokens, int n_seqs, int n_heads, const int* seq_first,
                           const int* seq_slots, float* state, long long state_stride, long long m_offset, float* gates,
                           void* stream) {
    if (n_seqs <= 0 || n_tokens <= 0) return MU_OK;
    if (!i_raw || !f_raw || !i_bias || !f_bias || !(cap > 0.0f) || !seq_first || !seq_slots || !state || !gates ||
        n_heads <= 0)
        return MU_ERR_BAD_ARGUMENT;
    if ((uintptr_t)gates & 15) return MU_ERR_ALIGNMENT;
    const dim3 grid(n_seqs, n_heads), block(n_tokens <= 32 * n_seqs ? 32 : 256);
    return mu::launch_pdl(mu::exp_gates_kernel, grid, block, 0, (cudaStream_t)stream, 1, i_raw, f_raw, ld, i_bias, f_bias,
                          cap, n_heads, seq_first, seq_slots, state, state_stride, m_offset, (float4*)gates);
}

// One or two low-rank projections of the same rows `low` (float32, a part's entries from its `col` on): `parts` is an
// array of n_parts.  The weights are bfloat16 or float32.
MU_EXPORT int mu_low_rank(const float* low, long long ldl, int n_tokens, const mu::LowRankPart* parts, int n_parts,
                          int w_bf16, void* stream) {
    if (n_tokens <= 0) return MU_OK;
    if (!low || !parts || n_parts < 1 || n_parts > 2) return MU_ERR_BAD_ARGUMENT;
    int blocks[2] = {0, 0}, rank = 0;
    for (int i = 0; i < n_parts; ++i) {
        const mu::LowRankPart& p = parts[i];
        if (!p.w || !p.out || p.rank <= 0 || p.n <= 0 || p.col < 0 || p.ldw < p.rank || p.fn < 0 || p.fn > 3 ||
            (p.fn == 2 && (!p.a_log || p.per_head <= 0)))
            return MU_ERR_BAD_ARGUMENT;
        blocks[i] = (p.n + mu::LR_CHANNELS - 1) / mu::LR_CHANNELS;
        rank = p.rank > rank ? p.rank : rank;
    }
    const mu::LowRankPart p0 = parts[0], p1 = n_parts > 1 ? parts[1] : parts[0];
    cudaStream_t s = (cudaStream_t)stream;
    // steps of many tokens with weights in whole 16-byte pieces: tensor cores
    bool tc = w_bf16 && n_tokens >= 64;
    for (int i = 0; i < n_parts; ++i)
        tc = tc && parts[i].rank % 16 == 0 && parts[i].rank <= 384 && parts[i].ldw % 8 == 0 && ((uintptr_t)parts[i].w & 15) == 0;
    if (tc) {
        int by[2] = {0, 0};
        for (int i = 0; i < n_parts; ++i) by[i] = (parts[i].n + mu::LM_CH - 1) / mu::LM_CH;
        const size_t bytes = (size_t)(mu::LM_CH + 2 * mu::LM_TOK) * (rank + mu::LM_PAD) * sizeof(__nv_bfloat16);
        if (!mu::allow_shared((const void*)mu::low_rank_mma_kernel, 220 * 1024)) return MU_ERR_LAUNCH;
        return mu::launch_pdl(mu::low_rank_mma_kernel, dim3((n_tokens + mu::LM_TOK - 1) / mu::LM_TOK, by[0] + by[1]),
                              dim3(mu::LM_THREADS),
                              bytes, s, 1, low, ldl, n_tokens, p0, p1, by[0]);
    }
    if (n_tokens < 64) {
        int by[2] = {0, 0};
        for (int i = 0; i < n_parts; ++i) by[i] = (parts[i].n + mu::LF_CHANNELS - 1) / mu::LF_CHANNELS;
        const dim3 few((n_tokens + mu::LF_TOK - 1) / mu::LF_TOK, by[0] + by[1]), threads(mu::LF_THREADS);
        if (w_bf16)
            return mu::launch_pdl(mu::low_rank_few_kernel<__nv_bfloat16>, few, threads, 0, s, 1, low, ldl, n_tokens, p0, p1, by[0]);
        return mu::launch_pdl(mu::low_rank_few_kernel<float>, few, threads, 0, s, 1, low, ldl, n_tokens, p0, p1, by[0]);
    }
    const size_t smem = (size_t)mu::LR_TOK * ((rank + 7) / 8 * 8) * sizeof(float);
    if (smem > 48 * 1024) return MU_ERR_UNSUPPORTED_SIZE;
    const dim3 grid((n_tokens + mu::LR_TOK - 1) / mu::LR_TOK, blocks[0] + blocks[1]), block(mu::LR_THREADS);
#define MU_LOW_RANK(T)                                                                                                \
    return mu::launch_pdl(mu::low_rank_kernel<T>, grid, block, smem, s, 1, low, ldl, n_tokens, p0, p1, blocks[0])
    if (w_bf16) MU_LOW_RANK(__nv_bfloat16);
    MU_LOW_RANK(float);
#undef MU_LOW_RANK
}
