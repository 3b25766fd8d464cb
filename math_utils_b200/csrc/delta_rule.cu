// The gated delta rule: a recurrent mixer with a matrix state S [dk][dv] per head, token by token.
//
// Per sequence the mixer keeps, in float32,
//     state[slot] = [ conv tail: (taps - 1) x channels, oldest first | S: heads x dv x dk ]
// (a head's S is stored column after column: the dk entries that one value entry reads lie together).  The short
// convolution with silu is mu_ssd_conv's; its float32 output row is [ q: kv heads x dk | k: kv heads x dk |
// v: heads x dv ].  Head h reads the queries and keys of kv head h / (heads / kv_heads).
//
// mu_delta_prepare   per token: every kv head's q and k become unit vectors, x / sqrt(sum x^2 + 1e-6), q also times
//                    q_scale, in place; kq = q . k of the finished vectors; per head beta = sigmoid(b_raw) and
//                    decay = exp(-exp(A_log) * softplus(a_raw + dt_bias)).  Everything float32.
// mu_delta_scan      per (sequence, head, a few columns of S), the step's tokens in order:
//                        S <- decay S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                    Two columns of S (two value entries) live in the registers of up to 16 lanes, two entries to a
//                    64-bit register; a key and a query read from shared memory serve both columns.  A token waits for
//                    one exchange between the lanes only, that of S^T k, made of the state as the token found it:
//                    (decay S)^T k = decay (S^T k).  The read-out of the written state is decay (S^T q) + u (k . q);
//                    nothing waits for it, so the lanes keep their shares of it for as many (token, column) pairs as
//                    there are lanes and add them crosswise.
//                    q, k, v, beta, decay and k . q of 16 tokens at a time are copied to shared memory
//                    asynchronously, the next 16 while these are worked on.
//                    The order of every sum is fixed by the column alone: a token's result does not depend on how
//                    the sequence was cut into steps or on the batch.
//
// Option: a decay per head and key channel instead of one per head (the rows of S decay each by its own number).  The
// decays are then made by mu_low_rank (linear_scan.cu) and staged beside the keys; S decays before the two sums, which
// are S^T k and S^T q of the decayed state, and the read-out is S^T q + u (k . q): one exchange a token again.
#include "common.cuh"

#include <math.h>
#include <stdint.h>

namespace mu {

template <typename TE>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(float* __restrict__ qkv, int channels, const TE* __restrict__ b_raw, long long ldb,
                     const TE* __restrict__ a_raw, long long lda, const float* __restrict__ a_log,
                     const float* __restrict__ dt_bias, int n_heads, int n_kv_heads, int dk, float q_scale,
                     float* __restrict__ kq, float* __restrict__ beta, float* __restrict__ decay) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    float* row = qkv + (long long)t * channels;
    for (int g = warp; g < n_kv_heads; g += warps) {
        float* qv = row + (long long)g * dk;
        float* kv = row + (long long)(n_kv_heads + g) * dk;
        float sq = 0.0f, sk = 0.0f;
        for (int d = lane; d < dk; d += 32) {
            sq = fmaf(qv[d], qv[d], sq);
            sk = fmaf(kv[d], kv[d], sk);
        }
        const float iq = q_scale / sqrtf(warp_sum(sq) + 1e-6f), ik = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
        float dot = 0.0f;
        for (int d = lane; d < dk; d += 32) {
            const float a = qv[d] * iq, b = kv[d] * ik;
            qv[d] = a;
            kv[d] = b;
            dot = fmaf(a, b, dot);
        }
        dot = warp_sum(dot);
        if (lane == 0) kq[(long long)t * n_kv_heads + g] = dot;
    }
    for (int h = tid; h < n_heads; h += blockDim.x) {
        const float b = to_float(b_raw[(long long)t * ldb + h]);
        beta[(long long)t * n_heads + h] = 1.0f / (1.0f + expf(-b));
        if (!a_raw) continue;                                // (decays per channel come from elsewhere)
        const float a = to_float(a_raw[(long long)t * lda + h]);
        decay[(long long)t * n_heads + h] = expf(-expf(a_log[h]) * softplus(a + dt_bias[h]));
    }
}

constexpr int DL_THREADS = 128;
constexpr int DL_PER = 2;         // columns of S whose entries a lane holds
constexpr int DL_CHUNK = 16;      // tokens staged at a time
constexpr int DL_MAX_DK = 256;    // the longest column

// Columns a block takes: LANES lanes share two columns.
__host__ __device__ constexpr int dl_columns(int lanes) { return DL_PER * DL_THREADS / lanes; }
// Floats of one staged chunk: keys, queries (and the channels' decays) padded to DKP entries, the block's values,
// (beta, decay, k . q, -).
__host__ __device__ constexpr int dl_chunk_floats(int dkp, int cols, bool per_channel) {
    return DL_CHUNK * ((per_channel ? 3 : 2) * dkp + cols + 4);
}

// LANES lanes hold two columns of S, R entries of each a lane (a multiple of 4; dk <= LANES R).  The columns are dealt
// to the lanes four entries at a time: lane l holds entries 4 (l + LANES i) .. 4 (l + LANES i) + 3, i < R / 4, so that
// neighbouring lanes read consecutive bytes of a staged key, and what a lane reads serves both of its columns.  LANES
// and R follow from dk alone, so the order of the sums does too.
// VEC: dk, dv, the row length and the state's offset and stride are all multiples of 4, so keys, queries, values and
// the state move 16 bytes at a time.  PER_CHANNEL: `decay` is [T][n_heads * dk] (else [T][n_heads]).
template <int R, int LANES, bool VEC, bool PER_CHANNEL>
__global__ void __launch_bounds__(DL_THREADS, R > 8 ? 2 : 4)
delta_scan_kernel(const float* __restrict__ qkv, int channels, const float* __restrict__ kq,
                  const float* __restrict__ beta, const float* __restrict__ decay, int n_heads, int n_kv_heads, int dk,
                  int dv, const int* __restrict__ seq_first, const int* __restrict__ seq_slots,
                  float* __restrict__ state, long long state_stride, long long state_offset, float* __restrict__ out) {
    constexpr int DKP = LANES * R, Q = R / 4, COLS = dl_columns(LANES), BUF = dl_chunk_floats(DKP, COLS, PER_CHANNEL);
    constexpr int GROUP = LANES / DL_PER;                    // tokens whose read-outs are summed together
    extern __shared__ __align__(16) float dl_smem[];
    const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, c0 = DL_PER * (tid / LANES), l = tid % LANES;
    const int g = h / (n_heads / n_kv_heads);
    const int n_live = min(DL_PER, dv - col0 - c0);          // (may be negative)
    for (int i = tid; i < 2 * BUF; i += DL_THREADS) dl_smem[i] = 0.0f;   // the padding past dk and dv stays zero
    pdl_wait();
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    float* const mine = state + (long long)seq_slots[s] * state_stride + state_offset + ((long long)h * dv + col0 + c0) * dk;
    float2x S[DL_PER][2 * Q];                                // the lane's entries in pairs
#pragma unroll
    for (int c = 0; c < DL_PER; ++c)
#pragma unroll
        for (int i = 0; i < Q; ++i) {
            const int d = 4 * (l + LANES * i);
            const float* col = mine + (long long)c * dk;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (c < n_live) {
                if (VEC) {
                    if (d < dk) x = *reinterpret_cast<const float4*>(col + d);
                } else {
                    if (d < dk) x.x = col[d];
                    if (d + 1 < dk) x.y = col[d + 1];
                    if (d + 2 < dk) x.z = col[d + 2];
                    if (d + 3 < dk) x.w = col[d + 3];
                }
            }
            S[c][2 * i] = pair_of_floats(x.x, x.y);
            S[c][2 * i + 1] = pair_of_floats(x.z, x.w);
        }
    const long long q_off = (long long)g * dk, k_off = (long long)(n_kv_heads + g) * dk;
    const long long v_off = (long long)2 * n_kv_heads * dk + (long long)h * dv + col0;
    // stages the chunk that starts at the sequence's li0-th token of this step into buffer `b`
    auto stage = [&](int li0, int b) {
        float* ks = dl_smem + b * BUF;
        float* qs = ks + DL_CHUNK * DKP;
        float* gs = qs + DL_CHUNK * DKP;
        float* vs = gs + (PER_CHANNEL ? DL_CHUNK * DKP : 0);
        float* sc = vs + DL_CHUNK * COLS;
        const int n = min(DL_CHUNK, count - li0);
        if (VEC) {
            const int per = dk / 4;
            for (int i = tid; i < n * per; i += DL_THREADS) {
                const int tok = i / per, d = 4 * (i % per);
                const float* row = qkv + (long long)(first + li0 + tok) * channels;
                copy_async16(ks + tok * DKP + d, row + k_off + d);
                copy_async16(qs + tok * DKP + d, row + q_off + d);
                if (PER_CHANNEL) copy_async16(gs + tok * DKP + d, decay + ((long long)(first + li0 + tok) * n_heads + h) * dk + d);
            }
            for (int i = tid; i < n * (COLS / 4); i += DL_THREADS) {
                const int tok = i / (COLS / 4), cc = 4 * (i % (COLS / 4));
                if (col0 + cc < dv)
                    copy_async16(vs + tok * COLS + cc, qkv + (long long)(first + li0 + tok) * channels + v_off + cc);
            }
        } else {
            for (int i = tid; i < n * dk; i += DL_THREADS) {
                const int tok = i / dk, d = i % dk;
                const float* row = qkv + (long long)(first + li0 + tok) * channels;
                copy_async4(ks + tok * DKP + d, row + k_off + d);
                copy_async4(qs + tok * DKP + d, row + q_off + d);
                if (PER_CHANNEL) copy_async4(gs + tok * DKP + d, decay + ((long long)(first + li0 + tok) * n_heads + h) * dk + d);
            }
            for (int i = tid; i < n * COLS; i += DL_THREADS) {
                const int tok = i / COLS, cc = i % COLS;
                if (col0 + cc < dv)
                    copy_async4(vs + tok * COLS + cc, qkv + (long long)(first + li0 + tok) * channels + v_off + cc);
            }
        }
        for (int tok = tid; tok < n; tok += DL_THREADS) {
            const long long t = first + li0 + tok;
            copy_async4(sc + tok * 4 + 0, beta + t * n_heads + h);
            if (!PER_CHANNEL) copy_async4(sc + tok * 4 + 1, decay + t * n_heads + h);
            copy_async4(sc + tok * 4 + 2, kq + t * n_kv_heads + g);
        }
        copy_async_commit();
    };
    __syncthreads();                                         // the zeros are down before the first copies land
    if (count > 0) stage(0, 0);
    int b = 0;
    for (int li0 = 0; li0 < count; li0 += DL_CHUNK, b ^= 1) {
        const int n = min(DL_CHUNK, count - li0);
        if (li0 + DL_CHUNK < count) {
            stage(li0 + DL_CHUNK, b ^ 1);                    // the next chunk is on its way while this one is worked on
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        const float* ks = dl_smem + b * BUF;
        const float* qs = ks + DL_CHUNK * DKP;
        const float* gs = qs + DL_CHUNK * DKP;
        const float* vs = gs + (PER_CHANNEL ? DL_CHUNK * DKP : 0);
        const float* sc = vs + DL_CHUNK * COLS;
        // One token.  S^T k has to come round the lanes before the state can move on; the read-out need not: the lane's
        // share of it goes to `sum`, u (k . q) into lane 0's.
        auto step = [&](int tok, float* sum) {
            const float4 par = *reinterpret_cast<const float4*>(sc + tok * 4);           // beta, decay, k . q
            const float2 v = *reinterpret_cast<const float2*>(vs + tok * COLS + c0);
            ulonglong2 kr[Q];
            float2x a[DL_PER] = {0, 0}, o[DL_PER] = {0, 0};                              // (two zeros each)
#pragma unroll
            for (int i = 0; i < Q; ++i) {
                const int at = tok * DKP + 4 * (l + LANES * i);
                kr[i] = *reinterpret_cast<const ulonglong2*>(ks + at);
                const ulonglong2 qr = *reinterpret_cast<const ulonglong2*>(qs + at);
                ulonglong2 gr = make_ulonglong2(0, 0);
                if (PER_CHANNEL) gr = *reinterpret_cast<const ulonglong2*>(gs + at);
#pragma unroll
                for (int c = 0; c < DL_PER; ++c) {
                    if (PER_CHANNEL) {
                        S[c][2 * i] = pair_mul(gr.x, S[c][2 * i]);
                        S[c][2 * i + 1] = pair_mul(gr.y, S[c][2 * i + 1]);
                    }
                    a[c] = pair_fma(S[c][2 * i], kr[i].x, a[c]);
                    a[c] = pair_fma(S[c][2 * i + 1], kr[i].y, a[c]);
                    o[c] = pair_fma(S[c][2 * i], qr.x, o[c]);
                    o[c] = pair_fma(S[c][2 * i + 1], qr.y, o[c]);
                }
            }
            float sk[DL_PER];
#pragma unroll
            for (int c = 0; c < DL_PER; ++c) {
                const float2 x = floats_of_pair(a[c]);
                sk[c] = x.x + x.y;
            }
#pragma unroll
            for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
                for (int c = 0; c < DL_PER; ++c) sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], w);
            const float2x dec2 = pair_of_floats(par.y, par.y);
#pragma unroll
            for (int c = 0; c < DL_PER; ++c) {
                // (one decay for the head: the sums are of the state before it, (decay S)^T k = decay (S^T k))
                const float u = par.x * ((c ? v.y : v.x) - (PER_CHANNEL ? sk[c] : par.y * sk[c]));
                const float2x u2 = pair_of_floats(u, u);
#pragma unroll
                for (int i = 0; i < Q; ++i) {
                    S[c][2 * i] = pair_fma(kr[i].x, u2, PER_CHANNEL ? S[c][2 * i] : pair_mul(dec2, S[c][2 * i]));
                    S[c][2 * i + 1] = pair_fma(kr[i].y, u2, PER_CHANNEL ? S[c][2 * i + 1] : pair_mul(dec2, S[c][2 * i + 1]));
                }
                const float2 x = floats_of_pair(o[c]);
                const float share = PER_CHANNEL ? x.x + x.y : par.y * (x.x + x.y);
                sum[c] = l == 0 ? fmaf(u, par.z, share) : share;
            }
        };
        for (int t0 = 0; t0 < n; t0 += GROUP) {
            float acc[LANES];                                // token t0 + i, column c at [2 i + c]
            const int left = n - t0;
            if (left >= GROUP) {                             // a whole group: no branch between the tokens
#pragma unroll
                for (int i = 0; i < GROUP; ++i) step(t0 + i, acc + DL_PER * i);
            } else {
#pragma unroll
                for (int i = 0; i < GROUP; ++i) {
#pragma unroll
                    for (int c = 0; c < DL_PER; ++c) acc[DL_PER * i + c] = 0.0f;
                    if (i < left) step(t0 + i, acc + DL_PER * i);
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
            const int tok = l / DL_PER, c = l % DL_PER;      // what this lane's sum is of
            if (tok < left && c < n_live)
                out[((long long)(first + li0 + t0 + tok) * n_heads + h) * dv + col0 + c0 + c] = acc[0];
        }
        __syncthreads();                                     // this buffer is free for the chunk after the next
    }
    // Only now may the next kernel start: its blocks would wait beside this one's for the whole scan, and a block
    // here has one warp a scheduler, which every waiting warp there slows down.
    pdl_trigger();
#pragma unroll
    for (int c = 0; c < DL_PER; ++c)
#pragma unroll
        for (int i = 0; i < Q; ++i) {
            const int d = 4 * (l + LANES * i);
            const float2 lo = floats_of_pair(S[c][2 * i]), hi = floats_of_pair(S[c][2 * i + 1]);
            if (c >= n_live) continue;
            float* col = mine + (long long)c * dk;
            if (VEC) {
                if (d < dk) *reinterpret_cast<float4*>(col + d) = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
                if (d < dk) col[d] = lo.x;
                if (d + 1 < dk) col[d + 1] = lo.y;
                if (d + 2 < dk) col[d + 2] = hi.x;
                if (d + 3 < dk) col[d + 3] = hi.y;
            }
        }
}

}  // namespace mu

// qkv: the convolution's float32 output rows [T][channels], channels = 2 * kv_heads * dk + heads * dv; q and k are
// finished in place.  b_raw, a_raw: [T][heads] views of the projection, both bfloat16 or both float32; a_raw null: no
// decay per head is made (a_log, dt_bias and decay are not touched).
MU_EXPORT int mu_delta_prepare(float* qkv, int channels, const void* b_raw, long long ldb, const void* a_raw,
                               long long lda, const float* a_log, const float* dt_bias, int n_tokens, int n_heads,
                               int n_kv_heads, int dk, float q_scale, float* kq, float* beta, float* decay,
                               int is_bf16, void* stream) {
    if (n_tokens <= 0) return MU_OK;
    if (!qkv || !b_raw || (a_raw && (!a_log || !dt_bias || !decay)) || !kq || !beta || n_heads <= 0 || n_kv_heads <= 0 ||
        n_heads % n_kv_heads || dk <= 0 || channels < 2 * n_kv_heads * dk)
        return MU_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid(n_tokens), block(128);
    typedef __nv_bfloat16 bf;
    if (is_bf16)
        return mu::launch_pdl(mu::delta_prepare_kernel<bf>, grid, block, 0, s, 1, qkv, channels, (const bf*)b_raw, ldb,
                              (const bf*)a_raw, lda, a_log, dt_bias, n_heads, n_kv_heads, dk, q_scale, kq, beta, decay);
    return mu::launch_pdl(mu::delta_prepare_kernel<float>, grid, block, 0, s, 1, qkv, channels, (const float*)b_raw, ldb,
                          (const float*)a_raw, lda, a_log, dt_bias, n_heads, n_kv_heads, dk, q_scale, kq, beta, decay);
}

// The largest key size the scan takes.
MU_EXPORT int mu_delta_scan_max_dk() { return mu::DL_MAX_DK; }

MU_EXPORT int mu_delta_scan(const float* qkv, int channels, const float* kq, const float* beta, const float* decay,
                            int n_seqs, int n_heads, int n_kv_heads, int dk, int dv, const int* seq_first,
                            const int* seq_slots, float* state, long long state_stride, long long state_offset,
                            float* out, int long_steps, void* stream, int per_channel) {
    if (n_seqs <= 0) return MU_OK;
    if (!qkv || !kq || !beta || !decay || !seq_first || !seq_slots || !state || !out || n_heads <= 0 ||
        n_kv_heads <= 0 || n_heads % n_kv_heads || dk <= 0 || dv <= 0 ||
        channels != 2 * n_kv_heads * dk + n_heads * dv)
        return MU_ERR_BAD_ARGUMENT;
    if (dk > mu::DL_MAX_DK) return MU_ERR_UNSUPPORTED_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = dk % 4 == 0 && dv % 4 == 0 && channels % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(state) |
                      (per_channel ? reinterpret_cast<uintptr_t>(decay) : 0)) % 16 == 0;
    // long_steps: many tokens a sequence (a prompt step).  The blocks then run for a long time with one warp a
    // scheduler; they start in plain stream order, on an empty device.
    // the two staging buffers of a block are most of what it needs of an SM: with the largest share of the on-chip
    // memory as shared memory several blocks fit, and the state is read once, so the L1 is no loss
#define MU_DELTA_SCAN_V(R, LANES, V, PC)                                                                              \
    do {                                                                                                              \
        const size_t smem = 2 * sizeof(float) * mu::dl_chunk_floats(LANES * R, mu::dl_columns(LANES), PC);            \
        const dim3 grid(n_seqs, n_heads, (dv + mu::dl_columns(LANES) - 1) / mu::dl_columns(LANES));                   \
        auto kernel = mu::delta_scan_kernel<R, LANES, V, PC>;                                                         \
        if (!mu::allow_shared((const void*)kernel, smem)) return MU_ERR_LAUNCH;                                       \
        mu::prefer_shared_memory((const void*)kernel);                                                                \
        const dim3 block(mu::DL_THREADS);                                                                             \
        if (long_steps)                                                                                               \
            return mu::launch_after(kernel, grid, block, smem, s, qkv, channels, kq, beta, decay, n_heads,            \
                                    n_kv_heads, dk, dv, seq_first, seq_slots, state, state_stride, state_offset, out); \
        return mu::launch_pdl(kernel, grid, block, smem, s, 1, qkv, channels, kq, beta, decay, n_heads, n_kv_heads,   \
                              dk, dv, seq_first, seq_slots, state, state_stride, state_offset, out);                  \
    } while (0)
#define MU_DELTA_SCAN(R, LANES)                                                                                       \
    do {                                                                                                              \
        if (vec && per_channel) MU_DELTA_SCAN_V(R, LANES, true, true);                                                \
        if (per_channel) MU_DELTA_SCAN_V(R, LANES, false, true);                                                      \
        if (vec) MU_DELTA_SCAN_V(R, LANES, true, false);                                                              \
        MU_DELTA_SCAN_V(R, LANES, false, false);                                                                      \
    } while (0)
    if (dk <= 32) MU_DELTA_SCAN(4, 8);
    if (dk <= 64) MU_DELTA_SCAN(4, 16);
    if (dk <= 128) MU_DELTA_SCAN(8, 16);
    MU_DELTA_SCAN(16, 16);
#undef MU_DELTA_SCAN_V
#undef MU_DELTA_SCAN
}
