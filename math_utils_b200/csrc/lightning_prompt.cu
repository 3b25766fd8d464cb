// Prompt steps of lightning attention (linear attention with one constant decay per head) on tensor cores:
//     S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   q, k, v = silu of the rows given.
// A sequence's tokens of the step are cut into chunks of 64.  With S the state before a chunk of n tokens (numbered
// from 0 within it),
//     o_t = d^(t + 1) S^T q_t + sum_{s <= t} d^(t - s) (q_t . k_s) v_s,
//     S'  = d^n S + sum_s d^(n - 1 - s) k_s v_s^T,
// so all chunks work at once but for the states between them.  Three launches:
//   mu::lightning_sums    per (chunk, head, 64 value columns): U = sum_s d^(n - 1 - s) v_s k_s^T, float32, to scratch.
//   mu::lightning_states  per (sequence, head, 4 entries of S): walks over the chunks' U, leaves in each place the state
//                         before that chunk, and moves the sequence's state on.
//   mu::lightning_outputs per (chunk, head, 64 value columns): the three products of o.
// Products are mma.sync.m16n8k16 with float32 accumulators.  q, k and v enter as bfloat16; everything that carries a
// decay or the state (d^i k, the weights d^(t - s) q . k, S) enters as two bfloat16 terms, so it acts with 16 bits of
// mantissa; the state itself stays float32.  A result depends on where the step's chunks begin only through rounding.
//
// Places in scratch: a chunk's is seq_first[s] / 64 + s + its number within the sequence, which no two chunks share.
#include "mma_sync.cuh"

#include <math.h>

namespace mu {

constexpr int LP_TOK = 64, LP_COLS = 64, LP_PAD = 8, LP_SUM_THREADS = 128, LP_OUT_THREADS = 256;

__device__ __forceinline__ float lp_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// Rows flat0 .. flat0 + count - 1 (zeros up to 64), `width` entries each (zeros up to `padded`), silu applied, into
// `hi` [64][pitch]; with `power`, row r is multiplied by power[count - 1 - r] and goes to `hi` and `lo` in two terms.
template <int THREADS>
__device__ __forceinline__ void lp_stage(__nv_bfloat16* hi, __nv_bfloat16* lo, int pitch, const __nv_bfloat16* src,
                                         long long ld, long long flat0, int count, int width, int padded, const float* power) {
    constexpr int STEP = THREADS / 16, N = LP_TOK / STEP;    // sixteen threads a row
    const int row0 = threadIdx.x >> 4, piece0 = threadIdx.x & 15;
    for (int c = 8 * piece0; c < padded; c += 128) {
        uint4 raw[N];
        const int from = min(c, width - 8);
#pragma unroll
        for (int i = 0; i < N; ++i)
            raw[i] = *reinterpret_cast<const uint4*>(src + (flat0 + min(row0 + STEP * i, count - 1)) * ld + from);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const int r = row0 + STEP * i;
            const bool in = r < count && c < width;
            const float f = power && r < count ? power[count - 1 - r] : 1.0f;
            const __nv_bfloat162* z = reinterpret_cast<const __nv_bfloat162*>(&raw[i]);
            uint32_t h[4], l[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 x = __bfloat1622float2(z[k]);
                const __nv_bfloat162 y = __floats2bfloat162_rn(in ? lp_silu(x.x) : 0.0f, in ? lp_silu(x.y) : 0.0f);
                if (power) split_bf16(f * __low2float(y), f * __high2float(y), h[k], l[k]);
                else h[k] = *reinterpret_cast<const uint32_t*>(&y);
            }
            *reinterpret_cast<uint4*>(hi + r * pitch + c) = make_uint4(h[0], h[1], h[2], h[3]);
            if (power) *reinterpret_cast<uint4*>(lo + r * pitch + c) = make_uint4(l[0], l[1], l[2], l[3]);
        }
    }
}

__device__ __forceinline__ long long lp_place(int flat0, int s, int first) { return first / LP_TOK + s + (flat0 - first) / LP_TOK; }

__global__ void __launch_bounds__(LP_SUM_THREADS)
lightning_sums_kernel(const __nv_bfloat16* __restrict__ k, const __nv_bfloat16* __restrict__ v, long long ld,
                      const int* __restrict__ tiles, const int* __restrict__ tok_seq, const int* __restrict__ seq_first,
                      const float* __restrict__ powers, int n_heads, int dk, int dkp, int dv, float* __restrict__ sums) {
    extern __shared__ __align__(16) unsigned char lp_raw[];
    const int pitch = dkp + LP_PAD, vp = LP_COLS + LP_PAD;
    __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(lp_raw);              // [64][pitch]
    __nv_bfloat16* kl = kh + LP_TOK * pitch;
    __nv_bfloat16* vs = kl + LP_TOK * pitch;                                   // [64][vp]
    pdl_trigger();
    pdl_wait();
    const int flat0 = tiles[2 * blockIdx.x], count = min(tiles[2 * blockIdx.x + 1], LP_TOK);
    const int h = blockIdx.y, col0 = blockIdx.z * LP_COLS, cols = min(LP_COLS, dv - col0);
    const int s = tok_seq[flat0];
    float* dst = sums + (lp_place(flat0, s, seq_first[s]) * n_heads + h) * (long long)dv * dk;
    lp_stage<LP_SUM_THREADS>(kh, kl, pitch, k + (long long)h * dk, ld, flat0, count, dk, dkp, powers + h * (LP_TOK + 1));
    lp_stage<LP_SUM_THREADS>(vs, nullptr, vp, v + (long long)h * dv + col0, ld, flat0, count, cols, LP_COLS, nullptr);
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    // this warp's 16 value columns, as rows of the product: V^T [16 x 64 tokens]
    uint32_t a[LP_TOK / 16][4];
#pragma unroll
    for (int kk = 0; kk < LP_TOK / 16; ++kk)
        ldsm_x4_trans(a[kk], vs + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * vp + warp * 16 + ((lane >> 3) & 1) * 8);
    for (int n0 = 0; n0 < dkp; n0 += 16) {
        float acc[2][4] = {};
#pragma unroll
        for (int kk = 0; kk < LP_TOK / 16; ++kk) {
            uint32_t bh[4], bl[4];
            const int at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + n0 + (lane >> 4) * 8;
            ldsm_x4_trans(bh, kh + at);
            ldsm_x4_trans(bl, kl + at);
            mma_bf16(acc[0], a[kk], bh[0], bh[1]);
            mma_bf16(acc[1], a[kk], bh[2], bh[3]);
            mma_bf16(acc[0], a[kk], bl[0], bl[1]);
            mma_bf16(acc[1], a[kk], bl[2], bl[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int n = n0 + 8 * j + 2 * tig;
            if (n >= dk) continue;
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int col = warp * 16 + gid + 8 * r;
                if (col < cols)
                    *reinterpret_cast<float2*>(dst + (long long)(col0 + col) * dk + n) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
            }
        }
    }
}

constexpr int LP_AHEAD = 8;       // chunks whose sums are on their way at once

__global__ void __launch_bounds__(128)
lightning_states_kernel(float* __restrict__ sums, const int* __restrict__ seq_first, const int* __restrict__ seq_slots,
                        const float* __restrict__ powers, int n_heads, int entries, float* __restrict__ state,
                        long long state_stride, long long state_offset) {
    pdl_trigger();
    pdl_wait();
    const int s = blockIdx.z, h = blockIdx.y, at = 4 * (blockIdx.x * blockDim.x + threadIdx.x);
    if (at >= entries) return;
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    if (count <= 0) return;
    const int chunks = (count + LP_TOK - 1) / LP_TOK;
    const long long step = (long long)n_heads * entries;
    float* u = sums + (lp_place(first, s, first) * n_heads + h) * (long long)entries + at;
    float4* kept = reinterpret_cast<float4*>(state + (long long)seq_slots[s] * state_stride + state_offset + (long long)h * entries + at);
    const float* power = powers + h * (LP_TOK + 1);
    const float whole = power[LP_TOK];
    float4 S = *kept;
    for (int c0 = 0; c0 < chunks; c0 += LP_AHEAD) {
        float4 x[LP_AHEAD];
#pragma unroll
        for (int i = 0; i < LP_AHEAD; ++i) x[i] = *reinterpret_cast<const float4*>(u + min(c0 + i, chunks - 1) * step);
#pragma unroll
        for (int i = 0; i < LP_AHEAD; ++i) {
            if (c0 + i >= chunks) break;
            *reinterpret_cast<float4*>(u + (c0 + i) * step) = S;
            const float d = c0 + i + 1 < chunks ? whole : power[count - LP_TOK * (chunks - 1)];
            S = make_float4(fmaf(d, S.x, x[i].x), fmaf(d, S.y, x[i].y), fmaf(d, S.z, x[i].z), fmaf(d, S.w, x[i].w));
        }
    }
    *kept = S;
}

__global__ void __launch_bounds__(LP_OUT_THREADS, 2)
lightning_outputs_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k,
                         const __nv_bfloat16* __restrict__ v, long long ld, const int* __restrict__ tiles,
                         const int* __restrict__ tok_seq, const int* __restrict__ seq_first, const float* __restrict__ powers,
                         int n_heads, int dk, int dkp, int dv, const float* __restrict__ sums, float* __restrict__ out,
                         long long ldo) {
    extern __shared__ __align__(16) unsigned char lp_raw[];
    __shared__ float power[LP_TOK + 1];
    const int pitch = dkp + LP_PAD, vp = LP_COLS + LP_PAD;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(lp_raw);              // [64][pitch]
    __nv_bfloat16* ks = qs + LP_TOK * pitch;
    __nv_bfloat16* sh = ks + LP_TOK * pitch;                                   // the state's columns, two terms: [64][pitch] each
    __nv_bfloat16* sl = sh + LP_COLS * pitch;
    __nv_bfloat16* vs = sl + LP_COLS * pitch;                                  // [64][vp]
    pdl_trigger();
    pdl_wait();
    const int flat0 = tiles[2 * blockIdx.x], count = min(tiles[2 * blockIdx.x + 1], LP_TOK);
    const int h = blockIdx.y, col0 = blockIdx.z * LP_COLS, cols = min(LP_COLS, dv - col0);
    const int s = tok_seq[flat0];
    const float* S = sums + (lp_place(flat0, s, seq_first[s]) * n_heads + h) * (long long)dv * dk + (long long)col0 * dk;
    if (threadIdx.x <= LP_TOK) power[threadIdx.x] = powers[h * (LP_TOK + 1) + threadIdx.x];
    lp_stage<LP_OUT_THREADS>(qs, nullptr, pitch, q + (long long)h * dk, ld, flat0, count, dk, dkp, nullptr);
    lp_stage<LP_OUT_THREADS>(ks, nullptr, pitch, k + (long long)h * dk, ld, flat0, count, dk, dkp, nullptr);
    lp_stage<LP_OUT_THREADS>(vs, nullptr, vp, v + (long long)h * dv + col0, ld, flat0, count, cols, LP_COLS, nullptr);
    {
        constexpr int STEP = LP_OUT_THREADS / 16, N = LP_COLS / STEP;
        const int row0 = threadIdx.x >> 4, piece0 = threadIdx.x & 15;
        for (int c = 8 * piece0; c < dkp; c += 128) {
            float4 raw[N][2];
            const int from = min(c, dk - 8);
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const float* src = S + (long long)min(row0 + STEP * i, cols - 1) * dk + from;
                raw[i][0] = *reinterpret_cast<const float4*>(src);
                raw[i][1] = *reinterpret_cast<const float4*>(src + 4);
            }
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const int r = row0 + STEP * i;
                const float f = r < cols && c < dk ? 1.0f : 0.0f;
                uint32_t hw[4], lw[4];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    split_bf16(f * raw[i][e].x, f * raw[i][e].y, hw[2 * e], lw[2 * e]);
                    split_bf16(f * raw[i][e].z, f * raw[i][e].w, hw[2 * e + 1], lw[2 * e + 1]);
                }
                *reinterpret_cast<uint4*>(sh + r * pitch + c) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
                *reinterpret_cast<uint4*>(sl + r * pitch + c) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
            }
        }
    }
    __syncthreads();
    // a warp 16 tokens and 32 of the columns
    constexpr int WCOLS = LP_COLS / 2;
    const int warp = (threadIdx.x >> 5) & 3, half0 = (threadIdx.x >> 7) * WCOLS;
    const int lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    if (warp * 16 >= count || half0 >= cols) return;
    const int t0 = warp * 16 + gid;                          // this thread's two tokens: t0 and t0 + 8
    float o[WCOLS / 8][4] = {}, w[LP_TOK / 8][4] = {};
    const int steps = warp + 1;                              // runs of 16 keys that this warp's tokens see
    for (int kk = 0; kk < dkp / 16; ++kk) {
        uint32_t a[4];
        ldsm_x4(a, qs + (warp * 16 + (lane & 15)) * pitch + kk * 16 + (lane >> 4) * 8);
        const int at = ((lane & 7) + (lane >> 4) * 8) * pitch + kk * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int j = 0; j < WCOLS / 16; ++j) {
            uint32_t bh[4], bl[4];
            ldsm_x4(bh, sh + (half0 + j * 16) * pitch + at);
            ldsm_x4(bl, sl + (half0 + j * 16) * pitch + at);
            mma_bf16(o[2 * j], a, bh[0], bh[1]);
            mma_bf16(o[2 * j + 1], a, bh[2], bh[3]);
            mma_bf16(o[2 * j], a, bl[0], bl[1]);
            mma_bf16(o[2 * j + 1], a, bl[2], bl[3]);
        }
#pragma unroll
        for (int j = 0; j < LP_TOK / 16; ++j) {
            if (j >= steps) break;
            uint32_t b[4];
            ldsm_x4(b, ks + j * 16 * pitch + at);
            mma_bf16(w[2 * j], a, b[0], b[1]);
            mma_bf16(w[2 * j + 1], a, b[2], b[3]);
        }
    }
    const float f0 = power[t0 + 1], f1 = power[min(t0 + 9, LP_TOK)];
#pragma unroll
    for (int j = 0; j < WCOLS / 8; ++j) {
        o[j][0] *= f0, o[j][1] *= f0;
        o[j][2] *= f1, o[j][3] *= f1;
    }
#pragma unroll
    for (int kk = 0; kk < LP_TOK / 16; ++kk) {
        if (kk >= steps) break;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int half = 0; half < 2; ++half)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int j = 2 * kk + half, age = t0 + 8 * r - (8 * j + 2 * tig);         // of the thread's first key
                const float p0 = age >= 0 ? w[j][2 * r] * power[max(age, 0)] : 0.0f;
                const float p1 = age >= 1 ? w[j][2 * r + 1] * power[max(age - 1, 0)] : 0.0f;
                split_bf16(p0, p1, ph[2 * half + r], pl[2 * half + r]);
            }
#pragma unroll
        for (int j = 0; j < WCOLS / 16; ++j) {
            uint32_t b[4];
            ldsm_x4_trans(b, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vp + half0 + j * 16 + (lane >> 4) * 8);
            mma_bf16(o[2 * j], ph, b[0], b[1]);
            mma_bf16(o[2 * j + 1], ph, b[2], b[3]);
            mma_bf16(o[2 * j], pl, b[0], b[1]);
            mma_bf16(o[2 * j + 1], pl, b[2], b[3]);
        }
    }
#pragma unroll
    for (int j = 0; j < WCOLS / 8; ++j) {
        const int col = half0 + 8 * j + 2 * tig;
        if (col >= cols) continue;
#pragma unroll
        for (int r = 0; r < 2; ++r)
            if (t0 + 8 * r < count)
                *reinterpret_cast<float2*>(out + (long long)(flat0 + t0 + 8 * r) * ldo + (long long)h * dv + col0 + col) =
                    make_float2(o[j][2 * r], o[j][2 * r + 1]);
    }
}

}  // namespace mu

// Whether mu_lightning_prompt takes these sizes: whole 16-byte pieces of bfloat16 rows.
MU_EXPORT int mu_lightning_prompt_fits(int dk, int dv) { return dk >= 8 && dv >= 8 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256; }

// Floats of scratch for a step of n_tokens tokens of n_seqs sequences.
MU_EXPORT long long mu_lightning_prompt_scratch(int n_tokens, int n_seqs, int n_heads, int dk, int dv) {
    return ((long long)n_tokens / mu::LP_TOK + n_seqs + 1) * n_heads * dk * dv;
}

// q, k [T][heads * dk], v [T][heads * dv]: bfloat16 slices of rows `ld` apart (before silu).  tiles: [n_tiles][2] = (first
// flat token, count <= 64), every sequence cut from its first token of the step on.  powers: [heads][65], decay^0 .. decay^64.
// State of a slot from state_offset on: heads x dv x dk float32.
MU_EXPORT int mu_lightning_prompt(const void* q, const void* k, const void* v, long long ld, const int* tiles, int n_tiles,
                                  const int* tok_seq, int n_seqs, const int* seq_first, const int* seq_slots,
                                  const float* powers, int n_heads, int dk, int dv, float* scratch, float* state,
                                  long long state_stride, long long state_offset, float* out, long long ldo, void* stream) {
    if (n_tiles <= 0 || n_seqs <= 0) return MU_OK;
    if (!q || !k || !v || !tiles || !tok_seq || !seq_first || !seq_slots || !powers || !scratch || !state || !out || n_heads <= 0)
        return MU_ERR_BAD_ARGUMENT;
    if (!mu_lightning_prompt_fits(dk, dv)) return MU_ERR_UNSUPPORTED_SIZE;
    if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)scratch | (uintptr_t)state) & 15 || ((uintptr_t)out & 7) || ld % 8 ||
        ldo % 2 || state_stride % 4 || state_offset % 4)
        return MU_ERR_ALIGNMENT;
    typedef __nv_bfloat16 bf;
    cudaStream_t s = (cudaStream_t)stream;
    const int dkp = (dk + 15) / 16 * 16, pitch = dkp + mu::LP_PAD, vp = mu::LP_COLS + mu::LP_PAD;
    const dim3 grid(n_tiles, n_heads, (dv + mu::LP_COLS - 1) / mu::LP_COLS);
    const size_t smem1 = ((size_t)2 * mu::LP_TOK * pitch + mu::LP_TOK * vp) * sizeof(bf);
    const size_t smem3 = ((size_t)(2 * mu::LP_TOK + 2 * mu::LP_COLS) * pitch + mu::LP_TOK * vp) * sizeof(bf);
    if (!mu::allow_shared((const void*)mu::lightning_sums_kernel, 100 * 1024) ||
        !mu::allow_shared((const void*)mu::lightning_outputs_kernel, 160 * 1024))
        return MU_ERR_LAUNCH;
    mu::prefer_shared_memory((const void*)mu::lightning_sums_kernel);
    mu::prefer_shared_memory((const void*)mu::lightning_outputs_kernel);
    int code = mu::launch_pdl(mu::lightning_sums_kernel, grid, dim3(mu::LP_SUM_THREADS), smem1, s, 1, (const bf*)k, (const bf*)v, ld, tiles, tok_seq,
                              seq_first, powers, n_heads, dk, dkp, dv, scratch);
    if (code != MU_OK) return code;
    const int entries = dk * dv;
    code = mu::launch_pdl(mu::lightning_states_kernel, dim3((entries / 4 + 127) / 128, n_heads, n_seqs), dim3(128), 0, s, 1, scratch,
                          seq_first, seq_slots, powers, n_heads, entries, state, state_stride, state_offset);
    if (code != MU_OK) return code;
    return mu::launch_pdl(mu::lightning_outputs_kernel, grid, dim3(mu::LP_OUT_THREADS), smem3, s, 1, (const bf*)q, (const bf*)k,
                          (const bf*)v, ld, tiles, tok_seq, seq_first, powers, n_heads, dk, dkp, dv, (const float*)scratch, out, ldo);
}
