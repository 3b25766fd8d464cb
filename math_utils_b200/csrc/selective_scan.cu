// The selective scan of a state-space mixer whose decay differs by channel AND state entry (Mamba; Gu, Dao, "Mamba:
// Linear-Time Sequence Modeling with Selective State Spaces"), with the gate that follows it:
//     S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c x_c B_n,    y_c = (sum_n S[c][n] C_n + D_c x_c) * silu(z_c).
// The state, decays, step sizes, B, C and all sums are float32; x, z and y are in the compute dtype.
//
// A channel's N state entries live in the registers of LPC lanes, NS entries each (pairs dealt to the lanes in turn;
// N <= LPC NS), with their rates A log2(e), so a token costs a lane NS exponentials (the hardware's 2^x), NS multiply-adds
// of the state and NS of the read-out, two entries to a 64-bit register.  Few entries a lane make many warps: a lone
// warp a scheduler would wait for its own exponentials.  Nothing waits for a token's read-out: a lane keeps its partial sums of
// GROUP tokens, which are then added crosswise, after which lane i holds token i's sum.  The step's tokens come 16 (for
// large states 8) at a time: B and C by asynchronous copies in two stages, x, dt and z through registers (read ahead while
// the ones before are worked on), which also carry x and z to the gate.  Tokens past a sequence's end are staged with
// dt = 0, which leaves the state as it is.  The order of every sum is fixed by N alone: a token's result does not depend on
// how the sequence was cut into steps or on the batch.
#include "common.cuh"

#include <math.h>

namespace mu {

constexpr int SS_THREADS = 128;
__host__ __device__ constexpr int ss_channels(int lanes) { return SS_THREADS / lanes; }

__device__ __forceinline__ float exp2_fast(float x) {        // results below 2^-126 are zero
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <typename TE> __device__ __forceinline__ float gated(float v, float z) { return v * z / (1.0f + expf(-z)); }
template <> __device__ __forceinline__ float gated<__nv_bfloat16>(float v, float z) {      // rounded right after
    return __fdividef(v * z, 1.0f + __expf(-z));
}

// SS_CHUNK: tokens staged at a time.  VEC: every pair of a channel's state starts on an 8-byte boundary.
template <typename TE, int LPC, int NS, bool VEC, int SS_CHUNK>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(const TE* __restrict__ x, long long ldx, const TE* __restrict__ z, long long ldz,
                      const float* __restrict__ dt, long long lddt, const float* __restrict__ bc, long long ldbc, int b_at,
                      int c_at, const float* __restrict__ rates, const float* __restrict__ skip, int inner, int N,
                      const int* __restrict__ seq_first, const int* __restrict__ seq_slots, float* __restrict__ state,
                      long long state_stride, long long state_offset, TE* __restrict__ y, long long ldy) {
    constexpr int NPAD = LPC * NS, Q = NS / 2, COLS = ss_channels(LPC), GROUP = LPC < SS_CHUNK ? LPC : SS_CHUNK;
    constexpr int ROWS = SS_THREADS / COLS;                  // tokens of a chunk that are staged at once, a channel a thread
    constexpr int PER = (SS_CHUNK + ROWS - 1) / ROWS;
    constexpr int PIECES = NPAD / 4, COPIES = (SS_CHUNK * PIECES + SS_THREADS - 1) / SS_THREADS;
    __shared__ __align__(16) float Bs[2][SS_CHUNK][NPAD], Cs[2][SS_CHUNK][NPAD];
    __shared__ __align__(16) float2 ds[2][SS_CHUNK][COLS];                   // (dt, dt x)
    __shared__ float ys[SS_CHUNK][COLS];
    const int tid = threadIdx.x, ch = tid / LPC, l = tid % LPC;
    const int s = blockIdx.x, c0 = blockIdx.y * COLS, c = c0 + ch;
    const int n4 = (N + 3) & ~3;
    for (int i = tid; i < 2 * SS_CHUNK * NPAD; i += SS_THREADS) {
        (&Bs[0][0][0])[i] = 0.0f;
        (&Cs[0][0][0])[i] = 0.0f;
    }
    // the rates do not depend on the launches before this one
    float2x A[Q], S[Q];
    const bool live = c < inner;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 2 * (l + LPC * q);
        const float a0 = live && n < N ? rates[(long long)c * N + n] : 0.0f;
        const float a1 = live && n + 1 < N ? rates[(long long)c * N + n + 1] : 0.0f;
        A[q] = pair_of_floats(a0, a1);
    }
    // staging: this thread's channel and first token of a chunk
    const int col = c0 + tid % COLS, row = tid / COLS;
    const bool real = col < inner;
    const float d_skip = real ? skip[col] : 0.0f;
    pdl_wait();
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    float* const mine = state + (long long)seq_slots[s] * state_stride + state_offset + (long long)c * N;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 2 * (l + LPC * q);
        float2 v = make_float2(0.0f, 0.0f);
        if (live) {
            if (VEC) {
                if (n < N) v = *reinterpret_cast<const float2*>(mine + n);
            } else {
                if (n < N) v.x = mine[n];
                if (n + 1 < N) v.y = mine[n + 1];
            }
        }
        S[q] = pair_of_floats(v.x, v.y);
    }
    const long long at = first + row, place = real ? col : inner - 1;
    const TE* xp = x + at * ldx + place;
    const TE* zp = z + at * ldz + place;
    const float* dp = dt + at * lddt + place;
    TE* yp = y + at * ldy + place;
    auto copy_bc = [&](int li0, int b) {
        const float* from = bc + (long long)(first + li0) * ldbc;
#pragma unroll
        for (int k = 0; k < COPIES; ++k) {
            const int i = tid + SS_THREADS * k, tok = i / PIECES, n = 4 * (i % PIECES);
            if (tok < SS_CHUNK && li0 + tok < count && n < n4) {
                copy_async16(&Bs[b][tok][n], from + tok * ldbc + b_at + n);
                copy_async16(&Cs[b][tok][n], from + tok * ldbc + c_at + n);
            }
        }
        copy_async_commit();
    };
    // (rows are read as they are, from places that always exist: nothing may wait for a load before all are on their way)
    TE xr[PER], zr[PER];
    float dr[PER], gate_x[PER], gate_z[PER];
    auto read_rows = [&](int li0) {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int li = min(li0 + row + ROWS * k, count - 1) - row;           // (pointers stand at the step's row-th token)
            xr[k] = xp[li * ldx];
            dr[k] = dp[li * lddt];
            zr[k] = zp[li * ldz];
        }
    };
    auto stage_rows = [&](int li0, int b) {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int tok = row + ROWS * k;
            const float step = li0 + tok < count ? dr[k] : 0.0f;
            gate_x[k] = to_float(xr[k]);
            gate_z[k] = to_float(zr[k]);
            if (tok < SS_CHUNK) ds[b][tok][tid % COLS] = make_float2(step, step * gate_x[k]);
        }
    };
    __syncthreads();                                         // the zeros are down before the first copies land
    if (count > 0) {
        copy_bc(0, 0);
        read_rows(0);
        stage_rows(0, 0);
    }
    int b = 0;
    for (int li0 = 0; li0 < count; li0 += SS_CHUNK, b ^= 1) {
        const int n = min(SS_CHUNK, count - li0);
        const bool more = li0 + SS_CHUNK < count;
        if (more) {
            copy_bc(li0 + SS_CHUNK, b ^ 1);
            read_rows(li0 + SS_CHUNK);
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        for (int t0 = 0; t0 < n; t0 += GROUP) {
            float acc[GROUP];
#pragma unroll
            for (int i = 0; i < GROUP; ++i) {
                const float2 d = ds[b][t0 + i][ch];
                const float2x d2 = pair_of_floats(d.x, d.x), x2 = pair_of_floats(d.y, d.y);
                float2x a = 0;                               // (two zeros)
#pragma unroll
                for (int q = 0; q < Q; ++q) {
                    const float2x bb = *reinterpret_cast<const float2x*>(&Bs[b][t0 + i][2 * (l + LPC * q)]);
                    const float2x cc = *reinterpret_cast<const float2x*>(&Cs[b][t0 + i][2 * (l + LPC * q)]);
                    const float2 e = floats_of_pair(pair_mul(d2, A[q]));
                    S[q] = pair_fma(pair_of_floats(exp2_fast(e.x), exp2_fast(e.y)), S[q], pair_mul(x2, bb));
                    a = pair_fma(S[q], cc, a);
                }
                const float2 sum = floats_of_pair(a);
                acc[i] = sum.x + sum.y;
            }
#pragma unroll
            for (int width = LPC / 2; width >= GROUP; width >>= 1) {
#pragma unroll
                for (int i = 0; i < GROUP; ++i) acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], width);
            }
#pragma unroll
            for (int width = GROUP / 2; width >= 1; width >>= 1) {
#pragma unroll
                for (int i = 0; i < width; ++i) {
                    const bool upper = (l & width) != 0;
                    const float send = upper ? acc[i] : acc[i + width];
                    const float keep = upper ? acc[i + width] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, width);
                }
            }
            if (l < GROUP) ys[t0 + l][ch] = acc[0];
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int tok = row + ROWS * k;
            if (tok < n && real)
                yp[(li0 + ROWS * k) * ldy] = from_float<TE>(gated<TE>(fmaf(d_skip, gate_x[k], ys[tok][tid % COLS]), gate_z[k]));
        }
        if (more) stage_rows(li0 + SS_CHUNK, b ^ 1);
    }
    pdl_trigger();
    if (!live) return;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 2 * (l + LPC * q);
        const float2 v = floats_of_pair(S[q]);
        if (VEC) {
            if (n < N) *reinterpret_cast<float2*>(mine + n) = v;
        } else {
            if (n < N) mine[n] = v.x;
            if (n + 1 < N) mine[n + 1] = v.y;
        }
    }
}

}  // namespace mu

// The largest state size per channel that the scan takes.
MU_EXPORT int mu_selective_scan_max_state() { return 256; }

// x, z, y [T][inner] views (compute dtype), dt [T][inner] float32; bc float32 rows with B from column b_at and C from
// c_at on (N rounded up to four entries each, 16-byte aligned); rates [inner][N] = A log2(e).  State of a slot from
// state_offset on: [inner][N].  long_steps: many tokens a sequence; the launch then waits for an empty device.
MU_EXPORT int mu_selective_scan(const void* x, long long ldx, const void* z, long long ldz, const float* dt, long long lddt,
                                const float* bc, long long ldbc, int b_at, int c_at, const float* rates, const float* skip,
                                int n_seqs, int inner, int N, const int* seq_first, const int* seq_slots, float* state,
                                long long state_stride, long long state_offset, void* y, long long ldy, int is_bf16,
                                int long_steps, void* stream) {
    if (n_seqs <= 0) return MU_OK;
    if (!x || !z || !dt || !bc || !rates || !skip || !seq_first || !seq_slots || !state || !y || inner <= 0 || N <= 0 ||
        b_at < 0 || c_at < 0)
        return MU_ERR_BAD_ARGUMENT;
    if (N > 256) return MU_ERR_UNSUPPORTED_SIZE;
    if (b_at % 4 || c_at % 4 || ldbc % 4 || ((uintptr_t)bc & 15)) return MU_ERR_ALIGNMENT;
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
    const bool vec = N % 2 == 0 && state_stride % 2 == 0 && state_offset % 2 == 0 && ((uintptr_t)state & 7) == 0;
#define MU_SELECTIVE_V(TE, LPC, NS, V)                                                                                 \
    do {                                                                                                               \
        const dim3 grid(n_seqs, (inner + mu::ss_channels(LPC) - 1) / mu::ss_channels(LPC)), block(mu::SS_THREADS);     \
        auto kernel = mu::selective_scan_kernel<TE, LPC, NS, V, NS <= 4 ? 16 : 8>;                                                       \
        if (long_steps)                                                                                                \
            return mu::launch_after(kernel, grid, block, 0, s, (const TE*)x, ldx, (const TE*)z, ldz, dt, lddt, bc,     \
                                    ldbc, b_at, c_at, rates, skip, inner, N, seq_first, seq_slots, state,              \
                                    state_stride, state_offset, (TE*)y, ldy);                                          \
        return mu::launch_pdl(kernel, grid, block, 0, s, 1, (const TE*)x, ldx, (const TE*)z, ldz, dt, lddt, bc, ldbc,  \
                              b_at, c_at, rates, skip, inner, N, seq_first, seq_slots, state, state_stride,            \
                              state_offset, (TE*)y, ldy);                                                              \
    } while (0)
#define MU_SELECTIVE(LPC, NS)                                                                                          \
    do {                                                                                                               \
        if (is_bf16 && vec) MU_SELECTIVE_V(bf, LPC, NS, true);                                                         \
        if (is_bf16) MU_SELECTIVE_V(bf, LPC, NS, false);                                                               \
        if (vec) MU_SELECTIVE_V(float, LPC, NS, true);                                                                 \
        MU_SELECTIVE_V(float, LPC, NS, false);                                                                         \
    } while (0)
    if (N <= 8) MU_SELECTIVE(4, 2);
    if (N <= 16) MU_SELECTIVE(8, 2);
    if (N <= 32) MU_SELECTIVE(16, 2);
    if (N <= 64) MU_SELECTIVE(32, 2);
    if (N <= 128) MU_SELECTIVE(32, 4);
    MU_SELECTIVE(32, 8);
#undef MU_SELECTIVE
#undef MU_SELECTIVE_V
}
