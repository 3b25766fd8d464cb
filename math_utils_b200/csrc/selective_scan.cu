// The selective scan of a state-space mixer whose decay differs by channel AND state entry (Mamba; Gu, Dao, "Mamba:
// Linear-Time Sequence Modeling with Selective State Spaces"), with the gate that follows it:
//     S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c x_c B_n,    y_c = (sum_n S[c][n] C_n + D_c x_c) * silu(z_c).
// The state, decays, step sizes, B, C and all sums are float32; x, z and y are in the compute dtype.
//
// A channel's N state entries live in the registers of LPC lanes, NS entries each (multiples of four; N <= LPC NS),
// with their rates A log2(e), so a token costs a lane NS exponentials (the hardware's 2^x), NS multiply-adds of the
// state and NS of the read-out, two entries to a 64-bit register.  Nothing waits for a token's read-out: a lane keeps
// its partial sums of GROUP tokens, which are then added crosswise, after which lane i holds token i's sum.  The step's tokens
// come 16 (for large states 8) at a time: B and C by asynchronous copies in two stages, x, dt and z through registers (read ahead while the
// ones before are worked on), which also carry x and z to the gate.  Tokens past a sequence's end are staged with
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

// VEC: every channel's state starts on a 16-byte boundary and N is a multiple of four.
template <typename TE> __device__ __forceinline__ float gated(float v, float z) { return v * z / (1.0f + expf(-z)); }
template <> __device__ __forceinline__ float gated<__nv_bfloat16>(float v, float z) {      // rounded right after
    return __fdividef(v * z, 1.0f + __expf(-z));
}

// SS_CHUNK: tokens staged at a time.
template <typename TE, int LPC, int NS, bool VEC, int SS_CHUNK>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(const TE* __restrict__ x, long long ldx, const TE* __restrict__ z, long long ldz,
                      const float* __restrict__ dt, long long lddt, const float* __restrict__ bc, long long ldbc, int b_at,
                      int c_at, const float* __restrict__ rates, const float* __restrict__ skip, int inner, int N,
                      const int* __restrict__ seq_first, const int* __restrict__ seq_slots, float* __restrict__ state,
                      long long state_stride, long long state_offset, TE* __restrict__ y, long long ldy) {
    constexpr int NPAD = LPC * NS, Q = NS / 4, COLS = ss_channels(LPC), GROUP = LPC < SS_CHUNK ? LPC : SS_CHUNK;
    constexpr int PER = (SS_CHUNK * COLS + SS_THREADS - 1) / SS_THREADS;     // (token, channel) pairs of a chunk a thread stages
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
    float2x A[2 * Q], S[2 * Q];
    const bool live = c < inner;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 4 * (l + LPC * q);
        float a[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (live && n + e < N) a[e] = rates[(long long)c * N + n + e];
        A[2 * q] = pair_of_floats(a[0], a[1]);
        A[2 * q + 1] = pair_of_floats(a[2], a[3]);
    }
    pdl_wait();
    const int first = seq_first[s], count = seq_first[s + 1] - first;
    float* const mine = state + (long long)seq_slots[s] * state_stride + state_offset + (long long)c * N;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 4 * (l + LPC * q);
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live) {
            if (VEC) {
                if (n < N) v = *reinterpret_cast<const float4*>(mine + n);
            } else {
                if (n < N) v.x = mine[n];
                if (n + 1 < N) v.y = mine[n + 1];
                if (n + 2 < N) v.z = mine[n + 2];
                if (n + 3 < N) v.w = mine[n + 3];
            }
        }
        S[2 * q] = pair_of_floats(v.x, v.y);
        S[2 * q + 1] = pair_of_floats(v.z, v.w);
    }
    auto copy_bc = [&](int li0, int b) {
        const int pieces = n4 / 4, left = min(SS_CHUNK, count - li0);
        for (int i = tid; i < left * pieces; i += SS_THREADS) {
            const int tok = i / pieces, n = 4 * (i % pieces);
            const float* row = bc + (long long)(first + li0 + tok) * ldbc;
            copy_async16(&Bs[b][tok][n], row + b_at + n);
            copy_async16(&Cs[b][tok][n], row + c_at + n);
        }
        copy_async_commit();
    };
    // (read as they are, from places that always exist: nothing may wait for a load before all are on their way)
    TE xr[PER], zr[PER];
    float dr[PER], gate_x[PER], gate_z[PER];
    auto read_rows = [&](int li0) {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int i = tid + SS_THREADS * k, col = min(c0 + i % COLS, inner - 1);
            const long long t = first + min(li0 + i / COLS, count - 1);
            xr[k] = x[t * ldx + col];
            dr[k] = dt[t * lddt + col];
            zr[k] = z[t * ldz + col];
        }
    };
    auto stage_rows = [&](int li0, int b) {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int i = tid + SS_THREADS * k;
            const float step = li0 + i / COLS < count ? dr[k] : 0.0f;
            gate_x[k] = to_float(xr[k]);
            gate_z[k] = to_float(zr[k]);
            if (i < SS_CHUNK * COLS) ds[b][i / COLS][i % COLS] = make_float2(step, step * gate_x[k]);
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
                float2x a0 = 0, a1 = 0;                      // (two zeros each)
#pragma unroll
                for (int q = 0; q < Q; ++q) {
                    const ulonglong2 bb = *reinterpret_cast<const ulonglong2*>(&Bs[b][t0 + i][4 * (l + LPC * q)]);
                    const ulonglong2 cc = *reinterpret_cast<const ulonglong2*>(&Cs[b][t0 + i][4 * (l + LPC * q)]);
                    const float2 e0 = floats_of_pair(pair_mul(d2, A[2 * q])), e1 = floats_of_pair(pair_mul(d2, A[2 * q + 1]));
                    S[2 * q] = pair_fma(pair_of_floats(exp2_fast(e0.x), exp2_fast(e0.y)), S[2 * q], pair_mul(x2, bb.x));
                    S[2 * q + 1] = pair_fma(pair_of_floats(exp2_fast(e1.x), exp2_fast(e1.y)), S[2 * q + 1], pair_mul(x2, bb.y));
                    a0 = pair_fma(S[2 * q], cc.x, a0);
                    a1 = pair_fma(S[2 * q + 1], cc.y, a1);
                }
                const float2 s0 = floats_of_pair(a0), s1 = floats_of_pair(a1);
                acc[i] = (s0.x + s0.y) + (s1.x + s1.y);
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
            const int i = tid + SS_THREADS * k, tok = i / COLS, col = c0 + i % COLS;
            if (i < SS_CHUNK * COLS && tok < n && col < inner) {
                const float v = fmaf(skip[col], gate_x[k], ys[tok][i % COLS]), zz = gate_z[k];
                y[(long long)(first + li0 + tok) * ldy + col] = from_float<TE>(gated<TE>(v, zz));
            }
        }
        if (more) stage_rows(li0 + SS_CHUNK, b ^ 1);
    }
    pdl_trigger();
    if (!live) return;
#pragma unroll
    for (int q = 0; q < Q; ++q) {
        const int n = 4 * (l + LPC * q);
        const float2 lo = floats_of_pair(S[2 * q]), hi = floats_of_pair(S[2 * q + 1]);
        if (VEC) {
            if (n < N) *reinterpret_cast<float4*>(mine + n) = make_float4(lo.x, lo.y, hi.x, hi.y);
        } else {
            if (n < N) mine[n] = lo.x;
            if (n + 1 < N) mine[n + 1] = lo.y;
            if (n + 2 < N) mine[n + 2] = hi.x;
            if (n + 3 < N) mine[n + 3] = hi.y;
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
    const bool vec = N % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define MU_SELECTIVE_V(TE, LPC, NS, V)                                                                                 \
    do {                                                                                                               \
        const dim3 grid(n_seqs, (inner + mu::ss_channels(LPC) - 1) / mu::ss_channels(LPC)), block(mu::SS_THREADS);     \
        auto kernel = mu::selective_scan_kernel<TE, LPC, NS, V, NS == 4 ? 16 : 8>;                                                       \
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
    if (N <= 8) MU_SELECTIVE(2, 4);
    if (N <= 16) MU_SELECTIVE(4, 4);
    if (N <= 32) MU_SELECTIVE(8, 4);
    if (N <= 64) MU_SELECTIVE(16, 4);
    if (N <= 128) MU_SELECTIVE(32, 4);
    MU_SELECTIVE(32, 8);
#undef MU_SELECTIVE
#undef MU_SELECTIVE_V
}
