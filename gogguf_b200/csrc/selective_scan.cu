// The selective scan: a diagonal state per channel, its decay and its input made from the token.
//
//     dt = softplus(xdt_c)                                                  xdt: a projection with its bias, float32
//     S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x_c B_n,   y_c = sum_n S[c, n] C_n + D_c x_c,   out_c = y_c silu(z_c)
//
// S [inner][N] (float32, zero at a sequence's start) lives in the cache's per-slot state.  x, z, B and C come in the
// compute dtype (columns of wider rows), xdt in float32; everything from there to the store is float32.
//
// A group of L neighbouring lanes owns a channel, a lane SPT of its states in registers; a CTA owns CPB channels and
// walks its rows in tiles of SS_TB tokens.  A tile's numbers are asked for while the tile before is being worked on;
// softplus and dt * x are made once per (token, channel) as a tile is put into shared memory.  Four tokens' partial
// sums are put together by one exchange (each lane ends with one token's), so a token costs fewer shuffles than levels.
//
// phase 0: blockIdx.x is a sequence, walked from the slot's state and into it.  Prompts with few channels are cut into
// chunks, which are independent once their starting states are known: phase 1 runs a chunk from zero and leaves what it
// adds to the state and the sum of its dt (the chunk's decay is exp(A sum dt)), a walk over a sequence's chunks makes
// the starting states, phase 2 runs the chunks again from those and makes the outputs.
#include "common.cuh"

#define SS_TB 16

template <bool FAST> __device__ __forceinline__ float ss_exp2(float x) {
    if (FAST) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
    return exp2f(x);
}
__device__ __forceinline__ float ss_softplus(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.f); }

template <int L> struct SsShape {
    static constexpr int THREADS = L <= 4 ? 128 : (L == 8 ? 256 : 512);
    static constexpr int CPB = THREADS / L;
};

// (sequence, rows) of chunk `item`: chunks are numbered sequence after sequence, padding rows have none
__device__ __forceinline__ bool ss_find_chunk(int item, const int* cu_seqlens, const int* seq_of_token, int n_seqs, int chunk,
                                              int& b, int& start, int& end) {
    for (int i = 0; i < n_seqs; ++i) {
        const int a = cu_seqlens[i], e = cu_seqlens[i + 1];
        if (e <= a || seq_of_token[a] < 0) continue;
        const int nc = (e - a + chunk - 1) / chunk;
        if (item < nc) { b = i; start = a + item * chunk; end = min(start + chunk, e); return true; }
        item -= nc;
    }
    return false;
}

template <typename T, int SPT, int L>
__global__ void __launch_bounds__(SsShape<L>::THREADS) selective_scan_kernel(
    const T* x, long long ldx, const T* z, long long ldz, const T* bc, long long ldbc, int b_off, int c_off, const float* xdt,
    long long lddt, T* out, float* state, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
    const int* __restrict__ seq_of_token, const float* __restrict__ A, const float* __restrict__ D, int inner, int N,
    int n_seqs, int phase, int chunk, float* chunk_state, float* chunk_dt) {
    pdl_launch();
    constexpr bool FAST = sizeof(T) == 2;
    constexpr int THREADS = SsShape<L>::THREADS, CPB = SsShape<L>::CPB, NP = L * SPT;
    constexpr int EPT = (SS_TB * CPB + THREADS - 1) / THREADS;          // (token, channel) elements a thread stages
    constexpr int BPT = (SS_TB * NP + THREADS - 1) / THREADS;           // elements of B (and of C) a thread stages
    __shared__ float2 du[SS_TB][CPB];                                   // dt, dt * x
    __shared__ float ys[SS_TB][CPB + 1];
    __shared__ __align__(16) float Bs[SS_TB][NP];
    __shared__ __align__(16) float Cs[SS_TB][NP];
    const int c0 = blockIdx.y * CPB;
    const int cl = threadIdx.x / L, lane = threadIdx.x % L;             // channel of the block, lane of its group
    const int c = c0 + cl;
    int b = blockIdx.x, start, end;
    if (phase == 0) {
        start = cu_seqlens[b];
        end = cu_seqlens[b + 1];
    } else if (!ss_find_chunk(blockIdx.x, cu_seqlens, seq_of_token, n_seqs, chunk, b, start, end)) {
        pdl_wait();
        return;
    }
    float a2[SPT], S[SPT];
#pragma unroll
    for (int i = 0; i < SPT; ++i) {
        const int n = lane * SPT + i;
        a2[i] = (c < inner && n < N) ? A[(size_t)c * N + n] * 1.4426950408889634f : 0.f;
        S[i] = 0.f;
    }
    pdl_wait();
    if (end <= start) return;
    if (seq_of_token[start] < 0) {                                      // padding rows of a replayed batch
        for (int t = start; t < end; ++t)
            for (int j = threadIdx.x; j < CPB; j += THREADS)
                if (c0 + j < inner) out[(size_t)t * inner + c0 + j] = from_f<T>(0.f);
        return;
    }
    float* sp = phase == 0 ? state + ((size_t)slots[b] * inner + c) * N : chunk_state + ((size_t)blockIdx.x * inner + c) * N;
    if (phase != 1 && c < inner) {
#pragma unroll
        for (int i = 0; i < SPT; ++i)
            if (lane * SPT + i < N) S[i] = sp[lane * SPT + i];
    }
    const bool emit = phase != 1;
    // what a thread stages of a tile, in registers until the tile before is done with shared memory
    float r_dt[EPT], r_x[EPT], r_z[EPT], r_b[BPT], r_c[BPT];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int k = 0; k < EPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / CPB, j = c0 + e % CPB;
            const bool in = tt < SS_TB && t0 + tt < end && j < inner;
            const size_t t = (size_t)(t0 + tt);
            r_dt[k] = in ? xdt[t * lddt + j] : 0.f;
            r_x[k] = in ? to_f<T>(x[t * ldx + j]) : 0.f;
            r_z[k] = (in && emit) ? to_f<T>(z[t * ldz + j]) : 0.f;
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / NP, n = e % NP;
            const bool in = tt < SS_TB && t0 + tt < end && n < N;
            const size_t row = (size_t)(t0 + tt) * ldbc;
            r_b[k] = in ? to_f<T>(bc[row + b_off + n]) : 0.f;
            r_c[k] = in ? to_f<T>(bc[row + c_off + n]) : 0.f;
        }
    };
    fetch(start);
    float dts = 0.f;                                                    // (phase 1) sum of dt of this group's channel
    for (int t0 = start; t0 < end; t0 += SS_TB) {
        const int nb = min(SS_TB, end - t0);
        float o_x[EPT], o_z[EPT];
#pragma unroll
        for (int k = 0; k < EPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / CPB;
            if (tt < nb) {
                const float dt = ss_softplus(r_dt[k]);
                du[tt][e % CPB] = make_float2(dt, dt * r_x[k]);
            } else if (tt < SS_TB) {
                du[tt][e % CPB] = make_float2(0.f, 0.f);                // a row that is not there leaves the state as it is
            }
            o_x[k] = r_x[k];
            o_z[k] = r_z[k];
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / NP;
            if (tt < SS_TB) { Bs[tt][e % NP] = r_b[k]; Cs[tt][e % NP] = r_c[k]; }
        }
        __syncthreads();
        if (t0 + SS_TB < end) fetch(t0 + SS_TB);
#pragma unroll 1
        for (int q0 = 0; q0 < nb; q0 += 4) {
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float2 d = du[q0 + q][cl];
                const float* bp = &Bs[q0 + q][lane * SPT];
                const float* cp = &Cs[q0 + q][lane * SPT];
                float acc = 0.f;
#pragma unroll
                for (int i = 0; i < SPT; ++i) {
                    S[i] = fmaf(ss_exp2<FAST>(d.x * a2[i]), S[i], d.y * bp[i]);
                    acc = fmaf(S[i], cp[i], acc);
                }
                y[q] = acc;
                dts += d.x;
            }
            if (emit) {
                if (L >= 4) {
                    // lanes exchange halves twice: lane (bits 1, 0) = (hi, lo) ends with token 2 hi + lo of the four
                    const bool hi = lane & 2, lo = lane & 1;
                    float s0 = hi ? y[0] : y[2], s1 = hi ? y[1] : y[3];
                    float k0 = hi ? y[2] : y[0], k1 = hi ? y[3] : y[1];
                    k0 += __shfl_xor_sync(0xffffffffu, s0, 2);
                    k1 += __shfl_xor_sync(0xffffffffu, s1, 2);
                    const float s = lo ? k0 : k1;
                    float k = lo ? k1 : k0;
                    k += __shfl_xor_sync(0xffffffffu, s, 1);
#pragma unroll
                    for (int o = 4; o < L; o <<= 1) k += __shfl_xor_sync(0xffffffffu, k, o);
                    if (lane < 4) ys[q0 + lane][cl] = k;
                } else {
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
#pragma unroll
                        for (int o = 1; o < L; o <<= 1) y[q] += __shfl_xor_sync(0xffffffffu, y[q], o);
                        if (lane == 0) ys[q0 + q][cl] = y[q];
                    }
                }
            }
        }
        __syncthreads();
        if (emit) {
#pragma unroll
            for (int k = 0; k < EPT; ++k) {
                const int e = threadIdx.x + k * THREADS, tt = e / CPB, j = e % CPB;
                if (tt < nb && c0 + j < inner) {
                    const float v = fmaf(D[c0 + j], o_x[k], ys[tt][j]), g = o_z[k];
                    out[(size_t)(t0 + tt) * inner + c0 + j] = from_f<T>(v * (g / (1.0f + (FAST ? __expf(-g) : expf(-g)))));
                }
            }
        }
        // (the next round writes du, Bs and Cs, which nobody reads after the barrier above; ys is written again only
        // after that round's first barrier)
    }
    if (phase == 2 || c >= inner) return;
#pragma unroll
    for (int i = 0; i < SPT; ++i)
        if (lane * SPT + i < N) sp[lane * SPT + i] = S[i];
    if (phase == 1 && lane == 0) chunk_dt[(size_t)blockIdx.x * inner + c] = dts;
}

// The walk between the chunked phases: S_in(k + 1) = exp(A sum dt_k) S_in(k) + U_k along a sequence's chunks, from the
// slot's state and into it; every chunk's U is replaced by its S_in.  grid (sequence, ceil(inner N / 256)).
__global__ void __launch_bounds__(256) selective_walk_kernel(float* chunk_state, const float* chunk_dt, float* state,
                                                             const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
                                                             const int* __restrict__ seq_of_token, const float* __restrict__ A,
                                                             int inner, int N, int chunk) {
    pdl_launch();
    pdl_wait();
    const int s = blockIdx.x;
    const long long e = (long long)blockIdx.y * blockDim.x + threadIdx.x, n = (long long)inner * N;
    const int start = cu_seqlens[s], end = cu_seqlens[s + 1];
    if (e >= n || end <= start || seq_of_token[start] < 0) return;
    int k0 = 0;
    for (int i = 0; i < s; ++i) {
        const int a = cu_seqlens[i], z = cu_seqlens[i + 1];
        if (z > a && seq_of_token[a] >= 0) k0 += (z - a + chunk - 1) / chunk;
    }
    const int nc = (end - start + chunk - 1) / chunk, c = (int)(e / N);
    const float a = A[e];
    float* sp = state + (size_t)slots[s] * n + e;
    float S = *sp;
    for (int k = k0; k < k0 + nc; k += 8) {              // eight chunks' loads in flight, then the chain
        float U[8], d[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (k + i < k0 + nc) {
                U[i] = chunk_state[(size_t)(k + i) * n + e];
                d[i] = chunk_dt[(size_t)(k + i) * inner + c];
            }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (k + i < k0 + nc) {
                chunk_state[(size_t)(k + i) * n + e] = S;
                S = fmaf(expf(a * d[i]), S, U[i]);
            }
    }
    *sp = S;
}

// x [T, inner] (rows ldx apart), z alike, B and C at columns b_off and c_off of bc, all in `dtype`; xdt float32; out
// [T, inner] in `dtype`; state [slots][inner][N]; A [inner][N] (negative), D [inner] float32; N <= 256.
// chunk > 0: the three-launch form over chunks of that many rows, with scratch of (ntok / chunk + n_seqs) * inner *
// (N + 1) floats; chunk == 0: every sequence walked whole.
GG_API gg_selective_scan(const void* x, long long ldx, const void* z, long long ldz, const void* bc, long long ldbc, int b_off,
                         int c_off, const float* xdt, long long lddt, void* out, int dtype, float* state, const int* cu_seqlens,
                         const int* slots, const int* seq_of_token, const float* A, const float* D, int ntok, int n_seqs,
                         int inner, int N, int chunk, float* scratch, cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0) return 0;
    if (inner <= 0 || N <= 0 || N > 256 || chunk < 0 || (chunk > 0 && scratch == nullptr) || state == nullptr || A == nullptr ||
        D == nullptr || xdt == nullptr)
        return GG_ERR_ARG;
    const int chunks = chunk ? ntok / chunk + n_seqs : 0;
    float* cs = scratch;
    float* cd = chunk ? scratch + (size_t)chunks * inner * N : nullptr;
#define GG_SS_ONE(T_, S_, L_, items_, phase_)                                                                            \
    gg_launch(selective_scan_kernel<T_, S_, L_>, dim3(items_, (inner + SsShape<L_>::CPB - 1) / SsShape<L_>::CPB),       \
              dim3(SsShape<L_>::THREADS), 0, stream, 1, (const T_*)x, ldx, (const T_*)z, ldz, (const T_*)bc, ldbc, b_off, c_off, \
              xdt, lddt, (T_*)out, state, cu_seqlens, slots, seq_of_token, A, D, inner, N, n_seqs, phase_, chunk, cs, cd)
#define GG_SS(T_, S_, L_)                                                                                                \
    do {                                                                                                                 \
        if ((inner + SsShape<L_>::CPB - 1) / SsShape<L_>::CPB > 65535) return GG_ERR_ARG;                                \
        if (chunk == 0) { GG_SS_ONE(T_, S_, L_, n_seqs, 0); }                                                            \
        else {                                                                                                           \
            GG_SS_ONE(T_, S_, L_, chunks, 1);                                                                            \
            gg_launch(selective_walk_kernel, dim3(n_seqs, (unsigned)(((long long)inner * N + 255) / 256)), dim3(256), 0, stream, 1, \
                      cs, (const float*)cd, state, cu_seqlens, slots, seq_of_token, A, inner, N, chunk);                 \
            GG_SS_ONE(T_, S_, L_, chunks, 2);                                                                            \
        }                                                                                                                \
    } while (0)
    GG_DISPATCH_DTYPE(dtype, T,
        if (N <= 4) GG_SS(T, 4, 1);
        else if (N <= 8) GG_SS(T, 4, 2);
        else if (N <= 16) GG_SS(T, 4, 4);
        else if (N <= 32) GG_SS(T, 4, 8);
        else if (N <= 64) GG_SS(T, 4, 16);
        else if (N <= 128) GG_SS(T, 4, 32);
        else GG_SS(T, 8, 32));
#undef GG_SS
#undef GG_SS_ONE
    return gg_last_error();
}
