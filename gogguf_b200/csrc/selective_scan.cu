// The selective scan: a diagonal state per channel, its decay and its input made from the token.
//
//     dt = softplus(xdt_c)                                                  xdt: a projection with its bias, float32
//     S_cj becomes e^(dt a_cj) S_cj + dt x_c B_j,     out_c = (sum_j S_cj C_j + D_c x_c) silu(z_c)
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
// The same to about 5e-6 of its value, from the hardware's exponential and logarithm: log(1 + e) by its series where e is
// small (there the logarithm of a number near one would lose it).
__device__ __forceinline__ float ss_softplus_fast(float z) {
    const float e = __expf(-fabsf(z));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333334f), -0.5f), 1.0f);
    return (e < 0.03125f ? series : __logf(1.0f + e)) + fmaxf(z, 0.f);
}
// pairs of float32 in one 64-bit register for the packed arithmetic of sm_100
__device__ __forceinline__ unsigned long long ss_pack(float lo, float hi) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void ss_unpack(unsigned long long v, float& lo, float& hi) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ unsigned long long ss_fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ unsigned long long ss_mul2(unsigned long long a, unsigned long long b) {
    unsigned long long d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
// four neighbouring numbers as they come
template <typename T> struct Raw4;
template <> struct Raw4<float> {
    float4 v;
    __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float4*>(p); }
    __device__ __forceinline__ void clear() { v = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ float4 get() const { return v; }
    static __device__ __forceinline__ void store(float* p, float4 a) { *reinterpret_cast<float4*>(p) = a; }
};
template <> struct Raw4<bf16> {
    uint2 v;
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint2*>(p); }
    __device__ __forceinline__ void clear() { v = make_uint2(0u, 0u); }
    __device__ __forceinline__ float4 get() const {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(bf16* p, float4 a) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(a.x, a.y), hi = __floats2bfloat162_rn(a.z, a.w);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    }
};

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

// VEC: channels and states by fours (sizes, offsets and strides are multiples of four, rows on their boundaries).
template <typename T, int SPT, int L, bool EMIT, bool VEC>
__global__ void __launch_bounds__(SsShape<L>::THREADS) selective_scan_kernel(
    const T* x, long long ldx, const T* z, long long ldz, const T* bc, long long ldbc, int b_off, int c_off, const float* xdt,
    long long lddt, T* out, float* state, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
    const int* __restrict__ seq_of_token, const float* __restrict__ A, const float* __restrict__ D, int inner, int N,
    int n_seqs, int phase, int chunk, float* chunk_state, float* chunk_dt) {
    pdl_launch();
    constexpr bool FAST = sizeof(T) == 2;
    constexpr int THREADS = SsShape<L>::THREADS, CPB = SsShape<L>::CPB, NP = L * SPT;
    constexpr int E = VEC ? 4 : 1, CG = CPB / E, NG = NP / E;
    constexpr int EPT = (SS_TB * CG + THREADS - 1) / THREADS;           // (token, channels) elements a thread stages
    constexpr int BPT = (SS_TB * NG + THREADS - 1) / THREADS;           // elements of B (and of C) a thread stages
    static_assert(SPT % 4 == 0 && CPB % 4 == 0, "states and channels come by fours");
    __shared__ __align__(16) float dts[SS_TB][CPB];                     // dt
    __shared__ __align__(16) float us[SS_TB][CPB];                      // dt * x
    __shared__ __align__(16) float ys[SS_TB][CPB + 4];
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
    // what a thread stages of a tile, in registers (as it comes: nothing waits for it yet) until the tile before is done
    // with shared memory
    Raw4<float> v_dt[VEC ? EPT : 1];
    Raw4<T> v_x[VEC ? EPT : 1], v_z[VEC ? EPT : 1], v_b[VEC ? BPT : 1], v_c[VEC ? BPT : 1];
    float s_dt[VEC ? 1 : EPT];
    T s_x[VEC ? 1 : EPT], s_z[VEC ? 1 : EPT], s_b[VEC ? 1 : BPT], s_c[VEC ? 1 : BPT];
    const T zero = from_f<T>(0.f);
    auto fetch = [&](int t0) {
#pragma unroll
        for (int k = 0; k < EPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / CG, j = c0 + E * (e % CG);
            const bool in = tt < SS_TB && t0 + tt < end && j < inner;
            const size_t t = (size_t)(t0 + tt);
            if (VEC) {
                v_dt[k].clear(); v_x[k].clear();
                if (EMIT) v_z[k].clear();
                if (in) {
                    v_dt[k].load(xdt + t * lddt + j);
                    v_x[k].load(x + t * ldx + j);
                    if (EMIT) v_z[k].load(z + t * ldz + j);
                }
            } else {
                s_dt[k] = in ? xdt[t * lddt + j] : 0.f;
                s_x[k] = in ? x[t * ldx + j] : zero;
                if (EMIT) s_z[k] = in ? z[t * ldz + j] : zero;
            }
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / NG, n = E * (e % NG);
            const bool in = tt < SS_TB && t0 + tt < end && n < N;
            const T* row = bc + (size_t)(t0 + tt) * ldbc + n;
            if (VEC) {
                v_b[k].clear();
                if (EMIT) v_c[k].clear();
                if (in) {
                    v_b[k].load(row + b_off);
                    if (EMIT) v_c[k].load(row + c_off);
                }
            } else {
                s_b[k] = in ? row[b_off] : zero;
                if (EMIT) s_c[k] = in ? row[c_off] : zero;
            }
        }
    };
    auto step_size = [&](float v, bool there) { return there ? (FAST ? ss_softplus_fast(v) : ss_softplus(v)) : 0.f; };
    fetch(start);
    float dsum = 0.f;                                                   // (phase 1) sum of dt of this group's channel
    for (int t0 = start; t0 < end; t0 += SS_TB) {
        const int nb = min(SS_TB, end - t0);
        Raw4<T> o_x[VEC ? EPT : 1], o_z[VEC ? EPT : 1];
        T p_x[VEC ? 1 : EPT], p_z[VEC ? 1 : EPT];
#pragma unroll
        for (int k = 0; k < EPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / CG, j = E * (e % CG);
            // (a row that is not there has no step: it leaves the state as it is)
            if (VEC) {
                if (tt < SS_TB) {
                    const float4 r = v_dt[k].get(), xx = v_x[k].get();
                    const bool on = tt < nb;
                    const float4 d = make_float4(step_size(r.x, on), step_size(r.y, on), step_size(r.z, on), step_size(r.w, on));
                    *reinterpret_cast<float4*>(&dts[tt][j]) = d;
                    *reinterpret_cast<float4*>(&us[tt][j]) = make_float4(d.x * xx.x, d.y * xx.y, d.z * xx.z, d.w * xx.w);
                }
                o_x[k] = v_x[k];
                if (EMIT) o_z[k] = v_z[k];
            } else {
                if (tt < SS_TB) {
                    const float d = step_size(s_dt[k], tt < nb);
                    dts[tt][j] = d;
                    us[tt][j] = d * to_f<T>(s_x[k]);
                }
                p_x[k] = s_x[k];
                if (EMIT) p_z[k] = s_z[k];
            }
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int e = threadIdx.x + k * THREADS, tt = e / NG, n = E * (e % NG);
            if (tt < SS_TB) {
                if (VEC) {
                    *reinterpret_cast<float4*>(&Bs[tt][n]) = v_b[k].get();
                    if (EMIT) *reinterpret_cast<float4*>(&Cs[tt][n]) = v_c[k].get();
                } else {
                    Bs[tt][n] = to_f<T>(s_b[k]);
                    if (EMIT) Cs[tt][n] = to_f<T>(s_c[k]);
                }
            }
        }
        __syncthreads();
        if (t0 + SS_TB < end) fetch(t0 + SS_TB);
#pragma unroll 2
        for (int q0 = 0; q0 < nb; q0 += 4) {
            float y[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float dt = dts[q0 + q][cl], u = us[q0 + q][cl];
                const unsigned long long dt2 = ss_pack(dt, dt), u2 = ss_pack(u, u);
                unsigned long long acc = ss_pack(0.f, 0.f);
#pragma unroll
                for (int i = 0; i < SPT; i += 4) {
                    const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(&Bs[q0 + q][lane * SPT + i]);
                    ulonglong2 c4;
                    if (EMIT) c4 = *reinterpret_cast<const ulonglong2*>(&Cs[q0 + q][lane * SPT + i]);
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        float e0, e1;
                        ss_unpack(ss_mul2(dt2, ss_pack(a2[i + 2 * h], a2[i + 2 * h + 1])), e0, e1);
                        const unsigned long long g = ss_pack(ss_exp2<FAST>(e0), ss_exp2<FAST>(e1));
                        const unsigned long long s2 = ss_fma2(g, ss_pack(S[i + 2 * h], S[i + 2 * h + 1]), ss_mul2(u2, h ? b4.y : b4.x));
                        ss_unpack(s2, S[i + 2 * h], S[i + 2 * h + 1]);
                        if (EMIT) acc = ss_fma2(s2, h ? c4.y : c4.x, acc);
                    }
                }
                float a0, a1;
                ss_unpack(acc, a0, a1);
                y[q] = a0 + a1;
                if (!EMIT) dsum += dt;
            }
            if (EMIT) {
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
        if (EMIT) {
            auto finish = [&](float y, float skip, float xv, float g) {
                return fmaf(skip, xv, y) * (g / (1.0f + (FAST ? __expf(-g) : expf(-g))));
            };
#pragma unroll
            for (int k = 0; k < EPT; ++k) {
                const int e = threadIdx.x + k * THREADS, tt = e / CG, j = E * (e % CG);
                if (tt < nb && c0 + j < inner) {
                    T* op = out + (size_t)(t0 + tt) * inner + c0 + j;
                    if (VEC) {
                        const float4 y = *reinterpret_cast<const float4*>(&ys[tt][j]), xx = o_x[k].get(), g = o_z[k].get();
                        const float4 d = __ldg(reinterpret_cast<const float4*>(D + c0 + j));
                        Raw4<T>::store(op, make_float4(finish(y.x, d.x, xx.x, g.x), finish(y.y, d.y, xx.y, g.y),
                                                       finish(y.z, d.z, xx.z, g.z), finish(y.w, d.w, xx.w, g.w)));
                    } else {
                        *op = from_f<T>(finish(ys[tt][j], D[c0 + j], to_f<T>(p_x[k]), to_f<T>(p_z[k])));
                    }
                }
            }
        }
        // (the next round writes dts, us, Bs and Cs, which nobody reads after the barrier above; ys is written again only
        // after that round's first barrier)
    }
    if (phase == 2 || c >= inner) return;
#pragma unroll
    for (int i = 0; i < SPT; ++i)
        if (lane * SPT + i < N) sp[lane * SPT + i] = S[i];
    if (phase == 1 && lane == 0) chunk_dt[(size_t)blockIdx.x * inner + c] = dsum;
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

// A token each: a stream of the states.  A group of L lanes owns a channel, a lane four of its states; what does not change
// while a step runs, and the states, which earlier steps wrote, is asked for before the kernels ahead are waited for.
template <typename T, int L, bool VEC>
__global__ void __launch_bounds__(256) selective_step_kernel(
    const T* x, long long ldx, const T* z, long long ldz, const T* bc, long long ldbc, int b_off, int c_off, const float* xdt,
    long long lddt, T* out, float* state, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
    const int* __restrict__ seq_of_token, const float* __restrict__ A, const float* __restrict__ D, int inner, int N) {
    pdl_launch();
    constexpr int CPB = 256 / L;
    const int b = blockIdx.x, c = blockIdx.y * CPB + threadIdx.x / L, lane = threadIdx.x % L, n0 = lane * 4;
    const int t = cu_seqlens[b];
    const bool there = cu_seqlens[b + 1] > t, live = there && seq_of_token[t] >= 0;
    const bool own = live && c < inner && n0 < N;
    float* sp = state + ((size_t)slots[b] * inner + c) * N + n0;
    float S[4] = {0.f, 0.f, 0.f, 0.f}, a[4] = {0.f, 0.f, 0.f, 0.f};
    if (own) {
        const float* ap = A + (size_t)c * N + n0;
        if (VEC) {
            const float4 s4 = *reinterpret_cast<const float4*>(sp), a4 = __ldg(reinterpret_cast<const float4*>(ap));
            S[0] = s4.x; S[1] = s4.y; S[2] = s4.z; S[3] = s4.w;
            a[0] = a4.x; a[1] = a4.y; a[2] = a4.z; a[3] = a4.w;
        } else {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (n0 + i < N) { S[i] = sp[i]; a[i] = ap[i]; }
        }
    }
    const float skip = own ? D[c] : 0.f;
    pdl_wait();
    if (!there) return;
    float y = 0.f, xv = 0.f, g = 0.f;
    if (own) {
        const T* bp = bc + (size_t)t * ldbc + n0;
        float bb[4], cc[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            bb[i] = n0 + i < N ? to_f<T>(bp[b_off + i]) : 0.f;
            cc[i] = n0 + i < N ? to_f<T>(bp[c_off + i]) : 0.f;
        }
        xv = to_f<T>(x[(size_t)t * ldx + c]);
        g = to_f<T>(z[(size_t)t * ldz + c]);
        const float dt = ss_softplus(xdt[(size_t)t * lddt + c]), u = dt * xv;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            S[i] = fmaf(expf(dt * a[i]), S[i], u * bb[i]);
            y = fmaf(S[i], cc[i], y);
        }
        if (VEC) {
            *reinterpret_cast<float4*>(sp) = make_float4(S[0], S[1], S[2], S[3]);
        } else {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (n0 + i < N) sp[i] = S[i];
        }
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (lane == 0 && c < inner) out[(size_t)t * inner + c] = from_f<T>(live ? fmaf(skip, xv, y) * (g / (1.0f + expf(-g))) : 0.f);
}

// x [T, inner] (rows ldx apart), z alike, B and C at columns b_off and c_off of bc, all in `dtype`; xdt float32; out
// [T, inner] in `dtype`; state [slots][inner][N]; A [inner][N] (negative), D [inner] float32; N <= 256.
// chunk > 0: the three-launch form over chunks of that many rows, with scratch of (ntok / chunk + n_seqs) * inner *
// (N + 1) floats; chunk == 0: every sequence walked whole.  max_new: the most tokens one sequence brings, where the caller
// knows it (1: the form for a token each).
GG_API gg_selective_scan(const void* x, long long ldx, const void* z, long long ldz, const void* bc, long long ldbc, int b_off,
                         int c_off, const float* xdt, long long lddt, void* out, int dtype, float* state, const int* cu_seqlens,
                         const int* slots, const int* seq_of_token, const float* A, const float* D, int ntok, int n_seqs,
                         int inner, int N, int chunk, int max_new, float* scratch, cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0) return 0;
    if (inner <= 0 || N <= 0 || N > 256 || chunk < 0 || (chunk > 0 && scratch == nullptr) || state == nullptr || A == nullptr ||
        D == nullptr || xdt == nullptr)
        return GG_ERR_ARG;
    if (max_new == 1 && N <= 128) {
        const bool vec = N % 4 == 0 && (((uintptr_t)state | (uintptr_t)A) & 15) == 0;
#define GG_STEP(T_, L_, V_)                                                                                              \
    gg_launch(selective_step_kernel<T_, L_, V_>, dim3(n_seqs, (inner + 256 / L_ - 1) / (256 / L_)), dim3(256), 0, stream, 1, \
              (const T_*)x, ldx, (const T_*)z, ldz, (const T_*)bc, ldbc, b_off, c_off, xdt, lddt, (T_*)out, state, cu_seqlens,  \
              slots, seq_of_token, A, D, inner, N)
#define GG_STEP_V(T_, L_) do { if (vec) GG_STEP(T_, L_, true); else GG_STEP(T_, L_, false); } while (0)
        if ((inner + 7) / 8 > 65535) return GG_ERR_ARG;
        GG_DISPATCH_DTYPE(dtype, T,
            if (N <= 4) GG_STEP_V(T, 1);
            else if (N <= 8) GG_STEP_V(T, 2);
            else if (N <= 16) GG_STEP_V(T, 4);
            else if (N <= 32) GG_STEP_V(T, 8);
            else if (N <= 64) GG_STEP_V(T, 16);
            else GG_STEP_V(T, 32));
#undef GG_STEP_V
#undef GG_STEP
        return gg_last_error();
    }
    const uintptr_t el = dtype == GG_BF16 ? 7 : 15;
    const bool vec = ((inner | N | b_off | c_off) & 3) == 0 && ((ldx | ldz | ldbc | lddt) & 3) == 0 &&
                     (((uintptr_t)x | (uintptr_t)z | (uintptr_t)bc | (uintptr_t)out) & el) == 0 &&
                     (((uintptr_t)xdt | (uintptr_t)D) & 15) == 0;
    const int chunks = chunk ? ntok / chunk + n_seqs : 0;
    float* cs = scratch;
    float* cd = chunk ? scratch + (size_t)chunks * inner * N : nullptr;
#define GG_SS_RUN(T_, S_, L_, E_, V_, items_, phase_)                                                                    \
    gg_launch(selective_scan_kernel<T_, S_, L_, E_, V_>, dim3(items_, (inner + SsShape<L_>::CPB - 1) / SsShape<L_>::CPB),       \
              dim3(SsShape<L_>::THREADS), 0, stream, 1, (const T_*)x, ldx, (const T_*)z, ldz, (const T_*)bc, ldbc, b_off, c_off, \
              xdt, lddt, (T_*)out, state, cu_seqlens, slots, seq_of_token, A, D, inner, N, n_seqs, phase_, chunk, cs, cd)
#define GG_SS_ONE(T_, S_, L_, E_, items_, phase_)                                                                        \
    do { if (vec) GG_SS_RUN(T_, S_, L_, E_, true, items_, phase_); else GG_SS_RUN(T_, S_, L_, E_, false, items_, phase_); } while (0)
#define GG_SS(T_, S_, L_)                                                                                                \
    do {                                                                                                                 \
        if ((inner + SsShape<L_>::CPB - 1) / SsShape<L_>::CPB > 65535) return GG_ERR_ARG;                                \
        if (chunk == 0) { GG_SS_ONE(T_, S_, L_, true, n_seqs, 0); }                                                            \
        else {                                                                                                           \
            GG_SS_ONE(T_, S_, L_, false, chunks, 1);                                                                            \
            gg_launch(selective_walk_kernel, dim3(n_seqs, (unsigned)(((long long)inner * N + 255) / 256)), dim3(256), 0, stream, 1, \
                      cs, (const float*)cd, state, cu_seqlens, slots, seq_of_token, A, inner, N, chunk);                 \
            GG_SS_ONE(T_, S_, L_, true, chunks, 2);                                                                            \
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
#undef GG_SS_RUN
    return gg_last_error();
}
