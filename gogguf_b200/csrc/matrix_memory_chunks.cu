// The matrix memory of matrix_memory.cu for prompts of the 16-bit path: chunks of MC_PC tokens, every (chunk, head) a CTA
// of its own, on the tensor cores (mma.sync m16n8k16, float32 accumulation), in three kernels.
//
// With i, j counting a chunk's tokens from 0, F_i the sum of the log forget gates up to i and b_j = i_j - F_j, the weight
// that token j's k v^T has in token i's memory is e^(F_i + b_j), so with M_i = max(m_in, max_(j <= i) b_j) (m_in the
// running maximum before the chunk) the maximum is m_i = F_i + M_i and
//     o_i ~ e^(m_in - M_i) S_in^T q_i + sum_(j <= i) e^(b_j - M_i) (q_i . k_j) v_j            n_i . q_i alike with n_in and 1
//   1. what a chunk adds:   U = sum_j e^(b_j - B) k_j v_j^T,  u = sum_j e^(b_j - B) k_j,  B = max_j b_j;  F = F_(last), F + B
//   2. a walk over a sequence's chunks, in scaled form: S_in and n_in of every chunk (in U's and u's place), m_in, and
//      the state after the last one
//   3. the outputs of a chunk, with the norm over the head, the weight and the output gate; the last chunk's CTA leaves m
// No exponent is ever positive.  q, k and v are exact as they come (bfloat16); what is float32 (the weighted v, the weights
// of a chunk, the state) enters its product as two bfloat16 terms, the rounded number and the rounded rest, so a product
// loses 2^-17 of a term.  Sums run in an order that depends on the chunk alone.  d and dv multiples of 8 up to 128.
#include "common.cuh"

#define MC_PC 64
#define MC_DEN_EPS 1e-6f

namespace {

__device__ __forceinline__ float mc_in_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mc_log_forget(float z, float cap) {
    const float u = cap * tanhf(z / cap);
    return fminf(u, 0.f) - log1pf(expf(-fabsf(u)));
}
__device__ __forceinline__ void mc_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mc_ldsm(uint32_t* r, const bf16* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void mc_ldsm_t(uint32_t* r, const bf16* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
// two numbers as two pairs of bfloat16: the rounded numbers and the rounded rests
__device__ __forceinline__ void mc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

__device__ __forceinline__ bool mc_find_chunk(int item, const int* cu_seqlens, const int* seq_of_token, int n_seqs, int& b, int& t0,
                                              int& n, bool& last) {
    for (int i = 0; i < n_seqs; ++i) {
        const int a = cu_seqlens[i], e = cu_seqlens[i + 1];
        if (e <= a || seq_of_token[a] < 0) continue;
        const int nc = (e - a + MC_PC - 1) / MC_PC;
        if (item < nc) { b = i; t0 = a + item * MC_PC; n = min(MC_PC, e - t0); last = item == nc - 1; return true; }
        item -= nc;
    }
    return false;
}

// F_i (running sum of the log forget gates) and b_i = i_i - F_i of the chunk's n tokens into shared memory; warp 0 only,
// two tokens a lane.  Tokens that are not there keep F and get b = -inf.
__device__ __forceinline__ void mc_gates(const float* zi, const float* zf, long long ldz, int t0, int n, int h, float cap, float* F,
                                         float* bs) {
    const int lane = threadIdx.x & 31, j0 = 2 * lane, j1 = j0 + 1;
    const float f0 = j0 < n ? mc_log_forget(zf[(size_t)(t0 + j0) * ldz + h], cap) : 0.f;
    const float f1 = j1 < n ? mc_log_forget(zf[(size_t)(t0 + j1) * ldz + h], cap) : 0.f;
    float run = f0 + f1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += v;
    }
    const float F1 = run, F0 = run - f1;
    F[j0] = F0;
    F[j1] = F1;
    bs[j0] = j0 < n ? mc_in_gate(zi[(size_t)(t0 + j0) * ldz + h], cap) - F0 : -INFINITY;
    bs[j1] = j1 < n ? mc_in_gate(zi[(size_t)(t0 + j1) * ldz + h], cap) - F1 : -INFINITY;
}

// n rows of `cols` numbers (a multiple of 8) from row t0 of x, column off, into tile [MC_PC][ld]; the rest up to `pad`
// columns and MC_PC rows is zeros.
__device__ __forceinline__ void mc_stage(const bf16* x, long long ldx, long long off, int t0, int n, int cols, int pad, bf16* tile,
                                         int ld) {
    const int ch = pad / 8;
    for (int idx = threadIdx.x; idx < MC_PC * ch; idx += blockDim.x) {
        const int r = idx / ch, c = (idx - r * ch) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < n && c < cols) v = *reinterpret_cast<const uint4*>(x + (size_t)(t0 + r) * ldx + off + c);
        *reinterpret_cast<uint4*>(tile + r * ld + c) = v;
    }
}

__host__ __device__ constexpr int mc_pad(int n) { return (n + 15) & ~15; }

// 1. U [item][H][d][dv], u [item][H][d], stats [item][H][2] = (F, F + B).  Eight warps, 16 rows of the state each.
template <int DVT>
__global__ void __launch_bounds__(256) memory_chunk_state_kernel(
    const bf16* x, long long ld, int k_off, int v_off, const float* zi, const float* zf, long long ldz, float* U, float* u,
    float* stats, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_of_token, int n_seqs, int H, int d, int dv,
    float cap) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t mc_smem[];
    __shared__ float F[MC_PC], bs[MC_PC], wj[MC_PC];
    int b, t0, n;
    bool last;
    if (!mc_find_chunk(blockIdx.x, cu_seqlens, seq_of_token, n_seqs, b, t0, n, last)) return;
    const int h = blockIdx.y, dp = mc_pad(d), dvp = mc_pad(dv), lk = dp + 8, lv = dvp + 8;
    bf16* Ks = reinterpret_cast<bf16*>(mc_smem);          // [MC_PC][lk]
    bf16* Vh = Ks + MC_PC * lk;                           // [MC_PC][lv]
    bf16* Vl = Vh + MC_PC * lv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp == 0) {
        mc_gates(zi, zf, ldz, t0, n, h, cap, F, bs);
        __syncwarp();
        const float B = warp_max(fmaxf(bs[2 * lane], bs[2 * lane + 1]));
        wj[2 * lane] = expf(bs[2 * lane] - B);
        wj[2 * lane + 1] = expf(bs[2 * lane + 1] - B);
        if (lane == 0) {
            float* st = stats + ((size_t)blockIdx.x * H + h) * 2;
            st[0] = F[MC_PC - 1];
            st[1] = F[MC_PC - 1] + B;
        }
    }
    mc_stage(x, ld, (long long)k_off + (long long)h * d, t0, n, d, dp, Ks, lk);
    __syncthreads();
    const int pairs = dvp / 2;
    for (int idx = threadIdx.x; idx < MC_PC * pairs; idx += blockDim.x) {
        const int r = idx / pairs, c = (idx - r * pairs) * 2;
        float v0 = 0.f, v1 = 0.f;
        if (r < n && c < dv) {
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(x + (size_t)(t0 + r) * ld + v_off + (size_t)h * dv + c);
            v0 = __low2float(v) * wj[r];
            v1 = __high2float(v) * wj[r];
        }
        uint32_t hi, lo;
        mc_split(v0, v1, hi, lo);
        *reinterpret_cast<uint32_t*>(Vh + r * lv + c) = hi;
        *reinterpret_cast<uint32_t*>(Vl + r * lv + c) = lo;
    }
    for (int r = threadIdx.x; r < d; r += blockDim.x) {
        float s = 0.f;
        for (int j = 0; j < n; ++j) s = fmaf(wj[j], __bfloat162float(Ks[j * lk + r]), s);
        u[((size_t)blockIdx.x * H + h) * d + r] = s;
    }
    __syncthreads();
    const int m0 = warp * 16;
    if (m0 >= dp) return;
    float acc[DVT / 8][4];
#pragma unroll
    for (int i = 0; i < DVT / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const int kmax = (n + 15) / 16;
    for (int kk = 0; kk < kmax; ++kk) {
        uint32_t a[4];
        mc_ldsm_t(a, Ks + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * lk + m0 + (((lane >> 3) & 1) << 3));
#pragma unroll
        for (int np = 0; np < DVT / 16; ++np) {
            if (np * 16 < dv) {
                const int at = (kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * lv + np * 16 + ((lane >> 4) << 3);
                uint32_t v[4];
                mc_ldsm_t(v, Vh + at);
                mc_mma(acc[2 * np], a, v[0], v[1]);
                mc_mma(acc[2 * np + 1], a, v[2], v[3]);
                mc_ldsm_t(v, Vl + at);
                mc_mma(acc[2 * np], a, v[0], v[1]);
                mc_mma(acc[2 * np + 1], a, v[2], v[3]);
            }
        }
    }
    float* up = U + ((size_t)blockIdx.x * H + h) * d * dv;
    const int g = lane >> 2, t = lane & 3;
#pragma unroll
    for (int i = 0; i < DVT / 8; ++i) {
        const int c = i * 8 + 2 * t;
        if (i * 8 < dv) {
            if (m0 + g < d) *reinterpret_cast<float2*>(up + (size_t)(m0 + g) * dv + c) = make_float2(acc[i][0], acc[i][1]);
            if (m0 + g + 8 < d) *reinterpret_cast<float2*>(up + (size_t)(m0 + g + 8) * dv + c) = make_float2(acc[i][2], acc[i][3]);
        }
    }
}

// 2. The walk.  grid (sequence, head, blocks of 256 elements of [S | n]); m_state is only read here (every block of a head
// needs the old one): kernel 3 moves it on.
__global__ void __launch_bounds__(256) memory_chunk_walk_kernel(
    float* U, float* u, const float* stats, float* m_in, float* S_state, float* n_state, const float* m_state,
    const int* __restrict__ cu_seqlens, const int* __restrict__ slots, const int* __restrict__ seq_of_token, int H, int d, int dv) {
    pdl_launch();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, e = blockIdx.z * 256 + threadIdx.x;
    const int start = cu_seqlens[s], end = cu_seqlens[s + 1];
    if (e >= d * dv + d || end <= start || seq_of_token[start] < 0) return;
    int k0 = 0;
    for (int i = 0; i < s; ++i) {
        const int a = cu_seqlens[i], z = cu_seqlens[i + 1];
        if (z > a && seq_of_token[a] >= 0) k0 += (z - a + MC_PC - 1) / MC_PC;
    }
    const int nc = (end - start + MC_PC - 1) / MC_PC;
    const bool mat = e < d * dv;
    const size_t step = mat ? (size_t)H * d * dv : (size_t)H * d;
    float* p = mat ? U + ((size_t)k0 * H + h) * d * dv + e : u + ((size_t)k0 * H + h) * d + (e - d * dv);
    const size_t hs = (size_t)slots[s] * H + h;
    float* sp = mat ? S_state + hs * d * dv + e : n_state + hs * d + (e - d * dv);
    float S = *sp, m = m_state[hs];
    const float* st = stats + ((size_t)k0 * H + h) * 2;
    for (int k = 0; k < nc; k += 8) {                     // eight chunks' loads in flight, then the chain
        float a[8], f[8], fb[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (k + i < nc) {
                a[i] = p[(size_t)(k + i) * step];
                f[i] = st[(size_t)(k + i) * H * 2];
                fb[i] = st[(size_t)(k + i) * H * 2 + 1];
            }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (k + i < nc) {
                p[(size_t)(k + i) * step] = S;
                if (e == 0) m_in[(size_t)(k0 + k + i) * H + h] = m;
                const float mn = fmaxf(f[i] + m, fb[i]);
                S = fmaf(expf(f[i] + m - mn), S, expf(fb[i] - mn) * a[i]);
                m = mn;
            }
    }
    *sp = S;
}

// 3. The outputs.  Four warps, 16 of the chunk's rows each; the state comes by in slabs of 64 of its rows.
template <int DVT>
__global__ void __launch_bounds__(128) memory_chunk_out_kernel(
    const bf16* x, long long ld, int q_off, int k_off, int v_off, int g_off, const float* zi, const float* zf, long long ldz, bf16* out,
    const float* Sin, const float* nin, const float* m_in, float* m_state, const int* __restrict__ cu_seqlens,
    const int* __restrict__ slots, const int* __restrict__ seq_of_token, const float* __restrict__ w, int n_seqs, int H, int d, int dv,
    float q_scale, float cap, float eps) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t mc_smem[];
    __shared__ float F[MC_PC], bs[MC_PC], Ms[MC_PC], ns[128];
    int b, t0, n;
    bool last;
    if (!mc_find_chunk(blockIdx.x, cu_seqlens, seq_of_token, n_seqs, b, t0, n, last)) return;
    const int h = blockIdx.y, dp = mc_pad(d), dvp = mc_pad(dv), lk = dp + 8, lv = dvp + 8;
    bf16* Qs = reinterpret_cast<bf16*>(mc_smem);          // [MC_PC][lk]
    bf16* Ks = Qs + MC_PC * lk;                           // [MC_PC][lk]
    bf16* Vs = Ks + MC_PC * lk;                           // [MC_PC][lv]
    bf16* Sh = Vs + MC_PC * lv;                           // [64][lv]
    bf16* Sl = Sh + 64 * lv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const float mi = m_in[(size_t)blockIdx.x * H + h];
    if (warp == 0) {
        mc_gates(zi, zf, ldz, t0, n, h, cap, F, bs);
        __syncwarp();
        float p1 = fmaxf(bs[2 * lane], bs[2 * lane + 1]);             // running maximum of b
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, p1, o);
            if (lane >= o) p1 = fmaxf(p1, v);
        }
        float p0 = __shfl_up_sync(0xffffffffu, p1, 1);
        p0 = lane == 0 ? bs[0] : fmaxf(p0, bs[2 * lane]);
        Ms[2 * lane] = fmaxf(mi, p0);
        Ms[2 * lane + 1] = fmaxf(mi, p1);
        __syncwarp();
        if (last && lane == 0) m_state[(size_t)slots[b] * H + h] = F[n - 1] + Ms[n - 1];
    }
    mc_stage(x, ld, (long long)q_off + (long long)h * d, t0, n, d, dp, Qs, lk);
    mc_stage(x, ld, (long long)k_off + (long long)h * d, t0, n, d, dp, Ks, lk);
    mc_stage(x, ld, (long long)v_off + (long long)h * dv, t0, n, dv, dvp, Vs, lv);
    for (int r = threadIdx.x; r < 128; r += 128) ns[r] = r < d ? nin[((size_t)blockIdx.x * H + h) * d + r] : 0.f;
    const float* S = Sin + ((size_t)blockIdx.x * H + h) * d * dv;
    const int r0 = warp * 16, i0 = r0 + g, i1 = r0 + g + 8;
    float o[DVT / 8][4], nq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < DVT / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    // S_in^T q and n_in . q
    const int quads = dvp / 4;
    for (int s0 = 0; s0 < dp; s0 += 64) {
        const int rows = min(64, dp - s0);
        if (s0) __syncthreads();                          // the slab before is used up
        for (int idx = threadIdx.x; idx < rows * quads; idx += 128) {
            const int r = idx / quads, c = (idx - r * quads) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (s0 + r < d && c < dv) v = *reinterpret_cast<const float4*>(S + (size_t)(s0 + r) * dv + c);
            uint2 hi, lo;
            mc_split(v.x, v.y, hi.x, lo.x);
            mc_split(v.z, v.w, hi.y, lo.y);
            *reinterpret_cast<uint2*>(Sh + r * lv + c) = hi;
            *reinterpret_cast<uint2*>(Sl + r * lv + c) = lo;
        }
        __syncthreads();
        for (int kk = 0; kk < rows / 16; ++kk) {
            uint32_t a[4];
            mc_ldsm(a, Qs + (r0 + (lane & 15)) * lk + s0 + kk * 16 + ((lane >> 4) << 3));
            {   // a tile of eight columns of which the first is n_in
                const float* np = ns + s0 + kk * 16 + 2 * t;
                uint32_t h0 = 0, l0 = 0, h1 = 0, l1 = 0;
                if (g == 0) { mc_split(np[0], np[1], h0, l0); mc_split(np[8], np[9], h1, l1); }
                mc_mma(nq, a, h0, h1);
                mc_mma(nq, a, l0, l1);
            }
#pragma unroll
            for (int np = 0; np < DVT / 16; ++np) {
                if (np * 16 < dv) {
                    const int at = (kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * lv + np * 16 + ((lane >> 4) << 3);
                    uint32_t v[4];
                    mc_ldsm_t(v, Sh + at);
                    mc_mma(o[2 * np], a, v[0], v[1]);
                    mc_mma(o[2 * np + 1], a, v[2], v[3]);
                    mc_ldsm_t(v, Sl + at);
                    mc_mma(o[2 * np], a, v[0], v[1]);
                    mc_mma(o[2 * np + 1], a, v[2], v[3]);
                }
            }
        }
    }
    const float M0 = Ms[i0], M1 = Ms[i1];
    const float f0 = expf(mi - M0) * q_scale, f1 = expf(mi - M1) * q_scale;
#pragma unroll
    for (int i = 0; i < DVT / 8; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
    // column 0 of the tile sits with the quad's first lane
    float den0 = __shfl_sync(0xffffffffu, nq[0], lane & ~3) * f0, den1 = __shfl_sync(0xffffffffu, nq[2], lane & ~3) * f1;
    // the chunk's own tokens: q k^T up to the warp's last row, weighted
    float s[MC_PC / 8][4];
#pragma unroll
    for (int i = 0; i < MC_PC / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    for (int kk = 0; kk < dp / 16; ++kk) {
        uint32_t a[4];
        mc_ldsm(a, Qs + (r0 + (lane & 15)) * lk + kk * 16 + ((lane >> 4) << 3));
#pragma unroll
        for (int np = 0; np < MC_PC / 16; ++np) {
            if (np <= warp) {
                uint32_t k[4];
                mc_ldsm(k, Ks + (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * lk + kk * 16 + (((lane >> 3) & 1) << 3));
                mc_mma(s[2 * np], a, k[0], k[1]);
                mc_mma(s[2 * np + 1], a, k[2], k[3]);
            }
        }
    }
    float l0 = 0.f, l1 = 0.f;
#pragma unroll
    for (int i = 0; i < MC_PC / 8; ++i) {
        if (i <= 2 * warp + 1) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int j = i * 8 + 2 * t + e;
                const float bj = bs[j];
                s[i][e] = j <= i0 ? s[i][e] * q_scale * expf(bj - M0) : 0.f;
                s[i][2 + e] = j <= i1 ? s[i][2 + e] * q_scale * expf(bj - M1) : 0.f;
                l0 += s[i][e];
                l1 += s[i][2 + e];
            }
        }
    }
#pragma unroll
    for (int m = 1; m < 4; m <<= 1) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, m);
        l1 += __shfl_xor_sync(0xffffffffu, l1, m);
    }
    den0 += l0;
    den1 += l1;
#pragma unroll
    for (int kk = 0; kk < MC_PC / 16; ++kk) {
        if (kk <= warp) {
            uint32_t ah[4], al[4];
            mc_split(s[2 * kk][0], s[2 * kk][1], ah[0], al[0]);
            mc_split(s[2 * kk][2], s[2 * kk][3], ah[1], al[1]);
            mc_split(s[2 * kk + 1][0], s[2 * kk + 1][1], ah[2], al[2]);
            mc_split(s[2 * kk + 1][2], s[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
            for (int np = 0; np < DVT / 16; ++np) {
                if (np * 16 < dv) {
                    uint32_t v[4];
                    mc_ldsm_t(v, Vs + (kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * lv + np * 16 + ((lane >> 4) << 3));
                    mc_mma(o[2 * np], ah, v[0], v[1]);
                    mc_mma(o[2 * np + 1], ah, v[2], v[3]);
                    mc_mma(o[2 * np], al, v[0], v[1]);
                    mc_mma(o[2 * np + 1], al, v[2], v[3]);
                }
            }
        }
    }
    // normaliser, norm over the head, weight, output gate
    const float inv0 = 1.0f / (fmaxf(fabsf(den0), expf(-(F[i0] + M0))) + MC_DEN_EPS);
    const float inv1 = 1.0f / (fmaxf(fabsf(den1), expf(-(F[i1] + M1))) + MC_DEN_EPS);
    float q0 = 0.f, q1 = 0.f;
#pragma unroll
    for (int i = 0; i < DVT / 8; ++i) {                  // (columns beyond dv are zeros)
        o[i][0] *= inv0; o[i][1] *= inv0; o[i][2] *= inv1; o[i][3] *= inv1;
        q0 = fmaf(o[i][0], o[i][0], fmaf(o[i][1], o[i][1], q0));
        q1 = fmaf(o[i][2], o[i][2], fmaf(o[i][3], o[i][3], q1));
    }
#pragma unroll
    for (int m = 1; m < 4; m <<= 1) {
        q0 += __shfl_xor_sync(0xffffffffu, q0, m);
        q1 += __shfl_xor_sync(0xffffffffu, q1, m);
    }
    const float n0 = 1.0f / sqrtf(q0 / (float)dv + eps), n1 = 1.0f / sqrtf(q1 / (float)dv + eps);
    const size_t HV = (size_t)H * dv;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int i = half ? i1 : i0;
        if (i >= n) continue;
        const float f = half ? n1 : n0;
        const bf16* gp = x + (size_t)(t0 + i) * ld + g_off + (size_t)h * dv;
        bf16* op = out + (size_t)(t0 + i) * HV + (size_t)h * dv;
#pragma unroll
        for (int k = 0; k < DVT / 8; ++k) {
            if (k * 8 < dv) {
                const int c = k * 8 + 2 * t;
                const __nv_bfloat162 gg = *reinterpret_cast<const __nv_bfloat162*>(gp + c);
                const float2 ww = *reinterpret_cast<const float2*>(w + (size_t)h * dv + c);
                const float a = o[k][2 * half] * f * ww.x / (1.0f + __expf(-__low2float(gg)));
                const float c2 = o[k][2 * half + 1] * f * ww.y / (1.0f + __expf(-__high2float(gg)));
                *reinterpret_cast<__nv_bfloat162*>(op + c) = __floats2bfloat162_rn(a, c2);
            }
        }
    }
}

int mc_smem_state(int d, int dv) { return MC_PC * ((mc_pad(d) + 8) + 2 * (mc_pad(dv) + 8)) * 2; }
int mc_smem_out(int d, int dv) { return (MC_PC * (2 * (mc_pad(d) + 8) + (mc_pad(dv) + 8)) + 2 * 64 * (mc_pad(dv) + 8)) * 2; }

template <int DVT>
int launch_chunks(const bf16* x, long long ld, int q_off, int k_off, int v_off, int g_off, const float* zi, const float* zf,
                  long long ldz, bf16* out, float* S_state, float* n_state, float* m_state, const int* cu_seqlens, const int* slots,
                  const int* seq_of_token, const float* w, int ntok, int n_seqs, int H, int d, int dv, float q_scale, float cap,
                  float eps, float* scratch, cudaStream_t stream) {
    const int chunks = ntok / MC_PC + n_seqs;
    float* U = scratch;
    float* u = U + (size_t)chunks * H * d * dv;
    float* stats = u + (size_t)chunks * H * d;
    float* m_in = stats + (size_t)chunks * H * 2;
    const int sa = mc_smem_state(d, dv), sc = mc_smem_out(d, dv);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(memory_chunk_state_kernel<DVT>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             mc_smem_state(128, DVT));
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(memory_chunk_out_kernel<DVT>, cudaFuncAttributeMaxDynamicSharedMemorySize, mc_smem_out(128, DVT));
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    int rc = gg_launch(memory_chunk_state_kernel<DVT>, dim3(chunks, H), dim3(256), sa, stream, 1, x, ld, k_off, v_off, zi, zf, ldz, U, u,
                       stats, cu_seqlens, seq_of_token, n_seqs, H, d, dv, cap);
    if (rc) return rc;
    rc = gg_launch(memory_chunk_walk_kernel, dim3(n_seqs, H, (d * dv + d + 255) / 256), dim3(256), 0, stream, 1, U, u, (const float*)stats,
                   m_in, S_state, n_state, (const float*)m_state, cu_seqlens, slots, seq_of_token, H, d, dv);
    if (rc) return rc;
    return gg_launch(memory_chunk_out_kernel<DVT>, dim3(chunks, H), dim3(128), sc, stream, 1, x, ld, q_off, k_off, v_off, g_off, zi, zf,
                     ldz, out, (const float*)U, (const float*)u, (const float*)m_in, m_state, cu_seqlens, slots, seq_of_token, w, n_seqs, H,
                     d, dv, q_scale, cap, eps);
}

}  // namespace

// The arguments of gg_memory_scan for bfloat16 rows x and out; scratch of (ntok / 64 + n_seqs) * H * (d * dv + d + 3)
// floats.  Padding rows of out are not written: a step that has them does not take this form.
GG_API gg_memory_chunks(const void* x, long long ld, int q_off, int k_off, int v_off, int g_off, const float* zi, const float* zf,
                        long long ldz, void* out, float* S_state, float* n_state, float* m_state, const int* cu_seqlens,
                        const int* slots, const int* seq_of_token, const float* w, int ntok, int n_seqs, int H, int d, int dv,
                        float q_scale, float cap, float eps, float* scratch, cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0) return 0;
    if (H <= 0 || H > 65535 || d <= 0 || dv <= 0 || d > 128 || dv > 128 || (d & 7) || (dv & 7) || !(cap > 0.f) || scratch == nullptr ||
        S_state == nullptr || n_state == nullptr || m_state == nullptr || w == nullptr || zi == nullptr || zf == nullptr)
        return GG_ERR_ARG;
    if ((ld & 7) || ((q_off | k_off | v_off | g_off) & 7) ||
        (((uintptr_t)x | (uintptr_t)out | (uintptr_t)w | (uintptr_t)scratch) & 15))
        return GG_ERR_ARG;
    if (dv <= 64)
        return launch_chunks<64>((const bf16*)x, ld, q_off, k_off, v_off, g_off, zi, zf, ldz, (bf16*)out, S_state, n_state, m_state,
                                 cu_seqlens, slots, seq_of_token, w, ntok, n_seqs, H, d, dv, q_scale, cap, eps, scratch, stream);
    return launch_chunks<128>((const bf16*)x, ld, q_off, k_off, v_off, g_off, zi, zf, ldz, (bf16*)out, S_state, n_state, m_state,
                              cu_seqlens, slots, seq_of_token, w, ntok, n_seqs, H, d, dv, q_scale, cap, eps, scratch, stream);
}
