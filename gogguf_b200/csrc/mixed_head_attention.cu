// Attention whose heads' weights are mixed before they meet the values ("talking heads" after the softmax), over the
// paged cache.
//
//   s_h(i, j) = cap tanh(scale tau(i) q_h,i . k_g(h),j / cap)         cap 0: the score itself;  tau(i): see below
//   p_h(i, j) = exp(s_h(i, j)) / (one + sum over the seen j of exp(s_h(i, j)))          one: 0 or 1
//   o_h(i)    = gate_h(i) sum_j ( sum_g T[h, g] p_g(i, j) ) v_g(h),j
//
// Query head h reads kv head g(h) = h / (H / G).  tau(i) = 1 + coef log(1 + floor((pos_i + 1) / every)) is the query
// temperature (coef 0: none).  gate_h(i) = sigmoid of a logit per token and head (null: no gate).  The mix is linear
// in the weights, so it may also be applied to the heads' results on every kv head's values:
//
//   u_g,G'(i) = sum_j p_g(i, j) v_G',j        o_h(i) = gate_h(i) sum_g T[h, g] u_g,g(h)(i)
//
// which is what the tensor-core form does: a head's softmax is finished before its weights leave the kernel, and the
// mixing works on H x G vectors per token instead of H weights per key.
//
// A token's projection row holds q [H][d], k [G][d], v [G][dv], then H gate logits; the kernels read it in place.
#include "common.cuh"

// ----------------------------------------------------------------------------- keys and values into the cache
// k goes into the pool as it is.  v: each head's run of dv is divided by its root mean square (unit != 0), then mixed
// with the step's first such layer's values, v <- v + lambda (first - v), where `first` is given and `keep` is
// null; with `keep` the layer is the first one and leaves its values there ([T][G][dv] float32).
template <typename T>
__global__ void __launch_bounds__(128) head_kv_prep_kernel(const T* row, long long ld, int k_off, int v_off, T* k_pool,
                                                           T* v_pool, const int* __restrict__ positions,
                                                           const int* __restrict__ seq_of_token,
                                                           const int* __restrict__ page_table, int max_pages, int page_size,
                                                           int G, int d, int dv, int unit, float eps, const float* first,
                                                           float lambda, float* keep, const PageBounds pb) {
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x;
    const int b = seq_of_token[t];
    if (b < 0) return;
    const int pos = positions[t];
    const int page = gg_page_w(page_table + (size_t)b * max_pages, pos / page_size, max_pages, pb, 52);
    const int slot = pos % page_size;
    const T* src = row + (size_t)t * ld;
    if (page >= 0) {
        for (int idx = threadIdx.x; idx < G * d; idx += blockDim.x) {
            const int g = idx / d, i = idx - g * d;
            k_pool[(((size_t)page * G + g) * page_size + slot) * d + i] = src[k_off + idx];
        }
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    for (int g = warp; g < G; g += nwarps) {
        const T* vs = src + v_off + (size_t)g * dv;
        float f = 1.f;
        if (unit) {
            float ss = 0.f;
            for (int i = lane; i < dv; i += 32) { const float v = to_f<T>(vs[i]); ss = fmaf(v, v, ss); }
            ss = warp_sum(ss);
            f = 1.0f / sqrtf(ss / (float)dv + eps);
        }
        const size_t at = ((size_t)t * G + g) * dv;
        for (int i = lane; i < dv; i += 32) {
            float v = to_f<T>(vs[i]) * f;
            if (keep != nullptr) keep[at + i] = v;
            else if (first != nullptr) v = (1.0f - lambda) * v + lambda * first[at + i];
            if (page >= 0) v_pool[(((size_t)page * G + g) * page_size + slot) * dv + i] = from_f<T>(v);
        }
    }
}

// row [T, ld] in `dtype` with k at column k_off and v at column v_off; pools k [page][G][page_size][d], v [..][dv].
GG_API gg_head_kv_prep(const void* row, long long ld, int dtype, int k_off, int v_off, void* k_pool, void* v_pool,
                       const int* positions, const int* seq_of_token, const int* page_table, int max_pages, int page_size,
                       int n_pages, int ntok, int G, int d, int dv, int unit, float eps, const float* first, float lambda,
                       float* keep, int* status, cudaStream_t stream) {
    if (ntok <= 0) return 0;
    if (G <= 0 || d <= 0 || dv <= 0 || page_size <= 0 || k_pool == nullptr || v_pool == nullptr || k_off < 0 || v_off < 0)
        return GG_ERR_ARG;
    GG_DISPATCH_DTYPE(dtype, T,
        gg_launch(head_kv_prep_kernel<T>, dim3(ntok), dim3(128), 0, stream, 1, (const T*)row, ld, k_off, v_off, (T*)k_pool,
                  (T*)v_pool, positions, seq_of_token, page_table, max_pages, page_size, G, d, dv, unit, eps, first, lambda,
                  keep, PageBounds{n_pages, status}));
    return gg_last_error();
}

__device__ __forceinline__ float mh_temperature(int pos, float coef, float every) {
    return coef == 0.f ? 1.0f : 1.0f + coef * logf(floorf((float)(pos + 1) / every) + 1.0f);
}

// ----------------------------------------------------------------------------- attention, plain
// One block per token, all heads: a first pass over the keys finds every head's maximum and sum, a second one makes the
// weights of 32 keys, mixes them and adds the values.  Everything between the loads and the store is float32.
#define MP_KEYS 32
template <typename T>
__global__ void __launch_bounds__(256) mixed_head_attention_plain_kernel(
    const T* row, long long ld, int g_off, const T* k_pool, const T* v_pool, T* out, long long ldo,
    const float* __restrict__ talk, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
    const int* __restrict__ page_table, int max_pages, int page_size, int H, int G, int d, int dv, float scale, float cap,
    float coef, float every, float one, int window, const PageBounds pb) {
    pdl_launch();
    pdl_wait();
    extern __shared__ float sm[];
    float* qs = sm;                         // [H][d]
    float* os = qs + (size_t)H * d;         // [H][dv]
    float* P = os + (size_t)H * dv;         // [H][MP_KEYS]
    float* Wm = P + H * MP_KEYS;            // [H][MP_KEYS]
    float* M = Wm + H * MP_KEYS;            // [H]
    float* L = M + H;                       // [H]
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    T* o = out + (size_t)t * ldo;
    const int b = seq_of_token[t];
    if (b < 0) {
        for (int i = threadIdx.x; i < H * dv; i += blockDim.x) o[i] = from_f<T>(0.f);
        return;
    }
    const int pos = positions[t];
    const int hpg = H / G;
    const float sc = scale * mh_temperature(pos, coef, every);
    const T* src = row + (size_t)t * ld;
    for (int i = threadIdx.x; i < H * d; i += blockDim.x) qs[i] = to_f<T>(src[i]);
    for (int i = threadIdx.x; i < H * dv; i += blockDim.x) os[i] = 0.f;
    for (int h = threadIdx.x; h < H; h += blockDim.x) { M[h] = one > 0.f ? 0.f : -INFINITY; L[h] = one; }
    __syncthreads();
    const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    const int* pt = page_table + (size_t)b * max_pages;

    auto scores = [&](int j0) {              // P[h][kk] = the bounded score of key j0 + kk (-inf beyond the last one seen)
        for (int kk = warp; kk < MP_KEYS; kk += nwarps) {
            const int j = j0 + kk;
            if (j > pos) {
                for (int h = lane; h < H; h += 32) P[h * MP_KEYS + kk] = -INFINITY;
                continue;
            }
            const int page = gg_page(pt, j / page_size, max_pages, pb, 53);
            for (int g = 0; g < G; ++g) {
                const T* kp = k_pool + (((size_t)page * G + g) * page_size + (j % page_size)) * d;
                for (int h = g * hpg; h < (g + 1) * hpg; ++h) {
                    float s = 0.f;
                    for (int i = lane; i < d; i += 32) s = fmaf(qs[(size_t)h * d + i], to_f<T>(kp[i]), s);
                    s = warp_sum(s) * sc;
                    if (cap > 0.f) s = cap * tanhf(s / cap);
                    if (lane == 0) P[h * MP_KEYS + kk] = s;
                }
            }
        }
        __syncthreads();
    };
    for (int j0 = lo; j0 <= pos; j0 += MP_KEYS) {
        scores(j0);
        for (int h = warp; h < H; h += nwarps) {
            const float s = P[h * MP_KEYS + lane];
            const float m0 = M[h], m1 = fmaxf(m0, warp_max(s));
            const float sum = warp_sum(expf(s - m1));
            if (lane == 0) { L[h] = L[h] * expf(m0 - m1) + sum; M[h] = m1; }
        }
        __syncthreads();
    }
    for (int j0 = lo; j0 <= pos; j0 += MP_KEYS) {
        scores(j0);
        for (int i = threadIdx.x; i < H * MP_KEYS; i += blockDim.x) P[i] = expf(P[i] - M[i / MP_KEYS]) / L[i / MP_KEYS];
        __syncthreads();
        for (int i = threadIdx.x; i < H * MP_KEYS; i += blockDim.x) {
            const int h = i / MP_KEYS, kk = i - h * MP_KEYS;
            float w = 0.f;
            for (int g = 0; g < H; ++g) w = fmaf(talk[h * H + g], P[g * MP_KEYS + kk], w);
            Wm[i] = w;
        }
        __syncthreads();
        const int nk = min(MP_KEYS, pos - j0 + 1);
        for (int i = threadIdx.x; i < H * dv; i += blockDim.x) {
            const int h = i / dv, e = i - h * dv;
            float a = os[i];
            for (int kk = 0; kk < nk; ++kk) {
                const int j = j0 + kk;
                const int page = gg_page(pt, j / page_size, max_pages, pb, 53);
                a = fmaf(Wm[h * MP_KEYS + kk], to_f<T>(v_pool[(((size_t)page * G + h / hpg) * page_size + (j % page_size)) * dv + e]), a);
            }
            os[i] = a;
        }
        __syncthreads();
    }
    for (int i = threadIdx.x; i < H * dv; i += blockDim.x) {
        float f = 1.f;
        if (g_off >= 0) f = 1.0f / (1.0f + expf(-to_f<T>(src[g_off + i / dv])));
        o[i] = from_f<T>(os[i] * f);
    }
}

// row [T, ld] in `dtype`: q at column 0, the gate logits at column g_off (negative: no gate); out [T, H dv] with row
// stride ldo; talk [H][H] float32.  cap 0: scores not bounded; coef 0: no temperature; one: 0 or 1; window <= 0: none.
GG_API gg_mixed_head_attention_plain(const void* row, long long ld, int g_off, const void* k_pool, const void* v_pool,
                                     void* out, long long ldo, int dtype, const float* talk, const int* positions,
                                     const int* seq_of_token, const int* page_table, int max_pages, int page_size,
                                     int n_pages, int ntok, int H, int G, int d, int dv, float scale, float cap, float coef,
                                     float every, float one, int window, int* status, cudaStream_t stream) {
    if (ntok <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || page_size <= 0 || talk == nullptr || cap < 0.f || ldo < H * dv ||
        (coef != 0.f && !(every > 0.f)))
        return GG_ERR_ARG;
    const size_t smem = ((size_t)H * d + (size_t)H * dv + 2 * (size_t)H * MP_KEYS + 2 * H) * sizeof(float);
    if (smem > 220 * 1024) return GG_ERR_ARG;
    GG_DISPATCH_DTYPE(dtype, T,
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(mixed_head_attention_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        gg_launch(mixed_head_attention_plain_kernel<T>, dim3(ntok), dim3(256), smem, stream, 1, (const T*)row, ld, g_off,
                  (const T*)k_pool, (const T*)v_pool, (T*)out, ldo, talk, positions, seq_of_token, page_table, max_pages,
                  page_size, H, G, d, dv, scale, cap, coef, every, one, window, PageBounds{n_pages, status}));
    return gg_last_error();
}

// ----------------------------------------------------------------------------- the same on the tensor cores (bfloat16)
// mixed_head_mma_kernel: a CTA of four warps takes 64 query rows, the hpg = H / G query heads of one kv head for
// tpt = 64 / hpg consecutive tokens of one sequence (row r: token r / hpg, head r % hpg), and NV kv heads' values.  The
// key tiles are the sequence's pages (64 positions), brought into shared memory by cp.async in two stages.  Per tile
// S = Q K^T (mma.sync m16n8k16, fragments by ldmatrix), temperature, bound and mask in float32, an online softmax in
// float32, P as the A operand of U_n += P V_n for the NV value heads.  Unnormalised results go to scratch,
// u [row of the step][head][share][kv head][dv], with each row's maximum (log2 units) and sum, ml [..][share][2].
// WK (tiles of at most 16 rows: decode steps): the four warps all hold the tile's rows and take 16 of a page's 64 keys
// each.  nsplit > 1: the key tiles of a CTA are shared out over nsplit CTAs.
// mixed_head_combine_kernel: a block per (token, kv head) puts the shares together, divides by the softmax's sum (with
// the one that joins it), mixes the heads with T and applies the gate.
__device__ __forceinline__ void mh_ldsm4(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mh_ldsm4_t(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mh_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mh_cp16(void* dst, const void* src) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ uint32_t mh_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float mh_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// The bounded score in log2 units from x = 2 log2(e) s / cap: cap log2(e) tanh(s / cap), tanh from one exponential.
__device__ __forceinline__ float mh_bound(float x, float cap_log2) {
    return cap_log2 - __fdividef(2.0f * cap_log2, mh_ex2(x) + 1.0f);
}
#define MH_LOG2E 1.4426950408889634f
#define MH_ROWS 64
#define MH_KEYS 64

template <int D, int DV, int NV, bool WK>
__global__ void __launch_bounds__(128) mixed_head_mma_kernel(
    const bf16* row, long long ld, const bf16* k_pool, const bf16* v_pool, float* u, float* ml,
    const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens,
    const int* __restrict__ page_table, int max_pages, int n_seqs, int H, int G, int hpg, int tpt, int d, int dv,
    float scale, float cap, float coef, float every, int window, int nsplit, const PageBounds pb) {
    pdl_wait();
    constexpr int QS = D + 8, VS = DV + 8;                          // row strides in elements (16 bytes of padding)
    extern __shared__ __align__(16) unsigned char mh_smem[];
    bf16* Qs = reinterpret_cast<bf16*>(mh_smem);                    // [64][QS]
    bf16* Ks = Qs + MH_ROWS * QS;                                   // [2][64][QS]
    bf16* Vs = Ks + 2 * MH_KEYS * QS;                               // [2][NV][64][VS]
    __shared__ int info[3];
    const int g = blockIdx.y % G, v0 = (blockIdx.y / G) * NV;       // the rows' kv head, the first value head
    if (threadIdx.x == 0) {
        // (the step's last tiles first: they read the most keys)
        int tile = (int)gridDim.x - 1 - (int)blockIdx.x, b = 0, found = 0;
        for (; b < n_seqs; ++b) {
            const int n = cu_seqlens[b + 1] - cu_seqlens[b];
            const int nt = (n + tpt - 1) / tpt;
            if (tile < nt) { found = 1; break; }
            tile -= nt;
        }
        info[0] = found ? b : -1;
        info[1] = found ? cu_seqlens[b] + tile * tpt : 0;
        info[2] = found ? min(tpt, cu_seqlens[b + 1] - (cu_seqlens[b] + tile * tpt)) : 0;
    }
    __syncthreads();
    const int b = info[0], t0 = info[1], ntok = info[2];
    if (b < 0 || seq_of_token[t0] < 0) return;                      // (padding rows: the combining kernel writes zeros)
    const int nrows = ntok * hpg;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int idx = threadIdx.x; idx < MH_ROWS * (D / 8); idx += blockDim.x) {
        const int r = idx / (D / 8), c = (idx - r * (D / 8)) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < nrows && c < d)
            v = *reinterpret_cast<const uint4*>(row + (size_t)(t0 + r / hpg) * ld + (size_t)(g * hpg + r % hpg) * d + c);
        *reinterpret_cast<uint4*>(Qs + r * QS + c) = v;
    }
    const int pos0 = positions[t0];
    const int pos_last = pos0 + ntok - 1;
    const int lo_key = (window > 0 && pos0 - window + 1 > 0) ? pos0 - window + 1 : 0;
    int j_lo = lo_key / MH_KEYS, j_hi = pos_last / MH_KEYS;
    if (nsplit > 1) {                                               // this CTA's share of the tiles (it may be empty)
        const int per = (j_hi - j_lo + nsplit) / nsplit;
        j_lo += (int)blockIdx.z * per;
        j_hi = min(j_hi, j_lo + per - 1);
    }
    const int* pt = page_table + (size_t)b * max_pages;

    auto load_tile = [&](int j, int stage) {
        const int page = gg_page(pt, j, max_pages, pb, 53);
        const bf16* kp = k_pool + ((size_t)page * G + g) * MH_KEYS * d;
        bf16* kd = Ks + stage * MH_KEYS * QS;
        for (int idx = threadIdx.x; idx < MH_KEYS * (D / 8); idx += blockDim.x) {
            const int r = idx / (D / 8), c = (idx - r * (D / 8)) * 8;
            if (c < d) mh_cp16(kd + r * QS + c, kp + (size_t)r * d + c);
            else *reinterpret_cast<uint4*>(kd + r * QS + c) = make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            if (v0 + n >= G) break;
            const bf16* vp = v_pool + ((size_t)page * G + v0 + n) * MH_KEYS * dv;
            bf16* vd = Vs + (stage * NV + n) * MH_KEYS * VS;
            for (int idx = threadIdx.x; idx < MH_KEYS * (DV / 8); idx += blockDim.x) {
                const int r = idx / (DV / 8), c = (idx - r * (DV / 8)) * 8;
                if (c < dv) mh_cp16(vd + r * VS + c, vp + (size_t)r * dv + c);
                else *reinterpret_cast<uint4*>(vd + r * VS + c) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    const int gq = lane >> 2, t4 = lane & 3;                        // this thread's two rows of its warp's sixteen
    const int rbase = WK ? 0 : warp * 16, kbase = WK ? warp * 16 : 0;
    constexpr int NP = WK ? 1 : 4;                                  // runs of 16 keys the warp takes of a page
    int rpos[2], rlo[2];
    float rfac[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = rbase + gq + 8 * i;
        rpos[i] = r < nrows ? pos0 + r / hpg : -1;
        rlo[i] = window > 0 ? rpos[i] - window + 1 : 0;
        rfac[i] = scale * mh_temperature(max(rpos[i], 0), coef, every) * (cap > 0.f ? 2.0f * MH_LOG2E / cap : MH_LOG2E);
    }
    const float cap_log2 = cap * MH_LOG2E;
    const int wlast = min(rbase + 15, nrows - 1);
    const int wmax = rbase < nrows ? pos0 + wlast / hpg : -1;       // the warp's largest position (-1: no rows)
    float O[NV][DV / 8][4];
    float mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int c = 0; c < DV / 8; ++c) { O[n][c][0] = O[n][c][1] = O[n][c][2] = O[n][c][3] = 0.f; }

    if (j_lo <= j_hi) load_tile(j_lo, 0);
    for (int j = j_lo; j <= j_hi; ++j) {
        const int stage = (j - j_lo) & 1;
        if (j < j_hi) {
            load_tile(j + 1, stage ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int key0 = j * MH_KEYS;
        if (key0 <= wmax) {
            const bf16* Kt = Ks + stage * MH_KEYS * QS;
            float s[2 * NP][4];
#pragma unroll
            for (int n = 0; n < 2 * NP; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
#pragma unroll
            for (int ks = 0; ks < D / 16; ++ks) {
                uint32_t a[4];
                mh_ldsm4(a, Qs + (rbase + (lane & 7) + ((lane >> 3) & 1) * 8) * QS + ks * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int np = 0; np < NP; ++np) {
                    uint32_t bb[4];
                    mh_ldsm4(bb, Kt + (kbase + np * 16 + (lane & 7) + (lane >> 4) * 8) * QS + ks * 16 + ((lane >> 3) & 1) * 8);
                    mh_mma(s[2 * np], a, bb[0], bb[1]);
                    mh_mma(s[2 * np + 1], a, bb[2], bb[3]);
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int n = 0; n < 2 * NP; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = e >> 1;
                    const int key = key0 + kbase + n * 8 + 2 * t4 + (e & 1);
                    float v = s[n][e] * rfac[i];
                    if (cap > 0.f) v = mh_bound(v, cap_log2);
                    v = (key <= rpos[i] && key >= rlo[i]) ? v : -INFINITY;
                    s[n][e] = v;
                    mx[i] = fmaxf(mx[i], v);
                }
            }
            float corr[2], muse[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
                const float mn = fmaxf(mrun[i], mx[i]);
                muse[i] = mn == -INFINITY ? 0.f : mn;
                corr[i] = mh_ex2(mrun[i] - muse[i]);
                mrun[i] = mn;
                lrun[i] *= corr[i];
            }
            uint32_t p[NP][4];
#pragma unroll
            for (int n = 0; n < 2 * NP; ++n) {
                const float p0 = mh_ex2(s[n][0] - muse[0]), p1 = mh_ex2(s[n][1] - muse[0]);
                const float p2 = mh_ex2(s[n][2] - muse[1]), p3 = mh_ex2(s[n][3] - muse[1]);
                lrun[0] += p0 + p1;
                lrun[1] += p2 + p3;
                p[n >> 1][(n & 1) * 2] = mh_pack(p0, p1);
                p[n >> 1][(n & 1) * 2 + 1] = mh_pack(p2, p3);
            }
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                if (v0 + n >= G) break;
                const bf16* Vt = Vs + (stage * NV + n) * MH_KEYS * VS;
#pragma unroll
                for (int c = 0; c < DV / 8; ++c) {
                    O[n][c][0] *= corr[0]; O[n][c][1] *= corr[0];
                    O[n][c][2] *= corr[1]; O[n][c][3] *= corr[1];
                }
#pragma unroll
                for (int kk = 0; kk < NP; ++kk) {
#pragma unroll
                    for (int np = 0; np < DV / 16; ++np) {
                        uint32_t bb[4];
                        mh_ldsm4_t(bb, Vt + (kbase + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VS + np * 16 + (lane >> 4) * 8);
                        mh_mma(O[n][2 * np], p[kk], bb[0], bb[1]);
                        mh_mma(O[n][2 * np + 1], p[kk], bb[2], bb[3]);
                    }
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        lrun[i] += __shfl_xor_sync(0xffffffffu, lrun[i], 1);
        lrun[i] += __shfl_xor_sync(0xffffffffu, lrun[i], 2);
    }
    if (WK) {
        // the four warps' shares of the keys, put together in shared memory (the pipeline's stages are free now)
        constexpr int RS = NV * DV + 2;
        float* mg = reinterpret_cast<float*>(mh_smem);               // [warp][16 rows][2 + NV * DV]
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int r = gq + 8 * i;
            if (rpos[i] < 0) continue;
            float* pm = mg + (size_t)(warp * 16 + r) * RS;
            if (t4 == 0) { pm[0] = mrun[i]; pm[1] = lrun[i]; }
#pragma unroll
            for (int n = 0; n < NV; ++n)
#pragma unroll
                for (int c = 0; c < DV / 8; ++c)
                    *reinterpret_cast<float2*>(pm + 2 + n * DV + c * 8 + 2 * t4) = make_float2(O[n][c][2 * i], O[n][c][2 * i + 1]);
        }
        __syncthreads();
        for (int r = warp; r < nrows; r += 4) {                     // a warp a row
            float M = -INFINITY, L = 0.f, f[4];
#pragma unroll
            for (int w = 0; w < 4; ++w) M = fmaxf(M, mg[(size_t)(w * 16 + r) * RS]);
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                const float* pm = mg + (size_t)(w * 16 + r) * RS;
                f[w] = pm[0] == -INFINITY ? 0.f : mh_ex2(pm[0] - M);
                L += pm[1] * f[w];
            }
            const size_t at = ((size_t)(t0 + r / hpg) * H + g * hpg + r % hpg) * nsplit + blockIdx.z;
            if (lane == 0 && v0 == 0) { ml[at * 2] = M; ml[at * 2 + 1] = L; }
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                if (v0 + n >= G) break;
                for (int c = lane; c < dv; c += 32) {
                    float a = 0.f;
#pragma unroll
                    for (int w = 0; w < 4; ++w) a += mg[(size_t)(w * 16 + r) * RS + 2 + n * DV + c] * f[w];
                    u[(at * G + v0 + n) * dv + c] = a;
                }
            }
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = rbase + gq + 8 * i;
        if (rpos[i] < 0) continue;
        const size_t at = ((size_t)(t0 + r / hpg) * H + g * hpg + r % hpg) * nsplit + blockIdx.z;
        if (t4 == 0 && v0 == 0) { ml[at * 2] = mrun[i]; ml[at * 2 + 1] = lrun[i]; }
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            if (v0 + n >= G) break;
            float* po = u + (at * G + v0 + n) * dv;
#pragma unroll
            for (int c = 0; c < DV / 8; ++c) {
                const int e = c * 8 + 2 * t4;
                if (e < dv) *reinterpret_cast<float2*>(po + e) = make_float2(O[n][c][2 * i], O[n][c][2 * i + 1]);
            }
        }
    }
}

// u [T][H][nsplit][G][dv] and ml [T][H][nsplit][2] (float32) -> out [T, H dv] (row stride ldo).  Eight warps share out
// the (head, share) pairs, a lane holds four columns; dv a multiple of 4, at most 128.
#define MC_WARPS 8
__global__ void __launch_bounds__(MC_WARPS * 32) mixed_head_combine_kernel(
    const float* u, const float* ml, const bf16* row, long long ld, int g_off, bf16* out, long long ldo,
    const float* __restrict__ talk, const int* __restrict__ seq_of_token, int H, int G, int dv, int nsplit, float one) {
    pdl_launch();
    pdl_wait();
    extern __shared__ __align__(16) float mc_sm[];
    float* red = mc_sm;                                 // [MC_WARPS][4][128] (first: it is written 16 bytes at a time)
    float* f = red + MC_WARPS * 4 * 128;                // [H][nsplit]: share z's factor for head g
    const int t = blockIdx.x, gv = blockIdx.y, hpg = H / G;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    bf16* o = out + (size_t)t * ldo + (size_t)gv * hpg * dv;
    if (seq_of_token[t] < 0) {
        for (int i = threadIdx.x; i < hpg * dv; i += blockDim.x) o[i] = __float2bfloat16_rn(0.f);
        return;
    }
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        const float* p = ml + ((size_t)t * H + h) * nsplit * 2;
        float M = one > 0.f ? 0.f : -INFINITY;
        for (int z = 0; z < nsplit; ++z) M = fmaxf(M, p[2 * z]);
        float L = one > 0.f ? one * mh_ex2(-M) : 0.f;
        for (int z = 0; z < nsplit; ++z) L += p[2 * z] == -INFINITY ? 0.f : p[2 * z + 1] * mh_ex2(p[2 * z] - M);
        for (int z = 0; z < nsplit; ++z) f[h * nsplit + z] = p[2 * z] == -INFINITY ? 0.f : mh_ex2(p[2 * z] - M) / L;
    }
    __syncthreads();
    const int c = 4 * lane;
    for (int h0 = 0; h0 < hpg; h0 += 4) {
        float acc[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[k][0] = acc[k][1] = acc[k][2] = acc[k][3] = 0.f;
        for (int gz = warp; gz < H * nsplit; gz += MC_WARPS) {
            const float fz = f[gz];
            const int gh = gz / nsplit;
            if (c < dv && fz != 0.f) {
                const float4 v = *reinterpret_cast<const float4*>(u + (((size_t)t * H * nsplit + gz) * G + gv) * dv + c);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    if (h0 + k < hpg) {
                        const float w = talk[(size_t)(gv * hpg + h0 + k) * H + gh] * fz;
                        acc[k][0] = fmaf(w, v.x, acc[k][0]); acc[k][1] = fmaf(w, v.y, acc[k][1]);
                        acc[k][2] = fmaf(w, v.z, acc[k][2]); acc[k][3] = fmaf(w, v.w, acc[k][3]);
                    }
                }
            }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k)
            *reinterpret_cast<float4*>(red + (warp * 4 + k) * 128 + c) = make_float4(acc[k][0], acc[k][1], acc[k][2], acc[k][3]);
        __syncthreads();
        for (int i = threadIdx.x; i < 4 * 128; i += blockDim.x) {
            const int k = i >> 7, e = i & 127;
            if (h0 + k >= hpg || e >= dv) continue;
            float a = 0.f;
#pragma unroll
            for (int w = 0; w < MC_WARPS; ++w) a += red[(w * 4 + k) * 128 + e];
            const int h = gv * hpg + h0 + k;
            if (g_off >= 0) a = a / (1.0f + mh_ex2(-MH_LOG2E * __bfloat162float(row[(size_t)t * ld + g_off + h])));
            o[(h0 + k) * dv + e] = __float2bfloat16_rn(a);
        }
        __syncthreads();
    }
}

// The same for one share (prompts): a warp per token and kv head, a lane four columns, a block the tokens of one kv head, so
// that the rows of T it needs sit in shared memory, HC heads of the kv head at a time.
template <int HC>
__global__ void __launch_bounds__(MC_WARPS * 32) mixed_head_combine_rows_kernel(
    const float* u, const float* ml, const bf16* row, long long ld, int g_off, bf16* out, long long ldo,
    const float* __restrict__ talk, const int* __restrict__ seq_of_token, int ntok, int H, int G, int dv, float one) {
    pdl_launch();
    extern __shared__ __align__(16) float cr_sm[];
    const int gv = blockIdx.y, hpg = H / G;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* tk = cr_sm;                                  // [H][HC]
    float* f = tk + H * HC + warp * H;                  // [H] of this warp's token
    const int t = blockIdx.x * MC_WARPS + warp, c = 4 * lane;
    const bool have = t < ntok, live = have && seq_of_token[have ? t : 0] >= 0;
    pdl_wait();
    if (live) {
        for (int h = lane; h < H; h += 32) {
            const float m = ml[((size_t)t * H + h) * 2], l = ml[((size_t)t * H + h) * 2 + 1];
            const float M = one > 0.f ? fmaxf(m, 0.f) : m;
            const float e = mh_ex2(m - M);
            f[h] = e / (l * e + (one > 0.f ? one * mh_ex2(-M) : 0.f));
        }
    }
    for (int h0 = 0; h0 < hpg; h0 += HC) {
        __syncthreads();
        for (int i = threadIdx.x; i < H * HC; i += blockDim.x) {
            const int g = i / HC, k = i - g * HC;
            tk[i] = h0 + k < hpg ? talk[(size_t)(gv * hpg + h0 + k) * H + g] : 0.f;
        }
        __syncthreads();
        if (!have || c >= dv) continue;
        float acc[HC][4];
#pragma unroll
        for (int k = 0; k < HC; ++k) acc[k][0] = acc[k][1] = acc[k][2] = acc[k][3] = 0.f;
        if (live) {
            const float* ub = u + ((size_t)t * H * G + gv) * dv + c;
#pragma unroll 4
            for (int g = 0; g < H; ++g) {
                const float4 v = *reinterpret_cast<const float4*>(ub + (size_t)g * G * dv);
                const float fg = f[g];
#pragma unroll
                for (int k = 0; k < HC; ++k) {
                    const float w = tk[g * HC + k] * fg;
                    acc[k][0] = fmaf(w, v.x, acc[k][0]); acc[k][1] = fmaf(w, v.y, acc[k][1]);
                    acc[k][2] = fmaf(w, v.z, acc[k][2]); acc[k][3] = fmaf(w, v.w, acc[k][3]);
                }
            }
        }
#pragma unroll
        for (int k = 0; k < HC; ++k) {
            if (h0 + k >= hpg) break;
            const int h = gv * hpg + h0 + k;
            float s = 1.f;
            if (live && g_off >= 0) s = 1.0f / (1.0f + mh_ex2(-MH_LOG2E * __bfloat162float(row[(size_t)t * ld + g_off + h])));
            const uint32_t a = mh_pack(acc[k][0] * s, acc[k][1] * s), b = mh_pack(acc[k][2] * s, acc[k][3] * s);
            *reinterpret_cast<uint2*>(out + (size_t)t * ldo + (size_t)h * dv + c) = make_uint2(a, b);
        }
    }
}

// 1 if the tensor-core form takes these sizes (bfloat16 only), else 0.
GG_API gg_mixed_head_mma_takes(int H, int G, int d, int dv, int page_size) {
    return (d > 0 && d <= 128 && d % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0 && page_size == MH_KEYS && G > 0 &&
            H % G == 0 && H / G <= MH_ROWS && H <= 512 && G <= 4096) ? 1 : 0;
}

// u [ntok][H][nsplit][G][dv] and ml [ntok][H][nsplit][2] (float32: unnormalised results of the shares of the keys on every
// kv head's values, their references in log2 units and sums) -> out [ntok, H dv] (bfloat16, row stride ldo): the shares put
// together, divided by the softmax's sum (with `one` joining it), the heads mixed by talk [H][H], gated by the logits at
// row + t ld + g_off (g_off negative: no gate).
GG_API gg_mixed_head_combine(const float* u, const float* ml, const void* row, long long ld, int g_off, void* out, long long ldo,
                             const float* talk, const int* seq_of_token, int ntok, int H, int G, int dv, int nsplit, float one,
                             cudaStream_t stream) {
    if (ntok <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dv <= 0 || dv > 128 || dv % 4 || nsplit < 1 || ldo < (long long)H * dv || (((uintptr_t)u) & 15))
        return GG_ERR_ARG;
    if (nsplit == 1 && ntok >= 64 && (ldo % 4) == 0 && (((uintptr_t)out) & 7) == 0) {
        const int hc = H / G > 2 ? 4 : (H / G > 1 ? 2 : 1);
        const size_t sm = (size_t)H * (hc + MC_WARPS) * sizeof(float);
        if (sm <= 48 * 1024) {
            auto kern = hc == 4 ? mixed_head_combine_rows_kernel<4> : (hc == 2 ? mixed_head_combine_rows_kernel<2> : mixed_head_combine_rows_kernel<1>);
            return gg_launch(kern, dim3((ntok + MC_WARPS - 1) / MC_WARPS, G), dim3(MC_WARPS * 32), sm, stream, 1, u, ml, (const bf16*)row,
                             ld, g_off, (bf16*)out, ldo, talk, seq_of_token, ntok, H, G, dv, one);
        }
    }
    const size_t smem = ((size_t)H * nsplit + MC_WARPS * 4 * 128) * sizeof(float);
    if (smem > 220 * 1024) return GG_ERR_ARG;
    if (smem > 48 * 1024) cudaFuncSetAttribute(mixed_head_combine_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return gg_launch(mixed_head_combine_kernel, dim3(ntok, G), dim3(MC_WARPS * 32), smem, stream, 1, u, ml, (const bf16*)row, ld,
                     g_off, (bf16*)out, ldo, talk, seq_of_token, H, G, dv, nsplit, one);
}

template <int D, int DV, int NV, bool WK>
static int mh_launch(const bf16* row, long long ld, const bf16* k_pool, const bf16* v_pool, float* u, float* ml,
                     const int* positions, const int* seq_of_token, const int* cu_seqlens, const int* page_table,
                     int max_pages, int n_pages, int ntok, int n_seqs, int H, int G, int d, int dv, float scale, float cap,
                     float coef, float every, int window, int nsplit, int* status, cudaStream_t stream) {
    const int hpg = H / G;
    const int tpt = (WK ? 16 : MH_ROWS) / hpg;
    size_t smem = ((size_t)MH_ROWS * (D + 8) + 2 * MH_KEYS * (D + 8) + 2 * NV * MH_KEYS * (DV + 8)) * sizeof(bf16);
    if (WK) { const size_t m = (size_t)4 * 16 * (NV * DV + 2) * sizeof(float); if (m > smem) smem = m; }
    static bool configured = false;                                  // per instantiation
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(mixed_head_mma_kernel<D, DV, NV, WK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const int tiles = (ntok + tpt - 1) / tpt + n_seqs;             // an upper bound on the sequences' tiles
    return gg_launch(mixed_head_mma_kernel<D, DV, NV, WK>, dim3(tiles, G * ((G + NV - 1) / NV), nsplit), dim3(128), smem, stream,
                     1, row, ld, k_pool, v_pool, u, ml, positions, seq_of_token, cu_seqlens, page_table, max_pages, n_seqs, H,
                     G, hpg, tpt, d, dv, scale, cap, coef, every, window, nsplit, PageBounds{n_pages, status});
}

// As gg_mixed_head_attention_plain for bfloat16 tensors whose rows start on 16-byte boundaries, with the step's
// cu_seqlens [n_seqs + 1].  u: scratch of ntok * H * nsplit * G * dv floats, ml of ntok * H * nsplit * 2.  max_new: the most
// rows one sequence brings (0: not known); where max_new * (H / G) <= 16 a tile holds 16 rows and its four warps share
// out every page's keys.  nsplit > 1: every tile is the work of nsplit CTAs, each with a share of the key tiles.
GG_API gg_mixed_head_attention_mma(const void* row, long long ld, int g_off, const void* k_pool, const void* v_pool, void* out,
                                   long long ldo, const float* talk, const int* positions, const int* seq_of_token,
                                   const int* cu_seqlens, const int* page_table, int max_pages, int page_size, int n_pages,
                                   int ntok, int n_seqs, int H, int G, int d, int dv, float scale, float cap, float coef,
                                   float every, float one, int window, int nsplit, float* u, float* ml, int max_new,
                                   int* status, cudaStream_t stream) {
    if (ntok <= 0 || n_seqs <= 0) return 0;
    if (!gg_mixed_head_mma_takes(H, G, d, dv, page_size) || talk == nullptr || u == nullptr || ml == nullptr || nsplit < 1 ||
        nsplit > 64 || cap < 0.f || ldo < H * dv || (coef != 0.f && !(every > 0.f)) || (ld % 8) ||
        (((uintptr_t)row | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)u) & 15))
        return GG_ERR_ARG;
    const bool wk = max_new > 0 && max_new * (H / G) <= 16;
    const bool two = G > 1;
    int rc = GG_ERR_ARG;
#define MH_ARGS (const bf16*)row, ld, (const bf16*)k_pool, (const bf16*)v_pool, u, ml, positions, seq_of_token, cu_seqlens, \
        page_table, max_pages, n_pages, ntok, n_seqs, H, G, d, dv, scale, cap, coef, every, window, nsplit, status, stream
#define MH_GO(D_, V_) rc = two ? (wk ? mh_launch<D_, V_, 2, true>(MH_ARGS) : mh_launch<D_, V_, 2, false>(MH_ARGS)) \
                               : (wk ? mh_launch<D_, V_, 1, true>(MH_ARGS) : mh_launch<D_, V_, 1, false>(MH_ARGS))
    if (d <= 32) { if (dv <= 32) MH_GO(32, 32); else if (dv <= 64) MH_GO(32, 64); else MH_GO(32, 128); }
    else if (d <= 64) { if (dv <= 32) MH_GO(64, 32); else if (dv <= 64) MH_GO(64, 64); else MH_GO(64, 128); }
    else { if (dv <= 32) MH_GO(128, 32); else if (dv <= 64) MH_GO(128, 64); else MH_GO(128, 128); }
#undef MH_GO
#undef MH_ARGS
    if (rc != 0) return rc;
    return gg_mixed_head_combine(u, ml, row, ld, g_off, out, ldo, talk, seq_of_token, ntok, H, G, dv, nsplit, one, stream);
}

// 1 if this library was built with checked page tables (the debug build), else 0.
GG_API gg_mixed_head_attention_checked() { return gg_debug_bounds(); }
