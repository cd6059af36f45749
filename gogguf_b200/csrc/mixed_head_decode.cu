// Attention with mixed heads (see mixed_head_attention.cu) of steps that bring few rows over long contexts (decode
// steps), bfloat16.  The heads' weights can only be mixed once every head's softmax sum is known, so the step goes over
// the keys first and over the values afterwards, each read once, with the scores (a float per head and position) kept
// in between:
//
//   mixed_head_scores_kernel   a CTA per (token, kv head, share of the pages): bounded scores in log2 units of the kv head's
//                              query heads into scores [token][head][position], each share's maximum and sum into ml
//   mixed_head_values_kernel   a CTA per (token, kv head, share): the weights of all heads at its positions from the scores,
//                              mixed by T into the rows of the kv head's heads, times the values; float32 partial sums
//   mixed_head_merge_kernel    the shares' sums added up, the heads' gates, the output
//
// In both passes each of a CTA's four warps takes 16 of a page's 64 positions through a ring of its own (cp.async), so no
// barrier stands in the loop.  Products are mma.sync m16n8k16 with the heads as rows; the mixed weights enter the second
// one as two bfloat16 terms.
#include "common.cuh"

#define MD_LOG2E 1.4426950408889634f
#define MD_STAGES 4

__device__ __forceinline__ void md_ldsm4(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void md_ldsm4_t(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void md_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void md_cp16(void* dst, const void* src) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ float md_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// The pages of share z of a sequence whose tokens up to `pos` are seen.
__device__ __forceinline__ void md_share(int pos, int window, int nsplit, int z, int& j_lo, int& j_hi, int& lo_key) {
    lo_key = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    j_lo = lo_key / 64;
    j_hi = pos / 64;
    const int per = (j_hi - j_lo + nsplit) / nsplit;
    j_lo += z * per;
    j_hi = min(j_hi, j_lo + per - 1);
}

// A warp's ring: 16 rows of W columns (the first w of them read, the rest zeros), rows W + 8 elements apart.
template <int W>
struct MdRing {
    static constexpr int LD = W + 8, STAGE = 16 * LD;
    bf16* base;
    int lane, w;
    __device__ __forceinline__ void clear() {            // the columns beyond w are never written again
        for (int i = lane; i < MD_STAGES * 16 * (W / 8); i += 32) {
            const int r = i / (W / 8), c = (i % (W / 8)) * 8;
            if (c >= w) *reinterpret_cast<uint4*>(base + r * LD + c) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    __device__ __forceinline__ void load(int stage, const bf16* src) {
        bf16* dst = base + stage * STAGE;
#pragma unroll
        for (int i = lane; i < 16 * (W / 8); i += 32) {
            const int r = i / (W / 8), c = (i % (W / 8)) * 8;
            if (c < w) md_cp16(dst + r * LD + c, src + (size_t)r * w + c);
        }
    }
};

template <int D>
__global__ void __launch_bounds__(128) mixed_head_scores_kernel(
    const bf16* row, long long ld, const bf16* k_pool, float* scores, long long ctx_pad, float* ml,
    const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ page_table, int max_pages,
    int H, int G, int d, float scale, float cap, float coef, float every, int window, int nsplit, const PageBounds pb) {
    pdl_launch();
    extern __shared__ __align__(16) unsigned char md_smem[];
    constexpr int LD = D + 8;
    bf16* Qs = reinterpret_cast<bf16*>(md_smem);                    // [16][LD]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    MdRing<D> ring{Qs + 16 * LD + warp * MD_STAGES * MdRing<D>::STAGE, lane, d};
    __shared__ float red[4][16][2];
    const int t = blockIdx.x, g = blockIdx.y, hpg = H / G;
    const int b = seq_of_token[t];
    if (b < 0) return;
    const int pos = positions[t];
    int j_lo, j_hi, lo_key;
    md_share(pos, window, nsplit, blockIdx.z, j_lo, j_hi, lo_key);
    const int* pt = page_table + (size_t)b * max_pages;
    const int n = j_hi - j_lo + 1;
    ring.clear();
    auto fetch = [&](int i) {                                       // page j_lo + i into stage i % MD_STAGES
        if (i < n) {
            const int page = gg_page(pt, j_lo + i, max_pages, pb, 53);
            ring.load(i % MD_STAGES, k_pool + (((size_t)page * G + g) * 64 + warp * 16) * d);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    pdl_wait();
#pragma unroll
    for (int i = 0; i < MD_STAGES - 1; ++i) fetch(i);
    for (int i = threadIdx.x; i < 16 * (D / 8); i += 128) {
        const int r = i / (D / 8), c = (i % (D / 8)) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < hpg && c < d) v = *reinterpret_cast<const uint4*>(row + (size_t)t * ld + (size_t)(g * hpg + r) * d + c);
        *reinterpret_cast<uint4*>(Qs + r * LD + c) = v;
    }
    __syncthreads();
    uint32_t qa[D / 16][4];
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) md_ldsm4(qa[ks], Qs + (lane & 15) * LD + ks * 16 + (lane >> 4) * 8);
    const int gq = lane >> 2, t4 = lane & 3;
    const float tau = coef == 0.f ? 1.0f : 1.0f + coef * logf(floorf((float)(pos + 1) / every) + 1.0f);
    const float fac = scale * tau * (cap > 0.f ? 2.0f * MD_LOG2E / cap : MD_LOG2E), cap_log2 = cap * MD_LOG2E;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    for (int i = 0; i < n; ++i) {
        fetch(i + MD_STAGES - 1);
        asm volatile("cp.async.wait_group %0;" :: "n"(MD_STAGES - 1) : "memory");
        __syncwarp();
        const bf16* kt = ring.base + (i % MD_STAGES) * MdRing<D>::STAGE;
        float s[2][4];
#pragma unroll
        for (int x = 0; x < 2; ++x) s[x][0] = s[x][1] = s[x][2] = s[x][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
            uint32_t bb[4];
            md_ldsm4(bb, kt + ((lane & 7) + (lane >> 4) * 8) * LD + ks * 16 + ((lane >> 3) & 1) * 8);
            md_mma(s[0], qa[ks], bb[0], bb[1]);
            md_mma(s[1], qa[ks], bb[2], bb[3]);
        }
        const int key0 = (j_lo + i) * 64 + warp * 16;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = key0 + x * 8 + 2 * t4 + (e & 1);
                float v = s[x][e] * fac;
                if (cap > 0.f) v = cap_log2 - __fdividef(2.0f * cap_log2, md_ex2(v) + 1.0f);
                s[x][e] = (key <= pos && key >= lo_key) ? v : -INFINITY;
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float mn = fmaxf(fmaxf(fmaxf(s[0][2 * r], s[0][2 * r + 1]), fmaxf(s[1][2 * r], s[1][2 * r + 1])), m[r]);
            const float mu = mn == -INFINITY ? 0.f : mn;
            l[r] = l[r] * md_ex2(m[r] - mu) + md_ex2(s[0][2 * r] - mu) + md_ex2(s[0][2 * r + 1] - mu) + md_ex2(s[1][2 * r] - mu) +
                   md_ex2(s[1][2 * r + 1] - mu);
            m[r] = mn;
            if (gq + 8 * r < hpg) {
                float* dst = scores + ((size_t)t * H + g * hpg + gq + 8 * r) * ctx_pad + key0 + 2 * t4;
                *reinterpret_cast<float2*>(dst) = make_float2(s[0][2 * r], s[0][2 * r + 1]);
                *reinterpret_cast<float2*>(dst + 8) = make_float2(s[1][2 * r], s[1][2 * r + 1]);
            }
        }
        __syncwarp();
    }
    // the four threads of a row, then the four warps
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
        for (int o = 1; o <= 2; o <<= 1) {
            const float mo = __shfl_xor_sync(0xffffffffu, m[r], o), lo = __shfl_xor_sync(0xffffffffu, l[r], o);
            const float mn = fmaxf(m[r], mo), mu = mn == -INFINITY ? 0.f : mn;
            l[r] = l[r] * md_ex2(m[r] - mu) + lo * md_ex2(mo - mu);
            m[r] = mn;
        }
        if (t4 == 0) { red[warp][gq + 8 * r][0] = m[r]; red[warp][gq + 8 * r][1] = l[r]; }
    }
    __syncthreads();
    if (threadIdx.x < hpg) {
        float M = -INFINITY, L = 0.f;
        for (int w = 0; w < 4; ++w) M = fmaxf(M, red[w][threadIdx.x][0]);
        for (int w = 0; w < 4; ++w)
            if (red[w][threadIdx.x][0] != -INFINITY) L += red[w][threadIdx.x][1] * md_ex2(red[w][threadIdx.x][0] - M);
        float* p = ml + (((size_t)t * H + g * hpg + threadIdx.x) * nsplit + blockIdx.z) * 2;
        p[0] = M;
        p[1] = L;
    }
}

// HP: query heads of a kv head, rounded up to 4, 8 or 16.  STAGED: the scores come through the ring with the values (models
// of few heads; the ring's stages are then longer by 64 bytes a head).
template <int DV, int HP, bool STAGED>
__global__ void __launch_bounds__(128) mixed_head_values_kernel(
    const float* scores, long long ctx_pad, const float* ml, const bf16* v_pool, float* part, const float* __restrict__ talk,
    const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ page_table, int max_pages,
    int H, int G, int dv, float one, int window, int nsplit, const PageBounds pb) {
    pdl_launch();
    extern __shared__ __align__(16) unsigned char md_smem[];
    constexpr int LD = DV + 8, WL = 24;                             // a row of mixed weights: 16 keys and padding
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    bf16* rings = reinterpret_cast<bf16*>(md_smem);                 // four warps' rings; at the end [4][HP][DV] float32
    MdRing<DV> ring{rings + warp * MD_STAGES * MdRing<DV>::STAGE, lane, dv};
    bf16* Ws = rings + 4 * MD_STAGES * MdRing<DV>::STAGE + warp * 2 * 16 * WL;          // [2 terms][16][WL]
    float* tk = reinterpret_cast<float*>(rings + 4 * MD_STAGES * MdRing<DV>::STAGE + 4 * 2 * 16 * WL);     // [H][HP]
    float* fm = tk + H * HP;                                        // [H][2]: maximum, 1 / sum
    float* Ss = fm + 2 * ((H + 1) & ~1) + warp * MD_STAGES * H * 16;            // STAGED: [stage][H][16]
    const int t = blockIdx.x, g = blockIdx.y, hpg = H / G;
    const int b = seq_of_token[t];
    if (b < 0) return;
    const int pos = positions[t];
    int j_lo, j_hi, lo_key;
    md_share(pos, window, nsplit, blockIdx.z, j_lo, j_hi, lo_key);
    const int* pt = page_table + (size_t)b * max_pages;
    const int n = j_hi - j_lo + 1;
    ring.clear();
    for (int i = lane; i < 2 * 16 * WL / 8; i += 32) reinterpret_cast<uint4*>(Ws)[i] = make_uint4(0u, 0u, 0u, 0u);
    for (int i = threadIdx.x; i < H * HP; i += 128) {
        const int gh = i / HP, r = i - gh * HP;
        tk[i] = r < hpg ? talk[(size_t)(g * hpg + r) * H + gh] : 0.f;
    }
    auto fetch = [&](int i) {
        if (i < n) {
            const int page = gg_page(pt, j_lo + i, max_pages, pb, 53);
            ring.load(i % MD_STAGES, v_pool + (((size_t)page * G + g) * 64 + warp * 16) * dv);
            if (STAGED) {
                const float* src = scores + (size_t)t * H * ctx_pad + (size_t)(j_lo + i) * 64 + warp * 16;
                for (int x = lane; x < H * 4; x += 32)
                    md_cp16(Ss + (i % MD_STAGES) * H * 16 + x * 4, src + (size_t)(x >> 2) * ctx_pad + (x & 3) * 4);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    pdl_wait();
#pragma unroll
    for (int i = 0; i < MD_STAGES - 1; ++i) fetch(i);
    for (int h = threadIdx.x; h < H; h += 128) {
        const float* p = ml + ((size_t)t * H + h) * nsplit * 2;
        float M = one > 0.f ? 0.f : -INFINITY;
        for (int z = 0; z < nsplit; ++z) M = fmaxf(M, p[2 * z]);
        float L = one > 0.f ? one * md_ex2(-M) : 0.f;
        for (int z = 0; z < nsplit; ++z) L += p[2 * z + 1] * md_ex2(p[2 * z] - M);       // (an empty share: sum 0, 2^-inf 0)
        fm[2 * h] = M;
        fm[2 * h + 1] = 1.0f / L;
    }
    __syncthreads();
    float O[DV / 8][4];
#pragma unroll
    for (int c = 0; c < DV / 8; ++c) O[c][0] = O[c][1] = O[c][2] = O[c][3] = 0.f;
    const int kk = lane & 15, half = lane >> 4;
    const float* sp = scores + (size_t)t * H * ctx_pad + warp * 16 + kk;
    for (int i = 0; i < n; ++i) {
        fetch(i + MD_STAGES - 1);
        if (STAGED) {
            asm volatile("cp.async.wait_group %0;" :: "n"(MD_STAGES - 1) : "memory");
            __syncwarp();
        }
        // this lane's key: every second head's weight there, its share of the mixed weights of all rows
        float w[HP];
#pragma unroll
        for (int r = 0; r < HP; ++r) w[r] = 0.f;
        const float* sk = STAGED ? Ss + (i % MD_STAGES) * H * 16 + kk : sp + (size_t)(j_lo + i) * 64;
        const long long sstep = STAGED ? 16 : ctx_pad;
#pragma unroll 8
        for (int gh = half; gh < H; gh += 2) {
            const float p = md_ex2(sk[gh * sstep] - fm[2 * gh]) * fm[2 * gh + 1];
            const float4* tr = reinterpret_cast<const float4*>(tk + gh * HP);
#pragma unroll
            for (int q = 0; q < HP / 4; ++q) {
                const float4 c = tr[q];
                w[4 * q] = fmaf(c.x, p, w[4 * q]); w[4 * q + 1] = fmaf(c.y, p, w[4 * q + 1]);
                w[4 * q + 2] = fmaf(c.z, p, w[4 * q + 2]); w[4 * q + 3] = fmaf(c.w, p, w[4 * q + 3]);
            }
        }
#pragma unroll
        for (int r = 0; r < HP; ++r) {
            w[r] += __shfl_xor_sync(0xffffffffu, w[r], 16);
            const bf16 hi = __float2bfloat16_rn(w[r]);
            Ws[half * 16 * WL + r * WL + kk] = half ? __float2bfloat16_rn(w[r] - __bfloat162float(hi)) : hi;
        }
        if (!STAGED) asm volatile("cp.async.wait_group %0;" :: "n"(MD_STAGES - 1) : "memory");
        __syncwarp();
        uint32_t ah[4], al[4];
        md_ldsm4(ah, Ws + (lane & 15) * WL + (lane >> 4) * 8);
        md_ldsm4(al, Ws + 16 * WL + (lane & 15) * WL + (lane >> 4) * 8);
        const bf16* vt = ring.base + (i % MD_STAGES) * MdRing<DV>::STAGE;
#pragma unroll
        for (int np = 0; np < DV / 16; ++np) {
            uint32_t bb[4];
            md_ldsm4_t(bb, vt + ((lane & 7) + ((lane >> 3) & 1) * 8) * LD + np * 16 + (lane >> 4) * 8);
            md_mma(O[2 * np], ah, bb[0], bb[1]);
            md_mma(O[2 * np + 1], ah, bb[2], bb[3]);
            md_mma(O[2 * np], al, bb[0], bb[1]);
            md_mma(O[2 * np + 1], al, bb[2], bb[3]);
        }
        __syncwarp();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float* sum = reinterpret_cast<float*>(md_smem);                 // [warp][HP][DV]
    const int gq = lane >> 2, t4 = lane & 3;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        if (gq + 8 * r >= hpg) continue;
#pragma unroll
        for (int c = 0; c < DV / 8; ++c)
            *reinterpret_cast<float2*>(sum + (size_t)(warp * HP + gq + 8 * r) * DV + c * 8 + 2 * t4) = make_float2(O[c][2 * r], O[c][2 * r + 1]);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < hpg * DV; i += 128) {
        const int r = i / DV, c = i - r * DV;
        if (c >= dv) continue;
        float a = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) a += sum[(size_t)(w * HP + r) * DV + c];
        part[(((size_t)t * H + g * hpg + r) * nsplit + blockIdx.z) * dv + c] = a;
    }
}

__global__ void __launch_bounds__(128) mixed_head_merge_kernel(const float* part, const bf16* row, long long ld, int g_off, bf16* out,
                                                               long long ldo, const int* __restrict__ seq_of_token, int H, int dv,
                                                               int nsplit) {
    pdl_launch();
    pdl_wait();
    const int t = blockIdx.x, n = H * dv;
    const bool live = seq_of_token[t] >= 0;
    for (int i = (blockIdx.y * 128 + threadIdx.x) * 4; i < n; i += gridDim.y * 512) {
        const int h = i / dv, c = i - h * dv;                       // (dv is a multiple of 4)
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live) {
            const float* p = part + ((size_t)t * H + h) * nsplit * dv + c;
#pragma unroll 4
            for (int z = 0; z < nsplit; ++z) {
                const float4 v = *reinterpret_cast<const float4*>(p + (size_t)z * dv);
                a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
            }
            if (g_off >= 0) {
                const float s = 1.0f / (1.0f + md_ex2(-MD_LOG2E * __bfloat162float(row[(size_t)t * ld + g_off + h])));
                a.x *= s; a.y *= s; a.z *= s; a.w *= s;
            }
        }
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a.x, a.y), hi = __floats2bfloat162_rn(a.z, a.w);
        *reinterpret_cast<uint2*>(out + (size_t)t * ldo + i) =
            make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
}

// 1 if the kernels take these sizes.
GG_API gg_mixed_head_decode_takes(int H, int G, int d, int dv, int page_size) {
    return (d > 0 && d <= 128 && d % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0 && page_size == 64 && G > 0 && G <= 65535 &&
            H % G == 0 && H / G <= 16 && H <= 256) ? 1 : 0;
}

template <int D>
static int md_scores(int ntok, int H, int G, int nsplit, cudaStream_t stream, const bf16* row, long long ld, const bf16* k_pool,
                     float* scores, long long ctx_pad, float* ml, const int* positions, const int* seq_of_token,
                     const int* page_table, int max_pages, int d, float scale, float cap, float coef, float every, int window,
                     const PageBounds pb) {
    const size_t smem = (size_t)(16 * (D + 8) + 4 * MD_STAGES * MdRing<D>::STAGE) * sizeof(bf16);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(mixed_head_scores_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return gg_launch(mixed_head_scores_kernel<D>, dim3(ntok, G, nsplit), dim3(128), smem, stream, 1, row, ld, k_pool, scores, ctx_pad,
                     ml, positions, seq_of_token, page_table, max_pages, H, G, d, scale, cap, coef, every, window, nsplit, pb);
}

template <int DV, int HP, bool STAGED>
static int md_values(int ntok, int H, int G, int nsplit, cudaStream_t stream, const float* scores, long long ctx_pad, const float* ml,
                     const bf16* v_pool, float* part, const float* talk, const int* positions, const int* seq_of_token,
                     const int* page_table, int max_pages, int dv, float one, int window, const PageBounds pb) {
    size_t smem = (size_t)(4 * MD_STAGES * MdRing<DV>::STAGE + 4 * 2 * 16 * 24) * sizeof(bf16);
    static_assert((size_t)4 * MD_STAGES * MdRing<DV>::STAGE * sizeof(bf16) >= (size_t)4 * HP * DV * sizeof(float),
                  "the rings must hold the warps' sums");
    smem += ((size_t)H * HP + 2 * ((H + 1) & ~1)) * sizeof(float);
    if (STAGED) smem += (size_t)4 * MD_STAGES * H * 16 * sizeof(float);
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(mixed_head_values_kernel<DV, HP, STAGED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    return gg_launch(mixed_head_values_kernel<DV, HP, STAGED>, dim3(ntok, G, nsplit), dim3(128), smem, stream, 1, scores, ctx_pad, ml, v_pool,
                     part, talk, positions, seq_of_token, page_table, max_pages, H, G, dv, one, window, nsplit, pb);
}

// row [ntok, ld] bfloat16: q [H][d] at column 0, gate logits at g_off (negative: none); pools as elsewhere; out [ntok, H dv]
// bfloat16 with row stride ldo.  Scratch (float32): scores [ntok][H][ctx_pad] (ctx_pad a multiple of 64, at least the longest
// sequence rounded up to pages), ml [ntok][H][nsplit][2], part [ntok][H][nsplit][dv].
GG_API gg_mixed_head_decode(const void* row, long long ld, int g_off, const void* k_pool, const void* v_pool, void* out,
                            long long ldo, const float* talk, const int* positions, const int* seq_of_token,
                            const int* page_table, int max_pages, int page_size, int n_pages, int ntok, int H, int G, int d,
                            int dv, float scale, float cap, float coef, float every, float one, int window, int nsplit,
                            float* scores, long long ctx_pad, float* ml, float* part, int* status, cudaStream_t stream) {
    if (ntok <= 0) return 0;
    if (!gg_mixed_head_decode_takes(H, G, d, dv, page_size) || talk == nullptr || scores == nullptr || ml == nullptr ||
        part == nullptr || nsplit < 1 || nsplit > 64 || cap < 0.f || ldo < (long long)H * dv || (ldo % 4) || (ld % 8) || ctx_pad <= 0 ||
        (ctx_pad % 64) || (coef != 0.f && !(every > 0.f)) ||
        (((uintptr_t)row | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)scores | (uintptr_t)part) & 15) || (((uintptr_t)out) & 7))
        return GG_ERR_ARG;
    const PageBounds pb{n_pages, status};
    const bf16 *r = (const bf16*)row, *kp = (const bf16*)k_pool, *vp = (const bf16*)v_pool;
#define MD_S(D_) md_scores<D_>(ntok, H, G, nsplit, stream, r, ld, kp, scores, ctx_pad, ml, positions, seq_of_token, page_table, \
                               max_pages, d, scale, cap, coef, every, window, pb)
    int rc = d <= 32 ? MD_S(32) : (d <= 64 ? MD_S(64) : MD_S(128));
#undef MD_S
    if (rc != 0) return rc;
    const int hpg = H / G;
#define MD_V(V_, P_) (H <= 32 ? MD_VS(V_, P_, true) : MD_VS(V_, P_, false))
#define MD_VS(V_, P_, S_) md_values<V_, P_, S_>(ntok, H, G, nsplit, stream, (const float*)scores, ctx_pad, (const float*)ml, vp, part, talk, \
                                       positions, seq_of_token, page_table, max_pages, dv, one, window, pb)
#define MD_VH(V_) (hpg <= 4 ? MD_V(V_, 4) : (hpg <= 8 ? MD_V(V_, 8) : MD_V(V_, 16)))
    rc = dv <= 32 ? MD_VH(32) : (dv <= 64 ? MD_VH(64) : MD_VH(128));
#undef MD_VH
#undef MD_V
#undef MD_VS
    if (rc != 0) return rc;
    const int chunks = (H * dv + 511) / 512;
    return gg_launch(mixed_head_merge_kernel, dim3(ntok, chunks > 64 ? 64 : chunks), dim3(128), 0, stream, 1, (const float*)part, r, ld,
                     g_off, (bf16*)out, ldo, seq_of_token, H, dv, nsplit);
}

// 1 if this library was built with checked page tables (the debug build), else 0.
GG_API gg_mixed_head_decode_checked() { return gg_debug_bounds(); }
