// Windowed softmax attention over bfloat16 cache rows [k | v] (the options and the mask of
// window_attention.cu), with the products on tensor cores and everything between them in 32-bit.
//
// The queries are 32-bit and so are the weights; both enter a bfloat16 product as TWO numbers,
// high + low = bf16(x) + bf16(x - bf16(x)), 16 bits of mantissa together, with one product each
// into the same 32-bit sums.  Keys and values are the cache's own bfloat16 numbers, exactly.
//
// wattn_mma_kernel (portions of prompts): a CTA of 4 warps takes 64 (query, head) pairs that
// share a key/value head, 16 a warp; keys go in blocks of 64 ABSOLUTE positions (the kept first
// tokens' before the window's), double buffered with cp.async, one block-table look-up per key,
// asked for two blocks ahead.  S = Q K^T and O += P V are mma.sync m16n8k16; scores, the cap,
// maxima, sums and weights stay in the accumulators' registers.
//
// wattn_decode_kernel (steps of single tokens): a CTA per (token, key/value head, share of the
// keys); a warp takes 32 keys at a time through a ring of its own in shared memory (cp.async, two
// blocks in flight while a third is worked on; no other warp waits for it): four neighbouring
// lanes share a key's row in 16-byte pieces for the scores, and a lane owns four value
// coordinates for the sums.  The warps' states are joined in
// shared memory in warp order; with several CTAs a token (a thread-block cluster, where the step
// leaves SMs idle) the first joins the others' through distributed shared memory in rank order.
#include "common.cuh"

namespace {
constexpr int NO_WINDOW = 1 << 30;
constexpr float LOG2E = 1.4426950408889634f;

struct Args {
    __nv_bfloat16* out;
    long out_ld;
    const float* q;                     // [T, heads * dim]
    const __nv_bfloat16* cache;         // [pages, kv_heads, page_size, dim + vdim]
    const int* block_table;
    const int* seq_of_token;
    const int* positions;
    const float* gate;
    long gate_ld;
    const float* slopes;
    const float* sinks;
    int n_tokens, heads, kv_heads, dim, vdim, page_size, max_pages, num_pages, window, keep_first;
    float scale, out_scale, softcap;
    int gate_per;
    int* status;
};

// 2^x in one instruction (results below the normal range are zero; 2^-inf = 0).
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// cap * tanh(s / cap) = cap - 2 cap / (e^(2 s / cap) + 1): one exponential and one reciprocal, off
// by a few 2^-23 of the cap (an infinite exponential gives cap, zero -cap).
__device__ __forceinline__ float capped(float s, float cap, float twice_log2e_over_cap) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(ex2(s * twice_log2e_over_cap) + 1.0f));
    return fmaf(-2.0f * cap, y, cap);
}
__device__ __forceinline__ float gate_of(const Args& a, size_t row, int h, int j) {
    if (a.gate == nullptr) return a.out_scale;
    const float z = a.gate[row * a.gate_ld + (size_t)h * a.gate_per + (a.gate_per > 1 ? j : 0)];
    return a.out_scale / (1.0f + expf(-z));
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
    return (uint32_t)__cvta_generic_to_shared(p);
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool real) {
    const int bytes = real ? 16 : 0;    // (0: the sixteen bytes are zeroed, nothing is read)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as two bfloat16 pairs: high parts, and what they leave out.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 hf = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - hf.x, y - hf.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// ------------------------------------------------------------------- portions of prompts
constexpr int WM_WARPS = 4;
constexpr int WM_ROWS = 16 * WM_WARPS;      // (query, head) pairs a CTA
constexpr int WM_KB = 64;                   // keys a block

// D: key and value sizes rounded up to a common multiple of 32 (the rest is zero).
// Three CTAs an SM up to 64, two beyond.
template <int D>
__global__ void __launch_bounds__(WM_WARPS * 32, D <= 64 ? 3 : 2) wattn_mma_kernel(Args a, int tq) {
    constexpr int PITCH = D + 8;            // (rows an odd number of 16-byte pieces apart)
    constexpr int NK = D / 16, NV = D / 8;
    extern __shared__ __align__(16) __nv_bfloat16 sm[];
    __nv_bfloat16* Qh = sm;                              // [WM_ROWS][PITCH]
    __nv_bfloat16* Ql = Qh + WM_ROWS * PITCH;
    __nv_bfloat16* Ks = Ql + WM_ROWS * PITCH;            // [2][WM_KB][PITCH]
    __nv_bfloat16* Vs = Ks + 2 * WM_KB * PITCH;
    __shared__ long long rows_s[2][WM_KB];               // a staged key's row of the cache, or -1
    prb_grid_launch_dependents();
    const int hg = a.heads / a.kv_heads;
    const int g = blockIdx.y;
    const int rowlen = a.dim + a.vdim;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r_begin = ((int)gridDim.x - 1 - (int)blockIdx.x) * tq;     // (long contexts first)
    const int r_end = min(a.n_tokens, r_begin + tq);
    const int win = a.window > 0 ? a.window : NO_WINDOW;
    const float cap_k = a.softcap > 0.0f ? 2.0f * LOG2E / a.softcap : 0.0f;
    const int kc = a.dim / 8, vc = a.vdim / 8;           // 16-byte pieces of a key, of a value
    // this thread's first piece of a block and the way to its next one
    const int per = kc + vc;
    const int kk0 = threadIdx.x / per, ch0 = threadIdx.x - kk0 * per;
    const int kstep = blockDim.x / per, cstep = blockDim.x - kstep * per;
    // columns beyond the real sizes stay zero in both buffers
    if (a.dim < D || a.vdim < D) {
        for (int e = threadIdx.x; e < 2 * WM_KB * PITCH; e += blockDim.x) {
            Ks[e] = __float2bfloat16_rn(0.0f);
            Vs[e] = __float2bfloat16_rn(0.0f);
        }
    }
    int r = r_begin;
    while (r < r_end) {
        const int b = a.seq_of_token[r];
        if (b < 0) {                                     // a padding row
            for (int j = threadIdx.x; j < hg * a.vdim; j += blockDim.x)
                a.out[(size_t)r * a.out_ld + (size_t)g * hg * a.vdim + j] = __float2bfloat16_rn(0.0f);
            ++r;
            continue;
        }
        const int p0 = a.positions[r];
        int r1 = r;
        while (r1 + 1 < r_end && a.seq_of_token[r1 + 1] == b && a.positions[r1 + 1] == p0 + (r1 + 1 - r)) ++r1;
        const int nq = r1 - r + 1;
        const int p_last = p0 + nq - 1;
        if (p0 < 0 || p_last >= a.max_pages * a.page_size) {
            if (threadIdx.x == 0) prb_set_status(a.status, PRB_S_POSITION_RANGE, r, p_last, a.max_pages * a.page_size);
            for (int j = threadIdx.x; j < nq * hg * a.vdim; j += blockDim.x) {
                const int qi = j / (hg * a.vdim), rest = j - qi * hg * a.vdim;
                a.out[(size_t)(r + qi) * a.out_ld + (size_t)g * hg * a.vdim + rest] = __float2bfloat16_rn(0.0f);
            }
            r = r1 + 1;
            continue;
        }
        const int lo_min = max(0, p0 - win + 1);
        const int win_start = (lo_min / WM_KB) * WM_KB;
        const int first_end = min(a.keep_first, win_start);
        const int first_blocks = (first_end + WM_KB - 1) / WM_KB;
        const int n_blocks = first_blocks + (p_last - win_start) / WM_KB + 1;
        const int* table = a.block_table + (size_t)b * a.max_pages;
        const int n_pairs = nq * hg;
        // the cache row of key `threadIdx.x` of a block, or -1 where no query of the pass looks
        auto row_of = [&](int blk) -> long long {
            if (threadIdx.x >= WM_KB || blk >= n_blocks) return -1;
            const int j0 = blk < first_blocks ? blk * WM_KB : win_start + (blk - first_blocks) * WM_KB;
            const int j_end = blk < first_blocks ? first_end : p_last + 1;
            const int jj = j0 + (int)threadIdx.x;
            if (jj >= j_end || !(jj >= lo_min || jj < a.keep_first)) return -1;
            const int pg = table[jj / a.page_size];
            if (pg < 0 || pg >= a.num_pages) {
                prb_set_status(a.status, PRB_S_PAGE_RANGE, r, jj, pg);
                return -1;
            }
            return ((long long)pg * a.kv_heads + g) * a.page_size + jj % a.page_size;
        };
        auto stage = [&](int blk) {                      // 16-byte pieces, neighbours of one row together
            const int s = blk & 1;
            int kk = kk0, ch = ch0;
            for (; kk < WM_KB; kk += kstep, ch += cstep) {
                if (ch >= per) {
                    ch -= per;
                    if (++kk >= WM_KB) break;
                }
                const long long row = rows_s[s][kk];
                const __nv_bfloat16* src = a.cache + (size_t)(row < 0 ? 0 : row) * rowlen + ch * 8;
                __nv_bfloat16* dst = ch < kc ? Ks + (s * WM_KB + kk) * PITCH + ch * 8
                                             : Vs + (s * WM_KB + kk) * PITCH + (ch - kc) * 8;
                cp_async16(smem_u32(dst), src, row >= 0);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        __syncthreads();                                 // the pass before is done with shared memory
        if (threadIdx.x < WM_KB) rows_s[0][threadIdx.x] = row_of(0);
        for (int e = threadIdx.x; e < WM_ROWS * (D / 2); e += blockDim.x) {
            const int pair = e / (D / 2), d = (e - pair * (D / 2)) * 2;
            float x = 0.0f, y = 0.0f;
            if (pair < n_pairs && d < a.dim) {           // (dim is even)
                const int qi = pair / hg, hh = pair - qi * hg;
                const float2 v = *reinterpret_cast<const float2*>(
                    a.q + ((size_t)(r + qi) * a.heads + g * hg + hh) * a.dim + d);
                x = v.x * a.scale;
                y = v.y * a.scale;
            }
            uint32_t hi, lo;
            split_pair(x, y, hi, lo);
            *reinterpret_cast<uint32_t*>(Qh + pair * PITCH + d) = hi;
            *reinterpret_cast<uint32_t*>(Ql + pair * PITCH + d) = lo;
        }
        __syncthreads();
        stage(0);
        if (threadIdx.x < WM_KB) rows_s[1][threadIdx.x] = row_of(1);
        // this lane's two rows: pairs warp * 16 + lane / 4 and the one eight further on
        int pi[2];
        float m[2], l[2], slope[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int pair = warp * 16 + (lane >> 2) + 8 * x;
            pi[x] = pair < n_pairs ? p0 + pair / hg : -1;
            slope[x] = (a.slopes && pair < n_pairs) ? a.slopes[g * hg + pair % hg] : 0.0f;
            m[x] = -INFINITY;
            l[x] = 0.0f;
        }
        // positions of the warp's first and last pair: blocks nobody of the warp sees are skipped
        const int w_first = warp * 16 < n_pairs ? p0 + (warp * 16) / hg : -1;
        const int w_last = w_first < 0 ? -1 : p0 + min(n_pairs - 1, warp * 16 + 15) / hg;
        const uint32_t qrow = (uint32_t)((warp * 16 + (lane & 15)) * PITCH + (lane >> 4) * 8) * 2;
        float o[NV][4];
#pragma unroll
        for (int n = 0; n < NV; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
        for (int blk = 0; blk < n_blocks; ++blk) {
            asm volatile("cp.async.wait_all;" ::: "memory");
            __syncthreads();                             // this block is here, the one before consumed
            if (blk + 1 < n_blocks) stage(blk + 1);
            const long long ahead = row_of(blk + 2);
            const int s = blk & 1;
            const int j0 = blk < first_blocks ? blk * WM_KB : win_start + (blk - first_blocks) * WM_KB;
            const int j_end = blk < first_blocks ? first_end : p_last + 1;
            const bool seen = w_last >= 0 && j0 <= w_last &&
                              (j0 + WM_KB - 1 >= w_first - win + 1 || j0 < a.keep_first);
            if (seen) {
                float c[WM_KB / 8][4];
#pragma unroll
                for (int n = 0; n < WM_KB / 8; ++n) c[n][0] = c[n][1] = c[n][2] = c[n][3] = 0.0f;
                // lanes 0-7 / 8-15: a tile's first / second eight dimensions; 16-31: the next tile
                const uint32_t krow = smem_u32(Ks + s * WM_KB * PITCH) +
                    (uint32_t)(((lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
                for (int k = 0; k < NK; ++k) {
                    uint32_t ah[4], al[4];
                    ldsm4(ah, smem_u32(Qh) + qrow + k * 32);
                    ldsm4(al, smem_u32(Ql) + qrow + k * 32);
#pragma unroll
                    for (int n = 0; n < WM_KB / 8; n += 2) {
                        uint32_t bb[4];
                        ldsm4(bb, krow + (uint32_t)(n * 8 * PITCH + k * 16) * 2);
                        mma(c[n], ah, bb[0], bb[1]);
                        mma(c[n], al, bb[0], bb[1]);
                        mma(c[n + 1], ah, bb[2], bb[3]);
                        mma(c[n + 1], al, bb[2], bb[3]);
                    }
                }
                // scores in place; a block wholly inside everybody's view needs no mask
                const bool whole = j0 + WM_KB - 1 <= w_first && j0 + WM_KB <= j_end &&
                                   ((w_last - j0 < win) || j0 + WM_KB <= a.keep_first);
                float mx[2] = {-INFINITY, -INFINITY};
                if (a.softcap > 0.0f) {
#pragma unroll
                    for (int n = 0; n < WM_KB / 8; ++n) {
#pragma unroll
                        for (int x = 0; x < 4; ++x) c[n][x] = capped(c[n][x], a.softcap, cap_k);
                    }
                }
                if (a.slopes != nullptr) {
#pragma unroll
                    for (int n = 0; n < WM_KB / 8; ++n) {
#pragma unroll
                        for (int x = 0; x < 4; ++x)
                            c[n][x] -= slope[x >> 1] *
                                       (float)(pi[x >> 1] - (j0 + n * 8 + (lane & 3) * 2 + (x & 1)));
                    }
                }
                if (!whole) {
#pragma unroll
                    for (int n = 0; n < WM_KB / 8; ++n) {
#pragma unroll
                        for (int x = 0; x < 4; ++x) {
                            const int j = j0 + n * 8 + (lane & 3) * 2 + (x & 1), i = pi[x >> 1];
                            if (!(j < j_end && j <= i && (i - j < win || j < a.keep_first))) c[n][x] = -INFINITY;
                        }
                    }
                }
#pragma unroll
                for (int n = 0; n < WM_KB / 8; ++n) {
#pragma unroll
                    for (int x = 0; x < 4; ++x) mx[x >> 1] = fmaxf(mx[x >> 1], c[n][x]);
                }
                float nb[2];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 1));
                    mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 2));
                    const float nm = fmaxf(m[x], mx[x]);
                    const float f = nm == -INFINITY ? 1.0f : ex2((m[x] - nm) * LOG2E);
                    m[x] = nm;
                    l[x] *= f;
                    nb[x] = nm == -INFINITY ? 0.0f : nm * LOG2E;
#pragma unroll
                    for (int n = 0; n < NV; ++n) {
                        o[n][2 * x] *= f;
                        o[n][2 * x + 1] *= f;
                    }
                }
#pragma unroll
                for (int n = 0; n < WM_KB / 8; ++n) {
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        c[n][x] = ex2(fmaf(c[n][x], LOG2E, -nb[x >> 1]));   // (exp(-inf) = 0)
                        l[x >> 1] += c[n][x];
                    }
                }
                // lanes 0-7 / 8-15: keys 0-7 / 8-15 of a step; 16-31: the next eight coordinates
                const uint32_t vrow = smem_u32(Vs + s * WM_KB * PITCH) +
                    (uint32_t)((lane & 15) * PITCH + (lane >> 4) * 8) * 2;
#pragma unroll
                for (int k = 0; k < WM_KB / 16; ++k) {
                    uint32_t ph[4], pl[4];
                    split_pair(c[2 * k][0], c[2 * k][1], ph[0], pl[0]);
                    split_pair(c[2 * k][2], c[2 * k][3], ph[1], pl[1]);
                    split_pair(c[2 * k + 1][0], c[2 * k + 1][1], ph[2], pl[2]);
                    split_pair(c[2 * k + 1][2], c[2 * k + 1][3], ph[3], pl[3]);
#pragma unroll
                    for (int n = 0; n < NV; n += 2) {
                        uint32_t bb[4];
                        ldsm4t(bb, vrow + (uint32_t)(k * 16 * PITCH + n * 8) * 2);
                        mma(o[n], ph, bb[0], bb[1]);
                        mma(o[n], pl, bb[0], bb[1]);
                        mma(o[n + 1], ph, bb[2], bb[3]);
                        mma(o[n + 1], pl, bb[2], bb[3]);
                    }
                }
            }
            if (threadIdx.x < WM_KB) rows_s[s][threadIdx.x] = ahead;
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int pair = warp * 16 + (lane >> 2) + 8 * x;
            l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
            l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
            if (pair >= n_pairs) continue;
            const int qi = pair / hg, h = g * hg + (pair - qi * hg);
            float f = 1.0f;
            if (a.sinks) {                               // the sink joins the denominator, once
                const float top = fmaxf(m[x], a.sinks[h]);
                f = ex2((m[x] - top) * LOG2E);
                l[x] = l[x] * f + ex2((a.sinks[h] - top) * LOG2E);
            }
            const float inv = l[x] > 0.0f ? f / l[x] : 0.0f;
            __nv_bfloat16* dst = a.out + (size_t)(r + qi) * a.out_ld + (size_t)h * a.vdim;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int j = n * 8 + (lane & 3) * 2;
                if (j >= a.vdim) continue;
                dst[j] = __float2bfloat16_rn(o[n][2 * x] * inv * gate_of(a, r + qi, h, j));
                dst[j + 1] = __float2bfloat16_rn(o[n][2 * x + 1] * inv * gate_of(a, r + qi, h, j + 1));
            }
        }
        r = r1 + 1;
    }
}

int mma_bucket(int dim, int vdim) {
    const int d = (dim > vdim ? dim : vdim);
    return (d + 31) / 32 * 32;
}
bool mma_takes(int heads, int kv_heads, int dim, int vdim) {
    return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && heads / kv_heads <= WM_ROWS && dim > 0 &&
           vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128;
}

// ------------------------------------------------------------------ steps of single tokens
constexpr int WD_WARPS = 4;
constexpr int WD_KEYS = 32;                 // keys a warp takes at a time
constexpr int WD_STAGES = 3;                // blocks in a warp's ring
// Words of shared memory before the rings: queries, the warps' states, the CTA's.
__host__ __device__ inline int decode_ring_at(int q_words, int hg, int vdim) {
    return (q_words + (WD_WARPS + 1) * hg * (vdim + 2) + 3) / 4 * 4;
}

__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float ld_cluster(const float* local, int rank) {
    uint32_t raddr;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(raddr) : "r"(smem_u32(local)), "r"(rank));
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(raddr) : "memory");
    return v;
}
__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

// HG: query heads of a key/value head (or a little more); WIDE: heads beyond 64 numbers (up to
// 128): a lane takes DC 16-byte pieces of a key's row, and a value row is shared by 32 lanes
// instead of 16 (four coordinates a lane).
template <int HG, bool WIDE>
__global__ void __launch_bounds__(WD_WARPS * 32) wattn_decode_kernel(Args a) {
    constexpr int DC = WIDE ? 4 : 2;
    constexpr int LPK = WIDE ? 32 : 16;              // lanes a value row
    constexpr int KPS = 32 / LPK;                    // value rows a step
    constexpr int STAGES = WD_STAGES;
    extern __shared__ __align__(16) float smf[];
    prb_grid_launch_dependents();
    const int hg = a.heads / a.kv_heads;
    const int r = blockIdx.x, g = blockIdx.y;
    const int splits = gridDim.z, split = blockIdx.z;            // the cluster and this CTA's rank
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int QPITCH = 40 * DC;                  // (32 numbers and 8 of padding, DC times: banks)
    const int jpitch = a.vdim + 2;
    const int per = (a.dim + a.vdim) / 8;            // 16-byte pieces of a cache row
    const int pitch = (per | 1) * 8;                 // staged rows an odd number of pieces apart
    float* Qs = smf;                                 // [HG][QPITCH], zero beyond dim
    float* Js = Qs + HG * QPITCH;                    // [WD_WARPS][hg][2 + vdim]
    float* Cs = Js + WD_WARPS * hg * jpitch;         // [hg][2 + vdim]: the CTA's own join
    __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smf + decode_ring_at(HG * QPITCH, hg, a.vdim)) +
                          (size_t)warp * STAGES * WD_KEYS * pitch;       // [STAGES][WD_KEYS][pitch]
    const int rowlen = a.dim + a.vdim;
    __nv_bfloat16* orow = a.out + (size_t)r * a.out_ld + (size_t)g * hg * a.vdim;
    const int b = a.seq_of_token[r];
    const int p = b < 0 ? 0 : a.positions[r];
    if (b < 0 || p < 0 || p >= a.max_pages * a.page_size) {      // a padding row, or a bad one
        if (split > 0) return;                                   // (so for the whole cluster)
        if (b >= 0 && threadIdx.x == 0)
            prb_set_status(a.status, PRB_S_POSITION_RANGE, r, p, a.max_pages * a.page_size);
        for (int j = threadIdx.x; j < hg * a.vdim; j += blockDim.x) orow[j] = __float2bfloat16_rn(0.0f);
        return;
    }
    const int win = a.window > 0 ? a.window : NO_WINDOW;
    const int lo_min = max(0, p - win + 1);
    const int win_start = (lo_min / WD_KEYS) * WD_KEYS;
    const int first_end = min(a.keep_first, win_start);
    const int first_blocks = (first_end + WD_KEYS - 1) / WD_KEYS;
    const int n_blocks = first_blocks + (p - win_start) / WD_KEYS + 1;
    const int* table = a.block_table + (size_t)b * a.max_pages;
    const float cap_k = a.softcap > 0.0f ? 2.0f * LOG2E / a.softcap : 0.0f;
    auto first_key = [&](int blk) {
        return blk < first_blocks ? blk * WD_KEYS : win_start + (blk - first_blocks) * WD_KEYS;
    };
    auto seen = [&](int blk, int j) {
        return blk < n_blocks && j < (blk < first_blocks ? first_end : p + 1) &&
               (p - j < win || j < a.keep_first);
    };
    // the row of this lane's key of a block, or -1
    auto row_of = [&](int blk) -> int {
        const int j = first_key(blk) + lane;
        if (!seen(blk, j)) return -1;
        const int pg = table[j / a.page_size];
        if (pg < 0 || pg >= a.num_pages) {
            prb_set_status(a.status, PRB_S_PAGE_RANGE, r, j, pg);
            return -1;
        }
        return (pg * a.kv_heads + g) * a.page_size + j % a.page_size;
    };
    // this lane's first piece of a block and the way to its next one
    const int kk0 = lane / per, ch0 = lane - kk0 * per;
    const int kstep = 32 / per, cstep = 32 - kstep * per;
    auto stage = [&](int n, int rows) {              // (all lanes take the same number of steps)
        __nv_bfloat16* base = ring + (size_t)(n % STAGES) * WD_KEYS * pitch;
        int kk = kk0, ch = ch0;
        for (int i = 0; i < per; ++i) {
            const int kr = __shfl_sync(0xffffffffu, rows, kk);
            cp_async16(smem_u32(base + kk * pitch + ch * 8),
                       a.cache + (size_t)(kr < 0 ? 0 : kr) * rowlen + ch * 8, kr >= 0);
            kk += kstep;
            ch += cstep;
            if (ch >= per) {
                ch -= per;
                ++kk;
            }
        }
    };
    const int stride = splits * WD_WARPS;
    const int blk_first = split * WD_WARPS + warp;
    // (asked for before the queries)
#pragma unroll
    for (int n = 0; n < STAGES - 1; ++n) {
        if (blk_first + n * stride < n_blocks) stage(n, row_of(blk_first + n * stride));
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    int row_ahead = row_of(blk_first + (STAGES - 1) * stride);
    for (int e = threadIdx.x; e < HG * 32 * DC; e += blockDim.x) {
        const int hh = e / (32 * DC), d = e - hh * 32 * DC;
        Qs[hh * QPITCH + d + d / 32 * 8] = hh < hg && d < a.dim
            ? a.q[((size_t)r * a.heads + g * hg + hh) * a.dim + d] * a.scale : 0.0f;
    }
    float m[HG], l[HG], acc[HG][4], slope[HG];
#pragma unroll
    for (int x = 0; x < HG; ++x) {
        m[x] = -INFINITY;
        l[x] = 0.0f;
        slope[x] = (a.slopes && x < hg) ? a.slopes[g * hg + x] : 0.0f;
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[x][c] = 0.0f;
    }
    const int quad = lane & 3, kc = a.dim / 8;
    const int vsub = lane / LPK, v0 = (lane % LPK) * 4;          // this lane's value row of a step, coordinates
    const bool vlive = v0 < a.vdim;
    __syncthreads();                                 // the queries are in place
    int n = 0;
    for (int blk = blk_first; blk < n_blocks; blk += stride, ++n) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncwarp();                                // this block is here, the one before consumed
        if (blk + (STAGES - 1) * stride < n_blocks) stage(n + STAGES - 1, row_ahead);
        asm volatile("cp.async.commit_group;" ::: "memory");
        row_ahead = row_of(blk + STAGES * stride);
        const __nv_bfloat16* rows = ring + (size_t)(n % STAGES) * WD_KEYS * pitch;
        float s[HG];
#pragma unroll
        for (int x = 0; x < HG; ++x) s[x] = 0.0f;
        float part[4][HG];                           // keys i * 8 + lane / 4, four lanes a key
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
            for (int x = 0; x < HG; ++x) part[i][x] = 0.0f;
        }
#pragma unroll
        for (int c = 0; c < DC; ++c) {
            const int ch = quad * 2 + (c & 1) + 8 * (c >> 1);            // (no two lanes in one bank)
            float kf[4][8];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                uint4 kv = make_uint4(0u, 0u, 0u, 0u);
                if (ch < kc)
                    kv = *reinterpret_cast<const uint4*>(rows + (i * 8 + (lane >> 2)) * pitch + ch * 8);
                kf[i][0] = bf_lo(kv.x); kf[i][1] = bf_hi(kv.x); kf[i][2] = bf_lo(kv.y); kf[i][3] = bf_hi(kv.y);
                kf[i][4] = bf_lo(kv.z); kf[i][5] = bf_hi(kv.z); kf[i][6] = bf_lo(kv.w); kf[i][7] = bf_hi(kv.w);
            }
#pragma unroll
            for (int x = 0; x < HG; ++x) {
                const float4* qp = reinterpret_cast<const float4*>(Qs + x * QPITCH + ch * 8 + ch / 4 * 8);
                const float4 u = qp[0], w = qp[1];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    part[i][x] = fmaf(u.w, kf[i][3], fmaf(u.z, kf[i][2], fmaf(u.y, kf[i][1], fmaf(u.x, kf[i][0], part[i][x]))));
                    part[i][x] = fmaf(w.w, kf[i][7], fmaf(w.z, kf[i][6], fmaf(w.y, kf[i][5], fmaf(w.x, kf[i][4], part[i][x]))));
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
            for (int x = 0; x < HG; ++x) {
                float v = part[i][x];
                v += __shfl_xor_sync(0xffffffffu, v, 1);
                v += __shfl_xor_sync(0xffffffffu, v, 2);
                // to the lane that owns the key: lane i * 8 + k has it from lane 4 k
                const float mine = __shfl_sync(0xffffffffu, v, (lane & 7) * 4);
                if ((lane >> 3) == i) s[x] = mine;
            }
        }
        const int j = first_key(blk) + lane;
        const bool vis = seen(blk, j);
        float e[HG];
#pragma unroll
        for (int x = 0; x < HG; ++x) {
            float v = s[x];
            if (a.softcap > 0.0f) v = capped(v, a.softcap, cap_k);
            v = vis ? v - slope[x] * (float)(p - j) : -INFINITY;
            const float nm = fmaxf(m[x], prb_warp_max(v));
            const float base = nm == -INFINITY ? 0.0f : nm;
            const float f = ex2((m[x] - base) * LOG2E);          // (exp(-inf) = 0)
            e[x] = ex2((v - base) * LOG2E);
            l[x] = l[x] * f + e[x];                              // (a lane's share; summed at the end)
            m[x] = nm;
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[x][c] *= f;
        }
        const __nv_bfloat16* vrow = rows + vsub * pitch + a.dim + (vlive ? v0 : 0);
#pragma unroll 8
        for (int i = 0; i < WD_KEYS / KPS; ++i) {
            const uint2 w = *reinterpret_cast<const uint2*>(vrow + i * KPS * pitch);
            const float u0 = bf_lo(w.x), u1 = bf_hi(w.x), u2 = bf_lo(w.y), u3 = bf_hi(w.y);
#pragma unroll
            for (int x = 0; x < HG; ++x) {
                const float pw = __shfl_sync(0xffffffffu, e[x], i * KPS + vsub);
                acc[x][0] = fmaf(pw, u0, acc[x][0]);
                acc[x][1] = fmaf(pw, u1, acc[x][1]);
                acc[x][2] = fmaf(pw, u2, acc[x][2]);
                acc[x][3] = fmaf(pw, u3, acc[x][3]);
            }
        }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll
    for (int x = 0; x < HG; ++x) {
        if (x >= hg) break;
        float* st = Js + ((size_t)warp * hg + x) * jpitch;
        const float total = prb_warp_sum(l[x]);
        if (lane == 0) {
            st[0] = m[x];
            st[1] = total;
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            float v = acc[x][c];
            if constexpr (KPS == 2) v += __shfl_xor_sync(0xffffffffu, v, 16);
            if (vsub == 0 && vlive) st[2 + v0 + c] = v;
        }
    }
    __syncthreads();
    // the CTA's warps in warp order, then the cluster's CTAs in rank order
    for (int e = threadIdx.x; e < hg * a.vdim; e += blockDim.x) {
        const int hh = e / a.vdim, jv = e - hh * a.vdim;
        float top = -INFINITY, lsum = 0.0f, sum = 0.0f;
#pragma unroll
        for (int w = 0; w < WD_WARPS; ++w) top = fmaxf(top, Js[(w * hg + hh) * jpitch]);
        const float base = top == -INFINITY ? 0.0f : top;
#pragma unroll
        for (int w = 0; w < WD_WARPS; ++w) {
            const float* st = Js + (w * hg + hh) * jpitch;
            const float f = ex2((st[0] - base) * LOG2E);
            lsum = fmaf(st[1], f, lsum);
            sum = fmaf(st[2 + jv], f, sum);
        }
        float* own = Cs + hh * jpitch;
        own[2 + jv] = sum;
        if (jv == 0) {
            own[0] = top;
            own[1] = lsum;
        }
    }
    if (splits > 1) cluster_sync();
    else __syncthreads();
    if (split == 0) {
        for (int e = threadIdx.x; e < hg * a.vdim; e += blockDim.x) {
            const int hh = e / a.vdim, jv = e - hh * a.vdim;
            const float* own = Cs + hh * jpitch;
            float mm[8], ll[8], vv[8], top = -INFINITY;
#pragma unroll
            for (int ss = 0; ss < 8; ++ss) {
                const bool in = ss < splits;
                mm[ss] = !in ? -INFINITY : splits > 1 ? ld_cluster(own, ss) : own[0];
                ll[ss] = !in ? 0.0f : splits > 1 ? ld_cluster(own + 1, ss) : own[1];
                vv[ss] = !in ? 0.0f : splits > 1 ? ld_cluster(own + 2 + jv, ss) : own[2 + jv];
            }
#pragma unroll
            for (int ss = 0; ss < 8; ++ss) top = fmaxf(top, mm[ss]);
            const int h = g * hg + hh;
            if (a.sinks) top = fmaxf(top, a.sinks[h]);
            const float base = top == -INFINITY ? 0.0f : top;
            float lsum = a.sinks ? ex2((a.sinks[h] - base) * LOG2E) : 0.0f, sum = 0.0f;
#pragma unroll
            for (int ss = 0; ss < 8; ++ss) {
                const float f = ex2((mm[ss] - base) * LOG2E);
                lsum = fmaf(ll[ss], f, lsum);
                sum = fmaf(vv[ss], f, sum);
            }
            orow[e] = __float2bfloat16_rn(lsum > 0.0f ? sum / lsum * gate_of(a, r, h, jv) : 0.0f);
        }
    }
    if (splits > 1) cluster_sync();                  // the states have been read: CTAs may leave
}

size_t decode_smem(int HG, int DC, int hg, int dim, int vdim) {
    const int pitch = ((dim + vdim) / 8 | 1) * 8;
    return (size_t)decode_ring_at(HG * 40 * DC, hg, vdim) * 4 + (size_t)WD_WARPS * WD_STAGES * WD_KEYS * pitch * 2;
}
bool decode_takes(int heads, int kv_heads, int dim, int vdim) {
    return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && heads / kv_heads <= 8 && dim > 0 && vdim > 0 &&
           dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128;
}
}  // namespace

// 1 if the tensor-core kernel (portions), bit 1 if the single-token kernel takes these sizes.
PRB_API int prb_wattn_bf16_supports(int heads, int kv_heads, int dim, int vdim) {
    return (mma_takes(heads, kv_heads, dim, vdim) ? 1 : 0) | (decode_takes(heads, kv_heads, dim, vdim) ? 2 : 0);
}

PRB_API int prb_wattn_bf16(void* out, long out_ld, const float* q, const void* cache,
                           const int* block_table, const int* seq_of_token, const int* positions,
                           const float* gate, long gate_ld, const float* slopes, int n_tokens,
                           int heads, int kv_heads, int dim, int vdim, int page_size, int max_pages,
                           int num_pages, int window, int keep_first, int single, float scale,
                           float out_scale, const float* sinks, int gate_per, float softcap,
                           int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (kv_heads <= 0 || kv_heads > 65535 || page_size <= 0 || max_pages <= 0 || num_pages < 0 || window < 0 ||
        keep_first < 0)
        return PRB_E_SIZE;
    if (!(single ? decode_takes(heads, kv_heads, dim, vdim) : mma_takes(heads, kv_heads, dim, vdim)))
        return PRB_E_SIZE;
    if ((long long)num_pages * kv_heads * page_size >= (1LL << 31)) return PRB_E_SIZE;
    if (((uintptr_t)cache) % 16 != 0 || ((uintptr_t)q) % 8 != 0) return PRB_E_ALIGN;
    Args a{(__nv_bfloat16*)out, out_ld, q, (const __nv_bfloat16*)cache, block_table, seq_of_token,
           positions, gate, gate_ld, slopes, sinks, n_tokens, heads, kv_heads, dim, vdim, page_size,
           max_pages, num_pages, window, keep_first, scale, out_scale, softcap, gate_per, status};
    const int hg = heads / kv_heads;
    if (!single) {
        const int tq = WM_ROWS / hg;
        const int d = mma_bucket(dim, vdim);
        const size_t smem = (size_t)(2 * WM_ROWS + 4 * WM_KB) * (d + 8) * 2;
        const dim3 grid((n_tokens + tq - 1) / tq, kv_heads);
#define WMMA(DN)                                                                                 \
    do {                                                                                         \
        if (smem > 40 * 1024)                                                                    \
            cudaFuncSetAttribute(wattn_mma_kernel<DN>,                                           \
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);        \
        wattn_mma_kernel<DN><<<grid, WM_WARPS * 32, smem, stream>>>(a, tq);                      \
    } while (0)
        switch (d) {
            case 32: WMMA(32); break;
            case 64: WMMA(64); break;
            case 96: WMMA(96); break;
            default: WMMA(128); break;
        }
#undef WMMA
        PRB_LAUNCH_CHECK();
        return 0;
    }
    // CTAs a (token, key/value head): as many as the SMs the step would leave idle allow, while a
    // request's keys (at most the window's and the kept ones) still give every CTA a round
    long long most = (long long)max_pages * page_size;
    if (window > 0 && (long long)window + keep_first + WD_KEYS < most) most = (long long)window + keep_first + WD_KEYS;
    const long long rounds = (most + WD_WARPS * WD_KEYS - 1) / (WD_WARPS * WD_KEYS);
    int splits = 1;
    while (splits < 8 && splits + 1 <= rounds &&
           (long long)n_tokens * kv_heads * (splits + 1) <= (dim + vdim <= 128 ? 2LL : 1LL) * prb_sm_count())
        ++splits;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(n_tokens, kv_heads, splits);
    cfg.blockDim = dim3(WD_WARPS * 32);
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = (unsigned)splits;
    cfg.attrs = attr;
    cfg.numAttrs = splits > 1 ? 1 : 0;
#define WD2(HN, WN)                                                                              \
    do {                                                                                         \
        cfg.dynamicSmemBytes = decode_smem(HN, WN ? 4 : 2, hg, dim, vdim);                            \
        if (cfg.dynamicSmemBytes > 40 * 1024)                                                    \
            cudaFuncSetAttribute(wattn_decode_kernel<HN, WN>,                                    \
                                 cudaFuncAttributeMaxDynamicSharedMemorySize,                    \
                                 (int)cfg.dynamicSmemBytes);                                     \
        cudaLaunchKernelEx(&cfg, wattn_decode_kernel<HN, WN>, a);                                \
    } while (0)
#define WD1(HN)                                                                                  \
    do {                                                                                         \
        if (dim <= 64 && vdim <= 64) WD2(HN, false);                                             \
        else WD2(HN, true);                                                                      \
    } while (0)
    switch (hg) {
        case 1: WD1(1); break;
        case 2: WD1(2); break;
        case 3: WD1(3); break;
        case 4: WD1(4); break;
        case 5: WD1(5); break;
        case 6: WD1(6); break;
        default: WD1(8); break;
    }
#undef WD1
#undef WD2
    PRB_LAUNCH_CHECK();
    return 0;
}
