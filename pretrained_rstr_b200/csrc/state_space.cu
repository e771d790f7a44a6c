// Mamba-2's state-space mixer (state-space duality) over a running 32-bit state per request.
//
// The projection of a token is [z | x B C | dt]: z and x are heads * vdim wide, B and C `groups`
// rows of `dim` numbers (head h uses group h / (heads / groups)), dt one number a head.
//
//     xBC = silu(causal convolution per channel of the projected x B C, with a bias)
//     dt  = softplus(dt + dt_bias)            a = exp(-exp(A_log) dt)
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T      y_t = S_t^T C_t + D x_t
//     out = y silu(z), RMS-normed in `parts` equal parts, times a weight (and a constant)
//
// ssm_prepare: convolution and silu (a thread per channel of 8 tokens), step sizes and decays.
// ssm_own / ssm_carry / ssm_out: bfloat16 serving, segments of 64 tokens side by side with every
//   product on tensor cores.  Convolved x, B and C are bfloat16 (operands of products); step sizes,
//   decays, their exponentials, scores and the state are 32-bit, and a 32-bit operand enters a
//   product as TWO bfloat16 numbers, high and low.  A segment's own sums S_own = (w x)^T B with
//   w_j = exp(cum_end - cum_j) dt_j; the carry walks a request's segments; outputs are exp(cum_i)
//   C S_start + sum_(j <= i) (C_i . B_j) exp(cum_i - cum_j) dt_j x_j, cum the running sum of log a.
//   32-bit runs (and sizes these do not take) use the recurrence of decayed_scan.cu instead.
// ssm_finish: norm in parts, a warp per (token, part) or a CTA per token; the saved inputs are brought
//   up to date.
// ssm_step: a step of single tokens in one launch: CTAs (head and share of its value columns,
//   request); state, saved inputs and taps are requested before the kernel waits for the
//   projection; the request's last CTA to arrive norms the token.
// The saved inputs are per-request state, [slots, taps, channels] in 32-bit (projected numbers before
// the convolution's bias): the token at position p lies in row p mod taps, so that saving one never
// touches a number that any CTA of the same step still reads.
#include "decayed_scan.cuh"

namespace {
using namespace dscan;
constexpr int SSM_TAPS = 8;

struct SsmArgs {
    const float* proj; long ld;
    int z_col, x_col, dt_col;        // x_col: the first of inner + 2 groups dim channels
    const float* conv_w;             // [taps, channels]
    const float* conv_b;             // [channels]
    const float* dt_bias; const float* neg_a; const float* d;      // [heads]; neg_a = -exp(A_log)
    float* conv_state;               // [slots, taps, channels], or null (one tap)
    float* state;                    // [slots, heads, vdim, dim]
    const int* seq; const int* q_start; const int* state_slot; const int* positions;
    int n_tokens, n_requests, heads, vdim, dim, groups, taps, n_slots;
    // finish
    float* raw; long raw_ld;         // [T, heads * vdim]: y silu(z) (or y, see ssm_finish)
    const float* norm_w;             // [heads * vdim]
    int parts;
    float eps, out_scale;
    void* out; long out_ld;
    int* status;
};

// The projected value of channel ch `m` tokens before token t (of request b, slot, `back` tokens
// into its portion, at position pos).
__device__ __forceinline__ float past_input(const SsmArgs& a, int channels, int t, int slot, int back,
                                            int pos, int ch, int m) {
    if (m > pos) return 0.0f;
    if (m <= back) return a.proj[(size_t)(t - m) * a.ld + a.x_col + ch];
    return a.conv_state[((size_t)slot * a.taps + (pos - m) % a.taps) * channels + ch];
}

__device__ __forceinline__ void store_as(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_as(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

constexpr int SP_TOKENS = 8;
// grid (tokens / 8, channels / 256 + 1): the last column of CTAs does the step sizes.
// TAPS: the most taps (fewer have weights of zero for the oldest).
template <typename X, int TAPS>
__global__ void __launch_bounds__(256) ssm_prepare_kernel(SsmArgs a, X* __restrict__ xbc, long xbc_ld,
                                                          float* __restrict__ dt_out,
                                                          float* __restrict__ decay_out, int as_log) {
    prb_grid_launch_dependents();
    const int channels = a.heads * a.vdim + 2 * a.groups * a.dim;
    const int t0 = blockIdx.x * SP_TOKENS, nt = min(SP_TOKENS, a.n_tokens - t0);
    if (blockIdx.y == gridDim.y - 1) {
        for (int e = threadIdx.x; e < nt * a.heads; e += blockDim.x) {
            const int tt = e / a.heads, h = e - tt * a.heads;
            const float dt = softplus(a.proj[(size_t)(t0 + tt) * a.ld + a.dt_col + h] + a.dt_bias[h]);
            const float la = a.neg_a[h] * dt;
            dt_out[(size_t)(t0 + tt) * a.heads + h] = dt;
            decay_out[(size_t)(t0 + tt) * a.heads + h] = as_log ? la : expm1f(la);
        }
        return;
    }
    const int ch = blockIdx.y * blockDim.x + threadIdx.x;
    if (ch >= channels) return;
    // w[TAPS - 1] is the current token's; win[j] the value TAPS - 1 - j tokens ago
    float w[TAPS], win[TAPS];
    const int skip = TAPS - a.taps;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = j >= skip ? a.conv_w[(size_t)(j - skip) * channels + ch] : 0.0f;
    const float bias = a.conv_b[ch];
    float cur[SP_TOKENS];
#pragma unroll
    for (int tt = 0; tt < SP_TOKENS; ++tt)
        cur[tt] = tt < nt ? a.proj[(size_t)(t0 + tt) * a.ld + a.x_col + ch] : 0.0f;
    int before = -2;
#pragma unroll
    for (int tt = 0; tt < SP_TOKENS; ++tt) {
        if (tt >= nt) break;
        const int t = t0 + tt, b = a.seq[t];
        if (b < 0) continue;
        if (b != before) {                           // the tile's first token, or another request's
            before = b;
            const int slot = a.state_slot[b], back = t - a.q_start[b], pos = a.positions[t];
            const bool fine = slot >= 0 && slot < a.n_slots;
            if (!fine && threadIdx.x == 0) prb_set_status(a.status, PRB_S_ROW_RANGE, t, slot, a.n_slots);
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j)
                win[j] = j >= skip && fine ? past_input(a, channels, t, slot, back, pos, ch, TAPS - 1 - j) : 0.0f;
        }
        win[TAPS - 1] = cur[tt];
        float s = bias;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) s = fmaf(w[j], win[j], s);
        store_as(xbc + (size_t)t * xbc_ld + ch, silu<X>(s));
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) win[j] = win[j + 1];
    }
}

// ------------------------------------------------------------- portions on tensor cores
using bf16 = __nv_bfloat16;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, "
                 "{%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float low_part(float x) { return x - __bfloat162float(__float2bfloat16_rn(x)); }

struct ChunkArgs {
    SsmArgs s;
    const bf16* xbc; long xbc_ld;
    const float* dt; const float* la;                // [T, heads]
    float* own;                                      // [segments, heads, vdim, dim]
    bf16* start_hi; bf16* start_lo;                  // the same shape: a segment's start as two numbers
    float* seg_decay;                                // [segments, heads]: product of decays minus one
};

// Running sums of log2 a over a segment's tokens, cum_s[64] (zero steps beyond nb), and dt_s.
__device__ __forceinline__ void running_sums(const ChunkArgs& c, int t0, int nb, int hd, float* cum_s,
                                             float* dt_s) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x, i0 = 2 * lane, i1 = i0 + 1;
        const float a0 = i0 < nb ? c.la[(size_t)(t0 + i0) * c.s.heads + hd] : 0.0f;
        const float a1 = i1 < nb ? c.la[(size_t)(t0 + i1) * c.s.heads + hd] : 0.0f;
        dt_s[i0] = i0 < nb ? c.dt[(size_t)(t0 + i0) * c.s.heads + hd] : 0.0f;
        dt_s[i1] = i1 < nb ? c.dt[(size_t)(t0 + i1) * c.s.heads + hd] : 0.0f;
        float sum = a0 + a1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        const float log2e = 1.4426950408889634f;
        cum_s[i1] = sum * log2e;
        cum_s[i0] = (sum - a1) * log2e;
    }
}

__device__ __forceinline__ bool chunk_of(const ChunkArgs& c, int z, int& b, int& s, int& nseg, int& t0, int& nb) {
    if (!find_segment(c.s.q_start, c.s.n_requests, z, b, s, nseg)) return false;
    const int first = c.s.q_start[b], end = c.s.q_start[b + 1];
    if (first < 0 || end > c.s.n_tokens) return false;
    t0 = first + s * DS_SEG;
    nb = min(DS_SEG, end - t0);
    return true;
}

// rows x n bfloat16 numbers from global rows into shared rows of `pitch` numbers, zeros beyond nb.
__device__ __forceinline__ void fetch_rows(bf16* dst, int pitch, const bf16* src, long ld, int n, int nb,
                                           int rows) {
    const int per = n / 8;
    for (int e = threadIdx.x; e < rows * per; e += blockDim.x) {
        const int r = e / per, i = (e - r * per) * 8;
        if (r < nb) copy16(dst + r * pitch + i, src + (size_t)r * ld + i);
        else *reinterpret_cast<uint4*>(dst + r * pitch + i) = make_uint4(0, 0, 0, 0);
    }
}

// Grid (head, segment); 128 threads: a warp takes 16 value rows at a time.
__global__ void __launch_bounds__(128) ssm_own_kernel(ChunkArgs c) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    prb_grid_launch_dependents();
    const int hd = blockIdx.x;
    int b, s, nseg, t0, nb;
    if (!chunk_of(c, blockIdx.y, b, s, nseg, t0, nb)) return;
    const int V = c.s.vdim, N = c.s.dim, vp = V + 8, np = N + 8;
    bf16* xh = reinterpret_cast<bf16*>(smem_raw);    // [64][V + 8]
    bf16* xl = xh + DS_SEG * vp;
    bf16* bs = xl + DS_SEG * vp;                     // [64][N + 8]
    float* cum_s = reinterpret_cast<float*>(bs + DS_SEG * np);
    float* dt_s = cum_s + DS_SEG;
    const bf16* row = c.xbc + (size_t)t0 * c.xbc_ld;
    const int inner = c.s.heads * V, g = hd / (c.s.heads / c.s.groups);
    fetch_rows(xh, vp, row + hd * V, c.xbc_ld, V, nb, DS_SEG);
    fetch_rows(bs, np, row + inner + g * N, c.xbc_ld, N, nb, DS_SEG);
    copy_commit();
    running_sums(c, t0, nb, hd, cum_s, dt_s);
    copy_wait<0>();
    __syncthreads();
    const float end = cum_s[DS_SEG - 1];
    if (threadIdx.x == 0) c.seg_decay[(size_t)blockIdx.y * c.s.heads + hd] = expm1f(end * 0.6931471805599453f);
    for (int e = threadIdx.x; e < DS_SEG * (V / 2); e += blockDim.x) {
        const int r = e / (V / 2), i = (e - r * (V / 2)) * 2;
        const float w = r < nb ? exp2f(end - cum_s[r]) * dt_s[r] : 0.0f;
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xh + r * vp + i);
        const float x0 = w * __bfloat162float(x.x), x1 = w * __bfloat162float(x.y);
        *reinterpret_cast<uint32_t*>(xh + r * vp + i) = pack2(x0, x1);
        *reinterpret_cast<uint32_t*>(xl + r * vp + i) = pack2(low_part(x0), low_part(x1));
    }
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* own = c.own + ((size_t)blockIdx.y * c.s.heads + hd) * V * N;
    const int kmax = (nb + 15) / 16 * 16;
    for (int v0 = warp * 16; v0 < V; v0 += 64) {
        for (int n0 = 0; n0 < N; n0 += 64) {
            const int nn = min(64, N - n0) / 16;     // pairs of 8-column tiles
            float acc[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
            for (int k0 = 0; k0 < kmax; k0 += 16) {
                // A = (w x)^T: rows v, columns j; stored [j][v], so transposed on the way
                uint32_t ah[4], al[4];
                const int ar = k0 + (lane & 7) + ((lane >> 4) & 1) * 8, ac = v0 + ((lane >> 3) & 1) * 8;
                ldsm4t(ah, xh + ar * vp + ac);
                ldsm4t(al, xl + ar * vp + ac);
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    if (p < nn) {
                        uint32_t bb[4];
                        ldsm4t(bb, bs + (k0 + (lane & 15)) * np + n0 + p * 16 + ((lane >> 4) & 1) * 8);
                        mma16816(acc[2 * p], ah, bb[0], bb[1]);
                        mma16816(acc[2 * p], al, bb[0], bb[1]);
                        mma16816(acc[2 * p + 1], ah, bb[2], bb[3]);
                        mma16816(acc[2 * p + 1], al, bb[2], bb[3]);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                if (i < 2 * nn) {
                    const int n = n0 + i * 8 + (lane & 3) * 2, v = v0 + (lane >> 2);
                    *reinterpret_cast<float2*>(own + (size_t)v * N + n) = make_float2(acc[i][0], acc[i][1]);
                    *reinterpret_cast<float2*>(own + (size_t)(v + 8) * N + n) = make_float2(acc[i][2], acc[i][3]);
                }
            }
        }
    }
}

// A thread per four state numbers of a (head, request); leaves every segment's start as two
// bfloat16 numbers and the state after the last segment in the slot.
__global__ void ssm_carry_kernel(ChunkArgs c) {
    prb_grid_launch_dependents();
    const int hd = blockIdx.x, b = blockIdx.y;
    const int t0 = c.s.q_start[b], t1 = c.s.q_start[b + 1];
    if (t1 <= t0 || t0 < 0 || t1 > c.s.n_tokens) return;
    const int slot = c.s.state_slot[b];
    if (slot < 0 || slot >= c.s.n_slots) {
        if (threadIdx.x == 0) prb_set_status(c.s.status, PRB_S_ROW_RANGE, t0, slot, c.s.n_slots);
        return;
    }
    int base = 0;
    for (int bb = 0; bb < b; ++bb) {
        const int n = c.s.q_start[bb + 1] - c.s.q_start[bb];
        base += n > 0 ? (n + DS_SEG - 1) / DS_SEG : 0;
    }
    const int nseg = (t1 - t0 + DS_SEG - 1) / DS_SEG;
    const size_t per_head = (size_t)c.s.vdim * c.s.dim, per_state = (size_t)c.s.heads * per_head;
    const size_t e = ((size_t)blockIdx.z * blockDim.x + threadIdx.x) * 4;
    if (e >= per_head) return;
    const size_t at = (size_t)hd * per_head + e;
    float* st = c.s.state + (size_t)slot * per_state + at;
    float4 S = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (c.s.positions[t0] > 0) S = *reinterpret_cast<const float4*>(st);
    auto leave = [&](int s) {
        const size_t to = (size_t)(base + s) * per_state + at;
        *reinterpret_cast<uint2*>(c.start_hi + to) = make_uint2(pack2(S.x, S.y), pack2(S.z, S.w));
        *reinterpret_cast<uint2*>(c.start_lo + to) =
            make_uint2(pack2(low_part(S.x), low_part(S.y)), pack2(low_part(S.z), low_part(S.w)));
    };
    auto join = [&](const float4& o, float p) {
        S.x += fmaf(p, S.x, o.x);
        S.y += fmaf(p, S.y, o.y);
        S.z += fmaf(p, S.z, o.z);
        S.w += fmaf(p, S.w, o.w);
    };
    int s = 0;
    for (; s + 4 <= nseg; s += 4) {                  // four segments' numbers requested at a time
        float4 o[4];
        float p[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[i] = *reinterpret_cast<const float4*>(c.own + (size_t)(base + s + i) * per_state + at);
            p[i] = c.seg_decay[(size_t)(base + s + i) * c.s.heads + hd];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            leave(s + i);
            join(o[i], p[i]);
        }
    }
    for (; s < nseg; ++s) {
        leave(s);
        join(*reinterpret_cast<const float4*>(c.own + (size_t)(base + s) * per_state + at),
             c.seg_decay[(size_t)(base + s) * c.s.heads + hd]);
    }
    *reinterpret_cast<float4*>(st) = S;
}

// Grid (head, segment); 256 threads: warps w and w + 4 share 16 tokens, each with half of the value
// columns.  VT: 8-column tiles a warp has room for.
template <int VT>
__global__ void __launch_bounds__(256) ssm_out_kernel(ChunkArgs c) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    prb_grid_launch_dependents();
    const int hd = blockIdx.x;
    int b, s, nseg, t0, nb;
    if (!chunk_of(c, blockIdx.y, b, s, nseg, t0, nb)) return;
    const int V = c.s.vdim, N = c.s.dim, vp = V + 8, np = N + 8;
    bf16* cs = reinterpret_cast<bf16*>(smem_raw);    // [64][N + 8]
    bf16* bs = cs + DS_SEG * np;
    bf16* xs = bs + DS_SEG * np;                     // [64][V + 8]
    bf16* sh = xs + DS_SEG * vp;                     // [V][N + 8]
    bf16* sl = sh + V * np;
    float* cum_s = reinterpret_cast<float*>(sl + V * np);
    float* dt_s = cum_s + DS_SEG;
    const bf16* row = c.xbc + (size_t)t0 * c.xbc_ld;
    const int inner = c.s.heads * V, gn = c.s.groups * N, g = hd / (c.s.heads / c.s.groups);
    const bool started = s > 0 || c.s.positions[t0] > 0;
    fetch_rows(cs, np, row + inner + gn + g * N, c.xbc_ld, N, nb, DS_SEG);
    fetch_rows(bs, np, row + inner + g * N, c.xbc_ld, N, nb, DS_SEG);
    fetch_rows(xs, vp, row + hd * V, c.xbc_ld, V, nb, DS_SEG);
    if (started) {
        const size_t at = ((size_t)blockIdx.y * c.s.heads + hd) * V * N;
        fetch_rows(sh, np, c.start_hi + at, N, N, V, V);
        fetch_rows(sl, np, c.start_lo + at, N, N, V, V);
    }
    copy_commit();
    running_sums(c, t0, nb, hd, cum_s, dt_s);
    copy_wait<0>();
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3;
    const int r0 = warp * 16;
    const int v_lo = (threadIdx.x >> 7) * VT * 8, v_n = min(V - v_lo, VT * 8);   // this warp's columns
    if (r0 >= nb || v_n <= 0) return;
    const int i0 = r0 + (lane >> 2), i1 = i0 + 8;    // this lane's token rows
    // the gates, asked for before the products
    float2 z[VT][2];
#pragma unroll
    for (int v = 0; v < VT; ++v)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = half ? i1 : i0;
            z[v][half] = v * 8 < v_n && i < nb
                ? *reinterpret_cast<const float2*>(c.s.proj + (size_t)(t0 + i) * c.s.ld + c.s.z_col + hd * V + v_lo +
                                                   v * 8 + (lane & 3) * 2)
                : make_float2(0.0f, 0.0f);
        }
    float acc[VT][4];
#pragma unroll
    for (int i = 0; i < VT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
    float gm[8][4];                                  // C B^T: 16 tokens x 64
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) gm[i][j] = 0.0f;
    for (int k0 = 0; k0 < N; k0 += 16) {
        uint32_t ca[4];
        ldsm4(ca, cs + (r0 + (lane & 15)) * np + k0 + (lane >> 4) * 8);
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            if (p <= warp) {                         // tokens j up to the warp's own
                uint32_t bb[4];
                ldsm4(bb, bs + (p * 16 + (lane & 7) + (lane >> 4) * 8) * np + k0 + ((lane >> 3) & 1) * 8);
                mma16816(gm[2 * p], ca, bb[0], bb[1]);
                mma16816(gm[2 * p + 1], ca, bb[2], bb[3]);
            }
        }
        if (started) {
#pragma unroll
            for (int p = 0; p < VT / 2; ++p) {
                if (p * 16 < v_n) {
                    const int at = (v_lo + p * 16 + (lane & 7) + (lane >> 4) * 8) * np + k0 + ((lane >> 3) & 1) * 8;
                    uint32_t hh[4], ll[4];
                    ldsm4(hh, sh + at);
                    ldsm4(ll, sl + at);
                    mma16816(acc[2 * p], ca, hh[0], hh[1]);
                    mma16816(acc[2 * p], ca, ll[0], ll[1]);
                    mma16816(acc[2 * p + 1], ca, hh[2], hh[3]);
                    mma16816(acc[2 * p + 1], ca, ll[2], ll[3]);
                }
            }
        }
    }
    const float cum0 = cum_s[i0], cum1 = cum_s[i1];
    if (started) {
        const float e0 = exp2f(cum0), e1 = exp2f(cum1);
#pragma unroll
        for (int i = 0; i < VT; ++i) {
            acc[i][0] *= e0; acc[i][1] *= e0;
            acc[i][2] *= e1; acc[i][3] *= e1;
        }
    }
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        if (p > warp) break;
        uint32_t mh[4], ml[4];
        float w[2][4];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int j0 = p * 16 + q * 8 + (lane & 3) * 2, j1 = j0 + 1;
            const float* gq = gm[2 * p + q];
            w[q][0] = j0 <= i0 ? gq[0] * exp2f(cum0 - cum_s[j0]) * dt_s[j0] : 0.0f;
            w[q][1] = j1 <= i0 ? gq[1] * exp2f(cum0 - cum_s[j1]) * dt_s[j1] : 0.0f;
            w[q][2] = j0 <= i1 ? gq[2] * exp2f(cum1 - cum_s[j0]) * dt_s[j0] : 0.0f;
            w[q][3] = j1 <= i1 ? gq[3] * exp2f(cum1 - cum_s[j1]) * dt_s[j1] : 0.0f;
        }
        mh[0] = pack2(w[0][0], w[0][1]); ml[0] = pack2(low_part(w[0][0]), low_part(w[0][1]));
        mh[1] = pack2(w[0][2], w[0][3]); ml[1] = pack2(low_part(w[0][2]), low_part(w[0][3]));
        mh[2] = pack2(w[1][0], w[1][1]); ml[2] = pack2(low_part(w[1][0]), low_part(w[1][1]));
        mh[3] = pack2(w[1][2], w[1][3]); ml[3] = pack2(low_part(w[1][2]), low_part(w[1][3]));
#pragma unroll
        for (int v = 0; v < VT / 2; ++v) {
            if (v * 16 < v_n) {
                uint32_t xx[4];
                ldsm4t(xx, xs + (p * 16 + (lane & 15)) * vp + v_lo + v * 16 + (lane >> 4) * 8);
                mma16816(acc[2 * v], mh, xx[0], xx[1]);
                mma16816(acc[2 * v], ml, xx[0], xx[1]);
                mma16816(acc[2 * v + 1], mh, xx[2], xx[3]);
                mma16816(acc[2 * v + 1], ml, xx[2], xx[3]);
            }
        }
    }
    const float dd = c.s.d[hd];
#pragma unroll
    for (int v = 0; v < VT; ++v) {
        if (v * 8 < v_n) {
            const int col = v_lo + v * 8 + (lane & 3) * 2;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int i = half ? i1 : i0;
                if (i < nb) {
                    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xs + i * vp + col);
                    const float y0 = fmaf(dd, __bfloat162float(x.x), acc[v][2 * half]);
                    const float y1 = fmaf(dd, __bfloat162float(x.y), acc[v][2 * half + 1]);
                    *reinterpret_cast<float2*>(c.s.raw + (size_t)(t0 + i) * c.s.raw_ld + hd * V + col) =
                        make_float2(y0 * silu<bf16>(z[v][half].x), y1 * silu<bf16>(z[v][half].y));
                }
            }
        }
    }
}

// ----------------------------------------------------------------------------- finish
// A part of a token's row by the warp: the gated numbers (or, with z, the ungated ones) stay in
// registers while they fit (up to 2,048, in pieces of four).
constexpr int FIN_PIECES = 16;
template <typename O>
__device__ __forceinline__ void norm_part_warp(const SsmArgs& a, const float* row, const float* z, O* o, int lo,
                                               int part, int lane) {
    if (part % 4 == 0 && part <= FIN_PIECES * 128 && (lo | a.raw_ld | a.out_ld) % 4 == 0 && z == nullptr &&
        (((uintptr_t)a.raw | (uintptr_t)a.norm_w) % 16) == 0 && ((uintptr_t)a.out) % (4 * sizeof(O)) == 0) {
        float4 y[FIN_PIECES];
        float ss = 0.0f;
#pragma unroll
        for (int p = 0; p < FIN_PIECES; ++p) {
            const int i = p * 128 + lane * 4;
            y[p] = i < part ? *reinterpret_cast<const float4*>(row + lo + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll
        for (int p = 0; p < FIN_PIECES; ++p)
            ss = fmaf(y[p].x, y[p].x, fmaf(y[p].y, y[p].y, fmaf(y[p].z, y[p].z, fmaf(y[p].w, y[p].w, ss))));
        const float inv = a.out_scale / sqrtf(prb_warp_sum(ss) / (float)part + a.eps);
#pragma unroll
        for (int p = 0; p < FIN_PIECES; ++p) {
            const int i = p * 128 + lane * 4;
            if (i < part) {
                const float4 w = *reinterpret_cast<const float4*>(a.norm_w + lo + i);
                prb_store4(o + lo + i, y[p].x * inv * w.x, y[p].y * inv * w.y, y[p].z * inv * w.z,
                           y[p].w * inv * w.w);
            }
        }
        return;
    }
    float ss = 0.0f;
    for (int i = lane; i < part; i += 32) {
        const float y = z ? row[lo + i] * silu<O>(z[lo + i]) : row[lo + i];
        ss = fmaf(y, y, ss);
    }
    const float inv = a.out_scale / sqrtf(prb_warp_sum(ss) / (float)part + a.eps);
    for (int i = lane; i < part; i += 32) {
        const float y = z ? row[lo + i] * silu<O>(z[lo + i]) : row[lo + i];
        o[lo + i] = prb_from_float<O>(y * inv * a.norm_w[lo + i]);
    }
}

// Every part of one token's row by the CTA (few parts: the CTA a part; many: a warp a part).
constexpr int FIN_KEPT = 4;
template <typename O>
__device__ __forceinline__ void norm_row_cta(const SsmArgs& a, const float* row, int t, float* scratch) {
    const int part = a.heads * a.vdim / a.parts;
    O* o = (O*)a.out + (size_t)t * a.out_ld;
    if (a.parts >= 4) {
        for (int p = threadIdx.x >> 5; p < a.parts; p += blockDim.x >> 5)
            norm_part_warp<O>(a, row, nullptr, o, p * part, part, threadIdx.x & 31);
        return;
    }
    for (int p = 0; p < a.parts; ++p) {
        const int lo = p * part;
        float y[FIN_KEPT], ss = 0.0f;
#pragma unroll
        for (int k = 0; k < FIN_KEPT; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            y[k] = i < part ? row[lo + i] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < FIN_KEPT; ++k) ss = fmaf(y[k], y[k], ss);
        for (int i = threadIdx.x + FIN_KEPT * blockDim.x; i < part; i += blockDim.x)
            ss = fmaf(row[lo + i], row[lo + i], ss);
        ss = prb_block_sum(ss, scratch);
        const float inv = a.out_scale / sqrtf(ss / (float)part + a.eps);
#pragma unroll
        for (int k = 0; k < FIN_KEPT; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            if (i < part) o[lo + i] = prb_from_float<O>(y[k] * inv * a.norm_w[lo + i]);
        }
        for (int i = threadIdx.x + FIN_KEPT * blockDim.x; i < part; i += blockDim.x)
            o[lo + i] = prb_from_float<O>(row[lo + i] * inv * a.norm_w[lo + i]);
    }
}

// A long part of a token's row by a CTA of FIN_WIDE threads.
constexpr int FIN_WIDE = 256;
template <typename O>
__device__ __forceinline__ void norm_part_cta(const SsmArgs& a, const float* row, const float* z, O* o, int lo,
                                              int part, float* scratch) {
    constexpr int KEPT = 16;
    float y[KEPT], ss = 0.0f;
    auto value = [&](int i) { return z ? row[lo + i] * silu<O>(z[lo + i]) : row[lo + i]; };
#pragma unroll
    for (int k = 0; k < KEPT; ++k) {
        const int i = threadIdx.x + k * FIN_WIDE;
        y[k] = i < part ? value(i) : 0.0f;
    }
#pragma unroll
    for (int k = 0; k < KEPT; ++k) ss = fmaf(y[k], y[k], ss);
    for (int i = threadIdx.x + KEPT * FIN_WIDE; i < part; i += FIN_WIDE) ss = fmaf(value(i), value(i), ss);
    ss = prb_block_sum(ss, scratch);
    const float inv = a.out_scale / sqrtf(ss / (float)part + a.eps);
#pragma unroll
    for (int k = 0; k < KEPT; ++k) {
        const int i = threadIdx.x + k * FIN_WIDE;
        if (i < part) o[lo + i] = prb_from_float<O>(y[k] * inv * a.norm_w[lo + i]);
    }
    for (int i = threadIdx.x + KEPT * FIN_WIDE; i < part; i += FIN_WIDE)
        o[lo + i] = prb_from_float<O>(value(i) * inv * a.norm_w[lo + i]);
}

// Warps (token, part), or CTAs where a part is longer than a warp keeps; behind them CTAs that save
// inputs: (request, one of its portion's last `taps` tokens, 512 channels).
constexpr int FIN_WARPS = 4, SAVE_CHANNELS = 512;
template <typename O, bool WIDE>
__global__ void __launch_bounds__(WIDE ? FIN_WIDE : FIN_WARPS * 32)
ssm_finish_kernel(SsmArgs a, int gate_here, int norm_blocks) {
    __shared__ float scratch[32];
    prb_grid_launch_dependents();
    if ((int)blockIdx.x >= norm_blocks) {
        const int channels = a.heads * a.vdim + 2 * a.groups * a.dim;
        const int pieces = (channels + SAVE_CHANNELS - 1) / SAVE_CHANNELS;
        int e = blockIdx.x - norm_blocks;
        const int piece = e % pieces;
        e /= pieces;
        const int back = e % a.taps, b = e / a.taps;
        const int t = a.q_start[b + 1] - 1 - back, slot = a.state_slot[b];
        if (t < a.q_start[b] || t < 0 || t >= a.n_tokens || slot < 0 || slot >= a.n_slots) return;
        float* st = a.conv_state + ((size_t)slot * a.taps + a.positions[t] % a.taps) * channels;
        const float* from = a.proj + (size_t)t * a.ld + a.x_col;
        const int end = min(channels, (piece + 1) * SAVE_CHANNELS);
#pragma unroll 4
        for (int ch = piece * SAVE_CHANNELS + (int)threadIdx.x; ch < end; ch += blockDim.x) st[ch] = from[ch];
        return;
    }
    const long unit = WIDE ? blockIdx.x : (long)blockIdx.x * FIN_WARPS + (threadIdx.x >> 5);
    if (unit >= (long)a.n_tokens * a.parts) return;
    const int t = (int)(unit / a.parts), p = (int)(unit - (long)t * a.parts);
    if (a.seq[t] < 0) return;
    const int part = a.heads * a.vdim / a.parts;
    const float* row = a.raw + (size_t)t * a.raw_ld;
    const float* z = gate_here ? a.proj + (size_t)t * a.ld + a.z_col : nullptr;
    O* o = (O*)a.out + (size_t)t * a.out_ld;
    if (WIDE) norm_part_cta<O>(a, row, z, o, p * part, part, scratch);
    else norm_part_warp<O>(a, row, z, o, p * part, part, threadIdx.x & 31);
}

// ------------------------------------------------------------------- single tokens
struct StepArgs {
    SsmArgs s;
    int splits, cols, lanes;         // a head's columns over `splits` CTAs of `cols`
    int* arrived;                    // [requests], zero between launches
};

constexpr int SS_CC = 4;             // value columns a thread holds
template <int KPL, int TAPS, typename O>
__global__ void __launch_bounds__(512, KPL == 4 ? 2 : 1) ssm_step_kernel(StepArgs g) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    __shared__ int last_s;
    const SsmArgs& a = g.s;
    const int L = g.lanes, dp = L * KPL, N = a.dim, V = a.vdim, cols = g.cols;
    float* q_s = sm;                                 // [dp] C
    float* k_s = q_s + dp;                           // [dp] B
    float* v_s = k_s + dp;                           // [cols]
    float* h_s = v_s + cols;                         // [taps][cols + 2 N]: saved inputs' share of the sum
    prb_grid_launch_dependents();
    const int hd = blockIdx.x / g.splits, cg = blockIdx.x % g.splits, b = blockIdx.y;
    // (the step's description, the state and the saved inputs lie behind launches that have
    // ended: they are read before the wait)
    const int t = a.q_start[b], t1 = a.q_start[b + 1], slot = a.state_slot[b];
    const bool run = t1 > t && t >= 0 && t1 <= a.n_tokens && slot >= 0 && slot < a.n_slots;
    const int pos = run ? a.positions[t] : 0;
    const int ln = threadIdx.x % L, cl = threadIdx.x / L;
    const int c0 = cg * cols + cl * SS_CC;
    const bool mine = cl * SS_CC < cols && c0 < V;
    float* sp = a.state + ((size_t)(run ? slot : 0) * a.heads + hd) * V * N;
    float S[SS_CC][KPL];
    load_state<SS_CC, KPL>(S, run && pos > 0 && mine ? sp : nullptr, ln, c0, N, V);
    const int inner = a.heads * V, channels = inner + 2 * a.groups * N, grp = hd / (a.heads / a.groups);
    const int first = cg * cols, live = max(0, min(cols, V - first));
    auto channel_of = [&](int i) {                   // [own x columns | B | C] -> channel
        return i < live ? hd * V + first + i : i < live + N ? inner + grp * N + (i - live)
                                                            : inner + a.groups * N + grp * N + (i - live - N);
    };
    const int todo = live + 2 * N;
    for (int i = threadIdx.x; i < todo; i += blockDim.x) {
        const int ch = channel_of(i);
        float s = a.conv_b[ch], w[TAPS - 1], u[TAPS - 1];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int m = a.taps - 1 - j;            // tokens ago
            const bool have = run && m >= 1 && m <= pos;
            w[j] = have ? a.conv_w[(size_t)j * channels + ch] : 0.0f;
            u[j] = have ? a.conv_state[((size_t)slot * a.taps + (pos - m) % a.taps) * channels + ch] : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) s = fmaf(w[j], u[j], s);
        h_s[i] = s;
        h_s[todo + i] = a.conv_w[(size_t)(a.taps - 1) * channels + ch];
    }
    const float dtb = a.dt_bias[hd], na = a.neg_a[hd], dd = a.d[hd];
    prb_grid_wait();
    if (!run) {
        if (t1 > t && threadIdx.x == 0) prb_set_status(a.status, PRB_S_ROW_RANGE, t, slot, a.n_slots);
        return;
    }
    const float* row = a.proj + (size_t)t * a.ld;
    // the column of this lane's sum, and its gate
    const int held = held_column<SS_CC>(ln, L);
    const bool writes = mine && (ln & (L / SS_CC - 1)) == 0 && cl * SS_CC + held < live;
    const float z = writes ? row[a.z_col + hd * V + c0 + held] : 0.0f;
    for (int i = threadIdx.x; i < todo; i += blockDim.x) {   // (the same thread as above)
        const float in = row[a.x_col + channel_of(i)];
        const float u = silu<O>(fmaf(h_s[todo + i], in, h_s[i]));
        // (a channel is saved by the one CTA that owns it; B and C by the group's first)
        if (a.taps > 1 && (i < live || (cg == 0 && hd % (a.heads / a.groups) == 0)))
            a.conv_state[((size_t)slot * a.taps + pos % a.taps) * channels + channel_of(i)] = in;
        if (i < live) v_s[i] = u;
        else if (i < live + N) k_s[i - live] = u;
        else q_s[i - live - N] = u;
    }
    for (int i = N + threadIdx.x; i < dp; i += blockDim.x) q_s[i] = k_s[i] = 0.0f;
    const float dt = softplus(row[a.dt_col + hd] + dtb);
    const float c1 = expm1f(na * dt);
    __syncthreads();
    float v[SS_CC], part[SS_CC];
#pragma unroll
    for (int j = 0; j < SS_CC; ++j) v[j] = mine && cl * SS_CC + j < live ? v_s[cl * SS_CC + j] * dt : 0.0f;
    advance<SS_CC, KPL, false, true>(S, k_s + ln * KPL, &c1, q_s + ln * KPL, v, part);
    const float sum = close_columns<SS_CC>(part, ln, L);
    if (writes)
        a.raw[(size_t)t * a.raw_ld + hd * V + c0 + held] = fmaf(dd, v_s[cl * SS_CC + held], sum) * silu<O>(z);
    if (mine) store_state<SS_CC, KPL>(S, sp, ln, c0, N, V);
    // the request's last CTA to arrive norms the token
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        const int n = atomicAdd(&g.arrived[b], 1);
        last_s = n == (int)gridDim.x - 1;
    }
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    if (threadIdx.x == 0) g.arrived[b] = 0;
    norm_row_cta<O>(a, a.raw + (size_t)t * a.raw_ld, t, scratch);
}

size_t own_smem(int V, int N) {
    return (size_t)DS_SEG * (2 * (V + 8) + (N + 8)) * 2 + 2 * DS_SEG * sizeof(float);
}
size_t out_smem(int V, int N) {
    return ((size_t)DS_SEG * (2 * (N + 8) + (V + 8)) + 2 * (size_t)V * (N + 8)) * 2 + 2 * DS_SEG * sizeof(float);
}
bool sizes_ok(const SsmArgs& a) {
    return a.heads > 0 && a.vdim > 0 && a.dim > 0 && a.groups > 0 && a.heads % a.groups == 0 && a.taps >= 1 &&
           a.taps <= SSM_TAPS && a.n_requests <= 65535 && (a.taps == 1 || a.conv_state != nullptr) &&
           a.parts > 0 && (a.heads * a.vdim) % a.parts == 0;
}
}  // namespace

PRB_API int prb_ssm_max_taps() { return SSM_TAPS; }

// 1: the tensor-core kernels take heads of these sizes.
PRB_API int prb_ssm_chunk_supports(int vdim, int dim) {
    return vdim > 0 && dim > 0 && vdim % 16 == 0 && dim % 16 == 0 && vdim <= 128 &&
           out_smem(vdim, dim) <= 200 * 1024 && own_smem(vdim, dim) <= 200 * 1024 ? 1 : 0;
}

#define SSM_PARAMS                                                                                        \
    const float *proj, long ld, int z_col, int x_col, int dt_col, const float *conv_w,                    \
        const float *conv_b, const float *dt_bias, const float *neg_a, const float *d, float *conv_state, \
        float *state, const int *seq, const int *q_start, const int *state_slot, const int *positions,    \
        int n_tokens, int n_requests, int heads, int vdim, int dim, int groups, int taps, int n_slots,    \
        float *raw, long raw_ld, const float *norm_w, int parts, float eps, float out_scale, void *out,   \
        long out_ld, int *status
#define SSM_ARGS                                                                                          \
    SsmArgs{proj,  ld,      z_col,     x_col,     dt_col,     conv_w, conv_b, dt_bias, neg_a,   d,        \
            conv_state, state, seq,    q_start, state_slot, positions, n_tokens, n_requests, heads, vdim, \
            dim,   groups,  taps,      n_slots,   raw,        raw_ld, norm_w, parts,   eps,     out_scale, \
            out,   out_ld,  status}

// Convolution, step sizes and decays: xbc [T, channels] in the given type, dt and decay [T, heads]
// (as_log: log a, else a - 1).
PRB_API int prb_ssm_prepare(SSM_PARAMS, void* xbc, long xbc_ld, int xbc_dtype, float* dt, float* decay,
                            int as_log, cudaStream_t stream) {
    const SsmArgs a = SSM_ARGS;
    if (n_tokens <= 0) return 0;
    if (!sizes_ok(a)) return PRB_E_SIZE;
    const int channels = heads * vdim + 2 * groups * dim;
    const dim3 grid((n_tokens + SP_TOKENS - 1) / SP_TOKENS, (channels + 255) / 256 + 1);
#define PREP(XT, TP) ssm_prepare_kernel<XT, TP><<<grid, 256, 0, stream>>>(a, (XT*)xbc, xbc_ld, dt, decay, as_log)
    if (xbc_dtype == PRB_F32) { if (taps <= 4) PREP(float, 4); else PREP(float, SSM_TAPS); }
    else if (xbc_dtype == PRB_BF16) { if (taps <= 4) PREP(bf16, 4); else PREP(bf16, SSM_TAPS); }
    else return PRB_E_DTYPE;
#undef PREP
    PRB_LAUNCH_CHECK();
    return 0;
}

// The recurrence of a step in segments on tensor cores: three launches, y silu(z) in raw.
PRB_API int prb_ssm_chunks(SSM_PARAMS, const void* xbc, long xbc_ld, const float* dt, const float* la,
                           float* own, void* start_hi, void* start_lo, float* seg_decay, int segments,
                           cudaStream_t stream) {
    const SsmArgs a = SSM_ARGS;
    if (n_tokens <= 0 || n_requests <= 0) return 0;
    if (!sizes_ok(a) || !prb_ssm_chunk_supports(vdim, dim)) return PRB_E_SIZE;
    const int need = n_tokens / DS_SEG + n_requests;
    if (segments < need || need > 65535) return PRB_E_SIZE;
    if (xbc_ld % 8 || ((uintptr_t)xbc) % 16 || ld % 2 || z_col % 2 || ((uintptr_t)proj) % 8 || raw_ld % 2 ||
        ((uintptr_t)raw) % 8 || ((uintptr_t)own | (uintptr_t)start_hi | (uintptr_t)start_lo | (uintptr_t)state) % 16)
        return PRB_E_ALIGN;
    const ChunkArgs c{a, (const bf16*)xbc, xbc_ld, dt, la, own, (bf16*)start_hi, (bf16*)start_lo, seg_decay};
    const size_t s1 = own_smem(vdim, dim), s2 = out_smem(vdim, dim);
    const dim3 grid(heads, need);
    if (s1 > 40 * 1024)
        cudaFuncSetAttribute(ssm_own_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    ssm_own_kernel<<<grid, 128, s1, stream>>>(c);
    PRB_LAUNCH_CHECK();
    ssm_carry_kernel<<<dim3(heads, n_requests, (vdim * dim / 4 + 127) / 128), 128, 0, stream>>>(c);
    PRB_LAUNCH_CHECK();
#define OUTRUN(VT)                                                                                        \
    do {                                                                                                  \
        if (s2 > 40 * 1024)                                                                               \
            cudaFuncSetAttribute(ssm_out_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2); \
        ssm_out_kernel<VT><<<grid, 256, s2, stream>>>(c);                                                 \
    } while (0)
    if (vdim <= 32) OUTRUN(2);
    else if (vdim <= 64) OUTRUN(4);
    else OUTRUN(8);
#undef OUTRUN
    PRB_LAUNCH_CHECK();
    return 0;
}

// Norm in parts of raw (gate_here: times silu(z) first) into out; saved inputs brought up to date.
PRB_API int prb_ssm_finish(SSM_PARAMS, int gate_here, int out_dtype, cudaStream_t stream) {
    const SsmArgs a = SSM_ARGS;
    if (n_tokens <= 0) return 0;
    if (!sizes_ok(a)) return PRB_E_SIZE;
    const bool wide = heads * vdim / parts > FIN_PIECES * 128;
    const long units = (long)n_tokens * parts;
    const int norm_blocks = (int)(wide ? units : (units + FIN_WARPS - 1) / FIN_WARPS);
    const int channels = heads * vdim + 2 * groups * dim;
    const int save_blocks = taps > 1 ? n_requests * taps * ((channels + SAVE_CHANNELS - 1) / SAVE_CHANNELS) : 0;
    const unsigned blocks = (unsigned)(norm_blocks + save_blocks);
#define FINISH(OT)                                                                                              \
    do {                                                                                                        \
        if (wide) ssm_finish_kernel<OT, true><<<blocks, FIN_WIDE, 0, stream>>>(a, gate_here, norm_blocks);       \
        else ssm_finish_kernel<OT, false><<<blocks, FIN_WARPS * 32, 0, stream>>>(a, gate_here, norm_blocks);     \
    } while (0)
    if (out_dtype == PRB_F32) FINISH(float);
    else if (out_dtype == PRB_BF16) FINISH(bf16);
    else return PRB_E_DTYPE;
#undef FINISH
    PRB_LAUNCH_CHECK();
    return 0;
}

static int step_cols(int vdim, int dim, int ctas) {
    const int lanes = lanes_of(dim);
    int cols = (vdim + SS_CC - 1) / SS_CC * SS_CC;
    while (cols > SS_CC && (cols / SS_CC * lanes > 512 ||
                            (long)ctas * ((vdim + cols - 1) / cols) < prb_sm_count() / 2))
        cols = (cols / SS_CC + 1) / 2 * SS_CC;
    return cols;
}

PRB_API int prb_ssm_step_supports(int vdim, int dim) { return vdim > 0 && lanes_of(dim) > 0 ? 1 : 0; }

// Every request brings one token.  arrived: [n_requests] zeros, left zero.
PRB_API int prb_ssm_step(SSM_PARAMS, int* arrived, int out_dtype, cudaStream_t stream) {
    const SsmArgs a = SSM_ARGS;
    if (n_tokens <= 0 || n_requests <= 0) return 0;
    if (!sizes_ok(a) || !prb_ssm_step_supports(vdim, dim)) return PRB_E_SIZE;
    const int lanes = lanes_of(dim), kpl = keys_per_lane(dim);
    const int cols = step_cols(vdim, dim, heads * n_requests);
    StepArgs g{a, (vdim + cols - 1) / cols, cols, lanes, arrived};
    const int threads = max((cols / SS_CC * lanes + 31) / 32 * 32, 256);
    const size_t smem = (size_t)(2 * lanes * kpl + cols + 2 * (cols + 2 * dim)) * sizeof(float);
    const dim3 grid(heads * g.splits, n_requests);
    cudaError_t e;
#define SSTEP1(KP, TP, OT) prb_launch_dependent(ssm_step_kernel<KP, TP, OT>, grid, dim3(threads), smem, stream, g)
#define SSTEP2(KP, OT) (taps <= 4 ? SSTEP1(KP, 4, OT) : SSTEP1(KP, SSM_TAPS, OT))
#define SSTEP(OT) e = kpl == 4 ? SSTEP2(4, OT) : kpl == 8 ? SSTEP2(8, OT) : SSTEP2(16, OT)
    if (out_dtype == PRB_F32) { SSTEP(float); }
    else if (out_dtype == PRB_BF16) { SSTEP(bf16); }
    else return PRB_E_DTYPE;
#undef SSTEP
#undef SSTEP2
#undef SSTEP1
    return e == cudaSuccess ? 0 : (int)e;
}
