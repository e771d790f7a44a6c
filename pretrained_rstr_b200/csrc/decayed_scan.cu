// A linear recurrence over a matrix state with decays (decayed_scan.cuh has the equations and
// the core), for whole steps of any mix of portions and single tokens, and the kernels of gated
// linear attention around it:
//
// dscan_seg / dscan_carry: portions in segments of DS_SEG tokens that run side by side.  Pass 1
//   builds every segment's own sums from zero and the product of its decays minus one; the carry
//   walks a request's segments in order from the carried state (zero at position 0); pass 2 runs
//   every segment from its start with outputs, and a request's last segment leaves the state in
//   its slot.  Operands come as (pointer, pitch, first column): heads may share a query or key
//   row (`share` heads each), a decay is per key channel or per head, keys may have a scale per
//   token and head, and a direct path adds direct_h * v to a head's result.  Operands of the next
//   16 tokens arrive by cp.async while a block is worked on.
// gla_decay: a = sigmoid(z)^(1 / tau) with z = W2 lr + b (lr: a low-rank projection), as a - 1.
// gla_step: a step of single tokens in one launch: decays, recurrence and finish, a CTA per (head,
//   request).  State and W2 are requested before the kernel waits for the projection.
// gla_finish (or inside pass 2 / the step): o / sqrt(mean(o^2) + eps) * weight * silu(gate) * out_scale,
//   the weight of `vdim` numbers shared by the heads.
// Everything here is 32-bit arithmetic.
#include "decayed_scan.cuh"

namespace {
using namespace dscan;
constexpr int DS_TB = 16;            // tokens staged at a time
constexpr int ds_threads(int kpl) { return kpl == 4 ? 512 : 256; }
constexpr int DS_CC = 8;             // value columns a thread of the segmented passes holds
constexpr int GS_CC = 4;             // and one of the single-token kernel

struct Finish {
    void* out;                       // null: raw sums
    long out_ld;
    const float* gate;               // [T, gate_ld], first column of head 0
    long gate_ld;
    const float* norm_w;             // [vdim]
    float eps, out_scale;
};

struct SegArgs {
    const float* q; long q_ld; int q_share;
    const float* k; long k_ld; int k_share;
    const float* v; long v_ld;
    const float* c; long c_ld;       // decay - 1: [T, heads * dim] or [T, heads]
    const float* ks;                 // [T, heads] or null
    const float* direct;             // [heads] or null
    float q_scale;
    float* raw; long raw_ld;
    float* state;
    const int* q_start; const int* state_slot; const int* positions;
    int n_tokens, n_requests, heads, dim, vdim, lanes, cols, n_slots;
    float* seg_own; float* seg_start; float* seg_decay;
    int* status;
    Finish fin;
};

// A token's row of a finish: a warp; src the head's sums, gp its gates (shared or global memory).
template <typename O>
__device__ __forceinline__ void finish_row(const Finish& f, const float* src, const float* gp, int t, int hd,
                                           int vdim, int lane) {
    float ss = 0.0f;
    for (int j = lane; j < vdim; j += 32) ss = fmaf(src[j], src[j], ss);
    ss = prb_warp_sum(ss);
    const float inv = f.out_scale / sqrtf(ss / (float)vdim + f.eps);
    O* o = (O*)f.out + (size_t)t * f.out_ld + (size_t)hd * vdim;
    for (int j = lane; j < vdim; j += 32)
        o[j] = prb_from_float<O>(src[j] * inv * f.norm_w[j] * silu<O>(gp[j]));
}

// MODE 1: a segment's own sums from zero; 2: a segment from its start with outputs.  Scales of the
// keys and the direct path go with decays per head.
template <int KPL, bool PER_KEY, int MODE, typename O>
__global__ void __launch_bounds__(ds_threads(KPL)) dscan_seg_kernel(SegArgs a) {
    extern __shared__ __align__(16) float sm[];
    prb_grid_launch_dependents();
    const int hd = blockIdx.x, cg = blockIdx.z;
    int b, s, nseg;
    if (!find_segment(a.q_start, a.n_requests, blockIdx.y, b, s, nseg)) return;
    int t0 = a.q_start[b], t1 = a.q_start[b + 1];
    if (t0 < 0 || t1 > a.n_tokens) return;
    const bool last = s == nseg - 1;
    if (MODE == 1 && last) return;                   // (a last segment's own sum is never needed)
    const int slot = a.state_slot[b];
    if (slot < 0 || slot >= a.n_slots) {
        if (MODE == 2 && threadIdx.x == 0) prb_set_status(a.status, PRB_S_ROW_RANGE, t0, slot, a.n_slots);
        return;
    }
    t0 += s * DS_SEG;
    t1 = min(t1, t0 + DS_SEG);
    const int L = a.lanes, dp = L * KPL, dim = a.dim, vdim = a.vdim, cols = a.cols;
    const int cw = PER_KEY ? dp : 4;
    const int stage = DS_TB * (2 * dp + cw + cols + 4);
    float* o_s = sm + 2 * stage;                     // [DS_TB][vdim], with the finish inside,
    float* g_s = o_s + DS_TB * vdim;                 // and twice [DS_TB][vdim] gates
    const int ln = threadIdx.x % L, cl = min((int)threadIdx.x / L * DS_CC, cols - DS_CC);
    const int c0 = cg * cols + cl;                   // this thread's first value column
    const bool mine = (int)threadIdx.x / L * DS_CC < cols;       // (threads beyond work along, and store nothing)
    const size_t per_head = (size_t)vdim * dim, per_state = (size_t)a.heads * per_head;
    float S[DS_CC][KPL], Pd[KPL];
    load_state<DS_CC, KPL>(S, MODE == 2 ? a.seg_start + (size_t)blockIdx.y * per_state + hd * per_head : nullptr,
                           ln, c0, dim, vdim);
#pragma unroll
    for (int i = 0; i < KPL; ++i) Pd[i] = 0.0f;
    const float* qb = a.q + (size_t)(hd / a.q_share) * dim;
    const float* kb = a.k + (size_t)(hd / a.k_share) * dim;
    const float* vb = a.v + (size_t)hd * vdim + cg * cols;
    const float* cb = PER_KEY ? a.c + (size_t)hd * dim : a.c + hd;
    const int vcols = min(cols, vdim - cg * cols);   // columns of this CTA that exist
    const bool vec = dim % 4 == 0 && vdim % 4 == 0 &&
                     (a.q_ld | a.k_ld | a.v_ld) % 4 == 0 && (!PER_KEY || a.c_ld % 4 == 0) &&
                     ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (PER_KEY ? (uintptr_t)a.c : 0)) % 16 == 0;
    const bool inside = MODE == 2 && a.fin.out != nullptr;
    const float* gb = inside ? a.fin.gate + (size_t)hd * vdim : nullptr;
    const bool gvec = inside && vdim % 4 == 0 && a.fin.gate_ld % 4 == 0 && ((uintptr_t)a.fin.gate) % 16 == 0;
    const float dd = !PER_KEY && a.direct ? a.direct[hd] : 0.0f;
    if (dp > dim) {                                  // keys beyond the head: zero in both stages
        for (int e = threadIdx.x; e < 2 * DS_TB * (dp - dim); e += blockDim.x) {
            const int row = e / (dp - dim), i = dim + e % (dp - dim);
            float* base = sm + (row / DS_TB) * stage + (row % DS_TB) * dp + i;
            base[0] = 0.0f;
            base[DS_TB * dp] = 0.0f;
            if (PER_KEY) base[2 * DS_TB * dp] = 0.0f;
        }
    }
    if (cols > vcols) {                              // and values beyond it
        for (int e = threadIdx.x; e < 2 * DS_TB * (cols - vcols); e += blockDim.x) {
            const int row = e / (cols - vcols), i = vcols + e % (cols - vcols);
            sm[(row / DS_TB) * stage + DS_TB * (2 * dp + cw) + (row % DS_TB) * cols + i] = 0.0f;
        }
    }
    auto fetch = [&](int tb, int into) {
        float* q_s = sm + into * stage;
        float* k_s = q_s + DS_TB * dp;
        float* c_s = k_s + DS_TB * dp;
        float* v_s = c_s + DS_TB * cw;
        float* d_s = v_s + DS_TB * cols;
        const int nb = min(DS_TB, t1 - tb);
        if (vec) {
            const int d4 = dim / 4, v4 = vcols / 4;
            for (int e = threadIdx.x; e < nb * d4; e += blockDim.x) {
                const int tok = e / d4, i = (e - tok * d4) * 4;
                const size_t t = tb + tok;
                if (MODE == 2) copy16(q_s + tok * dp + i, qb + t * a.q_ld + i);
                copy16(k_s + tok * dp + i, kb + t * a.k_ld + i);
                if (PER_KEY) copy16(c_s + tok * dp + i, cb + t * a.c_ld + i);
            }
            for (int e = threadIdx.x; e < nb * v4; e += blockDim.x) {
                const int tok = e / v4, i = (e - tok * v4) * 4;
                copy16(v_s + tok * cols + i, vb + (size_t)(tb + tok) * a.v_ld + i);
            }
        } else {
            for (int e = threadIdx.x; e < nb * dim; e += blockDim.x) {
                const int tok = e / dim, i = e - tok * dim;
                const size_t t = tb + tok;
                if (MODE == 2) q_s[tok * dp + i] = qb[t * a.q_ld + i];
                k_s[tok * dp + i] = kb[t * a.k_ld + i];
                if (PER_KEY) c_s[tok * dp + i] = cb[t * a.c_ld + i];
            }
            for (int e = threadIdx.x; e < nb * vcols; e += blockDim.x) {
                const int tok = e / vcols, i = e - tok * vcols;
                v_s[tok * cols + i] = vb[(size_t)(tb + tok) * a.v_ld + i];
            }
        }
        if (inside) {
            float* to = g_s + into * DS_TB * vdim;
            if (gvec) {
                for (int e = threadIdx.x; e < nb * (vdim / 4); e += blockDim.x) {
                    const int tok = e / (vdim / 4), i = (e - tok * (vdim / 4)) * 4;
                    copy16(to + tok * vdim + i, gb + (size_t)(tb + tok) * a.fin.gate_ld + i);
                }
            } else {
                for (int e = threadIdx.x; e < nb * vdim; e += blockDim.x) {
                    const int tok = e / vdim, i = e - tok * vdim;
                    to[e] = gb[(size_t)(tb + tok) * a.fin.gate_ld + i];
                }
            }
        }
        if (!PER_KEY) {
            for (int tok = threadIdx.x; tok < nb; tok += blockDim.x) {
                d_s[tok * 4] = a.ks ? a.ks[(size_t)(tb + tok) * a.heads + hd] : 1.0f;
                c_s[tok * 4] = cb[(size_t)(tb + tok) * a.c_ld];
            }
        }
        copy_commit();
    };
    const bool holder = mine && (ln & (L / DS_CC - 1)) == 0;
    const int held = held_column<DS_CC>(ln, L);
    const bool writes = holder && c0 + held < vdim;
    // where a token's sum of this lane goes: the finish's rows, or raw sums
    float* o_to = a.fin.out ? o_s + c0 + held : a.raw + (size_t)hd * vdim + c0 + held;
    const size_t o_ld = a.fin.out ? vdim : a.raw_ld;
    fetch(t0, 0);
    int turn = 0;
    for (int tb = t0; tb < t1; tb += DS_TB, turn ^= 1) {
        if (tb + DS_TB < t1) fetch(tb + DS_TB, turn ^ 1);
        else copy_commit();
        copy_wait<1>();
        __syncthreads();
        const float* q_s = sm + turn * stage;
        const float* k_s = q_s + DS_TB * dp;
        const float* c_s = k_s + DS_TB * dp;
        const float* v_s = c_s + DS_TB * cw + cl;
        const float* d_s = v_s - cl + DS_TB * cols;
        const int nb = min(DS_TB, t1 - tb);
        float* o_at = o_to + (a.fin.out ? 0 : (size_t)tb * o_ld);
#pragma unroll 4
        for (int tok = 0; tok < nb; ++tok) {
            float v[DS_CC], part[DS_CC];
#pragma unroll
            for (int j = 0; j < DS_CC; j += 4) {
                const float4 x = *reinterpret_cast<const float4*>(v_s + tok * cols + j);
                v[j] = x.x; v[j + 1] = x.y; v[j + 2] = x.z; v[j + 3] = x.w;
            }
            if (!PER_KEY) {
                const float ks = d_s[tok * 4];
#pragma unroll
                for (int j = 0; j < DS_CC; ++j) v[j] *= ks;
            }
            const float* c_at = PER_KEY ? c_s + tok * dp + ln * KPL : c_s + tok * 4;
            advance<DS_CC, KPL, PER_KEY, MODE == 2>(S, k_s + tok * dp + ln * KPL, c_at, q_s + tok * dp + ln * KPL,
                                                    v, part);
            if (MODE == 1) {                         // 1 + p <- (1 + p)(1 + c)
                if (PER_KEY) {
                    if (cl == 0) {
#pragma unroll
                        for (int i = 0; i < KPL; ++i) Pd[i] = fmaf(Pd[i], c_at[i], Pd[i] + c_at[i]);
                    }
                } else {
                    Pd[0] = fmaf(Pd[0], c_at[0], Pd[0] + c_at[0]);
                }
            }
            if (MODE == 2) {
                float sum = close_columns<DS_CC>(part, ln, L) * a.q_scale;
                if (!PER_KEY) sum = fmaf(dd, v_s[tok * cols + held], sum);
                if (writes) o_at[tok * o_ld] = sum;
            }
        }
        __syncthreads();
        if (inside) {
            for (int tok = threadIdx.x >> 5; tok < nb; tok += blockDim.x >> 5)
                finish_row<O>(a.fin, o_s + tok * vdim, g_s + (turn * DS_TB + tok) * vdim, tb + tok, hd, vdim,
                              threadIdx.x & 31);
        }
    }
    if (mine) {
        if (MODE == 1)
            store_state<DS_CC, KPL>(S, a.seg_own + (size_t)blockIdx.y * per_state + hd * per_head, ln, c0, dim, vdim);
        if (MODE == 2 && last)
            store_state<DS_CC, KPL>(S, a.state + (size_t)slot * per_state + hd * per_head, ln, c0, dim, vdim);
    }
    if (MODE == 1 && mine && cl == 0 && cg == 0) {
        if (PER_KEY) {
#pragma unroll
            for (int i = 0; i < KPL; ++i)
                if (ln * KPL + i < dim)
                    a.seg_decay[((size_t)blockIdx.y * a.heads + hd) * dim + ln * KPL + i] = Pd[i];
        } else if (ln == 0) {
            a.seg_decay[(size_t)blockIdx.y * a.heads + hd] = Pd[0];
        }
    }
}

// A thread per state number of a (head, request); the request's segments in order.
template <bool PER_KEY>
__global__ void dscan_carry_kernel(SegArgs a) {
    prb_grid_launch_dependents();
    const int hd = blockIdx.x, b = blockIdx.y;
    const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
    if (t1 <= t0 || t0 < 0 || t1 > a.n_tokens) return;
    const int slot = a.state_slot[b];
    if (slot < 0 || slot >= a.n_slots) return;
    int base = 0;
    for (int bb = 0; bb < b; ++bb) {
        const int n = a.q_start[bb + 1] - a.q_start[bb];
        base += n > 0 ? (n + DS_SEG - 1) / DS_SEG : 0;
    }
    const int nseg = (t1 - t0 + DS_SEG - 1) / DS_SEG;
    const size_t per_head = (size_t)a.vdim * a.dim, per_state = (size_t)a.heads * per_head;
    const size_t e = (size_t)blockIdx.z * blockDim.x + threadIdx.x;
    if (e >= per_head) return;
    const size_t at = (size_t)hd * per_head + e;
    const int kk = (int)(e % a.dim);
    const float* own = a.seg_own + (size_t)base * per_state + at;
    float* start = a.seg_start + (size_t)base * per_state + at;
    const float* dec = PER_KEY ? a.seg_decay + ((size_t)base * a.heads + hd) * a.dim + kk
                               : a.seg_decay + (size_t)base * a.heads + hd;
    const size_t dec_step = PER_KEY ? (size_t)a.heads * a.dim : a.heads;
    float S = a.positions[t0] > 0 ? a.state[(size_t)slot * per_state + at] : 0.0f;
    int s = 0;
    for (; s + 4 < nseg; s += 4) {                   // four segments' numbers requested at a time
        float o[4], p[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[i] = own[(size_t)(s + i) * per_state];
            p[i] = dec[(size_t)(s + i) * dec_step];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            start[(size_t)(s + i) * per_state] = S;
            S += fmaf(p[i], S, o[i]);
        }
    }
    for (; s < nseg; ++s) {
        start[(size_t)s * per_state] = S;
        if (s + 1 < nseg) S += fmaf(dec[(size_t)s * dec_step], S, own[(size_t)s * per_state]);
    }
}

template <typename O>
__global__ void gla_finish_kernel(Finish f, const float* __restrict__ raw, long raw_ld,
                                  const int* __restrict__ seq_of_token, int n_tokens, int heads, int vdim) {
    prb_grid_launch_dependents();
    const int lane = threadIdx.x & 31;
    const long unit = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= (long)n_tokens * heads) return;
    const int t = (int)(unit / heads), hd = (int)(unit - (long)t * heads);
    if (seq_of_token[t] < 0) return;
    finish_row<O>(f, raw + (size_t)t * raw_ld + (size_t)hd * vdim, f.gate + (size_t)t * f.gate_ld + (size_t)hd * vdim,
                  t, hd, vdim, lane);
}

__device__ __forceinline__ float decay_minus_one(float z, float inv_tau) {
    return expm1f(-softplus(-z) * inv_tau);
}

// A CTA per GD_TOKENS tokens: a thread per channel walks its row of W2 once for all of them.
constexpr int GD_TOKENS = 8;
__global__ void gla_decay_kernel(float* __restrict__ c_out, long c_ld, const float* __restrict__ lr, long lr_ld,
                                 const float* __restrict__ w2t, const float* __restrict__ bias, int n_tokens,
                                 int channels, int rank, float inv_tau) {
    extern __shared__ float th[];                    // [GD_TOKENS][rank]
    prb_grid_launch_dependents();
    const int t0 = blockIdx.x * GD_TOKENS;
    const int nt = min(GD_TOKENS, n_tokens - t0);
    for (int e = threadIdx.x; e < GD_TOKENS * rank; e += blockDim.x) {
        const int tt = e / rank, j = e - tt * rank;
        th[e] = tt < nt ? lr[(size_t)(t0 + tt) * lr_ld + j] : 0.0f;
    }
    __syncthreads();
    for (int ch = blockIdx.y * blockDim.x + threadIdx.x; ch < channels; ch += gridDim.y * blockDim.x) {
        float z[GD_TOKENS];
#pragma unroll
        for (int tt = 0; tt < GD_TOKENS; ++tt) z[tt] = 0.0f;
        for (int j = 0; j < rank; ++j) {
            const float wj = w2t[(size_t)j * channels + ch];
#pragma unroll
            for (int tt = 0; tt < GD_TOKENS; ++tt) z[tt] = fmaf(wj, th[tt * rank + j], z[tt]);
        }
        const float bb = bias[ch];
#pragma unroll
        for (int tt = 0; tt < GD_TOKENS; ++tt)
            if (tt < nt) c_out[(size_t)(t0 + tt) * c_ld + ch] = decay_minus_one(z[tt] + bb, inv_tau);
    }
}

struct GlaStepArgs {
    const float* proj; long ld;
    int q_col, k_col, v_col, lr_col;
    const float* w2t;                // [rank, heads * dim]
    const float* bias;               // [heads * dim]
    float inv_tau, q_scale;
    float* state;
    const int* q_start; const int* state_slot; const int* positions;
    int n_tokens, n_requests, heads, dim, vdim, rank, lanes, n_slots;
    int* status;
    Finish fin;
};

constexpr int GS_RANK = 16;          // rows of W2 a thread asks for before the projection is there

template <int KPL, typename O>
__global__ void __launch_bounds__(KPL == 4 ? 1024 : 512) gla_step_kernel(GlaStepArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int L = a.lanes, dp = L * KPL, dim = a.dim, vdim = a.vdim;
    float* q_s = sm;                                 // [dp]
    float* k_s = q_s + dp;
    float* c_s = k_s + dp;
    float* v_s = c_s + dp;                           // [vdim rounded to GS_CC]
    float* o_s = v_s + (vdim + GS_CC - 1) / GS_CC * GS_CC;
    float* g_s = o_s + (vdim + GS_CC - 1) / GS_CC * GS_CC;
    prb_grid_launch_dependents();
    const int hd = blockIdx.x, b = blockIdx.y;
    // (the step's description and the state of the step before lie behind launches that have
    // ended: they are read before the wait)
    const int t = a.q_start[b], t1 = a.q_start[b + 1];
    const int slot = a.state_slot[b];
    const bool run = t1 > t && t >= 0 && t1 <= a.n_tokens && slot >= 0 && slot < a.n_slots;
    const int ln = threadIdx.x % L, cl = threadIdx.x / L;
    const int c0 = cl * GS_CC;
    float* sp = a.state + ((size_t)(run ? slot : 0) * a.heads + hd) * vdim * dim;
    const bool carried = run && a.positions[t] > 0;
    float S[GS_CC][KPL];
    load_state<GS_CC, KPL>(S, carried && c0 < vdim ? sp : nullptr, ln, c0, dim, vdim);
    float w2[GS_RANK];
    const int ch = hd * dim + (int)threadIdx.x, channels = a.heads * dim;
    const bool decays = (int)threadIdx.x < dim;
#pragma unroll
    for (int j = 0; j < GS_RANK; ++j)
        w2[j] = decays && j < a.rank ? a.w2t[(size_t)j * channels + ch] : 0.0f;
    const float bias = decays ? a.bias[ch] : 0.0f;
    prb_grid_wait();
    if (!run) {
        if (t1 > t && threadIdx.x == 0) prb_set_status(a.status, PRB_S_ROW_RANGE, t, slot, a.n_slots);
        return;
    }
    const float* row = a.proj + (size_t)t * a.ld;
    for (int i = threadIdx.x; i < dp; i += blockDim.x) {
        q_s[i] = i < dim ? row[a.q_col + hd * dim + i] : 0.0f;
        k_s[i] = i < dim ? row[a.k_col + hd * dim + i] : 0.0f;
        if (i >= dim) c_s[i] = 0.0f;
    }
    for (int i = threadIdx.x; i < (vdim + GS_CC - 1) / GS_CC * GS_CC; i += blockDim.x)
        v_s[i] = i < vdim ? row[a.v_col + hd * vdim + i] : 0.0f;
    for (int i = threadIdx.x; i < vdim; i += blockDim.x)
        g_s[i] = a.fin.gate[(size_t)t * a.fin.gate_ld + (size_t)hd * vdim + i];
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float z = 0.0f;
        if (i == (int)threadIdx.x) {
#pragma unroll
            for (int j = 0; j < GS_RANK; ++j)
                if (j < a.rank) z = fmaf(w2[j], row[a.lr_col + j], z);
            for (int j = GS_RANK; j < a.rank; ++j) z = fmaf(a.w2t[(size_t)j * channels + ch], row[a.lr_col + j], z);
            z += bias;
        } else {                                     // (fewer threads than keys)
            for (int j = 0; j < a.rank; ++j)
                z = fmaf(a.w2t[(size_t)j * channels + hd * dim + i], row[a.lr_col + j], z);
            z += a.bias[hd * dim + i];
        }
        c_s[i] = decay_minus_one(z, a.inv_tau);
    }
    __syncthreads();
    float v[GS_CC], part[GS_CC];
#pragma unroll
    for (int j = 0; j < GS_CC; ++j) v[j] = c0 < vdim ? v_s[c0 + j] : 0.0f;
    advance<GS_CC, KPL, true, true>(S, k_s + ln * KPL, c_s + ln * KPL, q_s + ln * KPL, v, part);
    const float sum = close_columns<GS_CC>(part, ln, L);
    if ((ln & ((L >> 2) - 1)) == 0) {
        const int j = held_column<GS_CC>(ln, L);
        if (c0 + j < vdim) o_s[c0 + j] = sum * a.q_scale;
    }
    if (c0 < vdim) store_state<GS_CC, KPL>(S, sp, ln, c0, dim, vdim);
    __syncthreads();
    if (threadIdx.x < 32) finish_row<O>(a.fin, o_s, g_s, t, hd, vdim, threadIdx.x);
}

// Value columns a CTA of a pass takes (the pass with outputs likes whole heads, for the finish; the
// other several CTAs an SM).
int seg_cols(int dim, int vdim, int mode = 2) {
    const int lanes = lanes_of(dim);
    int cols = min(ds_threads(keys_per_lane(dim)), mode == 1 ? 256 : 1024) / lanes * DS_CC;
    if (cols > vdim) cols = (vdim + DS_CC - 1) / DS_CC * DS_CC;
    return cols;
}
size_t seg_smem(int dim, int vdim, int cols, bool per_key, bool fin) {
    const int dp = lanes_of(dim) * keys_per_lane(dim);
    return (size_t)(2 * DS_TB * (2 * dp + (per_key ? dp : 4) + cols + 4) +
                    (fin ? 3 * DS_TB * vdim : 0)) * sizeof(float);
}
}  // namespace

PRB_API int prb_dscan_segment() { return DS_SEG; }
PRB_API int prb_dscan_max_segments(int t_cap, int b_cap) { return t_cap / DS_SEG + b_cap; }
// 0: not at all; 1: raw sums; 3: also with the finish inside pass 2 (a CTA holds a whole head).
PRB_API int prb_dscan_supports(int dim, int vdim) {
    if (lanes_of(dim) == 0 || vdim <= 0 || vdim > 4096) return 0;
    const int cols = seg_cols(dim, vdim);
    if (seg_smem(dim, vdim, cols, true, false) > 200 * 1024) return 0;
    return cols >= vdim && seg_smem(dim, vdim, cols, true, true) <= 200 * 1024 ? 3 : 1;
}

// Three launches.  Workspaces: seg_own, seg_start [segments, heads, vdim, dim], seg_decay
// [segments, heads, dim] (per_key) or [segments, heads].  out != null: the finish inside.
PRB_API int prb_dscan_segments(float* raw, long raw_ld, const float* q, long q_ld, int q_share,
                               const float* k, long k_ld, int k_share, const float* v, long v_ld,
                               const float* c, long c_ld, int per_key, const float* ks, const float* direct,
                               float q_scale, float* state, const int* q_start, const int* state_slot,
                               const int* positions, int n_tokens, int n_requests, int heads, int dim,
                               int vdim, int n_slots, float* seg_own, float* seg_start, float* seg_decay,
                               int segments, void* out, long out_ld, const float* gate, long gate_ld,
                               const float* norm_w, float eps, float out_scale, int out_dtype, int* status,
                               cudaStream_t stream) {
    if (n_requests <= 0 || n_tokens <= 0) return 0;
    const int ok = prb_dscan_supports(dim, vdim);
    if (!ok || heads <= 0 || q_share <= 0 || k_share <= 0 || n_requests > 65535) return PRB_E_SIZE;
    if (out != nullptr && (ok != 3 || gate == nullptr || norm_w == nullptr)) return PRB_E_ARG;
    if (out == nullptr && raw == nullptr) return PRB_E_ARG;
    if (per_key && (ks != nullptr || direct != nullptr)) return PRB_E_ARG;
    const int need = prb_dscan_max_segments(n_tokens, n_requests);
    if (segments < need || need > 65535) return PRB_E_SIZE;
    if (out_dtype != PRB_F32 && out_dtype != PRB_BF16) return PRB_E_DTYPE;
    const int lanes = lanes_of(dim), kpl = keys_per_lane(dim), cols = seg_cols(dim, vdim);
    SegArgs a{q, q_ld, q_share, k, k_ld, k_share, v, v_ld, c, c_ld, ks, direct, q_scale, raw, raw_ld,
              state, q_start, state_slot, positions, n_tokens, n_requests, heads, dim, vdim, lanes,
              cols, n_slots, seg_own, seg_start, seg_decay, status,
              Finish{out, out_ld, gate, gate_ld, norm_w, eps, out_scale}};
#define SEGRUN(KP, PK, MD, OT)                                                                     \
    do {                                                                                           \
        a.cols = MD == 1 ? seg_cols(dim, vdim, 1) : cols;                                          \
        const int threads = (a.cols / DS_CC * lanes + 31) / 32 * 32;                               \
        const size_t smem = seg_smem(dim, vdim, a.cols, PK, MD == 2 && out != nullptr);            \
        const dim3 grid(heads, need, (vdim + a.cols - 1) / a.cols);                                \
        if (smem > 40 * 1024)                                                                      \
            cudaFuncSetAttribute(dscan_seg_kernel<KP, PK, MD, OT>,                                 \
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
        dscan_seg_kernel<KP, PK, MD, OT><<<grid, threads, smem, stream>>>(a);                      \
    } while (0)
#define SEGK(PK, MD, OT)                                                                           \
    do {                                                                                           \
        if (kpl == 4) SEGRUN(4, PK, MD, OT);                                                       \
        else if (kpl == 8) SEGRUN(8, PK, MD, OT);                                                  \
        else SEGRUN(16, PK, MD, OT);                                                               \
    } while (0)
    const dim3 cgrid(heads, n_requests, (unsigned)(((size_t)vdim * dim + 255) / 256));
    if (per_key) {
        SEGK(true, 1, float);
        PRB_LAUNCH_CHECK();
        dscan_carry_kernel<true><<<cgrid, 256, 0, stream>>>(a);
        PRB_LAUNCH_CHECK();
        if (out_dtype == PRB_F32) SEGK(true, 2, float);
        else SEGK(true, 2, __nv_bfloat16);
    } else {
        SEGK(false, 1, float);
        PRB_LAUNCH_CHECK();
        dscan_carry_kernel<false><<<cgrid, 256, 0, stream>>>(a);
        PRB_LAUNCH_CHECK();
        if (out_dtype == PRB_F32) SEGK(false, 2, float);
        else SEGK(false, 2, __nv_bfloat16);
    }
#undef SEGK
#undef SEGRUN
    PRB_LAUNCH_CHECK();
    return 0;
}

PRB_API int prb_gla_finish(void* out, long out_ld, const float* raw, long raw_ld, const float* gate,
                           long gate_ld, const float* norm_w, const int* seq_of_token, int n_tokens,
                           int heads, int vdim, float eps, float out_scale, int out_dtype,
                           cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (heads <= 0 || vdim <= 0) return PRB_E_SIZE;
    const Finish f{out, out_ld, gate, gate_ld, norm_w, eps, out_scale};
    const unsigned blocks = (unsigned)(((long)n_tokens * heads + 3) / 4);
    if (out_dtype == PRB_F32)
        gla_finish_kernel<float><<<blocks, 128, 0, stream>>>(f, raw, raw_ld, seq_of_token, n_tokens, heads, vdim);
    else if (out_dtype == PRB_BF16)
        gla_finish_kernel<__nv_bfloat16><<<blocks, 128, 0, stream>>>(f, raw, raw_ld, seq_of_token, n_tokens, heads, vdim);
    else
        return PRB_E_DTYPE;
    PRB_LAUNCH_CHECK();
    return 0;
}

// w2t: [rank, channels]; c_out [n_tokens, c_ld].
PRB_API int prb_gla_decay(float* c_out, long c_ld, const float* lr, long lr_ld, const float* w2t,
                          const float* bias, int n_tokens, int channels, int rank, float inv_tau,
                          cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const size_t smem = (size_t)GD_TOKENS * rank * sizeof(float);
    if (channels <= 0 || rank <= 0 || smem > 40 * 1024) return PRB_E_SIZE;
    const dim3 grid((n_tokens + GD_TOKENS - 1) / GD_TOKENS, (channels + 255) / 256);
    gla_decay_kernel<<<grid, 256, smem, stream>>>(c_out, c_ld, lr, lr_ld, w2t, bias, n_tokens, channels,
                                                  rank, inv_tau);
    PRB_LAUNCH_CHECK();
    return 0;
}

PRB_API int prb_gla_step_supports(int dim, int vdim) {
    const int lanes = lanes_of(dim);
    return lanes > 0 && vdim > 0 && (vdim + GS_CC - 1) / GS_CC * lanes <= (keys_per_lane(dim) == 4 ? 1024 : 512) ? 1 : 0;
}

// Every request brings one token.
PRB_API int prb_gla_step(void* out, long out_ld, const float* proj, long ld, int q_col, int k_col, int v_col,
                         int lr_col, int g_col, const float* w2t, const float* bias, float inv_tau,
                         float q_scale, const float* norm_w, float eps, float out_scale, float* state,
                         const int* q_start, const int* state_slot, const int* positions, int n_tokens,
                         int n_requests, int heads, int dim, int vdim, int rank, int n_slots, int out_dtype,
                         int* status, cudaStream_t stream) {
    if (n_tokens <= 0 || n_requests <= 0) return 0;
    if (heads <= 0 || rank <= 0 || n_requests > 65535 || !prb_gla_step_supports(dim, vdim)) return PRB_E_SIZE;
    const int lanes = lanes_of(dim), kpl = keys_per_lane(dim);
    const int vp = (vdim + GS_CC - 1) / GS_CC * GS_CC;
    const int threads = (vp / GS_CC * lanes + 31) / 32 * 32;
    const size_t smem = (size_t)(3 * lanes * kpl + 3 * vp) * sizeof(float);
    GlaStepArgs a{proj, ld, q_col, k_col, v_col, lr_col, w2t, bias, inv_tau, q_scale, state, q_start,
                  state_slot, positions, n_tokens, n_requests, heads, dim, vdim, rank, lanes, n_slots,
                  status, Finish{out, out_ld, proj + g_col, ld, norm_w, eps, out_scale}};
    const dim3 grid(heads, n_requests);
    cudaError_t e;
#define GSTEP(OT)                                                                                      \
    e = kpl == 4   ? prb_launch_dependent(gla_step_kernel<4, OT>, grid, dim3(threads), smem, stream, a)  \
        : kpl == 8 ? prb_launch_dependent(gla_step_kernel<8, OT>, grid, dim3(threads), smem, stream, a)  \
                   : prb_launch_dependent(gla_step_kernel<16, OT>, grid, dim3(threads), smem, stream, a)
    if (out_dtype == PRB_F32) { GSTEP(float); }
    else if (out_dtype == PRB_BF16) { GSTEP(__nv_bfloat16); }
    else return PRB_E_DTYPE;
#undef GSTEP
    return e == cudaSuccess ? 0 : (int)e;
}
