// What windowed attention does to a step's queries and keys before it attends, head by head
// (window_attention.cu holds the attention itself and the form with a norm over whole
// projections):
//
//   u    = projection (+ bias)
//   u    = sum_j w[c, j] u_(t - taps + 1 + j)       a causal convolution per channel of q and k,
//                                                  zeros before the sequence's start (optional)
//   v    = the value projection (+ bias), or the key as it is now
//   u    = u / sqrt(mean(u^2) + eps) * w            a norm per head before the rotation, or after
//                                                  it without a weight (optional)
//   u    = the first rot_dims coordinates turned by the position: pairs (i, i + rot_dims / 2), or
//          (2i, 2i + 1) in the interleaved layout
//
// A warp per (token, head): heads are independent, so a single token's heads spread over many
// SMs.  The convolution's inputs from before the step are per-request state, [slots, taps - 1,
// (heads + kv_heads) * dim] in 32-bit (the query's channels first); in a step whose requests bring
// one token each the same warp brings them up to date (its lanes own the same channels in
// every pass, and read before they write); in a step with portions they are read by a portion's
// first tokens while they would be written from its last, so wattn_conv_state does it afterwards.
//
// rotary_angles: cosine and sine of every token's angles, times one magnitude, once per step, for
//   all layers and heads.
// All arithmetic is 32-bit, the angles' products 64-bit.
#include "common.cuh"

namespace {
struct PrepArgs {
    float* q_out;               // [T, heads * dim]
    void* cache;                // [pages, kv_heads, page_size, dim + vdim]
    const float* proj;          // [T, ld]
    long ld;
    int q_col, k_col, v_col;    // v_col < 0: the (convolved) keys are the values
    const float* q_norm;        // [dim], norm_mode 2
    const float* k_norm;
    const float* q_bias;
    const float* k_bias;
    const float* v_bias;
    const float* conv_q;        // [heads * dim, taps], or null
    const float* conv_k;        // [kv_heads * dim, taps]
    int taps;
    float* conv_state;          // [slots, taps - 1, (heads + kv_heads) * dim]
    int n_slots, write_state;   // write_state: every request brings one token
    const int* seq;             // [T]   (these three with a convolution only)
    const int* q_start;         // [requests + 1]
    const int* state_slot;      // [requests]
    const int* slots;           // [T], or null: nothing is cached
    const int* positions;
    const float* freq;
    const float* freq_lo;
    const float2* angles;       // [T, rot_dims / 2] cosine and sine, or null: computed here
    int n_tokens, heads, kv_heads, dim, vdim, rot_dims, interleaved, norm_mode;
    float eps, temp_coef;
    int temp_every, page_size, num_pages;
    int* status;
};

// One head's channels of one token, as the projection (and the convolution) leaves them.
struct HeadInput {
    const float* row;           // this token's projected numbers of the head
    const float* bias;
    const float* w;             // taps of the head's first channel, or null
    const float* state;         // saved inputs of the head's first channel (stride channels), or null
    long ld;
    int taps, channels, back, pos;      // back: tokens of this portion before this one
    __device__ __forceinline__ float raw(int i) const { return row[i] + (bias ? bias[i] : 0.0f); }
    // the projected value `m` tokens ago
    __device__ __forceinline__ float past(int i, int m) const {
        if (m > pos) return 0.0f;
        if (m <= back) return row[i - (long)m * ld] + (bias ? bias[i] : 0.0f);
        return state ? state[(long)(taps - 1 - (m - back)) * channels + i] : 0.0f;
    }
    __device__ __forceinline__ float get(int i) const {
        if (w == nullptr) return raw(i);
        float s = 0.0f;
        if (back >= taps - 1 && bias == nullptr) {       // everything lies in this portion
            for (int j = 0; j < taps; ++j) s = fmaf(w[i * taps + j], row[i - (long)(taps - 1 - j) * ld], s);
            return s;
        }
        for (int j = 0; j < taps; ++j) s = fmaf(w[i * taps + j], past(i, taps - 1 - j), s);
        return s;
    }
};

__device__ __forceinline__ void store_pair(float* p, float x, float y) {
    *reinterpret_cast<float2*>(p) = make_float2(x, y);
}
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float x, float y) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y);
}

// U: pairs (or coordinates that stay) a lane owns at most; their numbers are computed once and stay
// in registers.  0: any size, computed again in every pass.
template <typename C, int U>
__global__ void __launch_bounds__(256) wattn_prepare_heads_kernel(PrepArgs a) {
    prb_grid_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int per_token = a.heads + a.kv_heads;
    const long unit = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= (long)a.n_tokens * per_token) return;
    const int t = (int)(unit / per_token), which = (int)(unit - (long)t * per_token);
    const bool is_key = which >= a.heads;
    const int hd = is_key ? which - a.heads : which;
    const int dim = a.dim;
    // where the results go: the query buffer, or the token's cache row of this head
    C* crow = nullptr;
    if (is_key) {
        const int slot = a.slots ? a.slots[t] : -1;
        if (slot < 0) {
            if (a.conv_q == nullptr || !a.write_state || a.seq[t] < 0) return;
        } else {
            const int page = slot / a.page_size, off = slot - page * a.page_size;
            if (page >= a.num_pages) {
                if (lane == 0) prb_set_status(a.status, PRB_S_SLOT_RANGE, t, slot, a.num_pages);
                return;
            }
            crow = reinterpret_cast<C*>(a.cache) +
                   (((size_t)page * a.kv_heads + hd) * a.page_size + off) * (dim + a.vdim);
        }
    }
    HeadInput in;
    in.row = a.proj + (size_t)t * a.ld + (is_key ? a.k_col : a.q_col) + hd * dim;
    const float* bias = is_key ? a.k_bias : a.q_bias;
    in.bias = bias ? bias + hd * dim : nullptr;
    in.w = nullptr;
    in.state = nullptr;
    in.ld = a.ld;
    in.taps = a.taps;
    in.channels = per_token * dim;
    in.pos = a.positions[t];
    in.back = 0;
    float* state = nullptr;
    if (a.conv_q != nullptr) {
        const int b = a.seq[t];
        in.w = (is_key ? a.conv_k : a.conv_q) + (size_t)hd * dim * a.taps;
        if (b >= 0) {
            in.back = t - a.q_start[b];
            const int slot = a.state_slot[b];
            if (slot < 0 || slot >= a.n_slots) {
                if (lane == 0) prb_set_status(a.status, PRB_S_SLOT_RANGE, t, slot, a.n_slots);
            } else if (a.taps > 1) {
                state = a.conv_state + (size_t)slot * (a.taps - 1) * in.channels + which * dim;
            }
        } else {
            in.pos = 0;                                  // a padding row: nothing before it
        }
        in.state = state;
    }
    const int half = a.rot_dims / 2;
    const int units = half + (dim - a.rot_dims);         // pairs, then coordinates that stay
    const float pos = (float)in.pos;
    const float2* ang = a.angles ? a.angles + (size_t)t * half : nullptr;
    auto angle = [&](int u, float& cs, float& sn) {
        if (ang) {
            const float2 v = ang[u];
            cs = v.x;
            sn = v.y;
        } else {
            prb_sincos_angle(pos, a.freq[u], &sn, &cs, a.freq_lo ? a.freq_lo[u] : 0.0f);
        }
    };
    auto first_of = [&](int u) { return a.interleaved ? 2 * u : u; };
    auto second_of = [&](int u) { return a.interleaved ? 2 * u + 1 : u + half; };
    constexpr int NU = U > 0 ? U : 1;
    float r0[NU], r1[NU];                                // (r1: a pair's second number)
    if constexpr (U > 0) {
#pragma unroll
        for (int k = 0; k < U; ++k) {
            const int u = lane + 32 * k;
            r0[k] = u < units ? in.get(u < half ? first_of(u) : u - half + a.rot_dims) : 0.0f;
            r1[k] = u < half ? in.get(second_of(u)) : 0.0f;
        }
    }
    // unit u's numbers: from the registers, or computed
    auto first_number = [&](int u, int k) {
        if constexpr (U > 0) return r0[k];
        else return in.get(u < half ? first_of(u) : u - half + a.rot_dims);
    };
    auto second_number = [&](int u, int k) {
        if constexpr (U > 0) return r1[k];
        else return in.get(second_of(u));
    };
    // every unit of the lane in turn (a loop the compiler can unroll when U is given)
    auto each_unit = [&](auto f) {
        if constexpr (U > 0) {
#pragma unroll
            for (int k = 0; k < U; ++k)
                if (lane + 32 * k < units) f(lane + 32 * k, k);
        } else {
            for (int u = lane; u < units; u += 32) f(u, 0);
        }
    };
    float pre = 1.0f, post = 1.0f;
    if (!is_key && a.temp_every > 0)
        post = 1.0f + a.temp_coef * logf((float)((in.pos + 1) / a.temp_every) + 1.0f);
    if (a.norm_mode == 2 || a.norm_mode == 3) {
        float ss = 0.0f;
        each_unit([&](int u, int k) {
            const float x0 = first_number(u, k);
            if (u >= half) {
                ss = fmaf(x0, x0, ss);
                return;
            }
            const float x1 = second_number(u, k);
            if (a.norm_mode == 2) {
                ss = fmaf(x0, x0, fmaf(x1, x1, ss));
            } else {
                float sn, cs;
                angle(u, cs, sn);
                const float y0 = x0 * cs - x1 * sn, y1 = x1 * cs + x0 * sn;
                ss = fmaf(y0, y0, fmaf(y1, y1, ss));
            }
        });
        const float inv = 1.0f / sqrtf(prb_warp_sum(ss) / (float)dim + a.eps);
        if (a.norm_mode == 2) pre = inv;
        else post *= inv;
    }
    const float* nw = a.norm_mode == 2 ? (is_key ? a.k_norm : a.q_norm) : nullptr;
    float* qrow = is_key ? nullptr : a.q_out + ((size_t)t * a.heads + hd) * dim;
    const bool keys_are_values = is_key && a.v_col < 0;
    auto store = [&](int i, float v) {
        if (!is_key) qrow[i] = v;
        else if (crow) crow[i] = prb_from_float<C>(v);
    };
    // pairs whose two numbers are neighbours go out in one piece
    const bool together = a.interleaved && dim % 2 == 0 && a.vdim % 2 == 0;
    auto store2 = [&](int i0, int i1, float y0, float y1, float x0, float x1) {
        if (!is_key) {
            if (together) {
                *reinterpret_cast<float2*>(qrow + i0) = make_float2(y0, y1);
            } else {
                qrow[i0] = y0;
                qrow[i1] = y1;
            }
            return;
        }
        if (crow == nullptr) return;
        if (together) {
            store_pair(crow + i0, y0, y1);
            if (keys_are_values) store_pair(crow + dim + i0, x0, x1);
        } else {
            crow[i0] = prb_from_float<C>(y0);
            crow[i1] = prb_from_float<C>(y1);
            if (keys_are_values) {
                crow[dim + i0] = prb_from_float<C>(x0);
                crow[dim + i1] = prb_from_float<C>(x1);
            }
        }
    };
    each_unit([&](int u, int k) {
        const float x0 = first_number(u, k);
        if (u < half) {
            const int i0 = first_of(u), i1 = second_of(u);
            const float x1 = second_number(u, k);
            float sn, cs;
            angle(u, cs, sn);
            const float y0 = x0 * pre * (nw ? nw[i0] : 1.0f), y1 = x1 * pre * (nw ? nw[i1] : 1.0f);
            store2(i0, i1, (y0 * cs - y1 * sn) * post, (y1 * cs + y0 * sn) * post, x0, x1);
        } else {
            const int i = u - half + a.rot_dims;
            store(i, x0 * pre * (nw ? nw[i] : 1.0f) * post);
            if (keys_are_values && crow) crow[dim + i] = prb_from_float<C>(x0);
        }
    });
    if (is_key && a.v_col >= 0 && crow) {
        const float* vrow = a.proj + (size_t)t * a.ld + a.v_col + hd * a.vdim;
        for (int j = lane; j < a.vdim; j += 32)
            crow[dim + j] = prb_from_float<C>(vrow[j] + (a.v_bias ? a.v_bias[hd * a.vdim + j] : 0.0f));
    }
    if (state != nullptr && a.write_state) {             // (the lane's own channels, as read above)
        auto shift = [&](int i) {
            for (int j = 0; j + 1 < a.taps - 1; ++j)
                state[(long)j * in.channels + i] = state[(long)(j + 1) * in.channels + i];
            state[(long)(a.taps - 2) * in.channels + i] = in.raw(i);
        };
        for (int u = lane; u < units; u += 32) {
            if (u < half) {
                shift(first_of(u));
                shift(second_of(u));
            } else {
                shift(u - half + a.rot_dims);
            }
        }
    }
}

// The saved inputs after a step with portions: a thread per (request, channel).
__global__ void wattn_conv_state_kernel(PrepArgs a) {
    prb_grid_launch_dependents();
    const int b = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int nq = a.heads * a.dim, channels = nq + a.kv_heads * a.dim;
    if (c >= channels) return;
    const int t0 = a.q_start[b], t1 = a.q_start[b + 1];
    if (t1 <= t0 || t0 < 0 || t1 > a.n_tokens) return;
    const int slot = a.state_slot[b];
    if (slot < 0 || slot >= a.n_slots) return;          // (said by the kernel before)
    const int keep = a.taps - 1, n = t1 - t0;
    float* st = a.conv_state + (size_t)slot * keep * channels + c;
    const int col = c < nq ? a.q_col + c : a.k_col + (c - nq);
    const float* bias = c < nq ? a.q_bias : a.k_bias;
    const float bv = bias ? bias[c < nq ? c : c - nq] : 0.0f;
    for (int j = 0; j < keep; ++j) {                     // (what is read lies at or behind what is written)
        const int src = j + n;                           // place in [saved inputs | the portion]
        st[(long)j * channels] = src < keep ? st[(long)src * channels]
                                            : a.proj[(size_t)(t0 + src - keep) * a.ld + col] + bv;
    }
}

__global__ void rotary_angles_kernel(float2* __restrict__ out, const int* __restrict__ positions,
                                     const float* __restrict__ freq, const float* __restrict__ freq_lo,
                                     int n_tokens, int half, float magnitude) {
    prb_grid_launch_dependents();
    const long e = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= (long)n_tokens * half) return;
    const int t = (int)(e / half), i = (int)(e - (long)t * half);
    float sn, cs;
    prb_sincos_angle((float)positions[t], freq[i], &sn, &cs, freq_lo ? freq_lo[i] : 0.0f);
    out[e] = make_float2(cs * magnitude, sn * magnitude);
}
}  // namespace

PRB_API int prb_rotary_angles(void* out, const int* positions, const float* freq, const float* freq_lo,
                              int n_tokens, int half, float magnitude, cudaStream_t stream) {
    if (n_tokens <= 0 || half <= 0) return 0;
    if (((uintptr_t)out) % 8 != 0) return PRB_E_ALIGN;
    const long total = (long)n_tokens * half;
    rotary_angles_kernel<<<(unsigned)((total + 127) / 128), 128, 0, stream>>>(
        (float2*)out, positions, freq, freq_lo, n_tokens, half, magnitude);
    PRB_LAUNCH_CHECK();
    return 0;
}

// n_requests > 0 with a convolution: the saved inputs are brought up to date by a second kernel
// (a step with portions); 0: by the first (every request brings one token).
PRB_API int prb_wattn_prepare_heads(float* q_out, void* cache, const float* proj, long ld, int q_col,
                                    int k_col, int v_col, const float* q_norm, const float* k_norm,
                                    const float* q_bias, const float* k_bias, const float* v_bias,
                                    const float* conv_q, const float* conv_k, int taps,
                                    float* conv_state, int n_slots, const int* seq,
                                    const int* q_start, const int* state_slot, int n_requests,
                                    const int* slots, const int* positions, const float* freq,
                                    const float* freq_lo, const void* angles, int n_tokens, int heads,
                                    int kv_heads, int dim, int vdim, int rot_dims, int interleaved,
                                    int norm_mode, float eps, float temp_coef, int temp_every,
                                    int page_size, int num_pages, int cache_dtype, int* status,
                                    cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || rot_dims < 0 || rot_dims % 2 ||
        rot_dims > dim || page_size <= 0 || n_requests < 0 || n_requests > 65535)
        return PRB_E_SIZE;
    if (norm_mode != 0 && norm_mode != 2 && norm_mode != 3) return PRB_E_ARG;
    if (v_col < 0 && vdim != dim) return PRB_E_SIZE;
    if (norm_mode == 2 && (q_norm == nullptr || (slots != nullptr && k_norm == nullptr))) return PRB_E_ARG;
    if (conv_q != nullptr && (conv_k == nullptr || taps < 1 || seq == nullptr || q_start == nullptr ||
                              state_slot == nullptr || (taps > 1 && conv_state == nullptr)))
        return PRB_E_ARG;
    PrepArgs a{q_out, cache, proj, ld, q_col, k_col, v_col, q_norm, k_norm, q_bias, k_bias, v_bias,
               conv_q, conv_k, taps, conv_state, n_slots, n_requests == 0 ? 1 : 0, seq, q_start,
               state_slot, slots, positions, freq, freq_lo, (const float2*)angles, n_tokens, heads,
               kv_heads, dim, vdim, rot_dims, interleaved, norm_mode, eps, temp_coef, temp_every,
               page_size, num_pages, status};
    const long units = (long)n_tokens * (heads + kv_heads);
    // few units: two warps a CTA, so that they spread over the SMs
    const int warps = units <= 4L * prb_sm_count() ? 2 : 8;
    const unsigned blocks = (unsigned)((units + warps - 1) / warps);
    const int lane_units = (dim - rot_dims / 2 + 31) / 32;
#define PREP1(CT, UN) wattn_prepare_heads_kernel<CT, UN><<<blocks, warps * 32, 0, stream>>>(a)
#define PREP(CT)                                                                                 \
    do {                                                                                         \
        if (lane_units == 1) PREP1(CT, 1);                                                       \
        else if (lane_units == 2) PREP1(CT, 2);                                                  \
        else if (lane_units <= 4) PREP1(CT, 4);                                                  \
        else PREP1(CT, 0);                                                                       \
    } while (0)
    if (cache_dtype == PRB_F32) PREP(float);
    else if (cache_dtype == PRB_BF16) PREP(__nv_bfloat16);
    else return PRB_E_DTYPE;
#undef PREP
#undef PREP1
    PRB_LAUNCH_CHECK();
    if (conv_q != nullptr && taps > 1 && n_requests > 0) {
        const int channels = (heads + kv_heads) * dim;
        wattn_conv_state_kernel<<<dim3((channels + 127) / 128, n_requests), 128, 0, stream>>>(a);
        PRB_LAUNCH_CHECK();
    }
    return 0;
}
