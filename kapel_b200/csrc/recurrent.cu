// Mechanisms that carry something from a request's last row to its next one, for mixers whose inputs
// come as one stacked product [rows, row_width] (a tensor or split-K partial sums).
//
//  token_shift       y[r] = h[r] + (h[r-1] - h[r]) * mu, channel by channel; the row before a request's
//                    first row of the step comes from its slot of a state table (zeros for a new request);
//                    `keep_last` then leaves the request's last h there.
//  conv_append       a short causal convolution over time on every channel of a query and a key
//                    projection (bias first, one filter a channel, no activation), the queries written
//                    out, the keys to the paged cache at each row's line; the last taps - 1 inputs of every
//                    channel live in a slot of a state table (`conv_history`).
//  decay_scan        a matrix memory S [d, e] a head with a decay a key channel and, optionally, the removal
//                    of what lies along a unit key:
//                        S <- diag(w) S - b (u^T S) + k v^T,   o = S^T r      (both first terms read the old S)
//                    Written on the old memory: with p = u^T S and q = (w r)^T S, o = q - p (b.r) + v (k.r),
//                    so both dot products of a row are reduced together. `gdelta_prep` (the generalized
//                    delta rule: decay through a small two-layer net, removal rate, unit keys),
//                    `gate_prep` (tied gates: a forget gate with a lower bound, and one minus it as the input gate:
//                    w = f, k = 1 - f, no removal), `cdelta_prep` (the gated delta rule with a decay a key channel:
//                    S <- diag(w) S + b (v - p)^T, o = q + (v - p) (b.r)) and `retention_prep` (a fixed decay a
//                    head, rotated queries and keys) make its inputs.
//  conv_rows         the convolution alone: a bias, the filter, another bias, written out in 32-bit.
//  weighted_sum2     out = a * va + b * vb + vc with a weight a channel on each branch.
//
// Everything here is 32-bit; only the projections may come in bfloat16.
#include "common.cuh"

namespace kb {

// retention.cu: a fixed decay's memory by chunks of rows
long long retention_chunk_floats(int rows, int entries, int heads, int d, int e);
int run_retention_chunks(float* out, const float* vec, const float* val, const float* scal, const float* decay, float* sums, float* state,
                         int n_slots, const int* entry_start, const int* entry_end, const int* slots, int entries, int longest, int heads,
                         int d, int e, cudaStream_t s);

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float rc_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// ------------------------------------------------------------------------------------------ token shift
template <typename T>
__global__ void token_shift_kernel(T* __restrict__ out, const T* __restrict__ h, const float* __restrict__ mu,
                                   const float* __restrict__ state, const int* __restrict__ row_entry,
                                   const int* __restrict__ entry_start, const int* __restrict__ slots, int entries, int n_slots,
                                   int width, int out_stride) {
    const int r = blockIdx.x;
    const int entry = row_entry[r];
    int r0 = r, slot = 0;
    if (entry >= 0 && entry < entries) {
        r0 = entry_start[entry];
        slot = slots[entry];
    }
    const bool kept = slot > 0 && slot < n_slots;
    for (int c = threadIdx.x; c < out_stride; c += blockDim.x) {
        float y = 0.f;
        if (c < width) {
            const float cur = Elem<T>::load(h + (size_t)r * width + c);
            const float before = r > r0 ? Elem<T>::load(h + (size_t)(r - 1) * width + c) : (kept ? state[(size_t)slot * width + c] : 0.f);
            y = fmaf(before - cur, mu[c], cur);
        }
        Elem<T>::store(out + (size_t)r * out_stride + c, y);
    }
}

template <typename T>
__global__ void keep_last_kernel(float* __restrict__ state, const T* __restrict__ h, const int* __restrict__ entry_start,
                                 const int* __restrict__ entry_end, const int* __restrict__ slots, int n_slots, int width) {
    const int entry = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int r0 = entry_start[entry], r1 = entry_end[entry];
    const int slot = slots[entry];
    if (c >= width || r1 <= r0 || slot <= 0 || slot >= n_slots) return;
    state[(size_t)slot * width + c] = Elem<T>::load(h + (size_t)(r1 - 1) * width + c);
}

// ------------------------------------------------------------------------------------------ convolutions ahead of attention
constexpr int CONV_MAX_TAPS = 16;

struct ConvParams {
    int row_width, q_off, k_off, nq, nk;      // columns of the stacked product; nq = hq d, nk = hkv d
    const float* bias;                        // [nq + nk] or null
    const float* conv;                        // [nq + nk, taps]: the last weight is the row's own
    const float* after;                       // [nq + nk] or null: added behind the filter
    float* state;                             // [slots, (taps - 1) (nq + nk)]
    const int* row_entry;
    const int* entry_start;
    const int* entry_end;
    const int* slots;
    const int* lines;
    int n_slots, entries, rows, taps, hkv, d, page_size, q_stride;
    long long table_lines;
};

template <typename TS, typename TO>
__global__ void conv_append_kernel(const Src<TS> src, const ConvParams p, TO* __restrict__ q_out, TO* __restrict__ k_table) {
    const int r = blockIdx.x;
    const int channels = p.nq + p.nk;
    const int entry = p.row_entry[r];
    int r0 = r, slot = 0;
    if (entry >= 0 && entry < p.entries) {
        r0 = p.entry_start[entry];
        slot = p.slots[entry];
    }
    const bool kept = slot > 0 && slot < p.n_slots;
    const float* hist = p.state + (size_t)(kept ? slot : 0) * (p.taps - 1) * channels;
    long long line = -1;
    if (k_table != nullptr) {
        line = p.lines[r];
        if (line >= p.table_lines) line = -1;
    }
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
        const bool is_q = c < p.nq;
        if (!is_q && line < 0) continue;
        const int col = is_q ? p.q_off + c : p.k_off + (c - p.nq);
        const float b = p.bias != nullptr ? p.bias[c] : 0.f;
        float y = 0.f;
        for (int j = 0; j < p.taps; ++j) {                      // the input j rows back
            const int t = r - j;
            float x;
            if (t >= r0) x = src.at((size_t)t * p.row_width + col) + b;
            else if (kept) x = hist[(size_t)(p.taps - 1 + (t - r0)) * channels + c];
            else x = 0.f;
            y = fmaf(p.conv[(size_t)c * p.taps + (p.taps - 1 - j)], x, y);
        }
        if (p.after != nullptr) y += p.after[c];
        if (is_q) {
            Elem<TO>::store(q_out + (size_t)r * p.q_stride + c, y);
        } else {
            const int ck = c - p.nq, h = ck / p.d, i = ck - h * p.d;
            Elem<TO>::store(k_table + kv_row(line, h, p.hkv, p.page_size) * p.d + i, y);
        }
    }
    for (int c = p.nq + threadIdx.x; c < p.q_stride; c += blockDim.x) Elem<TO>::store(q_out + (size_t)r * p.q_stride + c, 0.f);
}

// history <- the last taps - 1 inputs (bias added) of (history, this step's rows), per channel of a request.
template <typename TS>
__global__ void conv_history_kernel(const Src<TS> src, const ConvParams p) {
    const int entry = blockIdx.y;
    const int channels = p.nq + p.nk;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    const int slot = p.slots[entry];
    const int keep = p.taps - 1;
    if (r1 <= r0 || slot <= 0 || slot >= p.n_slots || keep <= 0) return;
    float* hist = p.state + (size_t)slot * keep * channels;
    const int col = c < p.nq ? p.q_off + c : p.k_off + (c - p.nq);
    const float b = p.bias != nullptr ? p.bias[c] : 0.f;
    const int n = r1 - r0;
    float fresh[CONV_MAX_TAPS];
#pragma unroll
    for (int i = 0; i < CONV_MAX_TAPS; ++i) {
        fresh[i] = 0.f;
        if (i < keep) {
            const int t = n - keep + i;
            fresh[i] = t >= 0 ? src.at((size_t)(r0 + t) * p.row_width + col) + b : hist[(size_t)(keep + t) * channels + c];
        }
    }
#pragma unroll
    for (int i = 0; i < CONV_MAX_TAPS; ++i)
        if (i < keep) hist[(size_t)i * channels + c] = fresh[i];
}

// ------------------------------------------------------------------------------------------ the scan's inputs
// Scratch of a step: vectors [rows, heads, NV, d] as the scan's mode lists them below, values [rows, heads, e],
// scalars [rows, heads, 2] = (b.r, k.r).
struct ScanInputs {
    float* vec;
    float* val;
    float* scal;
    int nv;
};

struct GDeltaParams {
    int row_width, r_off, k_off, v_off, a_off, w1_off, lora;
    const float* w2;            // [lora, heads d]: the net's second layer turned, so that neighbouring threads read neighbouring weights
    const float* w0;            // [heads d]
    const float* a_bias;        // [heads d]
    float decay_scale;          // w = exp(-decay_scale * sigmoid(.))
    float unit_eps;
    int heads, d;
};

// One block RB rows. The small net's hidden layers tanh(w1 h) of the block's rows lie in shared memory; a thread a channel
// reads its weights of the second layer once for all RB rows and leaves the decay and the removal rate in the scratch
// (which the same block reads back below); a warp a (row, head) then makes the unit key and the two dot products.
// RB is 8 for prompt portions (the second layer's weights cross from L2 once in eight rows) and 1 for a few rows.
template <typename TS, int RB>
__global__ void __launch_bounds__(1024)
gdelta_prep_kernel(const Src<TS> src, const GDeltaParams p, const ScanInputs s, int rows) {
    extern __shared__ float hid[];                              // [RB][lora]
    const int r0 = blockIdx.x * RB;
    const int nr = min(RB, rows - r0);
    const int n = p.heads * p.d, d = p.d;
    for (int idx = threadIdx.x; idx < RB * p.lora; idx += blockDim.x) {
        const int rr = idx / p.lora, j = idx - rr * p.lora;
        hid[idx] = rr < nr ? tanhf(src.at((size_t)(r0 + rr) * p.row_width + p.w1_off + j)) : 0.f;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        float z[RB];
#pragma unroll
        for (int rr = 0; rr < RB; ++rr) z[rr] = 0.f;
        for (int j = 0; j < p.lora; ++j) {
            const float wj = p.w2[(size_t)j * n + c];
#pragma unroll
            for (int rr = 0; rr < RB; ++rr) z[rr] = fmaf(wj, hid[rr * p.lora + j], z[rr]);
        }
        const float w0 = p.w0[c], ab = p.a_bias[c];
        const int h = c / d, i = c - h * d;
#pragma unroll
        for (int rr = 0; rr < RB; ++rr) {
            if (rr < nr) {
                float* vec = s.vec + ((size_t)(r0 + rr) * p.heads + h) * 5 * d;
                vec[d + i] = expf(-p.decay_scale * rc_sigmoid(z[rr] + w0));
                vec[4 * d + i] = rc_sigmoid(src.at((size_t)(r0 + rr) * p.row_width + p.a_off + c) + ab);      // the rate; times the unit key below
            }
        }
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int pair = warp; pair < nr * p.heads; pair += warps) {
        const int rr = pair / p.heads, h = pair - rr * p.heads;
        const int r = r0 + rr;
        const size_t base = (size_t)r * p.row_width;
        float kk = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float k = src.at(base + p.k_off + h * d + i);
            kk = fmaf(k, k, kk);
        }
        kk = warp_sum(kk);
        const float inv = 1.f / sqrtf(kk + p.unit_eps);
        float br = 0.f, kr = 0.f;
        float* vec = s.vec + ((size_t)r * p.heads + h) * 5 * d;
        for (int i = lane; i < d; i += 32) {
            const int c = h * d + i;
            const float k = src.at(base + p.k_off + c), q = src.at(base + p.r_off + c);
            const float u = k * inv, b = vec[4 * d + i] * u, w = vec[d + i];
            vec[i] = w * q;
            vec[2 * d + i] = k;
            vec[3 * d + i] = u;
            vec[4 * d + i] = b;
            br = fmaf(b, q, br);
            kr = fmaf(k, q, kr);
            s.val[(size_t)r * n + c] = src.at(base + p.v_off + c);
        }
        br = warp_sum(br);
        kr = warp_sum(kr);
        if (lane == 0) {
            s.scal[((size_t)r * p.heads + h) * 2] = br;
            s.scal[((size_t)r * p.heads + h) * 2 + 1] = kr;
        }
    }
}

struct GateParams {
    int row_width, q_off, f_off, v_off;
    const float* f_bias;        // [heads d]
    const float* lower;         // [heads d]
    int heads, d, e;
};

// One block a row: q = silu(.), f = l + (1 - l) sigmoid(. + bias); the scan's inputs are w r = f q, w = f, k = 1 - f.
template <typename TS>
__global__ void __launch_bounds__(256)
gate_prep_kernel(const Src<TS> src, const GateParams p, const ScanInputs s) {
    const int r = blockIdx.x;
    const size_t base = (size_t)r * p.row_width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int h = warp; h < p.heads; h += warps) {
        float kr = 0.f;
        float* vec = s.vec + ((size_t)r * p.heads + h) * 3 * p.d;
        for (int i = lane; i < p.d; i += 32) {
            const int c = h * p.d + i;
            const float z = src.at(base + p.q_off + c);
            const float q = z * rc_sigmoid(z);
            const float l = p.lower[c];
            const float f = fmaf(1.f - l, rc_sigmoid(src.at(base + p.f_off + c) + p.f_bias[c]), l);
            vec[i] = f * q;
            vec[p.d + i] = f;
            vec[2 * p.d + i] = 1.f - f;
            kr = fmaf(1.f - f, q, kr);
        }
        kr = warp_sum(kr);
        if (lane == 0) {
            s.scal[((size_t)r * p.heads + h) * 2] = 0.f;
            s.scal[((size_t)r * p.heads + h) * 2 + 1] = kr;
        }
    }
    const int nv = p.heads * p.e;
    for (int i = threadIdx.x; i < nv; i += blockDim.x) s.val[(size_t)r * nv + i] = src.at(base + p.v_off + i);
}

struct CDeltaParams {
    int row_width, q_off, k_off, v_off, b_off, a1_off, rank;
    const float* a2;            // [rank, heads d]: the decay's second factor turned, so that neighbouring threads read neighbouring weights
    const float* dt_bias;       // [heads d]
    const float* a_log;         // [heads]
    const float* conv;          // [2 kv_heads d + heads e, taps]: q's channels, then k's, then v's
    const float* state;         // [slots, (taps - 1) channels]: the convolutions' last inputs
    const int* row_entry;
    const int* entry_start;
    const int* slots;
    int n_slots, entries, heads, kv_heads, d, e, taps;
    float q_scale, unit_eps;
};

__device__ __forceinline__ float rc_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// The convolution and silu of one channel of a row: the inputs before the step come from the request's history.
template <typename TS>
__device__ __forceinline__ float conv_silu(const Src<TS>& src, const CDeltaParams& p, int r, int r0, const float* hist, int channels, int col, int c) {
    float y = 0.f;
    for (int j = 0; j < p.taps; ++j) {                          // the input j rows back
        const int t = r - j;
        float x = 0.f;
        if (t >= r0) x = src.at((size_t)t * p.row_width + col);
        else if (hist != nullptr) x = hist[(size_t)(p.taps - 1 + (t - r0)) * channels + c];
        y = fmaf(p.conv[(size_t)c * p.taps + (p.taps - 1 - j)], x, y);
    }
    return y * rc_sigmoid(y);
}

// One block RB rows. The decay of every (head, key channel) is a thread's: exp(-exp(A_log) softplus(a2 . hidden + dt_bias)), its
// column of a2 read once for the block's rows; a warp a (row, head) then convolves that head's query and key, makes them unit
// vectors and leaves (g q, g, beta k, g k) and beta k.q; a thread a channel the values.
template <typename TS, int RB>
__global__ void __launch_bounds__(1024)
cdelta_prep_kernel(const Src<TS> src, const CDeltaParams p, const ScanInputs s, int rows) {
    extern __shared__ float hid[];                              // [RB][rank]
    const int r0 = blockIdx.x * RB;
    const int nr = min(RB, rows - r0);
    const int d = p.d, n = p.heads * d, nq = p.kv_heads * d, nv = p.heads * p.e;
    const int channels = 2 * nq + nv;
    for (int idx = threadIdx.x; idx < RB * p.rank; idx += blockDim.x) {
        const int rr = idx / p.rank, j = idx - rr * p.rank;
        hid[idx] = rr < nr ? src.at((size_t)(r0 + rr) * p.row_width + p.a1_off + j) : 0.f;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        float z[RB];
#pragma unroll
        for (int rr = 0; rr < RB; ++rr) z[rr] = 0.f;
        for (int j = 0; j < p.rank; ++j) {
            const float wj = p.a2[(size_t)j * n + c];
#pragma unroll
            for (int rr = 0; rr < RB; ++rr) z[rr] = fmaf(wj, hid[rr * p.rank + j], z[rr]);
        }
        const float bias = p.dt_bias[c];
        const int h = c / d, i = c - h * d;
        const float rate = expf(p.a_log[h]);
#pragma unroll
        for (int rr = 0; rr < RB; ++rr)
            if (rr < nr) s.vec[((size_t)(r0 + rr) * p.heads + h) * 4 * d + d + i] = expf(-rate * rc_softplus(z[rr] + bias));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int per = p.heads / p.kv_heads;
    for (int pair = warp; pair < nr * p.heads; pair += warps) {
        const int rr = pair / p.heads, h = pair - rr * p.heads;
        const int r = r0 + rr, kvh = h / per;
        const int entry = p.row_entry[r];
        const bool known = entry >= 0 && entry < p.entries;
        const int first = known ? p.entry_start[entry] : r;
        const int slot = known ? p.slots[entry] : 0;
        const float* hist = slot > 0 && slot < p.n_slots ? p.state + (size_t)slot * (p.taps - 1) * channels : nullptr;
        float q[8], k[8];                                       // d <= 256
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const int i = lane + 32 * x;
            q[x] = k[x] = 0.f;
            if (i < d) {
                const int c = kvh * d + i;
                q[x] = conv_silu(src, p, r, first, hist, channels, p.q_off + c, c);
                k[x] = conv_silu(src, p, r, first, hist, channels, p.k_off + c, nq + c);
                sq = fmaf(q[x], q[x], sq);
                sk = fmaf(k[x], k[x], sk);
            }
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        const float iq = p.q_scale / sqrtf(sq + p.unit_eps), ik = 1.f / sqrtf(sk + p.unit_eps);
        const float beta = rc_sigmoid(src.at((size_t)r * p.row_width + p.b_off + h));
        float* vec = s.vec + ((size_t)r * p.heads + h) * 4 * d;
        float br = 0.f;
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const int i = lane + 32 * x;
            if (i < d) {
                const float g = vec[d + i], qn = q[x] * iq, kn = k[x] * ik;
                vec[i] = g * qn;
                vec[2 * d + i] = beta * kn;
                vec[3 * d + i] = g * kn;
                br = fmaf(beta * kn, qn, br);
            }
        }
        br = warp_sum(br);
        if (lane == 0) {
            s.scal[((size_t)r * p.heads + h) * 2] = br;
            s.scal[((size_t)r * p.heads + h) * 2 + 1] = 0.f;
        }
    }
    for (int idx = threadIdx.x; idx < nr * nv; idx += blockDim.x) {
        const int rr = idx / nv, c = idx - rr * nv;
        const int r = r0 + rr;
        const int entry = p.row_entry[r];
        const bool known = entry >= 0 && entry < p.entries;
        const int first = known ? p.entry_start[entry] : r;
        const int slot = known ? p.slots[entry] : 0;
        const float* hist = slot > 0 && slot < p.n_slots ? p.state + (size_t)slot * (p.taps - 1) * channels : nullptr;
        s.val[(size_t)r * nv + c] = conv_silu(src, p, r, first, hist, channels, p.v_off + c, 2 * nq + c);
    }
}

struct RetentionParams {
    int row_width, q_off, k_off, v_off;
    const float* decay;         // [heads]
    const float2* cos_sin;      // [rows, rotary / 2]
    int rotary, heads, d, e;
    float k_scale;
    int act;                    // 1: silu on queries, keys and values as they come from the product
};

// One block a row, a warp a head: queries, keys and values through the activation, queries and keys turned (component i with
// i + rotary / 2), keys scaled; the scan's inputs are decay q and k.
template <typename TS>
__global__ void __launch_bounds__(1024)
retention_prep_kernel(const Src<TS> src, const RetentionParams p, const ScanInputs s) {
    const int r = blockIdx.x;
    const size_t base = (size_t)r * p.row_width;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int half = p.rotary >> 1, d = p.d;
    auto at = [&](size_t i) {
        const float v = src.at(i);
        return p.act == 1 ? v * rc_sigmoid(v) : v;
    };
    for (int h = warp; h < p.heads; h += warps) {
        float kr = 0.f;
        const float decay = p.decay[h];
        float* vec = s.vec + ((size_t)r * p.heads + h) * 2 * d;
        auto put = [&](int i, float q, float k) {
            k *= p.k_scale;
            vec[i] = decay * q;
            vec[d + i] = k;
            kr = fmaf(k, q, kr);
        };
        const size_t qa = base + p.q_off + (size_t)h * d, ka = base + p.k_off + (size_t)h * d;
        for (int i = lane; i < half; i += 32) {
            float q0 = at(qa + i), q1 = at(qa + half + i), k0 = at(ka + i), k1 = at(ka + half + i);
            const float2 cs = p.cos_sin[(size_t)r * half + i];
            rope_rotate(q0, q1, cs);
            rope_rotate(k0, k1, cs);
            put(i, q0, k0);
            put(half + i, q1, k1);
        }
        for (int i = 2 * half + lane; i < d; i += 32) put(i, at(qa + i), at(ka + i));
        kr = warp_sum(kr);
        if (lane == 0) {
            s.scal[((size_t)r * p.heads + h) * 2] = 0.f;
            s.scal[((size_t)r * p.heads + h) * 2 + 1] = kr;
        }
    }
    const int nv = p.heads * p.e;
    for (int i = threadIdx.x; i < nv; i += blockDim.x) s.val[(size_t)r * nv + i] = at(base + p.v_off + i);
}

// ------------------------------------------------------------------------------------------ the scan
// What the vectors of a row are, and what a row does:
//   SCAN_GATE     (w r, w, k)         S <- diag(w) S + k v^T
//   SCAN_REMOVAL  (w r, w, k, u, b)   S <- diag(w) S - b (u^T S) + k v^T
//   SCAN_WRITE    (w r, w, b, u)      S <- diag(w) S + b (v - u^T S)^T
//   SCAN_FIXED    (w r, k)            S <- w S + k v^T with one w a head
enum ScanMode { SCAN_GATE = 0, SCAN_REMOVAL = 1, SCAN_WRITE = 2, SCAN_FIXED = 3 };
__host__ __device__ constexpr int scan_vectors(int mode) { return mode == SCAN_REMOVAL ? 5 : (mode == SCAN_WRITE ? 4 : (mode == SCAN_FIXED ? 2 : 3)); }
constexpr int SC = 4;                  // warps a block
constexpr int SCAN_R = 8;              // memory rows a lane can hold: d <= 32 * SCAN_R

struct ScanParams {
    const float* vec;           // [rows, heads, NV, d]
    const float* val;           // [rows, heads, e]
    const float* scal;          // [rows, heads, 2]
    const float* fixed;         // [heads] the decay of SCAN_FIXED
    float* state;               // [slots, heads, e, d]: a column of a head's memory lies together
    const int* entry_start;
    const int* entry_end;
    const int* slots;
    int n_slots, heads, d, e;
    float* out;                 // [rows, heads, e]
};

__device__ __forceinline__ void scan_copy4(float* dst, const float* src) {
    const uint32_t d32 = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d32), "l"(src) : "memory");
}
__device__ __forceinline__ void scan_copy16(float* dst, const float* src) {
    const uint32_t d32 = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d32), "l"(src) : "memory");
}

// R values that lie together, by the widest loads that fit (shared memory, 16-byte aligned where R >= 4).
template <int R>
__device__ __forceinline__ void scan_load(float (&dst)[R], const float* p) {
    if constexpr (R % 4 == 0) {
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const float4 v = reinterpret_cast<const float4*>(p)[i];
            dst[4 * i] = v.x; dst[4 * i + 1] = v.y; dst[4 * i + 2] = v.z; dst[4 * i + 3] = v.w;
        }
    } else if constexpr (R == 2) {
        const float2 v = *reinterpret_cast<const float2*>(p);
        dst[0] = v.x; dst[1] = v.y;
    } else {
#pragma unroll
        for (int i = 0; i < R; ++i) dst[i] = p[i];
    }
}

// One block = one request of the step x one head x SC * DW columns of the memory; a warp DW columns, lane l
// the rows R l .. R l + R - 1 of them in registers (a row's vectors then come from shared memory 16 bytes a load). R: rows a lane holds; CH: rows of the step staged at a time
// (asynchronous copies, the next chunk while this one is walked).
template <int R, int CH, int DW, int MODE>
__global__ void __launch_bounds__(SC * 32)
decay_scan_kernel(const ScanParams p) {
    constexpr int NV = scan_vectors(MODE);
    constexpr bool TWO_SUMS = MODE == SCAN_REMOVAL || MODE == SCAN_WRITE;      // p = u^T S beside q
    constexpr int DP = R * 32;
    constexpr int COLS = SC * DW;
    constexpr int tail = NV * DP;                               // v [COLS] | b.r | k.r | padding
    constexpr int rowf = NV * DP + COLS + 4;
    extern __shared__ __align__(16) float staged[];             // [2][CH][rowf]
    const int entry = blockIdx.x, head = blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int c0 = blockIdx.z * COLS + warp * DW;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    if (r1 <= r0) return;
    const int slot = p.slots[entry];
    const int d = p.d, e = p.e;
    if (slot <= 0 || slot >= p.n_slots) {                       // rows of no request: zeros, no state
        if (lane < DW && c0 + lane < e)
            for (int r = r0; r < r1; ++r) p.out[((size_t)r * p.heads + head) * e + c0 + lane] = 0.f;
        return;
    }
    float* st = p.state + ((size_t)slot * p.heads + head) * e * d;
    float S[DW][R];
#pragma unroll
    for (int ci = 0; ci < DW; ++ci)
#pragma unroll
        for (int i = 0; i < R; ++i) S[ci][i] = (c0 + ci < e && lane * R + i < d) ? st[(size_t)(c0 + ci) * d + lane * R + i] : 0.f;

    const bool wide = d % 4 == 0 && ((uintptr_t)p.vec & 15) == 0;
    auto stage = [&](int chunk, int buf) {
        const int rbase = r0 + chunk * CH;
        const int nr = min(CH, r1 - rbase);
        float* base = staged + (size_t)buf * CH * rowf;
        for (int t = warp; t < nr; t += SC) {
            float* row = base + (size_t)t * rowf;
            const float* vp = p.vec + ((size_t)(rbase + t) * p.heads + head) * NV * d;
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                if (wide) {
                    for (int x = lane * 4; x < d; x += 128) scan_copy16(row + v * DP + x, vp + v * d + x);
                } else {
                    for (int x = lane; x < d; x += 32) scan_copy4(row + v * DP + x, vp + v * d + x);
                }
            }
        }
        for (int idx = tid; idx < nr * (COLS + 2); idx += SC * 32) {
            const int t = idx / (COLS + 2), x = idx - t * (COLS + 2);
            float* dst = base + (size_t)t * rowf + tail + x;
            const size_t r = (size_t)(rbase + t);
            if (x < COLS) {
                const int cc = blockIdx.z * COLS + x;
                if (cc < e) scan_copy4(dst, p.val + (r * p.heads + head) * e + cc);
                else *dst = 0.f;
            } else {
                scan_copy4(dst, p.scal + (r * p.heads + head) * 2 + (x - COLS));
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (d < DP) {                                               // the vectors' padding, once: no copy ever writes it
        const int pad = DP - d;
        for (int idx = tid; idx < 2 * CH * NV * pad; idx += SC * 32) {
            const int t = idx / (NV * pad), x = idx - t * NV * pad;
            const int v = x / pad, i = x - v * pad;
            staged[(size_t)t * rowf + v * DP + d + i] = 0.f;
        }
    }
    const bool hi16 = lane & 16;
    const float fixed = MODE == SCAN_FIXED ? p.fixed[head] : 0.f;
    const int chunks = (r1 - r0 + CH - 1) / CH;
    stage(0, 0);
    for (int ch = 0; ch < chunks; ++ch) {
        if (ch + 1 < chunks) {
            stage(ch + 1, (ch + 1) & 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int rbase = r0 + ch * CH;
        const int nr = min(CH, r1 - rbase);
        const float* rows = staged + (size_t)(ch & 1) * CH * rowf;
        for (int t = 0; t < nr; ++t) {
            const float* in = rows + (size_t)t * rowf;
            const float br = in[tail + COLS], kr = in[tail + COLS + 1];
            float wr[R], w[R], k[R], u[TWO_SUMS ? R : 1], b[MODE == SCAN_REMOVAL ? R : 1];
            scan_load<R>(wr, in + lane * R);
            if constexpr (MODE == SCAN_FIXED) {
                scan_load<R>(k, in + DP + lane * R);
            } else {
                scan_load<R>(w, in + DP + lane * R);
                scan_load<R>(k, in + 2 * DP + lane * R);
            }
            if constexpr (TWO_SUMS) scan_load<R>(u, in + 3 * DP + lane * R);
            if constexpr (MODE == SCAN_REMOVAL) scan_load<R>(b, in + 4 * DP + lane * R);
#pragma unroll
            for (int ci = 0; ci < DW; ++ci) {
                const float v = in[tail + warp * DW + ci];
                float o;
                if constexpr (TWO_SUMS) {
                    float xp = 0.f, xq = 0.f;
#pragma unroll
                    for (int i = 0; i < R; ++i) {
                        xp = fmaf(S[ci][i], u[i], xp);
                        xq = fmaf(S[ci][i], wr[i], xq);
                    }
                    // two sums over 32 lanes: the halves swap one of them, then both are reduced side by side (the lower lanes
                    // end with p, the upper with q). Two broadcasts then give every lane both; one exchange between the halves
                    // and a choice a lane instead measured a fifth slower (1.23 against 1.03 ms at 2,048 rows, 16 heads of 128).
                    float y = (hi16 ? xq : xp) + __shfl_xor_sync(0xffffffffu, hi16 ? xp : xq, 16);
                    y += __shfl_xor_sync(0xffffffffu, y, 8);
                    y += __shfl_xor_sync(0xffffffffu, y, 4);
                    y += __shfl_xor_sync(0xffffffffu, y, 2);
                    y += __shfl_xor_sync(0xffffffffu, y, 1);
                    const float pp = __shfl_sync(0xffffffffu, y, 0), qq = __shfl_sync(0xffffffffu, y, 16);
                    if constexpr (MODE == SCAN_REMOVAL) {
#pragma unroll
                        for (int i = 0; i < R; ++i) S[ci][i] = fmaf(k[i], v, fmaf(-b[i], pp, w[i] * S[ci][i]));
                        o = fmaf(v, kr, fmaf(-pp, br, qq));
                    } else {
                        const float x = v - pp;
#pragma unroll
                        for (int i = 0; i < R; ++i) S[ci][i] = fmaf(k[i], x, w[i] * S[ci][i]);
                        o = fmaf(x, br, qq);
                    }
                } else {
                    float xq = 0.f;
#pragma unroll
                    for (int i = 0; i < R; ++i) {
                        xq = fmaf(S[ci][i], wr[i], xq);
                        S[ci][i] = fmaf(k[i], v, (MODE == SCAN_FIXED ? fixed : w[i]) * S[ci][i]);
                    }
                    xq = warp_sum(xq);
                    o = fmaf(v, kr, xq);
                }
                if (lane == 0 && c0 + ci < e) p.out[((size_t)(rbase + t) * p.heads + head) * e + c0 + ci] = o;
            }
        }
        __syncthreads();                                        // the chunk's buffer may be written again
    }
#pragma unroll
    for (int ci = 0; ci < DW; ++ci)
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (c0 + ci < e && lane * R + i < d) st[(size_t)(c0 + ci) * d + lane * R + i] = S[ci][i];
}

// ------------------------------------------------------------------------------------------ two branches with a weight a channel
template <typename TA, typename TB>
__global__ void weighted_sum2_kernel(float* __restrict__ out, const Src<TA> a, const float* __restrict__ va, const Src<TB> b,
                                     const float* __restrict__ vb, const float* __restrict__ vc, long long total, int width, bool has_b) {
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int c = (int)(idx % width);
    float y = a.at((size_t)idx) * va[c];
    if (has_b) y = fmaf(b.at((size_t)idx), vb[c], y);
    if (vc != nullptr) y += vc[c];
    out[idx] = y;
}

}  // namespace kb

using namespace kb;

extern "C" int kb_token_shift(void* out, const void* h, int dt, const float* mu, float* state, const int* row_entry,
                              const int* entry_start, const int* entry_end, const int* slots, int entries, int n_slots, int rows,
                              int width, int out_stride, int keep, void* stream) {
    KB_REQUIRE(rows >= 0 && width > 0 && out_stride >= width && entries >= 0 && n_slots >= 1, "token_shift: rows %d, width %d (out %d), %d requests, %d slots",
               rows, width, out_stride, entries, n_slots);
    KB_REQUIRE(out && h && mu && state && row_entry && entry_start && entry_end && slots, "token_shift: a tensor is missing");
    KB_REQUIRE(entries <= 65535, "token_shift: too many requests for one launch");
    if (rows == 0 || entries == 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = width >= 1024 ? 256 : 128;
    const dim3 kgrid((unsigned)((width + 127) / 128), entries);
    if (dt == KB_DT_F32) {
        token_shift_kernel<float><<<rows, threads, 0, s>>>((float*)out, (const float*)h, mu, state, row_entry, entry_start, slots, entries, n_slots, width, out_stride);
        if (int err = check_launch("token_shift")) return err;
        if (keep) keep_last_kernel<float><<<kgrid, 128, 0, s>>>(state, (const float*)h, entry_start, entry_end, slots, n_slots, width);
    } else if (dt == KB_DT_BF16) {
        token_shift_kernel<bf16><<<rows, threads, 0, s>>>((bf16*)out, (const bf16*)h, mu, state, row_entry, entry_start, slots, entries, n_slots, width, out_stride);
        if (int err = check_launch("token_shift")) return err;
        if (keep) keep_last_kernel<bf16><<<kgrid, 128, 0, s>>>(state, (const bf16*)h, entry_start, entry_end, slots, n_slots, width);
    } else {
        return fail("token_shift: dtype code %d is not known", dt);
    }
    return check_launch("token_shift keep");
}

extern "C" int kb_conv_append(void* q_out, int q_stride, void* k_table, int out_dt, const void* src, int in_dt, int splits,
                              long long split_stride, int row_width, int q_off, int k_off, const float* bias, const float* conv,
                              float* state, int n_slots, const int* row_entry, const int* entry_start, const int* entry_end,
                              const int* slots, const int* lines, int entries, int rows, int hq, int hkv, int d, int taps,
                              int write_kv, long long table_lines, int page_size, void* stream) {
    KB_REQUIRE(rows >= 0 && entries >= 0 && hq > 0 && hkv > 0 && d > 0, "conv_append: rows %d, heads %d / %d of %d", rows, hq, hkv, d);
    KB_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "conv_append: a convolution of %d taps (1 to %d)", taps, CONV_MAX_TAPS);
    const int nq = hq * d, nk = hkv * d;
    KB_REQUIRE(row_width > 0 && q_off >= 0 && q_off + nq <= row_width && k_off >= 0 && k_off + nk <= row_width && q_stride >= nq,
               "conv_append: columns q %d, k %d do not fit a row of %d", q_off, k_off, row_width);
    KB_REQUIRE(splits >= 1 && (splits == 1 || split_stride >= (long long)rows * row_width), "conv_append: %d slices %lld apart", splits, split_stride);
    KB_REQUIRE(q_out && conv && state && n_slots >= 1 && row_entry && entry_start && entry_end && slots, "conv_append: a tensor is missing");
    KB_REQUIRE(!write_kv || (lines && k_table && table_lines > 0 && page_size > 0), "conv_append: no cache to write");
    KB_REQUIRE(entries <= 65535, "conv_append: too many requests for one launch");
    if (rows == 0 || entries == 0) return 0;
    ConvParams p;
    p.row_width = row_width; p.q_off = q_off; p.k_off = k_off; p.nq = nq; p.nk = nk; p.bias = bias; p.conv = conv; p.after = nullptr; p.state = state;
    p.row_entry = row_entry; p.entry_start = entry_start; p.entry_end = entry_end; p.slots = slots; p.lines = lines;
    p.n_slots = n_slots; p.entries = entries; p.rows = rows; p.taps = taps; p.hkv = hkv; p.d = d; p.page_size = page_size;
    p.q_stride = q_stride; p.table_lines = table_lines;
    cudaStream_t s = (cudaStream_t)stream;
    void* kt = write_kv ? k_table : nullptr;
    const int channels = nq + nk;
    const int threads = channels >= 2048 ? 512 : 256;
#define KB_CONV(TS, TO)                                                                                                    \
    do {                                                                                                                   \
        conv_append_kernel<TS, TO><<<rows, threads, 0, s>>>(Src<TS>{(const TS*)src, splits, (size_t)split_stride}, p, (TO*)q_out, (TO*)kt); \
        if (int err = check_launch("conv_append")) return err;                                                             \
        if (taps > 1 && write_kv)                                                                                          \
            conv_history_kernel<TS><<<dim3((unsigned)((channels + 127) / 128), entries), 128, 0, s>>>(                      \
                Src<TS>{(const TS*)src, splits, (size_t)split_stride}, p);                                                 \
    } while (0)
    if (in_dt == KB_DT_F32 && out_dt == KB_DT_F32) KB_CONV(float, float);
    else if (in_dt == KB_DT_F32 && out_dt == KB_DT_BF16) KB_CONV(float, bf16);
    else if (in_dt == KB_DT_BF16 && out_dt == KB_DT_BF16) KB_CONV(bf16, bf16);
    else return fail("conv_append: dtype codes %d -> %d are not known", in_dt, out_dt);
#undef KB_CONV
    return check_launch("conv_append history");
}

// Floats of scratch for a step of `rows` rows of the scan in this mode: the vectors, the values, the two scalars.
extern "C" long long kb_decay_scan_scratch_floats(int rows, int heads, int d, int e, int mode) {
    return (long long)rows * heads * ((long long)scan_vectors(mode) * d + e + 2);
}

// 0: the launcher chooses how many columns of the memory a warp of the scan holds; 1 or 2: that many (for tests and measurements).
static int g_scan_columns = 0;
extern "C" void kb_decay_scan_columns(int n) { g_scan_columns = (n == 1 || n == 2 || n == 4) ? n : 0; }

static int run_decay_scan(float* out, const ScanInputs& in, float* state, int n_slots, const int* entry_start, const int* entry_end,
                          const int* slots, int entries, int heads, int d, int e, int mode, const float* fixed, cudaStream_t s) {
    ScanParams p;
    p.fixed = fixed;
    p.vec = in.vec; p.val = in.val; p.scal = in.scal; p.state = state; p.entry_start = entry_start; p.entry_end = entry_end;
    p.slots = slots; p.n_slots = n_slots; p.heads = heads; p.d = d; p.e = e; p.out = out;
    int sms = 148;
    {
        int dev = 0;
        if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    }
    // columns a warp: the most that still leaves about four warps a multiprocessor (a warp reads a row's vectors once for all
    // its columns, and walks them as independent chains)
    const long long columns = (long long)entries * heads * e;
    int dw = g_scan_columns ? g_scan_columns : (columns / 4 >= 4ll * sms ? 4 : (columns / 2 >= 4ll * sms ? 2 : 1));
    KB_REQUIRE((e + SC * dw - 1) / (SC * dw) <= 65535 && heads <= 65535, "decay_scan: too many heads or value components for one launch");
    dim3 grid(entries, heads, (e + SC * dw - 1) / (SC * dw));
    const int need = (d + 31) / 32;
#define KB_SCAN(R, CH, W, MODE)                                                                                   \
    do {                                                                                                          \
        const size_t smem = (size_t)2 * CH * (scan_vectors(MODE) * R * 32 + SC * W + 4) * sizeof(float);          \
        if (smem > 48 * 1024) cudaFuncSetAttribute(decay_scan_kernel<R, CH, W, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        decay_scan_kernel<R, CH, W, MODE><<<grid, SC * 32, smem, s>>>(p);                                         \
    } while (0)
#define KB_SCAN_M(R, CH, MODE)                                        \
    do {                                                              \
        if (dw == 4) KB_SCAN(R, CH, (R <= 4 ? 4 : 2), MODE);          \
        else if (dw == 2) KB_SCAN(R, CH, 2, MODE);                    \
        else KB_SCAN(R, CH, 1, MODE);                                 \
    } while (0)
#define KB_SCAN_W(R, CH)                                              \
    do {                                                              \
        switch (mode) {                                               \
            case SCAN_REMOVAL: KB_SCAN_M(R, CH, SCAN_REMOVAL); break; \
            case SCAN_WRITE: KB_SCAN_M(R, CH, SCAN_WRITE); break;     \
            case SCAN_FIXED: KB_SCAN_M(R, CH, SCAN_FIXED); break;     \
            default: KB_SCAN_M(R, CH, SCAN_GATE); break;              \
        }                                                             \
    } while (0)
    if (need <= 1) KB_SCAN_W(1, 16);
    else if (need <= 2) KB_SCAN_W(2, 16);
    else if (need <= 4) KB_SCAN_W(4, 8);
    else {                                                  // eight rows a lane: at most two columns a warp fit the registers
        if (dw == 4) {
            dw = 2;
            grid.z = (e + SC * dw - 1) / (SC * dw);
        }
        KB_SCAN_W(SCAN_R, 4);
    }
#undef KB_SCAN_W
#undef KB_SCAN_M
#undef KB_SCAN
    return check_launch("decay_scan");
}

static int scan_common_checks(const char* what, const void* src, int splits, long long split_stride, int row_width, int rows, int entries,
                              int heads, int d, int e, const float* state, int n_slots, const void* a, const void* b, const void* c) {
    KB_REQUIRE(entries >= 0 && rows >= 0 && heads > 0 && d > 0 && e > 0, "%s: entries %d, rows %d, heads %d, sizes %d / %d", what, entries, rows, heads, d, e);
    KB_REQUIRE(d <= 32 * SCAN_R, "%s: a key size of %d is more than the kernel's %d", what, d, 32 * SCAN_R);
    KB_REQUIRE(splits >= 1 && (splits == 1 || split_stride >= (long long)rows * row_width), "%s: %d slices %lld apart", what, splits, split_stride);
    KB_REQUIRE(src && state && n_slots >= 1 && a && b && c, "%s: state, ranges or slots are missing", what);
    KB_REQUIRE(entries <= 65535, "%s: too many requests for one launch", what);
    return 0;
}

// The generalized delta rule's read-out [rows, heads, d] over the rows of a step.
extern "C" int kb_gdelta_scan(float* out, float* scratch, const void* src, int in_dt, int splits, long long split_stride, int row_width,
                              int r_off, int k_off, int v_off, int a_off, int w1_off, int lora, const float* w2, const float* w0,
                              const float* a_bias, float decay_scale, float unit_eps, float* state, int n_slots,
                              const int* entry_start, const int* entry_end, const int* slots, int entries, int rows, int heads, int d,
                              void* stream) {
    if (int err = scan_common_checks("gdelta", src, splits, split_stride, row_width, rows, entries, heads, d, d, state, n_slots, entry_start, entry_end, slots))
        return err;
    const long long n = (long long)heads * d;
    KB_REQUIRE(row_width > 0 && lora > 0 && r_off >= 0 && r_off + n <= row_width && k_off >= 0 && k_off + n <= row_width && v_off >= 0 &&
                   v_off + n <= row_width && a_off >= 0 && a_off + n <= row_width && w1_off >= 0 && w1_off + lora <= row_width,
               "gdelta: columns r %d, k %d, v %d, a %d, w1 %d (+%d) do not fit a row of %d", r_off, k_off, v_off, a_off, w1_off, lora, row_width);
    KB_REQUIRE(out && scratch && w2 && w0 && a_bias, "gdelta: weights or scratch are missing");
    const bool few = rows <= DEPENDENT_ROWS;
    const size_t smem = (size_t)(few ? 1 : 8) * lora * sizeof(float);
    KB_REQUIRE(smem <= 200 * 1024, "gdelta: a decay net of %d hidden values does not fit the shared memory of a block", lora);
    if (entries == 0 || rows == 0) return 0;
    GDeltaParams g;
    g.row_width = row_width; g.r_off = r_off; g.k_off = k_off; g.v_off = v_off; g.a_off = a_off; g.w1_off = w1_off; g.lora = lora;
    g.w2 = w2; g.w0 = w0; g.a_bias = a_bias; g.decay_scale = decay_scale; g.unit_eps = unit_eps; g.heads = heads; g.d = d;
    ScanInputs in;
    in.vec = scratch;
    in.val = in.vec + (size_t)rows * heads * 5 * d;
    in.scal = in.val + (size_t)rows * n;
    in.nv = 5;
    cudaStream_t s = (cudaStream_t)stream;
#define KB_GD(TS)                                                                                                          \
    do {                                                                                                                   \
        if (few) {                                                                                                         \
            if (smem > 48 * 1024) cudaFuncSetAttribute(gdelta_prep_kernel<TS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            gdelta_prep_kernel<TS, 1><<<rows, 1024, smem, s>>>(Src<TS>{(const TS*)src, splits, (size_t)split_stride}, g, in, rows); /* few rows: a channel or two a thread */ \
        } else {                                                                                                           \
            if (smem > 48 * 1024) cudaFuncSetAttribute(gdelta_prep_kernel<TS, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            gdelta_prep_kernel<TS, 8><<<(rows + 7) / 8, 512, smem, s>>>(Src<TS>{(const TS*)src, splits, (size_t)split_stride}, g, in, rows); \
        }                                                                                                                  \
    } while (0)
    if (in_dt == KB_DT_F32) KB_GD(float);
    else if (in_dt == KB_DT_BF16) KB_GD(bf16);
    else return fail("gdelta: dtype code %d is not known", in_dt);
#undef KB_GD
    if (int err = check_launch("gdelta prep")) return err;
    return run_decay_scan(out, in, state, n_slots, entry_start, entry_end, slots, entries, heads, d, d, SCAN_REMOVAL, nullptr, s);
}

// The read-out [rows, heads, e] of the memory behind a forget gate with a lower bound.
extern "C" int kb_gate_scan(float* out, float* scratch, const void* src, int in_dt, int splits, long long split_stride, int row_width,
                            int q_off, int f_off, int v_off, const float* f_bias, const float* lower, float* state, int n_slots,
                            const int* entry_start, const int* entry_end, const int* slots, int entries, int rows, int heads, int d,
                            int e, void* stream) {
    if (int err = scan_common_checks("gate_scan", src, splits, split_stride, row_width, rows, entries, heads, d, e, state, n_slots, entry_start, entry_end, slots))
        return err;
    const long long nq = (long long)heads * d, nv = (long long)heads * e;
    KB_REQUIRE(row_width > 0 && q_off >= 0 && q_off + nq <= row_width && f_off >= 0 && f_off + nq <= row_width && v_off >= 0 && v_off + nv <= row_width,
               "gate_scan: columns q %d, f %d, v %d do not fit a row of %d", q_off, f_off, v_off, row_width);
    KB_REQUIRE(out && scratch && f_bias && lower, "gate_scan: weights or scratch are missing");
    if (entries == 0 || rows == 0) return 0;
    GateParams g;
    g.row_width = row_width; g.q_off = q_off; g.f_off = f_off; g.v_off = v_off; g.f_bias = f_bias; g.lower = lower;
    g.heads = heads; g.d = d; g.e = e;
    ScanInputs in;
    in.vec = scratch;
    in.val = in.vec + (size_t)rows * heads * 3 * d;
    in.scal = in.val + (size_t)rows * nv;
    in.nv = 3;
    cudaStream_t s = (cudaStream_t)stream;
    if (in_dt == KB_DT_F32) gate_prep_kernel<float><<<rows, 256, 0, s>>>(Src<float>{(const float*)src, splits, (size_t)split_stride}, g, in);
    else if (in_dt == KB_DT_BF16) gate_prep_kernel<bf16><<<rows, 256, 0, s>>>(Src<bf16>{(const bf16*)src, splits, (size_t)split_stride}, g, in);
    else return fail("gate_scan: dtype code %d is not known", in_dt);
    if (int err = check_launch("gate_scan prep")) return err;
    return run_decay_scan(out, in, state, n_slots, entry_start, entry_end, slots, entries, heads, d, e, SCAN_GATE, nullptr, s);
}

// The read-out [rows, heads, e] of the gated delta rule with a decay a key channel; `history` [slots, (taps - 1) channels]
// holds the convolutions' last inputs and `memory` [slots, heads, e, d] the memories.
extern "C" int kb_cdelta_scan(float* out, float* scratch, const void* src, int in_dt, int splits, long long split_stride, int row_width,
                              int q_off, int k_off, int v_off, int b_off, int a1_off, int rank, const float* a2, const float* dt_bias,
                              const float* a_log, const float* conv, float* history, float* memory, int n_slots, const int* row_entry,
                              const int* entry_start, const int* entry_end, const int* slots, int entries, int rows, int heads,
                              int kv_heads, int d, int e, int taps, float q_scale, float unit_eps, void* stream) {
    if (int err = scan_common_checks("cdelta", src, splits, split_stride, row_width, rows, entries, heads, d, e, memory, n_slots, entry_start, entry_end, slots))
        return err;
    KB_REQUIRE(kv_heads > 0 && heads % kv_heads == 0, "cdelta: %d heads over %d", heads, kv_heads);
    KB_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "cdelta: a convolution of %d taps (1 to %d)", taps, CONV_MAX_TAPS);
    const long long nq = (long long)kv_heads * d, nv = (long long)heads * e, n = (long long)heads * d;
    KB_REQUIRE(row_width > 0 && q_off >= 0 && k_off == q_off + nq && v_off == k_off + nq && v_off + nv <= row_width,
               "cdelta: columns q %d, k %d, v %d must follow one another in a row of %d", q_off, k_off, v_off, row_width);
    KB_REQUIRE(b_off >= 0 && b_off + heads <= row_width && rank > 0 && a1_off >= 0 && a1_off + rank <= row_width,
               "cdelta: columns b %d, a1 %d (+%d) do not fit a row of %d", b_off, a1_off, rank, row_width);
    KB_REQUIRE(out && scratch && a2 && dt_bias && a_log && conv && history && row_entry, "cdelta: weights, history or scratch are missing");
    const bool few = rows <= DEPENDENT_ROWS;
    const size_t smem = (size_t)(few ? 1 : 8) * rank * sizeof(float);
    KB_REQUIRE(smem <= 200 * 1024, "cdelta: a decay of rank %d does not fit the shared memory of a block", rank);
    if (entries == 0 || rows == 0) return 0;
    CDeltaParams g;
    g.row_width = row_width; g.q_off = q_off; g.k_off = k_off; g.v_off = v_off; g.b_off = b_off; g.a1_off = a1_off; g.rank = rank;
    g.a2 = a2; g.dt_bias = dt_bias; g.a_log = a_log; g.conv = conv; g.state = history; g.row_entry = row_entry; g.entry_start = entry_start;
    g.slots = slots; g.n_slots = n_slots; g.entries = entries; g.heads = heads; g.kv_heads = kv_heads; g.d = d; g.e = e; g.taps = taps;
    g.q_scale = q_scale; g.unit_eps = unit_eps;
    ScanInputs in;
    in.vec = scratch;
    in.val = in.vec + (size_t)rows * n * 4;
    in.scal = in.val + (size_t)rows * nv;
    in.nv = 4;
    ConvParams c = {};
    c.row_width = row_width; c.q_off = q_off; c.nq = (int)(2 * nq + nv); c.conv = conv; c.state = history; c.row_entry = row_entry;
    c.entry_start = entry_start; c.entry_end = entry_end; c.slots = slots; c.n_slots = n_slots; c.entries = entries; c.rows = rows; c.taps = taps;
    cudaStream_t s = (cudaStream_t)stream;
#define KB_CD(TS)                                                                                                          \
    do {                                                                                                                   \
        const Src<TS> x{(const TS*)src, splits, (size_t)split_stride};                                                      \
        if (few) {                                                                                                         \
            if (smem > 48 * 1024) cudaFuncSetAttribute(cdelta_prep_kernel<TS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            cdelta_prep_kernel<TS, 1><<<rows, 1024, smem, s>>>(x, g, in, rows);                                            \
        } else {                                                                                                           \
            if (smem > 48 * 1024) cudaFuncSetAttribute(cdelta_prep_kernel<TS, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            cdelta_prep_kernel<TS, 8><<<(rows + 7) / 8, 512, smem, s>>>(x, g, in, rows);                                   \
        }                                                                                                                  \
        if (int err = check_launch("cdelta prep")) return err;                                                             \
        if (taps > 1) conv_history_kernel<TS><<<dim3((unsigned)((c.nq + 127) / 128), entries), 128, 0, s>>>(x, c);          \
    } while (0)
    if (in_dt == KB_DT_F32) KB_CD(float);
    else if (in_dt == KB_DT_BF16) KB_CD(bf16);
    else return fail("cdelta: dtype code %d is not known", in_dt);
#undef KB_CD
    if (int err = check_launch("cdelta history")) return err;
    return run_decay_scan(out, in, memory, n_slots, entry_start, entry_end, slots, entries, heads, d, e, SCAN_WRITE, nullptr, s);
}

// From how many rows of a request on the memory is walked by chunks (retention.cu) instead of row by row; 0: never (for tests and measurements).
static int g_retention_chunk_rows = 128;
extern "C" void kb_retention_chunk_rows(int rows) { g_retention_chunk_rows = rows >= 0 ? rows : 128; }
static bool by_chunks(int longest) { return g_retention_chunk_rows > 0 && longest >= g_retention_chunk_rows; }

// Floats of scratch kb_retention_scan takes for a step of `rows` rows whose longest portion has `longest`.
extern "C" long long kb_retention_scratch_floats(int rows, int entries, int longest, int heads, int d, int e) {
    return kb_decay_scan_scratch_floats(rows, heads, d, e, SCAN_FIXED) + (by_chunks(longest) ? retention_chunk_floats(rows, entries, heads, d, e) : 0);
}

// The read-out [rows, heads, e] of a matrix memory with a fixed decay a head behind rotated queries and keys. `longest`: the
// most rows a request brings (every request's rows lie behind the earlier requests').
extern "C" int kb_retention_scan(float* out, float* scratch, const void* src, int in_dt, int splits, long long split_stride, int row_width,
                                 int q_off, int k_off, int v_off, const float* decay, const float* cos_sin, int rotary, float k_scale, int act,
                                 float* state, int n_slots, const int* entry_start, const int* entry_end, const int* slots, int entries,
                                 int rows, int longest, int heads, int d, int e, void* stream) {
    if (int err = scan_common_checks("retention", src, splits, split_stride, row_width, rows, entries, heads, d, e, state, n_slots, entry_start, entry_end, slots))
        return err;
    const long long nq = (long long)heads * d, nv = (long long)heads * e;
    KB_REQUIRE(row_width > 0 && q_off >= 0 && q_off + nq <= row_width && k_off >= 0 && k_off + nq <= row_width && v_off >= 0 && v_off + nv <= row_width,
               "retention: columns q %d, k %d, v %d do not fit a row of %d", q_off, k_off, v_off, row_width);
    KB_REQUIRE(rotary >= 0 && rotary <= d && rotary % 2 == 0 && (rotary == 0 || cos_sin), "retention: a rotation of %d components of %d", rotary, d);
    KB_REQUIRE(out && scratch && decay, "retention: decays or scratch are missing");
    KB_REQUIRE(act == 0 || act == 1, "retention: activation code %d is not known (0 none, 1 silu)", act);
    if (entries == 0 || rows == 0) return 0;
    RetentionParams g;
    g.row_width = row_width; g.q_off = q_off; g.k_off = k_off; g.v_off = v_off; g.decay = decay; g.cos_sin = (const float2*)cos_sin;
    g.rotary = rotary; g.heads = heads; g.d = d; g.e = e; g.k_scale = k_scale; g.act = act;
    ScanInputs in;
    in.vec = scratch;
    in.val = in.vec + (size_t)rows * nq * 2;
    in.scal = in.val + (size_t)rows * nv;
    in.nv = 2;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = rows <= DEPENDENT_ROWS ? 1024 : 256;      // few rows: latency counts
    if (in_dt == KB_DT_F32) retention_prep_kernel<float><<<rows, threads, 0, s>>>(Src<float>{(const float*)src, splits, (size_t)split_stride}, g, in);
    else if (in_dt == KB_DT_BF16) retention_prep_kernel<bf16><<<rows, threads, 0, s>>>(Src<bf16>{(const bf16*)src, splits, (size_t)split_stride}, g, in);
    else return fail("retention: dtype code %d is not known", in_dt);
    if (int err = check_launch("retention prep")) return err;
    if (by_chunks(longest))
        return run_retention_chunks(out, in.vec, in.val, in.scal, decay, in.scal + (size_t)rows * heads * 2, state, n_slots, entry_start, entry_end,
                                    slots, entries, longest, heads, d, e, s);
    return run_decay_scan(out, in, state, n_slots, entry_start, entry_end, slots, entries, heads, d, e, SCAN_FIXED, decay, s);
}

// out [rows, channels] = the convolution of columns off.. (bias added first, `after` behind the filter), in 32-bit; `state`
// [slots, (taps - 1) channels] holds every request's last inputs.
extern "C" int kb_conv_rows(float* out, const void* src, int in_dt, int splits, long long split_stride, int row_width, int off,
                            int channels, const float* bias, const float* conv, const float* after, float* state, int n_slots,
                            const int* row_entry, const int* entry_start, const int* entry_end, const int* slots, int entries, int rows,
                            int taps, void* stream) {
    KB_REQUIRE(rows >= 0 && entries >= 0 && channels > 0, "conv_rows: rows %d, requests %d, channels %d", rows, entries, channels);
    KB_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "conv_rows: a convolution of %d taps (1 to %d)", taps, CONV_MAX_TAPS);
    KB_REQUIRE(row_width > 0 && off >= 0 && off + (long long)channels <= row_width, "conv_rows: columns %d.. do not fit a row of %d", off, row_width);
    KB_REQUIRE(splits >= 1 && (splits == 1 || split_stride >= (long long)rows * row_width), "conv_rows: %d slices %lld apart", splits, split_stride);
    KB_REQUIRE(out && src && conv && state && n_slots >= 1 && row_entry && entry_start && entry_end && slots, "conv_rows: a tensor is missing");
    KB_REQUIRE(entries <= 65535, "conv_rows: too many requests for one launch");
    if (rows == 0 || entries == 0) return 0;
    ConvParams p = {};
    p.row_width = row_width; p.q_off = off; p.nq = channels; p.bias = bias; p.conv = conv; p.after = after; p.state = state;
    p.row_entry = row_entry; p.entry_start = entry_start; p.entry_end = entry_end; p.slots = slots; p.n_slots = n_slots; p.entries = entries;
    p.rows = rows; p.taps = taps; p.q_stride = channels;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = channels >= 2048 ? 512 : 256;
#define KB_CR(TS)                                                                                                          \
    do {                                                                                                                   \
        const Src<TS> x{(const TS*)src, splits, (size_t)split_stride};                                                      \
        conv_append_kernel<TS, float><<<rows, threads, 0, s>>>(x, p, out, (float*)nullptr);                                 \
        if (int err = check_launch("conv_rows")) return err;                                                               \
        if (taps > 1) conv_history_kernel<TS><<<dim3((unsigned)((channels + 127) / 128), entries), 128, 0, s>>>(x, p);      \
    } while (0)
    if (in_dt == KB_DT_F32) KB_CR(float);
    else if (in_dt == KB_DT_BF16) KB_CR(bf16);
    else return fail("conv_rows: dtype code %d is not known", in_dt);
#undef KB_CR
    return check_launch("conv_rows history");
}

extern "C" int kb_weighted_sum2(float* out, const void* a, int a_dt, int a_splits, long long a_stride, const float* va, const void* b,
                                int b_dt, int b_splits, long long b_stride, const float* vb, const float* vc, long long rows, int width,
                                void* stream) {
    KB_REQUIRE(rows >= 0 && width > 0 && out && a && va, "weighted_sum2: rows %lld, width %d", rows, width);
    KB_REQUIRE(b == nullptr || vb != nullptr, "weighted_sum2: a second branch without its weights");
    KB_REQUIRE(a_splits >= 1 && b_splits >= 1, "weighted_sum2: %d / %d slices", a_splits, b_splits);
    if (rows == 0) return 0;
    const long long total = rows * width;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    cudaStream_t s = (cudaStream_t)stream;
    const bool has_b = b != nullptr;
    const void* bp = has_b ? b : a;
    if (!has_b) { b_dt = a_dt; b_splits = 1; b_stride = 0; }
#define KB_WS(TA, TB)                                                                                                       \
    weighted_sum2_kernel<TA, TB><<<blocks, 256, 0, s>>>(out, Src<TA>{(const TA*)a, a_splits, (size_t)a_stride}, va,           \
                                                       Src<TB>{(const TB*)bp, b_splits, (size_t)b_stride}, vb, vc, total, width, has_b)
    if (a_dt == KB_DT_F32 && b_dt == KB_DT_F32) KB_WS(float, float);
    else if (a_dt == KB_DT_F32 && b_dt == KB_DT_BF16) KB_WS(float, bf16);
    else if (a_dt == KB_DT_BF16 && b_dt == KB_DT_F32) KB_WS(bf16, float);
    else if (a_dt == KB_DT_BF16 && b_dt == KB_DT_BF16) KB_WS(bf16, bf16);
    else return fail("weighted_sum2: dtype codes %d, %d are not known", a_dt, b_dt);
#undef KB_WS
    return check_launch("weighted_sum2");
}
