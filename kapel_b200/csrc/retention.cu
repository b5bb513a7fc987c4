// A matrix memory with a fixed decay a head, by chunks of rows: the same steps as the decay scan's SCAN_FIXED
// (S <- w S + k v^T, o = S^T q) summed in another order, for the long portions of prompts.
//
// With the memory S_0 before a chunk of n <= 64 rows, its row t reads
//     o_t = w^t (w q_t)^T S_0 + sum_{s < t} w^(t-s-1) (w q_t . k_s) v_s + (q_t . k_t) v_t
// and the memory behind it is w^n S_0 + sum_s w^(n-1-s) k_s v_s^T. Three kernels: `retention_sums` makes every
// chunk's own sum (all chunks side by side), `retention_states` walks a request's chunks and puts in each sum's
// place the memory before that chunk (the one part that is a chain: one multiply-add a chunk), and
// `retention_rows` makes the rows' read-outs (all chunks side by side again). Chunks are counted from a
// request's first row of the step. Everything is 32-bit multiply-adds; powers of w come from powf (w = 0 is
// allowed: no division by w anywhere).
#include "common.cuh"

namespace kb {

constexpr int RT_C = 64;               // rows a chunk
constexpr int RT_K = 32;               // inner steps staged at a time
constexpr int RT_THREADS = 256;

struct RetentionChunks {
    const float* vec;           // [rows, heads, 2, d]: w q, then k
    const float* val;           // [rows, heads, e]
    const float* scal;          // [rows, heads, 2]: the second is k.q
    const float* decay;         // [heads]
    float* sums;                // [chunks, heads, d, e]
    float* state;               // [slots, heads, e, d]
    const int* entry_start;
    const int* entry_end;
    const int* slots;
    int n_slots, heads, d, e;
    float* out;                 // [rows, heads, e]
};

// Where a request's first chunk lies: requests' rows follow one another, so ceil(n / 64) chunks fit between two of these.
__device__ __forceinline__ int first_chunk(int entry, int r0) { return r0 / RT_C + entry; }

// sums[chunk, head, i, c] = sum_s w^(n-1-s) k_s[i] v_s[c]. One block = 64 key channels x 128 value components of a chunk; a
// thread 8 x 4 of them.
__global__ void __launch_bounds__(RT_THREADS)
retention_sums_kernel(const RetentionChunks p, int etiles) {
    __shared__ __align__(16) float sk[RT_K][64], sv[RT_K][128];
    __shared__ float pw[RT_C];
    const int entry = blockIdx.z, head = blockIdx.y;
    const int dtiles = (p.d + 63) / 64;
    const int chunk = blockIdx.x / (dtiles * etiles), tile = blockIdx.x % (dtiles * etiles);
    const int i0 = tile / etiles * 64, c0 = tile % etiles * 128;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    const int first = r0 + chunk * RT_C, n = min(RT_C, r1 - first);
    const int slot = p.slots[entry];
    if (n <= 0 || slot <= 0 || slot >= p.n_slots) return;
    const int tid = threadIdx.x, ti = tid / 32, tc = tid % 32;
    const float w = p.decay[head];
    if (tid < RT_C) pw[tid] = powf(w, (float)tid);
    __syncthreads();
    float acc[8][4] = {};
    for (int s0 = 0; s0 < n; s0 += RT_K) {
        for (int idx = tid; idx < RT_K * 64; idx += RT_THREADS) {
            const int s = idx / 64, i = idx % 64;
            sk[s][i] = (s0 + s < n && i0 + i < p.d) ? p.vec[((size_t)(first + s0 + s) * p.heads + head) * 2 * p.d + p.d + i0 + i] : 0.f;
        }
        for (int idx = tid; idx < RT_K * 128; idx += RT_THREADS) {
            const int s = idx / 128, c = idx % 128;
            sv[s][c] = (s0 + s < n && c0 + c < p.e) ? pw[n - 1 - s0 - s] * p.val[((size_t)(first + s0 + s) * p.heads + head) * p.e + c0 + c] : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int s = 0; s < RT_K; ++s) {
            const float4 ka = *reinterpret_cast<const float4*>(&sk[s][ti * 8]), kb4 = *reinterpret_cast<const float4*>(&sk[s][ti * 8 + 4]);
            const float4 v4 = *reinterpret_cast<const float4*>(&sv[s][tc * 4]);
            const float k[8] = {ka.x, ka.y, ka.z, ka.w, kb4.x, kb4.y, kb4.z, kb4.w};
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                acc[x][0] = fmaf(k[x], v4.x, acc[x][0]);
                acc[x][1] = fmaf(k[x], v4.y, acc[x][1]);
                acc[x][2] = fmaf(k[x], v4.z, acc[x][2]);
                acc[x][3] = fmaf(k[x], v4.w, acc[x][3]);
            }
        }
        __syncthreads();
    }
    float* dst = p.sums + ((size_t)(first_chunk(entry, r0) + chunk) * p.heads + head) * p.d * p.e;
#pragma unroll
    for (int x = 0; x < 8; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const int i = i0 + ti * 8 + x, c = c0 + tc * 4 + y;
            if (i < p.d && c < p.e) dst[(size_t)i * p.e + c] = acc[x][y];
        }
}

// Every chunk's sum becomes the memory before that chunk; the last one behind goes to the request's slot. A thread a value of
// the memory; the sums of eight chunks are asked for before the chain walks them.
__global__ void retention_states_kernel(const RetentionChunks p) {
    const int entry = blockIdx.z, head = blockIdx.y;
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    const int size = p.d * p.e;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    const int slot = p.slots[entry];
    if (idx >= size || r1 <= r0 || slot <= 0 || slot >= p.n_slots) return;
    const int i = idx / p.e, c = idx - i * p.e;
    float* st = p.state + ((size_t)slot * p.heads + head) * size + (size_t)c * p.d + i;      // a column of the memory lies together there
    const size_t stride = (size_t)p.heads * size;
    float* at = p.sums + (size_t)first_chunk(entry, r0) * stride + (size_t)head * size + idx;
    const float w = p.decay[head];
    const float whole = powf(w, (float)RT_C);
    const int chunks = (r1 - r0 + RT_C - 1) / RT_C;
    float S = *st;
    for (int ch = 0; ch < chunks; ch += 8) {
        float x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = ch + j < chunks ? at[(size_t)(ch + j) * stride] : 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (ch + j < chunks) {
                at[(size_t)(ch + j) * stride] = S;
                const int n = min(RT_C, r1 - r0 - (ch + j) * RT_C);
                S = fmaf(n == RT_C ? whole : powf(w, (float)n), S, x[j]);
            }
    }
    *st = S;
}

// The read-outs of a chunk's rows for 128 value components: a thread 8 rows x 4 components, and 8 rows x 2 of the rows' scores
// against one another on the way.
__global__ void __launch_bounds__(RT_THREADS)
retention_rows_kernel(const RetentionChunks p) {
    __shared__ __align__(16) float sqk[2 * RT_K][RT_C + 4], sb[RT_K][128];
    auto sq = sqk, sk = sqk + RT_K;
    auto ss = sqk;                                              // [s][t]: what row s gives to row t, once queries and keys are done with
    static_assert(RT_C == 2 * RT_K, "the scores take the place of queries and keys");
    __shared__ float pw[RT_C + 1];
    const int entry = blockIdx.z, head = blockIdx.y;
    const int etiles = (p.e + 127) / 128;
    const int chunk = blockIdx.x / etiles, c0 = blockIdx.x % etiles * 128;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    const int first = r0 + chunk * RT_C, n = min(RT_C, r1 - first);
    if (n <= 0) return;
    const int tid = threadIdx.x, tr = tid / 32, tc = tid % 32;
    const int slot = p.slots[entry];
    const int d = p.d, e = p.e;
    if (slot <= 0 || slot >= p.n_slots) {                       // rows of no request: zeros
        for (int idx = tid; idx < n * 128; idx += RT_THREADS) {
            const int t = idx / 128, c = c0 + idx % 128;
            if (c < e) p.out[((size_t)(first + t) * p.heads + head) * e + c] = 0.f;
        }
        return;
    }
    const float w = p.decay[head];
    if (tid <= RT_C) pw[tid] = powf(w, (float)tid);
    const float* before = p.sums + ((size_t)(first_chunk(entry, r0) + chunk) * p.heads + head) * d * e;
    float o[8][4] = {}, sc[8][2] = {};
    for (int k0 = 0; k0 < d; k0 += RT_K) {
        for (int idx = tid; idx < RT_C * RT_K; idx += RT_THREADS) {
            const int t = idx / RT_K, k = idx % RT_K;
            const bool in = t < n && k0 + k < d;
            const float* row = p.vec + ((size_t)(first + t) * p.heads + head) * 2 * d + k0 + k;
            sq[k][t] = in ? row[0] : 0.f;
            sk[k][t] = in ? row[d] : 0.f;
        }
        for (int idx = tid; idx < RT_K * 128; idx += RT_THREADS) {
            const int k = idx / 128, c = idx % 128;
            sb[k][c] = (k0 + k < d && c0 + c < e) ? before[(size_t)(k0 + k) * e + c0 + c] : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int k = 0; k < RT_K; ++k) {
            const float4 qa = *reinterpret_cast<const float4*>(&sq[k][tr * 8]), qb = *reinterpret_cast<const float4*>(&sq[k][tr * 8 + 4]);
            const float2 k2 = *reinterpret_cast<const float2*>(&sk[k][tc * 2]);
            const float4 b4 = *reinterpret_cast<const float4*>(&sb[k][tc * 4]);
            const float q[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                o[x][0] = fmaf(q[x], b4.x, o[x][0]);
                o[x][1] = fmaf(q[x], b4.y, o[x][1]);
                o[x][2] = fmaf(q[x], b4.z, o[x][2]);
                o[x][3] = fmaf(q[x], b4.w, o[x][3]);
                sc[x][0] = fmaf(q[x], k2.x, sc[x][0]);
                sc[x][1] = fmaf(q[x], k2.y, sc[x][1]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < 8; ++x) {
        const int t = tr * 8 + x;
#pragma unroll
        for (int y = 0; y < 2; ++y) {
            const int s = tc * 2 + y;
            float g = 0.f;
            if (s < t && t < n) g = pw[t - s - 1] * sc[x][y];
            else if (s == t && t < n) g = p.scal[((size_t)(first + t) * p.heads + head) * 2 + 1];
            ss[s][t] = g;
        }
#pragma unroll
        for (int y = 0; y < 4; ++y) o[x][y] *= pw[t];
    }
    for (int s0 = 0; s0 < n; s0 += RT_K) {
        for (int idx = tid; idx < RT_K * 128; idx += RT_THREADS) {
            const int s = idx / 128, c = idx % 128;
            sb[s][c] = (s0 + s < n && c0 + c < e) ? p.val[((size_t)(first + s0 + s) * p.heads + head) * e + c0 + c] : 0.f;
        }
        __syncthreads();
        if (tr * 8 + 7 >= s0) {                                 // rows before these sources take nothing from them
#pragma unroll 4
            for (int s = 0; s < RT_K; ++s) {
                const float4 ga = *reinterpret_cast<const float4*>(&ss[s0 + s][tr * 8]), gb = *reinterpret_cast<const float4*>(&ss[s0 + s][tr * 8 + 4]);
                const float4 v4 = *reinterpret_cast<const float4*>(&sb[s][tc * 4]);
                const float g[8] = {ga.x, ga.y, ga.z, ga.w, gb.x, gb.y, gb.z, gb.w};
#pragma unroll
                for (int x = 0; x < 8; ++x) {
                    o[x][0] = fmaf(g[x], v4.x, o[x][0]);
                    o[x][1] = fmaf(g[x], v4.y, o[x][1]);
                    o[x][2] = fmaf(g[x], v4.z, o[x][2]);
                    o[x][3] = fmaf(g[x], v4.w, o[x][3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < 8; ++x) {
        const int t = tr * 8 + x;
#pragma unroll
        for (int y = 0; y < 4; ++y) {
            const int c = c0 + tc * 4 + y;
            if (t < n && c < e) p.out[((size_t)(first + t) * p.heads + head) * e + c] = o[x][y];
        }
    }
}

long long retention_chunk_floats(int rows, int entries, int heads, int d, int e) {
    return ((long long)rows / RT_C + entries) * heads * d * e;
}

// vec, val, scal: the decay scan's inputs in its SCAN_FIXED order. `longest`: the most rows a request brings.
int run_retention_chunks(float* out, const float* vec, const float* val, const float* scal, const float* decay, float* sums, float* state,
                         int n_slots, const int* entry_start, const int* entry_end, const int* slots, int entries, int longest, int heads,
                         int d, int e, cudaStream_t s) {
    RetentionChunks p;
    p.vec = vec; p.val = val; p.scal = scal; p.decay = decay; p.sums = sums; p.state = state; p.entry_start = entry_start;
    p.entry_end = entry_end; p.slots = slots; p.n_slots = n_slots; p.heads = heads; p.d = d; p.e = e; p.out = out;
    const long long chunks = (longest + RT_C - 1) / RT_C;
    const int dtiles = (d + 63) / 64, etiles = (e + 127) / 128;
    KB_REQUIRE(heads <= 65535 && entries <= 65535 && chunks * dtiles * etiles <= 0x7fffffffll, "retention: too many heads, requests or rows for one launch");
    retention_sums_kernel<<<dim3((unsigned)(chunks * dtiles * etiles), heads, entries), RT_THREADS, 0, s>>>(p, etiles);
    if (int err = check_launch("retention sums")) return err;
    retention_states_kernel<<<dim3((unsigned)((d * e + 127) / 128), heads, entries), 128, 0, s>>>(p);
    if (int err = check_launch("retention states")) return err;
    retention_rows_kernel<<<dim3((unsigned)(chunks * etiles), heads, entries), RT_THREADS, 0, s>>>(p);
    return check_launch("retention rows");
}

}  // namespace kb
