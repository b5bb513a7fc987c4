// Several residual streams a row (hyper-connections): x [rows, S, width], float32, one row's streams side by side.
//
//  stream_step   what happens between two sublayers, one kernel a row. With a branch y (the sublayer's result, times a
//                weight a channel): x_t <- sum_s mix[s, t] x_s + out[t] y, all streams at once from the old ones. Then, where
//                a sublayer follows, u = sum_s in[s] x_s and h = norm(u): a layer norm (or an RMS norm) with a weight and
//                perhaps a bias. Without a branch only the second half runs (the first sublayer of a model).
//                The branch may be a tensor, the split-K partial sums of a product, or the sum of two such
//                branches that are each RMS-normed first: y = rms(a) wa + rms(b) wb.
//  stream_sum    out[i] = sum_s x_s[rows[i]]: the rows whose logits are wanted, their streams added up.
//
// Everything is 32-bit; only the branch and h may be bfloat16. The order of the additions depends on the width and the
// block size only, never on the number of rows.
#include <algorithm>
#include "common.cuh"

namespace kb {

typedef __nv_bfloat16 bf16;

constexpr int STREAMS_MAX = 16;
constexpr int STREAM_THREADS = 512;

// V neighbouring values (4: 16 bytes of float32) of a branch, its slices added in slice order, eight in flight.
template <int V, typename T> struct Pack;
template <> struct Pack<4, float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Pack<4, bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(t.x << 16); v[1] = __uint_as_float(t.x & 0xffff0000u);
        v[2] = __uint_as_float(t.y << 16); v[3] = __uint_as_float(t.y & 0xffff0000u);
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
};
template <typename T> struct Pack<1, T> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = Elem<T>::load(p); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { Elem<T>::store(p, v[0]); }
};

template <int V, typename T, bool MANY>
__device__ __forceinline__ void branch_at(const Src<T>& src, size_t i, float (&v)[V]) {
    Pack<V, T>::load(src.p + i, v);
    if constexpr (!MANY) return;
    for (int s = 1; s < src.splits; s += 8) {
        float t[8][V];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (s + j < src.splits) {
                Pack<V, T>::load(src.p + (size_t)(s + j) * src.stride + i, t[j]);
            } else {
#pragma unroll
                for (int e = 0; e < V; ++e) t[j][e] = 0.f;
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] += t[j][e];
    }
}

struct StreamParams {
    float* x;                   // [rows, S, width]
    int streams, width;
    // the write: null `mix` for none
    const float* mix;           // [S, S], from and to
    const float* out;           // [S]
    const float* scale;         // [width] or null: the branch's weight a channel
    const float* norm_a;        // [width] or null: the branch is rms(a) norm_a + rms(b) norm_b
    const float* norm_b;
    float eps_ab;
    // the read: null `in` for none
    const float* in;            // [S]
    const float* weight;        // [width]
    const float* bias;          // [width] or null
    float eps, offset;
    int center;
};

// Two sums over the block at once; `scratch` holds 64 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) { scratch[warp] = a; scratch[32 + warp] = b; }
    __syncthreads();
    const int n = (blockDim.x + 31) >> 5;
    return make_float2(warp_sum(lane < n ? scratch[lane] : 0.f), warp_sum(lane < n ? scratch[32 + lane] : 0.f));
}

// SM: room for streams; MANY: branches of more than one slice (a decoding step, as a rule); a thread owns V neighbouring channels of every stream at a time. Shared memory: u [width], and with two
// normed branches their rows [2 width].
template <typename TB, typename TH, int V, int SM, bool MANY>
__global__ void __launch_bounds__(STREAM_THREADS, SM <= 4 && !MANY ? 2 : 1)
stream_step_kernel(const StreamParams p, const Src<TB> a, const Src<TB> b, TH* __restrict__ h) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[64];
    const int S = p.streams, width = p.width, chunks = width / V;
    const size_t base = (size_t)blockIdx.x * width;
    float* x = p.x + base * S;
    const bool write = p.mix != nullptr, read = p.in != nullptr;
    // A handful of numbers that every thread needs, constants of the layer: what goes to stream t lies together.
    __shared__ __align__(16) float held[SM * SM];
    __shared__ float out[SM], in[SM];
    for (int i = threadIdx.x; i < SM * SM; i += blockDim.x) {
        const int t = i / SM, f = i % SM;
        held[i] = write && f < S && t < S ? p.mix[f * S + t] : 0.f;
        if (f == 0) {
            out[t] = write && t < S ? p.out[t] : 0.f;
            in[t] = read && t < S ? p.in[t] : 0.f;
        }
    }
    __syncthreads();
    dependent_wait();
    dependent_trigger();
    const bool dual = write && p.norm_a != nullptr;
    if (dual) {
        float ssa = 0.f, ssb = 0.f;
        for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
            float va[V], vb[V];
            branch_at<V, TB, MANY>(a, base + (size_t)c * V, va);
            branch_at<V, TB, MANY>(b, base + (size_t)c * V, vb);
#pragma unroll
            for (int e = 0; e < V; ++e) { ssa = fmaf(va[e], va[e], ssa); ssb = fmaf(vb[e], vb[e], ssb); }
            Pack<V, float>::store(row + width + c * V, va);
            Pack<V, float>::store(row + 2 * width + c * V, vb);
        }
        const float2 ss = block_sum2(ssa, ssb, scratch);
        const float inv_a = 1.f / sqrtf(ss.x / (float)width + p.eps_ab), inv_b = 1.f / sqrtf(ss.y / (float)width + p.eps_ab);
        for (int c = threadIdx.x; c < chunks; c += blockDim.x) {        // their sum in the first one's place (this thread's own values)
            float va[V], vb[V], wa[V], wb[V];
            Pack<V, float>::load(row + width + c * V, va);
            Pack<V, float>::load(row + 2 * width + c * V, vb);
            Pack<V, float>::load(p.norm_a + c * V, wa);
            Pack<V, float>::load(p.norm_b + c * V, wb);
#pragma unroll
            for (int e = 0; e < V; ++e) va[e] = va[e] * inv_a * wa[e] + vb[e] * inv_b * wb[e];
            Pack<V, float>::store(row + width + c * V, va);
        }
    }
    float sum = 0.f;
    for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
        float v[SM][V];
#pragma unroll
        for (int s = 0; s < SM; ++s)
            if (s < S) Pack<V, float>::load(x + (size_t)s * width + c * V, v[s]);
        float u[V];
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
        if (write) {
            float y[V];
            if (dual) {
                Pack<V, float>::load(row + width + c * V, y);
            } else {
                branch_at<V, TB, MANY>(a, base + (size_t)c * V, y);
            }
            if (p.scale != nullptr) {
                float w[V];
                Pack<V, float>::load(p.scale + c * V, w);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] *= w[e];
            }
#pragma unroll
            for (int t = 0; t < SM; ++t) {
                if (t < S) {
                    float n[V];
#pragma unroll
                    for (int e = 0; e < V; ++e) n[e] = out[t] * y[e];
#pragma unroll
                    for (int s = 0; s < SM; ++s)
                        if (s < S) {
#pragma unroll
                            for (int e = 0; e < V; ++e) n[e] = fmaf(held[t * SM + s], v[s][e], n[e]);
                        }
                    Pack<V, float>::store(x + (size_t)t * width + c * V, n);
#pragma unroll
                    for (int e = 0; e < V; ++e) u[e] = fmaf(in[t], n[e], u[e]);
                }
            }
        } else {
#pragma unroll
            for (int s = 0; s < SM; ++s)
                if (s < S) {
#pragma unroll
                    for (int e = 0; e < V; ++e) u[e] = fmaf(in[s], v[s][e], u[e]);
                }
        }
        if (read) {
            Pack<V, float>::store(row + c * V, u);              // read back by this thread only
#pragma unroll
            for (int e = 0; e < V; ++e) sum += u[e];
        }
    }
    if (!read) return;
    const float mean = p.center ? block_sum(sum, scratch) / (float)width : 0.f;
    float ss = 0.f;
    for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
        float u[V];
        Pack<V, float>::load(row + c * V, u);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(u[e] - mean, u[e] - mean, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)width + p.eps);
    for (int c = threadIdx.x; c < chunks; c += blockDim.x) {
        float u[V], w[V];
        Pack<V, float>::load(row + c * V, u);
        Pack<V, float>::load(p.weight + c * V, w);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = (u[e] - mean) * inv * (p.offset + w[e]);
        if (p.bias != nullptr) {
            Pack<V, float>::load(p.bias + c * V, w);
#pragma unroll
            for (int e = 0; e < V; ++e) u[e] += w[e];
        }
        Pack<V, TH>::store(h + base + (size_t)c * V, u);
    }
}

__global__ void stream_sum_kernel(float* __restrict__ out, const float* __restrict__ x, const int* __restrict__ rows, int width, int streams,
                                  int src_rows) {
    const int i = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= width) return;
    const int r = rows[i];
    float v = __int_as_float(0x7fc00000);
    if (r >= 0 && r < src_rows) {
        v = 0.f;
        for (int s = 0; s < streams; ++s) v += x[((size_t)r * streams + s) * width + c];
    }
    out[(size_t)i * width + c] = v;
}

template <typename TB, typename TH, int V, int SM, bool MANY>
static int launch_stream_step(const StreamParams& p, const Src<TB>& a, const Src<TB>& b, void* h, int rows, cudaStream_t s) {
    const size_t smem = (size_t)p.width * sizeof(float) * (p.norm_a != nullptr && p.mix != nullptr ? 3 : 1);
    KB_REQUIRE(smem <= 200 * 1024, "stream_step: rows of %d values do not fit the shared memory of a block", p.width);
    if (smem > 40 * 1024) cudaFuncSetAttribute(stream_step_kernel<TB, TH, V, SM, MANY>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int chunks = p.width / V;
    const int threads = std::min(STREAM_THREADS, std::max(64, (chunks + 31) / 32 * 32));
    launch_dependent_if(rows <= DEPENDENT_ROWS, stream_step_kernel<TB, TH, V, SM, MANY>, dim3(rows), dim3(threads), smem, s, p, a, b, (TH*)h);
    return check_launch("stream_step");
}

template <typename TB, typename TH>
static int run_stream_step(const StreamParams& p, const Src<TB>& a, const Src<TB>& b, void* h, int rows, bool wide, cudaStream_t s) {
    const bool many = a.splits > 1 || b.splits > 1;
#define KB_SS2(V, SM) (many ? launch_stream_step<TB, TH, V, SM, true>(p, a, b, h, rows, s) : launch_stream_step<TB, TH, V, SM, false>(p, a, b, h, rows, s))
#define KB_SS(SM) (wide ? KB_SS2(4, SM) : KB_SS2(1, SM))
    if (p.streams <= 2) return KB_SS(2);
    if (p.streams <= 4) return KB_SS(4);
    if (p.streams <= 8) return KB_SS(8);
    return launch_stream_step<TB, TH, 1, STREAMS_MAX, true>(p, a, b, h, rows, s);
#undef KB_SS
#undef KB_SS2
}

}  // namespace kb

using namespace kb;

extern "C" int kb_streams_max() { return STREAMS_MAX; }

// x [rows, streams, width]. Write: mix, out and branch `a` (and, with norm_a and norm_b, `b`: slices of the same dtype), each
// `*_splits` slices `*_stride` elements apart. Read: in, weight and h.
extern "C" int kb_stream_step(float* x, int rows, int streams, int width, const void* a, int a_splits, long long a_stride, const void* b,
                              int b_splits, long long b_stride, int branch_dt, const float* norm_a, const float* norm_b, float eps_ab,
                              const float* scale, const float* mix, const float* out, const float* in,
                              const float* weight, const float* bias, float eps, float offset, int center, void* h, int h_dt, void* stream) {
    KB_REQUIRE(rows >= 0 && width > 0 && streams >= 1 && streams <= STREAMS_MAX, "stream_step: rows %d, width %d, %d streams (1 to %d)", rows, width, streams, STREAMS_MAX);
    KB_REQUIRE(x != nullptr && (mix != nullptr || in != nullptr), "stream_step: nothing to write and nothing to read");
    KB_REQUIRE((mix == nullptr) == (out == nullptr) && (mix == nullptr) == (a == nullptr), "stream_step: a write takes a branch, mix and out");
    KB_REQUIRE((norm_a == nullptr) == (norm_b == nullptr) && (norm_a == nullptr) == (b == nullptr), "stream_step: two normed branches take two weights");
    KB_REQUIRE((in == nullptr) == (h == nullptr) && (in == nullptr) == (weight == nullptr), "stream_step: a read takes its weights and an output");
    KB_REQUIRE(a == nullptr || (a_splits >= 1 && (a_splits == 1 || a_stride >= (long long)rows * width)), "stream_step: %d slices %lld apart", a_splits, a_stride);
    KB_REQUIRE(b == nullptr || (b_splits >= 1 && (b_splits == 1 || b_stride >= (long long)rows * width)), "stream_step: %d slices %lld apart", b_splits, b_stride);
    if (rows == 0) return 0;
    StreamParams p;
    p.x = x; p.streams = streams; p.width = width; p.mix = mix; p.out = out; p.scale = scale; p.norm_a = norm_a; p.norm_b = norm_b;
    p.eps_ab = eps_ab; p.in = in; p.weight = weight; p.bias = bias; p.eps = eps; p.offset = offset; p.center = center;
    const uintptr_t f32s = (uintptr_t)x | (uintptr_t)norm_a | (uintptr_t)norm_b | (uintptr_t)scale | (uintptr_t)weight | (uintptr_t)bias;
    const bool strides = (a_splits <= 1 || a_stride % 4 == 0) && (b == nullptr || b_splits <= 1 || b_stride % 4 == 0);
    const bool wide = width % 4 == 0 && strides && ((f32s | (uintptr_t)a | (uintptr_t)b | (uintptr_t)h) & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
#define KB_STEP(TB, TH)                                                                                              \
    return run_stream_step<TB, TH>(p, Src<TB>{(const TB*)a, a_splits, (size_t)a_stride}, Src<TB>{(const TB*)b, b_splits, (size_t)b_stride}, h, rows, wide, s)
    if (branch_dt == KB_DT_F32 && h_dt == KB_DT_F32) KB_STEP(float, float);
    if (branch_dt == KB_DT_F32 && h_dt == KB_DT_BF16) KB_STEP(float, bf16);
    if (branch_dt == KB_DT_BF16 && h_dt == KB_DT_BF16) KB_STEP(bf16, bf16);
    if (branch_dt == KB_DT_BF16 && h_dt == KB_DT_F32) KB_STEP(bf16, float);
#undef KB_STEP
    return fail("stream_step: dtype codes %d (branch), %d (output) are not known", branch_dt, h_dt);
}

extern "C" int kb_stream_sum(float* out, const float* x, const int* rows, int n, int width, int streams, int src_rows, void* stream) {
    KB_REQUIRE(n >= 0 && width > 0 && streams >= 1, "stream_sum: n %d, width %d, %d streams", n, width, streams);
    KB_REQUIRE(n <= 65535, "stream_sum: %d rows are too many for one launch", n);
    if (n == 0) return 0;
    stream_sum_kernel<<<dim3((unsigned)((width + 255) / 256), n), 256, 0, (cudaStream_t)stream>>>(out, x, rows, width, streams, src_rows);
    return check_launch("stream_sum");
}
