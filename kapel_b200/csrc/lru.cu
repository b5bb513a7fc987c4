// The real-gated linear recurrent unit (Griffin's RG-LRU), over the rows of a step.
//
// For a channel c in part b of `blocks` equal parts, with u the convolved branch (32-bit, [rows, width]):
//     r = sigmoid(ra[b] u_b + ra_bias)_c,   i = sigmoid(ri[b] u_b + ri_bias)_c,
//     log a = -rate r softplus(lam_c),   S <- a S + sqrt(1 - a^2) i u_c,   out = S gelu_tanh(y_c + y_bias_c)
// S is one float a channel in a slot of a state table, one slot a request, carried from a request's last
// row in this step to its first row in the next. Everything here is 32-bit.
//
// Two kernels. The gates' kernel makes (a - 1, sqrt(1 - a^2) i u) of every row and channel: two square products
// a part, taken in true 32-bit (tiles of 64 rows by 32 channels; for a few rows a warp a channel). A memory of
// thousands of rows has decays so near 1 that rounding a itself would be most of the error: a - 1 keeps its own
// precision, and a row is S <- S + ((a - 1) S + b), rounded once. The scan's kernel walks a request's rows: a
// step composes ((x1, b1) then (x2, b2) is (x1 + x2 + x1 x2, b1 + x2 b1 + b2) with x = a - 1), so a block takes
// 16 channels and 32 runs of 8 rows at a time, each thread composing one run, the runs joined by a scan over a
// warp's lanes; then every thread walks its rows again from the state before them. A step of few rows a request
// is walked by one thread a channel.
#include "common.cuh"

namespace kb {

typedef __nv_bfloat16 bf16;

struct LruGateParams {
    const float* u;             // [rows, width]
    const float* ra_bias;       // [width]
    const float* ri_bias;
    const float* lam;           // [width]
    float2* ab;                 // [rows, width]: (a - 1, what is added)
    float rate;
    int rows, width, part;      // part = width / blocks
};

__device__ __forceinline__ float lru_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

__device__ __forceinline__ float2 lru_step(const LruGateParams& p, int c, float zr, float zi, float u) {
    const float lam = p.lam[c];
    const float sp = lam > 20.f ? lam : log1pf(expf(lam));
    const float log_a = -p.rate * lru_sigmoid(zr + p.ra_bias[c]) * sp;
    const float x = expm1f(log_a);                              // a - 1; 1 - a^2 = -x (x + 2)
    return make_float2(x, sqrtf(-x * (x + 2.f)) * lru_sigmoid(zi + p.ri_bias[c]) * u);
}

// A step (x, b) on a state, and on what an earlier step does (b1; its x1 likewise with b = x).
__device__ __forceinline__ float lru_apply(float x, float b, float S) { return S + fmaf(x, S, b); }

constexpr int LG_ROWS = 64, LG_COLS = 32, LG_K = 32, LG_THREADS = 256;

// One block = 64 rows x 32 channels of one part; a thread 4 rows x 2 channels of both products.
template <typename TW>
__global__ void __launch_bounds__(LG_THREADS)
lru_gates_kernel(const TW* __restrict__ ra, const TW* __restrict__ ri, const LruGateParams p) {
    __shared__ __align__(16) float su[LG_K][LG_ROWS + 4];
    __shared__ __align__(16) float sr[LG_K][LG_COLS + 2], si[LG_K][LG_COLS + 2];
    const int b = blockIdx.z, c0 = blockIdx.y * LG_COLS, r0 = blockIdx.x * LG_ROWS;
    const int tid = threadIdx.x, tr = tid / 16, tc = tid % 16;
    const TW* wr = ra + (size_t)b * p.part * p.part;
    const TW* wi = ri + (size_t)b * p.part * p.part;
    float zr[4][2] = {}, zi[4][2] = {};
    for (int k0 = 0; k0 < p.part; k0 += LG_K) {
        for (int idx = tid; idx < LG_ROWS * LG_K; idx += LG_THREADS) {
            const int rr = idx / LG_K, k = idx % LG_K;
            su[k][rr] = (r0 + rr < p.rows && k0 + k < p.part) ? p.u[(size_t)(r0 + rr) * p.width + b * p.part + k0 + k] : 0.f;
        }
        for (int idx = tid; idx < LG_COLS * LG_K; idx += LG_THREADS) {
            const int cc = idx / LG_K, k = idx % LG_K;
            const bool in = c0 + cc < p.part && k0 + k < p.part;
            sr[k][cc] = in ? Elem<TW>::load(wr + (size_t)(c0 + cc) * p.part + k0 + k) : 0.f;
            si[k][cc] = in ? Elem<TW>::load(wi + (size_t)(c0 + cc) * p.part + k0 + k) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < LG_K; ++k) {
            const float4 u4 = *reinterpret_cast<const float4*>(&su[k][tr * 4]);
            const float2 r2 = *reinterpret_cast<const float2*>(&sr[k][tc * 2]), i2 = *reinterpret_cast<const float2*>(&si[k][tc * 2]);
            const float u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                zr[x][0] = fmaf(u[x], r2.x, zr[x][0]);
                zr[x][1] = fmaf(u[x], r2.y, zr[x][1]);
                zi[x][0] = fmaf(u[x], i2.x, zi[x][0]);
                zi[x][1] = fmaf(u[x], i2.y, zi[x][1]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
            const int r = r0 + tr * 4 + x, cp = c0 + tc * 2 + y;
            if (r < p.rows && cp < p.part) {
                const int c = b * p.part + cp;
                p.ab[(size_t)r * p.width + c] = lru_step(p, c, zr[x][y], zi[x][y], p.u[(size_t)r * p.width + c]);
            }
        }
}

// A few rows: a warp a channel, eight rows at a time.
constexpr int LF_WARPS = 8, LF_ROWS = 8;
template <typename TW>
__global__ void __launch_bounds__(LF_WARPS * 32)
lru_gates_few_kernel(const TW* __restrict__ ra, const TW* __restrict__ ri, const LruGateParams p) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * LF_WARPS + warp;
    if (c >= p.width) return;
    const int b = c / p.part;
    const int r0 = blockIdx.y * LF_ROWS, nr = min(LF_ROWS, p.rows - r0);
    const TW* wr = ra + (size_t)c * p.part;                     // [blocks, part, part]: row c of the stack
    const TW* wi = ri + (size_t)c * p.part;
    const float* u = p.u + (size_t)r0 * p.width + b * p.part;
    float zr[LF_ROWS] = {}, zi[LF_ROWS] = {};
    for (int k = lane; k < p.part; k += 32) {
        const float a = Elem<TW>::load(wr + k), g = Elem<TW>::load(wi + k);
#pragma unroll
        for (int x = 0; x < LF_ROWS; ++x) {
            const float v = x < nr ? u[(size_t)x * p.width + k] : 0.f;
            zr[x] = fmaf(a, v, zr[x]);
            zi[x] = fmaf(g, v, zi[x]);
        }
    }
#pragma unroll
    for (int x = 0; x < LF_ROWS; ++x) {
        zr[x] = warp_sum(zr[x]);
        zi[x] = warp_sum(zi[x]);
    }
    for (int x = 0; x < nr; ++x)
        if (lane == x) {
            float a = 0.f, g = 0.f;
#pragma unroll
            for (int y = 0; y < LF_ROWS; ++y) { a = y == x ? zr[y] : a; g = y == x ? zi[y] : g; }
            p.ab[(size_t)(r0 + x) * p.width + c] = lru_step(p, c, a, g, p.u[(size_t)(r0 + x) * p.width + c]);
        }
}

struct LruScanParams {
    const float2* ab;           // [rows, width]
    const float* y_bias;        // [width]
    float* state;               // [slots, width]
    const int* entry_start;
    const int* entry_end;
    const int* slots;
    int n_slots, width, row_width, y_off, out_stride;
};

constexpr int LS_CH = 16, LS_RUNS = 32, LS_ROWS = 8;            // channels a block; runs of rows at a time; rows a run

template <typename TS, typename TO>
__global__ void __launch_bounds__(LS_CH * LS_RUNS)
lru_scan_kernel(const Src<TS> src, const LruScanParams p, TO* __restrict__ out) {
    __shared__ float2 run[LS_RUNS][LS_CH + 1];                  // what a run does to a state; then the state before it in .x
    __shared__ float carry[LS_CH];
    const int entry = blockIdx.y;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    if (r1 <= r0) return;
    const int slot = p.slots[entry];
    const bool live = slot > 0 && slot < p.n_slots;
    const int cl = threadIdx.x % LS_CH, s = threadIdx.x / LS_CH;
    const int c = blockIdx.x * LS_CH + cl;
    const bool mine = c < p.width;
    if (blockIdx.x == 0)                                        // the product behind may want rows wider than the channels
        for (int idx = threadIdx.x; idx < (r1 - r0) * (p.out_stride - p.width); idx += LS_CH * LS_RUNS) {
            const int r = idx / (p.out_stride - p.width), x = idx - r * (p.out_stride - p.width);
            Elem<TO>::store(out + (size_t)(r0 + r) * p.out_stride + p.width + x, 0.f);
        }
    if (!live) {                                                // rows of no request: zeros, no state
        if (mine)
            for (int r = r0 + s; r < r1; r += LS_RUNS) Elem<TO>::store(out + (size_t)r * p.out_stride + c, 0.f);
        return;
    }
    if (s == 0 && mine) carry[cl] = p.state[(size_t)slot * p.width + c];
    const float bias = mine ? p.y_bias[c] : 0.f;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float2 next[LS_ROWS];
    auto fetch = [&](int base) {
#pragma unroll
        for (int j = 0; j < LS_ROWS; ++j) {
            const int r = base + s * LS_ROWS + j;
            next[j] = (mine && r < r1) ? p.ab[(size_t)r * p.width + c] : make_float2(0.f, 0.f);
        }
    };
    fetch(r0);
    for (int base = r0; base < r1; base += LS_RUNS * LS_ROWS) {
        float2 ab[LS_ROWS];
        float y[LS_ROWS];
#pragma unroll
        for (int j = 0; j < LS_ROWS; ++j) {
            ab[j] = next[j];
            const int r = base + s * LS_ROWS + j;
            y[j] = (mine && r < r1) ? src.at((size_t)r * p.row_width + p.y_off + c) : 0.f;
        }
        if (base + LS_RUNS * LS_ROWS < r1) fetch(base + LS_RUNS * LS_ROWS);
        float X = 0.f, B = 0.f;
#pragma unroll
        for (int j = 0; j < LS_ROWS; ++j) {
            X = lru_apply(ab[j].x, ab[j].x, X);
            B = lru_apply(ab[j].x, ab[j].y, B);
        }
        run[s][cl] = make_float2(X, B);
        __syncthreads();
        {                                                       // warp w joins the runs of channel w, lane l being run l
            float2 f = run[lane][warp];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x1 = __shfl_up_sync(0xffffffffu, f.x, o), b1 = __shfl_up_sync(0xffffffffu, f.y, o);
                if (lane >= o) {                                // f after (x1, b1)
                    f.y = lru_apply(f.x, f.y, b1);
                    f.x = lru_apply(f.x, f.x, x1);
                }
            }
            const float start = carry[warp];
            const float after = lru_apply(f.x, f.y, start);          // the state behind this lane's run
            float before = __shfl_up_sync(0xffffffffu, after, 1);
            if (lane == 0) before = start;
            __syncwarp();
            run[lane][warp].x = before;
            if (lane == 31) carry[warp] = after;
        }
        __syncthreads();
        float S = run[s][cl].x;
#pragma unroll
        for (int j = 0; j < LS_ROWS; ++j) {
            const int r = base + s * LS_ROWS + j;
            S = lru_apply(ab[j].x, ab[j].y, S);
            if (mine && r < r1) Elem<TO>::store(out + (size_t)r * p.out_stride + c, S * gelu_tanh(y[j] + bias));
        }
        __syncthreads();                                        // the runs may be written again
    }
    if (s == 0 && mine) p.state[(size_t)slot * p.width + c] = carry[cl];
}
static_assert(LS_CH * LS_RUNS == LS_CH * 32 && LS_RUNS == 32, "a warp a channel, a lane a run");

// Few rows a request: a thread a channel walks them.
template <typename TS, typename TO>
__global__ void lru_scan_few_kernel(const Src<TS> src, const LruScanParams p, TO* __restrict__ out) {
    const int entry = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= p.out_stride) return;
    const int r0 = p.entry_start[entry], r1 = p.entry_end[entry];
    const int slot = p.slots[entry];
    const bool live = slot > 0 && slot < p.n_slots && c < p.width;
    float S = live && r1 > r0 ? p.state[(size_t)slot * p.width + c] : 0.f;
    const float bias = live ? p.y_bias[c] : 0.f;
    for (int r = r0; r < r1; ++r) {
        float o = 0.f;
        if (live) {
            const float2 ab = p.ab[(size_t)r * p.width + c];
            S = lru_apply(ab.x, ab.y, S);
            o = S * gelu_tanh(src.at((size_t)r * p.row_width + p.y_off + c) + bias);
        }
        Elem<TO>::store(out + (size_t)r * p.out_stride + c, o);
    }
    if (live && r1 > r0) p.state[(size_t)slot * p.width + c] = S;
}

}  // namespace kb

using namespace kb;

// ab [rows, width, 2] = (a - 1, sqrt(1 - a^2) i u) of every row and channel.
extern "C" int kb_lru_gates(float* ab, const float* u, const void* ra, const void* ri, int w_dt, const float* ra_bias, const float* ri_bias,
                            const float* lam, float rate, int rows, int width, int blocks, void* stream) {
    KB_REQUIRE(rows >= 0 && width > 0 && blocks > 0 && width % blocks == 0, "lru_gates: rows %d, %d channels in %d parts", rows, width, blocks);
    KB_REQUIRE(ab && u && ra && ri && ra_bias && ri_bias && lam, "lru_gates: a tensor is missing");
    KB_REQUIRE(rate > 0.f, "lru_gates: rate %g must be positive", rate);
    if (rows == 0) return 0;
    LruGateParams p;
    p.u = u; p.ra_bias = ra_bias; p.ri_bias = ri_bias; p.lam = lam; p.ab = (float2*)ab; p.rate = rate; p.rows = rows; p.width = width;
    p.part = width / blocks;
    cudaStream_t s = (cudaStream_t)stream;
    const bool few = rows <= DEPENDENT_ROWS;
    const dim3 fgrid((width + LF_WARPS - 1) / LF_WARPS, (rows + LF_ROWS - 1) / LF_ROWS);
    const dim3 grid((rows + LG_ROWS - 1) / LG_ROWS, (p.part + LG_COLS - 1) / LG_COLS, blocks);
    KB_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "lru_gates: %d parts of %d channels is too many for one launch", blocks, p.part);
    if (w_dt == KB_DT_F32) {
        if (few) lru_gates_few_kernel<float><<<fgrid, LF_WARPS * 32, 0, s>>>((const float*)ra, (const float*)ri, p);
        else lru_gates_kernel<float><<<grid, LG_THREADS, 0, s>>>((const float*)ra, (const float*)ri, p);
    } else if (w_dt == KB_DT_BF16) {
        if (few) lru_gates_few_kernel<bf16><<<fgrid, LF_WARPS * 32, 0, s>>>((const bf16*)ra, (const bf16*)ri, p);
        else lru_gates_kernel<bf16><<<grid, LG_THREADS, 0, s>>>((const bf16*)ra, (const bf16*)ri, p);
    } else {
        return fail("lru_gates: dtype code %d is not known", w_dt);
    }
    return check_launch("lru_gates");
}

// out [rows, out_stride] (zeros behind the channels): the unit's state times the gelu branch, request by request from and into
// `state` [slots, width]; `longest`: the most rows a request brings.
extern "C" int kb_lru_scan(void* out, int out_dt, int out_stride, const float* ab, const void* src, int in_dt, int splits,
                           long long split_stride, int row_width, int y_off, const float* y_bias, float* state, int n_slots,
                           const int* entry_start, const int* entry_end, const int* slots, int entries, int rows, int longest, int width,
                           void* stream) {
    KB_REQUIRE(rows >= 0 && entries >= 0 && width > 0 && out_stride >= width, "lru_scan: rows %d, requests %d, %d channels in rows of %d", rows, entries, width, out_stride);
    KB_REQUIRE(row_width > 0 && y_off >= 0 && y_off + (long long)width <= row_width, "lru_scan: columns %d.. do not fit a row of %d", y_off, row_width);
    KB_REQUIRE(splits >= 1 && (splits == 1 || split_stride >= (long long)rows * row_width), "lru_scan: %d slices %lld apart", splits, split_stride);
    KB_REQUIRE(out && ab && src && y_bias && state && n_slots >= 1 && entry_start && entry_end && slots, "lru_scan: a tensor is missing");
    KB_REQUIRE(entries <= 65535, "lru_scan: too many requests for one launch");
    if (rows == 0 || entries == 0) return 0;
    LruScanParams p;
    p.ab = (const float2*)ab; p.y_bias = y_bias; p.state = state; p.entry_start = entry_start; p.entry_end = entry_end; p.slots = slots;
    p.n_slots = n_slots; p.width = width; p.row_width = row_width; p.y_off = y_off; p.out_stride = out_stride;
    cudaStream_t s = (cudaStream_t)stream;
    const bool few = longest <= 2 * LS_ROWS;
    const dim3 grid((width + LS_CH - 1) / LS_CH, entries), fgrid((out_stride + 127) / 128, entries);
#define KB_LS(TS, TO)                                                                                                      \
    do {                                                                                                                   \
        const Src<TS> x{(const TS*)src, splits, (size_t)split_stride};                                                      \
        if (few) lru_scan_few_kernel<TS, TO><<<fgrid, 128, 0, s>>>(x, p, (TO*)out);                                         \
        else lru_scan_kernel<TS, TO><<<grid, LS_CH * LS_RUNS, 0, s>>>(x, p, (TO*)out);                                      \
    } while (0)
    if (in_dt == KB_DT_F32 && out_dt == KB_DT_F32) KB_LS(float, float);
    else if (in_dt == KB_DT_F32 && out_dt == KB_DT_BF16) KB_LS(float, bf16);
    else if (in_dt == KB_DT_BF16 && out_dt == KB_DT_BF16) KB_LS(bf16, bf16);
    else return fail("lru_scan: dtype codes %d -> %d are not known", in_dt, out_dt);
#undef KB_LS
    return check_launch("lru_scan");
}
