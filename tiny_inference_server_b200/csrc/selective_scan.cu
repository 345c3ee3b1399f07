// A selective scan whose decay differs from channel to channel and from state to state (Mamba's first form).  Per channel c a
// state of N numbers, 32-bit, carried from step to step for each request:
//   dt = softplus(dt_in[c] + dt_bias[c]),  A[c][n] = -exp(A_log[c][n]),
//   S[c][n] <- exp(dt A[c][n]) S[c][n] + dt x[c] B[n],   y[c] = sum_n S[c][n] C[n] + D[c] x[c],   out[c] = y[c] * silu(z[c]).
//
// Every channel is a recurrence of its own.  LANES neighbouring lanes share a channel, DL states each in registers; a CTA
// takes 128 / LANES channels of one request and walks its rows 32 at a time: all threads prepare (dt, dt x) of the chunk's
// rows and channels and the rows' B and C in shared memory (the raw values of the next chunk are already on their way in
// registers), then every lane walks LANES rows in a row without exchanging anything and the lanes of a channel add their
// LANES partial sums of LANES rows at once (LANES - 1 shuffles instead of LANES * log2(LANES)), one row a lane; then
// the chunk's outputs are gated and stored.  The step from S to S is one multiply-add; everything else of a row is off
// the chain of dependences.
#include "common.cuh"

namespace {

constexpr int SCAN_THREADS = 128;
constexpr int SCAN_ROWS = 32;          // rows of a chunk

// softplus and x * sigmoid(x): the exact functions for 32-bit activations.  Otherwise the fast exponential and logarithm, and
// for small e the series log(1 + e) = e - e^2 / 2 + e^3 / 3 - .. (the logarithm of a number next to 1 would lose its digits):
// relative errors below 1e-5.
template <typename T> __device__ __forceinline__ float scan_softplus(float x);
template <> __device__ __forceinline__ float scan_softplus<float>(float x) { return x > 20.f ? x : log1pf(expf(x)); }
template <> __device__ __forceinline__ float scan_softplus<bf16>(float x) {
    const float e = __expf(fminf(x, 20.f));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.f / 3.f), -0.5f), 1.f);
    return x > 20.f ? x : (e < 0.03125f ? series : __logf(1.f + e));
}
template <typename T> __device__ __forceinline__ float scan_silu(float x);
template <> __device__ __forceinline__ float scan_silu<float>(float x) { return x / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float scan_silu<bf16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }

// 2^x: exact to the last bits for 32-bit activations, the fast form otherwise
template <typename T> __device__ __forceinline__ float scan_exp2(float x);
template <> __device__ __forceinline__ float scan_exp2<float>(float x) { return exp2f(x); }
template <> __device__ __forceinline__ float scan_exp2<bf16>(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

// Two multiply-adds (multiplications) in one instruction: neighbouring states of a lane.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("{\n.reg .b64 a, b, c, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmov.b64 c, {%6, %7};\nfma.rn.f32x2 d, a, b, c;\n"
        "mov.b64 {%0, %1}, d;\n}\n"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("{\n.reg .b64 a, b, d;\nmov.b64 a, {%2, %3};\nmov.b64 b, {%4, %5};\nmul.rn.f32x2 d, a, b;\nmov.b64 {%0, %1}, d;\n}\n"
        : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
    return d;
}

struct ScanParams {
    const void* x; int ldx;            // inputs (n, channels)
    const float* dt_in; int ldd;       // step sizes before the bias and the softplus (n, channels)
    const float* dt_bias;
    const float* A_log;                // (channels, N)
    const void* b; const void* c; int ldbc;     // (n, N) each
    const float* D;
    const void* z; int ldz;            // gates (n, channels)
    float* state; size_t state_stride; // [slots][channels][N]
    void* out; int ldo;
    const int* row_slot; const int* row_last; const int* seg_row0;
    int channels, N;
};

template <int LANES, int DL>
struct ScanShared {
    static constexpr int CB = SCAN_THREADS / LANES, NP = LANES * DL;
    static constexpr int YS = (CB + 31) / 32 * 32 + 32 / LANES;      // row stride of the sums: the lanes of a channel meet no bank twice
    float b[SCAN_ROWS][NP];
    float c[SCAN_ROWS][NP];
    float2 dt[SCAN_ROWS][CB];          // (dt, dt x)
    float y[SCAN_ROWS][YS];
};

template <typename T, int LANES, int DL>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_scan_kernel(const ScanParams p) {
    constexpr int CB = SCAN_THREADS / LANES;               // channels of a CTA
    constexpr int NP = LANES * DL;                         // states of a channel, padded
    constexpr int XPT = SCAN_ROWS / LANES;                 // (row, channel) pairs a thread prepares
    constexpr int BPT = SCAN_ROWS * NP / SCAN_THREADS;     // elements of B (and of C) a thread brings
    static_assert(SCAN_ROWS % LANES == 0 && BPT >= 1, "a chunk is whole groups of LANES rows");
    extern __shared__ __align__(16) unsigned char scan_smem[];
    ScanShared<LANES, DL>& sh = *reinterpret_cast<ScanShared<LANES, DL>*>(scan_smem);
    auto& sdt = sh.dt;
    auto& sb = sh.b;
    auto& sc = sh.c;
    auto& sy = sh.y;
    pdl_launch_dependents();
    const int r0 = p.seg_row0 != nullptr ? p.seg_row0[blockIdx.y] : (int)blockIdx.y;
    const int slot = p.row_slot[r0];
    if (slot < 0) return;
    if (p.seg_row0 == nullptr && r0 > 0 && p.row_slot[r0 - 1] == slot) return;
    const int rows = p.row_last[r0] - r0 + 1;
    const int tid = threadIdx.x, part = tid % LANES, cl = tid / LANES;
    const int c0 = blockIdx.x * CB, ch = c0 + cl;
    const bool mine = ch < p.channels;
    constexpr int DP = DL / 2;                             // a lane's states in pairs
    float2 A2[DP], S[DP];                                  // decay rates in units of log2
#pragma unroll
    for (int i = 0; i < DP; ++i) {
        const int n = part * DL + 2 * i;
        A2[i].x = mine && n < p.N ? -expf(p.A_log[(size_t)ch * p.N + n]) * 1.4426950408889634f : 0.f;
        A2[i].y = mine && n + 1 < p.N ? -expf(p.A_log[(size_t)ch * p.N + n + 1]) * 1.4426950408889634f : 0.f;
    }
    // what a thread prepares of every row: channel `tid % CB` of rows tid / CB, + LANES, ...
    const int pc = tid % CB, pr = tid / CB, pch = c0 + pc;
    const bool prepares = pch < p.channels;
    const float bias = prepares ? p.dt_bias[pch] : 0.f, skip = prepares ? p.D[pch] : 0.f;
    const T* x = static_cast<const T*>(p.x);
    const T* z = static_cast<const T*>(p.z);
    const T* bs = static_cast<const T*>(p.b);
    const T* cs = static_cast<const T*>(p.c);
    // raw values: a conversion next to the load would wait for it
    const T none = from_f32<T>(0.f);
    T rx[XPT], rb[BPT], rc[BPT];
    float rd[XPT];
    auto fetch = [&](int at) {
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = at + pr + k * LANES;
            const bool live = prepares && t < rows;
            const size_t rr = (size_t)(r0 + (live ? t : 0));
            rx[k] = live ? x[rr * p.ldx + pch] : none;
            rd[k] = live ? p.dt_in[rr * p.ldd + pch] : 0.f;
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int idx = tid + k * SCAN_THREADS, t = at + idx / NP, n = idx % NP;
            const bool live = t < rows && n < p.N;
            const size_t rr = (size_t)(r0 + (live ? t : 0));
            rb[k] = live ? bs[rr * p.ldbc + n] : none;
            rc[k] = live ? cs[rr * p.ldbc + n] : none;
        }
    };
    pdl_wait();
    float* S_glob = p.state + (size_t)slot * p.state_stride + (size_t)ch * p.N + part * DL;
#pragma unroll
    for (int i = 0; i < DP; ++i) {
        S[i].x = mine && part * DL + 2 * i < p.N ? S_glob[2 * i] : 0.f;
        S[i].y = mine && part * DL + 2 * i + 1 < p.N ? S_glob[2 * i + 1] : 0.f;
    }
    fetch(0);
    for (int at = 0; at < rows; at += SCAN_ROWS) {
        const int cnt = min(SCAN_ROWS, rows - at);
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = pr + k * LANES;
            if (k * LANES < cnt) {
                const float dt = t < cnt ? scan_softplus<T>(rd[k] + bias) : 0.f;      // (a row that does not exist changes nothing)
                const float xv = to_f32(rx[k]);
                sdt[t][pc] = make_float2(dt, dt * xv);
                sy[t][pc] = skip * xv;
            }
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int idx = tid + k * SCAN_THREADS;
            sb[idx / NP][idx % NP] = to_f32(rb[k]);
            sc[idx / NP][idx % NP] = to_f32(rc[k]);
        }
        __syncthreads();
        // the gates of this chunk and the raw values of the next one are on their way while this one is walked
        T rz[XPT];
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = pr + k * LANES;
            rz[k] = prepares && t < cnt ? z[(size_t)(r0 + at + t) * p.ldz + pch] : none;
        }
        if (at + SCAN_ROWS < rows) fetch(at + SCAN_ROWS);
        // with few lanes the operands of the group after are read from shared memory before this group is walked
        constexpr bool AHEAD = LANES <= 8;
        constexpr int AG = AHEAD ? LANES : 1;
        float2 dn[AG];
        float2 bn[AG][DP], cn[AG][DP];
        auto operands = [&](int t, float2& d, float2 (&bv)[DP], float2 (&cv)[DP]) {
            d = sdt[t][cl];
            if (DL % 4 == 0) {
#pragma unroll
                for (int i = 0; i < DP; i += 2) {
                    const float4 b4 = *reinterpret_cast<const float4*>(&sb[t][part * DL + 2 * i]);
                    const float4 c4 = *reinterpret_cast<const float4*>(&sc[t][part * DL + 2 * i]);
                    bv[i] = make_float2(b4.x, b4.y); bv[(i + 1) % DP] = make_float2(b4.z, b4.w);
                    cv[i] = make_float2(c4.x, c4.y); cv[(i + 1) % DP] = make_float2(c4.z, c4.w);
                }
            } else {
#pragma unroll
                for (int i = 0; i < DP; ++i) {
                    bv[i] = *reinterpret_cast<const float2*>(&sb[t][part * DL + 2 * i]);
                    cv[i] = *reinterpret_cast<const float2*>(&sc[t][part * DL + 2 * i]);
                }
            }
        };
        if (AHEAD) {
#pragma unroll
            for (int k = 0; k < AG; ++k) operands(k, dn[k], bn[k], cn[k]);
        }
#pragma unroll(AHEAD ? 2 : 1)
        for (int t0 = 0; t0 < cnt; t0 += LANES) {
            float y[LANES];
            float2 dc[AG];
            float2 bc[AG][DP], cc[AG][DP];
            if (AHEAD) {
#pragma unroll
                for (int k = 0; k < AG; ++k) {
                    dc[k] = dn[k];
#pragma unroll
                    for (int i = 0; i < DP; ++i) { bc[k][i] = bn[k][i]; cc[k][i] = cn[k][i]; }
                }
                const int nx = t0 + LANES < cnt ? t0 + LANES : t0;
#pragma unroll
                for (int k = 0; k < AG; ++k) operands(nx + k, dn[k], bn[k], cn[k]);
            }
#pragma unroll
            for (int k = 0; k < LANES; ++k) {
                constexpr int LAST = AG - 1;
                const int kk = AHEAD ? k : LAST;
                if (!AHEAD) operands(t0 + k, dc[0], bc[0], cc[0]);
                const float2 dt2 = make_float2(dc[kk].x, dc[kk].x), dx2 = make_float2(dc[kk].y, dc[kk].y);
                float2 acc = make_float2(0.f, 0.f);
#pragma unroll
                for (int i = 0; i < DP; ++i) {
                    float2 a = mul2(dt2, A2[i]);
                    a.x = scan_exp2<T>(a.x);
                    a.y = scan_exp2<T>(a.y);
                    S[i] = fma2(a, S[i], mul2(dx2, bc[kk][i]));
                    acc = fma2(S[i], cc[kk][i], acc);
                }
                y[k] = acc.x + acc.y;
            }
            // lane `part` ends with the sum of row t0 + part: at every step a lane hands the half of its rows that the
            // other lane is to keep over and adds what it gets to its own half
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) {
                const bool upper = (part & o) != 0;
#pragma unroll
                for (int i = 0; i < o; ++i) {
                    const float give = upper ? y[i] : y[i + o], keep = upper ? y[i + o] : y[i];
                    y[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            }
            sy[t0 + part][cl] += y[0];
        }
        __syncthreads();
        T* out = static_cast<T*>(p.out);
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = pr + k * LANES;
            if (prepares && t < cnt) out[(size_t)(r0 + at + t) * p.ldo + pch] = from_f32<T>(sy[t][pc] * scan_silu<T>(to_f32(rz[k])));
        }
        // (the next chunk's sums are written by the threads that read these, its other arrays were read before the barrier)
    }
    if (mine) {
#pragma unroll
        for (int i = 0; i < DP; ++i) {
            if (part * DL + 2 * i < p.N) S_glob[2 * i] = S[i].x;
            if (part * DL + 2 * i + 1 < p.N) S_glob[2 * i + 1] = S[i].y;
        }
    }
}

template <typename T, int LANES, int DL>
void launch_scan(const ScanParams& p, int segments, cudaStream_t stream) {
    constexpr int CB = SCAN_THREADS / LANES;
    constexpr size_t smem = sizeof(ScanShared<LANES, DL>);
    if (smem > 48 * 1024)
        cudaFuncSetAttribute(selective_scan_kernel<T, LANES, DL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    tis_launch(selective_scan_kernel<T, LANES, DL>, dim3((p.channels + CB - 1) / CB, segments), dim3(SCAN_THREADS), smem, stream, p);
}

template <typename T>
void launch_scan_any(const ScanParams& p, int segments, int fine, cudaStream_t stream) {
    if (fine && p.N <= 4) launch_scan<T, 4, 2>(p, segments, stream);
    else if (fine && p.N <= 16) launch_scan<T, 8, 2>(p, segments, stream);
    else if (fine && p.N <= 32) launch_scan<T, 16, 2>(p, segments, stream);
    else if (p.N <= 16) launch_scan<T, 4, 4>(p, segments, stream);
    else if (p.N <= 32) launch_scan<T, 8, 4>(p, segments, stream);
    else if (p.N <= 64) launch_scan<T, 16, 4>(p, segments, stream);
    else if (p.N <= 128) launch_scan<T, 32, 4>(p, segments, stream);
    else launch_scan<T, 32, 8>(p, segments, stream);
}

}  // namespace

// x, z, out (n, channels), b, c (n, N), of the storage type; dt_in (n, channels) float32; A_log (channels, N), dt_bias and D
// (channels) float32; `state` [slots][channels][N] float32 with a free slot stride.  seg_row0: the first rows of the step's
// requests (null: `segments` is n and every row is looked at).  fine: fewer states a lane (twice the CTAs).  N at most 256.
TIS_API int tis_selective_scan(int dtype, const void* x, int ldx, const float* dt_in, int ldd, const float* dt_bias,
                               const float* A_log, const void* b, const void* c, int ldbc, const float* D, const void* z, int ldz,
                               float* state, size_t state_stride, void* out, int ldo, const int* row_slot, const int* row_last,
                               const int* seg_row0, int segments, int n, int channels, int N, int fine, cudaStream_t stream) {
    if (n <= 0) return TIS_OK;
    if (seg_row0 == nullptr) segments = n;
    if (channels <= 0 || N <= 0 || N > 256 || segments <= 0 || segments > 65535) {
        tis_set_error("selective_scan: %d channels of %d states (at most 256), %d requests", channels, N, segments);
        return TIS_BAD_SIZE;
    }
    ScanParams p;
    p.x = x; p.ldx = ldx; p.dt_in = dt_in; p.ldd = ldd; p.dt_bias = dt_bias; p.A_log = A_log; p.b = b; p.c = c; p.ldbc = ldbc;
    p.D = D; p.z = z; p.ldz = ldz; p.state = state; p.state_stride = state_stride; p.out = out; p.ldo = ldo;
    p.row_slot = row_slot; p.row_last = row_last; p.seg_row0 = seg_row0; p.channels = channels; p.N = N;
    TIS_DISPATCH_DTYPE(dtype, T, launch_scan_any<T>(p, segments, fine, stream));
    return tis_check_launch("selective_scan");
}
