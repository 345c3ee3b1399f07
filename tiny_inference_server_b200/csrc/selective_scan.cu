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

__device__ __forceinline__ float scan_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// 2^x: exact to the last bits for 32-bit activations, the fast form otherwise
template <typename T> __device__ __forceinline__ float scan_exp2(float x);
template <> __device__ __forceinline__ float scan_exp2<float>(float x) { return exp2f(x); }
template <> __device__ __forceinline__ float scan_exp2<bf16>(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
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
    float A2[DL], S[DL];                                   // decay rates in units of log2
#pragma unroll
    for (int i = 0; i < DL; ++i) {
        const int n = part * DL + i;
        A2[i] = mine && n < p.N ? -expf(p.A_log[(size_t)ch * p.N + n]) * 1.4426950408889634f : 0.f;
    }
    // what a thread prepares of every row: channel `tid % CB` of rows tid / CB, + LANES, ...
    const int pc = tid % CB, pr = tid / CB, pch = c0 + pc;
    const bool prepares = pch < p.channels;
    const float bias = prepares ? p.dt_bias[pch] : 0.f, skip = prepares ? p.D[pch] : 0.f;
    const T* x = static_cast<const T*>(p.x);
    const T* z = static_cast<const T*>(p.z);
    const T* bs = static_cast<const T*>(p.b);
    const T* cs = static_cast<const T*>(p.c);
    float rx[XPT], rd[XPT];
    float rb[BPT], rc[BPT];
    auto fetch = [&](int at) {
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = at + pr + k * LANES;
            const bool live = prepares && t < rows;
            const size_t rr = (size_t)(r0 + (live ? t : 0));
            rx[k] = live ? to_f32(x[rr * p.ldx + pch]) : 0.f;
            rd[k] = live ? p.dt_in[rr * p.ldd + pch] : 0.f;
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int idx = tid + k * SCAN_THREADS, t = at + idx / NP, n = idx % NP;
            const bool live = t < rows && n < p.N;
            const size_t rr = (size_t)(r0 + (live ? t : 0));
            rb[k] = live ? to_f32(bs[rr * p.ldbc + n]) : 0.f;
            rc[k] = live ? to_f32(cs[rr * p.ldbc + n]) : 0.f;
        }
    };
    pdl_wait();
    float* S_glob = p.state + (size_t)slot * p.state_stride + (size_t)ch * p.N + part * DL;
#pragma unroll
    for (int i = 0; i < DL; ++i) S[i] = mine && part * DL + i < p.N ? S_glob[i] : 0.f;
    fetch(0);
    for (int at = 0; at < rows; at += SCAN_ROWS) {
        const int cnt = min(SCAN_ROWS, rows - at);
#pragma unroll
        for (int k = 0; k < XPT; ++k) {
            const int t = pr + k * LANES;
            if (k * LANES < cnt) {
                const float dt = t < cnt ? scan_softplus(rd[k] + bias) : 0.f;      // (a row that does not exist changes nothing)
                sdt[t][pc] = make_float2(dt, dt * rx[k]);
                sy[t][pc] = skip * rx[k];
            }
        }
#pragma unroll
        for (int k = 0; k < BPT; ++k) {
            const int idx = tid + k * SCAN_THREADS;
            sb[idx / NP][idx % NP] = rb[k];
            sc[idx / NP][idx % NP] = rc[k];
        }
        __syncthreads();
        if (at + SCAN_ROWS < rows) fetch(at + SCAN_ROWS);
#pragma unroll 1
        for (int t0 = 0; t0 < cnt; t0 += LANES) {
            float y[LANES];
#pragma unroll
            for (int k = 0; k < LANES; ++k) {
                const float2 d = sdt[t0 + k][cl];
                float bv[DL], cv[DL];
                if (DL % 4 == 0) {
#pragma unroll
                    for (int i = 0; i < DL; i += 4) {
                        const float4 b4 = *reinterpret_cast<const float4*>(&sb[t0 + k][part * DL + i]);
                        const float4 c4 = *reinterpret_cast<const float4*>(&sc[t0 + k][part * DL + i]);
                        bv[i] = b4.x; bv[(i + 1) % DL] = b4.y; bv[(i + 2) % DL] = b4.z; bv[(i + 3) % DL] = b4.w;
                        cv[i] = c4.x; cv[(i + 1) % DL] = c4.y; cv[(i + 2) % DL] = c4.z; cv[(i + 3) % DL] = c4.w;
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < DL; i += 2) {
                        const float2 b2 = *reinterpret_cast<const float2*>(&sb[t0 + k][part * DL + i]);
                        const float2 c2 = *reinterpret_cast<const float2*>(&sc[t0 + k][part * DL + i]);
                        bv[i] = b2.x; bv[i + 1] = b2.y;
                        cv[i] = c2.x; cv[i + 1] = c2.y;
                    }
                }
                float acc = 0.f;
#pragma unroll
                for (int i = 0; i < DL; ++i) {
                    S[i] = fmaf(scan_exp2<T>(d.x * A2[i]), S[i], d.y * bv[i]);
                    acc = fmaf(S[i], cv[i], acc);
                }
                y[k] = acc;
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
            if (prepares && t < cnt) {
                const size_t rr = (size_t)(r0 + at + t);
                const float zz = to_f32(z[rr * p.ldz + pch]);
                out[rr * p.ldo + pch] = from_f32<T>(sy[t][pc] * (zz / (1.f + expf(-zz))));
            }
        }
        // (the next chunk's sums are written by the threads that read these, its other arrays were read before the barrier)
    }
    if (mine) {
#pragma unroll
        for (int i = 0; i < DL; ++i)
            if (part * DL + i < p.N) S_glob[i] = S[i];
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
