// Selective scan with a diagonal state per channel (Mamba) over a ragged batch.  Per channel c and state n, with a step dt
// per token and channel and one B and one C row per token:
//
//     S[c, n] <- exp(-dt_c exp(A_log[c, n])) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
//
// and out = y * silu(z).  Everything is fp32 (`out` may be bfloat16: it is the operand of the next product).  The decay is
// taken as 2^(dt a) with a = -exp(A_log) log2(e) made once when the weights are loaded.
//
// A step's tokens are S runs (query_start [S + 1]); run s belongs to state slot slots[s], whose row holds S as [inner, N].
// A block walks one run for CB channels: LPC neighbouring lanes share a channel, each with NS of its states in registers,
// so the loop over tokens has no exchange between lanes at all: a lane leaves its partial of sum_n S C in shared memory
// and the pass that finishes a chunk of CT tokens adds the LPC partials in lane order.  While a chunk is computed the next
// one's inputs travel into registers.  A prompt portion and a single decoded token are the same code (CT 16 and 1), so
// the state after a step does not depend on how the tokens were cut into steps.
#include "common.cuh"

EMBER_DEFINE_LAST_ERROR

namespace ember {

__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

constexpr int SS_THREADS = 128;

struct SelectiveArgs {
    const float* x; int ld_x;                  // [T, inner] after convolution and silu
    const float* dt; int ld_dt;                // [T, inner] steps
    const float* bc; int ld_bc;                // [T, B (N) | C (N)]
    const float* z; int ld_z;                  // [T, inner] gate
    const float* a; const float* skip;         // [inner, N], [inner]
    float* state; long long state_stride;      // [slot][inner][N]
    void* out;                                 // [T, inner]
    const int* query_start; const int* slots;
    int inner, N;
    int vec;                                   // states of a lane lie on vector boundaries in global memory
};

// NS neighbouring floats: the widest vectors NS allows.
template <int NS>
__device__ __forceinline__ void read_row(const float* p, float (&v)[NS]) {
    if (NS % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NS / 4; i++) {
            const float4 f = reinterpret_cast<const float4*>(p)[i];
            v[4 * i] = f.x; v[4 * i + 1] = f.y; v[4 * i + 2] = f.z; v[4 * i + 3] = f.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < NS / 2; i++) {
            const float2 f = reinterpret_cast<const float2*>(p)[i];
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
}
template <int NS>
__device__ __forceinline__ void write_row(float* p, const float (&v)[NS]) {
    if (NS % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NS / 4; i++) reinterpret_cast<float4*>(p)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < NS / 2; i++) reinterpret_cast<float2*>(p)[i] = make_float2(v[2 * i], v[2 * i + 1]);
    }
}
// z sigmoid(z); the bfloat16 form with the fast exponential and division.
template <typename TO>
__device__ __forceinline__ float silu_(float z);
template <>
__device__ __forceinline__ float silu_<float>(float z) { return z / (1.0f + expf(-z)); }
template <>
__device__ __forceinline__ float silu_<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

template <int LPC, int NS, int CT, typename TO>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(SelectiveArgs p) {
    constexpr int CB = SS_THREADS / LPC, NP = LPC * NS;            // channels a block, states a channel (with padding)
    constexpr int EPT = (CT * CB + SS_THREADS - 1) / SS_THREADS;   // (token, channel) elements of a chunk a thread stages
    constexpr int BPT = (2 * CT * NP + SS_THREADS - 1) / SS_THREADS;
    constexpr bool EVEN = CT * CB % SS_THREADS == 0;               // every thread has EPT elements, all of one channel
    static_assert(NS % 2 == 0, "a lane's states are read in pairs or fours");
    extern __shared__ __align__(16) float smem[];
    float2* du = reinterpret_cast<float2*>(smem);      // 2 x [CT][CB] (step, step times input)
    float* bs = smem + 4 * CT * CB;                    // 2 x [CT][NP] pairs (B, C)
    float* yp = bs + 4 * CT * NP;                      // [CT][SS_THREADS] partial read-outs
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.y, c0 = blockIdx.x * CB, inner = p.inner, N = p.N;
    const int cl = threadIdx.x / LPC, l = threadIdx.x % LPC, c = c0 + cl, n0 = l * NS;
    const int first = p.query_start[s], end = p.query_start[s + 1];
    float* S = p.state + (size_t)p.slots[s] * p.state_stride + (size_t)c * N + n0;
    const float* A = p.a + (size_t)c * N + n0;
    // what this thread stages and finishes: tokens threadIdx.x / CB, + SS_THREADS / CB, ... of a chunk, all of channel ec
    const int ec = c0 + threadIdx.x % CB, et = threadIdx.x / CB;
    const bool mine = ec < inner && (EVEN || threadIdx.x < CT * CB);
    const float skip = mine ? p.skip[ec] : 0.0f;
    const float* px = p.x + ec;
    const float* pd = p.dt + ec;
    const float* pz = p.z + ec;

    float fx[EPT], fd[EPT], fz[EPT], fb[BPT], gx[EPT], gz[EPT];
    auto fetch = [&](int t0) {                 // the chunk from t0 on: into registers
#pragma unroll
        for (int e = 0; e < EPT; e++) {
            const int t = t0 + et + e * (SS_THREADS / CB);
            const bool in = mine && t < end;
            fx[e] = in ? px[(size_t)t * p.ld_x] : 0.0f;
            fd[e] = in ? pd[(size_t)t * p.ld_dt] : 0.0f;
            fz[e] = in ? pz[(size_t)t * p.ld_z] : 0.0f;
        }
#pragma unroll
        for (int e = 0; e < BPT; e++) {
            const int i = threadIdx.x + e * SS_THREADS, t = t0 + i / (2 * NP), w = i % (2 * NP), n = w % NP;
            const bool in = (2 * CT * NP % SS_THREADS == 0 || i < 2 * CT * NP) && t < end && n < N;
            fb[e] = in ? p.bc[(size_t)t * p.ld_bc + (w < NP ? 0 : N) + n] : 0.0f;
        }
    };
    auto stage = [&](int buf) {                // and from there into shared memory
#pragma unroll
        for (int e = 0; e < EPT; e++) {
            gx[e] = fx[e];
            gz[e] = fz[e];
            if (EVEN || threadIdx.x < CT * CB) du[buf * CT * CB + threadIdx.x + e * SS_THREADS] = make_float2(fd[e], fd[e] * fx[e]);
        }
#pragma unroll
        for (int e = 0; e < BPT; e++) {
            const int i = threadIdx.x + e * SS_THREADS, w = i % (2 * NP);
            if (2 * CT * NP % SS_THREADS == 0 || i < 2 * CT * NP) bs[(buf * CT + i / (2 * NP)) * 2 * NP + (w % NP) * 2 + w / NP] = fb[e];
        }
    };

    fetch(first);
    float st[NS], a[NS];
    const bool whole = p.vec && c < inner && n0 + NS <= N;
    if (whole) {
        read_row<NS>(S, st);
        read_row<NS>(A, a);
    } else {
#pragma unroll
        for (int i = 0; i < NS; i++) {
            const bool in = c < inner && n0 + i < N;
            st[i] = in ? S[i] : 0.0f;
            a[i] = in ? A[i] : 0.0f;           // (a padded state decays by 1 and gets B = 0: it stays zero)
        }
    }
    stage(0);
    __syncthreads();
    int cur = 0;
    for (int t0 = first; t0 < end; t0 += CT, cur ^= 1) {
        const bool more = t0 + CT < end;
        if (more) fetch(t0 + CT);
        const int n_tok = min(CT, end - t0);
        const float2* dc = du + cur * CT * CB + cl;
        const float* bc = bs + (cur * CT * NP + n0) * 2;
        auto token = [&](int tt) {
            const float2 d = dc[tt * CB];
            float pair[2 * NS];                // B and C in turn
            read_row<2 * NS>(bc + tt * 2 * NP, pair);
            float acc = 0.0f;
#pragma unroll
            for (int i = 0; i < NS; i++) {
                st[i] = fmaf(exp2_approx(d.x * a[i]), st[i], d.y * pair[2 * i]);
                acc = fmaf(st[i], pair[2 * i + 1], acc);
            }
            yp[tt * SS_THREADS + threadIdx.x] = acc;
        };
        if (n_tok == CT) {
#pragma unroll 16
            for (int tt = 0; tt < CT; tt++) token(tt);
        } else {
            for (int tt = 0; tt < n_tok; tt++) token(tt);
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EPT; e++) {
            const int tt = et + e * (SS_THREADS / CB);
            if (mine && tt < n_tok) {
                const float* part = yp + tt * SS_THREADS + (threadIdx.x % CB) * LPC;
                float y = 0.0f;
#pragma unroll
                for (int k = 0; k < LPC / 4; k++) {
                    const float4 f = reinterpret_cast<const float4*>(part)[k];
                    y += f.x; y += f.y; y += f.z; y += f.w;
                }
                y = fmaf(skip, gx[e], y);
                ((TO*)p.out)[(size_t)(t0 + tt) * inner + ec] = from_float<TO>(y * silu_<TO>(gz[e]));
            }
        }
        if (more) stage(cur ^ 1);
        __syncthreads();
    }
    if (whole) write_row<NS>(S, st);
    else {
#pragma unroll
        for (int i = 0; i < NS; i++)
            if (c < inner && n0 + i < N) S[i] = st[i];
    }
}

template <int LPC, int NS, int CT, typename TO>
int launch_selective(const SelectiveArgs& p, int S, cudaStream_t st) {
    constexpr int CB = SS_THREADS / LPC, NP = LPC * NS;
    const size_t smem = (size_t)(4 * CT * CB + 4 * CT * NP + CT * SS_THREADS) * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<LPC, NS, CT, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("selective_scan: shared memory %zu: %s", smem, cudaGetErrorString(e));
    }
    SelectiveArgs q = p;
    constexpr int VW = NS % 4 == 0 ? 4 : 2;
    q.vec = p.N % VW == 0 && p.state_stride % VW == 0 && ((((uintptr_t)p.state) | ((uintptr_t)p.a)) & 15) == 0;
    launch_kernel(selective_scan_kernel<LPC, NS, CT, TO>, dim3((p.inner + CB - 1) / CB, S), SS_THREADS, smem, st, q);
    return check_launch("selective_scan");
}

// Lanes a channel and states a lane by the number of states.
template <int CT, typename TO>
int pick_selective(const SelectiveArgs& p, int S, cudaStream_t st) {
    const int N = p.N;
    if (N <= 8) return launch_selective<4, 2, CT, TO>(p, S, st);
    if (N <= 16) return launch_selective<8, 2, CT, TO>(p, S, st);
    if (N <= 32) return launch_selective<8, 4, CT, TO>(p, S, st);
    if (N <= 64) return launch_selective<16, 4, CT, TO>(p, S, st);
    if (N <= 128) return launch_selective<32, 4, CT, TO>(p, S, st);
    return launch_selective<32, 8, CT, TO>(p, S, st);
}

}  // namespace ember

using namespace ember;

EMBER_API int ember_selective_scan_max_states() { return 256; }

// T == S (every run is one token): the form with chunks of one token.
EMBER_API int ember_selective_scan(const float* x, int ld_x, const float* dt, int ld_dt, const float* bc, int ld_bc, const float* z, int ld_z,
                                   const float* a, const float* skip, float* state, long long state_stride,
                                   void* out, int out_dtype, const int* query_start, const int* slots, int T, int S, int inner, int N,
                                   void* stream) {
    if (T <= 0 || S <= 0) return 0;
    if (inner <= 0 || N <= 0 || N > ember_selective_scan_max_states()) return fail("selective_scan: %d channels of %d states (at most %d)", inner, N, ember_selective_scan_max_states());
    if (ld_x < inner || ld_dt < inner || ld_z < inner || ld_bc < 2 * N || state_stride < (long long)inner * N)
        return fail("selective_scan: rows of %d / %d / %d / %d, state rows of %lld do not hold %d channels of %d states", ld_x, ld_dt, ld_z, ld_bc, state_stride, inner, N);
    if (S > 65535) return fail("selective_scan: %d runs are too many for one launch", S);
    SelectiveArgs p{x, ld_x, dt, ld_dt, bc, ld_bc, z, ld_z, a, skip, state, state_stride, out, query_start, slots, inner, N, 0};
    cudaStream_t st = (cudaStream_t)stream;
    const bool single = T == S;
    if (out_dtype == EMBER_F32) return single ? pick_selective<1, float>(p, S, st) : pick_selective<16, float>(p, S, st);
    if (out_dtype == EMBER_BF16) return single ? pick_selective<1, __nv_bfloat16>(p, S, st) : pick_selective<16, __nv_bfloat16>(p, S, st);
    return fail("selective_scan: unsupported output dtype %d", out_dtype);
}
