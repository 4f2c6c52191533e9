// Selective scan with a diagonal state per channel (Mamba) over a ragged batch.  With a step d = softplus(raw step + bias) per
// token and channel, and one B and one C row per token,
//
//     M[n, c] <- e^(-d_c a[n, c]) M[n, c] + d_c u_c B[n];   r_c = <M[:, c], C> + D_c u_c
//
// and out = r * silu(z).  Everything is fp32 (`out` may be bfloat16: it is the operand of the next product).  The decay is
// taken as a power of two, whose exponents' factor -a log2(e) is made once when the weights are loaded.
//
// A step's tokens are S runs (query_start [S + 1]); run s belongs to state slot slots[s], whose row holds M as [N, inner]
// (neighbouring channels side by side, like every other operand).  A block walks one run for 32 channels: a lane is a
// channel, and the block's NW warps share its states, NS each, in registers.  A token's B and C are then the same address for
// a whole warp, the loop over tokens has no exchange between threads at all, and a warp leaves its partials of the read-out in
// shared memory for the pass that finishes a chunk of CT tokens, which adds the warps' partials in order.  (With neighbouring
// lanes sharing a channel the B and C reads were four shared-memory wavefronts a warp and token and bounded the kernel.)
// States go two by two through packed fp32 arithmetic.  More warps bring the inputs, by cp.async into a ring of
// chunks some way ahead (what a block has in flight is what keeps the memory busy: with one chunk in flight the kernel waited
// for it), and finish the chunk before (sums, gate, store) while a chunk is computed: one barrier a chunk.
// A step whose runs are single tokens takes a kernel of its own, a thread a channel with all its states.
#include "common.cuh"

EMBER_DEFINE_LAST_ERROR

namespace ember {

__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

constexpr int SS_CHUNK = 32;          // tokens a chunk
constexpr int SS_STEPS = 4;           // tokens a turn of the computing loop
constexpr int SS_RING = 5;            // chunks of inputs in shared memory: one being finished, one computed, the rest on their way

struct SelectiveArgs {
    const float* x; int ld_x;                  // [T, inner] after convolution and silu
    const float* dt; int ld_dt;                // [T, inner] raw steps
    const float* bc; int ld_bc;                // [T, B (N) | C (N)]
    const float* z; int ld_z;                  // [T, inner] gate
    const float* dt_bias; const float* a; const float* skip;      // [inner], [N, inner], [inner]
    float* state; long long state_stride;      // [slot][N][inner]
    void* out;                                 // [T, inner]
    const int* query_start; const int* slots;
    int inner, N;
    int by16, bc16;                            // rows of x, dt and z, and of B and C, can be copied 16 bytes at a time
};

// Packed fp32 pairs.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pk2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "r"(__float_as_uint(lo)), "r"(__float_as_uint(hi)));
    return r;
}
__device__ __forceinline__ float2 up2(f32x2 v) {
    uint32_t lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=r"(lo), "=r"(hi) : "l"(v));
    return make_float2(__uint_as_float(lo), __uint_as_float(hi));
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
// softplus(z) = log(1 + e^z).  The bfloat16 form takes the logarithm's series where e^z is small (the fast logarithm has no
// relative precision near 1): an error of a few 1e-6.
template <typename TO>
__device__ __forceinline__ float softplus_(float z);
template <>
__device__ __forceinline__ float softplus_<float>(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
template <>
__device__ __forceinline__ float softplus_<__nv_bfloat16>(float z) {
    const float e = __expf(z);
    const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 1.0f / 3.0f), -0.5f), 1.0f);
    return z > 20.0f ? z : (e < 0.0625f ? series : __logf(1.0f + e));
}
// z sigmoid(z); the bfloat16 form with the fast exponential and division.
template <typename TO>
__device__ __forceinline__ float silu_(float z);
template <>
__device__ __forceinline__ float silu_<float>(float z) { return z / (1.0f + expf(-z)); }
template <>
__device__ __forceinline__ float silu_<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// NS neighbouring floats of shared memory in the widest reads NS allows.
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
__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// NW warps compute, NH warps feed them and finish what they leave.
template <int NW, int NS, int NH, int CT, int RING, typename TO>
__global__ void __launch_bounds__(32 * (NW + NH)) selective_scan_kernel(SelectiveArgs p) {
    constexpr int THREADS = 32 * NW, FEED = 32 * NH, NP = NW * NS, N2 = NS / 2;    // states a channel (with padding); pairs a thread
    constexpr int TILE = CT * 32;                                  // a chunk's elements of x, of dt and of z
    static_assert(NS % 2 == 0 && RING >= 4, "states go two by two");
    extern __shared__ __align__(16) float smem[];
    float* xs = smem;                                  // RING x [x | dt | z] x [CT][32]
    float* bs = xs + RING * 3 * TILE;                  // RING x [CT][B (NP) | C (NP)]
    float* yp = bs + RING * CT * NP * 2;               // 2 x [CT][NW][32] partial read-outs
    pdl_launch_dependents();
    const int s = blockIdx.y, inner = p.inner, N = p.N;
    const int lane = threadIdx.x & 31, c0 = blockIdx.x * 32, c = c0 + lane;
    const bool feeds = threadIdx.x >= THREADS;
    const int warp = (threadIdx.x >> 5) - (feeds ? NW : 0), tid = threadIdx.x - (feeds ? THREADS : 0);
    if (N < NP)                                        // (B and C of padded states stay zero)
        for (int i = threadIdx.x; i < RING * CT * NP * 2; i += THREADS + FEED) bs[i] = 0.0f;
    __syncthreads();
    pdl_wait();
    const int first = p.query_start[s], end = p.query_start[s + 1];
    const int chunks = (end - first + CT - 1) / CT;
    const bool live = c < inner;
    if (feeds) {
        const float skip = live ? p.skip[c] : 0.0f;
        const int n4 = N / 4;
        auto issue = [&](int i) {              // the inputs of chunk i on their way
            const int t0 = first + i * CT, n_tok = min(CT, end - t0);
            if (n_tok > 0) {
                float* xd = xs + (i % RING) * 3 * TILE;
                auto tile = [&](float* dst, const float* src, int ld) {
                    src += (size_t)t0 * ld + c0;
                    if (p.by16) {
#pragma unroll
                        for (int r = tid; r < CT * 8; r += FEED)
                            if (r / 8 < n_tok && c0 + (r % 8) * 4 < inner) copy16(dst + r * 4, src + (r / 8) * (size_t)ld + (r % 8) * 4);
                    } else {
                        for (int r = tid; r < TILE; r += FEED)
                            if (r / 32 < n_tok && live) copy4(dst + r, src + (r / 32) * (size_t)ld + lane);
                    }
                };
                tile(xd, p.x, p.ld_x);
                tile(xd + TILE, p.dt, p.ld_dt);
                tile(xd + 2 * TILE, p.z, p.ld_z);
                float* bd = bs + (i % RING) * CT * NP * 2;
                const float* src = p.bc + (size_t)t0 * p.ld_bc;
                if (p.bc16) {
                    constexpr int P4 = NP / 2;                     // 16-byte pieces of a token's B and C (with padding)
#pragma unroll
                    for (int r = tid; r < CT * P4; r += FEED) {
                        const int tt = r / P4, w = r % P4, n = w % (P4 / 2);
                        if (tt < n_tok && n < n4) copy16(bd + r * 4, src + (size_t)tt * p.ld_bc + (w < P4 / 2 ? 0 : N) + n * 4);
                    }
                } else {
                    for (int r = tid; r < CT * 2 * NP; r += FEED) {
                        const int tt = r / (2 * NP), w = r % (2 * NP), n = w % NP;
                        if (tt < n_tok && n < N) copy4(bd + r, src + (size_t)tt * p.ld_bc + (w < NP ? 0 : N) + n);
                    }
                }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        const float dt_bias = live ? p.dt_bias[c] : 0.0f;
        auto arrived = [&](int i) {            // chunk i is there: raw steps become steps
            asm volatile("cp.async.wait_group %0;" ::"n"(RING - 3) : "memory");
            asm volatile("bar.sync 1, %0;" ::"n"(FEED) : "memory");      // (pieces that other feeding threads copied)
            if (i < chunks) {
                float* xd = xs + (i % RING) * 3 * TILE + TILE + lane;
#pragma unroll
                for (int tt = warp; tt < CT; tt += NH) xd[tt * 32] = softplus_<TO>(xd[tt * 32] + dt_bias);
            }
        };
        auto finish = [&](int i) {             // chunk i: its partials, gate, store
            const int t0 = first + i * CT, n_tok = min(CT, end - t0);
            const float* xd = xs + (i % RING) * 3 * TILE + lane;
            const float* yc = yp + (i & 1) * CT * THREADS + lane;
#pragma unroll
            for (int tt = warp; tt < CT; tt += NH) {
                if (live && tt < n_tok) {
                    const float* part = yc + tt * THREADS;
                    float y0 = 0.0f, y1 = 0.0f;
#pragma unroll
                    for (int k = 0; k < NW; k += 2) { y0 += part[k * 32]; y1 += part[(k + 1) * 32]; }
                    const float y = fmaf(skip, xd[tt * 32], y0 + y1);
                    ((TO*)p.out)[(size_t)(t0 + tt) * inner + c] = from_float<TO>(y * silu_<TO>(xd[2 * TILE + tt * 32]));
                }
            }
        };
        for (int i = 0; i < RING - 2; i++) issue(i);
        arrived(0);
        __syncthreads();
        for (int i = 0; i < chunks; i++) {
            issue(i + RING - 2);               // (into the place of chunk i - 2, which has been finished)
            if (i > 0) finish(i - 1);
            arrived(i + 1);
            __syncthreads();
        }
        finish(chunks - 1);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        return;
    }
    const int n0 = warp * NS;
    float* S = p.state + (size_t)p.slots[s] * p.state_stride + c;
    const float* A = p.a + c;
    f32x2 st[N2], a[N2];
#pragma unroll
    for (int i = 0; i < N2; i++) {             // (a padded state decays by 1 and gets B = 0: it stays zero)
        const int n = n0 + 2 * i;
        const bool in0 = live && n < N, in1 = live && n + 1 < N;
        st[i] = pk2(in0 ? S[(size_t)n * inner] : 0.0f, in1 ? S[(size_t)(n + 1) * inner] : 0.0f);
        a[i] = pk2(in0 ? A[(size_t)n * inner] : 0.0f, in1 ? A[(size_t)(n + 1) * inner] : 0.0f);
    }
    __syncthreads();
    for (int i = 0; i < chunks; i++) {
        const int n_tok = min(CT, end - first - i * CT);
        const float* xc = xs + (i % RING) * 3 * TILE + lane;
        const float* bc = bs + (i % RING) * CT * 2 * NP + n0;
        float* yc = yp + (i & 1) * CT * THREADS + warp * 32 + lane;
        // A token in three steps, each one token behind the one before: its operands from shared memory, its decays and inputs,
        // the state.  (Left to the compiler the steps of a token follow one another, and a warp waits out every latency of
        // it.)  The two tokens looked at past the chunk's end lie in the ring and are not used.
        struct Operands { float d, x; float B[NS], C[NS]; };
        struct Prepared { f32x2 decay[N2], in[N2], out[N2]; };
        auto load = [&](int k) {
            Operands o;
            o.d = xc[TILE + k * 32];
            o.x = xc[k * 32];
            read_row<NS>(bc + k * 2 * NP, o.B);                                  // (the same addresses for the whole warp)
            read_row<NS>(bc + k * 2 * NP + NP, o.C);
            return o;
        };
        auto prepare = [&](const Operands& o) {
            Prepared t;
            const float u = o.d * o.x;
            const f32x2 dd = pk2(o.d, o.d), uu = pk2(u, u);
#pragma unroll
            for (int j = 0; j < N2; j++) {
                const float2 e = up2(mul2(dd, a[j]));
                t.decay[j] = pk2(exp2_approx(e.x), exp2_approx(e.y));
                t.in[j] = mul2(uu, pk2(o.B[2 * j], o.B[2 * j + 1]));
                t.out[j] = pk2(o.C[2 * j], o.C[2 * j + 1]);
            }
            return t;
        };
        Operands ahead = load(0);
        Prepared ready = prepare(ahead);
        ahead = load(1);
#pragma unroll SS_STEPS
        for (int k = 0; k < n_tok; k++) {
            const Prepared t = ready;
            ready = prepare(ahead);
            ahead = load(k + 2);
            f32x2 acc;
#pragma unroll
            for (int j = 0; j < N2; j++) {
                st[j] = fma2(t.decay[j], st[j], t.in[j]);
                acc = j == 0 ? mul2(st[j], t.out[j]) : fma2(st[j], t.out[j], acc);
            }
            const float2 r = up2(acc);
            yc[k * THREADS] = r.x + r.y;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < N2; i++) {
        const int n = n0 + 2 * i;
        const float2 v = up2(st[i]);
        if (live && n < N) S[(size_t)n * inner] = v.x;
        if (live && n + 1 < N) S[(size_t)(n + 1) * inner] = v.y;
    }
}

// One token a run: a thread takes a channel with all its states, ST of them in flight at a time.
constexpr int SS_STEP_THREADS = 128;
template <int ST, typename TO>
__global__ void __launch_bounds__(SS_STEP_THREADS) selective_step_kernel(SelectiveArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.y, inner = p.inner, N = p.N, c = blockIdx.x * SS_STEP_THREADS + threadIdx.x;
    if (c >= inner) return;
    const int t = p.query_start[s];
    float* S = p.state + (size_t)p.slots[s] * p.state_stride + c;
    const float* A = p.a + c;
    const float* bc = p.bc + (size_t)t * p.ld_bc;
    const float x = p.x[(size_t)t * p.ld_x + c], d = softplus_<TO>(p.dt[(size_t)t * p.ld_dt + c] + p.dt_bias[c]), z = p.z[(size_t)t * p.ld_z + c], skip = p.skip[c];
    const float u = d * x;
    float y0 = 0.0f, y1 = 0.0f;
    for (int n0 = 0; n0 < N; n0 += ST) {
        float st[ST], a[ST];
#pragma unroll
        for (int i = 0; i < ST; i++) {
            const bool in = n0 + i < N;
            st[i] = in ? S[(size_t)(n0 + i) * inner] : 0.0f;
            a[i] = in ? A[(size_t)(n0 + i) * inner] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < ST; i++) {
            const bool in = n0 + i < N;
            st[i] = fmaf(exp2_approx(d * a[i]), st[i], u * (in ? bc[n0 + i] : 0.0f));
            float& y = i & 1 ? y1 : y0;
            y = fmaf(st[i], in ? bc[N + n0 + i] : 0.0f, y);
            if (in) S[(size_t)(n0 + i) * inner] = st[i];
        }
    }
    ((TO*)p.out)[(size_t)t * inner + c] = from_float<TO>(fmaf(skip, x, y0 + y1) * silu_<TO>(z));
}

template <int NW, int NS, int NH, int CT, typename TO, int RING = SS_RING>
int launch_selective(const SelectiveArgs& p, int S, cudaStream_t st) {
    const size_t smem = (size_t)(RING * 3 * CT * 32 + RING * 2 * CT * NW * NS + 2 * CT * NW * 32) * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<NW, NS, NH, CT, RING, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("selective_scan: shared memory %zu: %s", smem, cudaGetErrorString(e));
    }
    launch_kernel(selective_scan_kernel<NW, NS, NH, CT, RING, TO>, dim3((p.inner + 31) / 32, S), 32 * (NW + NH), smem, st, p);
    return check_launch("selective_scan");
}

// Computing warps a block, states a thread and feeding warps by the number of states.  (Sixteen states, 2,048 tokens of 4,096
// channels: four warps of four states 103 us, eight of two 105, and when blocks share SMs four runs of 512 tokens 86 us either
// way: what is left is the instructions of both kinds of warps, 0.7 of the issue slots of the SMs that have a block.)
template <typename TO>
int pick_selective(const SelectiveArgs& p, int S, bool single, cudaStream_t st) {
    const int N = p.N;
    if (single) {
        const dim3 grid((p.inner + SS_STEP_THREADS - 1) / SS_STEP_THREADS, S);
        if (N <= 8) launch_kernel(selective_step_kernel<8, TO>, grid, SS_STEP_THREADS, 0, st, p);
        else launch_kernel(selective_step_kernel<16, TO>, grid, SS_STEP_THREADS, 0, st, p);
        return check_launch("selective_step");
    }
    if (N <= 8) return launch_selective<4, 2, 8, SS_CHUNK, TO>(p, S, st);
    if (N <= 16) return launch_selective<4, 4, 8, SS_CHUNK, TO>(p, S, st);
    if (N <= 32) return launch_selective<8, 4, 8, SS_CHUNK, TO>(p, S, st);
    if (N <= 64) return launch_selective<8, 8, 8, SS_CHUNK, TO>(p, S, st);
    if (N <= 128) return launch_selective<8, 16, 8, 16, TO, 4>(p, S, st);
    return launch_selective<16, 16, 8, 16, TO, 4>(p, S, st);
}

}  // namespace ember

using namespace ember;

EMBER_API int ember_selective_scan_max_states() { return 256; }

// T == S (every run is one token): the form with chunks of one token.
EMBER_API int ember_selective_scan(const float* x, int ld_x, const float* dt, int ld_dt, const float* bc, int ld_bc, const float* z, int ld_z,
                                   const float* dt_bias, const float* a, const float* skip, float* state, long long state_stride,
                                   void* out, int out_dtype, const int* query_start, const int* slots, int T, int S, int inner, int N,
                                   void* stream) {
    if (T <= 0 || S <= 0) return 0;
    if (inner <= 0 || N <= 0 || N > ember_selective_scan_max_states()) return fail("selective_scan: %d channels of %d states (at most %d)", inner, N, ember_selective_scan_max_states());
    if (ld_x < inner || ld_dt < inner || ld_z < inner || ld_bc < 2 * N || state_stride < (long long)inner * N)
        return fail("selective_scan: rows of %d / %d / %d / %d, state rows of %lld do not hold %d channels of %d states", ld_x, ld_dt, ld_z, ld_bc, state_stride, inner, N);
    if (S > 65535) return fail("selective_scan: %d runs are too many for one launch", S);
    SelectiveArgs p{x, ld_x, dt, ld_dt, bc, ld_bc, z, ld_z, dt_bias, a, skip, state, state_stride, out, query_start, slots, inner, N, 0, 0};
    p.by16 = inner % 4 == 0 && ld_x % 4 == 0 && ld_dt % 4 == 0 && ld_z % 4 == 0 && ((((uintptr_t)x) | ((uintptr_t)dt) | ((uintptr_t)z)) & 15) == 0;
    p.bc16 = N % 4 == 0 && ld_bc % 4 == 0 && (((uintptr_t)bc) & 15) == 0;
    cudaStream_t st = (cudaStream_t)stream;
    const bool single = T == S;
    if (out_dtype == EMBER_F32) return pick_selective<float>(p, S, single, st);
    if (out_dtype == EMBER_BF16) return pick_selective<__nv_bfloat16>(p, S, single, st);
    return fail("selective_scan: unsupported output dtype %d", out_dtype);
}
