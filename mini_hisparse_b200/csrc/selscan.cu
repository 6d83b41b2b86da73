// Recurrences whose gates read the current token only.
//
//   mingru_scan   per channel: z = sigmoid(zl + bz), u = xl + bx, c = u >= 0 ? u + 1/2 : sigmoid(u),
//                 S <- (1 - z) S + z c, out = S silu(gl): zl, xl, gl are columns of one float32 product
//   selective_split   from the product x W^T = [dt : rank | B : N | C : N] (possibly split-K parts): dt's columns in the
//                 compute dtype (padded with zeros), B and C as float32 rows
//   selective_scan    per channel c and state n (selective scan): dt = softplus(dtl_c + bias_c),
//                 S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x_c B_n,  y_c = sum_n S[c, n] C_n + D_c x_c,
//                 out = y silu(zl) * scale
//
// States are float32 and live in a request's slot; a segment that starts at position 0 starts from zero.  Inputs that
// come as split-K parts are summed in index order.
#include "common.cuh"

using namespace mhb;

MHB_EXPORT const char* mhb_last_error() { return error_buffer(); }

namespace {

// columns of a float32 matrix [T][ld] that may come as parts
struct Cols {
    const float* p;
    int nsplit;
    size_t stride;
    int ld;
    __device__ __forceinline__ float at(int row, int col) const {
        const float* q = p + (size_t)row * ld + col;
        float v = *q;
#pragma unroll 4
        for (int s = 1; s < nsplit; ++s) v += q[(size_t)s * stride];
        return v;
    }
};

__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float siluf(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplusf(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// ---- minGRU --------------------------------------------------------------------------------------------
struct GruArgs {
    Cols z, x, g;
    const float* bz;
    const float* bx;
    float* state;            // [slots][state_stride]: [W]
    size_t state_stride;
    const int* seg_offset;
    const int* seg_slot;
    const int* positions;
    void* out;               // [T][W]
    int W, writable;
};

__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoidf(u); }

// few tokens per segment: a thread per channel walks them
template <typename OT>
__global__ void __launch_bounds__(64)
mingru_walk_kernel(const GruArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, seg = blockIdx.y;
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    if (c >= a.W || t0 >= t1) return;
    float* slot = a.state + (size_t)a.seg_slot[seg] * a.state_stride;
    float S = a.positions[t0] == 0 ? 0.f : slot[c];
    const float bz = a.bz[c], bx = a.bx[c];
#pragma unroll 2
    for (int t = t0; t < t1; ++t) {
        const float z = sigmoidf(a.z.at(t, c) + bz), cand = gru_candidate(a.x.at(t, c) + bx), g = a.g.at(t, c);
        S = (1.f - z) * S + z * cand;
        ((OT*)a.out)[(size_t)t * a.W + c] = from_float<OT>(S * siluf(g));
    }
    if (a.writable) slot[c] = S;
}

// long segments: LANES lanes of time per channel, each RUN tokens in registers; a lane folds its run into (decay, sum),
// a warp per channel scans the lanes, and every lane walks its run again from its carry
constexpr int GRU_CH = 16, GRU_LANES = 64, GRU_RUN = 8;

template <typename OT>
__global__ void __launch_bounds__(GRU_CH * GRU_LANES)
mingru_scan_kernel(const GruArgs a) {
    __shared__ float fold_a[GRU_CH][GRU_LANES + 1], fold_b[GRU_CH][GRU_LANES + 1], carry[GRU_CH];
    pdl_launch_dependents();
    pdl_wait();
    const int cl = threadIdx.x % GRU_CH, lane_t = threadIdx.x / GRU_CH;
    const int c = blockIdx.x * GRU_CH + cl, seg = blockIdx.y;
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    if (t0 >= t1) return;
    const bool live = c < a.W;
    float* slot = a.state + (size_t)a.seg_slot[seg] * a.state_stride;
    if (lane_t == 0) carry[cl] = (live && a.positions[t0] != 0) ? slot[c] : 0.f;
    const float bz = live ? a.bz[c] : 0.f, bx = live ? a.bx[c] : 0.f;
    for (int r0 = t0; r0 < t1; r0 += GRU_LANES * GRU_RUN) {
        const int mine = r0 + lane_t * GRU_RUN;
        float da[GRU_RUN], db[GRU_RUN], g[GRU_RUN];
#pragma unroll
        for (int i = 0; i < GRU_RUN; ++i) {
            const int t = mine + i;
            const bool ok = live && t < t1;
            da[i] = ok ? a.z.at(t, c) : 0.f;
            db[i] = ok ? a.x.at(t, c) : 0.f;
            g[i] = ok ? a.g.at(t, c) : 0.f;
        }
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int i = 0; i < GRU_RUN; ++i) {
            if (mine + i < t1) {
                const float z = sigmoidf(da[i] + bz), cand = gru_candidate(db[i] + bx);
                da[i] = 1.f - z;
                db[i] = z * cand;
            } else {
                da[i] = 1.f;
                db[i] = 0.f;
            }
            A *= da[i];
            B = fmaf(da[i], B, db[i]);
        }
        fold_a[cl][lane_t] = A;
        fold_b[cl][lane_t] = B;
        __syncthreads();
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
        if (warp < GRU_CH) {                     // channel `warp`: two neighbouring runs per lane
            const float a0 = fold_a[warp][2 * lane], b0 = fold_b[warp][2 * lane];
            const float a1 = fold_a[warp][2 * lane + 1], b1 = fold_b[warp][2 * lane + 1];
            float pa = a0 * a1, pb = fmaf(a1, b0, b1);
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
                if (lane >= o) { pb = fmaf(pa, qb, pb); pa *= qa; }
            }
            const float S0 = carry[warp];
            const float ea = __shfl_up_sync(0xffffffffu, pa, 1), eb = __shfl_up_sync(0xffffffffu, pb, 1);
            const float before = lane ? fmaf(ea, S0, eb) : S0;
            fold_b[warp][2 * lane] = before;                          // what each run starts from
            fold_b[warp][2 * lane + 1] = fmaf(a0, before, b0);
            __syncwarp();
            if (lane == 31) carry[warp] = fmaf(pa, S0, pb);
        }
        __syncthreads();
        float S = fold_b[cl][lane_t];
#pragma unroll
        for (int i = 0; i < GRU_RUN; ++i) {
            S = fmaf(da[i], S, db[i]);
            if (live && mine + i < t1) ((OT*)a.out)[(size_t)(mine + i) * a.W + c] = from_float<OT>(S * siluf(g[i]));
        }
        __syncthreads();                         // the folds are free for the next round
    }
    if (a.writable && lane_t == 0 && live) slot[c] = carry[cl];
}

// ---- selective scan: the three column groups of the small product ------------------------------------------
template <typename OT>
__global__ void selective_split_kernel(Cols p, int rank, int N, OT* __restrict__ dt, int dt_ld, float* __restrict__ bc, int T) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < dt_ld; i += blockDim.x) dt[(size_t)t * dt_ld + i] = from_float<OT>(i < rank ? p.at(t, i) : 0.f);
    for (int i = threadIdx.x; i < 2 * N; i += blockDim.x) bc[(size_t)t * 2 * N + i] = p.at(t, rank + i);
}

struct ScanArgs {
    Cols z;                  // [T][>= C]: the output gate's columns
    Cols dt;                 // [T][>= C]: the step's logits (FUSE_DT: the small product, columns 0 .. rank - 1)
    Cols bc;                 // [T]: B in columns 0 .. N - 1, C in N .. 2 N - 1
    const float* x;          // [T][C]
    const void* dt_weight;   // FUSE_DT: [C][rank] compute dtype
    int rank, rank_ld;
    const float* dt_bias;    // [C]
    const float* A2;         // [C][N]: A log2(e)
    const float* D;          // [C]
    float* state;            // [slots][state_stride]: [C][N]
    size_t state_stride;
    const int* seg_offset;
    const int* seg_slot;
    const int* positions;
    void* out;               // [T][C]
    float scale;
    int C, N, writable;
};

__device__ __forceinline__ void copy_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// LPC lanes share a channel, each RPL states in registers (N <= LPC * RPL).  CH tokens are staged at once: dt and dt x
// per channel (softplus is taken once, by the thread that loads the element, which also finishes the element's output),
// B and C per state by cp.async while the CH tokens before are walked.
template <int LPC, int RPL, int CH, int THREADS, bool FUSE_DT, typename WT, typename OT>
__global__ void __launch_bounds__(THREADS)
selective_scan_kernel(const ScanArgs a) {
    constexpr int CPB = THREADS / LPC;                           // channels per CTA
    constexpr int RUN = RPL % 4 == 0 ? RPL + 4 : (RPL | 1);      // a lane's states in shared memory, padded against bank conflicts
    constexpr int E = (CH * CPB + THREADS - 1) / THREADS;        // elements a thread loads per stage
    __shared__ __align__(16) float Bs[2][CH][LPC * RUN];
    __shared__ __align__(16) float Cs[2][CH][LPC * RUN];
    __shared__ float dts[CH][CPB], dxs[CH][CPB], ys[CH][CPB];
    extern __shared__ float low[];                               // FUSE_DT: [CH][rank]
    pdl_launch_dependents();
    const int seg = blockIdx.y, c0 = blockIdx.x * CPB;
    const int sub = threadIdx.x % LPC, cl = threadIdx.x / LPC, c = c0 + cl;
    const int N = a.N;
    float A2[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int n = sub * RPL + r;
        A2[r] = (c < a.C && n < N) ? a.A2[(size_t)c * N + n] : 0.f;
    }
    for (int i = threadIdx.x; i < 2 * CH * LPC * RUN; i += THREADS) { (&Bs[0][0][0])[i] = 0.f; (&Cs[0][0][0])[i] = 0.f; }
    pdl_wait();
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    if (t0 >= t1) return;
    __syncthreads();
    auto stage_bc = [&](int st, int b) {
        const int n = min(CH, t1 - b);
        for (int i = threadIdx.x; i < n * 2 * N; i += THREADS) {
            const int tt = i / (2 * N), k = i - tt * 2 * N;
            const int s = k < N ? k : k - N;
            float* dst = (k < N ? &Bs[st][tt][0] : &Cs[st][tt][0]) + (s / RPL) * RUN + s % RPL;
            if (a.bc.nsplit == 1) copy_async4(dst, a.bc.p + (size_t)(b + tt) * a.bc.ld + k);
            else *dst = a.bc.at(b + tt, k);
        }
    };
    // this thread's elements of a stage: token tt, channel k
    float dt_r[E], x_r[E], z_r[E];
    auto load_elements = [&](int b) {
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
            const bool ok = tt < CH && b + tt < t1 && c0 + k < a.C;
            x_r[e] = ok ? a.x[(size_t)(b + tt) * a.C + c0 + k] : 0.f;
            z_r[e] = ok ? a.z.at(b + tt, c0 + k) : 0.f;
            if constexpr (!FUSE_DT) dt_r[e] = ok ? a.dt.at(b + tt, c0 + k) : 0.f;
        }
    };
    stage_bc(0, t0);
    copy_async_commit();
    load_elements(t0);
    float* slot = a.state + (size_t)a.seg_slot[seg] * a.state_stride;
    const bool fresh = a.positions[t0] == 0;
    float S[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int n = sub * RPL + r;
        S[r] = (!fresh && c < a.C && n < N) ? slot[(size_t)c * N + n] : 0.f;
    }
    int st = 0;
    for (int b = t0; b < t1; b += CH, st ^= 1) {
        const int n = min(CH, t1 - b);
        if constexpr (FUSE_DT) {
            // the step's logits from the rank columns: the lanes of a channel split the dot product
            for (int i = threadIdx.x; i < n * a.rank; i += THREADS) low[i] = a.dt.at(b + i / a.rank, i % a.rank);
            __syncthreads();
            const WT* w = (const WT*)a.dt_weight + (size_t)c * a.rank_ld;
            for (int tt = 0; tt < n; ++tt) {
                float d = 0.f;
                if (c < a.C)
                    for (int i = sub; i < a.rank; i += LPC) d = fmaf(to_float(w[i]), low[tt * a.rank + i], d);
#pragma unroll
                for (int o = 1; o < LPC; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
                if (sub == 0) dts[tt][cl] = d;
            }
            __syncthreads();
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
                dt_r[e] = tt < n ? dts[tt][k] : 0.f;
            }
        }
        float xd[E], zd[E];
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
            if (tt < n) {
                const float dt = c0 + k < a.C ? softplusf(dt_r[e] + a.dt_bias[c0 + k]) : 0.f;
                dts[tt][k] = dt;
                dxs[tt][k] = dt * x_r[e];
            }
            xd[e] = x_r[e];
            zd[e] = z_r[e];
        }
        copy_async_wait<0>();
        __syncthreads();
        if (b + CH < t1) {
            stage_bc(st ^ 1, b + CH);
            load_elements(b + CH);
        }
        copy_async_commit();
#pragma unroll 4
        for (int tt = 0; tt < n; ++tt) {
            const float dt = dts[tt][cl], dx = dxs[tt][cl];
            float Bv[RPL], Cv[RPL];
            const float* bp = &Bs[st][tt][sub * RUN];
            const float* cp = &Cs[st][tt][sub * RUN];
            if constexpr (RPL % 4 == 0) {
#pragma unroll
                for (int r = 0; r < RPL; r += 4) {
                    const float4 p = *(const float4*)(bp + r), q = *(const float4*)(cp + r);
                    Bv[r] = p.x; Bv[r + 1] = p.y; Bv[r + 2] = p.z; Bv[r + 3] = p.w;
                    Cv[r] = q.x; Cv[r + 1] = q.y; Cv[r + 2] = q.z; Cv[r + 3] = q.w;
                }
            } else {
#pragma unroll
                for (int r = 0; r < RPL; ++r) { Bv[r] = bp[r]; Cv[r] = cp[r]; }
            }
            float y = 0.f;
#pragma unroll
            for (int r = 0; r < RPL; ++r) {
                S[r] = fmaf(exp2_fast(dt * A2[r]), S[r], dx * Bv[r]);
                y = fmaf(S[r], Cv[r], y);
            }
#pragma unroll
            for (int o = 1; o < LPC; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (sub == 0) ys[tt][cl] = y;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
            if (tt < n && c0 + k < a.C)
                ((OT*)a.out)[(size_t)(b + tt) * a.C + c0 + k] =
                    from_float<OT>((ys[tt][k] + a.D[c0 + k] * xd[e]) * siluf(zd[e]) * a.scale);
        }
    }
    copy_async_wait<0>();
    if (a.writable)
#pragma unroll
        for (int r = 0; r < RPL; ++r) {
            const int n = sub * RPL + r;
            if (c < a.C && n < N) slot[(size_t)c * N + n] = S[r];
        }
}

template <int LPC, int RPL, int CH, bool FUSE_DT, typename WT, typename OT>
int launch_scan(const ScanArgs& a, int S, cudaStream_t stream) {
    constexpr int THREADS = 64;
    constexpr int CPB = THREADS / LPC;
    auto kern = selective_scan_kernel<LPC, RPL, CH, THREADS, FUSE_DT, WT, OT>;
    const size_t smem = FUSE_DT ? sizeof(float) * CH * (size_t)a.rank : 0;
    if (smem > 16 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("selective_scan: a rank of %d: %s", a.rank, cudaGetErrorString(e));
    }
    launch_kernel(kern, dim3((a.C + CPB - 1) / CPB, S), dim3(THREADS), smem, stream, a);
    return check_launch("selective_scan");
}

template <bool FUSE_DT, typename WT, typename OT>
int pick_scan(const ScanArgs& a, int S, cudaStream_t stream) {
    if (a.N <= 8) return launch_scan<4, 2, 16, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 16) return launch_scan<4, 4, 16, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 24) return launch_scan<4, 6, 16, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 32) return launch_scan<4, 8, 16, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 64) return launch_scan<8, 8, 16, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 128) return launch_scan<16, 8, 8, FUSE_DT, WT, OT>(a, S, stream);
    if (a.N <= 256) return launch_scan<32, 8, 4, FUSE_DT, WT, OT>(a, S, stream);
    return fail("selective_scan: %d states per channel (up to 256)", a.N);
}
}  // namespace

MHB_EXPORT int mhb_mingru_scan(const float* proj, int nsplit, long long split_stride, int ld, int z0, int x0, int g0,
                               const float* bz, const float* bx, float* state, long long state_stride,
                               const int* seg_offset, const int* seg_slot, const int* positions, void* out, int out_dtype,
                               int T, int S, int longest, int W, int writable, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (S > 65535) return fail("mingru_scan: %d segments", S);
    GruArgs a;
    a.z = Cols{proj + z0, nsplit, (size_t)split_stride, ld};
    a.x = Cols{proj + x0, nsplit, (size_t)split_stride, ld};
    a.g = Cols{proj + g0, nsplit, (size_t)split_stride, ld};
    a.bz = bz; a.bx = bx; a.state = state; a.state_stride = (size_t)state_stride; a.seg_offset = seg_offset;
    a.seg_slot = seg_slot; a.positions = positions; a.out = out; a.W = W; a.writable = writable;
    if (longest <= 16)
        MHB_DISPATCH_DTYPE(out_dtype, OT,
            launch_kernel(mingru_walk_kernel<OT>, dim3((W + 63) / 64, S), dim3(64), 0, stream, a));
    else
        MHB_DISPATCH_DTYPE(out_dtype, OT,
            launch_kernel(mingru_scan_kernel<OT>, dim3((W + GRU_CH - 1) / GRU_CH, S), dim3(GRU_CH * GRU_LANES), 0, stream, a));
    return check_launch("mingru_scan");
}

MHB_EXPORT int mhb_selective_split(const float* proj, int nsplit, long long split_stride, int ld, int rank, int N, void* dt,
                                   int dt_dtype, int dt_ld, float* bc, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    MHB_DISPATCH_DTYPE(dt_dtype, OT,
        launch_kernel(selective_split_kernel<OT>, dim3(T), dim3(128), 0, stream, Cols{proj, nsplit, (size_t)split_stride, ld},
                      rank, N, (OT*)dt, dt_ld, bc, T));
    return check_launch("selective_split");
}

// dt_weight null: `dt` holds the step's logits [T][C]; else `dt` holds the small product's rank columns and the logits
// are dt_weight [C][rank] times them
MHB_EXPORT int mhb_selective_scan(const float* z, int z_nsplit, long long z_stride, int z_ld, const float* dt, int dt_nsplit,
                                  long long dt_stride, int dt_ld, const float* bc, int bc_nsplit, long long bc_stride,
                                  int bc_ld, const float* x, const void* dt_weight, int rank, int rank_ld,
                                  const float* dt_bias, const float* A2, const float* D, float* state,
                                  long long state_stride, const int* seg_offset, const int* seg_slot, const int* positions,
                                  void* out, int dtype, float scale, int T, int S, int C, int N, int writable,
                                  cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (S > 65535) return fail("selective_scan: %d segments", S);
    ScanArgs a;
    a.z = Cols{z, z_nsplit, (size_t)z_stride, z_ld};
    a.dt = Cols{dt, dt_nsplit, (size_t)dt_stride, dt_ld};
    a.bc = Cols{bc, bc_nsplit, (size_t)bc_stride, bc_ld};
    a.x = x; a.dt_weight = dt_weight; a.rank = rank; a.rank_ld = rank_ld; a.dt_bias = dt_bias; a.A2 = A2; a.D = D;
    a.state = state; a.state_stride = (size_t)state_stride; a.seg_offset = seg_offset; a.seg_slot = seg_slot;
    a.positions = positions; a.out = out; a.scale = scale; a.C = C; a.N = N; a.writable = writable;
    if (dt_weight) MHB_DISPATCH_DTYPE(dtype, OT, return (pick_scan<true, OT, OT>(a, S, stream)));
    MHB_DISPATCH_DTYPE(dtype, OT, return (pick_scan<false, float, OT>(a, S, stream)));
}
