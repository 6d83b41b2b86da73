// Linear recurrences, element by element, with coefficients made from the input row alone (so they can be scanned).
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

// divisions by __fdividef (2 ulp; its zero for denominators beyond 2^126 is the limit here): without the branch of the
// full division several elements of a thread overlap
__device__ __forceinline__ float sigmoidf(float z) { return __fdividef(1.f, 1.f + expf(-z)); }
__device__ __forceinline__ float siluf(float z) { return __fdividef(z, 1.f + expf(-z)); }
__device__ __forceinline__ float softplusf(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
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
constexpr int GRU_CH = 8, GRU_LANES = 64, GRU_RUN = 8;

template <typename OT>
__global__ void __launch_bounds__(GRU_CH * GRU_LANES, 2)
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
    Cols dt;                 // [T][>= C]: the step's logits (dt_weight: the small product, columns 0 .. rank - 1)
    Cols bc;                 // [T]: B in columns 0 .. N - 1, C in N .. 2 N - 1
    const float* x;          // [T][C]
    const void* dt_weight;   // [C][rank] compute dtype (few tokens), or null
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

__device__ __forceinline__ void copy_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Few tokens per segment.  LPC lanes share a channel, each RPL states in registers (N <= LPC * RPL); up to CH tokens are
// staged at once.  The step's logits are formed here from the small product's rank columns (dt_weight), the lanes of a
// channel sharing the dot product: one launch less than a product of its own.
template <int LPC, int RPL, int CH, int THREADS, typename WT, typename OT>
__global__ void __launch_bounds__(THREADS, 7)
selective_step_kernel(const ScanArgs a) {
    constexpr int CPB = THREADS / LPC;                           // channels per CTA
    constexpr int E = (CH * CPB + THREADS - 1) / THREADS;        // elements a thread loads per stage
    __shared__ float Bs[CH][LPC * RPL], Cs[CH][LPC * RPL];
    __shared__ float dts[CH][CPB], dxs[CH][CPB], ys[CH][CPB];
    extern __shared__ __align__(16) float low[];                 // [CH][rank]
    pdl_launch_dependents();
    const int seg = blockIdx.y, c0 = blockIdx.x * CPB;
    const int sub = threadIdx.x % LPC, cl = threadIdx.x / LPC, c = c0 + cl;
    const int N = a.N;
    const bool live = c < a.C;
    float A2[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int n = sub * RPL + r;
        A2[r] = (live && n < N) ? a.A2[(size_t)c * N + n] : 0.f;
    }
    pdl_wait();
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    if (t0 >= t1) return;
    float* slot = a.state + (size_t)a.seg_slot[seg] * a.state_stride;
    const bool fresh = a.positions[t0] == 0;
    float S[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int n = sub * RPL + r;
        S[r] = (!fresh && live && n < N) ? slot[(size_t)c * N + n] : 0.f;
    }
    const WT* w = (const WT*)a.dt_weight + (size_t)(live ? c : 0) * a.rank_ld;
    for (int b = t0; b < t1; b += CH) {
        const int n = min(CH, t1 - b);
        float x_r[E], z_r[E];
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
            const bool ok = tt < n && c0 + k < a.C;
            x_r[e] = ok ? a.x[(size_t)(b + tt) * a.C + c0 + k] : 0.f;
            z_r[e] = ok ? a.z.at(b + tt, c0 + k) : 0.f;
        }
        for (int i = threadIdx.x; i < n * a.rank; i += THREADS) low[i] = a.dt.at(b + i / a.rank, i % a.rank);
        for (int i = threadIdx.x; i < n * LPC * RPL; i += THREADS) {
            const int tt = i / (LPC * RPL), k = i % (LPC * RPL);
            Bs[tt][k] = k < N ? a.bc.at(b + tt, k) : 0.f;
            Cs[tt][k] = k < N ? a.bc.at(b + tt, N + k) : 0.f;
        }
        __syncthreads();
        for (int tt = 0; tt < n; ++tt) {
            const float* lr = low + tt * a.rank;
            float d = 0.f;
            if (a.rank % 8 == 0) {
#pragma unroll 4
                for (int i = sub * 8; i < a.rank; i += LPC * 8) {
                    float wv[8];
                    if constexpr (sizeof(WT) == 2) {
                        const uint4 u = *(const uint4*)(w + i);
                        const __nv_bfloat162* h = (const __nv_bfloat162*)&u;
#pragma unroll
                        for (int j = 0; j < 4; ++j) { wv[2 * j] = __low2float(h[j]); wv[2 * j + 1] = __high2float(h[j]); }
                    } else {
#pragma unroll
                        for (int j = 0; j < 8; ++j) wv[j] = to_float(w[i + j]);
                    }
#pragma unroll
                    for (int j = 0; j < 8; ++j) d = fmaf(wv[j], lr[i + j], d);
                }
            } else
                for (int i = sub; i < a.rank; i += LPC) d = fmaf(to_float(w[i]), lr[i], d);
#pragma unroll
            for (int o = 1; o < LPC; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
            if (sub == 0) dts[tt][cl] = d;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = threadIdx.x + e * THREADS, tt = i / CPB, k = i % CPB;
            if (tt < n) {
                const float dt = c0 + k < a.C ? softplusf(dts[tt][k] + a.dt_bias[c0 + k]) : 0.f;
                dts[tt][k] = dt;
                dxs[tt][k] = dt * x_r[e];
            }
        }
        __syncthreads();
        for (int tt = 0; tt < n; ++tt) {
            const float dt = dts[tt][cl], dx = dxs[tt][cl];
            float y = 0.f;
#pragma unroll
            for (int r = 0; r < RPL; ++r) {
                S[r] = fmaf(exp2_fast(dt * A2[r]), S[r], dx * Bs[tt][sub * RPL + r]);
                y = fmaf(S[r], Cs[tt][sub * RPL + r], y);
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
                    from_float<OT>((ys[tt][k] + a.D[c0 + k] * x_r[e]) * siluf(z_r[e]) * a.scale);
        }
    }
    if (a.writable)
#pragma unroll
        for (int r = 0; r < RPL; ++r) {
            const int n = sub * RPL + r;
            if (live && n < N) slot[(size_t)c * N + n] = S[r];
        }
}

// Long segments: the recurrence walks token by token, so a CTA's warps are split.  WALKERS threads (LPC lanes a channel,
// RPL states each) do nothing but walk: dt and dt x of eight tokens as float4s, B and C rows, and the sums over a
// channel's lanes for eight tokens at once (each shuffle halves the tokens a lane carries).  HELPERS threads prepare the
// chunk after this one (softplus; B and C by cp.async; the loads of the chunk after that are already in flight) and
// finish the one before (D x, the gate, the store).  Tokens beyond the segment get dt = 0, which leaves the state alone.
template <int LPC, int RPL, int CH, typename OT>
__global__ void __launch_bounds__(256, 2)
selective_scan_kernel(const ScanArgs a) {
    constexpr int WALKERS = 128, HELPERS = 128;
    constexpr int CPB = WALKERS / LPC;
    constexpr int E = (CH * CPB + HELPERS - 1) / HELPERS;
    constexpr int NP = LPC * RPL;                                // states, padded
    constexpr int G = 8;                                         // tokens whose sums are finished together
    static_assert(LPC >= G && CH % G == 0, "");
    __shared__ __align__(16) float Bs[2][CH][NP], Cs[2][CH][NP];
    __shared__ __align__(16) float dts[2][CPB][CH + 4], dxs[2][CPB][CH + 4];
    __shared__ float ys[2][CPB][CH + 1];
    pdl_launch_dependents();
    const int seg = blockIdx.y, c0 = blockIdx.x * CPB, N = a.N;
    for (int i = threadIdx.x; i < 2 * CH * NP; i += 256) { (&Bs[0][0][0])[i] = 0.f; (&Cs[0][0][0])[i] = 0.f; }
    pdl_wait();
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    if (t0 >= t1) return;
    __syncthreads();
    const int chunks = (t1 - t0 + CH - 1) / CH;
    if (threadIdx.x >= WALKERS) {
        const int tid = threadIdx.x - WALKERS;
        float dt_r[E], x_r[E], z_r[E], skip[E], gate[E], bias[E], D[E];
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int k = (tid + e * HELPERS) % CPB;
            bias[e] = c0 + k < a.C ? a.dt_bias[c0 + k] : 0.f;
            D[e] = c0 + k < a.C ? a.D[c0 + k] : 0.f;
        }
        auto fetch = [&](int chunk) {
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = tid + e * HELPERS, tt = i / CPB, k = i % CPB, t = t0 + chunk * CH + tt;
                const bool ok = tt < CH && t < t1 && c0 + k < a.C;
                dt_r[e] = ok ? a.dt.at(t, c0 + k) : 0.f;
                x_r[e] = ok ? a.x[(size_t)t * a.C + c0 + k] : 0.f;
                z_r[e] = ok ? a.z.at(t, c0 + k) : 0.f;
            }
        };
        // B and C: rows of 2 N numbers, in runs of four where they allow it; a thread's next run is `dq` tokens and `dr` runs on
        const bool by4 = N % 4 == 0 && a.bc.nsplit == 1 && a.bc.ld % 4 == 0 && ((uintptr_t)a.bc.p & 15) == 0;
        const int per = by4 ? N / 2 : 2 * N, dq = HELPERS / per, dr = HELPERS % per, tt0 = tid / per, k0 = tid % per;
        auto stage_bc = [&](int st, int chunk) {
            const int b = t0 + chunk * CH, n = min(CH, t1 - b);
            for (int tt = tt0, k = k0; tt < n;) {
                const int i = by4 ? 4 * k : k;
                float* dst = i < N ? &Bs[st][tt][i] : &Cs[st][tt][i - N];
                if (by4) copy_async16(dst, a.bc.p + (size_t)(b + tt) * a.bc.ld + i);
                else *dst = a.bc.at(b + tt, i);
                tt += dq;
                k += dr;
                if (k >= per) { k -= per; ++tt; }
            }
            copy_async_commit();
        };
        auto stage = [&](int st, int chunk) {                    // what fetch() brought
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = tid + e * HELPERS, tt = i / CPB, k = i % CPB;
                if (tt >= CH) continue;
                const float dt = t0 + chunk * CH + tt < t1 ? softplusf(dt_r[e] + bias[e]) : 0.f;
                dts[st][k][tt] = dt;
                dxs[st][k][tt] = dt * x_r[e];
                skip[e] = D[e] * x_r[e];
                gate[e] = siluf(z_r[e]) * a.scale;
            }
        };
        float sk[E], ga[E];                                      // of the chunk that is walked
        auto finish = [&](int chunk) {
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = tid + e * HELPERS, tt = i / CPB, k = i % CPB, t = t0 + chunk * CH + tt;
                if (tt < CH && t < t1 && c0 + k < a.C)
                    ((OT*)a.out)[(size_t)t * a.C + c0 + k] = from_float<OT>((ys[chunk & 1][k][tt] + sk[e]) * ga[e]);
            }
        };
        fetch(0);
        stage_bc(0, 0);
        stage(0, 0);
        if (chunks > 1) fetch(1);
        copy_async_wait<0>();
        __syncthreads();                                         // chunk 0 is staged
        for (int k = 0; k < chunks; ++k) {
            if (k + 1 < chunks) stage_bc((k + 1) & 1, k + 1);
            if (k > 0) finish(k - 1);
#pragma unroll
            for (int e = 0; e < E; ++e) { sk[e] = skip[e]; ga[e] = gate[e]; }
            if (k + 1 < chunks) {
                stage((k + 1) & 1, k + 1);
                if (k + 2 < chunks) fetch(k + 2);
            }
            copy_async_wait<0>();
            __syncthreads();                                     // chunk k is walked, chunk k + 1 is staged
        }
        finish(chunks - 1);
        return;
    }
    const int sub = threadIdx.x % LPC, cl = threadIdx.x / LPC, c = c0 + cl;
    float* slot = a.state + (size_t)a.seg_slot[seg] * a.state_stride;
    const bool fresh = a.positions[t0] == 0;
    float A2[RPL], S[RPL];
#pragma unroll
    for (int r = 0; r < RPL; ++r) {
        const int n = sub * RPL + r;
        const bool ok = c < a.C && n < N;
        A2[r] = ok ? a.A2[(size_t)c * N + n] : 0.f;
        S[r] = (ok && !fresh) ? slot[(size_t)c * N + n] : 0.f;
    }
    __syncthreads();
    for (int k = 0; k < chunks; ++k) {
        const int st = k & 1;
#pragma unroll 1
        for (int g = 0; g < CH; g += G) {
            float dt[G], dx[G], y[G];
#pragma unroll
            for (int i = 0; i < G; i += 4) {
                const float4 p = *(const float4*)&dts[st][cl][g + i], q = *(const float4*)&dxs[st][cl][g + i];
                dt[i] = p.x; dt[i + 1] = p.y; dt[i + 2] = p.z; dt[i + 3] = p.w;
                dx[i] = q.x; dx[i + 1] = q.y; dx[i + 2] = q.z; dx[i + 3] = q.w;
            }
#pragma unroll
            for (int i = 0; i < G; ++i) {
                const float* bp = &Bs[st][g + i][sub * RPL];
                const float* cp = &Cs[st][g + i][sub * RPL];
                float Bv[RPL], Cv[RPL];
                if constexpr (RPL % 4 == 0) {
#pragma unroll
                    for (int r = 0; r < RPL; r += 4) {
                        const float4 p = *(const float4*)(bp + r), q = *(const float4*)(cp + r);
                        Bv[r] = p.x; Bv[r + 1] = p.y; Bv[r + 2] = p.z; Bv[r + 3] = p.w;
                        Cv[r] = q.x; Cv[r + 1] = q.y; Cv[r + 2] = q.z; Cv[r + 3] = q.w;
                    }
                } else if constexpr (RPL == 2) {
                    const float2 p = *(const float2*)bp, q = *(const float2*)cp;
                    Bv[0] = p.x; Bv[1] = p.y;
                    Cv[0] = q.x; Cv[1] = q.y;
                } else {
#pragma unroll
                    for (int r = 0; r < RPL; ++r) { Bv[r] = bp[r]; Cv[r] = cp[r]; }
                }
                y[i] = 0.f;
#pragma unroll
                for (int r = 0; r < RPL; ++r) {
                    S[r] = fmaf(exp2_fast(dt[i] * A2[r]), S[r], dx[i] * Bv[r]);
                    y[i] = fmaf(S[r], Cv[r], y[i]);
                }
            }
            // lane `sub` ends up with the sum of token g + sub % 8
#pragma unroll
            for (int half = G / 2, o = 1; half > 0; half >>= 1, o <<= 1) {
                const bool odd = sub & o;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float keep = odd ? y[2 * i + 1] : y[2 * i], send = odd ? y[2 * i] : y[2 * i + 1];
                    y[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
#pragma unroll
            for (int o = G; o < LPC; o <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
            if (sub < G) ys[st][cl][g + sub] = y[0];
        }
        __syncthreads();
    }
    if (a.writable)
#pragma unroll
        for (int r = 0; r < RPL; ++r) {
            const int n = sub * RPL + r;
            if (c < a.C && n < N) slot[(size_t)c * N + n] = S[r];
        }
}

template <int LPC, int RPL, int CH, typename WT>
int launch_step(const ScanArgs& a, int S, cudaStream_t stream) {
    constexpr int THREADS = 128;
    constexpr int CPB = THREADS / LPC;
    auto kern = selective_step_kernel<LPC, RPL, CH, THREADS, WT, WT>;
    const size_t smem = sizeof(float) * CH * (size_t)a.rank;
    if (smem > 8 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return fail("selective_scan: a rank of %d: %s", a.rank, cudaGetErrorString(e));
    }
    launch_kernel(kern, dim3((a.C + CPB - 1) / CPB, S), dim3(THREADS), smem, stream, a);
    return check_launch("selective_scan");
}

template <typename WT>
int pick_step(const ScanArgs& a, int S, cudaStream_t stream) {
    if (a.N <= 16) return launch_step<4, 4, 4, WT>(a, S, stream);
    if (a.N <= 32) return launch_step<4, 8, 4, WT>(a, S, stream);
    if (a.N <= 64) return launch_step<8, 8, 4, WT>(a, S, stream);
    if (a.N <= 128) return launch_step<16, 8, 4, WT>(a, S, stream);
    if (a.N <= 256) return launch_step<32, 8, 4, WT>(a, S, stream);
    return fail("selective_scan: %d states per channel (up to 256)", a.N);
}

template <int LPC, int RPL, int CH, typename OT>
int launch_scan(const ScanArgs& a, int S, cudaStream_t stream) {
    constexpr int CPB = 128 / LPC;
    launch_kernel(selective_scan_kernel<LPC, RPL, CH, OT>, dim3((a.C + CPB - 1) / CPB, S), dim3(256), 0, stream, a);
    return check_launch("selective_scan");
}

template <typename OT>
int pick_scan(const ScanArgs& a, int S, cudaStream_t stream) {
    // few channels: more lanes (and so more CTAs) share a channel, which a walk that is bound by latency needs
    const bool few = (long long)S * ((a.C + 15) / 16) < 200;
    if (a.N <= 16) return few ? launch_scan<16, 1, 32, OT>(a, S, stream) : launch_scan<8, 2, 32, OT>(a, S, stream);
    if (a.N <= 32 && few) return launch_scan<16, 2, 32, OT>(a, S, stream);
    if (a.N <= 24) return launch_scan<8, 3, 32, OT>(a, S, stream);
    if (a.N <= 32) return launch_scan<8, 4, 32, OT>(a, S, stream);
    if (a.N <= 64) return launch_scan<8, 8, 16, OT>(a, S, stream);
    if (a.N <= 128) return launch_scan<16, 8, 8, OT>(a, S, stream);
    if (a.N <= 256) return launch_scan<32, 8, 8, OT>(a, S, stream);
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
    if (dt_weight) MHB_DISPATCH_DTYPE(dtype, WT, return (pick_step<WT>(a, S, stream)));
    MHB_DISPATCH_DTYPE(dtype, OT, return (pick_scan<OT>(a, S, stream)));
}
