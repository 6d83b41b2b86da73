// The input of an attention layer whose q, k and v pass a short causal convolution over time before they are used:
//
//   y_t[c] = sum_j w[c, j] u_(t - taps + 1 + j)[c]      u: the projected columns; zeros before the start of the sequence
//   q, k:  y / sqrt(mean over the head of y^2 + eps) * weight (one [dim] for all heads, or none)
//   q:     times 1 + coef ln(floor((position + 1) / every) + 1)
//   q goes to a matrix [T][nq dk], k and v into the pages of the cache (v is not normalised)
//
// A row of the product holds [q: nq * dk | k: nkv * dk | v: nkv * dv | anything else], float32, possibly in split-K parts
// that are summed in index order; a layer that reads another layer's cache has [q | anything else] and has_kv = 0.
// A slot keeps the last taps - 1 projected rows of a sequence [taps - 1][channels] in float32.
//
// A warp owns one head (of q, k or v) and a tile of up to TILE tokens of one segment, so that the norm is a warp's sum.
// The first tile of a segment reads the slot's kept rows and, when it is done with them, writes the new ones, from the
// product itself if they lie in another tile: no other tile touches the slot (TILE >= taps - 1), and a lane reads and
// writes the same channels only.  Two kernels: heads up to 128 wide in float4 with up to four taps keep the window of
// projected values in registers and the next tokens' loads in flight; every other shape reads its taps again from the
// product (which the caches hold).
#include "common.cuh"

using namespace mhb;

MHB_EXPORT const char* mhb_last_error() { return error_buffer(); }

namespace {
constexpr int MAX_TAPS = 16;
constexpr int TILE = 16;
constexpr int AHEAD = 4;          // tokens whose loads are in flight together
constexpr int WARPS = 4;

struct Args {
    const float* proj;            // [nsplit][T][ld]
    int nsplit, ld;
    size_t split_stride;
    const float* taps;            // [ntaps][C], the last row is the current token's
    const float* q_weight;        // [dk] or null
    const float* k_weight;
    float eps;
    float* keep;                  // [slots][keep_stride]: [ntaps - 1][C]
    size_t keep_stride;
    const int* seg_offset;        // [S + 1]
    const int* seg_slot;
    const int* positions;         // [T]
    const int* block_table;       // [S][width]
    int width;
    void* q_out;
    void* cache;
    int* status;
    int nq, nkv, dk, dv, P, num_pages, has_kv, ntaps, C;
    float temp_coef;
    double temp_every;
};

__device__ __forceinline__ float4 load4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ void add4(float4& a, const float4 b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ void store4(float* p, const float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *(const uint32_t*)&a;
    u.y = *(const uint32_t*)&b;
    *(uint2*)p = u;
}

// the head of this warp: which part it belongs to, its first column of the product and its width
struct Head {
    int kind, index, col, d;      // kind 0: q, 1: k, 2: v
};
__device__ __forceinline__ Head head_of(const Args& a, int unit) {
    Head h;
    h.kind = unit < a.nq ? 0 : unit < a.nq + a.nkv ? 1 : 2;
    h.index = h.kind == 0 ? unit : h.kind == 1 ? unit - a.nq : unit - a.nq - a.nkv;
    h.d = h.kind == 2 ? a.dv : a.dk;
    h.col = h.kind == 0 ? h.index * a.dk : h.kind == 1 ? (a.nq + h.index) * a.dk : (a.nq + a.nkv) * a.dk + h.index * a.dv;
    return h;
}

__device__ __forceinline__ float temperature(const Args& a, int pos) {
    return a.temp_coef != 0.f ? 1.f + a.temp_coef * log1pf((float)floor((double)(pos + 1) / a.temp_every)) : 1.f;
}

// where a token's row of this head goes: its first element in q_out or in the pool (-1: the table names no page of the pool)
__device__ __forceinline__ long long target(const Args& a, const Head& h, int t, int seg, int pos) {
    if (h.kind == 0) return ((long long)t * a.nq + h.index) * a.dk;
    const int page = a.block_table[(size_t)seg * a.width + pos / a.P], within = pos % a.P;
    if (page < 0 || page >= a.num_pages) {          // never write outside the pool
        if (a.status) atomicOr(a.status, 2);
        return -1;
    }
    const long long base = (long long)page * ((long long)a.nkv * a.P * (a.dk + a.dv));
    if (h.kind == 1) return base + ((long long)h.index * a.P + within) * a.dk;
    return base + (long long)a.nkv * a.P * a.dk + ((long long)h.index * a.P + within) * a.dv;
}

// ---- heads up to 128 wide, multiples of four, up to four taps --------------------------------------------------
template <typename CT, int TAPS>
__global__ void __launch_bounds__(WARPS * 32)
window_kernel(const Args a) {
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int unit = blockIdx.x * WARPS + (threadIdx.x >> 5);
    const int units = a.nq + (a.has_kv ? 2 * a.nkv : 0);
    const bool any = unit < units;
    const Head h = head_of(a, any ? unit : 0);
    const int e = lane * 4;
    const bool inside = any && e < h.d;
    const int c = h.col + e;               // this lane's first channel
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 w[TAPS], gain = make_float4(1.f, 1.f, 1.f, 1.f);
    if (inside) {                          // constants: before the wait for the kernel in front
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = load4(a.taps + (size_t)j * a.C + c);
        const float* g = h.kind == 0 ? a.q_weight : a.k_weight;
        if (h.kind < 2 && g) gain = load4(g + e);
    }
    pdl_wait();
    if (!any) return;
    const int seg = blockIdx.y;
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    const int begin = t0 + blockIdx.z * TILE;
    if (begin >= t1) return;
    const int end = min(begin + TILE, t1);
    const bool first = begin == t0, fresh = a.positions[t0] == 0;
    float* kept = TAPS > 1 ? a.keep + (size_t)a.seg_slot[seg] * a.keep_stride : nullptr;
    auto raw = [&](int t) {
        const float* p = a.proj + (size_t)t * a.ld + c;
        float4 v = load4(p);
        for (int s = 1; s < a.nsplit; ++s) add4(v, load4(p + (size_t)s * a.split_stride));
        return v;
    };
    float4 win[TAPS > 1 ? TAPS - 1 : 1];   // win[j]: the value TAPS - 1 - j tokens before the one that is next
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
        const int back = TAPS - 1 - j;
        win[j] = zero;
        if (!inside) continue;
        if (begin - back >= t0) win[j] = raw(begin - back);
        else if (!fresh) win[j] = load4(kept + (size_t)j * a.C + c);        // only the first tile gets here
    }
    if constexpr (TAPS > 1) {
        if (first && end < t1 && inside)          // a segment of several tiles: its last rows are all its own
#pragma unroll
            for (int r = 0; r < TAPS - 1; ++r) store4(kept + (size_t)r * a.C + c, raw(t1 - (TAPS - 1) + r));
    }
    // lane l looks up where token begin + l goes and its temperature; the others ask it
    long long my_row = -1;
    float my_temp = 1.f;
    if (lane < TILE && begin + lane < end) {
        const int pos = a.positions[begin + lane];
        my_row = target(a, h, begin + lane, seg, pos);
        if (h.kind == 0) my_temp = temperature(a, pos);
    }
    CT* out = (CT*)(h.kind == 0 ? a.q_out : a.cache);
    for (int t = begin; t < end; t += AHEAD) {
        float4 u[AHEAD], y[AHEAD];
        float ss[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) u[i] = inside && t + i < end ? raw(t + i) : zero;
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            y[i] = zero;
            if (inside) {
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {              // the window runs on into this round's tokens
                    const int at = i + j - (TAPS - 1);
                    const float4 v = at >= 0 ? u[at >= 0 ? at : 0] : win[at >= 0 ? 0 : TAPS - 1 + at];
                    y[i].x = fmaf(w[j].x, v.x, y[i].x); y[i].y = fmaf(w[j].y, v.y, y[i].y);
                    y[i].z = fmaf(w[j].z, v.z, y[i].z); y[i].w = fmaf(w[j].w, v.w, y[i].w);
                }
            }
            ss[i] = y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
        }
        if (h.kind < 2) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < AHEAD; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const int from = (t + i - begin) & 31;
            const long long row = __shfl_sync(0xffffffffu, my_row, from);
            const float temp = __shfl_sync(0xffffffffu, my_temp, from);
            if (h.kind < 2) {
                const float f = temp / sqrtf(ss[i] / (float)h.d + a.eps);
                y[i].x *= f * gain.x; y[i].y *= f * gain.y; y[i].z *= f * gain.z; y[i].w *= f * gain.w;
            }
            if (t + i < end && row >= 0 && inside) store4(out + row + e, y[i]);
        }
        if constexpr (TAPS > 1) {                             // the window after the last token of this round that exists
            const int n = min(AHEAD, end - t);
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const float4 next = j + 1 < TAPS - 1 ? win[j + 1 < TAPS - 1 ? j + 1 : 0] : u[i];
                    if (i < n) win[j] = next;
                }
            }
        }
    }
    if constexpr (TAPS > 1) {
        if (first && end == t1 && inside)         // a segment of one tile: the window holds the last rows, older ones included
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) store4(kept + (size_t)j * a.C + c, win[j]);
    }
}

// ---- every other shape --------------------------------------------------------------------------------------------
template <typename CT>
__global__ void __launch_bounds__(WARPS * 32)
general_kernel(const Args a) {
    extern __shared__ float rows[];        // [WARPS][widest head]
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int unit = blockIdx.x * WARPS + warp;
    if (unit >= a.nq + (a.has_kv ? 2 * a.nkv : 0)) return;
    const Head h = head_of(a, unit);
    float* row = rows + (size_t)warp * max(a.dk, a.dv);
    const int seg = blockIdx.y;
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    const int begin = t0 + blockIdx.z * TILE;
    if (begin >= t1) return;
    const int end = min(begin + TILE, t1), R = a.ntaps - 1;
    const bool first = begin == t0, fresh = a.positions[t0] == 0;
    float* kept = R > 0 ? a.keep + (size_t)a.seg_slot[seg] * a.keep_stride : nullptr;
    auto raw = [&](int t, int c) {
        const float* p = a.proj + (size_t)t * a.ld + c;
        float v = *p;
        for (int s = 1; s < a.nsplit; ++s) v += p[(size_t)s * a.split_stride];
        return v;
    };
    for (int t = begin; t < end; ++t) {
        const int pos = a.positions[t];
        float ss = 0.f;
        for (int e = lane; e < h.d; e += 32) {
            const int c = h.col + e;
            float y = 0.f;
            for (int j = 0; j < a.ntaps; ++j) {
                const int back = R - j;
                float z = 0.f;
                if (t - back >= t0) z = raw(t - back, c);
                else if (!fresh) z = kept[(size_t)(R - (back - (t - t0))) * a.C + c];
                y = fmaf(a.taps[(size_t)j * a.C + c], z, y);
            }
            row[e] = y;
            ss += y * y;
        }
        float f = 1.f;
        const float* g = nullptr;
        if (h.kind < 2) {
            f = (h.kind == 0 ? temperature(a, pos) : 1.f) / sqrtf(warp_sum(ss) / (float)h.d + a.eps);
            g = h.kind == 0 ? a.q_weight : a.k_weight;
        }
        const long long at = target(a, h, t, seg, pos);
        CT* dst = (CT*)(h.kind == 0 ? a.q_out : a.cache) + (at >= 0 ? at : 0);
        if (at >= 0)
            for (int e = lane; e < h.d; e += 32) dst[e] = from_float<CT>(row[e] * (f * (g ? g[e] : 1.f)));
    }
    if (first && R > 0) {
        const int n = t1 - t0;
        for (int e = lane; e < h.d; e += 32) {
            const int c = h.col + e;
            for (int r = 0; r < R; ++r) {              // new row r: the value R - r positions before the segment's end
                const int back = R - r;
                float z = 0.f;
                if (back <= n) z = raw(t1 - back, c);
                else if (!fresh) z = kept[(size_t)(r + n) * a.C + c];       // an old row that is still inside (r + n > r)
                kept[(size_t)r * a.C + c] = z;
            }
        }
    }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }
}  // namespace

// taps [ntaps][C] float32 with C = nq dk (+ nkv (dk + dv) with has_kv); keep [slots][keep_stride].  temp_coef 0: no
// temperature.  longest: tokens of the longest segment.
MHB_EXPORT int mhb_head_conv_append(const float* proj, int nsplit, long long split_stride, int ld, const float* taps,
                                    int ntaps, const float* q_weight, const float* k_weight, float eps, float* keep,
                                    long long keep_stride, const int* seg_offset, const int* seg_slot,
                                    const int* positions, const int* block_table, int width, void* q_out, void* cache,
                                    int dtype, int T, int S, int longest, int nq, int nkv, int dk, int dv, int P,
                                    int num_pages, int has_kv, float temp_coef, double temp_every, int* status,
                                    cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (ntaps < 1 || ntaps > MAX_TAPS) return fail("head_conv_append: %d taps (1 to %d)", ntaps, MAX_TAPS);
    if (ntaps > 1 && !keep) return fail("head_conv_append: %d taps need kept rows", ntaps);
    if (nq < 1 || nkv < 1 || dk < 1 || dv < 1) return fail("head_conv_append: %d and %d heads of %d and %d", nq, nkv, dk, dv);
    if (temp_coef != 0.f && !(temp_every > 0.)) return fail("head_conv_append: a temperature needs a positive step");
    const int tiles = (longest + TILE - 1) / TILE;
    if (S > 65535 || tiles > 65535) return fail("head_conv_append: %d segments, the longest of %d tokens", S, longest);
    Args a;
    a.proj = proj; a.nsplit = nsplit; a.ld = ld; a.split_stride = (size_t)split_stride; a.taps = taps;
    a.q_weight = q_weight; a.k_weight = k_weight; a.eps = eps; a.keep = keep; a.keep_stride = (size_t)keep_stride;
    a.seg_offset = seg_offset; a.seg_slot = seg_slot; a.positions = positions; a.block_table = block_table; a.width = width;
    a.q_out = q_out; a.cache = cache; a.status = status; a.nq = nq; a.nkv = nkv; a.dk = dk; a.dv = dv; a.P = P;
    a.num_pages = num_pages; a.has_kv = has_kv; a.ntaps = ntaps; a.C = nq * dk + (has_kv ? nkv * (dk + dv) : 0);
    a.temp_coef = temp_coef; a.temp_every = temp_every;
    const int units = nq + (has_kv ? 2 * nkv : 0);
    const dim3 grid((units + WARPS - 1) / WARPS, S, tiles);
    const bool window = ntaps <= 4 && dk % 4 == 0 && dk <= 128 && (!has_kv || (dv % 4 == 0 && dv <= 128)) && ld % 4 == 0 &&
                        split_stride % 4 == 0 && keep_stride % 4 == 0 && aligned16(proj) && aligned16(taps) &&
                        aligned16(keep) && aligned16(q_out) && aligned16(cache) && aligned16(q_weight) && aligned16(k_weight);
    MHB_DISPATCH_DTYPE(dtype, CT, {
        cudaError_t e = cudaSuccess;
        if (!window) {
            const size_t smem = sizeof(float) * WARPS * (size_t)(dk > dv ? dk : dv);
            if (smem > 48 * 1024) return fail("head_conv_append: heads of %d and %d are too wide", dk, dv);
            e = launch_kernel(general_kernel<CT>, grid, dim3(WARPS * 32), smem, stream, a);
        } else if (ntaps == 1) e = launch_kernel(window_kernel<CT, 1>, grid, dim3(WARPS * 32), 0, stream, a);
        else if (ntaps == 2) e = launch_kernel(window_kernel<CT, 2>, grid, dim3(WARPS * 32), 0, stream, a);
        else if (ntaps == 3) e = launch_kernel(window_kernel<CT, 3>, grid, dim3(WARPS * 32), 0, stream, a);
        else e = launch_kernel(window_kernel<CT, 4>, grid, dim3(WARPS * 32), 0, stream, a);
        if (e != cudaSuccess) return fail("head_conv_append: %s", cudaGetErrorString(e));
    });
    return check_launch("head_conv_append");
}
