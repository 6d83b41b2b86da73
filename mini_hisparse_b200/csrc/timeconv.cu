// Short causal convolutions over time, one filter per channel, and what they are fused with.
//
//   conv(h)_t[c] = sum_j w[c, j] h_(t - taps + 1 + j)[c]          (zeros before the start of the sequence)
//
//   stream_conv   the input of a sublayer whose norm works element by element (dynamic tanh):
//                 v = x + d1 + d2 (the stream with pending products), h = tanh(alpha v) w + b,
//                 out = h + conv(h); v goes to ANOTHER buffer than x
//   rows_conv     out = h + conv(h) for rows h that are already normalised (any other norm)
//   product_conv  out = silu(conv(z) + bias) for columns z of a float32 product
//   dyt_rows      h alone, of chosen rows (the norm in front of the head)
//   stream_shift  x <- x + d (+ table[token] * scale) + row
//
// A slot keeps the last taps - 1 inputs of a sequence [taps - 1][C] in float32.  The grid is (channels, segments,
// tiles of a segment's tokens); a thread owns VEC channels and walks a tile with the window in registers.  The first
// tile of a segment reads the kept inputs and writes the new ones, which it computes itself (from the stream before
// this kernel, which is why the sum goes to another buffer): no other tile touches the slot, and no two kernels are
// needed.  Everything is float32; products may come as split-K parts, which are summed in index order.
#include "common.cuh"

using namespace mhb;

MHB_EXPORT const char* mhb_last_error() { return error_buffer(); }

namespace {
constexpr int MAX_TAPS = 16;
constexpr int TILE = 16;          // tokens per tile: at least MAX_TAPS - 1, so that later tiles never look into the slot
constexpr int AHEAD = 4;          // tokens whose loads are in flight together

enum { STREAM = 0, ROWS = 1, PRODUCT = 2 };

struct Delta {
    const float* p;
    int nsplit;
    size_t stride;
};

struct ConvArgs {
    const void* src;            // STREAM: x [T][C] float32; ROWS: h [T][C]; PRODUCT: first column of [T][ld] float32 parts
    int nsplit;
    size_t split_stride;
    int ld;
    Delta d1, d2;               // STREAM: pending products [T][C]
    float* x_out;               // STREAM: where the sum goes (null: nothing pending)
    const float* alpha;         // STREAM: one number
    const float* weight;        // STREAM: [C]
    const float* shift;         // STREAM: [C]
    const float* taps;          // [ntaps][C], the last row is the current token's
    const float* bias;          // PRODUCT: [C]
    float* keep;                // [slots][keep_stride]: [ntaps - 1][C]
    size_t keep_stride;
    const int* seg_offset;      // [S + 1]
    const int* seg_slot;
    const int* positions;
    void* out;                  // [T][C] compute dtype
    float* out32;               // PRODUCT: [T][C] float32, or null
    int C, ntaps, writable;
};

template <int VEC> __device__ __forceinline__ void load_f(const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const float4 f = *(const float4*)p;
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else v[0] = *p;
}
template <int VEC> __device__ __forceinline__ void load_f(const __nv_bfloat16* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const uint2 u = *(const uint2*)p;
        const __nv_bfloat162 a = *(const __nv_bfloat162*)&u.x, b = *(const __nv_bfloat162*)&u.y;
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    } else v[0] = __bfloat162float(*p);
}
template <int VEC> __device__ __forceinline__ void store_f(float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int VEC> __device__ __forceinline__ void store_f(__nv_bfloat16* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 u;
        u.x = *(const uint32_t*)&a;
        u.y = *(const uint32_t*)&b;
        *(uint2*)p = u;
    } else *p = __float2bfloat16_rn(v[0]);
}
template <int VEC> __device__ __forceinline__ void add_parts(const float* p, int nsplit, size_t stride, float (&v)[VEC]) {
#pragma unroll 4
    for (int s = 0; s < nsplit; ++s) {
        float d[VEC];
        load_f<VEC>(p + (size_t)s * stride, d);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] += d[i];
    }
}

__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.f + expf(-z)); }

// the raw input of one token: the stream with everything pending, or the rows themselves
template <int MODE, typename IT, int VEC>
__device__ __forceinline__ void raw_input(const ConvArgs& a, int t, int c, float (&v)[VEC]) {
    const size_t at = (size_t)t * a.ld + c;
    load_f<VEC>((const IT*)a.src + at, v);
    if constexpr (MODE == STREAM) {
        if (a.d1.p) add_parts<VEC>(a.d1.p + at, a.d1.nsplit, a.d1.stride, v);
        if (a.d2.p) add_parts<VEC>(a.d2.p + at, a.d2.nsplit, a.d2.stride, v);
    } else if constexpr (MODE == PRODUCT) {
        if (a.nsplit > 1) add_parts<VEC>((const float*)a.src + at + a.split_stride, a.nsplit - 1, a.split_stride, v);
    }
}

// TAPS >= ntaps: the filters are padded with zeros at the old end
template <int MODE, typename IT, typename OT, int VEC, int TAPS>
__global__ void __launch_bounds__(128)
conv_kernel(const ConvArgs a) {
    pdl_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    const bool inside = c < a.C;
    const int R = a.ntaps - 1;             // inputs a slot keeps
    float w[TAPS][VEC], gain[VEC], shift[VEC], bias[VEC];
    float alpha = 0.f;
    if (inside) {                          // constants: before the wait for the kernel in front
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const int k = j - (TAPS - a.ntaps);
            if (k >= 0) load_f<VEC>(a.taps + (size_t)k * a.C + c, w[j]);
            else
#pragma unroll
                for (int i = 0; i < VEC; ++i) w[j][i] = 0.f;
        }
        if constexpr (MODE == STREAM) {
            alpha = *a.alpha;
            load_f<VEC>(a.weight + c, gain);
            load_f<VEC>(a.shift + c, shift);
        }
        if constexpr (MODE == PRODUCT) {
            if (a.bias) load_f<VEC>(a.bias + c, bias);
            else
#pragma unroll
                for (int i = 0; i < VEC; ++i) bias[i] = 0.f;
        }
    }
    pdl_wait();
    const int seg = blockIdx.y;
    const int t0 = a.seg_offset[seg], t1 = a.seg_offset[seg + 1];
    const int begin = t0 + blockIdx.z * TILE;
    if (begin >= t1 || !inside) return;
    const int end = min(begin + TILE, t1);
    const bool first = begin == t0;
    const bool fresh = a.positions[t0] == 0;
    float* kept = a.keep + (size_t)a.seg_slot[seg] * a.keep_stride;

    auto activate = [&](float (&v)[VEC]) {
        if constexpr (MODE == STREAM)
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[i] = tanhf(alpha * v[i]) * gain[i] + shift[i];
    };
    // win[j]: the input TAPS - 1 - j tokens before the one that is next
    float win[TAPS > 1 ? TAPS - 1 : 1][VEC];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
        const int back = TAPS - 1 - j;
#pragma unroll
        for (int i = 0; i < VEC; ++i) win[j][i] = 0.f;
        if (back > R) continue;
        if (begin - back >= t0) {
            raw_input<MODE, IT, VEC>(a, begin - back, c, win[j]);
            activate(win[j]);
        } else if (!fresh) load_f<VEC>(kept + (size_t)(R - back) * a.C + c, win[j]);      // only the first tile gets here
    }
    if (first && a.writable && end < t1) {       // a segment of several tiles: its last R inputs are all its own (TILE >= R)
        for (int r = 0; r < R; ++r) {
            float v[VEC];
            raw_input<MODE, IT, VEC>(a, t1 - R + r, c, v);
            activate(v);
            store_f<VEC>(kept + (size_t)r * a.C + c, v);
        }
    }
    for (int t = begin; t < end; t += AHEAD) {
        float raw[AHEAD][VEC];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (t + u < end) raw_input<MODE, IT, VEC>(a, t + u, c, raw[u]);
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (t + u >= end) break;
            const size_t at = (size_t)(t + u) * a.C + c;
            if constexpr (MODE == STREAM) {
                if (a.x_out) store_f<VEC>(a.x_out + at, raw[u]);
            }
            float h[VEC], y[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) h[i] = raw[u][i];
            activate(h);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                float s = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) s = fmaf(w[j][i], win[j][i], s);
                s = fmaf(w[TAPS - 1][i], h[i], s);
                if constexpr (MODE == PRODUCT) y[i] = silu(s + bias[i]);
                else y[i] = h[i] + s;
            }
            store_f<VEC>((OT*)a.out + at, y);
            if constexpr (MODE == PRODUCT) {
                if (a.out32) store_f<VEC>(a.out32 + at, y);
            }
#pragma unroll
            for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
                for (int i = 0; i < VEC; ++i) win[j][i] = win[j + 1][i];
            if constexpr (TAPS > 1)
#pragma unroll
                for (int i = 0; i < VEC; ++i) win[TAPS - 2][i] = h[i];
        }
    }
    if (first && a.writable && end == t1) {      // a segment of one tile: the window holds the last inputs, older ones included
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int back = TAPS - 1 - j;
            if (back <= R) store_f<VEC>(kept + (size_t)(R - back) * a.C + c, win[j]);
        }
    }
}

template <int MODE, typename IT, typename OT>
int launch_conv(const ConvArgs& a, int S, int longest, bool vec, const char* what, cudaStream_t stream) {
    const int tiles = (longest + TILE - 1) / TILE;
    if (S > 65535 || tiles > 65535) return fail("%s: %d segments, the longest of %d tokens", what, S, longest);
    const int per = vec && a.ntaps <= 4 ? 4 : 1;
    // few tokens: small CTAs, so that more SMs take part
    int threads = (long long)S * tiles * a.C / (per * 128) < 296 ? 32 : 128;
    dim3 grid((a.C + per * threads - 1) / (per * threads), S, tiles);
    if (per == 4) launch_kernel(conv_kernel<MODE, IT, OT, 4, 4>, grid, dim3(threads), 0, stream, a);
    else if (a.ntaps <= 4) launch_kernel(conv_kernel<MODE, IT, OT, 1, 4>, grid, dim3(threads), 0, stream, a);
    else launch_kernel(conv_kernel<MODE, IT, OT, 1, MAX_TAPS>, grid, dim3(threads), 0, stream, a);
    return check_launch(what);
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

// ---- dynamic tanh of chosen rows ------------------------------------------------------------------
// out[r] = tanh(alpha v) * w + b with v = x[s] + d1[s] + d2[s], s = rows ? rows[r] : r; without rows and with a delta the
// sum is written back
template <typename OT>
__global__ void dyt_rows_kernel(float* __restrict__ x, Delta d1, Delta d2, const float* __restrict__ alpha,
                                const float* __restrict__ weight, const float* __restrict__ shift,
                                const int* __restrict__ rows, OT* __restrict__ out, int H) {
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const size_t s = rows ? rows[r] : r;
    const float al = *alpha;
    const bool back = !rows && (d1.p || d2.p);
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float v[1] = {x[s * H + i]};
        if (d1.p) add_parts<1>(d1.p + s * H + i, d1.nsplit, d1.stride, v);
        if (d2.p) add_parts<1>(d2.p + s * H + i, d2.nsplit, d2.stride, v);
        if (back) x[s * H + i] = v[0];
        out[(size_t)r * H + i] = from_float<OT>(tanhf(al * v[0]) * weight[i] + shift[i]);
    }
}

// ---- x <- x + d (+ table[token] scale) + row ---------------------------------------------------------
template <typename WT, int VEC>
__global__ void stream_shift_kernel(float* __restrict__ x, Delta d, const WT* __restrict__ table, const int* __restrict__ tokens,
                                    float scale, int vocab, const float* __restrict__ row, size_t n, int H) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t at = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (at >= n) return;
    const size_t t = at / H;
    const int i = (int)(at - t * H);
    float v[VEC], e[VEC], r[VEC];
    load_f<VEC>(x + at, v);
    load_f<VEC>(row + i, r);
    if (d.p) add_parts<VEC>(d.p + at, d.nsplit, d.stride, v);
    if (table) {
        const int tok = tokens[t];                    // an id outside the table gave zeros (and a status bit) in the embedding
        if (tok >= 0 && tok < vocab) {
            load_f<VEC>(table + (size_t)tok * H + i, e);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] += e[j] * scale;
        }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] += r[j];
    store_f<VEC>(x + at, v);
}
}  // namespace

// vec for all of them: four neighbours a thread when every row and every pointer allows float4
MHB_EXPORT int mhb_stream_conv(const float* x, const float* d1, int n1, long long s1, const float* d2, int n2, long long s2,
                               float* x_out, const float* alpha, const float* weight, const float* shift,
                               const float* taps, float* keep, long long keep_stride, const int* seg_offset,
                               const int* seg_slot, const int* positions, void* out, int out_dtype, int T, int S,
                               int longest, int C, int ntaps, int writable, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (ntaps < 1 || ntaps > MAX_TAPS) return fail("stream_conv: %d taps (1 to %d)", ntaps, MAX_TAPS);
    if (x_out == x) return fail("stream_conv: the sum must go to another buffer than the stream is read from");
    if ((d1 || d2) && !x_out) return fail("stream_conv: nowhere to put the sum");
    ConvArgs a = {};
    a.src = x; a.nsplit = 1; a.ld = C; a.d1 = Delta{d1, n1, (size_t)s1}; a.d2 = Delta{d2, n2, (size_t)s2}; a.x_out = x_out;
    a.alpha = alpha; a.weight = weight; a.shift = shift; a.taps = taps; a.keep = keep; a.keep_stride = (size_t)keep_stride;
    a.seg_offset = seg_offset; a.seg_slot = seg_slot; a.positions = positions; a.out = out; a.C = C; a.ntaps = ntaps;
    a.writable = writable && ntaps > 1;
    const bool vec = C % 4 == 0 && aligned16(x) && aligned16(d1) && aligned16(d2) && aligned16(x_out) && aligned16(weight) &&
                     aligned16(shift) && aligned16(taps) && aligned16(keep) && keep_stride % 4 == 0 && aligned16(out) &&
                     s1 % 4 == 0 && s2 % 4 == 0;
    MHB_DISPATCH_DTYPE(out_dtype, OT, return (launch_conv<STREAM, float, OT>(a, S, longest, vec, "stream_conv", stream)));
}

MHB_EXPORT int mhb_rows_conv(const void* h, int dtype, const float* taps, float* keep, long long keep_stride,
                             const int* seg_offset, const int* seg_slot, const int* positions, void* out, int T, int S,
                             int longest, int C, int ntaps, int writable, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (ntaps < 1 || ntaps > MAX_TAPS) return fail("rows_conv: %d taps (1 to %d)", ntaps, MAX_TAPS);
    if (out == h) return fail("rows_conv: input and output must be different buffers");
    ConvArgs a = {};
    a.src = h; a.nsplit = 1; a.ld = C; a.taps = taps; a.keep = keep; a.keep_stride = (size_t)keep_stride;
    a.seg_offset = seg_offset; a.seg_slot = seg_slot; a.positions = positions; a.out = out; a.C = C; a.ntaps = ntaps;
    a.writable = writable && ntaps > 1;
    const bool vec = C % 4 == 0 && aligned16(h) && aligned16(taps) && aligned16(keep) && keep_stride % 4 == 0 && aligned16(out);
    MHB_DISPATCH_DTYPE(dtype, OT, return (launch_conv<ROWS, OT, OT>(a, S, longest, vec, "rows_conv", stream)));
}

MHB_EXPORT int mhb_product_conv(const float* z, int nsplit, long long split_stride, int ld, const float* taps,
                                const float* bias, float* keep, long long keep_stride, const int* seg_offset,
                                const int* seg_slot, const int* positions, void* out, int out_dtype, float* out32, int T,
                                int S, int longest, int C, int ntaps, int writable, cudaStream_t stream) {
    if (T <= 0 || S <= 0) return 0;
    if (ntaps < 1 || ntaps > MAX_TAPS) return fail("product_conv: %d taps (1 to %d)", ntaps, MAX_TAPS);
    ConvArgs a = {};
    a.src = z; a.nsplit = nsplit; a.split_stride = (size_t)split_stride; a.ld = ld; a.taps = taps; a.bias = bias;
    a.keep = keep; a.keep_stride = (size_t)keep_stride; a.seg_offset = seg_offset; a.seg_slot = seg_slot;
    a.positions = positions; a.out = out; a.out32 = out32; a.C = C; a.ntaps = ntaps; a.writable = writable && ntaps > 1;
    const bool vec = C % 4 == 0 && ld % 4 == 0 && aligned16(z) && split_stride % 4 == 0 && aligned16(taps) &&
                     aligned16(bias) && aligned16(keep) && keep_stride % 4 == 0 && aligned16(out) && aligned16(out32);
    MHB_DISPATCH_DTYPE(out_dtype, OT, return (launch_conv<PRODUCT, float, OT>(a, S, longest, vec, "product_conv", stream)));
}

MHB_EXPORT int mhb_dyt_rows(float* x, const float* d1, int n1, long long s1, const float* d2, int n2, long long s2,
                            const float* alpha, const float* weight, const float* shift, const int* rows, void* out,
                            int out_dtype, int R, int H, cudaStream_t stream) {
    if (R <= 0) return 0;
    const int threads = H >= 1024 ? 256 : 128;
    MHB_DISPATCH_DTYPE(out_dtype, OT,
        launch_kernel(dyt_rows_kernel<OT>, dim3(R), dim3(threads), 0, stream, x, Delta{d1, n1, (size_t)s1},
                      Delta{d2, n2, (size_t)s2}, alpha, weight, shift, rows, (OT*)out, H));
    return check_launch("dyt_rows");
}

MHB_EXPORT int mhb_stream_shift(float* x, const float* d, int nd, long long sd, const void* table, int table_dtype,
                                const int* tokens, float scale, int vocab, const float* row, int T, int H,
                                cudaStream_t stream) {
    if (T <= 0) return 0;
    const size_t n = (size_t)T * H;
    const Delta delta{d, nd, (size_t)sd};
    const bool vec = H % 4 == 0 && aligned16(x) && aligned16(d) && sd % 4 == 0 && aligned16(table) && aligned16(row);
    const int per = vec ? 4 : 1, threads = 128;
    const unsigned blocks = (unsigned)((n / per + threads - 1) / threads);
    MHB_DISPATCH_DTYPE(table_dtype, WT, {
        if (vec) launch_kernel(stream_shift_kernel<WT, 4>, dim3(blocks), dim3(threads), 0, stream, x, delta, (const WT*)table, tokens, scale, vocab, row, n, H);
        else launch_kernel(stream_shift_kernel<WT, 1>, dim3(blocks), dim3(threads), 0, stream, x, delta, (const WT*)table, tokens, scale, vocab, row, n, H);
    });
    return check_launch("stream_shift");
}
