// Dynamic tanh, a norm without statistics, fused with the residual sum that precedes it:
//
//   norm(x) = tanh(alpha * x) * w + b          alpha one number, w and b one number per column
//
//   tb_dyt    per number of the stream h [rows, width] (32-bit), given a branch output a (a matrix in 32 or 16 bits, or
//             32-bit split-K partial sums [splits, rows, width], added in split order):
//               take 0   h stays (a is not read)
//               take 1   h <- h + norm_a(a)
//               take 2   h <- a               (a product that replaces the stream)
//             then, if asked for,
//               give 1   out <- norm_b(h)
//               give 2   out <- h             (the stream itself in the output's dtype)
//             with rows of `out` out_stride numbers apart, so that it may be a part of a wider matrix.
//             from 1: x is read from `a` instead of h and h is not touched (a norm on its own).
//
// No number waits for any other, so nothing is shared: a thread owns four columns (one where rows are not whole 16-byte
// pieces) of one or two rows, keeps the columns' weights in registers and has all of its rows on their way at once.
// Everything is 32-bit; only `out` is rounded.
#include "common.cuh"

TB_EXPORT_ERROR()

struct DytArgs {
    float* h;
    const void* a; int n_splits; long long split_stride;
    float alpha_a; const float* wa; const float* ba;
    float alpha_b; const float* wb; const float* bb;
    void* out; long long out_stride;
    int take, give, from;
    int rows, width;
};

// The argument block's size, for the Python mirror's check.
extern "C" int tb_dyt_args_bytes() { return (int)sizeof(DytArgs); }

template <int V> struct Pack { float v[V]; };
template <int V> __device__ __forceinline__ Pack<V> load_pack(const float* p) {
    Pack<V> r;
    if constexpr (V == 4) { const float4 q = *(const float4*)p; r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w; }
    else r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ Pack<V> load_pack(const bf16* p) {
    Pack<V> r;
    if constexpr (V == 4) {
        const uint2 q = *(const uint2*)p;
        r.v[0] = __uint_as_float(q.x << 16); r.v[1] = __uint_as_float(q.x & 0xffff0000u);
        r.v[2] = __uint_as_float(q.y << 16); r.v[3] = __uint_as_float(q.y & 0xffff0000u);
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_pack(float* p, const Pack<V>& r) {
    if constexpr (V == 4) *(float4*)p = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]); else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void store_pack(bf16* p, const Pack<V>& r) {
    if constexpr (V == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *(uint2*)p = make_uint2(*(uint32_t*)&lo, *(uint32_t*)&hi);
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}
template <int V> __device__ __forceinline__ void dyt(Pack<V>& x, float alpha, const Pack<V>& w, const Pack<V>& b) {
#pragma unroll
    for (int e = 0; e < V; e++) x.v[e] = fmaf(tanhf(alpha * x.v[e]), w.v[e], b.v[e]);
}

template <typename TA, typename TO, int V, int RPT>
__global__ void __launch_bounds__(256) dyt_kernel(DytArgs a) {
    pdl_launch_dependents();
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= a.width) return;
    const int r0 = blockIdx.x * RPT;
    Pack<V> wa = {}, ba = {}, wb = {}, bb = {};                       // weights do not depend on the kernel before this one
    if (a.take == 1) { wa = load_pack<V>(a.wa + c); ba = load_pack<V>(a.ba + c); }
    if (a.give == 1) { wb = load_pack<V>(a.wb + c); bb = load_pack<V>(a.bb + c); }
    pdl_wait();
    Pack<V> h[RPT], x[RPT];
    const bool reads_a = a.take != 0 || a.from != 0, reads_h = a.take < 2 && a.from == 0;
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        h[i] = {}; x[i] = {};
        if (r0 + i < a.rows) {
            const size_t at = (size_t)(r0 + i) * a.width + c;
            if (reads_h) h[i] = load_pack<V>(a.h + at);
            if (reads_a) x[i] = load_pack<V>((const TA*)a.a + at);
        }
    }
    if (reads_a && a.n_splits > 1) {
#pragma unroll
        for (int i = 0; i < RPT; i++) {
            if (r0 + i >= a.rows) continue;
            const TA* p = (const TA*)a.a + (size_t)(r0 + i) * a.width + c;
            for (int s0 = 1; s0 < a.n_splits; s0 += 8) {              // eight splits asked for at a time, added in order
                Pack<V> t[8];
#pragma unroll
                for (int k = 0; k < 8; k++) { t[k] = {}; if (s0 + k < a.n_splits) t[k] = load_pack<V>(p + (size_t)(s0 + k) * a.split_stride); }
#pragma unroll
                for (int k = 0; k < 8; k++)
#pragma unroll
                    for (int e = 0; e < V; e++) x[i].v[e] += t[k].v[e];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        if (r0 + i >= a.rows) break;
        const size_t at = (size_t)(r0 + i) * a.width + c;
        if (a.take == 1) {
            dyt<V>(x[i], a.alpha_a, wa, ba);
#pragma unroll
            for (int e = 0; e < V; e++) h[i].v[e] += x[i].v[e];
        } else if (a.take == 2 || a.from != 0) {
            h[i] = x[i];
        }
        if (a.take != 0) store_pack<V>(a.h + at, h[i]);
        if (a.give != 0) {
            if (a.give == 1) dyt<V>(h[i], a.alpha_b, wb, bb);
            store_pack<V>((TO*)a.out + (size_t)(r0 + i) * a.out_stride + c, h[i]);
        }
    }
}

extern "C" int tb_dyt(const DytArgs* args, int a_dtype, int out_dtype, cudaStream_t stream) {
    const DytArgs& a = *args;
    if (a.rows <= 0) return 0;
    if (a.width <= 0) return tb_refuse("dyt: width %d", a.width);
    if (a.take < 0 || a.take > 2 || a.give < 0 || a.give > 2 || (a.from && a.take)) return tb_refuse("dyt: take %d, give %d, from %d", a.take, a.give, a.from);
    const bool reads_a = a.take != 0 || a.from != 0;
    if (reads_a && (a.a == nullptr || a.n_splits < 1)) return tb_refuse("dyt: no branch output to take");
    if (reads_a && a.n_splits > 1 && a_dtype != TB_F32) return tb_refuse("dyt: partial sums must be 32-bit");
    if (a.take == 1 && (a.wa == nullptr || a.ba == nullptr)) return tb_refuse("dyt: the branch's norm has no weights");
    if (a.give == 1 && (a.wb == nullptr || a.bb == nullptr)) return tb_refuse("dyt: the output's norm has no weights");
    if (a.give != 0 && a.out == nullptr) return tb_refuse("dyt: no output");
    if (!a.from && a.h == nullptr) return tb_refuse("dyt: no stream");
    const size_t ea = a_dtype == TB_BF16 ? 2 : 4, eo = out_dtype == TB_BF16 ? 2 : 4;
    const bool vec = a.width % 4 == 0 && (uintptr_t)a.h % 16 == 0 && (!reads_a || ((uintptr_t)a.a % (4 * ea) == 0 && a.split_stride % 4 == 0))
        && (a.give == 0 || ((uintptr_t)a.out % (4 * eo) == 0 && a.out_stride % 4 == 0))
        && (uintptr_t)a.wa % 16 == 0 && (uintptr_t)a.ba % 16 == 0 && (uintptr_t)a.wb % 16 == 0 && (uintptr_t)a.bb % 16 == 0;
    const int cols = vec ? a.width / 4 : a.width;
    // few rows: one a thread, so that the launch spreads over the device; many: two a thread (measured at 2,048 rows of
    // 1,024 to 4,096 numbers: 13, 18 and 30 us, with four rows and 192 threads 15, 22 and 36)
    const bool many = a.rows >= 256;
    const int threads = many ? 128 : 64;
    const int rpt = many ? 2 : 1;
    const dim3 grid((a.rows + rpt - 1) / rpt, (cols + threads - 1) / threads);
    if (grid.y > 65535) return tb_refuse("dyt: rows of %d numbers are too wide", a.width);
#define GO(TA, TO) do { \
        if (vec && many) tb_launch(dyt_kernel<TA, TO, 4, 2>, grid, dim3(threads), 0, stream, a); \
        else if (vec) tb_launch(dyt_kernel<TA, TO, 4, 1>, grid, dim3(threads), 0, stream, a); \
        else if (many) tb_launch(dyt_kernel<TA, TO, 1, 2>, grid, dim3(threads), 0, stream, a); \
        else tb_launch(dyt_kernel<TA, TO, 1, 1>, grid, dim3(threads), 0, stream, a); } while (0)
    TB_DISPATCH_1(a_dtype, TA, TB_DISPATCH_1(out_dtype, TO, GO(TA, TO)));
#undef GO
    return tb_launch_status();
}
