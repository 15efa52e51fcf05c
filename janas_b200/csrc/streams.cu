// A residual stream kept as several streams per row (hyper-connections), float32 [n, streams, dm].
//
//   write:  X_t <- sum_s mix[s, t] X_s + mult * out[t] * (ls * y)      y: a sublayer's result, all t at once
//   read:   u = sum_s in[s] X_s;   h = (u - mean u) / sqrt(var u + eps) * w + b
//
// A launch does a write, a read, or a write and the read of what was just written (the next
// sublayer's), so that the streams go through the chip once per sublayer.  y is a stack of partial
// sums; ls (a factor per value) may be null; in null: every stream counts once; w null: u itself, in
// float32.  mix has a row per stream before and a column per stream after.  Everything is computed in float32; mean and variance are two
// passes over the row, and the order of the additions depends on the row's width alone.
#include "common.cuh"
#include "kernels.h"

namespace jb {

struct StreamWrite {
    const float *y;            // [S, n, dm] or null: nothing is written
    int S;
    size_t stride;
    const float *ls, *out, *mix;
    float mult;
};
struct StreamRead {
    const float *in, *w, *b;
    float eps;
};

constexpr int MAX_STREAMS = 32;

// Rows of up to 1024 NV values, a multiple of four, everything on 16-byte boundaries: a block of
// 256 threads per row, four values of every stream to a thread at a time, u in registers.
template <typename TO, int NS, int NV>
__global__ void __launch_bounds__(256)
streams_vec_kernel(float *__restrict__ x, StreamWrite wr, const int32_t *__restrict__ rows, StreamRead rd,
                   TO *__restrict__ out, int dm)
{
    __shared__ float red[32];
    pdl_trigger();
    int r = blockIdx.x, nv = dm / 4;
    float mix[NS * NS], wo[NS], wi[NS];
#pragma unroll
    for (int s = 0; s < NS; s++) {
        wo[s] = wr.y != nullptr ? wr.mult * wr.out[s] : 0.0f;
        wi[s] = rd.in != nullptr ? rd.in[s] : 1.0f;
#pragma unroll
        for (int t = 0; t < NS; t++)
            mix[s * NS + t] = wr.y != nullptr ? wr.mix[s * NS + t] : 0.0f;
    }
    pdl_wait();
    size_t src = rows != nullptr ? (size_t)rows[r] : (size_t)r;
    float *xr = x + src * NS * dm;
    float4 u[NV];
    float sum = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; k++) {
        int i = threadIdx.x + k * 256;
        u[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i >= nv)
            continue;
        float4 xs[NS];
#pragma unroll
        for (int s = 0; s < NS; s++)
            xs[s] = load4(xr + (size_t)s * dm + 4 * i);
        if (wr.y != nullptr) {
            const float *p = wr.y + src * dm + 4 * i;
            float4 y = load4(p);
            for (int sp = 1; sp < wr.S; sp++) {
                float4 t = load4(p + (size_t)sp * wr.stride);
                y.x += t.x; y.y += t.y; y.z += t.z; y.w += t.w;
            }
            if (wr.ls != nullptr) {
                float4 l = load4(wr.ls + 4 * i);
                y.x *= l.x; y.y *= l.y; y.z *= l.z; y.w *= l.w;
            }
            float4 nx[NS];
#pragma unroll
            for (int t = 0; t < NS; t++) {
                float4 a = make_float4(wo[t] * y.x, wo[t] * y.y, wo[t] * y.z, wo[t] * y.w);
#pragma unroll
                for (int s = 0; s < NS; s++) {
                    float c = mix[s * NS + t];
                    a.x = fmaf(c, xs[s].x, a.x);
                    a.y = fmaf(c, xs[s].y, a.y);
                    a.z = fmaf(c, xs[s].z, a.z);
                    a.w = fmaf(c, xs[s].w, a.w);
                }
                nx[t] = a;
                store4(xr + (size_t)t * dm + 4 * i, a);
            }
#pragma unroll
            for (int t = 0; t < NS; t++)
                xs[t] = nx[t];
        }
        float4 a = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int s = 0; s < NS; s++) {
            a.x = fmaf(wi[s], xs[s].x, a.x);
            a.y = fmaf(wi[s], xs[s].y, a.y);
            a.z = fmaf(wi[s], xs[s].z, a.z);
            a.w = fmaf(wi[s], xs[s].w, a.w);
        }
        u[k] = a;
        sum += (a.x + a.y) + (a.z + a.w);
    }
    if (out == nullptr)
        return;
    TO *o = out + (size_t)r * dm;
    if (rd.w == nullptr) {
#pragma unroll
        for (int k = 0; k < NV; k++)
            if (threadIdx.x + k * 256 < nv)
                store4(o + 4 * (threadIdx.x + k * 256), u[k]);
        return;
    }
    float mean = block_sum(sum, red) / (float)dm;
    float sq = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; k++)
        if (threadIdx.x + k * 256 < nv) {
            float dx = u[k].x - mean, dy = u[k].y - mean, dz = u[k].z - mean, dw = u[k].w - mean;
            sq = fmaf(dx, dx, sq); sq = fmaf(dy, dy, sq); sq = fmaf(dz, dz, sq); sq = fmaf(dw, dw, sq);
        }
    float inv = 1.0f / sqrtf(block_sum(sq, red) / (float)dm + rd.eps);
#pragma unroll
    for (int k = 0; k < NV; k++) {
        int i = threadIdx.x + k * 256;
        if (i < nv) {
            float4 w = load4(rd.w + 4 * i);
            float4 b = rd.b != nullptr ? load4(rd.b + 4 * i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            store4(o + 4 * i, make_float4(fmaf((u[k].x - mean) * inv, w.x, b.x), fmaf((u[k].y - mean) * inv, w.y, b.y),
                                          fmaf((u[k].z - mean) * inv, w.z, b.z), fmaf((u[k].w - mean) * inv, w.w, b.w)));
        }
    }
}

// One value of every stream: the write (when there is one), and u.
template <int NS>
__device__ __forceinline__ float stream_value(float *xr, const StreamWrite &wr, const StreamRead &rd, const float *mix,
                                              size_t src, int c, int dm, int ns)
{
    constexpr int CAP = NS > 0 ? NS : MAX_STREAMS, UN = NS > 0 ? NS : 1;
    const int n = NS > 0 ? NS : ns;
    float xs[CAP];
#pragma unroll(UN)
    for (int s = 0; s < CAP; s++)
        if (s < n)
            xs[s] = xr[(size_t)s * dm + c];
    float u = 0.0f;
    if (wr.y == nullptr) {
#pragma unroll(UN)
        for (int s = 0; s < CAP; s++)
            if (s < n)
                u = fmaf(rd.in != nullptr ? rd.in[s] : 1.0f, xs[s], u);
        return u;
    }
    float y = add_partials(0.0f, wr.y + src * dm + c, wr.S, wr.stride);
    if (wr.ls != nullptr)
        y *= wr.ls[c];
#pragma unroll(UN)
    for (int t = 0; t < CAP; t++)
        if (t < n) {
            float a = wr.mult * wr.out[t] * y;
#pragma unroll(UN)
            for (int s = 0; s < CAP; s++)
                if (s < n)
                    a = fmaf(mix[s * n + t], xs[s], a);
            xr[(size_t)t * dm + c] = a;
            u = fmaf(rd.in != nullptr ? rd.in[t] : 1.0f, a, u);
        }
    return u;
}

// Any sizes: a block per row, one value of every stream to a thread at a time, u in shared memory.
template <typename TO>
__global__ void __launch_bounds__(256)
streams_kernel(float *__restrict__ x, int ns, StreamWrite wr, const int32_t *__restrict__ rows, StreamRead rd,
               TO *__restrict__ out, int dm)
{
    extern __shared__ float row[];
    __shared__ float red[32], mix[MAX_STREAMS * MAX_STREAMS];
    pdl_trigger();
    int r = blockIdx.x;
    if (wr.y != nullptr)
        for (int i = threadIdx.x; i < ns * ns; i += blockDim.x)
            mix[i] = wr.mix[i];
    __syncthreads();
    pdl_wait();
    size_t src = rows != nullptr ? (size_t)rows[r] : (size_t)r;
    float *xr = x + src * ns * dm;
    float sum = 0.0f;
    for (int c = threadIdx.x; c < dm; c += blockDim.x) {
        float u = stream_value<0>(xr, wr, rd, mix, src, c, dm, ns);
        row[c] = u;
        sum += u;
    }
    if (out == nullptr)
        return;
    TO *o = out + (size_t)r * dm;
    if (rd.w == nullptr) {
        for (int c = threadIdx.x; c < dm; c += blockDim.x)
            o[c] = from_f<TO>(row[c]);
        return;
    }
    float mean = block_sum(sum, red) / (float)dm;
    float sq = 0.0f;
    for (int c = threadIdx.x; c < dm; c += blockDim.x) {
        float d = row[c] - mean;
        sq = fmaf(d, d, sq);
    }
    float inv = 1.0f / sqrtf(block_sum(sq, red) / (float)dm + rd.eps);
    for (int c = threadIdx.x; c < dm; c += blockDim.x)
        o[c] = from_f<TO>(fmaf((row[c] - mean) * inv, rd.w[c], rd.b != nullptr ? rd.b[c] : 0.0f));
}

// The same for few rows of the bfloat16 path: a cluster of C CTAs per row, each with `cols` columns
// (the sums cross the cluster as in layernorm_cluster_kernel).
template <typename TO, int NS, int C>
__global__ void __launch_bounds__(512)
streams_cluster_kernel(float *__restrict__ x, int ns, StreamWrite wr, const int32_t *__restrict__ rows, StreamRead rd,
                       TO *__restrict__ out, int dm, int cols)
{
    extern __shared__ float row[];          // this CTA's slice of u
    __shared__ float red[32], mix[MAX_STREAMS * MAX_STREAMS];
    __shared__ float part_sum[C], part_sq[C];
    pdl_trigger();
    if (wr.y != nullptr)
        for (int i = threadIdx.x; i < ns * ns; i += blockDim.x)
            mix[i] = wr.mix[i];
    __syncthreads();
    uint32_t rank = cluster_rank();
    int r = blockIdx.x / C;
    int c0 = (int)rank * cols, c1 = min(dm, c0 + cols);
    pdl_wait();
    size_t src = rows != nullptr ? (size_t)rows[r] : (size_t)r;
    float *xr = x + src * ns * dm;
    float sum = 0.0f;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float u = stream_value<NS>(xr, wr, rd, mix, src, c, dm, ns);
        row[c - c0] = u;
        sum += u;
    }
    if (out == nullptr)
        return;                             // the write alone: no CTA of the cluster waits for another
    sum = block_sum(sum, red);
    if (threadIdx.x < C)
        cluster_write(&part_sum[rank], threadIdx.x, sum);
    cluster_arrive();
    cluster_wait();
    float tot = 0.0f;
#pragma unroll
    for (int k = 0; k < C; k++)
        tot += part_sum[k];
    float mean = tot / (float)dm;
    float sq = 0.0f;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float d = row[c - c0] - mean;
        sq = fmaf(d, d, sq);
    }
    sq = block_sum(sq, red);
    if (threadIdx.x < C)
        cluster_write(&part_sq[rank], threadIdx.x, sq);
    cluster_arrive();
    cluster_wait();
    tot = 0.0f;
#pragma unroll
    for (int k = 0; k < C; k++)
        tot += part_sq[k];
    float inv = 1.0f / sqrtf(tot / (float)dm + rd.eps);
    TO *o = out + (size_t)r * dm;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x)
        o[c] = from_f<TO>(fmaf((row[c - c0] - mean) * inv, rd.w[c], rd.b != nullptr ? rd.b[c] : 0.0f));
}

// x[r, s, :] = e[r, :] for every stream s; V values a thread
template <int V>
__global__ void __launch_bounds__(256)
spread_streams_kernel(const float *__restrict__ e, float *__restrict__ x, int ns, int n, int dm)
{
    pdl_trigger();
    int per = dm / V;
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)n * per)
        return;
    size_t r = idx / per;
    int c = (int)(idx - r * per) * V;
    pdl_wait();
    if (V == 4) {
        float4 v = load4(e + r * dm + c);
        for (int s = 0; s < ns; s++)
            store4(x + (r * ns + s) * dm + c, v);
    } else {
        float v = e[r * dm + c];
        for (int s = 0; s < ns; s++)
            x[(r * ns + s) * dm + c] = v;
    }
}

}  // namespace jb

using namespace jb;

extern "C" int jb_max_streams(void) { return MAX_STREAMS; }

extern "C" int jb_spread_streams(const float *e, float *x, int ns, int n, int dm, cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (ns <= 0 || ns > MAX_STREAMS || dm <= 0 || e == nullptr || x == nullptr)
        return JB_EINVAL;
    bool vec = dm % 4 == 0 && (((uintptr_t)e | (uintptr_t)x) & 15) == 0;
    size_t threads = (size_t)n * (vec ? dm / 4 : dm);
    unsigned grid = (unsigned)((threads + 255) / 256);
    if (vec)
        launch(spread_streams_kernel<4>, grid, 256, 0, st, e, x, ns, n, dm);
    else
        launch(spread_streams_kernel<1>, grid, 256, 0, st, e, x, ns, n, dm);
    return launch_status();
}

// x: float32 [rows, ns, dm].  y: float32 [S, n, dm] with ls (float32 [dm] or null), out_w [ns] and
// mix [ns, ns]: the write, in place; null: none.  out ([n, dm] in out_dt): the read; null: none.  rows (n
// indices, or null): the rows that are read (then nothing is written to x).  w null: u in float32.
// few_rows: a cluster of CTAs per row (the bfloat16 path's decode steps).
extern "C" int jb_streams(float *x, int ns, const float *y, int S, long long stride, const float *ls, const float *out_w,
                          const float *mix, float mult, const int32_t *rows, const float *in_w, const float *w,
                          const float *b, float eps, void *out, int out_dt, int n, int dm, int few_rows,
                          cudaStream_t st)
{
    if (n <= 0)
        return JB_OK;
    if (ns <= 0 || ns > MAX_STREAMS || dm <= 0 || dm > 40960 / 4 || x == nullptr || (y == nullptr && out == nullptr) ||
        (y != nullptr && (S <= 0 || out_w == nullptr || mix == nullptr || rows != nullptr)) ||
        (out != nullptr && out_dt != JB_F32 && (out_dt != JB_BF16 || w == nullptr)))
        return JB_EINVAL;
    StreamWrite wr{y, S, (size_t)stride, ls, out_w, mix, mult};
    StreamRead rd{in_w, w, b, eps};
    constexpr int CL = 8;
    if (few_rows && n <= 32 && dm >= 64 * CL && (out == nullptr || (w != nullptr && out_dt == JB_BF16))) {
        int cols = (dm + CL - 1) / CL;
        unsigned threads = (unsigned)min(512, (cols + 31) / 32 * 32);
#define JB_STC(NS)                                                                                             \
    launch_cluster(streams_cluster_kernel<bf16, NS, CL>, dim3((unsigned)n * CL), threads, (size_t)cols * 4, st, CL, x, \
                   ns, wr, rows, rd, (bf16 *)out, dm, cols)
        if (ns == 1) JB_STC(1);
        else if (ns == 2) JB_STC(2);
        else if (ns == 3) JB_STC(3);
        else if (ns == 4) JB_STC(4);
        else JB_STC(0);
#undef JB_STC
        return launch_status();
    }
    auto al16 = [](const void *p) { return ((uintptr_t)p & 15) == 0; };
    bool vec = ns <= 4 && dm % 4 == 0 && dm <= 8192 && stride % 4 == 0 && al16(x) && al16(y) && al16(ls) && al16(w) &&
               al16(b) && al16(out);
#define JB_STV(TO, NS, NV) launch(streams_vec_kernel<TO, NS, NV>, (unsigned)n, 256, 0, st, x, wr, rows, rd, (TO *)out, dm)
#define JB_STV_N(TO, NV)                                                                                       \
    do {                                                                                                       \
        if (ns == 1) JB_STV(TO, 1, NV);                                                                        \
        else if (ns == 2) JB_STV(TO, 2, NV);                                                                   \
        else if (ns == 3) JB_STV(TO, 3, NV);                                                                   \
        else JB_STV(TO, 4, NV);                                                                                \
    } while (0)
#define JB_STV_ANY(TO)                                                                                         \
    do {                                                                                                       \
        if (dm <= 1024) JB_STV_N(TO, 1);                                                                       \
        else if (dm <= 2048) JB_STV_N(TO, 2);                                                                  \
        else if (dm <= 3072) JB_STV_N(TO, 3);                                                                  \
        else if (dm <= 4096) JB_STV_N(TO, 4);                                                                  \
        else JB_STV_N(TO, 8);                                                                                  \
    } while (0)
    bool half = out != nullptr && out_dt == JB_BF16;
    if (vec) {
        if (half) JB_STV_ANY(bf16);
        else JB_STV_ANY(float);
        return launch_status();
    }
    unsigned threads = (unsigned)min(256, (dm + 31) / 32 * 32);
    if (half)
        launch(streams_kernel<bf16>, (unsigned)n, threads, (size_t)dm * 4, st, x, ns, wr, rows, rd, (bf16 *)out, dm);
    else
        launch(streams_kernel<float>, (unsigned)n, threads, (size_t)dm * 4, st, x, ns, wr, rows, rd, (float *)out, dm);
    return launch_status();
#undef JB_STV_ANY
#undef JB_STV_N
#undef JB_STV
}
