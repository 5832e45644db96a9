// Hyper-connections: the residual is not one vector per row but `streams` of them, x_1 .. x_n.  A sublayer reads one
// weighted sum of the streams and its result goes back to all of them, while they also mix among themselves:
//
//   y     = scale * sum_s rmsnorm(delta[s] + bias[s]) * slice_w[s]      or plainly  sum_s (delta[s] + bias[s])
//   x_t  <- sum_s mix[s][t] x_s + out_w[t] y                            (all streams at once from the old ones)
//   u     = sum_s in_w[s] x_s                                           (the NEXT reader's weights)
//   out   = rmsnorm(u) * w
//
// One kernel does what lies between two sublayers: it finishes the sublayer before (its pending sums, possibly the
// results of two mixers side by side, each normed on its own), brings the streams up to date and norms what the next
// sublayer reads.  Without `mix` the old streams do not enter (the first reader of a step: all streams start as
// copies of the embedding row, which is then the pending result).  Without a pending result the streams stay as they
// are.  With chosen rows only those are produced and the streams are left alone: the model's last norm.
//
// ONE stream with one normed slice is a layer with a norm before and after each sublayer, and has a kernel of its own.
//
// All 32-bit up to the store of `out`.  One CTA per row; sums over a row are formed in a fixed order that depends on
// the width alone (for the one stream also on whether the step has few rows or many), so a row has the same bits in any
// such batch.
#include "common.cuh"

#define HC_MAX_STREAMS 32
#define HC_MAX_SLICES 4

struct StreamNormArgs {
    float* x;                        // [T][streams][H]
    const int* rows;                 // chosen rows, or null
    const float* delta; int S; size_t slice_stride;          // pending sums [S][T][H], or null
    const float* slice_bias;         // [S][H] or null
    const float* slice_w;            // [S][H] or null: every slice over its own root mean square, times this
    float slice_eps, slice_scale;
    const float* out_w;              // [streams]
    const float* mix;                // [streams from][streams to] or null
    const float* in_w;               // [streams]
    const float* w; float eps;       // the norm's weight [H]
    int update;                      // the streams are brought up to date
    int streams, H;
};

template <int VEC> __device__ __forceinline__ void hc_load(const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else {
        v[0] = p[0];
    }
}
template <int VEC> __device__ __forceinline__ void hc_store(float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
}
template <int VEC> __device__ __forceinline__ void hc_store(bf16* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 t;
        t.x = *reinterpret_cast<const unsigned*>(&a);
        t.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = t;
    } else {
        p[0] = __float2bfloat16_rn(v[0]);
    }
}

// sums over the CTA of up to HC_MAX_SLICES numbers a thread, in a fixed order, between two barriers
__device__ __forceinline__ void hc_block_sums(float (&v)[HC_MAX_SLICES], int count, float (*scratch)[32]) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
#pragma unroll
    for (int s = 0; s < HC_MAX_SLICES; ++s)
        if (s < count) {
            v[s] = ap_warp_sum(v[s]);
            if (lane == 0) scratch[s][warp] = v[s];
        }
    __syncthreads();
#pragma unroll
    for (int s = 0; s < HC_MAX_SLICES; ++s)
        if (s < count) {
            float total = 0.f;
            for (int w = 0; w < nwarps; ++w) total += scratch[s][w];
            v[s] = total;
        }
}

// NS: the number of streams the kernel is built for (0: any number up to HC_MAX_STREAMS).  ONE: the CTA has a thread for
// every VEC columns, whose numbers stay in registers between the sums over the row.
template <int NS, int VEC, bool ONE, typename TO>
__global__ void __launch_bounds__(ONE && NS <= 4 ? 1024 : 512) stream_norm_kernel(const StreamNormArgs A, TO* __restrict__ out) {
    constexpr int N = NS ? NS : HC_MAX_STREAMS;
    extern __shared__ __align__(16) float u_s[];             // [H] where not ONE
    __shared__ float slice_scratch[HC_MAX_SLICES][32], scratch[32];
    __shared__ float mix_s[N * N], out_s[N], in_s[N];
    const int n = NS ? NS : A.streams;
    ap_pdl_trigger();
    // the weights do not depend on earlier kernels
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        out_s[i] = A.out_w ? A.out_w[i] : 0.f;
        in_s[i] = A.in_w[i];
    }
    if (A.mix) for (int i = threadIdx.x; i < n * n; i += blockDim.x) mix_s[i] = A.mix[i];
    ap_pdl_wait();
    const int H = A.H;
    const size_t t = A.rows ? (size_t)A.rows[blockIdx.x] : (size_t)blockIdx.x;
    float* xr = A.x + t * n * H;
    const float* dr = A.delta ? A.delta + t * H : nullptr;
    const bool reads_old = A.delta == nullptr || A.mix != nullptr;
    const bool normed = dr != nullptr && A.slice_w != nullptr;

    auto load_old = [&](int c, float (&old)[N][VEC]) {
        if (reads_old) {
#pragma unroll(NS ? N : 1)
            for (int s = 0; s < N; ++s) {
                if (s >= n) break;
                hc_load<VEC>(xr + (size_t)s * H + c, old[s]);
            }
        }
    };
    auto load_slice = [&](int s, int c, float (&d)[VEC]) {
        hc_load<VEC>(dr + s * A.slice_stride + c, d);
        if (A.slice_bias) {
            float b[VEC];
            hc_load<VEC>(A.slice_bias + (size_t)s * H + c, b);
#pragma unroll
            for (int i = 0; i < VEC; ++i) d[i] += b[i];
        }
    };
    float factor[HC_MAX_SLICES];
#pragma unroll
    for (int s = 0; s < HC_MAX_SLICES; ++s) factor[s] = 0.f;
    auto square = [&](int s, const float (&d)[VEC]) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) factor[s] = fmaf(d[i], d[i], factor[s]);
    };
    auto finish_factors = [&]() {
        hc_block_sums(factor, A.S, slice_scratch);
#pragma unroll
        for (int s = 0; s < HC_MAX_SLICES; ++s) factor[s] = A.slice_scale / sqrtf(factor[s] / (float)H + A.slice_eps);
    };
    auto add_slice = [&](int s, int c, const float (&d)[VEC], float (&y)[VEC]) {
        if (normed) {
            float w[VEC];
            hc_load<VEC>(A.slice_w + (size_t)s * H + c, w);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] += d[i] * factor[s] * w[i];
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] += d[i];
        }
    };
    // the streams after the pending result, and what the next sublayer reads of them
    auto apply = [&](int c, const float (&old)[N][VEC], const float (&y)[VEC], float (&u)[VEC]) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = 0.f;
#pragma unroll(NS ? N : 1)
        for (int o = 0; o < N; ++o) {
            if (o >= n) break;
            float v[VEC];
            if (dr) {
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[i] = out_s[o] * y[i];
                if (A.mix) {
#pragma unroll(NS ? N : 1)
                    for (int s = 0; s < N; ++s) {
                        if (s >= n) break;
                        const float m = mix_s[s * n + o];
#pragma unroll
                        for (int i = 0; i < VEC; ++i) v[i] = fmaf(m, old[s][i], v[i]);
                    }
                }
                if (A.update) hc_store<VEC>(xr + (size_t)o * H + c, v);
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[i] = old[o][i];
            }
            const float wi = in_s[o];
#pragma unroll
            for (int i = 0; i < VEC; ++i) u[i] = fmaf(wi, v[i], u[i]);
        }
    };
    auto store = [&](int c, float (&u)[VEC], float inv) {
        float ww[VEC];
        hc_load<VEC>(A.w + c, ww);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = u[i] * inv * ww[i];
        hc_store<VEC>(out + (size_t)blockIdx.x * H + c, u);
    };

    float ss = 0.f;
    if constexpr (ONE) {
        const int c = threadIdx.x * VEC;
        const bool in = c < H;
        float old[N][VEC], d[HC_MAX_SLICES][VEC], y[VEC], u[VEC];
        if (in) {
#pragma unroll
            for (int s = 0; s < HC_MAX_SLICES; ++s)
                if (s < A.S) load_slice(s, c, d[s]);
            load_old(c, old);
        }
        if (normed) {
#pragma unroll
            for (int s = 0; s < HC_MAX_SLICES; ++s)
                if (in && s < A.S) square(s, d[s]);
            finish_factors();
        } else {
            __syncthreads();                                 // the weights are in shared memory
        }
        if (in) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = 0.f;
#pragma unroll
            for (int s = 0; s < HC_MAX_SLICES; ++s)
                if (s < A.S) add_slice(s, c, d[s], y);
            apply(c, old, y, u);
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(u[i], u[i], ss);
        }
        ss = ap_block_sum(ss, scratch);
        if (in) store(c, u, 1.0f / sqrtf(ss / (float)H + A.eps));
    } else {
        if (normed) {
            for (int c = threadIdx.x * VEC; c < H; c += blockDim.x * VEC) {
#pragma unroll
                for (int s = 0; s < HC_MAX_SLICES; ++s)
                    if (s < A.S) {
                        float d[VEC];
                        load_slice(s, c, d);
                        square(s, d);
                    }
            }
            finish_factors();
        } else {
            __syncthreads();
        }
        for (int c = threadIdx.x * VEC; c < H; c += blockDim.x * VEC) {
            float old[N][VEC], y[VEC], u[VEC];
            load_old(c, old);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = 0.f;
#pragma unroll
            for (int s = 0; s < HC_MAX_SLICES; ++s)
                if (s < A.S) {
                    float d[VEC];
                    load_slice(s, c, d);
                    add_slice(s, c, d, y);
                }
            apply(c, old, y, u);
            hc_store<VEC>(u_s + c, u);
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(u[i], u[i], ss);
        }
        ss = ap_block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)H + A.eps);
        // a thread reads back the columns it wrote itself
        for (int c = threadIdx.x * VEC; c < H; c += blockDim.x * VEC) {
            float u[VEC];
            hc_load<VEC>(u_s + c, u);
            store(c, u, inv);
        }
    }
}

// One stream, one pending slice over its own root mean square:
//   x <- mix x + out_w (scale rmsnorm(delta) slice_w)        out = rmsnorm(in_w x) w
// A thread holds PV runs of four columns of both rows in registers through the two sums over the row.
template <int PV, typename TO>
__global__ void __launch_bounds__(512) one_stream_norm_kernel(const StreamNormArgs A, TO* __restrict__ out) {
    __shared__ float first_s[32], second_s[32];
    ap_pdl_trigger();
    const float mix = A.mix[0], out_w = A.out_w[0] * A.slice_scale, in_w = A.in_w[0];
    ap_pdl_wait();
    const int H = A.H;
    const size_t t = A.rows ? (size_t)A.rows[blockIdx.x] : (size_t)blockIdx.x;
    float* xr = A.x + t * H;
    const float* dr = A.delta + t * H;
    float4 d[PV], x[PV];
#pragma unroll
    for (int j = 0; j < PV; ++j) {
        const int c = (j * (int)blockDim.x + (int)threadIdx.x) * 4;
        d[j] = x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < H) {
            d[j] = *reinterpret_cast<const float4*>(dr + c);
            x[j] = *reinterpret_cast<const float4*>(xr + c);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PV; ++j) ss = fmaf(d[j].x, d[j].x, fmaf(d[j].y, d[j].y, fmaf(d[j].z, d[j].z, fmaf(d[j].w, d[j].w, ss))));
    ss = ap_block_sum(ss, first_s);
    const float f = out_w / sqrtf(ss / (float)H + A.slice_eps);
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < PV; ++j) {
        const int c = (j * (int)blockDim.x + (int)threadIdx.x) * 4;
        if (c < H) {
            const float4 w = *reinterpret_cast<const float4*>(A.slice_w + c);
            x[j].x = fmaf(mix, x[j].x, f * d[j].x * w.x);
            x[j].y = fmaf(mix, x[j].y, f * d[j].y * w.y);
            x[j].z = fmaf(mix, x[j].z, f * d[j].z * w.z);
            x[j].w = fmaf(mix, x[j].w, f * d[j].w * w.w);
            if (A.update) *reinterpret_cast<float4*>(xr + c) = x[j];
        }
        x[j].x *= in_w; x[j].y *= in_w; x[j].z *= in_w; x[j].w *= in_w;
        ss = fmaf(x[j].x, x[j].x, fmaf(x[j].y, x[j].y, fmaf(x[j].z, x[j].z, fmaf(x[j].w, x[j].w, ss))));
    }
    ss = ap_block_sum(ss, second_s);
    const float inv = 1.0f / sqrtf(ss / (float)H + A.eps);
#pragma unroll
    for (int j = 0; j < PV; ++j) {
        const int c = (j * (int)blockDim.x + (int)threadIdx.x) * 4;
        if (c < H) {
            const float4 w = *reinterpret_cast<const float4*>(A.w + c);
            const float v[4] = {x[j].x * inv * w.x, x[j].y * inv * w.y, x[j].z * inv * w.z, x[j].w * inv * w.w};
            hc_store<4>(out + (size_t)blockIdx.x * H + c, v);
        }
    }
}

AP_EXPORT int ap_stream_norm(float* x, const int* rows, int R, const float* delta, int S, long long slice_stride,
                             const float* slice_bias, const float* slice_w, float slice_eps, float slice_scale,
                             const float* out_w, const float* mix, const float* in_w, const float* w, float eps,
                             int update, void* out, int out_dtype, int streams, int H, cudaStream_t stream) {
    AP_REQUIRE(R >= 0 && H > 0 && x && in_w && w && out, "stream_norm: bad arguments R=%d H=%d", R, H);
    AP_REQUIRE(streams >= 1 && streams <= HC_MAX_STREAMS, "stream_norm: %d streams are not in 1..%d", streams, HC_MAX_STREAMS);
    AP_REQUIRE(delta == nullptr || (S >= 1 && S <= HC_MAX_SLICES && out_w), "stream_norm: %d slices of pending sums are not "
               "in 1..%d, or the streams' weights on them are missing", S, HC_MAX_SLICES);
    AP_REQUIRE(!(update && rows), "stream_norm: chosen rows leave the streams alone");
    if (R == 0) return AP_OK;
    const bool vec = H % 4 == 0 && slice_stride % 4 == 0 &&
                     ((((uintptr_t)x) | ((uintptr_t)delta) | ((uintptr_t)slice_bias) | ((uintptr_t)slice_w) | ((uintptr_t)w)) & 15) == 0 &&
                     (((uintptr_t)out) & (out_dtype == AP_F32 ? 15 : 7)) == 0;
    int threads = ((vec ? H / 4 : H) + 31) / 32 * 32;
    const bool built = streams <= 4 || streams == 6 || streams == 8;       // (else the kernel for any number)
    const bool one = built && vec && threads <= (streams <= 4 ? 1024 : 512);   // a row in one pass, kept in registers
    if (!one && threads > 512) threads = 512;
    const size_t smem = one ? 0 : (size_t)H * sizeof(float);
    AP_REQUIRE(smem <= 200 * 1024, "stream_norm: a row of %d does not fit shared memory", H);
    StreamNormArgs A;
    A.x = x; A.rows = rows; A.delta = delta; A.S = delta ? S : 0; A.slice_stride = (size_t)slice_stride;
    A.slice_bias = slice_bias; A.slice_w = slice_w; A.slice_eps = slice_eps; A.slice_scale = slice_scale;
    A.out_w = out_w; A.mix = mix; A.in_w = in_w; A.w = w; A.eps = eps; A.update = (update && delta) ? 1 : 0;
    A.streams = streams; A.H = H;
    AP_REQUIRE(out_dtype == AP_F32 || out_dtype == AP_BF16, "stream_norm: unknown dtype %d", out_dtype);
    if (streams == 1 && vec && delta && S == 1 && slice_w && !slice_bias && mix && H <= 16384) {
        // runs of four columns to a thread: in a step of many rows more of them, so that an SM holds many rows at once
        const int runs = H / 4, want = R >= 4 * 148 ? 128 : 512;
        int pv = 1;
        while (pv < 8 && (runs + pv - 1) / pv > want) pv *= 2;
        const int nt = ((runs + pv - 1) / pv + 31) / 32 * 32;
#define LAUNCH_ONE(PV)                                                                                              \
        do {                                                                                                        \
            if (out_dtype == AP_F32)                                                                                \
                AP_CHECK_PDL_LAUNCH("stream_norm", ap_launch_pdl(one_stream_norm_kernel<PV, float>, dim3((unsigned)R), dim3(nt), 0, stream, A, (float*)out)); \
            else                                                                                                    \
                AP_CHECK_PDL_LAUNCH("stream_norm", ap_launch_pdl(one_stream_norm_kernel<PV, bf16>, dim3((unsigned)R), dim3(nt), 0, stream, A, (bf16*)out));   \
        } while (0)
        if (pv == 1) LAUNCH_ONE(1);
        else if (pv == 2) LAUNCH_ONE(2);
        else if (pv == 4) LAUNCH_ONE(4);
        else LAUNCH_ONE(8);
#undef LAUNCH_ONE
        return AP_OK;
    }
#define LAUNCH(N, V, ONE, TO)                                                                                       \
    do {                                                                                                            \
        auto kern = stream_norm_kernel<N, V, ONE, TO>;                                                                  \
        if (smem > 40 * 1024) {                                                                                     \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
            AP_REQUIRE(e == cudaSuccess, "stream_norm: cannot reserve %zu bytes of shared memory", smem);           \
        }                                                                                                           \
        AP_CHECK_PDL_LAUNCH("stream_norm", ap_launch_pdl(kern, dim3((unsigned)R), dim3(threads), smem, stream, A, (TO*)out)); \
    } while (0)
#define LAUNCH_T(N, V, ONE) do { if (out_dtype == AP_F32) LAUNCH(N, V, ONE, float); else LAUNCH(N, V, ONE, bf16); } while (0)
#define LAUNCH_V(N) do { if (one) LAUNCH_T(N, 4, true); else if (vec) LAUNCH_T(N, 4, false); else LAUNCH_T(N, 1, false); } while (0)
    switch (streams) {
        case 1: LAUNCH_V(1); break;
        case 2: LAUNCH_V(2); break;
        case 3: LAUNCH_V(3); break;
        case 4: LAUNCH_V(4); break;
        case 6: LAUNCH_V(6); break;
        case 8: LAUNCH_V(8); break;
        default: LAUNCH_T(0, 1, false);
    }
#undef LAUNCH_V
#undef LAUNCH_T
#undef LAUNCH
    return AP_OK;
}
