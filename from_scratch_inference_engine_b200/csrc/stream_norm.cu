// A residual of several streams (hyper-connections): per token `streams` rows x_1 .. x_s of the model's
// width, side by side in 32-bit.  One kernel settles what the sublayer before left pending, forms
// the next sublayer's input and norms it, in one pass over the token's streams:
//
//   settle     x_t <- sum_r mix[r, t] x_r + out[t] y      for all t at once, from the old streams
//              (only with a pending output y; written back when write_x; with y_scale [width] the
//              output is first multiplied by it column by column)
//   gather     u = sum_t in[t] x_t                        (in = null: the plain sum)
//   norm       centred: z = T( (u - mean) / sqrt(mean((u - mean)^2) + eps) * gain + bias )
//              else:    z = T( u / sqrt(mean(u^2) + eps) * gain + bias )
//
// With `start` [tokens, width] the streams do not exist yet: every one equals the token's row of it
// (they come into being with the first settled output).  Row r of z belongs to token rows ? rows[r]
// : r.  Everything is 32-bit but y and z, which have the storage type T.
#include "common.cuh"
#include <math.h>

namespace fsie {

struct StreamNormParams {
    float* x;                      // [tokens, streams, width]
    const float* start;            // [tokens, width] or null
    const void* y;                 // [tokens, width] of T, or null: nothing pending
    const float* y_scale;          // [width], or null: y as it is
    const float* mix;              // [streams, streams], from x to
    const float* out;              // [streams]
    const float* in;               // [streams] or null
    const float* gain;             // [width]
    const float* bias;             // [width] or null
    const int* rows;
    void* z;                       // [num_rows, width] of T, or null
    int streams, width, write_x, centred;
    float eps;
};

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store4(bf16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ void load4(const float* p, float (&v)[1]) { v[0] = *p; }
__device__ __forceinline__ void load4(const bf16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
__device__ __forceinline__ void store4(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void store4(bf16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }

// S: the number of streams, or 0: any number, a thread's old values wait in shared memory.
// STEP: columns per thread and trip (4: the width is a multiple of 4 and every row starts on 16
// bytes, or 8 for bfloat16).
template <typename T, int S, int STEP>
__global__ void __launch_bounds__(512, S > 0 && S <= 4 ? 2 : 1) stream_norm_kernel(const StreamNormParams p) {
    extern __shared__ __align__(16) float sn_smem[];
    __shared__ float scratch[32];
    const int streams = S > 0 ? S : p.streams, width = p.width;
    float* u = sn_smem;                               // [width], rounded up to 4
    float* mix = u + ((width + 3) & ~3);              // [streams, streams]
    float* out = mix + streams * streams;             // [streams]
    float* in = out + streams;                        // [streams]
    float* stash = in + streams;                      // S == 0: [streams][threads]
    // the coefficients are the model's: they are fetched while the kernel before still runs
    const bool settle = p.y != nullptr;
    for (int i = threadIdx.x; i < streams * streams; i += blockDim.x) mix[i] = settle ? p.mix[i] : 0.f;
    for (int i = threadIdx.x; i < streams; i += blockDim.x) {
        out[i] = settle ? p.out[i] : 0.f;
        in[i] = p.in ? p.in[i] : 1.f;
    }
    __syncthreads();
    grid_dependency_wait();
    grid_dependents_go();
    const int r = blockIdx.x;
    const size_t t = p.rows ? (size_t)p.rows[r] : (size_t)r;
    float* xr = p.x + t * streams * width;
    const float* sr = p.start ? p.start + t * width : nullptr;
    const T* yr = settle ? (const T*)p.y + t * width : nullptr;
    float sum = 0.f;
    for (int c = threadIdx.x * STEP; c < width; c += blockDim.x * STEP) {
        float acc[STEP], v[STEP];
#pragma unroll
        for (int i = 0; i < STEP; ++i) acc[i] = 0.f;
        if (S > 0) {
            float old[S > 0 ? S : 1][STEP], y[STEP];
            if (settle) {
                load4(yr + c, y);
                if (p.y_scale) {
                    load4(p.y_scale + c, v);
#pragma unroll
                    for (int i = 0; i < STEP; ++i) y[i] *= v[i];
                }
            }
            if (sr) {
                load4(sr + c, old[0]);
#pragma unroll
                for (int a = 1; a < S; ++a)
#pragma unroll
                    for (int i = 0; i < STEP; ++i) old[a][i] = old[0][i];
            } else {
#pragma unroll
                for (int a = 0; a < S; ++a) load4(xr + (size_t)a * width + c, old[a]);
            }
#pragma unroll
            for (int b = 0; b < S; ++b) {
                if (settle) {
                    const float ob = out[b];
#pragma unroll
                    for (int i = 0; i < STEP; ++i) v[i] = ob * y[i];
#pragma unroll
                    for (int a = 0; a < S; ++a) {
                        const float m = mix[a * S + b];
#pragma unroll
                        for (int i = 0; i < STEP; ++i) v[i] = fmaf(m, old[a][i], v[i]);
                    }
                    if (p.write_x) store4(xr + (size_t)b * width + c, v);
                } else {
#pragma unroll
                    for (int i = 0; i < STEP; ++i) v[i] = old[b][i];
                }
                const float w = in[b];
#pragma unroll
                for (int i = 0; i < STEP; ++i) acc[i] = fmaf(w, v[i], acc[i]);
            }
        } else {
            for (int i = 0; i < STEP; ++i) {
                float* mine = stash + threadIdx.x;
                for (int a = 0; a < streams; ++a)
                    mine[a * blockDim.x] = sr ? sr[c + i] : xr[(size_t)a * width + c + i];
                const float y = settle ? to_float(yr[c + i]) * (p.y_scale ? p.y_scale[c + i] : 1.f) : 0.f;
                for (int b = 0; b < streams; ++b) {
                    float nv = mine[b * blockDim.x];
                    if (settle) {
                        nv = out[b] * y;
                        for (int a = 0; a < streams; ++a) nv = fmaf(mix[a * streams + b], mine[a * blockDim.x], nv);
                        if (p.write_x) xr[(size_t)b * width + c + i] = nv;
                    }
                    acc[i] = fmaf(in[b], nv, acc[i]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < STEP; ++i) sum += p.centred ? acc[i] : acc[i] * acc[i];
        store4(u + c, acc);
    }
    if (!p.z) return;
    // every thread reads back only what it wrote itself: no barrier is needed before these loops
    float mean = 0.f, var = block_sum(sum, scratch) / (float)width;
    if (p.centred) {
        mean = var;
        float sq = 0.f;
        for (int c = threadIdx.x * STEP; c < width; c += blockDim.x * STEP) {
#pragma unroll
            for (int i = 0; i < STEP; ++i) {
                const float d = u[c + i] - mean;
                sq += d * d;
            }
        }
        var = block_sum(sq, scratch) / (float)width;
    }
    const float inv = 1.0f / sqrtf(var + p.eps);
    T* zr = (T*)p.z + (size_t)r * width;
    for (int c = threadIdx.x * STEP; c < width; c += blockDim.x * STEP) {
        float v[STEP], g[STEP], b[STEP];
        load4(u + c, v);
        load4(p.gain + c, g);
        if (p.bias) load4(p.bias + c, b);
#pragma unroll
        for (int i = 0; i < STEP; ++i) {
            v[i] = (v[i] - mean) * inv * g[i];
            if (p.bias) v[i] += b[i];
        }
        store4(zr + c, v);
    }
}

template <typename T, int S, int STEP>
static int stream_norm_launch(const StreamNormParams& p, int num_rows, cudaStream_t stream) {
    const int columns = (p.width + STEP - 1) / STEP;
    // few rows: as many threads as there is work for, so that a row is one trip to memory; many rows:
    // smaller blocks, more of which fit beside one another
    const int threads = S == 0 ? 128 : (num_rows <= 64 && columns >= 512 ? 512 : (columns >= 256 ? 256 : 128));
    const size_t floats = (size_t)((p.width + 3) & ~3) + (size_t)p.streams * p.streams + 2 * (size_t)p.streams +
                          (S == 0 ? (size_t)p.streams * threads : 0);
    const size_t smem = floats * sizeof(float);
    if (smem > 200 * 1024) return ERR_UNSUPPORTED;
    if (smem > 48 * 1024)
        cudaFuncSetAttribute(stream_norm_kernel<T, S, STEP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return launch_dependent(stream_norm_kernel<T, S, STEP>, num_rows, threads, smem, stream, p);
}

template <typename T, int STEP>
static int stream_norm_dispatch(const StreamNormParams& p, int num_rows, cudaStream_t stream) {
    switch (p.streams) {
        case 1: return stream_norm_launch<T, 1, STEP>(p, num_rows, stream);
        case 2: return stream_norm_launch<T, 2, STEP>(p, num_rows, stream);
        case 3: return stream_norm_launch<T, 3, STEP>(p, num_rows, stream);
        case 4: return stream_norm_launch<T, 4, STEP>(p, num_rows, stream);
        case 5: return stream_norm_launch<T, 5, STEP>(p, num_rows, stream);
        case 6: return stream_norm_launch<T, 6, STEP>(p, num_rows, stream);
        case 7: return stream_norm_launch<T, 7, STEP>(p, num_rows, stream);
        case 8: return stream_norm_launch<T, 8, STEP>(p, num_rows, stream);
        default: return stream_norm_launch<T, 0, 1>(p, num_rows, stream);
    }
}

}  // namespace fsie

using namespace fsie;

extern "C" {

int fsie_stream_norm(float* x, const float* start, const void* y, const float* y_scale, const float* mix, const float* out,
                     const float* in, const float* gain, const float* bias, const int* rows, void* z,
                     int num_rows, int streams, int width, float eps, int write_x, int centred, int dtype,
                     cudaStream_t stream) {
    if (num_rows <= 0) return 0;
    if (streams <= 0 || width <= 0 || !x || (y && (!mix || !out)) || (z && !gain) || (!y && !z)) return ERR_BAD_ARGUMENT;
    StreamNormParams p;
    p.x = x; p.start = start; p.y = y; p.y_scale = y_scale; p.mix = mix; p.out = out; p.in = in; p.gain = gain; p.bias = bias;
    p.rows = rows; p.z = z; p.streams = streams; p.width = width; p.write_x = write_x; p.centred = centred;
    p.eps = eps;
    const size_t wide = (size_t)x | (size_t)start | (size_t)gain | (size_t)bias | (size_t)y_scale;
    const size_t stored = (size_t)y | (size_t)z;
    const bool vec = width % 4 == 0 && (wide & 15) == 0 && (stored & (dtype == DTYPE_F32 ? 15 : 7)) == 0;
    if (dtype == DTYPE_F32)
        return vec ? stream_norm_dispatch<float, 4>(p, num_rows, stream) : stream_norm_dispatch<float, 1>(p, num_rows, stream);
    return vec ? stream_norm_dispatch<bf16, 4>(p, num_rows, stream) : stream_norm_dispatch<bf16, 1>(p, num_rows, stream);
}

}  // extern "C"
