// Linear attention with a per-head decay ("lightning attention") over per-request state.
//
//   q_t, k_t = silu(projected q, k)  [heads, dim]     v_t = silu(projected v)  [heads, vdim]
//   S_t = decay_h * S_{t-1} + k_t v_t^T               o_t = S_t^T q_t
//   y_t = T( o_t / sqrt(mean(o_t^2) + eps) * gain * sigmoid(g_t) )      over all heads together
//
// The state S [heads, dim, vdim] of a request is 32-bit and lives in its state slot; a step
// carries it on from where the step before left it, token by token in the order of the
// sequence, so the result does not depend on how the tokens were cut into steps beyond rounding
// (long prompts sum chunk by chunk).  The activations, the decay, the state and the output o are
// 32-bit whatever the storage type.
//
// The scan also serves recurrences with a decay per token, head and state row (`decay_row` [tokens, heads *
// dim]; gated linear attention: S_t = diag(a_t) S_(t-1) + k_t v_t^T) whose projections may be read as they
// are stored (T), and recurrences of the same form with a decay per token and head (`decay_tok`
// [tokens, heads] in place of the constant per head) and with q and k columns that `share` heads
// read together (head h reads the q and k of column group h / share): a state-space mixer's
// S_t = a_t S_(t-1) + B_t (dt_t x_t)^T, o_t = S_t^T C_t.  A request's state starts `state_stride`
// floats after the one before it (a slot may hold more than S).
#include "common.cuh"

namespace fsie {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

constexpr int SCAN_COLS = 32;      // value columns of one block
constexpr int SCAN_ROW_GROUPS = 16;// threads that share four columns; thread r owns rows r DR .. r DR + DR - 1

// four neighbouring values as 32-bit numbers; p starts on four elements
__device__ __forceinline__ float4 scan_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 scan_load4(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void scan_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void scan_store4(bf16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// where row d of a staged q or k vector lives: the DR rows of a thread are contiguous (one or
// more 16-byte loads) and the groups are four floats apart in the banks
template <int DR> __device__ __forceinline__ int scan_row_at(int d) {
    constexpr int PAD = DR > 4 ? DR + 4 : DR;
    return (d / DR) * PAD + d % DR;
}

// grid (column slices of 32, heads, segments), 128 threads.  Thread (row group r, column group c)
// keeps the DR x 4 patch S[r DR + i][4 c + x] in registers: a staged k or q value serves four
// columns and a v value DR rows, so the arithmetic, not shared memory, sets the pace; the
// output's sum over the rows is finished by shuffles among the 16 row groups.
//
// A block works on one segment of one request: the whole of its new tokens (seg_item == nullptr:
// segment z is request z, the state comes from and goes back to the request's slot), or one
// chunk of them.  Chunks make a long prompt parallel: every chunk first sums its own tokens
// from a zero state (`chunk_states` receives the sum, nothing else is written), a second kernel
// chains the sums into the state at every chunk's start, and every chunk then runs again from
// that state and writes the outputs.
// ROWS: a decay per state row (decay_row); the outputs are multiplied by out_scale.
template <int DR, typename T, bool ROWS>
__global__ void __launch_bounds__(SCAN_COLS / 4 * SCAN_ROW_GROUPS)
lightning_scan_kernel(const T* __restrict__ proj, int ld, int q_off, int k_off, int v_off,
                      const int* __restrict__ item_qstart, const int* __restrict__ item_qlen,
                      const int* __restrict__ item_slots, float* __restrict__ state,
                      const float* __restrict__ decay, float* __restrict__ out, int heads, int dim,
                      int vdim, const int* __restrict__ seg_item, const int* __restrict__ seg_row0,
                      int seg_tokens, float* __restrict__ chunk_states, int phase, int share,
                      const float* __restrict__ decay_tok, const float* __restrict__ decay_row,
                      float out_scale, long long state_stride, float* __restrict__ chunk_decay) {
    // tokens staged in shared memory at a time (fewer where q, k and the rows' decays of large heads are staged)
    constexpr int SCAN_TOKENS = ROWS && DR > 8 ? 8 : 16;
    constexpr int PAD = DR > 4 ? DR + 4 : DR;
    constexpr int ROW_LEN = SCAN_ROW_GROUPS * PAD;
    __shared__ __align__(16) float qs[SCAN_TOKENS * ROW_LEN];
    __shared__ __align__(16) float ks[SCAN_TOKENS * ROW_LEN];
    __shared__ __align__(16) float vs[SCAN_TOKENS * SCAN_COLS];
    __shared__ float ls[SCAN_TOKENS];                  // the decay of each staged token
    __shared__ __align__(16) float as[ROWS ? SCAN_TOKENS * ROW_LEN : 4];     // ... or of each of its state rows
    grid_dependency_wait();
    grid_dependents_go();
    const int item = seg_item ? seg_item[blockIdx.z] : blockIdx.z, head = blockIdx.y;
    const int slot = item_slots[item];
    if (slot < 0) return;                              // a padding entry of a fixed-size batch
    const int row0 = seg_item ? seg_row0[blockIdx.z] : 0;
    const int start = item_qstart[item] + row0;
    const int count = seg_item ? min(seg_tokens, item_qlen[item] - row0) : item_qlen[item];
    // phase 0: from the slot, outputs, back to the slot; 1: from zero, the sum to chunk_states;
    // 2: from chunk_states (the state at the chunk's start), outputs
    const bool from_zero = phase == 1, write_out = phase != 1;
    const int rg = threadIdx.x & (SCAN_ROW_GROUPS - 1), cg = threadIdx.x / SCAN_ROW_GROUPS;
    const int col0 = blockIdx.x * SCAN_COLS + cg * 4;
    const bool wide = (vdim & 3) == 0 && (state_stride & 3) == 0;                 // rows of the state start on 16 bytes
    // q and k rows of a head start on 16 bytes and end on them: staged four values at a time
    const bool vec = DR * SCAN_ROW_GROUPS >= 4 && ((dim | ld | q_off | k_off) & 3) == 0;
    float* mine = (phase == 0 ? state + (size_t)slot * state_stride + ((size_t)head * dim) * vdim
                              : chunk_states + (((size_t)blockIdx.z * heads + head) * dim) * vdim);
    const float head_decay = decay ? decay[head] : 1.f;
    const int qk_head = head / share;                  // `share` heads read the same q and k columns
    float through = 1.f;                               // the product of the chunk's decays (phase 1)
    float s[DR][4];
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int d = rg * DR + i;
        s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
        if (from_zero || d >= dim || col0 >= vdim) continue;
        const float* at = mine + (size_t)d * vdim + col0;
        if (wide) {
            const float4 v = *reinterpret_cast<const float4*>(at);
            s[i][0] = v.x; s[i][1] = v.y; s[i][2] = v.z; s[i][3] = v.w;
        } else {
#pragma unroll
            for (int x = 0; x < 4; ++x) if (col0 + x < vdim) s[i][x] = at[x];
        }
    }
    for (int t0 = 0; t0 < count; t0 += SCAN_TOKENS) {
        const int n = min(SCAN_TOKENS, count - t0);
        __syncthreads();
        if (vec) {
            constexpr int CHUNKS = SCAN_ROW_GROUPS * DR / 4 > 0 ? SCAN_ROW_GROUPS * DR / 4 : 1;
            for (int idx = threadIdx.x; idx < n * CHUNKS; idx += blockDim.x) {
                const int t = idx / CHUNKS, d = (idx - t * CHUNKS) * 4;
                const T* row = proj + (size_t)(start + t0 + t) * ld + qk_head * dim + d;
                const int at = t * ROW_LEN + scan_row_at<DR>(d);
                const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
                if (write_out)
                    *reinterpret_cast<float4*>(qs + at) = d < dim ? scan_load4(row + q_off) : zero;
                *reinterpret_cast<float4*>(ks + at) = d < dim ? scan_load4(row + k_off) : zero;
                if (ROWS)
                    *reinterpret_cast<float4*>(as + at) = d < dim ? scan_load4(decay_row + ((size_t)(start + t0 + t) * heads + head) * dim + d) : zero;
            }
        } else {
            for (int idx = threadIdx.x; idx < n * SCAN_ROW_GROUPS * DR; idx += blockDim.x) {
                const int t = idx / (SCAN_ROW_GROUPS * DR), d = idx - t * (SCAN_ROW_GROUPS * DR);
                const T* row = proj + (size_t)(start + t0 + t) * ld + qk_head * dim + d;
                const int at = t * ROW_LEN + scan_row_at<DR>(d);
                if (write_out) qs[at] = d < dim ? to_float(row[q_off]) : 0.f;
                ks[at] = d < dim ? to_float(row[k_off]) : 0.f;
                if (ROWS) as[at] = d < dim ? decay_row[((size_t)(start + t0 + t) * heads + head) * dim + d] : 0.f;
            }
        }
        for (int idx = threadIdx.x; idx < n * SCAN_COLS; idx += blockDim.x) {
            const int t = idx / SCAN_COLS, c = idx - t * SCAN_COLS;
            const int cc = blockIdx.x * SCAN_COLS + c;
            vs[idx] = cc < vdim ? to_float(proj[(size_t)(start + t0 + t) * ld + v_off + head * vdim + cc]) : 0.f;
        }
        if (!ROWS && threadIdx.x < n)
            ls[threadIdx.x] = decay_tok ? decay_tok[(size_t)(start + t0 + threadIdx.x) * heads + head] : head_decay;
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float lambda = ROWS ? 1.f : ls[t];
            through *= lambda;
            const float4 v4 = *reinterpret_cast<const float4*>(vs + t * SCAN_COLS + cg * 4);
            const float v[4] = {v4.x, v4.y, v4.z, v4.w};
            float kk[DR], qq[DR], aa[ROWS ? DR : 1];
            const float* kr = ks + t * ROW_LEN + rg * PAD;
            const float* ar = as + (ROWS ? t * ROW_LEN + rg * PAD : 0);
            const float* qr = qs + t * ROW_LEN + rg * PAD;
            if (DR >= 4) {
#pragma unroll
                for (int i = 0; i < DR; i += 4) {
                    const float4 a = *reinterpret_cast<const float4*>(kr + i);
                    kk[i] = a.x; kk[i + 1] = a.y; kk[i + 2] = a.z; kk[i + 3] = a.w;
                    if (ROWS) {
                        const float4 b = *reinterpret_cast<const float4*>(ar + i);
                        aa[i] = b.x; aa[i + 1] = b.y; aa[i + 2] = b.z; aa[i + 3] = b.w;
                    }
                    if (write_out) {
                        const float4 b = *reinterpret_cast<const float4*>(qr + i);
                        qq[i] = b.x; qq[i + 1] = b.y; qq[i + 2] = b.z; qq[i + 3] = b.w;
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < DR; ++i) {
                    kk[i] = kr[i];
                    if (ROWS) aa[i] = ar[i];
                    if (write_out) qq[i] = qr[i];
                }
            }
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < DR; ++i)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    s[i][x] = (ROWS ? aa[i] : lambda) * s[i][x] + kk[i] * v[x];
                    if (write_out) o[x] += s[i][x] * qq[i];
                }
            if (!write_out) continue;
            // the sum over the 16 row groups: the first two exchanges halve what a lane holds (four columns,
            // two, one), the last two add one column's parts; five exchanges, not sixteen
            const bool upper = rg & 1, odd = rg & 2;
            const float a0 = __shfl_xor_sync(0xffffffffu, upper ? o[0] : o[2], 1);
            const float a1 = __shfl_xor_sync(0xffffffffu, upper ? o[1] : o[3], 1);
            const float b0 = (upper ? o[2] : o[0]) + a0, b1 = (upper ? o[3] : o[1]) + a1;
            float sum = (odd ? b1 : b0) + __shfl_xor_sync(0xffffffffu, odd ? b0 : b1, 2);
            sum += __shfl_xor_sync(0xffffffffu, sum, 4);
            sum += __shfl_xor_sync(0xffffffffu, sum, 8);
            const int col = col0 + (upper ? 2 : 0) + (odd ? 1 : 0);
            if (rg < 4 && col < vdim)
                out[(size_t)(start + t0 + t) * heads * vdim + head * vdim + col] = sum * out_scale;
        }
    }
    if (!ROWS && phase == 1 && chunk_decay && blockIdx.x == 0 && threadIdx.x == 0)
        chunk_decay[(size_t)blockIdx.z * heads + head] = through;
    if (ROWS && phase == 1 && blockIdx.x == 0)         // the product of the chunk's decays, row by row
        for (int d = threadIdx.x; d < dim; d += blockDim.x) {
            const float* at = decay_row + ((size_t)start * heads + head) * dim + d;
            float product = 1.f;
#pragma unroll 8
            for (int t = 0; t < count; ++t) product *= at[(size_t)t * heads * dim];
            chunk_decay[((size_t)blockIdx.z * heads + head) * dim + d] = product;
        }
    if (phase != 2 && col0 < vdim) {
#pragma unroll
        for (int i = 0; i < DR; ++i) {
            const int d = rg * DR + i;
            if (d >= dim) continue;
            float* at = mine + (size_t)d * vdim + col0;
            if (wide) *reinterpret_cast<float4*>(at) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
            else {
#pragma unroll
                for (int x = 0; x < 4; ++x) if (col0 + x < vdim) at[x] = s[i][x];
            }
        }
    }
}

// act[t, c] = silu(proj[t, c]) for the first `width` columns (q, k and v), widened to 32-bit: the
// scan reads every value several times (once per column slice and walk), the activation is
// taken once.
template <typename T>
__global__ void silu_rows_kernel(const T* __restrict__ proj, int ld, int width, float* __restrict__ act,
                                 long long count) {
    grid_dependency_wait();
    grid_dependents_go();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < count;
         i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / width;
        const int c = (int)(i - t * width);
        act[i] = silu_f(to_float(proj[t * ld + c]));
    }
}

// Chains the chunks' sums of every request: chunk_states[c] (on entry the sum of chunk c's own
// tokens from a zero state) becomes the state at the start of chunk c, and the request's slot
// receives the state after its last chunk.  S_after = decay^len * S_before + sum.  One thread per
// state element; chunks are listed request by request, in order.
__global__ void lightning_chain_kernel(const int* __restrict__ item_qstart, const int* __restrict__ item_qlen,
                                       const int* __restrict__ item_slots,
                                       int items, float* __restrict__ state, const float* __restrict__ decay,
                                       float* __restrict__ chunk_states, int seg_tokens, int heads,
                                       int dim, int vdim, const float* __restrict__ chunk_decay, int by_row,
                                       long long state_stride) {
    const int item = blockIdx.y;
    const int slot = item_slots[item];
    if (slot < 0) return;
    const size_t per_head = (size_t)dim * vdim, per_state = per_head * heads;
    const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= per_state) return;
    int first = 0;                                         // index of this request's first chunk
    for (int i = 0; i < item; ++i) first += (item_qlen[i] + seg_tokens - 1) / seg_tokens;
    const int count = item_qlen[item];
    const int chunks = (count + seg_tokens - 1) / seg_tokens;
    const int head = (int)(e / per_head);
    const float lambda = decay ? decay[head] : 1.f;
    const int row = (int)((e - head * per_head) / vdim);
    float s = state[(size_t)slot * state_stride + e];
    for (int c = 0; c < chunks; ++c) {
        const int len = min(seg_tokens, count - c * seg_tokens);
        float* at = chunk_states + (size_t)(first + c) * per_state + e;
        const float sum = *at;
        *at = s;
        float power = 1.f;                                 // decay^len by the same products as the scan
        if (by_row) power = chunk_decay[((size_t)(first + c) * heads + head) * dim + row];
        else if (chunk_decay) power = chunk_decay[(size_t)(first + c) * heads + head];     // (what the chunk's walk multiplied)
        else for (int t = 0; t < len; ++t) power *= lambda;
        s = power * s + sum;
    }
    state[(size_t)slot * state_stride + e] = s;
}

// The decays of gated linear attention: a = sigmoid(z)^(1/tau) with z = low W^T + bias, low the token's `rank`
// columns of proj at low_off, W given as wt [rank, columns].  Through the logarithm, log sigmoid(z) = min(z, 0)
// - log(1 + e^-|z|), in 32-bit: what rounding 1 + e^-|z| loses is below a rounding of the result.  A thread owns a column of DECAY_TOKENS tokens: a weight is fetched once for all.
// The first DECAY_AHEAD of them are asked for while the kernel before still runs.
constexpr int DECAY_TOKENS = 16, DECAY_AHEAD = 16;
template <typename T>
__global__ void __launch_bounds__(128) row_decay_kernel(
        const T* __restrict__ proj, int ld, int low_off, int rank, const float* __restrict__ wt,
        const float* __restrict__ bias, float inv_tau, float* __restrict__ out, int tokens, int columns) {
    extern __shared__ __align__(16) float rd_low[];      // [rank][DECAY_TOKENS]
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    float w[DECAY_AHEAD];
#pragma unroll
    for (int r = 0; r < DECAY_AHEAD; ++r) w[r] = r < rank && c < columns ? wt[(size_t)r * columns + c] : 0.f;
    const float b = c < columns ? bias[c] : 0.f;
    grid_dependency_wait();
    grid_dependents_go();
    const int t0 = blockIdx.y * DECAY_TOKENS;
    const int n = min(DECAY_TOKENS, tokens - t0);
    for (int i = threadIdx.x; i < rank * DECAY_TOKENS; i += blockDim.x) {
        const int t = i / rank, r = i - t * rank;
        rd_low[r * DECAY_TOKENS + t] = t < n ? to_float(proj[(size_t)(t0 + t) * ld + low_off + r]) : 0.f;
    }
    __syncthreads();
    if (c >= columns) return;
    float z[DECAY_TOKENS];
#pragma unroll
    for (int t = 0; t < DECAY_TOKENS; ++t) z[t] = b;
    for (int r0 = 0; r0 < rank; r0 += DECAY_AHEAD) {
#pragma unroll
        for (int j = 0; j < DECAY_AHEAD; ++j) {
            if (r0 + j >= rank) break;
            const float4* low = reinterpret_cast<const float4*>(rd_low + (r0 + j) * DECAY_TOKENS);
#pragma unroll
            for (int q = 0; q < DECAY_TOKENS / 4; ++q) {
                const float4 v = low[q];
                z[4 * q] = fmaf(w[j], v.x, z[4 * q]);
                z[4 * q + 1] = fmaf(w[j], v.y, z[4 * q + 1]);
                z[4 * q + 2] = fmaf(w[j], v.z, z[4 * q + 2]);
                z[4 * q + 3] = fmaf(w[j], v.w, z[4 * q + 3]);
            }
        }
#pragma unroll
        for (int j = 0; j < DECAY_AHEAD; ++j) {
            const int r = r0 + DECAY_AHEAD + j;
            if (r < rank) w[j] = wt[(size_t)r * columns + c];
        }
    }
    float* dst = out + (size_t)t0 * columns + c;
#pragma unroll
    for (int t = 0; t < DECAY_TOKENS; ++t, dst += columns) {
        const float log_sigmoid = fminf(z[t], 0.f) - logf(1.0f + __expf(-fabsf(z[t])));
        const float a = expf(log_sigmoid * inv_tau);
        if (t < n) *dst = a;
    }
}

// A warp per (token, head): y = T( o / sqrt(mean(o^2) + eps) * gain * silu(gate) ), the mean over the head's vdim
// columns, the gain [vdim] shared by the heads.
// VEC columns side by side per lane.
template <typename T, int VEC>
__global__ void head_norm_silu_kernel(const float* __restrict__ o, const T* __restrict__ proj, int ld, int g_off,
                                      const float* __restrict__ gain, T* __restrict__ y, long long pairs, int heads,
                                      int vdim, float eps) {
    const int lane = threadIdx.x & 31;
    const long long pair = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    grid_dependency_wait();
    grid_dependents_go();
    if (pair >= pairs) return;
    const long long t = pair / heads;
    const int h = (int)(pair - t * heads);
    const float* row = o + pair * vdim;
    const T* gate = proj + t * ld + g_off + (size_t)h * vdim;
    T* yr = y + pair * vdim;
    float sq = 0.f;
    for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
        if (VEC == 4) {
            const float4 v = scan_load4(row + c);
            sq += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        } else {
            sq += row[c] * row[c];
        }
    }
    const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)vdim + eps);
    for (int c = lane * VEC; c < vdim; c += 32 * VEC) {
        if (VEC == 4) {
            const float4 v = scan_load4(row + c), w = scan_load4(gain + c), z = scan_load4(gate + c);
            scan_store4(yr + c, make_float4(v.x * inv * w.x * silu_f(z.x), v.y * inv * w.y * silu_f(z.y),
                                            v.z * inv * w.z * silu_f(z.z), v.w * inv * w.w * silu_f(z.w)));
        } else {
            yr[c] = from_float<T>(row[c] * inv * gain[c] * silu_f(to_float(gate[c])));
        }
    }
}

// One block per token: y = T( o * rsqrt(mean(o^2) + eps) * gain * sigmoid(gate) ).
template <typename T>
__global__ void gated_rmsnorm_kernel(const float* __restrict__ o, const T* __restrict__ proj, int ld,
                                     int g_off, const float* __restrict__ gain, T* __restrict__ y,
                                     int width, float eps) {
    __shared__ float scratch[32];
    grid_dependency_wait();
    grid_dependents_go();
    const size_t t = blockIdx.x;
    const float* row = o + t * width;
    float sq = 0.f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) sq += row[c] * row[c];
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)width + eps);
    const T* gate = proj + t * ld + g_off;
    T* yr = y + t * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float g = to_float(gate[c]);
        yr[c] = from_float<T>(row[c] * inv * gain[c] * (1.0f / (1.0f + expf(-g))));
    }
}

}  // namespace fsie

using namespace fsie;

extern "C" {

int fsie_silu_rows(const void* proj, int ld, int width, float* act, int tokens, int dtype,
                   cudaStream_t stream) {
    const long long count = (long long)tokens * width;
    if (count <= 0) return 0;
    const long long wanted = (count + 255) / 256;
    const unsigned blocks = (unsigned)(wanted > 8192 ? 8192 : wanted);
    if (dtype == DTYPE_F32)
        return launch_dependent(silu_rows_kernel<float>, blocks, 256, 0, stream, (const float*)proj, ld,
                                width, act, count);
    return launch_dependent(silu_rows_kernel<bf16>, blocks, 256, 0, stream, (const bf16*)proj, ld, width,
                            act, count);
}

// proj [tokens, ld] (float: the activations that fsie_silu_rows left) holds q at q_off, k at k_off
// (heads * dim each) and v at v_off (heads * vdim); state [slots, heads, dim, vdim]; out [tokens,
// heads * vdim] (float).
//
// With seg_item / seg_row0 (num_segs chunks of seg_tokens tokens, listed request by request) and
// chunk_states [num_segs, heads, dim, vdim] (with decay_tok: and num_segs * heads floats more, with decay_row
// num_segs * heads * dim more) the requests run chunk-parallel in three launches.  decay_row [tokens, heads *
// dim]: a decay per state row in place of the others; proj may then be of either storage type (`dtype`), else it
// is float.  The outputs are multiplied by out_scale.
int fsie_lightning_scan(const void* proj, int ld, int q_off, int k_off, int v_off,
                        const int* item_qstart, const int* item_qlen, const int* item_slots,
                        int items, float* state, const float* decay, float* out, int heads,
                        int dim, int vdim, const int* seg_item, const int* seg_row0, int num_segs,
                        int seg_tokens, float* chunk_states, int share, const float* decay_tok,
                        const float* decay_row, float out_scale, int dtype, long long state_stride,
                        cudaStream_t stream) {
    if (items <= 0) return 0;
    if (heads <= 0 || dim <= 0 || vdim <= 0 || heads > 65535 || items > 65535 || share <= 0 ||
        heads % share || (!decay && !decay_tok && !decay_row) || (dtype != DTYPE_F32 && !decay_row) || state_stride < (long long)heads * dim * vdim)
        return ERR_BAD_ARGUMENT;
    if (dim > SCAN_ROW_GROUPS * 16) return ERR_UNSUPPORTED;
    const bool chunked = seg_item != nullptr;
    if (chunked && (!seg_row0 || !chunk_states || num_segs <= 0 || num_segs > 65535 || seg_tokens <= 0))
        return ERR_BAD_ARGUMENT;
    // decays per token: every chunk's walk leaves the product of its decays behind its sums, for the chain
    float* chunk_decay = chunked && (decay_tok || decay_row) ? chunk_states + (size_t)num_segs * heads * dim * vdim : nullptr;
    dim3 grid((vdim + SCAN_COLS - 1) / SCAN_COLS, heads, chunked ? num_segs : items);
    int phase = chunked ? 1 : 0;
    const int threads = SCAN_COLS / 4 * SCAN_ROW_GROUPS;
    const int per_thread = (dim + SCAN_ROW_GROUPS - 1) / SCAN_ROW_GROUPS;
    int launch_code = 0;
#define FSIE_SCAN(T, R, DPT)                                                                     \
    launch_code = launch_dependent(lightning_scan_kernel<DPT, T, R>, grid, threads, 0, stream,   \
        (const T*)proj, ld, q_off, k_off, v_off, item_qstart, item_qlen, item_slots, state,      \
        decay, out, heads, dim, vdim, seg_item, seg_row0, seg_tokens, chunk_states, phase, share, \
        decay_tok, decay_row, out_scale, state_stride, chunk_decay)
#define FSIE_SCAN_SIZES(T, R)                                                                    \
    do {                                                                                         \
        if (per_thread <= 1) FSIE_SCAN(T, R, 1);                                                 \
        else if (per_thread <= 2) FSIE_SCAN(T, R, 2);                                            \
        else if (per_thread <= 4) FSIE_SCAN(T, R, 4);                                            \
        else if (per_thread <= 8) FSIE_SCAN(T, R, 8);                                            \
        else FSIE_SCAN(T, R, 16);                                                                \
    } while (0)
#define FSIE_SCAN_BY_SIZE()                                                                      \
    do {                                                                                         \
        if (!decay_row) FSIE_SCAN_SIZES(float, false);                                           \
        else if (dtype == DTYPE_F32) FSIE_SCAN_SIZES(float, true);                               \
        else FSIE_SCAN_SIZES(bf16, true);                                                        \
    } while (0)
    FSIE_SCAN_BY_SIZE();
    if (launch_code) return launch_code;
    if (chunked) {
        int code;
        const size_t per_state = (size_t)heads * dim * vdim;
        lightning_chain_kernel<<<dim3((unsigned)((per_state + 255) / 256), items), 256, 0, stream>>>(
            item_qstart, item_qlen, item_slots, items, state, decay, chunk_states, seg_tokens, heads, dim, vdim,
            chunk_decay, decay_row != nullptr, state_stride);
        code = FSIE_LAUNCH_CHECK();
        if (code) return code;
        phase = 2;
        FSIE_SCAN_BY_SIZE();
    }
#undef FSIE_SCAN_BY_SIZE
#undef FSIE_SCAN_SIZES
#undef FSIE_SCAN
    return launch_code;
}

// proj [tokens, ld] of storage type `dtype`, `rank` columns of it at low_off; wt float [rank, columns]; bias float
// [columns]; out float [tokens, columns] = sigmoid(low wt + bias)^inv_tau.
int fsie_row_decay(const void* proj, int ld, int low_off, int rank, const float* wt, const float* bias, float inv_tau,
                   float* out, int tokens, int columns, int dtype, cudaStream_t stream) {
    if (tokens <= 0 || columns <= 0) return 0;
    if (rank <= 0 || low_off < 0 || low_off + rank > ld) return ERR_BAD_ARGUMENT;
    const size_t smem = (size_t)rank * DECAY_TOKENS * sizeof(float);
    const int groups = (tokens + DECAY_TOKENS - 1) / DECAY_TOKENS;
    if (smem > 48 * 1024 || groups > 65535) return ERR_UNSUPPORTED;
    const dim3 grid((columns + 127) / 128, groups);
    if (dtype == DTYPE_F32)
        return launch_dependent(row_decay_kernel<float>, grid, dim3(128), smem, stream, (const float*)proj, ld, low_off,
                                rank, wt, bias, inv_tau, out, tokens, columns);
    return launch_dependent(row_decay_kernel<bf16>, grid, dim3(128), smem, stream, (const bf16*)proj, ld, low_off, rank,
                            wt, bias, inv_tau, out, tokens, columns);
}

// o float [tokens, heads * vdim]; gate columns of proj [tokens, ld] at g_off; gain float [vdim]; y [tokens, heads * vdim].
int fsie_head_norm_silu(const float* o, const void* proj, int ld, int g_off, const float* gain, void* y, int tokens,
                        int heads, int vdim, float eps, int dtype, cudaStream_t stream) {
    const long long pairs = (long long)tokens * heads;
    if (pairs <= 0 || vdim <= 0) return 0;
    const dim3 grid((unsigned)((pairs + 3) / 4));
    const bool vec = ((vdim | ld | g_off) & 3) == 0 && (((size_t)o | (size_t)gain | (size_t)proj | (size_t)y) & 15) == 0;
#define FSIE_HEAD_NORM(T, V)                                                                                     \
    launch_dependent(head_norm_silu_kernel<T, V>, grid, dim3(128), 0, stream, o, (const T*)proj, ld, g_off, gain, \
                     (T*)y, pairs, heads, vdim, eps)
    if (dtype == DTYPE_F32) return vec ? FSIE_HEAD_NORM(float, 4) : FSIE_HEAD_NORM(float, 1);
    return vec ? FSIE_HEAD_NORM(bf16, 4) : FSIE_HEAD_NORM(bf16, 1);
#undef FSIE_HEAD_NORM
}

int fsie_gated_rmsnorm(const float* o, const void* proj, int ld, int g_off, const float* gain,
                       void* y, int tokens, int width, float eps, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    const int threads = width >= 2048 ? 512 : (width >= 512 ? 256 : 128);
    if (dtype == DTYPE_F32)
        return launch_dependent(gated_rmsnorm_kernel<float>, tokens, threads, 0, stream, o,
                                (const float*)proj, ld, g_off, gain, (float*)y, width, eps);
    return launch_dependent(gated_rmsnorm_kernel<bf16>, tokens, threads, 0, stream, o,
                            (const bf16*)proj, ld, g_off, gain, (bf16*)y, width, eps);
}

}  // extern "C"
