// Kernels around a residual stream that norms touch only behind the branches, and of mixers whose
// norm or rotation is not one head's own:
//   * stream update: x += rmsnorm(branch) * w; optionally the result joins a record of all layers'
//     results and the stream becomes a weighted sum over that record (an average over depth);
//     then the stream in the compute dtype, or a norm of it
//   * RMS norm over all query rows and over all key rows of a projection at once, rotation, values
//     turned by their position, cache write; and the turn back of the heads' outputs
//   * latent cache row with a rotated tail: RMS norm of the latent, rotation of the key part that
//     all heads share and of every query's own part
// Norms, angles, sums and the stream are float32; inputs and outputs are float32 or bfloat16.
#include "common.cuh"
#include "rotation.cuh"
#include "vec4.cuh"

namespace somi {

// ------------------------------------------------------------------- stream update
// d = sum_s delta[s][row] (partial sums `split_stride` apart, added in order)
// r = x_in[row] + (weight_b ? d / sqrt(mean(d^2) + eps_b) * weight_b : d)      (no delta: x_in[row])
// with coef:  X_0 = start, X_j = results[j - 1] for 0 < j < n, X_n = r;
//             results[n - 1][row] = r;  x = sum_{j <= n} coef[j] X_j[row]       (j ascending)
// else        x = r
// if write_back: x_out[row] = x.  out[b] = x in TO, or with `weight` x / sqrt(mean(x^2) + eps) * weight;
// row = rows ? rows[b] : b.  V vectors of four columns a thread, kept in registers.
template <typename TD, typename TO, int V>
__global__ void __launch_bounds__(V == 4 ? 512 : 1024)
stream_update_kernel(const float* x_in, float* x_out,       // (may be the same rows)
                     const TD* __restrict__ delta, int splits, long long split_stride,
                     const void* __restrict__ weight_b, int wb_dtype, float eps_b,
                     const float* __restrict__ start, float* __restrict__ results,
                     long long result_stride, int n, const float* __restrict__ coef,
                     const void* __restrict__ weight, int w_dtype, float eps, TO* __restrict__ out,
                     const int* __restrict__ rows, int H, int write_back) {
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x;
    const int row = rows ? rows[b] : b;
    const size_t base = static_cast<size_t>(row) * H;
    float x[V][4], d[V][4], acc[V][4];
    float ss = 0.f;
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int i = (threadIdx.x + v * blockDim.x) * 4;
#pragma unroll
        for (int c = 0; c < 4; ++c) x[v][c] = d[v][c] = acc[v][c] = 0.f;
        if (i < H) {
            const F4 t = load4(x_in + base + i);
#pragma unroll
            for (int c = 0; c < 4; ++c) x[v][c] = t.v[c];
            if (delta != nullptr) {
                F4 s = load4(delta + base + i);
#pragma unroll 4
                for (int k = 1; k < splits; ++k) {
                    const F4 e = load4(delta + static_cast<size_t>(k) * split_stride + base + i);
#pragma unroll
                    for (int c = 0; c < 4; ++c) s.v[c] += e.v[c];
                }
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    d[v][c] = s.v[c];
                    ss = fmaf(s.v[c], s.v[c], ss);
                }
            }
            if (coef != nullptr) {                    // the earlier results do not wait for the sum
                const F4 t0 = load4(start + base + i);
                const float c0 = coef[0];
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[v][c] = c0 * t0.v[c];
#pragma unroll 4
                for (int j = 1; j < n; ++j) {
                    const F4 e = load4(results + static_cast<size_t>(j - 1) * result_stride + base + i);
                    const float cj = coef[j];
#pragma unroll
                    for (int c = 0; c < 4; ++c) acc[v][c] = fmaf(cj, e.v[c], acc[v][c]);
                }
            }
        }
    }
    if (delta != nullptr) {
        float inv = 1.0f;
        if (weight_b != nullptr) {
            ss = block_sum(ss, scratch);
            inv = 1.0f / sqrtf(ss / static_cast<float>(H) + eps_b);
        }
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int i = (threadIdx.x + v * blockDim.x) * 4;
            if (i < H) {
                F4 w{{1.f, 1.f, 1.f, 1.f}};
                if (weight_b != nullptr) w = load4_any(weight_b, wb_dtype, i);
#pragma unroll
                for (int c = 0; c < 4; ++c) x[v][c] += d[v][c] * inv * w.v[c];
            }
        }
    }
    if (coef != nullptr) {
        const float cn = coef[n];
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int i = (threadIdx.x + v * blockDim.x) * 4;
            if (i < H) {
                F4 r;
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    r.v[c] = x[v][c];
                    x[v][c] = fmaf(cn, x[v][c], acc[v][c]);
                }
                if (write_back) store4(results + static_cast<size_t>(n - 1) * result_stride + base + i, r);
            }
        }
    }
    float inv = 1.0f;
    if (weight != nullptr) {
        ss = 0.f;
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
            for (int c = 0; c < 4; ++c) ss = fmaf(x[v][c], x[v][c], ss);
        ss = block_sum(ss, scratch);
        inv = 1.0f / sqrtf(ss / static_cast<float>(H) + eps);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int i = (threadIdx.x + v * blockDim.x) * 4;
        if (i >= H) continue;
        F4 y;
#pragma unroll
        for (int c = 0; c < 4; ++c) y.v[c] = x[v][c];
        if (write_back) store4(x_out + base + i, y);
        if (out != nullptr) {
            if (weight != nullptr) {
                const F4 w = load4_any(weight, w_dtype, i);
#pragma unroll
                for (int c = 0; c < 4; ++c) y.v[c] = y.v[c] * inv * w.v[c];
            }
            store4(out + static_cast<size_t>(b) * H + i, y);
        }
    }
}

// The same for any width: one column at a time, the row in shared memory ([H] floats).
template <typename TD, typename TO>
__global__ void stream_update_any_kernel(const float* x_in, float* x_out,
                                         const TD* __restrict__ delta, int splits, long long split_stride,
                                         const void* __restrict__ weight_b, int wb_dtype, float eps_b,
                                         const float* __restrict__ start, float* __restrict__ results,
                                         long long result_stride, int n, const float* __restrict__ coef,
                                         const void* __restrict__ weight, int w_dtype, float eps,
                                         TO* __restrict__ out, const int* __restrict__ rows, int H,
                                         int write_back) {
    extern __shared__ float row_s[];
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int b = blockIdx.x;
    const int row = rows ? rows[b] : b;
    const size_t base = static_cast<size_t>(row) * H;
    float inv = 1.0f;
    if (delta != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            float d = to_float(delta[base + i]);
            for (int k = 1; k < splits; ++k) d += to_float(delta[static_cast<size_t>(k) * split_stride + base + i]);
            row_s[i] = d;
            ss = fmaf(d, d, ss);
        }
        if (weight_b != nullptr) {
            ss = block_sum(ss, scratch);
            inv = 1.0f / sqrtf(ss / static_cast<float>(H) + eps_b);
        }
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        float x = x_in[base + i];
        if (delta != nullptr) x += row_s[i] * inv * (weight_b != nullptr ? load_as_float(weight_b, wb_dtype, i) : 1.f);
        if (coef != nullptr) {
            const float r = x;
            x = coef[0] * start[base + i];
            for (int j = 1; j < n; ++j) x = fmaf(coef[j], results[static_cast<size_t>(j - 1) * result_stride + base + i], x);
            x = fmaf(coef[n], r, x);
            if (write_back) results[static_cast<size_t>(n - 1) * result_stride + base + i] = r;
        }
        if (write_back) x_out[base + i] = x;
        row_s[i] = x;
        ss = fmaf(x, x, ss);
    }
    if (out == nullptr) return;
    float iw = 1.0f;
    if (weight != nullptr) {
        ss = block_sum(ss, scratch);
        iw = 1.0f / sqrtf(ss / static_cast<float>(H) + eps);
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x)
        out[static_cast<size_t>(b) * H + i] =
            from_float<TO>(row_s[i] * iw * (weight != nullptr ? load_as_float(weight, w_dtype, i) : 1.f));
}

// ------------------- norm over whole projections + rotation + turned values + cache write
// A row of `qkv` holds nq query heads and nkv key heads of `hd` elements and nkv value heads of
// `vd` elements.  All query rows at once are divided by their root mean square (eps inside the
// root) and multiplied by q_w [nq hd]; all key rows likewise with k_w [nkv hd] (null: no norm).
// Then the pairs among the first `rot` entries of every query and key head turn by
// position * inv_freq[i], and (v_freq != null) the pairs of every value head, over all of vd, by
// position * v_freq[m].  Pairs: entries i and i + rot / 2 (`neighbours` 0) or 2i and 2i + 1.
// Queries are written back in place; keys and values go to their cache slots.
// turn (may be null): float32 [T, vd / 2, 2], cosine and sine of the value pairs' angles, from
// which the heads' outputs are turned back.
// One CTA per token; sines and cosines are formed once per token.  `vec`: four neighbours at once
// (halves layout, all widths multiples of 8).
template <typename T>
__global__ void __launch_bounds__(256)
rownorm_rotary_store_kernel(T* __restrict__ qkv, long long stride, const int* __restrict__ positions,
                            const double* __restrict__ inv_freq, const double* __restrict__ v_freq,
                            int nq, int nkv, int hd, int vd, int rot, int neighbours,
                            const void* __restrict__ q_w, const void* __restrict__ k_w, int w_dtype,
                            float eps, const int* __restrict__ slot_map, T* __restrict__ kcache,
                            T* __restrict__ vcache, int page_size, float* __restrict__ turn, int vec) {
    extern __shared__ float2 cs_s[];                   // [rot / 2] of q and k, then [vd / 2] of v
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, nthr = blockDim.x;
    T* row = qkv + static_cast<size_t>(t) * stride;
    const int slot = slot_map != nullptr ? slot_map[t] : -1;
    const size_t page = slot >= 0 ? slot / page_size : 0, off = slot >= 0 ? slot % page_size : 0;
    const int half = rot >> 1, vhalf = v_freq != nullptr ? vd >> 1 : 0;
    const double pos = static_cast<double>(positions[t]);
    for (int i = tid; i < half + vhalf; i += nthr) {
        const float2 cs = turn_by(pos, i < half ? inv_freq[i] : v_freq[i - half]);
        cs_s[i] = cs;
        if (i >= half && turn != nullptr)
            reinterpret_cast<float2*>(turn)[static_cast<size_t>(t) * vhalf + i - half] = cs;
    }
    const int nqe = nq * hd, nke = nkv * hd;
    float inv_q = 1.f, inv_k = 1.f;
    if (q_w != nullptr) {
        float sq = 0.f, sk = 0.f;
        if (vec) {
            for (int e = tid * 4; e < nqe + nke; e += nthr * 4) {
                const F4 f = load4(row + e);
                float s = 0.f;
#pragma unroll
                for (int c = 0; c < 4; ++c) s = fmaf(f.v[c], f.v[c], s);
                if (e < nqe) sq += s; else sk += s;
            }
        } else {
            for (int e = tid; e < nqe + nke; e += nthr) {
                const float f = to_float(row[e]);
                if (e < nqe) sq = fmaf(f, f, sq); else sk = fmaf(f, f, sk);
            }
        }
        sq = block_sum(sq, scratch);
        __syncthreads();
        sk = block_sum(sk, scratch);
        inv_q = 1.0f / sqrtf(sq / static_cast<float>(nqe) + eps);
        inv_k = 1.0f / sqrtf(sk / static_cast<float>(nke) + eps);
    }
    __syncthreads();
    auto key_slot = [&](int g) { return kcache + ((page * nkv + g) * page_size + off) * hd; };
    auto value_slot = [&](int g) { return vcache + ((page * nkv + g) * page_size + off) * vd; };
    if (vec) {
        // queries and keys: an item is a run of four pairs below `rot`, or four entries behind it
        const int pair_items = half >> 2, items = pair_items + ((hd - rot) >> 2);
        for (int it = tid; it < (nq + nkv) * items; it += nthr) {
            const int head = it / items, j = it - head * items;
            const bool is_q = head < nq;
            if (!is_q && slot < 0) continue;
            const T* src = row + static_cast<size_t>(head) * hd;
            T* dst = is_q ? row + static_cast<size_t>(head) * hd : key_slot(head - nq);
            const void* w = is_q ? q_w : k_w;
            const size_t w0 = static_cast<size_t>(is_q ? head : head - nq) * hd;
            const float r = is_q ? inv_q : inv_k;
            auto fetch = [&](int e) {
                F4 f = load4(src + e);
                if (w != nullptr) {
                    const F4 ww = load4_any(w, w_dtype, w0 + e);
#pragma unroll
                    for (int c = 0; c < 4; ++c) f.v[c] = f.v[c] * r * ww.v[c];
                }
                return f;
            };
            if (j < pair_items) {
                const int e = 4 * j;
                F4 a = fetch(e), b = fetch(e + half);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float2 cs = cs_s[e + c];
                    const float u = a.v[c], v = b.v[c];
                    a.v[c] = fmaf(u, cs.x, -(v * cs.y));
                    b.v[c] = fmaf(v, cs.x, u * cs.y);
                }
                store4(dst + e, a);
                store4(dst + e + half, b);
            } else {
                const int e = rot + 4 * (j - pair_items);
                store4(dst + e, fetch(e));
            }
        }
        if (slot >= 0) {
            const T* vrow = row + nqe + nke;
            const int per = (vhalf > 0 ? vhalf : vd) >> 2;
            for (int it = tid; it < nkv * per; it += nthr) {
                const int g = it / per, e = 4 * (it - g * per);
                T* dst = value_slot(g);
                F4 a = load4(vrow + static_cast<size_t>(g) * vd + e);
                if (vhalf > 0) {
                    F4 b = load4(vrow + static_cast<size_t>(g) * vd + vhalf + e);
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        const float2 cs = cs_s[half + e + c];
                        const float u = a.v[c], v = b.v[c];
                        a.v[c] = fmaf(u, cs.x, -(v * cs.y));
                        b.v[c] = fmaf(v, cs.x, u * cs.y);
                    }
                    store4(dst + vhalf + e, b);
                }
                store4(dst + e, a);
            }
        }
        return;
    }
    // any width: an item is a pair below `rot`, or one entry behind it
    const int items = half + (hd - rot);
    for (int it = tid; it < (nq + nkv) * items; it += nthr) {
        const int head = it / items, j = it - head * items;
        const bool is_q = head < nq;
        if (!is_q && slot < 0) continue;
        const T* src = row + static_cast<size_t>(head) * hd;
        T* dst = is_q ? row + static_cast<size_t>(head) * hd : key_slot(head - nq);
        const void* w = is_q ? q_w : k_w;
        const size_t w0 = static_cast<size_t>(is_q ? head : head - nq) * hd;
        const float r = is_q ? inv_q : inv_k;
        auto fetch = [&](int e) {
            const float f = to_float(src[e]);
            return w != nullptr ? f * r * load_as_float(w, w_dtype, w0 + e) : f;
        };
        if (j < half) {
            const int e0 = neighbours ? 2 * j : j, e1 = neighbours ? 2 * j + 1 : j + half;
            const float2 cs = cs_s[j];
            const float u = fetch(e0), v = fetch(e1);
            dst[e0] = from_float<T>(fmaf(u, cs.x, -(v * cs.y)));
            dst[e1] = from_float<T>(fmaf(v, cs.x, u * cs.y));
        } else {
            const int e = rot + (j - half);
            dst[e] = from_float<T>(fetch(e));
        }
    }
    if (slot >= 0) {
        const T* vrow = row + nqe + nke;
        const int per = vhalf > 0 ? vhalf : vd;
        for (int it = tid; it < nkv * per; it += nthr) {
            const int g = it / per, j = it - g * per;
            const T* src = vrow + static_cast<size_t>(g) * vd;
            T* dst = value_slot(g);
            if (vhalf > 0) {
                const int e0 = neighbours ? 2 * j : j, e1 = neighbours ? 2 * j + 1 : j + vhalf;
                const float2 cs = cs_s[half + j];
                const float u = to_float(src[e0]), v = to_float(src[e1]);
                dst[e0] = from_float<T>(fmaf(u, cs.x, -(v * cs.y)));
                dst[e1] = from_float<T>(fmaf(v, cs.x, u * cs.y));
            } else {
                dst[j] = src[j];
            }
        }
    }
}

// The pairs of every head of x [T, heads * vd] turned back, in place: turn [T, vd / 2, 2] holds
// cosine and sine of the angles by which the values' pairs were turned at this token's position.
template <typename T>
__global__ void turn_back_kernel(T* __restrict__ x, const float2* __restrict__ turn, int heads, int vd,
                                 int neighbours, long long rows, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const int half = vd >> 1;
    const int per = vec ? half >> 2 : half;
    const long long n = rows * heads * per;
    for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
         i += static_cast<long long>(gridDim.x) * blockDim.x) {
        const long long th = i / per;
        const int j = static_cast<int>(i - th * per);
        const long long t = th / heads;
        T* head = x + th * vd;
        const float2* tr = turn + t * half;
        if (vec) {
            const int e = 4 * j;
            F4 a = load4(head + e), b = load4(head + half + e);
            const float4 c01 = *reinterpret_cast<const float4*>(tr + e);
            const float4 c23 = *reinterpret_cast<const float4*>(tr + e + 2);
            const float cs[4] = {c01.x, c01.z, c23.x, c23.z}, sn[4] = {c01.y, c01.w, c23.y, c23.w};
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float u = a.v[c], v = b.v[c];
                a.v[c] = fmaf(u, cs[c], v * sn[c]);
                b.v[c] = fmaf(v, cs[c], -(u * sn[c]));
            }
            store4(head + e, a);
            store4(head + half + e, b);
        } else {
            const int e0 = neighbours ? 2 * j : j, e1 = neighbours ? 2 * j + 1 : j + half;
            const float u = to_float(head[e0]), v = to_float(head[e1]);
            const float2 cs = tr[j];
            head[e0] = from_float<T>(fmaf(u, cs.x, v * cs.y));
            head[e1] = from_float<T>(fmaf(v, cs.x, -(u * cs.y)));
        }
    }
}

// ------------------------------------- latent cache row with a rotated tail, queries' tails
// A row of `x` holds, from column q_at on, H query heads of qd + rot elements each (the last `rot`
// of a head turn), and from column c_at on a latent of `rank` elements with a key part of `rot`
// elements behind it.  Written: cache row of the token [rank + rot] = (latent / rms * weight | turned
// key part), and into qa [H, T, rank + rot] the turned tail of every query behind column `rank`
// (the columns before it are another kernel's).  Pairs: i and i + rot / 2, or neighbours.
// One CTA per token; sines and cosines are formed once per token.  `vec2`: two neighbours at once
// (neighbouring pairs, every offset even).
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_rotary_store_kernel(const T* __restrict__ x, long long stride, int q_at, int H, int qd, int rot,
                           int c_at, int rank, int neighbours, const int* __restrict__ positions,
                           const double* __restrict__ inv_freq, const void* __restrict__ weight,
                           int w_dtype, float eps, float magnitude, const int* __restrict__ slot_map,
                           T* __restrict__ cache, T* __restrict__ qa, int n_tokens, int vec2) {
    extern __shared__ float2 cs_s[];                       // [rot / 2]
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, nthr = blockDim.x;
    const T* row = x + static_cast<size_t>(t) * stride;
    const int half = rot >> 1, W = rank + rot;
    const double pos = static_cast<double>(positions[t]);
    for (int i = tid; i < half; i += nthr) {
        const float2 cs = turn_by(pos, inv_freq[i]);
        cs_s[i] = make_float2(cs.x * magnitude, cs.y * magnitude);
    }
    float ss = 0.f;
    if (vec2) {
        for (int e = 2 * tid; e < rank; e += 2 * nthr) {
            const float2 f = load2(row + c_at + e);
            ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss));
        }
    } else {
        for (int e = tid; e < rank; e += nthr) {
            const float f = to_float(row[c_at + e]);
            ss = fmaf(f, f, ss);
        }
    }
    ss = block_sum(ss, scratch);
    __syncthreads();
    const float inv = 1.0f / sqrtf(ss / static_cast<float>(rank) + eps);
    if (slot_map != nullptr) {
        T* dst = cache + static_cast<size_t>(slot_map[t]) * W;
        if (vec2) {
            for (int e = 2 * tid; e < rank; e += 2 * nthr) {
                const float2 f = load2(row + c_at + e);
                store2(dst + e, f.x * inv * load_as_float(weight, w_dtype, e),
                       f.y * inv * load_as_float(weight, w_dtype, e + 1));
            }
        } else {
            for (int e = tid; e < rank; e += nthr)
                dst[e] = from_float<T>(to_float(row[c_at + e]) * inv * load_as_float(weight, w_dtype, e));
        }
    }
    if (vec2 && !neighbours) {
        // two neighbouring pairs (j, j + half), (j + 1, j + 1 + half) at once
        for (int it = tid; it < (H + 1) * (half >> 1); it += nthr) {
            const int h = it / (half >> 1), j = 2 * (it - h * (half >> 1));
            const T* src = h < H ? row + q_at + static_cast<size_t>(h) * (qd + rot) + qd : row + c_at + rank;
            T* dst;
            if (h < H) dst = qa + (static_cast<size_t>(h) * n_tokens + t) * W + rank;
            else if (slot_map != nullptr) dst = cache + static_cast<size_t>(slot_map[t]) * W + rank;
            else continue;
            const float2 c0 = cs_s[j], c1 = cs_s[j + 1], u = load2(src + j), v = load2(src + j + half);
            store2(dst + j, fmaf(u.x, c0.x, -(v.x * c0.y)), fmaf(u.y, c1.x, -(v.y * c1.y)));
            store2(dst + j + half, fmaf(v.x, c0.x, u.x * c0.y), fmaf(v.y, c1.x, u.y * c1.y));
        }
        return;
    }
    for (int it = tid; it < (H + 1) * half; it += nthr) {
        const int h = it / half, j = it - h * half;
        const int e0 = neighbours ? 2 * j : j, e1 = neighbours ? 2 * j + 1 : j + half;
        const T* src = h < H ? row + q_at + static_cast<size_t>(h) * (qd + rot) + qd : row + c_at + rank;
        T* dst;
        if (h < H) dst = qa + (static_cast<size_t>(h) * n_tokens + t) * W + rank;
        else if (slot_map != nullptr) dst = cache + static_cast<size_t>(slot_map[t]) * W + rank;
        else continue;
        const float2 cs = cs_s[j];
        if (vec2) {
            const float2 f = load2(src + e0);
            store2(dst + e0, fmaf(f.x, cs.x, -(f.y * cs.y)), fmaf(f.y, cs.x, f.x * cs.y));
            continue;
        }
        const float u = to_float(src[e0]), v = to_float(src[e1]);
        dst[e0] = from_float<T>(fmaf(u, cs.x, -(v * cs.y)));
        dst[e1] = from_float<T>(fmaf(v, cs.x, u * cs.y));
    }
}

}  // namespace somi

using namespace somi;

static inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// delta: [rows, H] of delta_dtype, or float32 partial sums; start, results: float32 (results rows
// `result_stride` apart per layer); coef: float32 [n + 1] or null.  See stream_update_kernel.
SOMI_API int somi_stream_update(const float* x_in, float* x_out, const void* delta, int delta_dtype,
                                int splits, long long split_stride, const void* weight_b, int wb_dtype,
                                float eps_b, const float* start, float* results,
                                long long result_stride, int n, const float* coef, const void* weight,
                                int w_dtype, float eps, void* out, int out_dtype, const int* rows,
                                int n_out, int H, int write_back, cudaStream_t stream) {
    if (n_out <= 0) return 0;
    if (H <= 0 || (splits > 1 && delta_dtype != SOMI_F32) ||
        (coef != nullptr && (n < 1 || start == nullptr || results == nullptr)))
        return SOMI_ERR_UNSUPPORTED;
    const bool vec4 = (H & 3) == 0 && H <= 8192 && aligned16(x_in) && aligned16(x_out) && aligned16(delta) &&
                      aligned16(weight_b) && aligned16(start) && aligned16(results) && aligned16(weight) &&
                      aligned16(out) && (split_stride & 3) == 0 && (result_stride & 3) == 0;
    // few rows (a decode step): a thread per four columns, every load of the row in flight at once
    const int vecs = (H + 3) / 4;
    int v = n_out <= 512 ? 1 : 4;
    if (vecs < 64 * v) v = 1;
    if (v == 1 && vecs > 1024) v = 2;                     // (a CTA of V = 4 has at most 512 threads)
    const int threads = max(32, (((vecs + v - 1) / v + 31) / 32) * 32);
#define SOMI_SU_ARGS(TD, TO)                                                                       \
    x_in, x_out, static_cast<const TD*>(delta), splits, split_stride, weight_b, wb_dtype, eps_b,   \
        start, results, result_stride, n, coef, weight, w_dtype, eps, static_cast<TO*>(out), rows, \
        H, write_back
#define SOMI_LAUNCH_SU(TD, TO)                                                                     \
    do {                                                                                           \
        if (!vec4) {                                                                               \
            const size_t smem = sizeof(float) * H;                                                 \
            if (smem > 200 * 1024) return SOMI_ERR_UNSUPPORTED;                                    \
            if (smem > 48 * 1024)                                                                  \
                cudaFuncSetAttribute(stream_update_any_kernel<TD, TO>,                             \
                                     cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
            launch_pdl(stream_update_any_kernel<TD, TO>, dim3(n_out),                              \
                       dim3(min(256, max(32, ((H / 2 + 31) / 32) * 32))), smem, stream,            \
                       SOMI_SU_ARGS(TD, TO));                                                      \
        } else if (v == 1) {                                                                       \
            launch_pdl(stream_update_kernel<TD, TO, 1>, dim3(n_out), dim3(threads), 0, stream,     \
                       SOMI_SU_ARGS(TD, TO));                                                      \
        } else if (v == 2) {                                                                       \
            launch_pdl(stream_update_kernel<TD, TO, 2>, dim3(n_out), dim3(threads), 0, stream,     \
                       SOMI_SU_ARGS(TD, TO));                                                      \
        } else {                                                                                   \
            launch_pdl(stream_update_kernel<TD, TO, 4>, dim3(n_out), dim3(threads), 0, stream,     \
                       SOMI_SU_ARGS(TD, TO));                                                      \
        }                                                                                          \
    } while (0)
    if (delta_dtype == SOMI_F32 && out_dtype == SOMI_F32) SOMI_LAUNCH_SU(float, float);
    else if (delta_dtype == SOMI_F32) SOMI_LAUNCH_SU(float, __nv_bfloat16);
    else if (out_dtype == SOMI_F32) SOMI_LAUNCH_SU(__nv_bfloat16, float);
    else SOMI_LAUNCH_SU(__nv_bfloat16, __nv_bfloat16);
#undef SOMI_LAUNCH_SU
#undef SOMI_SU_ARGS
    return launch_status();
}

SOMI_API int somi_rownorm_rotary_store(void* qkv, int dtype, long long stride, const int* positions,
                                       const double* inv_freq, const double* v_freq, int T, int nq,
                                       int nkv, int hd, int vd, int rot, int neighbours,
                                       const void* q_w, const void* k_w, int w_dtype, float eps,
                                       const int* slot_map, void* kcache, void* vcache, int page_size,
                                       float* turn, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (nq <= 0 || nkv <= 0 || hd <= 0 || vd <= 0 || rot < 0 || rot > hd || (rot & 1) ||
        (v_freq != nullptr && (vd & 1)) || (q_w == nullptr) != (k_w == nullptr) || page_size <= 0)
        return SOMI_ERR_UNSUPPORTED;
    const size_t smem = sizeof(float2) * (rot / 2 + (v_freq != nullptr ? vd / 2 : 0) + 1);
    if (smem > 48 * 1024) return SOMI_ERR_UNSUPPORTED;
    const int vec = !neighbours && ((hd | vd | rot) & 7) == 0 && (stride & 3) == 0 && aligned16(qkv) &&
                    aligned16(kcache) && aligned16(vcache) && aligned16(q_w) && aligned16(k_w);
#define SOMI_LAUNCH_RRS(TT)                                                                        \
    launch_pdl(rownorm_rotary_store_kernel<TT>, dim3(T), dim3(256), smem, stream,                  \
               static_cast<TT*>(qkv), stride, positions, inv_freq, v_freq, nq, nkv, hd, vd, rot,   \
               neighbours, q_w, k_w, w_dtype, eps, slot_map, static_cast<TT*>(kcache),             \
               static_cast<TT*>(vcache), page_size, turn, vec)
    if (dtype == SOMI_F32) SOMI_LAUNCH_RRS(float);
    else SOMI_LAUNCH_RRS(__nv_bfloat16);
#undef SOMI_LAUNCH_RRS
    return launch_status();
}

SOMI_API int somi_turn_back(void* x, int dtype, const float* turn, long long rows, int heads, int vd,
                            int neighbours, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (heads <= 0 || vd <= 0 || (vd & 1)) return SOMI_ERR_UNSUPPORTED;
    const int vec = !neighbours && (vd & 7) == 0 && aligned16(x) && aligned16(turn);
    const long long n = rows * heads * (vd / 2) / (vec ? 4 : 1);
    const int blocks = static_cast<int>(min((n + 255) / 256, 148LL * 16));
    if (dtype == SOMI_F32)
        launch_pdl(turn_back_kernel<float>, dim3(blocks), dim3(256), 0, stream, static_cast<float*>(x),
                   reinterpret_cast<const float2*>(turn), heads, vd, neighbours, rows, vec);
    else
        launch_pdl(turn_back_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream,
                   static_cast<__nv_bfloat16*>(x), reinterpret_cast<const float2*>(turn), heads, vd,
                   neighbours, rows, vec);
    return launch_status();
}

SOMI_API int somi_latent_rotary_store(const void* x, int dtype, long long stride, int q_at, int H,
                                      int qd, int rot, int c_at, int rank, int neighbours,
                                      const int* positions, const double* inv_freq, const void* weight,
                                      int w_dtype, float eps, float magnitude, const int* slot_map,
                                      void* cache, void* qa, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || qd < 0 || rot < 0 || (rot & 1) || rot > 4096 || rank <= 0) return SOMI_ERR_UNSUPPORTED;
    const size_t smem = sizeof(float2) * (rot / 2 + 1);
    const int vec2 = (neighbours || (rot & 3) == 0) && ((q_at | qd | c_at | rank) & 1) == 0 && (stride & 1) == 0 && aligned16(x) &&
                     aligned16(cache) && aligned16(qa);
#define SOMI_LAUNCH_LRS(TT)                                                                        \
    launch_pdl(latent_rotary_store_kernel<TT>, dim3(T), dim3(256), smem, stream,                   \
               static_cast<const TT*>(x), stride, q_at, H, qd, rot, c_at, rank, neighbours,        \
               positions, inv_freq, weight, w_dtype, eps, magnitude, slot_map,                     \
               static_cast<TT*>(cache), static_cast<TT*>(qa), T, vec2)
    if (dtype == SOMI_F32) SOMI_LAUNCH_LRS(float);
    else SOMI_LAUNCH_LRS(__nv_bfloat16);
#undef SOMI_LAUNCH_LRS
    return launch_status();
}
