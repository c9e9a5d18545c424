// Prompt-portion attention over the paged cache on the 5th-generation tensor cores, two query
// tiles per CTA in ping-pong.
//
// One CTA = up to 256 consecutive query rows of one request x one query head, as two tiles A and
// B of 128 rows; key tiles of 128 positions aligned to multiples of 128, fetched once for both
// query tiles.  Tensor memory holds S_A, S_B (128 columns each) and O_A, O_B (head_dim columns
// each).  A softmax warp group of 128 threads serves each query tile, one thread per row (one
// lane of tensor memory): it reads its row of S, writes the probabilities back over the same
// columns as packed bfloat16 pairs, and the second product takes them from there as its A
// operand (`tcgen05.mma` with A in tensor memory), so P never passes through shared memory.
// One thread issues the products in the order
//     S_A(0) S_B(0) | PV_A(t) S_A(t+1) PV_B(t) S_B(t+1) | ...
// so that while warp group A works on tile t's scores the tensor core runs B's products of
// tile t-1 and B's scores of tile t, and the other way round.  The pipe executes in issue order,
// which is what makes the aliasing of P over S safe: S_X(t+1) is issued after PV_X(t).
// (Two issuing threads, one per query tile, fall into step with each other: both softmax warp
// groups then want the exponential unit at the same time and a round takes a third longer.)
// What the issuing thread does between products costs a hundred cycles and more apiece (a
// barrier test, a fence, a commit), during which the pipe runs dry, so it does as little of
// it as possible: it tests only the two p_full barriers in a round (the softmax warp group that
// announces P has seen the value tile and the next key tile arrive, before it waits for the
// scores, where it has time), it commits o_done only after a query tile's last key tile (the
// commit behind s_full covers the output products issued before it), and it hands both stages
// back at the end of a round.
// An accumulator is rescaled in tensor memory only when its row maximum grows by more than 2^8
// (probabilities up to 256 are harmless in float32 sums and bfloat16 operands).  Because tile B's
// rows come later in the sequence, tile A runs out of key tiles first and writes its output
// while B goes on.  Softmax is float32, base 2; scaling, subtraction and the row sum work on
// pairs of keys (`fma.rn.f32x2`, `add.rn.f32x2`), the maximum on three values at a time.  Every
// wait on an mbarrier is bounded and failure is recorded in an error word.
//
// Warp roles: warps 0-3 softmax of tile A, 4-7 softmax of tile B (both clear the value stages
// first), warp 8 key (and Q) producer, warp 9 MMA issuer and owner of tensor memory, warp 10
// value producer, warp 11 idle.  Two key stages and three value stages at head size 128 (a value
// tile is read a round later than the key tile that came with it), four and four at 64.
//
// With `TWO_MAPS` (attention in two maps, two_maps.cuh) the CTA's two query tiles are the two queries
// of the same 128 rows: a key row of HD elements holds the keys of both maps, map x being its half
// x, so the keys of both maps arrive in one tile and the values are fetched once for both.  Both
// tiles then have the same rows, positions and key tiles; at the end each softmax warp group takes
// half of the head's columns of both outputs, and the difference of the maps, its norm and the
// gate are made from the float32 accumulators.  There first tokens may stay visible beside a
// window (`keep`): the key tiles that hold them come in front of the window's.
//
// The reference's prefill kernel (somi_inference/core/flash_attention_triton.py:31-194) is a
// FlashAttention-2 loop on `tl.dot`; formulas in somi_inference/models/qwen2.py:158-186.
#include "tcgen05.cuh"
#include "two_maps.cuh"

namespace somi {

constexpr int kPpBM = 128;               // rows of one query tile
constexpr int kPpRows = 2 * kPpBM;       // rows of a CTA
constexpr int kPpBN = 128;               // keys per tile
constexpr int kPpThreads = 384;
constexpr int kPpMaxStages = 4;
// A value tile is read one key tile later than the key tile that arrived with it (its products
// wait for the softmax in between), so at the same distance of prefetch it needs a stage more.
__host__ __device__ constexpr int pp_k_stages(int hd) { return hd == 128 ? 2 : 4; }
__host__ __device__ constexpr int pp_v_stages(int hd) { return hd == 128 ? 3 : 4; }
constexpr int kPpQHalf = kPpBM * 128;    // bytes of one [128 rows][64 elements] swizzled block
constexpr int kPpKvHalf = kPpBN * 128;

__device__ int g_prefill_pp_error = 0;

template <int HD, bool TWO_MAPS>
__global__ void __launch_bounds__(kPpThreads, 1)
paged_prefill_pp_kernel(const __grid_constant__ CUtensorMap q_map,
                        const __grid_constant__ CUtensorMap kv_map, long long k_row0,
                        long long v_row0, const int* __restrict__ block_table, int bt_stride,
                        const int* __restrict__ cu_q, const int* __restrict__ ctx_len,
                        const int* __restrict__ tiles, int nq, int nkv, int page_size,
                        float scale_log2e, int window, const float* __restrict__ sinks,
                        const float2* __restrict__ turn, __nv_bfloat16* __restrict__ out,
                        int n_q_tiles, int keep, TwoMaps two) {
    constexpr int HALVES = HD / 64;
    constexpr int QTILE = HALVES * kPpQHalf;
    constexpr int TILE = HALVES * kPpKvHalf;
    constexpr int KST = pp_k_stages(HD), VST = pp_v_stages(HD);
    constexpr uint32_t TmemCols = 512;                   // S_A | S_B | O_A | O_B, 128 columns each
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>(
        (reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
    unsigned char* Qs = base;                            // two query tiles (two maps: one)
    unsigned char* Ks = Qs + (TWO_MAPS ? 1 : 2) * QTILE;                  // KST tiles
    unsigned char* Vs = Ks + KST * TILE;                 // VST tiles
    __shared__ __align__(8) unsigned long long q_full[2], k_full[kPpMaxStages], k_empty[kPpMaxStages],
        v_full[kPpMaxStages], v_empty[kPpMaxStages], s_full[2], p_full[2], o_done[2], v_zeroed;
    __shared__ uint32_t tmem_base_s;
    __shared__ int failed_s;
    __shared__ float map_scale_s[TWO_MAPS ? 2 : 1][kPpBM], map_square_s[TWO_MAPS ? 2 : 1][kPpBM];

    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int x = 0; x < 2; ++x) {
            mbar_init(smem_u32(&q_full[x]), 1);
            mbar_init(smem_u32(&s_full[x]), 1);
            mbar_init(smem_u32(&p_full[x]), 4);          // one arrival per warp of the group
            mbar_init(smem_u32(&o_done[x]), 1);
        }
        for (int s = 0; s < kPpMaxStages; ++s) {
            mbar_init(smem_u32(&k_full[s]), 1);
            mbar_init(smem_u32(&k_empty[s]), 1);
            mbar_init(smem_u32(&v_full[s]), 1);
            mbar_init(smem_u32(&v_empty[s]), 1);
        }
        mbar_init(smem_u32(&v_zeroed), 8);               // one arrival per softmax warp
        mbar_fence_init();
        failed_s = 0;
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(
                         smem_u32(&tmem_base_s)),
                     "r"(TmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    t5::fence_before();
    __syncthreads();
    t5::fence_after();
    pdl_wait();
    const uint32_t tmem_s = tmem_base_s;                 // S_A at column 0, S_B at 128
    const uint32_t tmem_o = tmem_base_s + 2 * kPpBN;     // O_A at 256, O_B at 384

    // Later tiles of a prompt see more keys.  Blocks are handed out longest first (heads
    // first, last tile first), so that the short ones fill the end.
    const int rank = blockIdx.x;
    const int tile = n_q_tiles - 1 - rank / nq;
    const int req = tiles[3 * tile], row0 = tiles[3 * tile + 1];
    const int rows = tiles[3 * tile + 2];
    const int head = rank % nq, kvh = head / (nq / nkv);
    const bool has_b = TWO_MAPS || rows > kPpBM;
    const int q_pos0 = ctx_len[req] + (row0 - cu_q[req]);
    const int kv_first = first_visible_key(q_pos0, window);
    const int kb0 = (kv_first / kPpBN) * kPpBN;
    const int end_a = q_pos0 + min(rows, kPpBM), end_all = q_pos0 + rows;
    // tiles of kept keys in front of the window's
    const int n_pre = TWO_MAPS && keep > 0 ? min((keep + kPpBN - 1) / kPpBN, kb0 / kPpBN) : 0;
    const int n_a = n_pre + (end_a - kb0 + kPpBN - 1) / kPpBN;    // key tiles that tile A reads
    const int n_t = n_pre + (end_all - kb0 + kPpBN - 1) / kPpBN;  // key tiles of the CTA
    auto key_tile = [&](int t) { return t < n_pre ? t * kPpBN : kb0 + (t - n_pre) * kPpBN; };
    const int* bt = block_table + static_cast<size_t>(req) * bt_stride;

    // The softmax threads hold a row of 128 scores in registers; the producer and issuing warps
    // need few.  Warps 8-11 give registers back and the softmax warp groups take them.  The
    // pool is what the CTA was given at launch, 12 warps x 168 registers a thread: 8 x 216 +
    // 4 x 72 uses exactly that.  `setmaxnreg.inc` waits, without a limit, until the pool has what
    // it asks for, so the two figures must never add up to more.
    static_assert(8 * 216 + 4 * 72 <= 12 * 168, "setmaxnreg would wait for registers that never come");
    if (warp >= 8) {
      asm volatile("setmaxnreg.dec.sync.aligned.u32 72;\n");
      if (warp == 8 || warp == 10) {
        // ---- producer warps, one for the keys (and Q) and one for the values.  Lane 0 keeps the
        // barriers, one lane per page looks its page up and issues that page's copies.
        if (warp == 8 && lane == 0) {
            for (int x = 0; x < (has_b && !TWO_MAPS ? 2 : 1); ++x) {
                mbar_expect_tx(smem_u32(&q_full[x]), kPpBM * HD * 2);
#pragma unroll
                for (int h = 0; h < HALVES; ++h)
                    tma_load_2d(smem_u32(Qs + x * QTILE + h * kPpQHalf), &q_map, head * HD + h * 64,
                                row0 + x * kPpBM, smem_u32(&q_full[x]));
            }
        }
        const int pages_per_tile = kPpBN / page_size;
        const int which = warp == 8 ? 0 : 1;
        const int n_st = which ? VST : KST;
        // no value copy before the softmax warps have cleared the value stages
        if (which && !mbar_wait(smem_u32(&v_zeroed), 0)) failed_s = 1;
        __syncwarp();
        for (int t = 0; t < n_t; ++t) {
            const int st = t % n_st;
            const int kb = key_tile(t);
            const int p_lo = max(kb, kv_first) / page_size;
            const int p_hi = (min(kb + kPpBN, end_all) - 1) / page_size;
            int my_page = -1, n_pages = p_hi - p_lo + 1;
            const int ap = kb / page_size + lane;
            bool mine = lane < pages_per_tile && ap >= p_lo && ap <= p_hi;
            if constexpr (TWO_MAPS) {
                mine = mine || (lane < pages_per_tile && ap <= p_hi && ap * page_size < keep);
                n_pages = __popc(__ballot_sync(0xffffffffu, mine));
            }
            if (mine) my_page = bt[ap];
            const uint32_t bar = smem_u32(which ? &v_full[st] : &k_full[st]);
            int ok = 1;
            if (lane == 0) {
                ok = mbar_wait(smem_u32(which ? &v_empty[st] : &k_empty[st]), ((t / n_st) & 1) ^ 1) ? 1 : 0;
                if (ok) mbar_expect_tx(bar, static_cast<uint32_t>(n_pages) * page_size * HD * 2);
                else failed_s = 1;
            }
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (!ok) break;
            if (my_page >= 0) {
                const long long prow = (static_cast<long long>(my_page) * nkv + kvh) * page_size;
                unsigned char* dst = (which ? Vs : Ks) + st * TILE + lane * page_size * 128;
#pragma unroll
                for (int h = 0; h < HALVES; ++h)
                    tma_load_2d(smem_u32(dst + h * kPpKvHalf), &kv_map, h * 64,
                                static_cast<int>((which ? v_row0 : k_row0) + prow), bar);
            }
        }
      } else if (warp == 9) {
        if (lane == 0) {
            // float32 accumulators, bf16 operands.  Scores: A and B K-major, N = 128 keys.
            // P.V: A (P) from tensor memory, B (V) MN-major, N = head_dim.
            const uint32_t idesc_qk = (1u << 4) | (1u << 7) | (1u << 10) |
                                      (static_cast<uint32_t>(kPpBN >> 3) << 17) |
                                      (static_cast<uint32_t>(kPpBM >> 4) << 24);
            const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) |
                                      (static_cast<uint32_t>(HD >> 3) << 17) |
                                      (static_cast<uint32_t>(kPpBM >> 4) << 24);
            const uint64_t q_desc = t5::desc_kmajor(smem_u32(Qs));
            const uint64_t k_desc = t5::desc_kmajor(smem_u32(Ks));
            const uint64_t v_desc = t5::desc_mnmajor(smem_u32(Vs), kPpKvHalf);
            bool ok = true;
            auto wait = [&](unsigned long long* bar, int parity) {
                if (ok && !mbar_wait(smem_u32(bar), parity)) ok = false;
                t5::fence_after();
            };
            // the same with the test that returns at once: this thread has nothing else to do,
            // and wakes up sooner than from the test that may suspend it
            auto spin = [&](unsigned long long* bar, int parity) {
                if (ok) {
                    int i = 0;
                    while (!mbar_test_now(smem_u32(bar), parity))
                        if (++i > 8000000) { ok = false; break; }
                }
                t5::fence_after();
            };
            auto scores = [&](int x, int t) {            // S_x(t) = Q_x K(t)^T
                const uint64_t kd = k_desc + (((t % KST) * TILE) >> 4);
                const uint64_t qd = q_desc + (TWO_MAPS ? 0 : (x * QTILE) >> 4);
                // (two maps: query x and key x are half x of the rows)
                const int first16 = TWO_MAPS ? x * (HD / 32) : 0;
#pragma unroll
                for (int i16 = 0; i16 < (TWO_MAPS ? HD / 32 : HD / 16); ++i16) {
                    const int k16 = first16 + i16;
                    t5::mma_ss(tmem_s + x * kPpBN,
                               qd + (((k16 >> 2) * kPpQHalf + (k16 & 3) * 32) >> 4),
                               kd + (((k16 >> 2) * kPpKvHalf + (k16 & 3) * 32) >> 4), idesc_qk,
                               i16 > 0 ? 1u : 0u);
                }
                t5::commit(smem_u32(&s_full[x]));
            };
            auto outputs = [&](int x, int t) {           // O_x += P_x(t) V(t)
                const uint64_t vd = v_desc + (((t % VST) * TILE) >> 4);
#pragma unroll
                for (int k16 = 0; k16 < kPpBN / 16; ++k16)
                    t5::mma_ts(tmem_o + x * kPpBN, tmem_s + x * kPpBN + 8 * k16,
                               vd + ((k16 * 16 * 128) >> 4), idesc_pv, (t > 0 || k16 > 0) ? 1u : 0u);
                // A commit covers every product issued so far: s_full of tile t + 1 also says
                // that O holds tile t, so o_done is only needed after a query tile's last.
                if (t + 1 == (x == 0 ? n_a : n_t)) t5::commit(smem_u32(&o_done[x]));
            };
            wait(&q_full[0], 0);
            wait(&k_full[0], 0);
            if (ok) scores(0, 0);
            if (has_b) {
                if (!TWO_MAPS) wait(&q_full[1], 0);
                if (ok) scores(1, 0);
            }
            if (ok) t5::commit(smem_u32(&k_empty[0]));
            for (int t = 0; t < n_t && ok; ++t) {
                // The key and value tiles these products read have been seen by the softmax
                // warp group that announces P (it waits for them before it arrives), so this
                // thread tests nothing but the two p_full barriers in an iteration: every test
                // and every commit is time in which this thread issues no product.
                if (t < n_a) {
                    spin(&p_full[0], t & 1);
                    if (!ok) break;
                    outputs(0, t);
                    if (t + 1 < n_a) scores(0, t + 1);
                }
                if (has_b) {
                    spin(&p_full[1], t & 1);
                    if (!ok) break;
                    outputs(1, t);
                    if (t + 1 < n_t) scores(1, t + 1);
                }
                // both stages are handed back at the end, so that no commit sits between the
                // products of a query tile
                t5::commit(smem_u32(&v_empty[t % VST]));
                if (t + 1 < n_t) t5::commit(smem_u32(&k_empty[(t + 1) % KST]));
            }
            if (!ok) failed_s = 1;       // the softmax warps run out of their bounded waits
        }
      }
    } else {
        asm volatile("setmaxnreg.inc.sync.aligned.u32 216;\n");
        // Value rows that no copy fills (pages outside the request's range) must be finite
        // numbers, whatever the shared memory held before.  These warps have nothing to do
        // until the first scores are there, so they clear the value stages while the keys and
        // queries are on their way; the value producer waits for them.
        for (int c = tid; c < VST * TILE / 16; c += 8 * 32)
            reinterpret_cast<uint4*>(Vs)[c] = make_uint4(0, 0, 0, 0);
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&v_zeroed));
        // ---- softmax: warp group x serves query tile x, one thread per row
        const int x = warp >> 2;
        if (x == 0 || has_b) {
            const int q = warp & 3;                                  // lane quarter this warp may access
            const int row = q * 32 + lane;                           // row within the query tile
            const uint32_t lane_addr = static_cast<uint32_t>(q * 32) << 16;
            const int tile_pos0 = q_pos0 + (TWO_MAPS ? 0 : x * kPpBM);   // position of the tile's first row
            const int pos = tile_pos0 + row;
            const int lo = first_visible_key(pos, window);
            // the highest first visible key among the tile's rows
            const int lo_max = first_visible_key(tile_pos0 + kPpBM - 1, window);
            const unsigned span = static_cast<unsigned>(pos - lo);
            const int keep_end = TWO_MAPS ? min(keep, pos + 1) : 0;  // keys below it are visible, too
            const int n_x = x == 0 ? n_a : n_t;
            const uint32_t s_addr = tmem_s + x * kPpBN + lane_addr;
            const uint32_t o_addr = tmem_o + x * kPpBN + lane_addr;
            float m = -INFINITY, l = 0.f;        // m: the reference maximum in use (log2 units)
            bool ok = true;
            for (int t = 0; t < n_x; ++t) {
                // On behalf of the issuing thread: the values of this tile and the keys of the
                // next have arrived before this warp group announces P(t).  They are tested
                // here, where the warp would wait for the scores anyway (a test costs a few
                // hundred cycles even on a completed barrier), by the whole warp, so that it
                // stays converged for the aligned instructions.
                if (q == 0) {
                    ok = mbar_wait(smem_u32(&v_full[t % VST]), (t / VST) & 1, ok ? 400000 : 1) && ok;
                    if (t + 1 < n_x)
                        ok = mbar_wait(smem_u32(&k_full[(t + 1) % KST]), ((t + 1) / KST) & 1,
                                       ok ? 400000 : 1) && ok;
                }
                ok = mbar_wait(smem_u32(&s_full[x]), t & 1, ok ? 400000 : 1) && ok;
                t5::fence_after();
                const int kb = key_tile(t);
                // a tile in which no row of this query tile has a hidden key takes the short way
                const bool tile_inner = kb + kPpBN - 1 <= tile_pos0 &&
                                        (kb >= lo_max || (TWO_MAPS && kb + kPpBN <= keep));
                // ---- the row's 128 scores into registers: four loads in flight, one wait
                uint32_t sv[128];
#pragma unroll
                for (int c = 0; c < 4; ++c) t5::ld32_nowait(s_addr + c * 32, sv + c * 32);
                t5::wait_ld();
                float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
                if (tile_inner) {
#pragma unroll
                    for (int j = 0; j < 128; j += 2)
                        mx[(j >> 1) & 3] = fmax3(mx[(j >> 1) & 3], __uint_as_float(sv[j]), __uint_as_float(sv[j + 1]));
                } else {
#pragma unroll
                    for (int j = 0; j < 128; ++j) {
                        // key in [lo, pos] as one unsigned comparison
                        const unsigned d = static_cast<unsigned>(kb + j - lo);
                        const bool seen = d <= span || (TWO_MAPS && kb + j < keep_end);
                        const float v = seen ? __uint_as_float(sv[j]) : -INFINITY;
                        sv[j] = __float_as_uint(v);
                        mx[j & 3] = fmaxf(mx[j & 3], v);
                    }
                }
                // the scale is positive: the maximum is taken over the raw scores and scaled once
                const float tmax = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * scale_log2e;
                // keep the old reference maximum unless the new one is more than 2^8 above it
                float alpha = 1.f;
                bool rescale = false;
                if (m == -INFINITY) {
                    m = tmax;                                   // nothing accumulated yet for this row
                } else if (tmax > m + 8.0f) {
                    alpha = fast_exp2(m - tmax);
                    m = tmax;
                    rescale = true;
                }
                if (__any_sync(0xffffffffu, rescale)) {
                    // O holds the tiles so far: the commit behind s_full covered the products
                    // of tile t - 1 as well (issued before S(t) by the same thread)
#pragma unroll
                    for (int c = 0; c < HD / 32; ++c) {
                        uint32_t ov[32];
                        t5::ld32_nowait(o_addr + c * 32, ov);
                        t5::wait_ld();
#pragma unroll
                        for (int j = 0; j < 32; ++j) ov[j] = __float_as_uint(__uint_as_float(ov[j]) * alpha);
                        t5::st32(o_addr + c * 32, ov);
                    }
                    t5::wait_st();
                    l *= alpha;
                }
                const float neg_m = m == -INFINITY ? 0.f : -m;
                // ---- probabilities, written over the scores as bfloat16 pairs: chunk c's 32 keys
                // become 16 columns at 16 c (every score is in registers by now)
                // (scaling, subtraction and the row sum on pairs of keys: one instruction for two)
                const uint64_t scale2 = pair_f32(scale_log2e, scale_log2e), neg_m2 = pair_f32(neg_m, neg_m);
                uint64_t ps2[2] = {pair_f32(0.f, 0.f), pair_f32(0.f, 0.f)};
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    uint32_t pk[16];
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        float a0, a1;
                        unpair_f32(fma_f32x2(pair_f32(__uint_as_float(sv[c * 32 + 2 * j]),
                                                      __uint_as_float(sv[c * 32 + 2 * j + 1])),
                                             scale2, neg_m2), a0, a1);
                        const float p0 = fast_exp2(a0), p1 = fast_exp2(a1);
                        ps2[j & 1] = add_f32x2(ps2[j & 1], pair_f32(p0, p1));
                        pk[j] = pack_bf16(p0, p1);
                    }
                    t5::st16(s_addr + c * 16, pk);
                }
                {
                    float s0, s1, s2, s3;
                    unpair_f32(ps2[0], s0, s1);
                    unpair_f32(ps2[1], s2, s3);
                    l += (s0 + s2) + (s1 + s3);
                }
                t5::wait_st();
                t5::fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&p_full[x]));
            }
            // ---- the output of this row
            ok = mbar_wait(smem_u32(&o_done[x]), 0, ok ? 400000 : 1) && ok;
            t5::fence_after();
            if constexpr (TWO_MAPS) {
                ok = mbar_wait(smem_u32(&o_done[x ^ 1]), 0, ok ? 400000 : 1) && ok;
                t5::fence_after();
                if (!ok) failed_s = 1;
                map_scale_s[x][row] = (x == 0 ? 1.0f : -two.factor) / l;
                asm volatile("bar.sync 1, 256;\n" ::: "memory");     // the two softmax warp groups
                const float c0 = map_scale_s[0][row], c1 = map_scale_s[1][row];
                const uint32_t col0 = x * (HD / 2);                  // this warp group's half of the head
                const uint32_t a_addr = tmem_o + lane_addr + col0, b_addr = a_addr + kPpBN;
                float dif[HD / 2];
                float ss = 0.f;
#pragma unroll
                for (int c = 0; c < HD / 64; ++c) {
                    uint32_t v[32], u[32];
                    t5::ld32_nowait(a_addr + c * 32, v);
                    t5::ld32_nowait(b_addr + c * 32, u);
                    t5::wait_ld();
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        const float y = fmaf(__uint_as_float(u[j]), c1, __uint_as_float(v[j]) * c0);
                        dif[c * 32 + j] = y;
                        ss = fmaf(y, y, ss);
                    }
                }
                map_square_s[x][row] = ss;
                asm volatile("bar.sync 1, 256;\n" ::: "memory");
                if (row < rows) {
                    const float mean = (map_square_s[0][row] + map_square_s[1][row]) / static_cast<float>(HD);
                    const float f = two.gain / sqrtf(mean + two.eps) *
                                    two_map_gate<__nv_bfloat16>(two, static_cast<size_t>(row0 + row), head);
                    __nv_bfloat16* dst = out + static_cast<size_t>(row0 + row) * nq * HD + head * HD + col0;
#pragma unroll
                    for (int d = 0; d < HD / 2; d += 8) {
                        uint4 w;
                        w.x = pack_bf16(dif[d] * f, dif[d + 1] * f);
                        w.y = pack_bf16(dif[d + 2] * f, dif[d + 3] * f);
                        w.z = pack_bf16(dif[d + 4] * f, dif[d + 5] * f);
                        w.w = pack_bf16(dif[d + 6] * f, dif[d + 7] * f);
                        *reinterpret_cast<uint4*>(dst + d) = w;
                    }
                }
            } else {
                if (!ok) failed_s = 1;
                // a sink: one more score in the denominator, without a value
                if (sinks != nullptr) l += fast_exp2(sinks[head] * 1.4426950408889634f - m);
                const float inv = 1.0f / l;
                const int r = x * kPpBM + row;
                __nv_bfloat16* dst = out + static_cast<size_t>(row0 + r) * nq * HD + head * HD;
                auto store8 = [](__nv_bfloat16* p, const float* y) {
                    uint4 w;
                    w.x = pack_bf16(y[0], y[1]);
                    w.y = pack_bf16(y[2], y[3]);
                    w.z = pack_bf16(y[4], y[5]);
                    w.w = pack_bf16(y[6], y[7]);
                    *reinterpret_cast<uint4*>(p) = w;
                };
                if (turn == nullptr) {
#pragma unroll
                    for (int c = 0; c < HD / 32; ++c) {
                        uint32_t v[32];
                        t5::ld32_nowait(o_addr + c * 32, v);
                        t5::wait_ld();
                        if (r < rows) {
#pragma unroll
                            for (int d = 0; d < 32; d += 8) {
                                float y[8];
#pragma unroll
                                for (int j = 0; j < 8; ++j) y[j] = __uint_as_float(v[d + j]) * inv;
                                store8(dst + c * 32 + d, y);
                            }
                        }
                    }
                } else {
                    // the pairs (d, d + HD / 2) are turned back by the row's angles before they are rounded
#pragma unroll
                    for (int c = 0; c < HD / 64; ++c) {
                        uint32_t v[32], u[32];
                        t5::ld32_nowait(o_addr + c * 32, v);
                        t5::ld32_nowait(o_addr + HD / 2 + c * 32, u);
                        t5::wait_ld();
                        if (r < rows) {
                            const float4* tr = reinterpret_cast<const float4*>(turn + static_cast<size_t>(row0 + r) * (HD / 2) + c * 32);
#pragma unroll
                            for (int d = 0; d < 32; d += 8) {
                                float y0[8], y1[8];
#pragma unroll
                                for (int j = 0; j < 8; j += 2) {
                                    const float4 cs = tr[(d + j) / 2];          // two pairs' cosine, sine
                                    const float p0 = __uint_as_float(v[d + j]) * inv, q0 = __uint_as_float(u[d + j]) * inv;
                                    const float p1 = __uint_as_float(v[d + j + 1]) * inv, q1 = __uint_as_float(u[d + j + 1]) * inv;
                                    y0[j] = fmaf(p0, cs.x, q0 * cs.y);
                                    y1[j] = fmaf(q0, cs.x, -(p0 * cs.y));
                                    y0[j + 1] = fmaf(p1, cs.z, q1 * cs.w);
                                    y1[j + 1] = fmaf(q1, cs.z, -(p1 * cs.w));
                                }
                                store8(dst + c * 32 + d, y0);
                                store8(dst + HD / 2 + c * 32 + d, y1);
                            }
                        }
                    }
                }
            }
        }
    }
    t5::fence_before();
    __syncthreads();
    if (warp == 9) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base_s),
                     "r"(TmemCols)
                     : "memory");
    }
    if (tid == 0 && failed_s) atomicExch(&g_prefill_pp_error, 1);
}

template <int HD, bool TWO_MAPS = false>
int launch_prefill_pp(const CUtensorMap* q_map, const CUtensorMap* kv_map, long long k_row0,
                      long long v_row0, const int* block_table, int bt_stride, const int* cu_q,
                      const int* ctx_len, const int* tiles, int n_tiles, int nq, int nkv,
                      int page_size, float scale, int window, const float* sinks, const float* turn,
                      void* out, cudaStream_t stream, int keep = 0, const TwoMaps& two = TwoMaps{}) {
    const size_t smem = (TWO_MAPS ? 1 : 2) * (HD / 64) * kPpQHalf +
                        (pp_k_stages(HD) + pp_v_stages(HD)) * (HD / 64) * kPpKvHalf + 1024;
    cudaFuncSetAttribute(paged_prefill_pp_kernel<HD, TWO_MAPS>,
                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    dim3 grid(static_cast<unsigned>(nq) * n_tiles);
    launch_pdl(paged_prefill_pp_kernel<HD, TWO_MAPS>, grid, dim3(kPpThreads), smem, stream, *q_map, *kv_map,
               k_row0, v_row0, block_table, bt_stride, cu_q, ctx_len, tiles, nq, nkv, page_size,
               scale * 1.4426950408889634f, window, sinks, reinterpret_cast<const float2*>(turn),
               static_cast<__nv_bfloat16*>(out), n_tiles, keep, two);
    return launch_status();
}

}  // namespace somi

using namespace somi;

SOMI_API int somi_prefill_pp_q_tile() { return kPpRows; }

SOMI_API int somi_prefill_pp_supported(int nq, int nkv, int hd, int page_size) {
    if (nkv <= 0 || nq % nkv) return 0;
    if (hd != 64 && hd != 128) return 0;
    return page_size >= 8 && page_size % 8 == 0 && kPpBN % page_size == 0;
}

SOMI_API int somi_prefill_pp_error() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_prefill_pp_error, sizeof(int)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_prefill_pp_error, &zero, sizeof(int));
    return v;
}

// `tiles`: int32 [n_tiles, 3] = (request, first row, rows <= 256) over the multi-token requests;
// `sinks`, `turn`: as for the decode kernel (attention_decode_tma.cu), or null;
// `q_map`: the projection buffer's map with boxes of 128 rows x 64 columns (as the one-tile kernel's).
SOMI_API int somi_paged_attention_prefill_pp(
    const void* q_map, const void* kv_map, long long k_row0, long long v_row0,
    const int* block_table, int bt_stride, const int* cu_q, const int* ctx_len, const int* tiles,
    int n_tiles, int nq, int nkv, int hd, int page_size, float scale, int window, const float* sinks,
    const float* turn, void* out, cudaStream_t stream) {
    if (n_tiles <= 0) return 0;
    if (!somi_prefill_pp_supported(nq, nkv, hd, page_size)) return SOMI_ERR_UNSUPPORTED;
    const CUtensorMap* qm = static_cast<const CUtensorMap*>(q_map);
    const CUtensorMap* km = static_cast<const CUtensorMap*>(kv_map);
    if (hd == 64)
        return launch_prefill_pp<64>(qm, km, k_row0, v_row0, block_table, bt_stride, cu_q, ctx_len,
                                     tiles, n_tiles, nq, nkv, page_size, scale, window, sinks, turn, out,
                                     stream);
    return launch_prefill_pp<128>(qm, km, k_row0, v_row0, block_table, bt_stride, cu_q, ctx_len, tiles,
                                  n_tiles, nq, nkv, page_size, scale, window, sinks, turn, out, stream);
}

// Attention in two maps (two_maps.cuh) of prompt portions.  hd (64 or 128): the width of a value and of
// the two queries, or keys, of a head together.  `tiles`: as above with rows <= 128.
SOMI_API int somi_two_map_attention_prefill(
    const void* q_map, const void* kv_map, long long k_row0, long long v_row0,
    const int* block_table, int bt_stride, const int* cu_q, const int* ctx_len, const int* tiles,
    int n_tiles, int nq, int nkv, int hd, int page_size, float scale, int window, int keep, float factor,
    float eps, float gain, const void* gate, long long gate_stride, void* out, cudaStream_t stream) {
    if (n_tiles <= 0) return 0;
    if (!somi_prefill_pp_supported(nq, nkv, hd, page_size) || window < 0 || keep < 0 || (keep > 0 && window == 0))
        return SOMI_ERR_UNSUPPORTED;
    const CUtensorMap* qm = static_cast<const CUtensorMap*>(q_map);
    const CUtensorMap* km = static_cast<const CUtensorMap*>(kv_map);
    const TwoMaps two{factor, eps, gain, gate, gate_stride};
    if (hd == 64)
        return launch_prefill_pp<64, true>(qm, km, k_row0, v_row0, block_table, bt_stride, cu_q, ctx_len,
                                           tiles, n_tiles, nq, nkv, page_size, scale, window, nullptr,
                                           nullptr, out, stream, keep, two);
    return launch_prefill_pp<128, true>(qm, km, k_row0, v_row0, block_table, bt_stride, cu_q, ctx_len,
                                        tiles, n_tiles, nq, nkv, page_size, scale, window, nullptr, nullptr,
                                        out, stream, keep, two);
}
