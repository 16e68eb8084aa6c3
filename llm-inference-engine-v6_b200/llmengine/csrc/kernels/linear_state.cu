// Mixers whose memory is a matrix per head ("linear state"): S [dk, dv] per request and head, float32, kept in the request's state
// slot, updated token after token by a rank-one write k v^T and read by a query. Four update rules share one kernel:
//
//   MODE 0  decay a key channel, write, read:   S <- diag(a_t) S + k_t v_t^T;              o_t = S^T q_t
//   MODE 1  read with a bonus, decay, write:    o_t = (S + diag(u) k_t v_t^T)^T q_t;       S <- diag(a_t) S + k_t v_t^T
//   MODE 2  delta rule with a decay a head:     S <- g_t S;  w = beta_t (v_t - S^T k_t);   S <- S + k_t w^T;   o_t = S^T q_t
//           (q and k made unit vectors per head first: x / sqrt(sum x^2 + unit_eps))
//   MODE 3  delta rule with a decay a channel:  S <- diag(a_t) S;  the rest as MODE 2, beta_t a number a head of its own
//
// Every column S[:, j] evolves by itself, so a block takes a (request, head, tile of columns) and walks the request's tokens of the
// step in order; a column's dk numbers are spread over R lanes of a warp (KPT = 16 numbers a lane), the two dot products of a
// token are sums over a lane's numbers and then over the R lanes (xor shuffles, a fixed order). The tokens' q, k, decays and v
// come through shared memory in tiles of a few tokens that warps of their own fetch ahead of the walk (the sums of the products'
// parts, the unit norms and the query's scale are applied there), so the walk itself only syncs once a tile. Results never depend
// on how a request was cut into steps, on the batch or on the slot: the same additions happen in the same order.
//
// In the slot a head's matrix is stored as the threads hold it: number (m, column j, lane r) at ((m * dv + j) * R + r), which is
// S[channel_of(m, r, R), j]; loads and stores of a warp are then 128 contiguous bytes. R = the power of two >= dk / 16.
//
// Beside it: token_shift (every projection's own blend of a token's input with the previous token's, the previous token of a
// portion's first token coming from the slot), delta_gates (the delta rule's decay and write strength per head), channel_gates
// (two low-rank maps and a sigmoid at once: a decay per head and key channel, the gate of the result, the write strength) and head_norm_gate (every head's
// result divided by its root mean square, times a weight, times silu or sigmoid of a gate; wide heads, or all heads as one, a block a
// row) and silu_sums (activated projections for portions, whose tiles then arrive as they are).
#include "common.cuh"
#include "mma_common.cuh"

#include <cmath>

namespace {

constexpr int KPT = 16;       // state numbers of a column that one lane holds
constexpr int LS_THREADS = 128;   // threads that hold the state, at most: fewer when the blocks would not fill the device
constexpr int LS_FETCHERS = 128;  // threads behind them that fetch the tiles of tokens ahead
constexpr int LS_BLOCK = LS_THREADS + LS_FETCHERS;
constexpr int LS_BUFFERS = 3;    // tiles in shared memory: walked, landing, issued
constexpr int WIDE_NORM_FROM = 512;  // rows of more numbers are normed by a block each
constexpr size_t LS_SMEM = 112 * 1024;  // of the tiles, at most (portions)

__device__ __forceinline__ float parts_sum(const float* __restrict__ p, int n_parts, size_t pstride, size_t i) {
  float s = p[i];
  for (int k = 1; k < n_parts; ++k) s += p[(size_t)k * pstride + i];
  return s;
}

struct Sums {  // columns off.. of float32 sums [parts, rows, width]
  const float* p; int n; size_t stride; int width, off;
};

struct LinearStateParams {
  Sums q, k, v, b;                                 // b: MODE 3, one number a head
  const float* decay; int decay_width, decay_off;  // float32 rows: MODE 0/1/3 a number a (head, key channel); MODE 2 [g: H | beta: H]
  const float* bonus;                              // MODE 1: [H, dk]
  float* state;                                    // [slots, H, R * KPT, dv] in the layout above
  const int* seq_qoff; const int* seq_ntok; const int* seq_slot;
  float* out;                                      // [tokens, H * dv]
  int H, G, dk, dv, R, tile;
  float q_scale, unit_eps;
  int silu;      // MODE 0: q, k and v are silu of the sums
  int walkers;   // threads of a block that hold the state (a multiple of 32 and of R); LS_FETCHERS more fetch
  int one_part;  // every product comes in one part
  int vec4;      // every row and column offset is a multiple of four numbers on a 16-byte boundary
};

// Key channel of a lane's number m: the lane holds four groups of four neighbouring channels, group c of lane r being channels
// 4 (c R + r) .. + 3, so that a lane reads a group with one 16-byte load and the R lanes of a column read 16 R contiguous bytes.
__device__ __forceinline__ int channel_of(int m, int lane_r, int R) { return (((m >> 2) * R + lane_r) << 2) + (m & 3); }

template <int R>
__device__ __forceinline__ void load16(float (&x)[KPT], const float* __restrict__ row) {
#pragma unroll
  for (int c = 0; c < KPT / 4; ++c) {
    const float4 t = *reinterpret_cast<const float4*>(row + 4 * c * R);
    x[4 * c] = t.x; x[4 * c + 1] = t.y; x[4 * c + 2] = t.z; x[4 * c + 3] = t.w;
  }
}

template <int R>
__device__ __forceinline__ float lanes_sum(float x) {  // over the R lanes of a column, a fixed order
#pragma unroll
  for (int o = R >> 1; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
  return x;
}

struct TileRows {  // a tile of tokens in shared memory
  float* q;  // [tile][dkp]
  float* k;  // [tile][dkp]
  float* a;  // [tile][dkp] (MODE 0/1/3) or [tile][2] (MODE 2)
  float* v;  // [tile][dv]
  float* b;  // [tile] (MODE 3)
};

// A tile of tokens through the rule: s the thread's numbers of its column, v[tt * dv + col] the column's value; out points at the
// column's result of the tile's first token. A lane's sixteen products are summed as four interleaved chains ((c0 + c1) +
// (c2 + c3), chain i taking m = i, i + 4, ...), which shortens the dependent chain of a token fourfold; the order is fixed, so a
// token's result is the same in every step that computes it. What the state does not wait for is moved out of its way: the next
// token's rows are read while this one is computed, and a result's sum over the lanes and its store happen one token late.
template <int MODE, int R>
__device__ __forceinline__ void walk_tile(float (&s)[KPT], const float (&u)[KPT], const TileRows& rows, int dv, int col, int cnt, int lane_r,
                                          bool live, float* __restrict__ out, size_t out_stride) {
  constexpr int dkp = R * KPT, a_stride = MODE == 2 ? 2 : dkp;
  float kk[KPT], qq[KPT], aa[KPT], vj, g = 0.f, beta = 0.f;
  auto read = [&](int tt, float (&k_)[KPT], float (&q_)[KPT], float (&a_)[KPT], float& v_, float& g_, float& b_) {
    load16<R>(k_, rows.k + tt * dkp + 4 * lane_r);
    load16<R>(q_, rows.q + tt * dkp + 4 * lane_r);
    if (MODE != 2) {
      load16<R>(a_, rows.a + tt * a_stride + 4 * lane_r);
    } else {
      g_ = rows.a[tt * a_stride];
      b_ = rows.a[tt * a_stride + 1];
    }
    if (MODE == 3) b_ = rows.b[tt];
    v_ = live ? rows.v[tt * dv + col] : 0.f;
  };
  read(0, kk, qq, aa, vj, g, beta);
  float pend = 0.f;
#pragma unroll 4
  for (int tt = 0; tt < cnt; ++tt) {
    float kn[KPT], qn[KPT], an[KPT], vn, gn = 0.f, bn = 0.f;
    read(min(tt + 1, cnt - 1), kn, qn, an, vn, gn, bn);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (MODE == 0) {
#pragma unroll
      for (int m = 0; m < KPT; ++m) {
        s[m] = fmaf(kk[m], vj, aa[m] * s[m]);
        acc[m & 3] = fmaf(s[m], qq[m], acc[m & 3]);
      }
    } else if (MODE == 1) {
#pragma unroll
      for (int m = 0; m < KPT; ++m) {
        const float kv = kk[m] * vj;
        acc[m & 3] = fmaf(fmaf(u[m], kv, s[m]), qq[m], acc[m & 3]);
        s[m] = fmaf(aa[m], s[m], kv);
      }
    } else {
      float dot[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int m = 0; m < KPT; ++m) {
        s[m] *= MODE == 3 ? aa[m] : g;
        dot[m & 3] = fmaf(s[m], kk[m], dot[m & 3]);
      }
      const float d = lanes_sum<R>((dot[0] + dot[1]) + (dot[2] + dot[3]));
      const float w = beta * (vj - d);
#pragma unroll
      for (int m = 0; m < KPT; ++m) {
        s[m] = fmaf(kk[m], w, s[m]);
        acc[m & 3] = fmaf(s[m], qq[m], acc[m & 3]);
      }
    }
    if (tt > 0) {
      const float o = lanes_sum<R>(pend);
      if (live && lane_r == 0) out[(size_t)(tt - 1) * out_stride] = o;
    }
    pend = (acc[0] + acc[1]) + (acc[2] + acc[3]);
#pragma unroll
    for (int m = 0; m < KPT; ++m) {
      kk[m] = kn[m];
      qq[m] = qn[m];
      if (MODE != 2) aa[m] = an[m];
    }
    vj = vn; g = gn; beta = bn;
  }
  const float o = lanes_sum<R>(pend);
  if (live && lane_r == 0) out[(size_t)(cnt - 1) * out_stride] = o;
}

__device__ __forceinline__ void copy4_async(float* smem_dst, const float* gmem_src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ void copy16_async(float* smem_dst, const float* gmem_src) {  // both on 16-byte boundaries
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(smem_dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(gmem_src) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copies_wait_but_last() { asm volatile("cp.async.wait_group 1;" ::: "memory"); }

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// A tile's rows into shared memory by the n_thr fetching threads (thread `tid` of them), in two steps so that two tiles can be
// on their way while a third is walked. fetch_issue: every thread takes elements of the whole tile in turn. Products in one
// part (a prompt's portion) are copied asynchronously (16 bytes a copy where every address allows it), no registers held, and
// the copies of a tile are one group. Products in several parts (few tokens, K cut) go through registers, a few elements at a
// time, the parts added in their order (and silu applied, where the rule reads activated projections). fetch_finish, once the tile's
// group has landed: the thread activates its own copies and scales its own queries; the
// delta rule's unit norms need a token's whole row, so the fetchers meet (barrier 1 is theirs alone) and a warp a token
// scales what was stored.
template <int MODE>
__device__ __forceinline__ void fetch_issue(const LinearStateParams& p, size_t row0, int cnt, int head, int kvh, int dk, int dkp, int dv,
                                            int tid, int n_thr, const TileRows& rows) {
  const bool unit = MODE >= 2 && p.unit_eps >= 0.f;
  const float qmul = unit ? 1.0f : p.q_scale;
  const int lg = __ffs(dkp) - 1;  // dkp is a power of two
  const int n_qk = cnt * dkp, n_v = cnt * dv;
  if (p.one_part) {
    if (p.vec4) {
      for (int e = tid; e < (n_qk >> 2); e += n_thr) {
        const int tt = e >> (lg - 2), i = (e << 2) & (dkp - 1);
        const size_t row = row0 + tt;
        if (i < dk) {
          copy16_async(rows.q + 4 * e, p.q.p + row * p.q.width + p.q.off + (size_t)kvh * dk + i);
          copy16_async(rows.k + 4 * e, p.k.p + row * p.k.width + p.k.off + (size_t)kvh * dk + i);
          if (MODE != 2) copy16_async(rows.a + 4 * e, p.decay + row * p.decay_width + p.decay_off + (size_t)head * dk + i);
        } else {
          const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
          *reinterpret_cast<float4*>(rows.q + 4 * e) = z;
          *reinterpret_cast<float4*>(rows.k + 4 * e) = z;
          if (MODE != 2) *reinterpret_cast<float4*>(rows.a + 4 * e) = z;
        }
      }
      const int dv4 = dv >> 2;
      for (int e = tid; e < (n_v >> 2); e += n_thr) {
        const int tt = e / dv4, j = (e - tt * dv4) << 2;
        copy16_async(rows.v + 4 * e, p.v.p + (row0 + tt) * p.v.width + p.v.off + (size_t)head * dv + j);
      }
    } else {
      for (int e = tid; e < n_qk; e += n_thr) {
        const int tt = e >> lg, i = e & (dkp - 1);
        const size_t row = row0 + tt;
        if (i < dk) {
          copy4_async(rows.q + e, p.q.p + row * p.q.width + p.q.off + (size_t)kvh * dk + i);
          copy4_async(rows.k + e, p.k.p + row * p.k.width + p.k.off + (size_t)kvh * dk + i);
          if (MODE != 2) copy4_async(rows.a + e, p.decay + row * p.decay_width + p.decay_off + (size_t)head * dk + i);
        } else {
          rows.q[e] = rows.k[e] = 0.f;
          if (MODE != 2) rows.a[e] = 0.f;
        }
      }
      for (int e = tid; e < n_v; e += n_thr) {
        const int tt = e / dv, j = e - tt * dv;
        copy4_async(rows.v + e, p.v.p + (row0 + tt) * p.v.width + p.v.off + (size_t)head * dv + j);
      }
    }
    if (MODE == 2)
      for (int e = tid; e < 2 * cnt; e += n_thr)
        copy4_async(rows.a + e, p.decay + (row0 + (e >> 1)) * p.decay_width + p.decay_off + (e & 1) * p.H + head);
    if (MODE == 3)
      for (int e = tid; e < cnt; e += n_thr) copy4_async(rows.b + e, p.b.p + (row0 + e) * p.b.width + p.b.off + head);
    return;
  }
  constexpr int U = 4;  // elements a thread has in flight: their loads are issued together, part after part in the parts' order
  for (int e0 = tid; e0 < n_qk; e0 += U * n_thr) {
    float qv[U], kv[U], av[U];
    size_t qi[U], ki[U];
    bool ok[U];
#pragma unroll
    for (int x = 0; x < U; ++x) {
      const int e = e0 + x * n_thr, tt = e >> lg, i = e & (dkp - 1);
      const size_t row = row0 + tt;
      ok[x] = e < n_qk && i < dk;
      qi[x] = row * p.q.width + p.q.off + (size_t)kvh * dk + i;
      ki[x] = row * p.k.width + p.k.off + (size_t)kvh * dk + i;
      qv[x] = kv[x] = 0.f;
      av[x] = (MODE != 2 && ok[x]) ? p.decay[row * p.decay_width + p.decay_off + (size_t)head * dk + i] : 0.f;
    }
    for (int part = 0; part < p.q.n; ++part) {
#pragma unroll
      for (int x = 0; x < U; ++x)
        if (ok[x]) qv[x] += p.q.p[(size_t)part * p.q.stride + qi[x]];
    }
    for (int part = 0; part < p.k.n; ++part) {
#pragma unroll
      for (int x = 0; x < U; ++x)
        if (ok[x]) kv[x] += p.k.p[(size_t)part * p.k.stride + ki[x]];
    }
#pragma unroll
    for (int x = 0; x < U; ++x) {
      const int e = e0 + x * n_thr;
      if (e < n_qk) {
        rows.q[e] = (MODE == 0 && p.silu ? silu_f(qv[x]) : qv[x]) * qmul;
        rows.k[e] = MODE == 0 && p.silu ? silu_f(kv[x]) : kv[x];
        if (MODE != 2) rows.a[e] = av[x];
      }
    }
  }
  for (int e0 = tid; e0 < n_v; e0 += U * n_thr) {
    float vv[U];
    size_t vi[U];
#pragma unroll
    for (int x = 0; x < U; ++x) {
      const int e = min(e0 + x * n_thr, n_v - 1), tt = e / dv, j = e - tt * dv;
      vi[x] = (row0 + tt) * p.v.width + p.v.off + (size_t)head * dv + j;
      vv[x] = 0.f;
    }
    for (int part = 0; part < p.v.n; ++part) {
#pragma unroll
      for (int x = 0; x < U; ++x) vv[x] += p.v.p[(size_t)part * p.v.stride + vi[x]];
    }
#pragma unroll
    for (int x = 0; x < U; ++x)
      if (e0 + x * n_thr < n_v) rows.v[e0 + x * n_thr] = MODE == 0 && p.silu ? silu_f(vv[x]) : vv[x];
  }
  if (MODE == 2)
    for (int e = tid; e < 2 * cnt; e += n_thr) rows.a[e] = p.decay[(row0 + (e >> 1)) * p.decay_width + p.decay_off + (e & 1) * p.H + head];
  if (MODE == 3)
    for (int e = tid; e < cnt; e += n_thr) rows.b[e] = parts_sum(p.b.p, p.b.n, p.b.stride, (row0 + e) * p.b.width + p.b.off + head);
}

template <int MODE>
__device__ __forceinline__ void fetch_finish(const LinearStateParams& p, int cnt, int dk, int dkp, int dv, int tid, int n_thr, const TileRows& rows) {
  const bool unit = MODE >= 2 && p.unit_eps >= 0.f;
  const float qmul = unit ? 1.0f : p.q_scale;
  const int n_qk = cnt * dkp;
  if (MODE == 0 && p.one_part && p.silu) {  // the thread's own copies, as fetch_issue dealt them (a group of four numbers or one)
    const int n_v = cnt * dv, V = p.vec4 ? 4 : 1;
    for (int e = tid * V; e < n_qk; e += n_thr * V)
      for (int i = e; i < e + V; ++i) {
        rows.q[i] = silu_f(rows.q[i]);
        rows.k[i] = silu_f(rows.k[i]);
      }
    for (int e = tid * V; e < n_v; e += n_thr * V)
      for (int i = e; i < e + V; ++i) rows.v[i] = silu_f(rows.v[i]);
  }
  if (p.one_part && qmul != 1.0f) {
    if (p.vec4) {
      for (int e = tid; e < (n_qk >> 2); e += n_thr) {
        float4 t = *reinterpret_cast<float4*>(rows.q + 4 * e);
        t.x *= qmul; t.y *= qmul; t.z *= qmul; t.w *= qmul;
        *reinterpret_cast<float4*>(rows.q + 4 * e) = t;
      }
    } else {
      for (int e = tid; e < n_qk; e += n_thr) rows.q[e] *= qmul;
    }
  }
  if (unit) {
    asm volatile("bar.sync 1, %0;" ::"r"(n_thr) : "memory");
    const int lane = tid & 31;
    for (int tt = tid >> 5; tt < cnt; tt += n_thr >> 5) {
      float ssq = 0.f, ssk = 0.f;
      for (int i = lane; i < dkp; i += 32) {
        ssq = fmaf(rows.q[tt * dkp + i], rows.q[tt * dkp + i], ssq);
        ssk = fmaf(rows.k[tt * dkp + i], rows.k[tt * dkp + i], ssk);
      }
      ssq = warp_sum(ssq);
      ssk = warp_sum(ssk);
      const float qm = p.q_scale / sqrtf(ssq + p.unit_eps), km = 1.0f / sqrtf(ssk + p.unit_eps);
      for (int i = lane; i < dkp; i += 32) {  // the lane's own numbers again
        rows.q[tt * dkp + i] *= qm;
        rows.k[tt * dkp + i] *= km;
      }
    }
  }
}

// Threads 0 .. p.walkers - 1 hold the state and walk; the LS_FETCHERS threads behind them only fetch. Three buffers: while the walkers are in
// tile i of the request's tokens, tile i + 1 lands and is finished and the copies of tile i + 2 are issued; the block meets once
// a tile. (A decode step has one tile of one token; the walkers read their state while it is fetched.)
// FEW: for steps of about a token a request (decoding). The same code held to half the registers, so that two blocks share a
// multiprocessor: such a step is a state's trip to memory and back, and more blocks in flight hide more of it.
template <int MODE, int R, bool FEW>
__global__ void __launch_bounds__(LS_BLOCK, FEW ? 2 : 1) linear_state_kernel(const LinearStateParams p) {
  extern __shared__ __align__(16) float sh_ls[];
  dep_launch();
  dep_wait();
  const int seq = blockIdx.z, head = blockIdx.y, dk = p.dk, dv = p.dv;
  const int n_tok = p.seq_ntok[seq];
  if (n_tok <= 0) return;
  const int first = p.seq_qoff[seq];
  constexpr int dkp = R * KPT, a_stride = MODE == 2 ? 2 : dkp;
  const int kvh = head / (p.H / p.G);
  const bool walker = threadIdx.x < p.walkers;
  const int lane_r = threadIdx.x & (R - 1);
  const int col = blockIdx.x * (p.walkers / R) + threadIdx.x / R;
  const bool live = walker && col < dv;
  const int tile = p.tile, n_tiles = (n_tok + tile - 1) / tile;
  const size_t a_floats = ((size_t)tile * a_stride + 3) & ~(size_t)3;
  const size_t buf_floats = ((size_t)tile * (2 * dkp + dv + (MODE == 3 ? 1 : 0)) + a_floats + 3) & ~(size_t)3;  // every region but the last starts on 16 bytes
  auto rows_of = [&](int i) {
    TileRows r;
    r.q = sh_ls + (size_t)(i % LS_BUFFERS) * buf_floats;
    r.k = r.q + (size_t)tile * dkp;
    r.a = r.k + (size_t)tile * dkp;
    r.v = r.a + a_floats;
    r.b = r.v + (size_t)tile * dv;
    return r;
  };
  const int ftid = threadIdx.x - p.walkers, n_fetch = LS_FETCHERS;
  auto issue = [&](int i) {  // a group of copies a call, empty behind the last tile
    if (i < n_tiles)
      fetch_issue<MODE>(p, (size_t)(first + i * tile), min(tile, n_tok - i * tile), head, kvh, dk, dkp, dv, ftid, n_fetch, rows_of(i));
    copies_commit();
  };
  auto finish = [&](int i) {
    if (i < n_tiles) fetch_finish<MODE>(p, min(tile, n_tok - i * tile), dk, dkp, dv, ftid, n_fetch, rows_of(i));
  };

  float* st = p.state + ((size_t)p.seq_slot[seq] * p.H + head) * (size_t)dkp * dv;
  float s[KPT], u[KPT];
  if (walker) {
#pragma unroll
    for (int m = 0; m < KPT; ++m) {
      s[m] = live ? st[((size_t)m * dv + col) * R + lane_r] : 0.f;
      const int i = channel_of(m, lane_r, R);
      u[m] = (MODE == 1 && i < dk) ? p.bonus[(size_t)head * dk + i] : 0.f;
    }
  } else {
    issue(0);
    issue(1);
    copies_wait_but_last();
    finish(0);
  }
  __syncthreads();
  for (int i = 0; i < n_tiles; ++i) {
    if (walker) {
      const int t0 = i * tile;
      walk_tile<MODE, R>(s, u, rows_of(i), dv, col, min(tile, n_tok - t0), lane_r, live,
                         p.out + (size_t)(first + t0) * p.H * dv + (size_t)head * dv + col, (size_t)p.H * dv);
    } else {
      issue(i + 2);
      copies_wait_but_last();
      finish(i + 1);
    }
    __syncthreads();  // tile i has been used up, tile i + 1 is in place
  }
  if (live) {
#pragma unroll
    for (int m = 0; m < KPT; ++m) st[((size_t)m * dv + col) * R + lane_r] = s[m];
  }
}

// out[s][t, c] = x[t, c] + (prev[c] - x[t, c]) * mu[s, c], prev = the request's token before t (of this step, or from the slot)
template <typename T>
__global__ void token_shift_kernel(const T* __restrict__ x, const float* __restrict__ mu, int n_out, const float* __restrict__ shift_state,
                                   const int* __restrict__ token_seq, const int* __restrict__ seq_qoff, const int* __restrict__ seq_slot,
                                   T* __restrict__ out, int n_tokens, int D) {
  dep_launch();
  dep_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= D) return;
  for (int tok = blockIdx.y; tok < n_tokens; tok += gridDim.y) {
    const int seq = token_seq[tok];
    const float cur = to_f32(x[(size_t)tok * D + c]);
    const float prev = tok > seq_qoff[seq] ? to_f32(x[(size_t)(tok - 1) * D + c]) : shift_state[(size_t)seq_slot[seq] * D + c];
    const float d = prev - cur;
    for (int s = 0; s < n_out; ++s) out[((size_t)s * n_tokens + tok) * D + c] = from_f32<T>(fmaf(d, mu[(size_t)s * D + c], cur));
  }
}

template <typename T>
__global__ void token_shift_state_kernel(const T* __restrict__ x, float* __restrict__ shift_state, const int* __restrict__ seq_qoff,
                                         const int* __restrict__ seq_ntok, const int* __restrict__ seq_slot, int n_seqs, int D) {
  dep_launch();
  dep_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)n_seqs * D) return;
  const int seq = (int)(i / D), c = (int)(i - (size_t)seq * D);
  const int n = seq_ntok[seq];
  if (n > 0) shift_state[(size_t)seq_slot[seq] * D + c] = to_f32(x[(size_t)(seq_qoff[seq] + n - 1) * D + c]);
}

// out[t] = [g: H | beta: H], g = exp(-exp(a_log[h]) * softplus(a[t, h] + dt_bias[h])), beta = sigmoid(b[t, h])
__global__ void delta_gates_kernel(const Sums a, const Sums b, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                   float* __restrict__ out, int n_tokens, int H) {
  dep_launch();
  dep_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)n_tokens * H) return;
  const size_t tok = i / H;
  const int h = (int)(i - tok * H);
  const float z = parts_sum(a.p, a.n, a.stride, tok * a.width + a.off + h) + dt_bias[h];
  const float sp = z > 20.0f ? z : log1pf(expf(z));
  out[tok * 2 * H + h] = expf(-expf(a_log[h]) * sp);
  out[tok * 2 * H + H + h] = 1.0f / (1.0f + expf(-parts_sum(b.p, b.n, b.stride, tok * b.width + b.off + h)));
}

// Two low-rank maps of one product's sums in one launch. Columns x0.off .. + R0 of the sums feed map 0, the decay of a delta rule
// with a decay per key channel: out0[t, c] = exp(-exp(a_log[c / per]) * softplus(bias0[c] + sum_r w0[c, r] x0[t, r])); columns
// x1.off .. + R1 feed map 1, out1[t, c] = sum_r w1[c, r] x1[t, r], the sums of the result's gate. Beside them
// beta[t, h] = sigmoid(xb[t, h]), the write strengths of H heads. All float32.
struct ChannelGates {
  Sums x0, x1, xb;
  int R0, R1, C0, C1, per, H;
  const float* bias0; const float* a_log;
  float* out0; float* out1; float* beta;
  int n_tokens;
};

// beta of a block's tokens t0 .. t1: the first block of every row of blocks does it
__device__ __forceinline__ void write_beta(const ChannelGates& p, int t0, int t1) {
  for (int i = threadIdx.x; i < (t1 - t0) * p.H; i += blockDim.x) {
    const int t = t0 + i / p.H, h = i % p.H;
    p.beta[(size_t)t * p.H + h] = 1.0f / (1.0f + expf(-parts_sum(p.xb.p, p.xb.n, p.xb.stride, (size_t)t * p.xb.width + p.xb.off + h)));
  }
}

__device__ __forceinline__ float channel_decay(float z, float a_log) {
  return expf(-expf(a_log) * (z > 20.0f ? z : log1pf(expf(z))));
}

// A block: 32 channels of one map x 8 tokens; its four warps take a quarter of the rank each, warp 0 adds the quarters in index
// order. wt: the maps stored transposed [R, C] (neighbouring channels read neighbouring words).
template <typename T>
__global__ void __launch_bounds__(128) channel_gates_kernel(const ChannelGates p, const T* __restrict__ wt0, const T* __restrict__ wt1) {
  extern __shared__ __align__(16) float sm_cg[];  // low [R][8], then quarters [4][32][8]
  dep_launch();
  dep_wait();
  const int blocks0 = (p.C0 + 31) / 32;
  const bool first = (int)blockIdx.x < blocks0;
  const Sums x = first ? p.x0 : p.x1;
  const T* wt = first ? wt0 : wt1;
  const int R = first ? p.R0 : p.R1, C = first ? p.C0 : p.C1, c0 = ((int)blockIdx.x - (first ? 0 : blocks0)) * 32;
  float* low = sm_cg;
  float* quarter = sm_cg + (size_t)R * 8;
  const int t0 = blockIdx.y * 8;
  constexpr int U = 8;  // numbers a thread has in flight, part after part in the parts' order
  for (int i0 = threadIdx.x; i0 < 8 * R; i0 += U * 128) {
    float v[U];
    size_t at[U];
    bool ok[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * 128, tl = i / R, r = i - tl * R;
      ok[u] = i < 8 * R && t0 + tl < p.n_tokens;
      at[u] = (size_t)(t0 + tl) * x.width + x.off + r;
      v[u] = 0.f;
    }
    for (int k = 0; k < x.n; ++k) {
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (ok[u]) v[u] += x.p[(size_t)k * x.stride + at[u]];
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * 128, tl = i / R, r = i - tl * R;
      if (i < 8 * R) low[r * 8 + tl] = v[u];
    }
  }
  if (blockIdx.x == 0) write_beta(p, t0, min(t0 + 8, p.n_tokens));
  __syncthreads();
  const int lane = threadIdx.x & 31, part = threadIdx.x >> 5;
  const int c = min(c0 + lane, C - 1);
  const int per = (R + 3) / 4, r_end = min(R, (part + 1) * per);
  float acc[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
#pragma unroll 8
  for (int r = part * per; r < r_end; ++r) {
    const float wv = to_f32(wt[(size_t)r * C + c]);
    const float4 v0 = *reinterpret_cast<const float4*>(low + r * 8), v1 = *reinterpret_cast<const float4*>(low + r * 8 + 4);
    acc[0] = fmaf(wv, v0.x, acc[0]); acc[1] = fmaf(wv, v0.y, acc[1]); acc[2] = fmaf(wv, v0.z, acc[2]); acc[3] = fmaf(wv, v0.w, acc[3]);
    acc[4] = fmaf(wv, v1.x, acc[4]); acc[5] = fmaf(wv, v1.y, acc[5]); acc[6] = fmaf(wv, v1.z, acc[6]); acc[7] = fmaf(wv, v1.w, acc[7]);
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) quarter[(part * 32 + lane) * 8 + i] = acc[i];
  __syncthreads();
  if (c0 + lane >= C) return;
  const float b = first ? p.bias0[c] : 0.f, al = first ? p.a_log[c / p.per] : 0.f;
  for (int i = part; i < 8; i += 4) {  // every warp finishes two of the tokens
    const int t = t0 + i;
    if (t >= p.n_tokens) break;
    const float z = ((quarter[lane * 8 + i] + quarter[(32 + lane) * 8 + i]) + quarter[(64 + lane) * 8 + i]) + quarter[(96 + lane) * 8 + i] + b;
    if (first) p.out0[(size_t)t * C + c] = channel_decay(z, al);
    else p.out1[(size_t)t * C + c] = z;
  }
}

// The same maps for prompt-sized steps in bfloat16, on tensor cores: a block takes 64 tokens x 128 channels of one map, eight warps
// of 16 x 64 each; w0 [C0, R0], w1 [C1, R1] as the checkpoint stores them. The low-rank numbers enter as the sum of two bfloat16
// numbers (the number rounded, and what the rounding left), a product each, so they count with about 16 bits of mantissa.
constexpr int CG_TOK = 64, CG_COLS = 128, CG_K = 64, CG_LD = CG_K + 8, CG_THREADS = 256;
__global__ void __launch_bounds__(CG_THREADS, 3) channel_gates_mma_kernel(const ChannelGates p, const bf16* __restrict__ w0, const bf16* __restrict__ w1) {
  __shared__ __align__(16) bf16 hi_s[CG_TOK][CG_LD], lo_s[CG_TOK][CG_LD], w_s[CG_COLS][CG_LD];
  dep_launch();
  dep_wait();
  const int blocks0 = (p.C0 + CG_COLS - 1) / CG_COLS;
  const bool first = (int)blockIdx.x < blocks0;
  const Sums x = first ? p.x0 : p.x1;
  const bf16* w = first ? w0 : w1;
  const int R = first ? p.R0 : p.R1, C = first ? p.C0 : p.C1, c0 = ((int)blockIdx.x - (first ? 0 : blocks0)) * CG_COLS;
  const int t0 = blockIdx.y * CG_TOK, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wm = warp & 3, wn = warp >> 2;
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const bool quads = R % 8 == 0 && (reinterpret_cast<uintptr_t>(w) & 15u) == 0;
  for (int k0 = 0; k0 < R; k0 += CG_K) {
    if (k0 > 0) __syncthreads();  // everyone is done with the block before
    constexpr int U = CG_TOK * CG_K / CG_THREADS;  // numbers a thread has in flight
    float v[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = tid + u * CG_THREADS, t = i / CG_K, k = i % CG_K;
      v[u] = 0.f;
      if (t0 + t < p.n_tokens && k0 + k < R) v[u] = x.p[(size_t)(t0 + t) * x.width + x.off + k0 + k];  // (one part)
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = tid + u * CG_THREADS, t = i / CG_K, k = i % CG_K;
      const bf16 h = __float2bfloat16_rn(v[u]);
      hi_s[t][k] = h;
      lo_s[t][k] = __float2bfloat16_rn(v[u] - __bfloat162float(h));
    }
    if (quads) {
      for (int i = tid; i < CG_COLS * (CG_K / 8); i += CG_THREADS) {
        const int c = i / (CG_K / 8), k = (i % (CG_K / 8)) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (c0 + c < C && k0 + k < R) v = *reinterpret_cast<const uint4*>(w + (size_t)(c0 + c) * R + k0 + k);
        *reinterpret_cast<uint4*>(&w_s[c][k]) = v;
      }
    } else {
      for (int i = tid; i < CG_COLS * CG_K; i += CG_THREADS) {
        const int c = i / CG_K, k = i % CG_K;
        w_s[c][k] = (c0 + c < C && k0 + k < R) ? w[(size_t)(c0 + c) * R + k0 + k] : __float2bfloat16_rn(0.f);
      }
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < CG_K / 16; ++ks) {
      if (k0 + ks * 16 >= R) break;
      uint32_t ah[4], al[4];
      ldmatrix_x4(ah, &hi_s[wm * 16 + (lane % 16)][ks * 16 + (lane / 16) * 8]);
      ldmatrix_x4(al, &lo_s[wm * 16 + (lane % 16)][ks * 16 + (lane / 16) * 8]);
#pragma unroll
      for (int j2 = 0; j2 < 4; ++j2) {
        uint32_t b[4];
        ldmatrix_x4(b, &w_s[wn * 64 + j2 * 16 + (lane % 8) + (lane / 16) * 8][ks * 16 + ((lane / 8) % 2) * 8]);
        mma_bf16(acc[2 * j2], al, b[0], b[1]);
        mma_bf16(acc[2 * j2], ah, b[0], b[1]);
        mma_bf16(acc[2 * j2 + 1], al, b[2], b[3]);
        mma_bf16(acc[2 * j2 + 1], ah, b[2], b[3]);
      }
    }
  }
  if (blockIdx.x == 0) write_beta(p, t0, min(t0 + CG_TOK, p.n_tokens));
  float* out = first ? p.out0 : p.out1;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = c0 + wn * 64 + j * 8 + 2 * (lane % 4);
    if (c >= C) continue;
    const bool two = c + 1 < C;
    float b0 = 0.f, b1 = 0.f, r0 = 0.f, r1 = 0.f;
    if (first) {
      b0 = p.bias0[c];
      r0 = expf(p.a_log[c / p.per]);
      if (two) {
        b1 = p.bias0[c + 1];
        r1 = expf(p.a_log[(c + 1) / p.per]);
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = t0 + wm * 16 + lane / 4 + half * 8;
      if (t >= p.n_tokens) continue;
      float y0 = acc[j][2 * half] + b0, y1 = acc[j][2 * half + 1] + b1;
      if (first) {
        y0 = expf(-r0 * (y0 > 20.0f ? y0 : log1pf(expf(y0))));
        y1 = expf(-r1 * (y1 > 20.0f ? y1 : log1pf(expf(y1))));
      }
      float* dst = out + (size_t)t * C + c;
      if (two && (C & 1) == 0) {  // both numbers, on an 8-byte boundary
        *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
      } else {
        dst[0] = y0;
        if (two) dst[1] = y1;
      }
    }
  }
}

// a warp a (token, head): out = o / sqrt(mean(o^2) + eps) * weight * act(gate), act silu or sigmoid; weight [dv] for all heads or
// [H * dv]
template <typename T>
__global__ void __launch_bounds__(128)
    head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ weight, int weight_per_head, const Sums gate, float eps,
                          T* __restrict__ out, int n_tokens, int H, int dv, int sigmoid) {
  dep_launch();
  dep_wait();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * H) return;
  const int lane = threadIdx.x & 31;
  const size_t tok = (size_t)(item / H);
  const int head = (int)(item - (long long)tok * H);
  const float* row = o + tok * (size_t)H * dv + (size_t)head * dv;
  float ss = 0.f;
  for (int d = lane; d < dv; d += 32) ss = fmaf(row[d], row[d], ss);
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  for (int d = lane; d < dv; d += 32) {
    float v = row[d] * inv * weight[weight_per_head ? (size_t)head * dv + d : d];
    if (gate.p) {
      const float g = parts_sum(gate.p, gate.n, gate.stride, tok * gate.width + gate.off + (size_t)head * dv + d);
      v *= (sigmoid ? 1.0f : g) / (1.0f + expf(-g));
    }
    out[tok * (size_t)H * dv + (size_t)head * dv + d] = from_f32<T>(v);
  }
}

template <int V>
__device__ __forceinline__ void load_n(float (&x)[V], const float* p) {
  if constexpr (V == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    x[0] = t.x; x[1] = t.y; x[2] = t.z; x[3] = t.w;
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = p[e];
  }
}
template <int V>
__device__ __forceinline__ void store_n(float* p, const float (&x)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  else
#pragma unroll
    for (int e = 0; e < V; ++e) p[e] = x[e];
}
template <int V>
__device__ __forceinline__ void store_n(bf16* p, const float (&x)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1]), b = __floats2bfloat162_rn(x[2], x[3]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a);
    u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) p[e] = __float2bfloat16_rn(x[e]);
  }
}

// The same for wide rows (all heads normed together): a block a (token, head), its numbers in the threads' turns, then block_sum.
// V 4: rows of a multiple of four numbers on 16-byte boundaries, moved four at a time.
template <typename T, int V>
__global__ void __launch_bounds__(1024)
    wide_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ weight, int weight_per_head, const Sums gate, float eps,
                          T* __restrict__ out, int H, int dv, int sigmoid) {
  __shared__ float red[33];
  dep_launch();
  dep_wait();
  const size_t item = blockIdx.x, tok = item / H;
  const int head = (int)(item - tok * H);
  const float* row = o + item * dv;
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < dv; d += blockDim.x * V) {
    float x[V];
    load_n<V>(x, row + d);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(x[e], x[e], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + eps);
  for (int d = threadIdx.x * V; d < dv; d += blockDim.x * V) {
    float x[V], w[V], g[V], t[V];
    load_n<V>(x, row + d);
    load_n<V>(w, weight + (weight_per_head ? (size_t)head * dv + d : d));
    if (gate.p) {  // the parts in index order
      const float* gp = gate.p + tok * gate.width + gate.off + (size_t)head * dv + d;
      load_n<V>(g, gp);
#pragma unroll 4
      for (int k = 1; k < gate.n; ++k) {
        load_n<V>(t, gp + (size_t)k * gate.stride);
#pragma unroll
        for (int e = 0; e < V; ++e) g[e] += t[e];
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      x[e] = x[e] * inv * w[e];
      if (gate.p) x[e] *= (sigmoid ? 1.0f : g[e]) / (1.0f + expf(-g[e]));
    }
    store_n<V>(out + item * dv + d, x);
  }
}

// out[t, c] = silu(columns off .. + C of the sums), float32: four neighbouring numbers a thread
template <int V>
__global__ void silu_sums_kernel(const Sums x, int C, float* __restrict__ out, size_t total) {
  dep_launch();
  dep_wait();
  const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= total) return;
  const size_t tok = i / C;
  const size_t src = tok * x.width + x.off + (i - tok * C);
  if constexpr (V == 4) {
    float4 s = *reinterpret_cast<const float4*>(x.p + src);
    for (int k = 1; k < x.n; ++k) {
      const float4 t = *reinterpret_cast<const float4*>(x.p + (size_t)k * x.stride + src);
      s.x += t.x; s.y += t.y; s.z += t.z; s.w += t.w;
    }
    *reinterpret_cast<float4*>(out + i) = make_float4(silu_f(s.x), silu_f(s.y), silu_f(s.z), silu_f(s.w));
  } else {
    out[i] = silu_f(parts_sum(x.p, x.n, x.stride, src));
  }
}

int device_sms() {
  static int n = 0;
  if (n == 0) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
  }
  return n;
}

// Rotation of float32 sums for mixers whose recurrence reads rotated queries and keys: for every token and each of `heads` heads
// of dk numbers that lie side by side from column `off` of the sums, the pair (i, i + rot_dims / 2) of the head's first rot_dims
// numbers turns by the token's position (cos / sin tables [positions, rot_dims / 2]); heads from `scaled_from` on are then
// multiplied by `scale`. out [tokens, heads * dk] float32: nothing is rounded on the way.
__global__ void rotate_sums_kernel(Sums x, int heads, int dk, int rot_dims, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                   const int* __restrict__ positions, float* __restrict__ out, int n_tokens, int scaled_from, float scale) {
  dep_launch();
  dep_wait();
  // a thread a pair of the rotated part, or a single number behind it: dk - half items a head, every number read and written once
  const int half = rot_dims / 2, items = dk - half, per = heads * items;
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)n_tokens * per) return;
  const int tok = (int)(i / per), c = (int)(i - (size_t)tok * per), head = c / items, j = c - head * items;
  const float mul = head >= scaled_from ? scale : 1.0f;
  const size_t src = (size_t)tok * x.width + x.off + (size_t)head * dk, dst = ((size_t)tok * heads + head) * dk;
  if (j < half) {
    const float u = parts_sum(x.p, x.n, x.stride, src + j), v = parts_sum(x.p, x.n, x.stride, src + j + half);
    const float cs = cos_t[(size_t)positions[tok] * half + j], sn = sin_t[(size_t)positions[tok] * half + j];
    out[dst + j] = (u * cs - v * sn) * mul;
    out[dst + j + half] = (v * cs + u * sn) * mul;
  } else {
    out[dst + j + half] = parts_sum(x.p, x.n, x.stride, src + j + half) * mul;
  }
}

int lanes_for(int dk) {
  int r = 1;
  while (r * KPT < dk) r *= 2;
  return r;
}

}  // namespace

// Lanes a column of the state is spread over (the slot holds lanes * 16 rows a head); 0 if dk is beyond the kernel.
extern "C" int llm_linear_state_lanes(int dk) {
  if (dk <= 0 || dk > 32 * KPT) return 0;
  return lanes_for(dk);
}

extern "C" int llm_linear_state(int mode, const float* q, int qn, long long qs, int qw, int qo, const float* k, int kn, long long ks, int kw,
                                int ko, const float* v, int vn, long long vs, int vw, int vo, const float* b, int bn, long long bs, int bw,
                                int bo, const float* decay, int decay_width, int decay_off, const float* bonus, float* state, const int* seq_qoff, const int* seq_ntok,
                                const int* seq_slot, float* out, int n_tokens, int n_seqs, int H, int G, int dk, int dv, float q_scale,
                                float unit_eps, int decay_const, int silu, cudaStream_t stream) {
  // decay_const: `decay` is one row that holds for every token (decays that are constants of the model); silu: q, k and v are silu of
  // the sums (before the query's scale)
  if (n_seqs == 0) return LLM_OK;
  LLM_REQUIRE(mode >= 0 && mode <= 3, "linear_state: unknown update rule %d", mode);
  LLM_REQUIRE(!silu || mode == 0, "linear_state: activated sums go with the first rule");
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && dv > 0, "linear_state: bad sizes");
  LLM_REQUIRE(llm_linear_state_lanes(dk) > 0, "linear_state: a key size of %d is not in 1..%d", dk, 32 * KPT);
  LLM_REQUIRE(mode >= 2 || G == H, "linear_state: only the delta rules share query/key heads");
  LLM_REQUIRE(mode != 3 || (b && bn >= 1 && bo >= 0 && bo + H <= bw), "linear_state: the delta rule with a decay a channel needs beta");
  LLM_REQUIRE(q && k && v && decay && state && out && qn >= 1 && kn >= 1 && vn >= 1 && (mode != 1 || bonus), "linear_state: missing tensors");
  LLM_REQUIRE(qo + G * dk <= qw && ko + G * dk <= kw && vo + H * dv <= vw && decay_off + (mode == 2 ? 2 * H : H * dk) <= decay_width,
              "linear_state: columns outside their rows");
  LinearStateParams p;
  p.q = Sums{q, qn, (size_t)qs, qw, qo}; p.k = Sums{k, kn, (size_t)ks, kw, ko}; p.v = Sums{v, vn, (size_t)vs, vw, vo};
  p.b = Sums{b, bn, (size_t)bs, bw, bo};
  p.decay = decay; p.decay_width = decay_const ? 0 : decay_width; p.decay_off = decay_off; p.bonus = bonus; p.state = state;
  p.seq_qoff = seq_qoff; p.seq_ntok = seq_ntok; p.seq_slot = seq_slot; p.out = out;
  p.H = H; p.G = G; p.dk = dk; p.dv = dv; p.R = lanes_for(dk); p.q_scale = q_scale; p.unit_eps = unit_eps; p.silu = silu;
  const int dkp = p.R * KPT;
  const int a_stride = mode == 2 ? 2 : dkp;
  auto smem_for = [&](int tile) {  // as the kernel lays a buffer out
    const size_t a_floats = ((size_t)tile * a_stride + 3) & ~(size_t)3;
    return LS_BUFFERS * ((((size_t)tile * (2 * dkp + dv + (mode == 3 ? 1 : 0)) + a_floats + 3) & ~(size_t)3) * sizeof(float));
  };
  const bool few = n_tokens <= 2 * n_seqs;
  p.tile = few ? 2 : 16;
  // a portion's blocks have a multiprocessor each, so they may take more than the default 48 KB: longer tiles, fewer meetings
  const size_t smem_limit = few ? 48 * 1024 : LS_SMEM;
  while (p.tile > 1 && smem_for(p.tile) > smem_limit) p.tile /= 2;
  LLM_REQUIRE(smem_for(p.tile) <= smem_limit, "linear_state: heads of %d / %d numbers exceed one block's shared memory", dk, dv);
  p.one_part = qn == 1 && kn == 1 && vn == 1 && (mode != 3 || bn == 1);
  auto quads = [](const void* ptr, long long width, long long off) { return ((uintptr_t)ptr & 15) == 0 && width % 4 == 0 && off % 4 == 0; };
  p.vec4 = dk % 4 == 0 && dv % 4 == 0 && quads(q, qw, qo) && quads(k, kw, ko) && quads(v, vw, vo) && (mode == 2 || quads(decay, p.decay_width, decay_off));
  // the walk is bound by what a multiprocessor's shared memory delivers a token, so few blocks are cut into more, down to a warp of walkers
  p.walkers = LS_THREADS;
  const long long per_column_block = (long long)H * n_seqs;
  while (p.walkers > 32 && 2 * per_column_block * ceil_div(dv, p.walkers / p.R) <= device_sms()) p.walkers /= 2;
  dim3 grid(ceil_div(dv, p.walkers / p.R), H, n_seqs);
  const size_t smem = smem_for(p.tile);
#define LS_LAUNCH(M, RR)                                                                                                              \
  if (few) {                                                                                                                         \
    launch_kernel(linear_state_kernel<M, RR, true>, grid, p.walkers + LS_FETCHERS, smem, stream, p);                                 \
  } else {                                                                                                                           \
    LLM_REQUIRE(smem <= 48 * 1024 || cudaFuncSetAttribute(linear_state_kernel<M, RR, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                          (int)LS_SMEM) == cudaSuccess, "linear_state: cannot raise the shared memory limit"); \
    launch_kernel(linear_state_kernel<M, RR, false>, grid, p.walkers + LS_FETCHERS, smem, stream, p);                                \
  }
#define LS_LANES(M)                  \
  switch (p.R) {                     \
    case 1: LS_LAUNCH(M, 1); break;  \
    case 2: LS_LAUNCH(M, 2); break;  \
    case 4: LS_LAUNCH(M, 4); break;  \
    case 8: LS_LAUNCH(M, 8); break;  \
    case 16: LS_LAUNCH(M, 16); break; \
    default: LS_LAUNCH(M, 32); break; \
  }
  if (mode == 0) { LS_LANES(0) } else if (mode == 1) { LS_LANES(1) } else if (mode == 2) { LS_LANES(2) } else { LS_LANES(3) }
#undef LS_LANES
#undef LS_LAUNCH
  LLM_CHECK_LAUNCH("linear_state");
  return LLM_OK;
}

extern "C" int llm_token_shift(const void* x, const float* mu, int n_out, float* shift_state, const int* token_seq, const int* seq_qoff,
                               const int* seq_ntok, const int* seq_slot, void* out, int dtype, int n_tokens, int n_seqs, int D,
                               cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && D > 0 && n_out >= 1, "token_shift: bad sizes");
  LLM_REQUIRE(dtype == LLM_F32 || dtype == LLM_BF16, "token_shift: unknown dtype %d", dtype);
  dim3 grid(ceil_div(D, 256), n_tokens < 65535 ? n_tokens : 65535);
  const int sblocks = ceil_div((long long)n_seqs * D, 256);
  if (dtype == LLM_F32) {
    launch_kernel(token_shift_kernel<float>, grid, 256, 0, stream, (const float*)x, mu, n_out, (const float*)shift_state, token_seq, seq_qoff,
                  seq_slot, (float*)out, n_tokens, D);
    launch_kernel(token_shift_state_kernel<float>, sblocks, 256, 0, stream, (const float*)x, shift_state, seq_qoff, seq_ntok, seq_slot, n_seqs, D);
  } else {
    launch_kernel(token_shift_kernel<bf16>, grid, 256, 0, stream, (const bf16*)x, mu, n_out, (const float*)shift_state, token_seq, seq_qoff,
                  seq_slot, (bf16*)out, n_tokens, D);
    launch_kernel(token_shift_state_kernel<bf16>, sblocks, 256, 0, stream, (const bf16*)x, shift_state, seq_qoff, seq_ntok, seq_slot, n_seqs, D);
  }
  LLM_CHECK_LAUNCH("token_shift");
  return LLM_OK;
}

extern "C" int llm_delta_gates(const float* a, int an, long long as, int aw, int ao, const float* b, int bn, long long bs, int bw, int bo,
                               const float* a_log, const float* dt_bias, float* out, int n_tokens, int H, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && H > 0 && a && b && a_log && dt_bias && out && an >= 1 && bn >= 1, "delta_gates: bad arguments");
  LLM_REQUIRE(ao + H <= aw && bo + H <= bw, "delta_gates: columns outside their rows");
  launch_kernel(delta_gates_kernel, ceil_div((long long)n_tokens * H, 128), 128, 0, stream, Sums{a, an, (size_t)as, aw, ao},
                Sums{b, bn, (size_t)bs, bw, bo}, a_log, dt_bias, out, n_tokens, H);
  LLM_CHECK_LAUNCH("delta_gates");
  return LLM_OK;
}

// x: float32 sums; columns x0.. (R0 of them) and x1.. (R1). wt0 [R0, C0], wt1 [R1, C1]: the maps transposed, in the engine's dtype;
// w0, w1 (bfloat16 alone, or null): the maps as they are stored, for steps of more than 64 tokens on tensor cores.
extern "C" int llm_channel_gates(const float* x, int xn, long long xs, int xw, int x0, int x1, int R0, int R1, const void* wt0, const void* wt1,
                                 const void* w0, const void* w1, const float* bias0, const float* a_log, int C0, int C1, int per, float* out0, float* out1,
                                 int xb, int H, float* beta, int dtype, int n_tokens, cudaStream_t stream) {
  // beta [n_tokens, H] = sigmoid of columns xb .. + H
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && x && xn >= 1 && wt0 && wt1 && bias0 && a_log && out0 && out1, "channel_gates: missing tensors");
  LLM_REQUIRE(R0 > 0 && R1 > 0 && C0 > 0 && C1 > 0 && per > 0 && C0 % per == 0, "channel_gates: bad sizes");
  LLM_REQUIRE(x0 >= 0 && x1 >= 0 && x0 + R0 <= xw && x1 + R1 <= xw, "channel_gates: columns outside the product");
  LLM_REQUIRE(dtype == LLM_F32 || dtype == LLM_BF16, "channel_gates: unknown dtype %d", dtype);
  ChannelGates p;
  LLM_REQUIRE(beta && H > 0 && xb >= 0 && xb + H <= xw, "channel_gates: columns of the write strengths outside the product");
  p.x0 = Sums{x, xn, (size_t)xs, xw, x0}; p.x1 = Sums{x, xn, (size_t)xs, xw, x1}; p.xb = Sums{x, xn, (size_t)xs, xw, xb};
  p.H = H; p.beta = beta;
  p.R0 = R0; p.R1 = R1; p.C0 = C0; p.C1 = C1; p.per = per; p.bias0 = bias0; p.a_log = a_log; p.out0 = out0; p.out1 = out1; p.n_tokens = n_tokens;
  if (dtype == LLM_BF16 && w0 && w1 && n_tokens > 64 && xn == 1) {
    dim3 tiles(ceil_div(C0, CG_COLS) + ceil_div(C1, CG_COLS), ceil_div(n_tokens, CG_TOK));
    LLM_REQUIRE(tiles.y <= 65535, "channel_gates: too many tokens in one step (%d)", n_tokens);
    launch_kernel(channel_gates_mma_kernel, tiles, CG_THREADS, 0, stream, p, (const bf16*)w0, (const bf16*)w1);
    LLM_CHECK_LAUNCH("channel_gates");
    return LLM_OK;
  }
  const size_t smem = ((size_t)max(R0, R1) * 8 + 4 * 32 * 8) * sizeof(float);
  LLM_REQUIRE(smem <= 48 * 1024, "channel_gates: ranks of %d / %d exceed one block's shared memory", R0, R1);
  dim3 grid(ceil_div(C0, 32) + ceil_div(C1, 32), ceil_div(n_tokens, 8));
  LLM_REQUIRE(grid.y <= 65535, "channel_gates: too many tokens in one step (%d)", n_tokens);
  if (dtype == LLM_F32) launch_kernel(channel_gates_kernel<float>, grid, 128, smem, stream, p, (const float*)wt0, (const float*)wt1);
  else launch_kernel(channel_gates_kernel<bf16>, grid, 128, smem, stream, p, (const bf16*)wt0, (const bf16*)wt1);
  LLM_CHECK_LAUNCH("channel_gates");
  return LLM_OK;
}

extern "C" int llm_head_norm_gate(const float* o, const float* weight, int weight_per_head, const float* gate, int gn, long long gs, int gw,
                                  int go, float eps, void* out, int dtype, int n_tokens, int H, int dv, int sigmoid, cudaStream_t stream) {
  // sigmoid 1: the gate is sigmoid(sums) instead of silu(sums)
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && H > 0 && dv > 0 && o && weight && out, "head_norm_gate: bad arguments");
  LLM_REQUIRE(gate == nullptr || (gn >= 1 && go >= 0 && go + H * dv <= gw), "head_norm_gate: gate columns outside the product");
  const Sums g{gate, gn, (size_t)gs, gw, go};
  LLM_REQUIRE(dtype == LLM_F32 || dtype == LLM_BF16, "head_norm_gate: unknown dtype %d", dtype);
  if (dv > WIDE_NORM_FROM) {  // a block a row; the threads' number depends on the row's size alone, and with it the order of the sum
    const int threads = min(1024, ceil_div(dv, 128) * 32);
    const long long rows = (long long)n_tokens * H;
    LLM_REQUIRE(rows <= 0x7fffffffLL, "head_norm_gate: too many rows");
    auto quads = [](const void* q) { return ((uintptr_t)q & 15u) == 0; };
    const bool vec = dv % 4 == 0 && gw % 4 == 0 && go % 4 == 0 && gs % 4 == 0 && quads(o) && quads(weight) && quads(gate) && quads(out);
#define LLM_WIDE_NORM(T, V) \
  launch_kernel(wide_norm_gate_kernel<T, V>, (int)rows, threads, 0, stream, o, weight, weight_per_head, g, eps, (T*)out, H, dv, sigmoid)
    if (dtype == LLM_F32 && vec) LLM_WIDE_NORM(float, 4);
    else if (dtype == LLM_F32) LLM_WIDE_NORM(float, 1);
    else if (vec) LLM_WIDE_NORM(bf16, 4);
    else LLM_WIDE_NORM(bf16, 1);
#undef LLM_WIDE_NORM
    LLM_CHECK_LAUNCH("head_norm_gate");
    return LLM_OK;
  }
  const int blocks = ceil_div((long long)n_tokens * H, 4);
  if (dtype == LLM_F32)
    launch_kernel(head_norm_gate_kernel<float>, blocks, 128, 0, stream, o, weight, weight_per_head, g, eps, (float*)out, n_tokens, H, dv, sigmoid);
  else
    launch_kernel(head_norm_gate_kernel<bf16>, blocks, 128, 0, stream, o, weight, weight_per_head, g, eps, (bf16*)out, n_tokens, H, dv, sigmoid);
  LLM_CHECK_LAUNCH("head_norm_gate");
  return LLM_OK;
}

extern "C" int llm_silu_sums(const float* x, int xn, long long xs, int xw, int xo, int C, float* out, int n_tokens, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && C > 0 && x && out && xn >= 1 && xo >= 0 && (long long)xo + C <= xw, "silu_sums: bad arguments");
  const Sums s{x, xn, (size_t)xs, xw, xo};
  const long long total = (long long)n_tokens * C;
  if (C % 4 == 0 && xw % 4 == 0 && xo % 4 == 0 && xs % 4 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15u) == 0)
    launch_kernel(silu_sums_kernel<4>, ceil_div(total / 4, 256), 256, 0, stream, s, C, out, (size_t)total);
  else
    launch_kernel(silu_sums_kernel<1>, ceil_div(total, 256), 256, 0, stream, s, C, out, (size_t)total);
  LLM_CHECK_LAUNCH("silu_sums");
  return LLM_OK;
}

extern "C" int llm_rotate_sums(const float* x, int xn, long long xs, int xw, int xo, int heads, int dk, int rot_dims, const float* cos_t,
                               const float* sin_t, const int* positions, float* out, int n_tokens, int scaled_from, float scale,
                               cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && heads > 0 && dk > 0 && x && out && xn >= 1 && xo >= 0 && (long long)xo + (long long)heads * dk <= xw, "rotate_sums: bad arguments");
  LLM_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dk && (rot_dims == 0 || (cos_t && sin_t && positions)), "rotate_sums: %d rotated numbers in a head of %d", rot_dims, dk);
  launch_kernel(rotate_sums_kernel, ceil_div((long long)n_tokens * heads * (dk - rot_dims / 2), 256), 256, 0, stream, Sums{x, xn, (size_t)xs, xw, xo}, heads, dk,
                rot_dims, cos_t, sin_t, positions, out, n_tokens, scaled_from, scale);
  LLM_CHECK_LAUNCH("rotate_sums");
  return LLM_OK;
}
