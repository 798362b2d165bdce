// Tensor-core softmax attention (bf16) for score shapes that the kernels of softmax_attention.cuh do not have (its head comment
// defines them): two score maps per head over the same values, scores over the key heads' channels side by side (the mixed queries
// of a talking attention), value heads of another size than the keys, and head sizes that are any multiple of 8.
//
// A UNIT is one softmax: a (query head, map) pair.  The units of one value head ("its units") share that head's value rows; their
// key rows are, per map, one slice of `dim` channels (wide: all units read the same rows).
//
//   multi_attention_prefill_kernel<DV16, KT>   rows in portions.  CTA of eight warps = `rt` query tiles (16 rows each, consecutive
//                        entries of the host's table) x `uw` units of a value head: a warp owns one (tile, unit) pair, S = Q K^T and
//                        O += P V on mma.sync m16n8k16 with fp32 accumulators, running maximum and sum in fp32 registers.  Tiles
//                        that continue one another share the staged keys and values (cp.async double buffer through the page map);
//                        tiles of different sequences are walked one after the other.  With two maps a head's units sit in
//                        neighbouring warps and their difference is taken (and normed) in the epilogue.
//   multi_attention_decode_kernel<SPW, DV16>   steps of single tokens: CTA = (row, units, key split), the products TRANSPOSED
//                        (S^T = K Q^T, O^T = V^T P^T), so the MMA's 16-row side carries keys / value columns and its 8-column side
//                        up to eight query heads.  A SET is up to eight heads that share a key slice and a value head: the two maps
//                        of a head group, or (wide) the head groups of several value heads.  Four warps = `4 / sg` slices of 16
//                        keys x `sg` groups of SPW sets; partial results meet in shared memory.
//
// Channels are padded to a multiple of 16 with zeros in shared memory.
#pragma once

#include "softmax_attention.cuh"

namespace mtx {

constexpr int kMatThreads = 256, kMatWarps = 8;

struct MultiMmaPlan {
  bool ok = false;
  int kt = 0, dv16 = 0, uw = 0, rt = 0, chunks = 0;
  size_t smem = 0;
};

inline int mat_pad16(int n) { return (n + 15) / 16 * 16; }

// bytes of the staged queries and of one key / value stage
inline size_t mat_query_bytes(int dim) { return size_t(kMatWarps) * 16 * (mat_pad16(dim) + 8) * sizeof(bf16); }
inline size_t mat_stage_bytes(int dim, int vdim, int maps, bool wide, bool same_kv, int kt) {
  return size_t(kt) * ((wide ? 1 : maps) * mat_pad16(dim) + 8 + (same_kv ? 0 : mat_pad16(vdim) + 8)) * sizeof(bf16);
}

// n_tiles: query tiles of the step, num_sms: fewer tiles per CTA when the grid would not cover the GPU
inline MultiMmaPlan multi_mma_plan(int heads, int kv_heads, int dim, int vdim, int maps, bool wide, bool same_kv, int n_tiles, int num_sms) {
  MultiMmaPlan p;
  if (dim % 8 != 0 || vdim % 8 != 0 || vdim > 256 || (same_kv && vdim > dim)) return p;
  const int d16 = mat_pad16(vdim) / 16, units = heads / kv_heads * maps;
  p.dv16 = d16 <= 4 ? 4 : (d16 <= 8 ? 8 : 16);
  p.uw = units < kMatWarps ? units : kMatWarps;
  if (maps == 2 && (p.uw & 1)) --p.uw;
  p.chunks = (units + p.uw - 1) / p.uw;
  p.rt = kMatWarps / p.uw;
  while (p.rt > 1 && (long long)((n_tiles + p.rt - 1) / p.rt) * kv_heads * p.chunks < num_sms) p.rt /= 2;
  // 64-key tiles when two CTAs then still share an SM, else 32
  for (int kt = p.dv16 <= 4 ? 64 : 32; kt >= 32; kt /= 2) {
    p.smem = mat_query_bytes(dim) + 2 * mat_stage_bytes(dim, vdim, maps, wide, same_kv, kt);
    if (maps == 2) {  // (the epilogue's exchange of the second maps' results)
      const size_t xch = size_t(kMatWarps / 2) * 16 * mat_pad16(vdim) * sizeof(float);
      if (xch > p.smem) p.smem = xch;
    }
    p.kt = kt;
    if (p.smem <= (kt == 64 ? 112 : 226) * size_t(1024)) {
      p.ok = true;
      break;
    }
  }
  return p;
}

__device__ __forceinline__ void mat_ldsm_x4(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mat_ldsm_x4_trans(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}

template <int DV16, int KT>
__global__ void __launch_bounds__(kMatThreads, DV16 <= 8 ? 2 : 1) multi_attention_prefill_kernel(const SoftmaxAttnArgs<bf16> a, int n_tiles, int uw, int rt, int chunks) {
  extern __shared__ __align__(16) unsigned char mat_raw[];
  constexpr int NB = 2 * DV16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int maps = a.maps > 1 ? a.maps : 1, rep_units = a.heads / a.kv_heads * maps, units = a.heads * maps;
  const bool same_kv = a.k_pages == a.v_pages;
  const int d = a.dim, dv = a.vdim, dp = (d + 15) & ~15, dvp = (dv + 15) & ~15, n_slices = a.wide ? 1 : maps;
  const int QP = dp + 8, KP = n_slices * dp + 8, VP = same_kv ? KP : dvp + 8, stage_elems = KT * (KP + (same_kv ? 0 : VP));
  bf16* const sQ = reinterpret_cast<bf16*>(mat_raw);  // [8 warps][16][QP]
  bf16* const stage0 = sQ + kMatWarps * 16 * QP;      // stage s: K [KT][KP], then V [KT][VP]
  if (dp != d || dvp != dv) {  // the padding channels are zero and stay so
    const int words = (kMatWarps * 16 * QP + 2 * stage_elems) / 2;
    for (int e = tid; e < words; e += kMatThreads) reinterpret_cast<uint32_t*>(mat_raw)[e] = 0u;
    __syncthreads();
  }
  griddep_wait();
  const int vh = blockIdx.y / chunks, unit0 = (blockIdx.y % chunks) * uw;
  const int tile0 = blockIdx.x * rt, my_tile = tile0 + warp / uw, my_unit = unit0 + warp % uw;
  const bool active = warp < uw * rt && my_tile < n_tiles && my_unit < rep_units;
  const int u_all = vh * rep_units + (active ? my_unit : 0), h = u_all / maps;  // unit and query head in the whole layer
  const int r0 = active ? a.tile_row0[my_tile] : 0, nr = active ? a.tile_row0[my_tile + 1] - r0 : 0;
  const int p0 = active ? a.pos[r0] : 0, p_last = p0 + nr - 1;

  // this warp's queries, rows beyond the tile zero
  bf16* const myQ = sQ + warp * 16 * QP;
  for (int r = 0; r < 16; ++r)
    for (int c = lane * 8; c < d; c += 256) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < nr) v = *reinterpret_cast<const uint4*>(a.q + (size_t(r0 + r) * units + u_all) * d + c);
      *reinterpret_cast<uint4*>(myQ + r * QP + c) = v;
    }
  __syncwarp();

  float o[NB][4];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nb][e] = 0.0f;
  constexpr float kLog2e = 1.4426950408889634f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};  // (maxima in units of log 2)
  if (a.sink) {
    m_run[0] = m_run[1] = a.sink[h] * kLog2e;
    l_run[0] = l_run[1] = t == 0 ? 1.0f : 0.0f;
  }
  const float mul = a.scale * kLog2e;
  const int pi0 = p0 + g, pi1 = p0 + g + 8;
  const int lo0 = smax_first(pi0, a.window, a.chunk), lo1 = smax_first(pi1, a.window, a.chunk);
  const int lo_first = smax_first(p0, a.window, a.chunk), lo_last = smax_first(p_last > 0 ? p_last : 0, a.window, a.chunk);

  const int tpp = a.tokens_per_page, page_shift = (tpp & (tpp - 1)) == 0 ? __ffs(tpp) - 1 : -1;
  const size_t pool_rows = size_t(a.num_pages) * tpp;
  const bf16* const kbase = a.k_pages + (a.wide ? 0 : size_t(vh) * maps * pool_rows * d);
  const bf16* const vbase = a.v_pages + size_t(vh) * pool_rows * dv;
  const int ld_row = tid >> 3, ld_sub = tid & 7;  // eight threads per key row
  const int map_of_warp = (u_all % maps) * (a.wide ? 0 : dp);

  // groups of tiles [ta, tb) that continue one another: they share their keys
  for (int ta = tile0, tb; ta < tile0 + rt && ta < n_tiles; ta = tb) {
    const int ra = a.tile_row0[ta], grp = a.group[ra], pa = a.pos[ra];
    int rb = a.tile_row0[ta + 1];
    for (tb = ta + 1; tb < tile0 + rt && tb < n_tiles; ++tb) {
      if (a.group[rb] != grp || a.pos[rb] != pa + (rb - ra)) break;
      rb = a.tile_row0[tb + 1];
    }
    const int lo = smax_first(pa, a.window, a.chunk), last = pa + (rb - ra) - 1, n_key_tiles = (last - lo) / KT + 1;
    const int* pages = a.page_map + size_t(grp) * a.max_pages;
    const bool mine = active && my_tile >= ta && my_tile < tb;
    auto load_tile = [&](int it, int stage) {
      bf16* sk = stage0 + size_t(stage) * stage_elems;
#pragma unroll
      for (int q = 0; q < KT / 32; ++q) {
        const int jj = ld_row + q * 32, j = lo + it * KT + jj;
        const bool ok = j <= last;
        const int pg = page_shift >= 0 ? (j >> page_shift) : j / tpp;
        const size_t row = ok ? size_t(pages[pg]) * tpp + (j - pg * tpp) : 0;
        for (int m = 0; m < n_slices; ++m) {
          const bf16* src = kbase + (m * pool_rows + row) * d;
          bf16* dst = sk + jj * KP + m * dp;
          for (int c = ld_sub * 8; c < d; c += 64) cp_async_16(dst + c, src + c, ok);
        }
        if (!same_kv) {
          const bf16* src = vbase + row * dv;
          bf16* dst = sk + KT * KP + jj * VP;
          for (int c = ld_sub * 8; c < dv; c += 64) cp_async_16(dst + c, src + c, ok);
        }
      }
      cp_async_commit();
    };
    load_tile(0, 0);
    for (int it = 0; it < n_key_tiles; ++it) {
      if (it + 1 < n_key_tiles) {
        load_tile(it + 1, (it + 1) & 1);
        cp_async_wait_pending(1);
      } else {
        cp_async_wait_pending(0);
      }
      __syncthreads();
      const int j0 = lo + it * KT;
      if (mine && j0 <= p_last && j0 + KT > lo_first) {
        const bf16* sk = stage0 + size_t(it & 1) * stage_elems;
        const bf16* sv = same_kv ? sk : sk + KT * KP;
        float s[KT / 8][4];
#pragma unroll
        for (int nb = 0; nb < KT / 8; ++nb)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[nb][e] = 0.0f;
        const bf16* qa = myQ + (lane & 15) * QP + (lane >> 4) * 8;
        const bf16* kb = sk + ((lane & 7) + (lane >> 4) * 8) * KP + map_of_warp + ((lane >> 3) & 1) * 8;
#pragma unroll 2
        for (int k0 = 0; k0 < dp; k0 += 16) {
          uint32_t qf[4];
          mat_ldsm_x4(qf, qa + k0);
#pragma unroll
          for (int nb = 0; nb < KT / 8; nb += 2) {
            uint32_t kf[4];
            mat_ldsm_x4(kf, kb + nb * 8 * KP + k0);
            mma_bf16_16816(s[nb], qf, kf[0], kf[1]);
            mma_bf16_16816(s[nb + 1], qf, kf[2], kf[3]);
          }
        }
        const bool every_key_seen = j0 + KT - 1 <= p0 && j0 >= lo_last;
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int nb = 0; nb < KT / 8; ++nb) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float sc = s[nb][e] * mul;
            if (!every_key_seen) {
              const int j = j0 + nb * 8 + 2 * t + (e & 1);
              if (j > ((e & 2) ? pi1 : pi0) || j < ((e & 2) ? lo1 : lo0)) sc = -INFINITY;
            }
            s[nb][e] = sc;
          }
          mx0 = fmaxf(mx0, fmaxf(s[nb][0], s[nb][1]));
          mx1 = fmaxf(mx1, fmaxf(s[nb][2], s[nb][3]));
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);
        const float base0 = mn0 == -INFINITY ? 0.0f : mn0, base1 = mn1 == -INFINITY ? 0.0f : mn1;
        const float fix0 = smax_ex2(m_run[0] - base0), fix1 = smax_ex2(m_run[1] - base1);
        m_run[0] = mn0;
        m_run[1] = mn1;
        float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
        for (int nb = 0; nb < KT / 8; ++nb) {
          s[nb][0] = smax_ex2(s[nb][0] - base0);
          s[nb][1] = smax_ex2(s[nb][1] - base0);
          s[nb][2] = smax_ex2(s[nb][2] - base1);
          s[nb][3] = smax_ex2(s[nb][3] - base1);
          sum0 += s[nb][0] + s[nb][1];
          sum1 += s[nb][2] + s[nb][3];
        }
        l_run[0] = l_run[0] * fix0 + sum0;  // (per-thread partial sums; the four lanes of a row are added at the end)
        l_run[1] = l_run[1] * fix1 + sum1;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
          o[nb][0] *= fix0;
          o[nb][1] *= fix0;
          o[nb][2] *= fix1;
          o[nb][3] *= fix1;
        }
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
          uint32_t pf[4];
          pf[0] = smax_pack_bf16(s[2 * kk][0], s[2 * kk][1]);
          pf[1] = smax_pack_bf16(s[2 * kk][2], s[2 * kk][3]);
          pf[2] = smax_pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
          pf[3] = smax_pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
          const bf16* vrow = sv + (kk * 16 + (lane & 15)) * VP + (lane >> 4) * 8;
#pragma unroll
          for (int nb = 0; nb < NB; nb += 2) {
            if (nb * 8 < dvp) {
              uint32_t vf[4];
              mat_ldsm_x4_trans(vf, vrow + nb * 8);
              mma_bf16_16816(o[nb], pf, vf[0], vf[1]);
              mma_bf16_16816(o[nb + 1], pf, vf[2], vf[3]);
            }
          }
        }
      }
      __syncthreads();  // the stage is free for the load after next
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
  }
  if (maps == 2) {
    // warp 2 n + 1 holds the second map of warp 2 n's head and rows: its normalised result goes through shared memory
    float* xch = reinterpret_cast<float*>(mat_raw) + (warp >> 1) * 16 * dvp;
    const float i0 = 1.0f / l_run[0], i1 = 1.0f / l_run[1];
    if ((warp & 1) && active) {
#pragma unroll
      for (int nb = 0; nb < NB; ++nb)
        if (nb * 8 < dvp) {
          *reinterpret_cast<float2*>(xch + g * dvp + nb * 8 + 2 * t) = make_float2(o[nb][0] * i0, o[nb][1] * i0);
          *reinterpret_cast<float2*>(xch + (g + 8) * dvp + nb * 8 + 2 * t) = make_float2(o[nb][2] * i1, o[nb][3] * i1);
        }
    }
    __syncthreads();
    if ((warp & 1) || !active) return;
    float ss0 = 0.0f, ss1 = 0.0f;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
      if (nb * 8 < dvp) {
        const float2 b0 = *reinterpret_cast<const float2*>(xch + g * dvp + nb * 8 + 2 * t), b1 = *reinterpret_cast<const float2*>(xch + (g + 8) * dvp + nb * 8 + 2 * t);
        o[nb][0] = fmaf(-a.diff_lambda, b0.x, o[nb][0] * i0);
        o[nb][1] = fmaf(-a.diff_lambda, b0.y, o[nb][1] * i0);
        o[nb][2] = fmaf(-a.diff_lambda, b1.x, o[nb][2] * i1);
        o[nb][3] = fmaf(-a.diff_lambda, b1.y, o[nb][3] * i1);
        ss0 += o[nb][0] * o[nb][0] + o[nb][1] * o[nb][1];  // (padding columns are zero)
        ss1 += o[nb][2] * o[nb][2] + o[nb][3] * o[nb][3];
      }
    ss0 += __shfl_xor_sync(0xffffffffu, ss0, 1);
    ss0 += __shfl_xor_sync(0xffffffffu, ss0, 2);
    ss1 += __shfl_xor_sync(0xffffffffu, ss1, 1);
    ss1 += __shfl_xor_sync(0xffffffffu, ss1, 2);
    const float f0 = a.diff_scale / sqrtf(ss0 / float(dv) + a.eps), f1 = a.diff_scale / sqrtf(ss1 / float(dv) + a.eps);
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int col = nb * 8 + 2 * t;
      if (col < dv) {  // (dv is even)
        bf16* out0 = a.out + size_t(r0 + g) * a.ld_out + h * dv + col;
        if (g < nr) *reinterpret_cast<uint32_t*>(out0) = smax_pack_bf16(o[nb][0] * f0, o[nb][1] * f0);
        if (g + 8 < nr) *reinterpret_cast<uint32_t*>(out0 + size_t(8) * a.ld_out) = smax_pack_bf16(o[nb][2] * f1, o[nb][3] * f1);
      }
    }
    return;
  }
  if (!active) return;
  const float f0 = a.out_scale / l_run[0] * (g < nr ? smax_gate(a.gate, a.ld_gate, r0 + g, h) : 1.0f);
  const float f1 = a.out_scale / l_run[1] * (g + 8 < nr ? smax_gate(a.gate, a.ld_gate, r0 + g + 8, h) : 1.0f);
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int col = nb * 8 + 2 * t;
    if (col < dv) {
      bf16* out0 = a.out + size_t(r0 + g) * a.ld_out + h * dv + col;
      if (g < nr) *reinterpret_cast<uint32_t*>(out0) = smax_pack_bf16(o[nb][0] * f0, o[nb][1] * f0);
      if (g + 8 < nr) *reinterpret_cast<uint32_t*>(out0 + size_t(8) * a.ld_out) = smax_pack_bf16(o[nb][2] * f1, o[nb][3] * f1);
    }
  }
}

// ---- steps of single tokens ---------------------------------------------------------------------------------------------------------

struct MultiDecodePlan {
  bool ok = false;
  int spw = 0, dv16 = 0, sg = 0, sets = 0;  // sets: of one CTA
  int groups = 0, chunks = 0;               // CTAs per (row, split): groups of value heads x chunks of eight heads
  size_t smem = 0;
};

inline size_t multi_decode_smem_bytes(int dim, int vdim, int sets, int slices, int vparts, bool same_kv, int kt) {
  const int dp = mat_pad16(dim), dvp = mat_pad16(vdim);
  const size_t q = size_t(sets) * 8 * (dp + 8) * sizeof(bf16);
  const size_t ring = size_t(2) * kt * (slices * dp + 8 + (same_kv ? 0 : vparts * dvp + 8)) * sizeof(bf16);
  const size_t merge = sizeof(float) * size_t(sets) * (kt / 16) * (8 * size_t(dvp) + 16);
  return q + (ring > merge ? ring : merge);
}

inline MultiDecodePlan multi_decode_plan(int heads, int kv_heads, int dim, int vdim, int maps, bool wide, bool same_kv) {
  MultiDecodePlan p;
  if (dim % 8 != 0 || vdim % 8 != 0 || vdim > 256 || (same_kv && vdim > dim)) return p;
  const int d16 = mat_pad16(vdim) / 16;
  p.dv16 = d16 <= 4 ? 4 : (d16 <= 8 ? 8 : 16);
  p.chunks = (heads / kv_heads + 7) / 8;
  // wide: up to four value heads per CTA, so that the key rows they share are staged once
  for (int want = wide ? (kv_heads >= 3 ? 4 : kv_heads) : maps; want >= 1; want /= 2) {
    p.sets = want;
    p.sg = want == 4 ? 2 : 1;
    p.spw = p.sets / p.sg;
    p.groups = wide ? (kv_heads + p.sets - 1) / p.sets : kv_heads;
    p.smem = multi_decode_smem_bytes(dim, vdim, p.sets, wide ? 1 : maps, wide ? p.sets : 1, same_kv, 64 / p.sg);
    if (p.smem <= 226 * size_t(1024)) {
      p.ok = true;
      break;
    }
    if (!wide) break;
  }
  return p;
}

template <int SPW, int DV16>
__global__ void __launch_bounds__(128) multi_attention_decode_kernel(const SoftmaxAttnArgs<bf16> a, int sets, int sg, int chunks) {
  extern __shared__ __align__(16) unsigned char mat_raw[];
  constexpr int NT = 128;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int maps = a.maps > 1 ? a.maps : 1, rep_all = a.heads / a.kv_heads, units = a.heads * maps;
  const bool same_kv = a.k_pages == a.v_pages;
  const int d = a.dim, dv = a.vdim, dp = (d + 15) & ~15, dvp = (dv + 15) & ~15;
  const int ks_n = 4 / sg, KT = 16 * ks_n, n_slices = a.wide ? 1 : maps, n_vals = a.wide ? sets : 1;
  const int QP = dp + 8, KP = n_slices * dp + 8, VP = same_kv ? KP : n_vals * dvp + 8, stage_elems = KT * (KP + (same_kv ? 0 : VP));
  bf16* const sQ = reinterpret_cast<bf16*>(mat_raw);  // [sets][8][QP]
  bf16* const stage0 = sQ + sets * 8 * QP;
  if (dp != d || dvp != dv) {
    const int words = (sets * 8 * QP + 2 * stage_elems) / 2;
    for (int e = tid; e < words; e += NT) reinterpret_cast<uint32_t*>(mat_raw)[e] = 0u;
    __syncthreads();
  }
  griddep_wait();
  const int row = blockIdx.x, vgroup = blockIdx.y / chunks, chunk = blockIdx.y % chunks;
  const int rep = rep_all - chunk * 8 < 8 ? rep_all - chunk * 8 : 8;
  const int pos = a.pos[row], grp = a.group[row], lo = smax_first(pos, a.window, a.chunk);
  const int* pages = a.page_map + size_t(grp) * a.max_pages;
  const int tpp = a.tokens_per_page, page_shift = (tpp & (tpp - 1)) == 0 ? __ffs(tpp) - 1 : -1;
  const size_t pool_rows = size_t(a.num_pages) * tpp;
  const int vh0 = a.wide ? vgroup * sets : vgroup;  // first value head of the CTA
  const bf16* const kbase = a.k_pages + (a.wide ? 0 : size_t(vgroup) * maps * pool_rows * d);
  const bf16* const vbase = a.v_pages + size_t(vh0) * pool_rows * dv;
  const int all_key_tiles = (pos - lo) / KT + 1, per = (all_key_tiles + a.splits - 1) / a.splits, tile_lo = int(blockIdx.z) * per;
  int n_key_tiles = all_key_tiles - tile_lo < per ? all_key_tiles - tile_lo : per;
  if (n_key_tiles < 0) n_key_tiles = 0;
  // unit of head slot hh of set s: -1 when there is none
  auto unit_of = [&](int s, int hh) -> int {
    if (hh >= rep) return -1;
    if (a.wide) return vh0 + s < a.kv_heads ? (vh0 + s) * rep_all + chunk * 8 + hh : -1;
    return (vgroup * rep_all + chunk * 8 + hh) * maps + s;
  };
  const int ld_row = tid >> 3, ld_sub = tid & 7;
  auto load_tile = [&](int it, int stage) {
    bf16* sk = stage0 + size_t(stage) * stage_elems;
    for (int jj = ld_row; jj < KT; jj += 16) {
      const int j = lo + (tile_lo + it) * KT + jj;
      const bool ok = j <= pos;
      const int pg = page_shift >= 0 ? (j >> page_shift) : j / tpp;
      const size_t r = ok ? size_t(pages[pg]) * tpp + (j - pg * tpp) : 0;
      for (int m = 0; m < n_slices; ++m) {
        const bf16* src = kbase + (m * pool_rows + r) * d;
        bf16* dst = sk + jj * KP + m * dp;
        for (int c = ld_sub * 8; c < d; c += 64) cp_async_16(dst + c, src + c, ok);
      }
      if (!same_kv)
        for (int v = 0; v < n_vals; ++v) {
          const bool okv = ok && vh0 + v < a.kv_heads;
          const bf16* src = vbase + (okv ? v * pool_rows + r : 0) * dv;
          bf16* dst = sk + KT * KP + jj * VP + v * dvp;
          for (int c = ld_sub * 8; c < dv; c += 64) cp_async_16(dst + c, src + c, okv);
        }
    }
    cp_async_commit();
  };
  if (n_key_tiles > 0) load_tile(0, 0);
  for (int s = 0; s < sets; ++s)
    for (int hh = warp; hh < 8; hh += 4) {
      const int u = unit_of(s, hh);
      for (int c = lane * 8; c < d; c += 256) {
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (u >= 0) v = *reinterpret_cast<const uint4*>(a.q + (size_t(row) * units + u) * d + c);
        *reinterpret_cast<uint4*>(sQ + (s * 8 + hh) * QP + c) = v;
      }
    }
  const int ks = warp % ks_n, set0 = warp / ks_n * SPW;
  float o[SPW][DV16][4];  // O^T: (column mb * 16 + g / g + 8, head 2t / 2t + 1)
  float m_run[SPW][2], l_run[SPW][2];
  constexpr float kLog2e = 1.4426950408889634f;
#pragma unroll
  for (int s = 0; s < SPW; ++s) {
#pragma unroll
    for (int mb = 0; mb < DV16; ++mb)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[s][mb][e] = 0.0f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      m_run[s][e] = -INFINITY;
      l_run[s][e] = 0.0f;
      const int u = unit_of(set0 + s, 2 * t + e);
      if (a.sink && ks == 0 && blockIdx.z == 0 && u >= 0) {  // (the first key slice of the first split carries the sink)
        m_run[s][e] = a.sink[u / maps] * kLog2e;
        l_run[s][e] = g == 0 ? 1.0f : 0.0f;
      }
    }
  }
  const float mul = a.scale * kLog2e;
  for (int it = 0; it < n_key_tiles; ++it) {
    if (it + 1 < n_key_tiles) {
      load_tile(it + 1, (it + 1) & 1);
      cp_async_wait_pending(1);
    } else {
      cp_async_wait_pending(0);
    }
    __syncthreads();
    const bf16* sk = stage0 + size_t(it & 1) * stage_elems;
    const bf16* sv = same_kv ? sk : sk + KT * KP;
    const int j0 = lo + (tile_lo + it) * KT + ks * 16;  // this warp's 16 keys
    if (j0 <= pos) {
      float c[SPW][4];
#pragma unroll
      for (int s = 0; s < SPW; ++s)
#pragma unroll
        for (int e = 0; e < 4; ++e) c[s][e] = 0.0f;
      const bf16* kb = sk + (ks * 16 + (lane & 15)) * KP + (lane >> 4) * 8;
      const bf16* qb = sQ + (set0 * 8 + g) * QP + 2 * t;
      if (a.wide) {
#pragma unroll 4
        for (int k0 = 0; k0 < dp; k0 += 16) {
          uint32_t af[4];
          mat_ldsm_x4(af, kb + k0);
#pragma unroll
          for (int s = 0; s < SPW; ++s)
            mma_bf16_16816(c[s], af, *reinterpret_cast<const uint32_t*>(qb + s * 8 * QP + k0), *reinterpret_cast<const uint32_t*>(qb + s * 8 * QP + k0 + 8));
        }
      } else {
#pragma unroll 2
        for (int k0 = 0; k0 < dp; k0 += 16) {
#pragma unroll
          for (int s = 0; s < SPW; ++s) {
            uint32_t af[4];
            mat_ldsm_x4(af, kb + (set0 + s) * dp + k0);
            mma_bf16_16816(c[s], af, *reinterpret_cast<const uint32_t*>(qb + s * 8 * QP + k0), *reinterpret_cast<const uint32_t*>(qb + s * 8 * QP + k0 + 8));
          }
        }
      }
      const bool sa = j0 + g <= pos, sb = j0 + g + 8 <= pos;  // (no tile starts before the first visible key)
#pragma unroll
      for (int s = 0; s < SPW; ++s) {
        c[s][0] = sa ? c[s][0] * mul : -INFINITY;
        c[s][1] = sa ? c[s][1] * mul : -INFINITY;
        c[s][2] = sb ? c[s][2] * mul : -INFINITY;
        c[s][3] = sb ? c[s][3] * mul : -INFINITY;
        float mx0 = fmaxf(c[s][0], c[s][2]), mx1 = fmaxf(c[s][1], c[s][3]);
#pragma unroll
        for (int sh = 4; sh < 32; sh <<= 1) {
          mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, sh));
          mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, sh));
        }
        const float mn0 = fmaxf(m_run[s][0], mx0), mn1 = fmaxf(m_run[s][1], mx1);  // (finite: the warp's first key is visible)
        const float fix0 = smax_ex2(m_run[s][0] - mn0), fix1 = smax_ex2(m_run[s][1] - mn1);
        m_run[s][0] = mn0;
        m_run[s][1] = mn1;
        c[s][0] = smax_ex2(c[s][0] - mn0);
        c[s][1] = smax_ex2(c[s][1] - mn1);
        c[s][2] = smax_ex2(c[s][2] - mn0);
        c[s][3] = smax_ex2(c[s][3] - mn1);
        l_run[s][0] = l_run[s][0] * fix0 + c[s][0] + c[s][2];  // (this lane's keys; the eight lanes of a head are added at the end)
        l_run[s][1] = l_run[s][1] * fix1 + c[s][1] + c[s][3];
#pragma unroll
        for (int mb = 0; mb < DV16; ++mb) {
          o[s][mb][0] *= fix0;
          o[s][mb][1] *= fix1;
          o[s][mb][2] *= fix0;
          o[s][mb][3] *= fix1;
        }
      }
      uint32_t pb[SPW][2];
#pragma unroll
      for (int s = 0; s < SPW; ++s) {
        pb[s][0] = smax_movmatrix_trans(smax_pack_bf16(c[s][0], c[s][1]));
        pb[s][1] = smax_movmatrix_trans(smax_pack_bf16(c[s][2], c[s][3]));
      }
      const bf16* v0 = sv + (ks * 16 + (lane & 7) + 8 * (lane >> 4)) * VP + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int mb = 0; mb < DV16; ++mb) {
        if (mb * 16 < dvp) {
          uint32_t vf[4];
          if (!a.wide) mat_ldsm_x4_trans(vf, v0 + mb * 16);
#pragma unroll
          for (int s = 0; s < SPW; ++s) {
            if (a.wide) mat_ldsm_x4_trans(vf, v0 + (set0 + s) * dvp + mb * 16);
            mma_bf16_16816(o[s][mb], vf, pb[s][0], pb[s][1]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int s = 0; s < SPW; ++s)
#pragma unroll
    for (int sh = 4; sh < 32; sh <<= 1) {
      l_run[s][0] += __shfl_xor_sync(0xffffffffu, l_run[s][0], sh);
      l_run[s][1] += __shfl_xor_sync(0xffffffffu, l_run[s][1], sh);
    }
  // merge of the key slices (the ring is free: the loop ended with a barrier)
  float* mo = reinterpret_cast<float*>(stage0);  // [set][key slice][8 heads][dvp]
  float* mm = mo + sets * ks_n * 8 * dvp;        // [set][key slice][8] maxima, then the sums
  float* ml = mm + sets * ks_n * 8;
#pragma unroll
  for (int s = 0; s < SPW; ++s) {
    const int at = ((set0 + s) * ks_n + ks) * 8;
#pragma unroll
    for (int mb = 0; mb < DV16; ++mb)
      if (mb * 16 < dvp) {
        mo[(at + 2 * t) * dvp + mb * 16 + g] = o[s][mb][0];
        mo[(at + 2 * t + 1) * dvp + mb * 16 + g] = o[s][mb][1];
        mo[(at + 2 * t) * dvp + mb * 16 + g + 8] = o[s][mb][2];
        mo[(at + 2 * t + 1) * dvp + mb * 16 + g + 8] = o[s][mb][3];
      }
    if (g == 0) {
      mm[at + 2 * t] = m_run[s][0];
      mm[at + 2 * t + 1] = m_run[s][1];
      ml[at + 2 * t] = l_run[s][0];
      ml[at + 2 * t + 1] = l_run[s][1];
    }
  }
  __syncthreads();
  const bool partial = a.splits > 1 || maps > 1;
  for (int sh = warp; sh < sets * 8; sh += 4) {
    const int s = sh >> 3, hh = sh & 7, u = unit_of(s, hh);
    if (u < 0) continue;
    float M = -INFINITY, L = 0.0f;
    for (int w = 0; w < ks_n; ++w) M = fmaxf(M, mm[(s * ks_n + w) * 8 + hh]);
    for (int w = 0; w < ks_n; ++w) {
      const float mw = mm[(s * ks_n + w) * 8 + hh];
      if (mw != -INFINITY) L = fmaf(smax_ex2(mw - M), ml[(s * ks_n + w) * 8 + hh], L);
    }
    const size_t base = (size_t(blockIdx.z) * a.rows + row) * units + u;
    if (partial && lane == 0) {
      a.part_ml[base * 2] = M * 0.6931471805599453f;  // (the merge kernels work with natural exponents)
      a.part_ml[base * 2 + 1] = L;
    }
    const float f = partial ? 1.0f : a.out_scale / L * smax_gate(a.gate, a.ld_gate, row, u / maps);
    for (int col = lane; col < dv; col += 32) {
      float acc = 0.0f;
      for (int w = 0; w < ks_n; ++w) {
        const float mw = mm[(s * ks_n + w) * 8 + hh];
        if (mw != -INFINITY) acc = fmaf(smax_ex2(mw - M), mo[((s * ks_n + w) * 8 + hh) * dvp + col], acc);
      }
      if (partial) a.part_o[base * dv + col] = acc;
      else a.out[size_t(row) * a.ld_out + u * dv + col] = __float2bfloat16_rn(acc * f);
    }
  }
}

}  // namespace mtx
