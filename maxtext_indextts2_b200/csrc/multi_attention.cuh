// Tensor-core softmax attention (bf16) for score shapes that the kernels of softmax_attention.cuh do not have (its head comment
// defines them): two score maps per head over the same values, scores over the key heads' channels side by side (the mixed queries
// of a talking attention), value heads of another size than the keys, and head sizes that are any multiple of 8.
//
// A UNIT is one softmax: a (query head, map) pair.  The units of one value head ("its units") share that head's value rows; their
// key rows are, per map, one slice of `dim` channels (wide: all units read the same rows).
//
//   multi_attention_prefill_kernel<DV16, KT>   rows in portions.  CTA of eight warps (four with 16-key tiles, for the widest keys) = `rt` query tiles (16 rows each, consecutive
//                        entries of the host's table) x `uw` units of a value head: a warp owns one (tile, unit) pair, S = Q K^T and
//                        O += P V on mma.sync m16n8k16 with fp32 accumulators, running maximum and sum in fp32 registers.  Tiles
//                        that continue one another share the staged keys and values (cp.async double buffer through the page map);
//                        tiles of different sequences are walked one after the other.  With two maps a head's units sit in
//                        neighbouring warps and their difference is taken (and normed) in the epilogue.
//   multi_attention_decode_kernel<NV, DV16>   steps of single tokens: CTA = (row, value heads, key split), the products TRANSPOSED
//                        (S^T = K Q^T, O^T = V^T P^T), so the MMA's 16-row side carries keys / value columns and its 8-column side
//                        up to eight units: those of NV neighbouring value heads (wide), or both maps of a value head's query heads
//                        (a unit's query is zero in the other map's slice of the key row, so the two maps are one product over the
//                        row).  Four warps = ks_n slices of 16 keys x sg groups of units; partial results meet in shared memory.
//
// Keys and values arrive by 16-byte cp.async, eight threads per row; rows beyond the last visible key repeat it (their scores are masked),
// and the page map is read one key tile ahead of the copies that need it.
//
// Channels are padded to a multiple of 16 with zeros in shared memory.
#pragma once

#include "softmax_attention.cuh"

namespace mtx {

constexpr int kMatMaxWarps = 8;

struct MultiMmaPlan {
  bool ok = false;
  int kt = 0, dv16 = 0, warps = 0, uw = 0, rt = 0, chunks = 0;
  size_t smem = 0;
};

inline int mat_pad16(int n) { return (n + 15) / 16 * 16; }

// bytes of the staged queries and of one key / value stage
inline size_t mat_query_bytes(int dim, int warps) { return size_t(warps) * 16 * (mat_pad16(dim) + 8) * sizeof(bf16); }
inline size_t mat_stage_bytes(int dim, int vdim, int maps, bool wide, bool same_kv, int kt) {
  return size_t(kt) * ((wide ? 1 : maps) * mat_pad16(dim) + 8 + (same_kv ? 0 : mat_pad16(vdim) + 8)) * sizeof(bf16);
}

// n_tiles: query tiles of the step, num_sms: fewer tiles per CTA when the grid would not cover the GPU
inline MultiMmaPlan multi_mma_plan(int heads, int kv_heads, int dim, int vdim, int maps, bool wide, bool same_kv, int n_tiles, int num_sms) {
  MultiMmaPlan p;
  if (dim % 8 != 0 || vdim % 8 != 0 || vdim > 256 || (same_kv && vdim > dim)) return p;
  const int d16 = mat_pad16(vdim) / 16, units = heads / kv_heads * maps;
  p.dv16 = d16 <= 4 ? 4 : (d16 <= 8 ? 8 : 16);
  // 64-key tiles when two CTAs then still share an SM (and the accumulators leave room for the scores), else 32; score vectors
  // that do not fit even so: four warps and 16-key tiles
  struct { int kt, warps, kib; } tries[3] = {{64, 8, 112}, {32, 8, 226}, {16, 4, 226}};
  for (int i = p.dv16 <= 4 ? 0 : 1; i < 3 && !p.ok; ++i) {
    p.kt = tries[i].kt;
    p.warps = tries[i].warps;
    p.smem = mat_query_bytes(dim, p.warps) + 2 * mat_stage_bytes(dim, vdim, maps, wide, same_kv, p.kt);
    if (maps == 2) {  // (the epilogue's exchange of the second maps' results)
      const size_t xch = size_t(p.warps / 2) * 16 * mat_pad16(vdim) * sizeof(float);
      if (xch > p.smem) p.smem = xch;
    }
    p.ok = p.smem <= size_t(tries[i].kib) * 1024;
  }
  p.uw = units < p.warps ? units : p.warps;
  if (maps == 2 && (p.uw & 1)) --p.uw;
  p.chunks = (units + p.uw - 1) / p.uw;
  p.rt = p.warps / p.uw;
  while (p.rt > 1 && (long long)((n_tiles + p.rt - 1) / p.rt) * kv_heads * p.chunks < num_sms) p.rt /= 2;
  return p;
}

__device__ __forceinline__ void mat_cp16(uint32_t dst, const char* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }

// the 16-byte chunks sub, sub + 8, .. of `n` slices of `chunks` chunks each (slice strides in bytes)
__device__ __forceinline__ void mat_copy_slices(uint32_t dst, const char* src, int n, int chunks, int sub, uint32_t dst_stride, size_t src_stride) {
  dst += sub * 16;
  src += sub * 16;
  for (int m = 0; m < n; ++m) {
    uint32_t d = dst;
    const char* s = src;
    for (int c = sub; c < chunks; c += 8) {
      mat_cp16(d, s);
      d += 128;
      s += 128;
    }
    dst += dst_stride;
    src += src_stride;
  }
}

__device__ __forceinline__ void mat_ldsm_x4(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mat_ldsm_x4_trans(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}

template <int DV16, int KT>
__global__ void __launch_bounds__(KT == 16 ? 128 : 256, DV16 <= 8 && KT >= 32 ? 2 : 1) multi_attention_prefill_kernel(const SoftmaxAttnArgs<bf16> a, int n_tiles, int uw, int rt, int chunks) {
  extern __shared__ __align__(16) unsigned char mat_raw[];
  constexpr int NB = 2 * DV16, NW = KT == 16 ? 4 : 8, NT = NW * 32;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int maps = a.maps > 1 ? a.maps : 1, rep_units = a.heads / a.kv_heads * maps, units = a.heads * maps;
  const bool same_kv = a.k_pages == a.v_pages;
  const int d = a.dim, dv = a.vdim, dp = (d + 15) & ~15, dvp = (dv + 15) & ~15, n_slices = a.wide ? 1 : maps;
  const int QP = dp + 8, KP = n_slices * dp + 8, VP = same_kv ? KP : dvp + 8, stage_elems = KT * (KP + (same_kv ? 0 : VP));
  bf16* const sQ = reinterpret_cast<bf16*>(mat_raw);  // [NW warps][16][QP]
  bf16* const stage0 = sQ + NW * 16 * QP;      // stage s: K [KT][KP], then V [KT][VP]
  if (dp != d || dvp != dv) {  // the padding channels are zero and stay so
    const int words = (NW * 16 * QP + 2 * stage_elems) / 2;
    for (int e = tid; e < words; e += NT) reinterpret_cast<uint32_t*>(mat_raw)[e] = 0u;
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
  for (int r = lane >> 3; r < 16; r += 4)
    for (int c = (lane & 7) * 8; c < d; c += 64) {
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
  const char* const kbase = reinterpret_cast<const char*>(a.k_pages + (a.wide ? 0 : size_t(vh) * maps * pool_rows * d));
  const char* const vbase = reinterpret_cast<const char*>(a.v_pages + size_t(vh) * pool_rows * dv);
  const int ld_row = tid >> 3, ld_sub = tid & 7;  // eight threads per key row
  constexpr int RPT = KT * 8 / NT;                // key rows per thread
  const uint32_t sk_addr = smem_u32(stage0) + ld_row * KP * 2, sv_addr = smem_u32(stage0) + (KT * KP + ld_row * VP) * 2;
  const int map_of_warp = (u_all % maps) * (a.wide ? 0 : dp);

  // groups of tiles [ta, tb) that continue one another: they share their keys
  for (int ta = tile0, tb; ta < tile0 + rt && ta < n_tiles; ta = tb) {
    const int ra = a.tile_row0[ta], grp = a.group[ra], pa = a.pos[ra];
    int rb = a.tile_row0[ta + 1];
    for (tb = ta + 1; tb < tile0 + rt && tb < n_tiles; ++tb) {
      if (a.group[rb] != grp || a.pos[rb] != pa + (rb - ra)) break;
      rb = a.tile_row0[tb + 1];
    }
    const int lo = smax_first(pa, a.window, a.chunk), last = pa + (rb - ra) - 1, lead = a.keep_first < lo ? a.keep_first : lo, skip = lo - lead,
              v_last = last - skip, n_key_tiles = v_last / KT + 1;  // virtual key indices: see softmax_attention.cuh
    const int* pages = a.page_map + size_t(grp) * a.max_pages;
    const bool mine = active && my_tile >= ta && my_tile < tb;
    int rows_next[RPT];  // cache rows of this thread's keys of the tile that is copied next
    auto find_rows = [&](int it) {
#pragma unroll
      for (int q = 0; q < RPT; ++q) {
        const int vn = it * KT + ld_row + q * (NT / 8), v = vn < v_last ? vn : v_last, j = v < lead ? v : v + skip;
        const int pg = page_shift >= 0 ? (j >> page_shift) : j / tpp;
        rows_next[q] = pages[pg] * tpp + (j - pg * tpp);
      }
    };
    auto load_tile = [&](int stage) {
#pragma unroll
      for (int q = 0; q < RPT; ++q) {
        const uint32_t at = stage * stage_elems * 2 + q * (NT / 8) * KP * 2;
        mat_copy_slices(sk_addr + at, kbase + size_t(rows_next[q]) * (2 * d), n_slices, d >> 3, ld_sub, dp * 2, pool_rows * d * 2);
        if (!same_kv) mat_copy_slices(sv_addr + stage * stage_elems * 2 + q * (NT / 8) * VP * 2, vbase + size_t(rows_next[q]) * (2 * dv), 1, dv >> 3, ld_sub, 0, 0);
      }
      cp_async_commit();
    };
    find_rows(0);
    load_tile(0);
    if (n_key_tiles > 1) find_rows(1);
    for (int it = 0; it < n_key_tiles; ++it) {
      if (it + 1 < n_key_tiles) {
        load_tile((it + 1) & 1);
        if (it + 2 < n_key_tiles) find_rows(it + 2);
        cp_async_wait_pending(1);
      } else {
        cp_async_wait_pending(0);
      }
      __syncthreads();
      const int v0 = it * KT, j0 = v0 < lead ? v0 : v0 + skip, j_end = v0 + KT <= lead ? v0 + KT : v0 + KT + skip;
      if (mine && j0 <= p_last && (j_end > lo_first || j0 < a.keep_first)) {
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
        const bool every_key_seen = v0 < lead ? v0 + KT <= lead : j_end - 1 <= p0 && j0 >= lo_last;
        float mx0 = -INFINITY, mx1 = -INFINITY;  // (of the raw products: the scale is positive)
        if (every_key_seen) {
#pragma unroll
          for (int nb = 0; nb < KT / 8; ++nb) {
            mx0 = fmaxf(mx0, fmaxf(s[nb][0], s[nb][1]));
            mx1 = fmaxf(mx1, fmaxf(s[nb][2], s[nb][3]));
          }
        } else {
#pragma unroll
          for (int nb = 0; nb < KT / 8; ++nb) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int v = v0 + nb * 8 + 2 * t + (e & 1), j = v < lead ? v : v + skip;
              if (j > ((e & 2) ? pi1 : pi0) || (j < ((e & 2) ? lo1 : lo0) && j >= a.keep_first)) s[nb][e] = -INFINITY;
            }
            mx0 = fmaxf(mx0, fmaxf(s[nb][0], s[nb][1]));
            mx1 = fmaxf(mx1, fmaxf(s[nb][2], s[nb][3]));
          }
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m_run[0], mx0 * mul), mn1 = fmaxf(m_run[1], mx1 * mul);
        const float base0 = mn0 == -INFINITY ? 0.0f : mn0, base1 = mn1 == -INFINITY ? 0.0f : mn1;
        const float fix0 = smax_ex2(m_run[0] - base0), fix1 = smax_ex2(m_run[1] - base1);
        m_run[0] = mn0;
        m_run[1] = mn1;
        float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
        for (int nb = 0; nb < KT / 8; ++nb) {
          s[nb][0] = smax_ex2(fmaf(s[nb][0], mul, -base0));
          s[nb][1] = smax_ex2(fmaf(s[nb][1], mul, -base0));
          s[nb][2] = smax_ex2(fmaf(s[nb][2], mul, -base1));
          s[nb][3] = smax_ex2(fmaf(s[nb][3], mul, -base1));
          sum0 += s[nb][0] + s[nb][1];
          sum1 += s[nb][2] + s[nb][3];
        }
        l_run[0] = l_run[0] * fix0 + sum0;  // (per-thread partial sums; the four lanes of a row are added at the end)
        l_run[1] = l_run[1] * fix1 + sum1;
        if (__any_sync(0xffffffffu, fix0 != 1.0f || fix1 != 1.0f)) {  // (most tiles leave every row's maximum as it is)
#pragma unroll
          for (int nb = 0; nb < NB; ++nb) {
            o[nb][0] *= fix0;
            o[nb][1] *= fix0;
            o[nb][2] *= fix1;
            o[nb][3] *= fix1;
          }
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
  const float f0 = a.out_scale / l_run[0] * (g < nr ? smax_gate(a, r0 + g, h) : 1.0f);
  const float f1 = a.out_scale / l_run[1] * (g + 8 < nr ? smax_gate(a, r0 + g + 8, h) : 1.0f);
  if (a.value_gate) {
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (nb * 8 + 2 * t < dv && g + (e & 2) * 4 < nr) o[nb][e] *= smax_value_gate(a, r0 + g + (e & 2) * 4, h, nb * 8 + 2 * t + (e & 1));
  }
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
  int nv = 0, dv16 = 0, sg = 0;
  int groups = 0, chunks = 0;  // CTAs per (row, split): groups of value heads x chunks of eight units
  size_t smem = 0;
};

inline size_t multi_decode_smem_bytes(int dim, int vdim, int maps, bool wide, int nv, int sg, bool same_kv) {
  const int kt = 64 / sg, kw = (wide ? 1 : maps) * mat_pad16(dim), dvp = mat_pad16(vdim);
  const size_t q = size_t(sg) * 8 * (kw + 8) * sizeof(bf16);
  const size_t ring = size_t(2) * kt * (kw + 8 + (same_kv ? 0 : (wide ? nv * sg : 1) * dvp + 8)) * sizeof(bf16);
  const size_t merge = sizeof(float) * 4 * (8 * size_t(dvp) + 16);
  return q + (ring > merge ? ring : merge);
}

inline MultiDecodePlan multi_decode_plan(int heads, int kv_heads, int dim, int vdim, int maps, bool wide, bool same_kv) {
  MultiDecodePlan p;
  if (dim % 8 != 0 || vdim % 8 != 0 || vdim > 256 || (same_kv && vdim > dim)) return p;
  const int d16 = mat_pad16(vdim) / 16, rep = heads / kv_heads;
  p.dv16 = d16 <= 4 ? 4 : (d16 <= 8 ? 8 : 16);
  p.chunks = (rep * maps + 7) / 8;
  p.nv = 1;
  // wide: the value heads whose query heads fill the eight columns, at most 16 accumulator tiles per warp
  if (wide)
    while (p.nv < 4 && p.nv * 2 * rep <= 8 && p.nv * 2 * p.dv16 <= 16 && p.nv < kv_heads) p.nv *= 2;
  // ... and as many groups of them per CTA as there are (up to four): the key rows they share are then staged once
  int sg = 1;
  if (wide)
    while (sg < 4 && sg * p.nv < kv_heads) sg *= 2;
  for (; sg >= 1; sg /= 2) {
    p.sg = sg;
    p.groups = wide ? (kv_heads + sg * p.nv - 1) / (sg * p.nv) : kv_heads;
    p.smem = multi_decode_smem_bytes(dim, vdim, maps, wide, p.nv, sg, same_kv);
    if (p.smem <= 226 * size_t(1024)) {
      p.ok = true;
      break;
    }
  }
  return p;
}

template <int NV, int DV16>
__global__ void __launch_bounds__(128) multi_attention_decode_kernel(const SoftmaxAttnArgs<bf16> a, int sg, int chunks) {
  extern __shared__ __align__(16) unsigned char mat_raw[];
  constexpr int NT = 128;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int maps = a.maps > 1 ? a.maps : 1, rep = a.heads / a.kv_heads, rep_units = rep * maps, units = a.heads * maps;
  const bool same_kv = a.k_pages == a.v_pages;
  const int d = a.dim, dv = a.vdim, dp = (d + 15) & ~15, dvp = (dv + 15) & ~15;
  const int ks_n = 4 / sg, KT = 16 * ks_n, n_slices = a.wide ? 1 : maps, n_vals = a.wide ? NV * sg : 1, kw = n_slices * dp;
  const int KP = kw + 8, VP = same_kv ? KP : n_vals * dvp + 8, stage_elems = KT * (KP + (same_kv ? 0 : VP));
  bf16* const sQ = reinterpret_cast<bf16*>(mat_raw);  // [sg][8 units][KP]
  bf16* const stage0 = sQ + sg * 8 * KP;              // stage s: K [KT][KP], then V [KT][VP]
  if (dp != d || dvp != dv) {  // the padding channels are zero and stay so
    const int words = (sg * 8 * KP + 2 * stage_elems) / 2;
    for (int e = tid; e < words; e += NT) reinterpret_cast<uint32_t*>(mat_raw)[e] = 0u;
    __syncthreads();
  }
  griddep_wait();
  const int row = blockIdx.x, vgroup = blockIdx.y / chunks, chunk = blockIdx.y % chunks;
  const int pos = a.pos[row], grp = a.group[row], lo = smax_first(pos, a.window, a.chunk);
  const int* pages = a.page_map + size_t(grp) * a.max_pages;
  const int tpp = a.tokens_per_page, page_shift = (tpp & (tpp - 1)) == 0 ? __ffs(tpp) - 1 : -1;
  const size_t pool_rows = size_t(a.num_pages) * tpp;
  const int vh0 = a.wide ? vgroup * NV * sg : vgroup;  // first value head of the CTA
  const char* const kbase = reinterpret_cast<const char*>(a.k_pages + (a.wide ? 0 : size_t(vgroup) * maps * pool_rows * d));
  const char* const vbase = reinterpret_cast<const char*>(a.v_pages + size_t(vh0) * pool_rows * dv);
  const int vals_here = n_vals < a.kv_heads - vh0 ? n_vals : a.kv_heads - vh0;  // (the last group may hold fewer value heads)
  const int lead = a.keep_first < lo ? a.keep_first : lo, skip = lo - lead, v_last = pos - skip;
  const int all_key_tiles = v_last / KT + 1, per = (all_key_tiles + a.splits - 1) / a.splits, tile_lo = int(blockIdx.z) * per;
  int n_key_tiles = all_key_tiles - tile_lo < per ? all_key_tiles - tile_lo : per;
  if (n_key_tiles < 0) n_key_tiles = 0;
  // column hh of unit group s: its unit (-1: none) and, among the group's value heads, its value head
  const int cols_v = rep_units - chunk * 8 < 8 ? rep_units - chunk * 8 : 8;  // columns of one value head
  auto value_of = [&](int hh) { return NV == 1 ? 0 : hh / cols_v; };
  auto unit_of = [&](int s, int hh) -> int {
    const int v = value_of(hh), vh = vh0 + s * NV + v, r = hh - v * cols_v;
    return v < NV && r < cols_v && vh < a.kv_heads ? vh * rep_units + chunk * 8 + r : -1;
  };
  const int ld_row = tid >> 3, ld_sub = tid & 7;
  const uint32_t sk_addr = smem_u32(stage0) + ld_row * KP * 2, sv_addr = smem_u32(stage0) + (KT * KP + ld_row * VP) * 2;
  int rows_next[4];  // cache rows of this thread's keys (ks_n of them) of the tile that is copied next
  auto find_rows = [&](int it) {
#pragma unroll
    for (int q = 0; q < 4; ++q)
      if (q < ks_n) {
        const int vn = (tile_lo + it) * KT + ld_row + q * 16, v = vn < v_last ? vn : v_last, j = v < lead ? v : v + skip;
        const int pg = page_shift >= 0 ? (j >> page_shift) : j / tpp;
        rows_next[q] = pages[pg] * tpp + (j - pg * tpp);
      }
  };
  auto load_tile = [&](int stage) {
    const uint32_t at = stage * stage_elems * 2;
#pragma unroll
    for (int q = 0; q < 4; ++q)
      if (q < ks_n) {
        mat_copy_slices(sk_addr + at + q * 32 * KP, kbase + size_t(rows_next[q]) * (2 * d), n_slices, d >> 3, ld_sub, dp * 2, pool_rows * d * 2);
        if (!same_kv) mat_copy_slices(sv_addr + at + q * 32 * VP, vbase + size_t(rows_next[q]) * (2 * dv), vals_here, dv >> 3, ld_sub, dvp * 2, pool_rows * dv * 2);
      }
    cp_async_commit();
  };
  if (n_key_tiles > 0) {
    find_rows(0);
    load_tile(0);
    if (n_key_tiles > 1) find_rows(1);
  }
  // the units' queries; two maps: zero in the other map's slice
  for (int sh = warp; sh < sg * 8; sh += 4) {
    const int u = unit_of(sh >> 3, sh & 7), slice = n_slices > 1 ? (u < 0 ? 0 : u % maps) : 0;
    for (int m = 0; m < n_slices; ++m)
      for (int c = lane * 8; c < d; c += 256) {
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (u >= 0 && m == slice) v = *reinterpret_cast<const uint4*>(a.q + (size_t(row) * units + u) * d + c);
        *reinterpret_cast<uint4*>(sQ + sh * KP + m * dp + c) = v;
      }
  }
  const int ks = warp % ks_n, set = warp / ks_n;
  float o[NV][DV16][4];  // O^T: (column mb * 16 + g / g + 8, unit 2t / 2t + 1)
#pragma unroll
  for (int v = 0; v < NV; ++v)
#pragma unroll
    for (int mb = 0; mb < DV16; ++mb)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[v][mb][e] = 0.0f;
  constexpr float kLog2e = 1.4426950408889634f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};  // units 2t, 2t + 1 (maxima in units of log 2)
  if (a.sink && ks == 0 && blockIdx.z == 0) {  // (the first key slice of the first split carries the sink)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int u = unit_of(set, 2 * t + e);
      if (u >= 0) {
        m_run[e] = a.sink[u / maps] * kLog2e;
        l_run[e] = g == 0 ? 1.0f : 0.0f;
      }
    }
  }
  const float mul = a.scale * kLog2e;
  for (int it = 0; it < n_key_tiles; ++it) {
    if (it + 1 < n_key_tiles) {
      load_tile((it + 1) & 1);
      if (it + 2 < n_key_tiles) find_rows(it + 2);
      cp_async_wait_pending(1);
    } else {
      cp_async_wait_pending(0);
    }
    __syncthreads();
    const bf16* sk = stage0 + size_t(it & 1) * stage_elems;
    const bf16* sv = same_kv ? sk : sk + KT * KP;
    const int j0 = (tile_lo + it) * KT + ks * 16;  // this warp's 16 keys
    if (j0 <= v_last) {
      float c[4] = {0.0f, 0.0f, 0.0f, 0.0f}, c2[4] = {0.0f, 0.0f, 0.0f, 0.0f};  // two chains
      const bf16* kb = sk + (ks * 16 + (lane & 15)) * KP + (lane >> 4) * 8;
      const bf16* qb = sQ + (set * 8 + (lane & 7)) * KP + (lane >> 3) * 8;  // (four 8-channel columns of the eight units per ldmatrix)
      int k0 = 0;
#pragma unroll 2
      for (; k0 + 32 <= kw; k0 += 32) {
        uint32_t af[4], bf[4], af2[4];
        mat_ldsm_x4(bf, qb + k0);
        mat_ldsm_x4(af, kb + k0);
        mat_ldsm_x4(af2, kb + k0 + 16);
        mma_bf16_16816(c, af, bf[0], bf[1]);
        mma_bf16_16816(c2, af2, bf[2], bf[3]);
      }
      if (k0 < kw) {
        uint32_t af[4];
        const bf16* q1 = sQ + (set * 8 + g) * KP + k0 + 2 * t;
        mat_ldsm_x4(af, kb + k0);
        mma_bf16_16816(c, af, *reinterpret_cast<const uint32_t*>(q1), *reinterpret_cast<const uint32_t*>(q1 + 8));
      }
      const bool sa = j0 + g <= v_last, sb = j0 + g + 8 <= v_last;  // (every key of the walk up to its end is visible)
      c[0] = sa ? (c[0] + c2[0]) * mul : -INFINITY;
      c[1] = sa ? (c[1] + c2[1]) * mul : -INFINITY;
      c[2] = sb ? (c[2] + c2[2]) * mul : -INFINITY;
      c[3] = sb ? (c[3] + c2[3]) * mul : -INFINITY;
      float mx0 = fmaxf(c[0], c[2]), mx1 = fmaxf(c[1], c[3]);
#pragma unroll
      for (int sh = 4; sh < 32; sh <<= 1) {
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, sh));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, sh));
      }
      const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);  // (finite: the warp's first key is visible)
      const float fix0 = smax_ex2(m_run[0] - mn0), fix1 = smax_ex2(m_run[1] - mn1);
      m_run[0] = mn0;
      m_run[1] = mn1;
      c[0] = smax_ex2(c[0] - mn0);
      c[1] = smax_ex2(c[1] - mn1);
      c[2] = smax_ex2(c[2] - mn0);
      c[3] = smax_ex2(c[3] - mn1);
      l_run[0] = l_run[0] * fix0 + c[0] + c[2];  // (this lane's keys; the eight lanes of a unit are added at the end)
      l_run[1] = l_run[1] * fix1 + c[1] + c[3];
      if (__any_sync(0xffffffffu, fix0 != 1.0f || fix1 != 1.0f)) {
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
          for (int mb = 0; mb < DV16; ++mb) {
            o[v][mb][0] *= fix0;
            o[v][mb][1] *= fix1;
            o[v][mb][2] *= fix0;
            o[v][mb][3] *= fix1;
          }
      }
      const uint32_t pb0 = smax_movmatrix_trans(smax_pack_bf16(c[0], c[1])), pb1 = smax_movmatrix_trans(smax_pack_bf16(c[2], c[3]));
      const bf16* v0 = sv + (ks * 16 + (lane & 7) + 8 * (lane >> 4)) * VP + ((lane >> 3) & 1) * 8 + set * NV * dvp;
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int mb = 0; mb < DV16; ++mb)
          if (mb * 16 < dvp) {
            uint32_t vf[4];
            mat_ldsm_x4_trans(vf, v0 + v * dvp + mb * 16);
            mma_bf16_16816(o[v][mb], vf, pb0, pb1);
          }
    }
    __syncthreads();
  }
#pragma unroll
  for (int sh = 4; sh < 32; sh <<= 1) {
    l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], sh);
    l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], sh);
  }
  // merge of the key slices (the ring is free: the loop ended with a barrier)
  float* mo = reinterpret_cast<float*>(stage0);  // [sg][ks_n][8 units][dvp]
  float* mm = mo + 32 * dvp;                     // [sg][ks_n][8] maxima, then the sums
  float* ml = mm + 32;
  {
    const int at = (set * ks_n + ks) * 8 + 2 * t, va = value_of(2 * t), vb = value_of(2 * t + 1);
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int mb = 0; mb < DV16; ++mb)
        if (mb * 16 < dvp) {
          float* dst = mo + size_t(at) * dvp + mb * 16 + g;
          if (v == va) {
            dst[0] = o[v][mb][0];
            dst[8] = o[v][mb][2];
          }
          if (v == vb) {
            dst[dvp] = o[v][mb][1];
            dst[dvp + 8] = o[v][mb][3];
          }
        }
    if (g == 0) {
      mm[at] = m_run[0];
      mm[at + 1] = m_run[1];
      ml[at] = l_run[0];
      ml[at + 1] = l_run[1];
    }
  }
  __syncthreads();
  const bool partial = a.splits > 1 || maps > 1;
  for (int sh = warp; sh < sg * 8; sh += 4) {
    const int s = sh >> 3, hh = sh & 7, u = unit_of(s, hh);
    if (u < 0) continue;
    float w[4], M = -INFINITY, L = 0.0f;  // the key slices' weights
    for (int i = 0; i < ks_n; ++i) M = fmaxf(M, mm[(s * ks_n + i) * 8 + hh]);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      w[i] = 0.0f;
      if (i < ks_n) {
        const float mw = mm[(s * ks_n + i) * 8 + hh];
        if (mw != -INFINITY) w[i] = smax_ex2(mw - M);
        L = fmaf(w[i], ml[(s * ks_n + i) * 8 + hh], L);
      }
    }
    const size_t base = (size_t(blockIdx.z) * a.rows + row) * units + u;
    if (partial && lane == 0) {
      a.part_ml[base * 2] = M * 0.6931471805599453f;  // (the merge kernels work with natural exponents)
      a.part_ml[base * 2 + 1] = L;
    }
    const float f = partial ? 1.0f : a.out_scale / L * smax_gate(a, row, u / maps);
    for (int col = lane; col < dv; col += 32) {
      float acc = 0.0f;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (i < ks_n) acc = fmaf(w[i], mo[((s * ks_n + i) * 8 + hh) * dvp + col], acc);
      if (partial) a.part_o[base * dv + col] = acc;
      else a.out[size_t(row) * a.ld_out + u * dv + col] = __float2bfloat16_rn(acc * f * smax_value_gate(a, row, u, col));
    }
  }
}

}  // namespace mtx
