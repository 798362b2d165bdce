"""The Fibelix design: a pre-norm decoder whose config.json lists its layers one by one.

    x += mixer(norm(x, norm1));   x += ff(norm(x, norm2))          (a routed feed-forward, or none)

with norm(x, w) = x / sqrt(mean(x^2) + eps) * (1 + w).  Mixers:

* ``attention``        -- grouped-query softmax attention with biases in its projections: rotate-half positions with linearly
                          scaled frequencies, a temperature per head on the scores, scores mixed over the heads (``talk``) before the
                          softmax, one added to the softmax's denominator; a query sees its own chunk of positions up to itself.
* ``attention_2``      -- differential attention: two softmax maps per head over the same values, the second one's result times
                          a layer-wide lambda taken off the first one's, each head brought to unit RMS, times (1 - diff); no
                          positions, chunked.  ``kv_from: j`` reads layer j's cache.
* ``latent_attention`` -- queries through a normed latent, keys and values expanded from a cached normed latent plus one rotated
                          key part shared by the heads (interleaved pairs, YaRN-scaled frequencies and amplitude), a sliding window,
                          a sigmoid gate per head.

Feed-forward: router logits with a bias, the ``top`` largest chosen, a softmax over the chosen logits as weights, silu-gated
experts.  The logits are the normed stream times the embedding table.

This module is the design's entry in the framework: config.json -> config keys (`config_keys`), checks (`validate_layer_specs`),
safetensors names -> layer descriptors of the layered engine (`model_plan`), random weights of any size (`random_tensors`).  On the
device every layer is a MTX_NORM_PRE layer without input convolution; the norms' weights are handed over as 1 + w.
"""

from __future__ import annotations

import math
from typing import Any, Dict, List, Optional, Tuple

import numpy as np
import torch

from .gugidra import TILE_ROWS, _interleave, _need, _shape, rot_frequencies

MIXERS = ("attention", "attention_2", "latent_attention")


def yarn_rot_frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[torch.Tensor, float]:
  """(radians per position of the channel pair i < dims / 2 in float64, factor on cosine and sine).  `scaling` {factor, original,
  fast, slow}: a pair that turns more than `fast` times within `original` positions keeps base^(-2i / dims), one that turns fewer
  than `slow` times is `factor` times slower, and between the two the frequency is blended linearly in i."""
  f = rot_frequencies(dims, base)
  if not scaling:
    return f, 1.0
  factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
  pair = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
  lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), dims - 1)
  ramp = torch.from_numpy(np.clip((np.arange(dims // 2, dtype=np.float64) - lo) / max(hi - lo, 0.001), 0.0, 1.0))
  return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def config_keys(model: dict) -> dict:
  """config.json of a Fibelix model -> keys of configs/base.yml."""
  layers = model["layers"]
  validate_layer_specs(layers)
  ffs = [int(l["mlp"]["expert"]["ff"]) for l in layers if l.get("mlp")]
  first = layers[0]["mixer"]
  return dict(
      base_emb_dim=int(model["width"]),
      vocab_size=int(model["vocab"]),
      base_num_decoder_layers=len(layers),
      global_parameter_scale=1,
      normalization_layer_epsilon=float(model["norm"]["eps"]),
      layer_specs=layers,
      # (the homogeneous keys describe the first layer; the engine reads layer_specs)
      base_num_query_heads=int(first["heads"]),
      base_num_kv_heads=int(first.get("kv_heads", first["heads"])),
      head_dim=int(first["dim"]),
      base_mlp_dim=max(ffs) if ffs else 0,
  )


def validate_layer_specs(specs: List[dict]) -> None:
  for i, l in enumerate(specs):
    kind = l.get("type")
    if kind not in MIXERS:
      raise ValueError(f"layer {i}: mixer type {kind!r}; this design has {MIXERS}")
    m = l["mixer"]
    where = f"layer {i}: mixer"
    if int((m.get("mask") or {}).get("size") or 0) < 0:
      raise ValueError(f"layer {i}: mask.size must not be negative")
    if kind == "latent_attention":
      _need(m, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale"), where)
      if int(m["rot_dim"]):
        _need(m, ("rot",), where)
        if int(m["rot_dim"]) % 2 or int(m["rot"]["dims"]) != int(m["rot_dim"]):
          raise ValueError(f"layer {i}: rot_dim must be even and equal to rot.dims")
        if m["rot"].get("scaling"):
          _need(m["rot"]["scaling"], ("factor", "original", "fast", "slow"), where + ".rot.scaling")
    else:
      _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
      if int(m["heads"]) % int(m["kv_heads"]):
        raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
      rot = m.get("rot")
      if kind == "attention_2":
        _need(m, ("diff",), where)
        if rot:
          raise ValueError(f"layer {i}: differential attention has no rotation")
      elif rot:
        if int(rot["dims"]) % 2 or int(rot["dims"]) > int(m["dim"]):
          raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
        if rot.get("scaling"):
          _need(rot["scaling"], ("factor",), where + ".rot.scaling")
      src = m.get("kv_from")
      if src is not None:
        src = int(src)
        if not 0 <= src < i or specs[src].get("type") != kind or specs[src]["mixer"].get("kv_from") is not None:
          raise ValueError(f"layer {i}: kv_from must name an earlier layer of the same type with projections of its own")
        o = specs[src]["mixer"]
        if any(int(o[k]) != int(m[k]) for k in ("kv_heads", "dim", "vdim")):
          raise ValueError(f"layer {i}: its key / value geometry differs from layer {src}'s, whose cache it reads")
    f = l.get("mlp")
    if f is not None:
      if f.get("kind", "moe") != "moe":
        raise ValueError(f"layer {i}: feed-forward kind {f.get('kind')!r}; this design has routed ones")
      _need(f, ("expert", "router"), f"layer {i}: mlp")
      n, top = int(f["router"]["experts"]), int(f["router"]["top"])
      if not 1 <= top <= n:
        raise ValueError(f"layer {i}: top {top} of {n} experts")


def difference_weight(lq1: torch.Tensor, lk1: torch.Tensor, lq2: torch.Tensor, lk2: torch.Tensor, diff: float) -> float:
  """exp(<lq1, lk1>) - exp(<lq2, lk2>) + diff."""
  dot = lambda a, b: float((a.to(torch.float64) * b.to(torch.float64)).sum())
  return math.exp(dot(lq1, lk1)) - math.exp(dot(lq2, lk2)) + diff


def layer_plan(config, tensors: Dict[str, torch.Tensor], i: int) -> Dict[str, Any]:
  """What layer i hands to the layered engine: sizes and scalars (python numbers) and host tensors; matrices keep their stored
  dtype.  All projections of the mixer's input are one matrix in the order the device reads them."""
  spec = config.layer_specs[i]
  E = int(config.emb_dim)
  t, p, m = tensors, f"l{i}.mix.", spec["mixer"]
  dev = tensors["embed"].device
  f32 = lambda name, shape: _shape(t[name].to(torch.float32), shape, name)
  plan: Dict[str, Any] = dict(mixer="composite", norm_style="pre", attn=None, rec=None, latent=None, moe=None, ff_kind="moe", ff=0,
                              residual_mult=1.0, conv_taps=0, conv1=None, conv2=None, norm1=1.0 + f32(f"l{i}.norm1", (E,)))
  rows: List[torch.Tensor] = []
  bias: List[torch.Tensor] = []

  def add(name: str, n: int, with_bias: bool = False) -> None:
    rows.append(_shape(t[p + name], (n, E), p + name))
    if with_bias:
      bias.append(f32(p + name + ".b", (n,)))

  H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
  size = int((m.get("mask") or {}).get("size") or 0)
  if spec["type"] == "latent_attention":
    dr, qr, kr = int(m["rot_dim"]), int(m["q_rank"]), int(m["kv_rank"])
    add("dq", qr)
    add("dkv", kr + dr)
    add("g", H)
    freq, amp = yarn_rot_frequencies(dr, float(m["rot"]["base"]), m["rot"].get("scaling")) if dr else (None, 1.0)
    uk = _shape(t[p + "uk"], (H * d, kr), p + "uk")
    plan["latent"] = dict(heads=H, dim=d, rot_dim=dr, vdim=dv, q_rank=qr, kv_rank=kr, rot_half=0, scale=float(m["scale"]), window=size,
                          rot_freq=freq, rot_amp=amp, sink=None, q_norm=f32(p + "dq.norm", (qr,)), kv_norm=f32(p + "dkv.norm", (kr,)),
                          w_uq=_shape(t[p + "uq"], (H * (d + dr), qr), p + "uq"),
                          w_uk_t=uk.reshape(H, d, kr).transpose(1, 2).contiguous(),  # [H, kv_rank, dim]
                          w_uv=_shape(t[p + "uv"], (H * dv, kr), p + "uv").reshape(H, dv, kr).contiguous())
  else:
    G, src = int(m["kv_heads"]), m.get("kv_from")
    talking = spec["type"] == "attention"
    maps = 1 if talking else 2
    add("q", H * maps * d, talking)
    if src is None:
      add("k", G * maps * d, talking)
      add("v", G * dv, talking)
    rot = m.get("rot") if talking else None
    rd = int(rot["dims"]) if rot else 0
    attn = dict(heads=H, kv_heads=G, dim=d, vdim=dv, window=0, chunk=size, maps=maps, rot_dims=rd, rot_half=1, values_are_keys=0, scale=float(m["scale"]),
                out_scale=1.0, rot_freq=None, shared_kv=0 if src is None else 1, kv_from=None if src is None else int(src), head_gate=0)
    if talking:
      if rd:
        attn["rot_freq"] = rot_frequencies(rd, float(rot["base"])) / float((rot.get("scaling") or {}).get("factor", 1.0))
      attn.update(temp=f32(p + "temp", (H,)), talk=f32(p + "talk", (H, H)), sink=torch.zeros(H, dtype=torch.float32, device=dev))
      plan["bo"] = f32(p + "o.b", (E,))
    else:
      diff = float(m["diff"])
      attn.update(diff_lambda=difference_weight(*(_shape(t[p + n], (d,), p + n) for n in ("lq1", "lk1", "lq2", "lk2")), diff), diff_scale=1.0 - diff)
    plan["attn"] = attn
  w_in = torch.cat(rows, dim=0)
  pad = (-w_in.shape[0]) % TILE_ROWS if E % 64 == 0 else 0
  if pad:  # zero rows up to a whole tile of the tensor-core GEMM
    w_in = torch.cat([w_in, torch.zeros(pad, E, dtype=w_in.dtype, device=dev)], dim=0)
  if bias:
    plan["b_in"] = torch.cat(bias + [torch.zeros(pad, dtype=torch.float32, device=dev)])
  plan.update(w_in=w_in, n_in=int(w_in.shape[0]), wo=_shape(t[p + "o"], (E, H * dv), p + "o"))
  f = spec.get("mlp")
  if f is not None:
    q, n_exp, F = f"l{i}.mlp.", int(f["router"]["experts"]), int(f["expert"]["ff"])
    plan["norm2"] = 1.0 + f32(f"l{i}.norm2", (E,))
    part = lambda e, name, shape: _shape(t[f"{q}e{e}.{name}"], shape, f"{q}e{e}.{name}")
    plan["moe"] = dict(experts=n_exp, top=int(f["router"]["top"]), groups=1, keep_groups=1, ff=F, limit=0.0, shared_ff=0, shared_limit=0.0, act_silu=1,
                       chosen_softmax=1, correction=None, w_router=_shape(t[q + "router"], (n_exp, E), q + "router"), router_bias=f32(q + "router.b", (n_exp,)),
                       w_gate_up=torch.stack([_interleave(part(e, "gate", (F, E)), part(e, "up", (F, E))) for e in range(n_exp)]),
                       w_down=torch.stack([part(e, "down", (E, F)) for e in range(n_exp)]), shared_gate_up=None, shared_down=None)
  return plan


def model_plan(config, tensors: Dict[str, torch.Tensor]) -> Dict[str, Any]:
  E, V = int(config.emb_dim), int(config.vocab_size)
  return dict(
      embedding=_shape(tensors["embed"], (V, E), "embed"), head=tensors["embed"], final_gain=1.0,
      final_norm=1.0 + _shape(tensors["final.norm"].to(torch.float32), (E,), "final.norm"),
      embed_scale=1.0, logit_softcap=0.0, logit_scale=1.0, norm_groups=1, layers=[layer_plan(config, tensors, i) for i in range(len(config.layer_specs))],
  )


def random_tensors(config, seed: int = 0, device: Any = "cpu") -> Dict[str, torch.Tensor]:
  """Random bf16 weights with the design's tensor names, for `config` (tests, benchmarks and smoke runs; made on `device`)."""
  g = torch.Generator(device=device).manual_seed(seed)
  E, V = int(config.emb_dim), int(config.vocab_size)

  def rn(*shape, std=1.0, mean=0.0):
    return (torch.randn(tuple(shape), generator=g, device=device) * std + mean).to(torch.bfloat16)

  lin = lambda n_, k: rn(n_, k, std=1.0 / math.sqrt(k))
  t = {"embed": rn(V, E), "final.norm": rn(E, std=0.1)}
  for i, l in enumerate(config.layer_specs):
    p, q, m = f"l{i}.", f"l{i}.mix.", l["mixer"]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    t[p + "norm1"], t[q + "o"] = rn(E, std=0.1), lin(E, H * dv)
    if l["type"] == "attention":
      G = int(m["kv_heads"])
      names = [("q", H * d)] + ([("k", G * d), ("v", G * dv)] if m.get("kv_from") is None else [])
      for n, r in names:
        t[q + n], t[q + n + ".b"] = lin(r, E), rn(r, std=0.1)
      t[q + "o.b"], t[q + "temp"] = rn(E, std=0.1), rn(H, std=0.1, mean=1.0)
      t[q + "talk"] = (torch.eye(H, device=device) + 0.3 * torch.randn(H, H, generator=g, device=device)).to(torch.bfloat16)
    elif l["type"] == "attention_2":
      G = int(m["kv_heads"])
      t[q + "q"] = lin(H * 2 * d, E)
      if m.get("kv_from") is None:
        t[q + "k"], t[q + "v"] = lin(G * 2 * d, E), lin(G * dv, E)
      for n in ("lq1", "lk1", "lq2", "lk2"):
        t[q + n] = rn(d, std=0.1)
    else:
      dr, qr, kr = int(m["rot_dim"]), int(m["q_rank"]), int(m["kv_rank"])
      t[q + "dq"], t[q + "dq.norm"], t[q + "uq"] = lin(qr, E), rn(qr, std=0.1, mean=1.0), lin(H * (d + dr), qr)
      t[q + "dkv"], t[q + "dkv.norm"] = lin(kr + dr, E), rn(kr, std=0.1, mean=1.0)
      t[q + "uk"], t[q + "uv"], t[q + "g"] = lin(H * d, kr), lin(H * dv, kr), lin(H, E)
    f = l.get("mlp")
    if f:
      n_exp, F = int(f["router"]["experts"]), int(f["expert"]["ff"])
      t[p + "norm2"] = rn(E, std=0.1)
      for e in range(n_exp):
        x = f"{p}mlp.e{e}."
        t[x + "gate"], t[x + "up"], t[x + "down"] = lin(F, E), lin(F, E), lin(E, F)
      t[p + "mlp.router"], t[p + "mlp.router.b"] = rn(n_exp, E, std=2.0 / math.sqrt(E)), rn(n_exp, std=0.3)
  return t


# -- config.json-shaped dicts (tests, benchmarks) ----------------------------------------------------------------------------


def model_dict(width: int, vocab: int, layers: List[dict], eps: float = 1e-6) -> dict:
  return {"architecture": "Fibelix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def moe_ff(experts: int, top: int, ff: int) -> dict:
  return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _mixer(kind: str, m: dict, size: int, mlp: Optional[dict]) -> dict:
  if size:
    m["mask"] = {"size": size}
  return {"type": kind, "mixer": m, "mlp": mlp}


def talking_layer(heads: int, kv_heads: int, dim: int, vdim: Optional[int] = None, chunk: int = 0, scale: float = 0.0, rot_dims: Optional[int] = None,
                  rot_base: float = 10000.0, rot_factor: float = 1.0, kv_from: Optional[int] = None, mlp: Optional[dict] = None) -> dict:
  m: Dict[str, Any] = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "scale": scale or dim**-0.5}
  rd = dim if rot_dims is None else rot_dims
  if rd:
    m["rot"] = {"base": rot_base, "dims": rd, "scaling": {"factor": rot_factor}}
  if kv_from is not None:
    m["kv_from"] = kv_from
  return _mixer("attention", m, chunk, mlp)


def differential_layer(heads: int, kv_heads: int, dim: int, vdim: Optional[int] = None, chunk: int = 0, scale: float = 0.0, diff: float = 0.3,
                       kv_from: Optional[int] = None, mlp: Optional[dict] = None) -> dict:
  m: Dict[str, Any] = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": 2 * dim if vdim is None else vdim, "scale": scale or dim**-0.5, "diff": diff}
  if kv_from is not None:
    m["kv_from"] = kv_from
  return _mixer("attention_2", m, chunk, mlp)


def latent_layer(heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, window: int = 0, rot_base: float = 10000.0,
                 rot_scaling: Optional[dict] = None, scale: float = 0.0, mlp: Optional[dict] = None) -> dict:
  m: Dict[str, Any] = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                       "rot": {"base": rot_base, "dims": rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5}
  if rot_scaling:
    m["rot"]["scaling"] = dict(rot_scaling)
  return _mixer("latent_attention", m, window, mlp)
