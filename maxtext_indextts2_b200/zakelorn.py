"""The Zakelorn design: a decoder whose config.json lists its layers one by one.

    x += s1 * ln(mixer(x), norm1);   x += s2 * ln(ff(x), norm2)          (the second part only if the layer has a feed-forward)

with ln the layer norm (weight and bias) and s1, s2 one factor per channel; both sublayers read the residual stream itself.  The
one mixer, ``parallel``, is ``left_scale * left + right_scale * right``:

* left  -- grouped-query softmax attention: interleaved rotary pairs on the leading channels, queries and keys of unit RMS per head,
           a sliding window that always keeps the sequence's first tokens, a learned sink per head in the softmax's denominator, and
           a sigmoid gate on every channel of the concatenated heads.
* right -- lightning attention: silu queries, keys and values, a matrix state per head that decays by one constant per head and
           token, unit RMS over all heads together, a sigmoid gate.

Feed-forward: ``down(gelu_tanh(up x))``, or routed silu-gated experts: softmax scores over all router outputs, chosen by score +
correction among the groups with the largest choice scores, weighted by the scores as they are; the last router outputs are
identity experts (their output is the input); a shared expert with a sigmoid gate per token.  The logits are the layer-normed stream
times the embedding table.

This module is the design's entry in the framework: config.json -> config keys (`config_keys`), checks (`validate_layer_specs`),
safetensors names -> layer descriptors of the layered engine (`model_plan`), random weights of any size (`random_tensors`).  On the
device every layer is a composite mixer under MTX_NORM_OUT_LAYER; s1, s2 are folded into the norms' weights and biases.
"""

from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

from .gugidra import TILE_ROWS, _interleave, _need, _shape, rot_frequencies

MIXERS = ("parallel",)
FF_KINDS = ("dense", "moe")


def config_keys(model: dict) -> dict:
  """config.json of a Zakelorn model -> keys of configs/base.yml."""
  layers = model["layers"]
  validate_layer_specs(layers)
  ffs = [int(f["ff"] if f.get("kind", "dense") == "dense" else f["expert"]["ff"]) for f in (l.get("mlp") for l in layers) if f]
  first = layers[0]["mixer"]["left"]
  return dict(
      base_emb_dim=int(model["width"]),
      vocab_size=int(model["vocab"]),
      base_num_decoder_layers=len(layers),
      global_parameter_scale=1,
      normalization_layer_epsilon=float(model["norm"]["eps"]),
      embedding_scale=float((model.get("embedding") or {}).get("scale", 1.0)),
      layer_specs=layers,
      # (the homogeneous keys describe the first layer; the engine reads layer_specs)
      base_num_query_heads=int(first["heads"]),
      base_num_kv_heads=int(first["kv_heads"]),
      head_dim=int(first["dim"]),
      base_mlp_dim=max(ffs) if ffs else 0,
  )


def _decays(right: dict) -> List[float]:
  d = right["decay"]
  return [float(x) for x in d] if isinstance(d, (list, tuple)) else [float(d)] * int(right["heads"])


def validate_layer_specs(specs: List[dict]) -> None:
  for i, l in enumerate(specs):
    if l.get("type") not in MIXERS:
      raise ValueError(f"layer {i}: mixer type {l.get('type')!r}; this design has {MIXERS}")
    m = l["mixer"]
    where = f"layer {i}: mixer"
    _need(m, ("left", "right", "left_scale", "right_scale"), where)
    a, r = m["left"], m["right"]
    _need(a, ("heads", "kv_heads", "dim", "vdim", "scale"), where + ".left")
    if int(a["heads"]) % int(a["kv_heads"]):
      raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
    rot = a.get("rot")
    if rot:
      _need(rot, ("base", "dims"), where + ".left.rot")
      if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(a["dim"]):
        raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
    mask = a.get("mask") or {}
    if int(mask.get("size") or 0) < 0 or int(mask.get("keep_first") or 0) < 0:
      raise ValueError(f"layer {i}: mask.size and mask.keep_first must not be negative")
    _need(r, ("heads", "dim", "vdim", "decay"), where + ".right")
    if len(_decays(r)) != int(r["heads"]):
      raise ValueError(f"layer {i}: {len(_decays(r))} decays for {r['heads']} heads")
    f = l.get("mlp")
    if f is None:
      continue
    kind = f.get("kind", "dense")
    if kind not in FF_KINDS:
      raise ValueError(f"layer {i}: feed-forward kind {kind!r}; this design has {FF_KINDS}")
    if kind == "dense":
      _need(f, ("ff",), f"layer {i}: mlp")
      continue
    _need(f, ("expert", "router"), f"layer {i}: mlp")
    q = f["router"]
    n = int(q["experts"]) + int(q.get("identity") or 0)
    g = q.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = int(g["count"]), int(g["keep"]), int(q["top"])
    if int(q["experts"]) < 1 or count < 1 or n % count or not 1 <= keep <= count:
      raise ValueError(f"layer {i}: {n} router outputs in {count} groups of which {keep} are kept")
    if not 1 <= top <= keep * (n // count):
      raise ValueError(f"layer {i}: top {top} of {keep * (n // count)} experts in the kept groups")


def layer_plan(config, tensors: Dict[str, torch.Tensor], i: int) -> Dict[str, Any]:
  """What layer i hands to the layered engine: sizes and scalars (python numbers) and host tensors; matrices keep their stored
  dtype.  All projections of the mixer's input are one matrix in the order the device reads them, and so are the two output
  projections (the two scales multiply the activations that enter it)."""
  spec = config.layer_specs[i]
  E = int(config.emb_dim)
  t, p, m = tensors, f"l{i}.", spec["mixer"]
  dev = tensors["embed"].device
  mat = lambda name, shape: _shape(t[name], shape, name)
  f32 = lambda name, shape: _shape(t[name].to(torch.float32), shape, name)
  plan: Dict[str, Any] = dict(mixer="composite", norm_style="out_layer", moe=None, ff_kind="none", ff=0)

  def norm(n: str, scale: str, weight_key: str, bias_key: str) -> None:
    s = f32(p + scale, (E,))
    plan[weight_key], plan[bias_key] = f32(p + n, (E,)) * s, f32(p + n + ".b", (E,)) * s

  norm("norm1", "ls1", "norm1", "norm1b")
  a, r, q = m["left"], m["right"], p + "mix.left."
  H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
  rot, mask = a.get("rot"), a.get("mask") or {}
  rd, size = int(rot["dims"]) if rot else 0, int(mask.get("size") or 0)
  ones = torch.ones(d, dtype=torch.float32, device=dev)
  plan["attn"] = dict(heads=H, kv_heads=G, dim=d, vdim=dv, window=size, keep_first=int(mask.get("keep_first") or 0) if size else 0, rot_dims=rd, rot_half=0,
                      values_are_keys=0, value_gate=1, scale=float(a["scale"]), out_scale=float(m["left_scale"]),
                      rot_freq=rot_frequencies(rd, float(rot["base"])) if rd else None, sink=f32(q + "sink", (H,)),
                      q_norm=ones, k_norm=ones)  # (a rotation leaves a head's RMS as it is: the device norms first)
  rows = [mat(q + "q", (H * d, E)), mat(q + "k", (G * d, E)), mat(q + "v", (G * dv, E)), mat(q + "g", (H * dv, E))]
  wo = [mat(q + "o", (E, H * dv))]
  q = p + "mix.right."
  H, d, dv = int(r["heads"]), int(r["dim"]), int(r["vdim"])
  plan["rec"] = dict(kind="decay", heads=H, dim=d, vdim=dv, decay_rank=0, gate_silu=0, q_scale=1.0, tau=1.0, gate_cap=0.0, denom_eps=0.0,
                     out_scale=float(m["right_scale"]), norm_whole=1, out_norm=f32(q + "norm", (H * dv,)),
                     head_decay=torch.tensor(_decays(r), dtype=torch.float32, device=dev))
  rows += [mat(q + "q", (H * d, E)), mat(q + "k", (H * d, E)), mat(q + "v", (H * dv, E)), mat(q + "g", (H * dv, E))]
  wo.append(mat(q + "o", (E, H * dv)))
  w_in = torch.cat(rows, dim=0)
  pad = (-w_in.shape[0]) % TILE_ROWS
  if pad and E % 64 == 0:  # zero rows up to a whole tile of the tensor-core GEMM
    w_in = torch.cat([w_in, torch.zeros(pad, E, dtype=w_in.dtype, device=dev)], dim=0)
  plan.update(w_in=w_in, n_in=int(w_in.shape[0]), wo=torch.cat(wo, dim=1))
  f = spec.get("mlp")
  if f is None:
    return plan
  norm("norm2", "ls2", "norm2", "norm2b")
  q = p + "mlp."
  if f.get("kind", "dense") == "dense":
    F = int(f["ff"])
    plan.update(ff_kind="gelu_up", ff=F, w_gate_up=mat(q + "up", (F, E)), w_down=mat(q + "down", (E, F)))
    return plan

  def gated(prefix: str, F: int):
    return _interleave(mat(prefix + "gate", (F, E)), mat(prefix + "up", (F, E))), mat(prefix + "down", (E, F))

  router, shared = f["router"], f.get("shared")
  n, ident, F = int(router["experts"]), int(router.get("identity") or 0), int(f["expert"]["ff"])
  groups = router.get("groups") or {"count": 1, "keep": 1}
  experts = [gated(f"{q}e{e}.", F) for e in range(n)]
  w_router = mat(q + "router", (n + ident, E))
  moe = dict(experts=n, identity=ident, top=int(router["top"]), groups=int(groups["count"]), keep_groups=int(groups["keep"]), groups_max=1, ff=F, limit=0.0,
             shared_ff=0, shared_limit=0.0, act_silu=1, score_softmax=1, plain_weights=1, correction=f32(q + "correction", (n + ident,)),
             w_gate_up=torch.stack([g for g, _ in experts]), w_down=torch.stack([dn for _, dn in experts]), shared_gate_up=None, shared_down=None)
  if shared:
    gu, dn = gated(q + "shared.", int(shared["ff"]))
    moe.update(shared_ff=int(shared["ff"]), shared_gate_up=gu, shared_down=dn, shared_gate=1)
    w_router = torch.cat([w_router, mat(q + "shared.sg", (1, E))], dim=0)  # (the gate's row rides on the router's product)
  plan.update(ff_kind="moe", moe=dict(moe, w_router=w_router))
  return plan


def model_plan(config, tensors: Dict[str, torch.Tensor]) -> Dict[str, Any]:
  E, V = int(config.emb_dim), int(config.vocab_size)
  final = lambda n: _shape(tensors[n].to(torch.float32), (E,), n)
  return dict(embedding=_shape(tensors["embed"], (V, E), "embed"), head=tensors["embed"], final_gain=1.0, final_norm=final("final.norm"),
              final_norm_b=final("final.norm.b"), embed_scale=float(config.embedding_scale), layers=[layer_plan(config, tensors, i) for i in range(len(config.layer_specs))])


def random_tensors(config, seed: int = 0, device: Any = "cpu") -> Dict[str, torch.Tensor]:
  """Random bf16 weights with the design's tensor names, for `config` (tests, benchmarks and smoke runs; made on `device`)."""
  g = torch.Generator(device=device).manual_seed(seed)
  E, V = int(config.emb_dim), int(config.vocab_size)

  def rn(*shape, std=1.0, mean=0.0):
    return (torch.randn(tuple(shape), generator=g, device=device) * std + mean).to(torch.bfloat16)

  lin = lambda n_, k: rn(n_, k, std=1.0 / math.sqrt(k))
  t = {"embed": rn(V, E, std=1.0 / float(config.embedding_scale))}

  def norm(name: str) -> None:
    t[name], t[name + ".b"] = rn(E, std=0.1, mean=1.0), rn(E, std=0.1)

  def heads(q: str, names) -> None:
    for n_, r in names:
      t[q + n_] = lin(r, E)

  norm("final.norm")
  for i, l in enumerate(config.layer_specs):
    p, a, r = f"l{i}.", l["mixer"]["left"], l["mixer"]["right"]
    norm(p + "norm1")
    t[p + "ls1"] = rn(E, std=0.1, mean=0.7)
    H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
    q = p + "mix.left."
    heads(q, (("q", H * d), ("k", G * d), ("v", G * dv), ("g", H * dv)))
    t[q + "o"], t[q + "sink"] = lin(E, H * dv), rn(H)
    H, d, dv = int(r["heads"]), int(r["dim"]), int(r["vdim"])
    q = p + "mix.right."
    heads(q, (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)))
    t[q + "o"], t[q + "norm"] = lin(E, H * dv), rn(H * dv, std=0.1, mean=1.0)
    f = l.get("mlp")
    if not f:
      continue
    norm(p + "norm2")
    t[p + "ls2"] = rn(E, std=0.1, mean=0.7)
    q = p + "mlp."
    if f.get("kind", "dense") == "dense":
      t[q + "up"], t[q + "down"] = lin(int(f["ff"]), E), lin(E, int(f["ff"]))
      continue
    names = [(f"{q}e{e}.", int(f["expert"]["ff"])) for e in range(int(f["router"]["experts"]))]
    if f.get("shared"):
      names.append((q + "shared.", int(f["shared"]["ff"])))
      t[q + "shared.sg"] = lin(1, E)
    for x, F in names:
      t[x + "gate"], t[x + "up"], t[x + "down"] = lin(F, E), lin(F, E), lin(E, F)
    n = int(f["router"]["experts"]) + int(f["router"].get("identity") or 0)
    t[q + "router"], t[q + "correction"] = rn(n, E, std=1.5 / math.sqrt(E)), rn(n, std=0.5 / n)
  return t


# -- config.json-shaped dicts (tests, benchmarks) ----------------------------------------------------------------------------


def model_dict(width: int, vocab: int, layers: List[dict], eps: float = 1e-6, embed_scale: float = 1.0) -> dict:
  return {"architecture": "Zakelorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}


def dense_ff(ff: int) -> dict:
  return {"kind": "dense", "ff": ff}


def moe_ff(experts: int, top: int, ff: int, identity: int = 0, groups: int = 1, keep: int = 1, shared_ff: int = 0) -> dict:
  out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}}
  if shared_ff:
    out["shared"] = {"ff": shared_ff}
  return out


def attention_part(heads: int, kv_heads: int, dim: int, vdim: Optional[int] = None, window: int = 0, keep_first: int = 0, scale: float = 0.0,
                   rot_dims: Optional[int] = None, rot_base: float = 10000.0) -> dict:
  a: Dict[str, Any] = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim if vdim is None else vdim, "scale": scale or dim**-0.5}
  rd = dim if rot_dims is None else rot_dims
  if rd:
    a["rot"] = {"base": rot_base, "dims": rd}
  if window:
    a["mask"] = {"size": window, "keep_first": keep_first}
  return a


def lightning_part(heads: int, dim: int, vdim: Optional[int] = None, decay: Optional[List[float]] = None) -> dict:
  if decay is None:  # half-lives from two tokens to a thousand
    decay = [2.0 ** (-1.0 / 2.0 ** (1.0 + 9.0 * h / max(1, heads - 1))) for h in range(heads)]
  return {"heads": heads, "dim": dim, "vdim": dim if vdim is None else vdim, "decay": list(decay)}


def parallel_layer(left: dict, right: dict, left_scale: float = 1.0, right_scale: float = 1.0, mlp: Optional[dict] = None) -> dict:
  return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}
