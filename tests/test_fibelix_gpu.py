"""The Fibelix design on the layered engine against the plain restatement in oracle/fibelix_ref.py (numpy float64, same weights).

Small configurations with random weights; where random weights would hide a fault (a far key among hundreds, the one in a softmax's
denominator, a chunk's or a window's edge) the weights are made so that it shows, and the oracle is told to make that fault to
prove it.  float32 engines are compared tightly, bfloat16 ones within rounding.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from maxtext_indextts2_b200 import fibelix as fx
from maxtext_indextts2_b200 import maxengine, pyconfig
from oracle import fibelix_ref as ref

pytestmark = pytest.mark.gpu

TIGHT = 3e-5
LOOSE = 3e-2
DTYPES = pytest.mark.parametrize("dtype,tol", [("float32", TIGHT), ("bfloat16", LOOSE)])


def as_torch(t):
  return {k: torch.from_numpy(np.asarray(v)).to(torch.bfloat16) for k, v in t.items()}


def make_engine(cfg_dict, tensors, dtype="float32", slots=4, tokens_per_page=4, num_pages=60, max_len=200, **kw):
  config = pyconfig.from_model_dict(cfg_dict, dtype=dtype, per_device_batch_size=slots, max_target_length=max_len,
                                    pagedattn_tokens_per_page=tokens_per_page, pagedattn_num_pages=num_pages, **kw)
  engine = maxengine.MaxEngine(config)
  engine.load_params(as_torch(tensors))
  engine.init_decode_state()
  return engine


def tokens_for(cfg_dict, n, seed=5):
  return np.random.Generator(np.random.PCG64(seed)).integers(0, cfg_dict["vocab"], size=n).tolist()


def rel_err(got, want):
  got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
  return float(np.abs(got - want).max() / np.abs(want).max())


def rms_err(got, want):
  got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
  return float(np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want**2).mean()))


def error(dtype):
  return rel_err if dtype == "float32" else rms_err


def whole(engine, toks, slot=0):
  out = engine.step([(slot, toks, list(range(len(toks))))]).cpu().numpy()
  engine.release_pages(slot)
  return out


def in_portions(engine, toks, cuts, slot=1, decode=0):
  """The sequence fed in portions of `cuts` tokens, then `decode` tokens one by one; every position's logits."""
  got, at = [], 0
  for c in cuts:
    got.append(engine.step([(slot, toks[at : at + c], list(range(c)))]).cpu().numpy())
    at += c
  got += [engine.step([(slot, [tok], [0])]).cpu().numpy() for tok in toks[at : at + decode]]
  engine.release_pages(slot)
  return np.concatenate(got)


YARN = {"factor": 3.0, "original": 90, "fast": 8.0, "slow": 0.5}


def tlk(mlp=None, **kw):
  args = dict(heads=4, kv_heads=2, dim=12, vdim=20, chunk=11, scale=0.31, rot_dims=8, rot_base=50.0, rot_factor=5.0)
  args.update(kw)
  return fx.talking_layer(mlp=mlp, **args)


def dif(mlp=None, **kw):
  args = dict(heads=4, kv_heads=2, dim=10, vdim=18, chunk=13, scale=0.4, diff=0.35)
  args.update(kw)
  return fx.differential_layer(mlp=mlp, **args)


def lat(mlp=None, **kw):
  args = dict(heads=3, dim=10, rot_dim=8, vdim=14, q_rank=22, kv_rank=26, window=9, rot_base=70.0, rot_scaling=YARN, scale=0.3)
  args.update(kw)
  return fx.latent_layer(mlp=mlp, **args)


def moe(experts=5, top=2, ff=14):
  return fx.moe_ff(experts, top, ff)


def model(layers, width=40, vocab=61):
  return fx.model_dict(width, vocab, layers, eps=1e-5)


def weights(cfg, seed, toks=None):
  """Random weights; of eight seeds the one whose routers make the least close call on `toks` (no test rests on which of two
  nearly equal experts is chosen)."""
  if toks is None or not any(l.get("mlp") for l in cfg["layers"]):
    return ref.random_model(cfg, seed=seed)
  models = [ref.random_model(cfg, seed=s) for s in range(seed, seed + 8)]
  return max(models, key=lambda t: ref.closest_router_gap(cfg, t, toks))


DEFAULT = lambda: model([dif(moe()), lat(moe(4, 1, 12)), tlk(moe()), dif(moe(6, 3, 10), kv_from=0, chunk=7, heads=6, diff=0.2), lat(window=5)])

# ---- each mechanism alone ------------------------------------------------------------------------------------------------------

CASES = {
    "talking_attention": lambda: model([tlk()]),
    "talking_attention_without_chunks": lambda: model([tlk(chunk=0)]),
    "talking_attention_without_rotation": lambda: model([tlk(rot_dims=0)]),
    "talking_attention_one_kv_head": lambda: model([tlk(kv_heads=1)]),
    "talking_attention_key_heads_of_their_own": lambda: model([tlk(kv_heads=4)]),
    "chunks_of_one": lambda: model([tlk(chunk=1), dif(chunk=1)]),
    "differential_attention": lambda: model([dif()]),
    "differential_attention_without_chunks": lambda: model([dif(chunk=0)]),
    "shared_keys_and_values_other_chunks_and_heads": lambda: model([dif(), dif(kv_from=0, chunk=5, heads=2, diff=0.6, scale=0.2)]),
    "talking_attention_on_a_shared_cache": lambda: model([tlk(), tlk(kv_from=0, chunk=4)]),
    "latent_attention": lambda: model([lat()]),
    "latent_attention_without_window": lambda: model([lat(window=0)]),
    "latent_attention_without_scaling": lambda: model([lat(rot_scaling=None)]),
    "window_of_one": lambda: model([lat(window=1)]),
    "routed_feed_forward": lambda: model([lat(moe())]),
    "routed_feed_forward_every_expert_chosen": lambda: model([tlk(moe(3, 3, 12))]),
    "all_mixers": DEFAULT,
}


def _without_kv_from_in_talking(cfg):
  return not any(l["type"] == "attention" and l["mixer"].get("kv_from") is not None for l in cfg["layers"])


@DTYPES
@pytest.mark.parametrize("case", sorted(CASES))
def test_each_mechanism_alone(case, dtype, tol):
  cfg = CASES[case]()
  toks = tokens_for(cfg, 37)
  if _without_kv_from_in_talking(cfg):
    t = weights(cfg, 11, toks)
    want = ref.forward(cfg, t, toks)
  else:  # (a layer of its own keys and values: the same weights twice, the second layer reading the first one's cache of equal input)
    base = model([cfg["layers"][0]])
    t = ref.random_model(base, seed=11)
    t["l0.mix.o"], t["l0.mix.o.b"] = t["l0.mix.o"] * 0.0, t["l0.mix.o.b"] * 0.0  # the first layer leaves the stream as it is
    two = ref.random_model(model([cfg["layers"][0], tlk(chunk=4)]), seed=12)
    t.update({k: v for k, v in two.items() if k.startswith("l1.")})
    t["l1.norm1"] = t["l0.norm1"]
    for n in ("k", "v", "k.b", "v.b"):
      t["l1.mix." + n] = t["l0.mix." + n]
    want = ref.forward(model([cfg["layers"][0], tlk(chunk=4)]), t, toks)
    for n in ("k", "v", "k.b", "v.b"):
      del t["l1.mix." + n]
  engine = make_engine(cfg, t, dtype=dtype)
  assert error(dtype)(whole(engine, toks), want) < tol
  assert error(dtype)(in_portions(engine, toks, [9, 2, 17], decode=9), want) < tol


# ---- schedules: the logits of a position do not depend on how it got there --------------------------------------------------------

def test_prefill_equals_token_by_token_decoding():
  cfg = DEFAULT()
  toks = tokens_for(cfg, 45)
  t = weights(cfg, 1, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t)
  first = whole(engine, toks)
  assert rel_err(first, want) < TIGHT
  rows = in_portions(engine, toks, [], decode=len(toks))
  assert rel_err(rows, want) < TIGHT
  assert rel_err(rows, first) < 1e-5


@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 5, 16, 17, 15], [7, 1, 1, 2, 33, 18], [1, 61], [16, 16, 30], [31, 31]])
def test_portions_of_any_size(sizes):
  cfg = DEFAULT()
  toks = tokens_for(cfg, sum(sizes))
  t = weights(cfg, 2, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, tokens_per_page=8)
  assert rel_err(in_portions(engine, toks, sizes, slot=2), want) < TIGHT


@DTYPES
def test_a_step_longer_than_the_engine_takes_at_once_runs_in_slices(dtype, tol):
  cfg = DEFAULT()
  toks = {0: tokens_for(cfg, 50, seed=1), 1: tokens_for(cfg, 27, seed=2)}
  t = weights(cfg, 4, toks[0] + toks[1])
  engine = make_engine(cfg, t, dtype=dtype, max_step_rows=19)  # slices cut both runs
  out = engine.step([(s, v, list(range(len(v)))) for s, v in toks.items()]).cpu().numpy()
  want = np.concatenate([ref.forward(cfg, t, v) for v in toks.values()])
  assert rms_err(out, want) < tol


@DTYPES
def test_unequal_requests_in_one_batch_equal_each_alone_and_freed_slots_and_pages_are_reused(dtype, tol):
  cfg = DEFAULT()
  lens = {"a": 43, "b": 9, "c": 1, "d": 14, "e": 37, "f": 6}
  toks = {k: tokens_for(cfg, n, seed=ord(k)) for k, n in lens.items()}
  t = weights(cfg, 3, sum(toks.values(), []))
  want = {k: ref.forward(cfg, t, v) for k, v in toks.items()}
  # 19 usable pages of 4 tokens: a + b + c + d take 11 + 3 + 1 + 4; e and f only fit into pages that were given back
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=4, num_pages=20, max_len=64)
  got, at = {k: [] for k in toks}, {k: 0 for k in toks}
  slot_of = {"a": 0, "b": 1, "c": 2, "d": 3}
  plan = [
      [("a", 5), ("b", 2), ("c", 1), ("d", 3)],
      [("a", 1), ("b", 7), ("d", 1)],
      [("a", 19), ("d", 10)],
      [("a", 1), ("e", 4), ("f", 2)],
      [("a", 17), ("e", 1), ("f", 4)],
      [("e", 32)],
  ]
  for step in plan:
    for k, _ in step:
      if k not in slot_of:
        done = [r for r, s in slot_of.items() if at[r] == lens[r]]
        slot_of[k] = slot_of.pop(done[0])
    out = engine.step([(slot_of[k], toks[k][at[k] : at[k] + n], list(range(n))) for k, n in step]).cpu().numpy()
    for k, n in step:
      got[k].append(out[:n])
      out = out[n:]
      at[k] += n
      if at[k] == lens[k]:
        engine.release_pages(slot_of[k])
  for k in toks:
    assert at[k] == lens[k]
    assert error(dtype)(np.concatenate(got[k]), want[k]) < (tol if dtype == "float32" else 2 * tol), k  # (single requests of few rows)


def test_pool_exhaustion_is_an_error_not_a_wrong_answer():
  cfg = DEFAULT()
  t = weights(cfg, 3)
  engine = make_engine(cfg, t, tokens_per_page=4, num_pages=5, max_len=64)
  engine.step([(0, tokens_for(cfg, 10), [9])])
  with pytest.raises(ValueError):
    engine.step([(1, tokens_for(cfg, 9), [8])])


@DTYPES
def test_long_decoding_across_many_pages(dtype, tol):
  cfg = DEFAULT()
  toks = tokens_for(cfg, 150)
  t = weights(cfg, 6, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=4, num_pages=50)
  assert error(dtype)(in_portions(engine, toks, [5], slot=3, decode=145), want) < tol


def test_first_tokens_of_a_sequence():
  cfg = DEFAULT()
  t = weights(cfg, 9)
  engine = make_engine(cfg, t)
  for n in (1, 2, 3, 4):
    toks = tokens_for(cfg, n, seed=n)
    assert rel_err(whole(engine, toks), ref.forward(cfg, t, toks)) < TIGHT
    assert rel_err(in_portions(engine, toks, [], decode=n), ref.forward(cfg, t, toks)) < TIGHT


# ---- far keys, edges of chunks and windows, the denominator, page borders ----------------------------------------------------------------

def _peaky(cfg, seed, toks, times):
  """Scores that spread widely, so that single keys (also far ones, also the key at an edge) carry most of a query's weight."""
  t = weights(cfg, seed, toks)
  for i, l in enumerate(cfg["layers"]):
    p = f"l{i}.mix."
    name = {"attention": "temp", "attention_2": "q", "latent_attention": "uq"}[l["type"]]
    t[p + name] = ref.bf16_values(t[p + name] * times)
  return t


@pytest.mark.parametrize("page", [4, 16, 64])
def test_far_keys_and_page_borders(page):
  cfg = model([tlk(chunk=0), dif(moe(), chunk=0), lat(window=0), tlk(chunk=200), dif(chunk=150, kv_from=1)])
  n = 330
  toks = tokens_for(cfg, n)
  t = _peaky(cfg, 21, toks, 4.0)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, tokens_per_page=page, num_pages=700 // page + 2, max_len=400)
  assert rel_err(whole(engine, toks), want) < 2 * TIGHT
  # a prompt that ends at, one before and one after a page border, then decoding across the next borders
  for cut in (2 * page - 1, 2 * page, 2 * page + 1):
    assert rel_err(in_portions(engine, toks, [cut], decode=page + 3), want[: cut + page + 3]) < 2 * TIGHT, cut
  # far keys seen from decoded tokens
  got = [engine.step([(2, toks[:310], [])]).cpu().numpy()] + [engine.step([(2, [tok], [0])]).cpu().numpy() for tok in toks[310:]]
  assert rel_err(np.concatenate(got[1:]), want[310:]) < 2 * TIGHT


def test_the_far_past_matters_in_these_tests():
  """The check that the test above would see a lost far key: the oracle fed only the last 100 tokens (a whole number of chunks
  further on) differs clearly in every layer kind."""
  for layers in ([tlk(chunk=0)], [dif(chunk=0)], [lat(window=0)], [tlk(chunk=230)], [dif(chunk=230)]):
    cfg = model(layers)
    toks = tokens_for(cfg, 330)
    t = _peaky(cfg, 21, toks, 4.0)
    cut = slice(230, 330) if not layers[0]["mixer"].get("mask") else slice(130, 230)  # (chunks: inside the first one)
    assert rms_err(ref.forward(cfg, t, toks[cut])[-20:], ref.forward(cfg, t, toks)[cut][-20:]) > 1e-2, layers[0]["type"]


@DTYPES
@pytest.mark.parametrize("kind,size", [(k, s) for k in ("talking", "differential", "latent") for s in (1, 2, 7, 16, 33, 64, 70)])
def test_keys_just_inside_and_just_outside_a_chunk_or_window(kind, size, dtype, tol):
  """Peaky scores: a query's weight often sits on the oldest key it may see.  The oracle with a chunk or a window one token longer or
  shorter, or with chunks counted from the second token, gives clearly different logits, so an edge that is one off would show; the
  engine agrees with the exact one over a whole prompt, over portions that end around the edges, and decoding across them."""
  if kind == "talking":
    layer = tlk(heads=4, kv_heads=2, dim=16, vdim=16, chunk=size)
    hooks = [{"size": 1}, {"size": -1}, {"shift": 1}]
  elif kind == "differential":
    layer = dif(heads=4, kv_heads=2, dim=16, vdim=32, chunk=size)
    hooks = [{"size": 1}, {"size": -1}]
  else:
    layer = lat(heads=4, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=24, window=size)
    hooks = [{"size": 1}, {"size": -1}]
  cfg = model([layer] if kind != "latent" else [layer, lat(window=size, heads=2, dim=12, rot_dim=4, vdim=16, q_rank=20, kv_rank=20)])
  n = 3 * size + 40
  toks = tokens_for(cfg, n, seed=size)
  t = _peaky(cfg, 30 + size, toks, 6.0 if kind == "latent" else 3.0)
  want = ref.forward(cfg, t, toks)
  for hook in hooks:
    if size + hook.get("size", 0) < 1 or (size == 1 and "shift" in hook):
      continue
    bad = ref.forward(cfg, t, toks, hooks={i: hook for i in range(len(cfg["layers"]))})
    assert rms_err(bad[size:], want[size:]) > 2 * LOOSE, hook
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=8, num_pages=80, max_len=320)
  err = error(dtype)
  assert err(whole(engine, toks), want) < tol
  for cuts in ([size - 1, 1, 1, size, 2], [size, size + 1, size - 1], [2 * size - 1, 2, size], [size + 1, 2 * size - 2, 3]):
    cuts = [c for c in cuts if c > 0]
    d = min(size + 5, n - sum(cuts))
    assert err(in_portions(engine, toks, cuts, decode=d), want[: sum(cuts) + d]) < tol, cuts


@DTYPES
def test_every_part_of_the_scores_shows(dtype, tol):
  """The one in the denominator, the temperatures, the mixing of the heads' scores, the second map, the rotation's amplitude: the
  oracle without each of them is clearly elsewhere."""
  cfg = model([tlk(heads=4, kv_heads=2, dim=16, vdim=16), dif(heads=4, kv_heads=2, dim=16, vdim=32), lat()])
  toks = tokens_for(cfg, 70)
  t = weights(cfg, 40, toks)
  t["l0.mix.q.b"], t["l0.mix.k.b"] = ref.bf16_values(t["l0.mix.q.b"] * 0.3), ref.bf16_values(t["l0.mix.k.b"] * 0.3)
  t["l2.mix.uq"] = ref.bf16_values(t["l2.mix.uq"] * 3.0)
  want = ref.forward(cfg, t, toks)
  for i, hook in ((0, "no_sink"), (0, "no_talk"), (0, "no_temp"), (1, "one_map"), (2, "no_amp")):
    assert rms_err(ref.forward(cfg, t, toks, hooks={i: {hook: True}}), want) > 0.04, hook
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=16, num_pages=20)
  assert error(dtype)(whole(engine, toks), want) < tol
  assert error(dtype)(in_portions(engine, toks, [50], decode=20), want) < tol


@DTYPES
def test_a_denominator_that_outweighs_the_keys(dtype, tol):
  cfg = model([tlk(heads=4, kv_heads=1, dim=16, vdim=16, chunk=40)])
  toks = tokens_for(cfg, 60)
  t = weights(cfg, 44, toks)
  # every head's scores far below zero: the mixing takes minus the sum of the heads' scores, all keys look alike and like the queries
  t["l0.mix.talk"] = np.full((4, 4), -1.0)
  t["l0.mix.q.b"], t["l0.mix.k.b"] = np.full(64, 1.0), np.full(16, 1.0)
  t["l0.mix.q"], t["l0.mix.k"] = ref.bf16_values(t["l0.mix.q"] * 0.2), ref.bf16_values(t["l0.mix.k"] * 0.2)
  t["l0.mix.v"] = ref.bf16_values(t["l0.mix.v"] * 2e6)
  cfg["layers"][0]["mixer"]["scale"] = 0.2
  del cfg["layers"][0]["mixer"]["rot"]
  want = ref.forward(cfg, t, toks)
  assert rms_err(ref.forward(cfg, t, toks, hooks={0: {"no_sink": True}}), want) > 0.5
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=16, num_pages=20)
  assert error(dtype)(whole(engine, toks), want) < 2 * tol
  assert error(dtype)(in_portions(engine, toks, [30], decode=30), want) < 2 * tol


# ---- other sizes ------------------------------------------------------------------------------------------------------------------

SIZES = {
    "odd_width": lambda: model([dif(moe(7, 3, 9)), tlk(moe()), lat()], width=37, vocab=47),
    "one_head_everywhere": lambda: model([dif(heads=1, kv_heads=1), tlk(heads=1, kv_heads=1), lat(heads=1)]),
    "heads_with_kv_heads_of_their_own": lambda: model([dif(kv_heads=4), tlk(kv_heads=4), lat(heads=4)]),
    "many_heads_on_one_key_head": lambda: model([tlk(heads=10, kv_heads=1, dim=8, vdim=8), dif(heads=9, kv_heads=1, dim=8, vdim=8), lat(heads=10)]),
    "three_and_five_key_heads": lambda: model([tlk(heads=6, kv_heads=3, dim=16, vdim=24), dif(heads=6, kv_heads=3, dim=8, vdim=24), tlk(heads=5, kv_heads=5, dim=8, vdim=16),
                                               dif(heads=10, kv_heads=5, dim=16, vdim=8)]),
    "three_query_heads_per_key_head": lambda: model([tlk(heads=9, kv_heads=3, dim=16, vdim=16), dif(heads=9, kv_heads=3, dim=8, vdim=16), dif(heads=15, kv_heads=3, dim=8, vdim=16)]),
    "one_expert": lambda: model([lat(moe(1, 1, 12)), tlk(moe(2, 2, 8))]),
    "value_size_over_key_size": lambda: model([tlk(dim=8, vdim=40), dif(dim=8, vdim=72)]),
    "key_size_over_value_size": lambda: model([tlk(dim=40, vdim=8, rot_dims=40), dif(dim=40, vdim=8)]),
    "rotation_of_two_channels": lambda: model([tlk(rot_dims=2), lat(rot_dim=2)]),
    "rotation_of_every_channel": lambda: model([tlk(rot_dims=12, rot_factor=1.0)]),
    "no_rotated_part": lambda: model([lat(rot_dim=0)]),
    "latent_sizes": lambda: model([lat(dim=4, rot_dim=12, vdim=30, q_rank=5, kv_rank=7), lat(heads=5, dim=20, rot_dim=6, vdim=3, q_rank=50, kv_rank=44)]),
    "wide_heads": lambda: model([dif(heads=2, kv_heads=1, dim=72, vdim=200), tlk(heads=4, kv_heads=4, dim=96, vdim=136, rot_dims=64), lat(heads=2, kv_rank=120, rot_dim=24)], width=64),
    "very_wide_scores": lambda: model([tlk(heads=6, kv_heads=6, dim=64, vdim=264, rot_dims=64), tlk(heads=3, kv_heads=3, dim=184, vdim=48, rot_dims=20)], width=48),
    "shared_cache_two_layers_back": lambda: model([dif(moe()), lat(), dif(kv_from=0, chunk=30), dif(kv_from=0, chunk=2)]),
    "layers_without_feed_forward": lambda: model([dif(), tlk(), lat()]),
    "many_experts_top_one": lambda: model([lat(moe(40, 1, 6))]),
    "more_than_64_experts": lambda: model([lat(moe(72, 5, 6)), tlk(moe(128, 4, 8))], width=64),
    "chunk_and_window_longer_than_the_sequence": lambda: model([dif(chunk=100), tlk(chunk=64), lat(window=99)]),
    "the_same_kind_twice_with_other_sizes": lambda: model([tlk(), tlk(heads=3, kv_heads=3, dim=6, vdim=9, chunk=5, rot_dims=4), dif(), dif(heads=2, kv_heads=2, dim=7, vdim=5, diff=0.8)]),
}


@DTYPES
@pytest.mark.parametrize("case", sorted(SIZES))
def test_other_sizes(case, dtype, tol):
  # (bfloat16: sizes that are not multiples of eight take the unvectorised loads of the projections and the row kernel of the attention)
  cfg = SIZES[case]()
  toks = tokens_for(cfg, 41)
  t = weights(cfg, 13, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=8)
  assert error(dtype)(in_portions(engine, toks, [22, 17], slot=0, decode=2), want) < tol


def test_sizes_made_of_whole_tensor_core_tiles_on_a_bfloat16_engine():
  cfg = model([dif(moe(8, 2, 128), heads=4, kv_heads=2, dim=32, vdim=64, chunk=48), lat(moe(8, 2, 64), heads=4, dim=32, rot_dim=32, vdim=64, q_rank=64, kv_rank=64, window=24),
               tlk(moe(4, 2, 128), heads=4, kv_heads=2, dim=64, vdim=64, chunk=40, rot_dims=32), dif(moe(8, 3, 64), heads=8, kv_heads=2, dim=32, vdim=64, chunk=20, kv_from=0)],
              width=128, vocab=256)
  toks = tokens_for(cfg, 90)
  t = weights(cfg, 15, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype="bfloat16", tokens_per_page=16, num_pages=30)
  assert rms_err(whole(engine, toks), want) < LOOSE
  assert rms_err(in_portions(engine, toks, [70], decode=20), want) < LOOSE


# ---- the tensor-core attention kernels over mixed schedules (bf16, head sizes in multiples of eight) -------------------------------------

SHAPES = {
    "talking_4x64_on_2": lambda: tlk(heads=4, kv_heads=2, dim=64, vdim=64, chunk=70, rot_dims=32),
    "talking_8x32_on_1": lambda: tlk(heads=8, kv_heads=1, dim=32, vdim=32, chunk=100, rot_dims=32),
    "talking_16x32_on_4_values_96": lambda: tlk(heads=16, kv_heads=4, dim=32, vdim=96, chunk=64, rot_dims=16),
    "talking_12x24_on_6_values_40": lambda: tlk(heads=12, kv_heads=6, dim=24, vdim=40, chunk=33, rot_dims=12),
    "talking_20x16_on_2": lambda: tlk(heads=20, kv_heads=2, dim=16, vdim=16, chunk=90, rot_dims=16),
    "talking_6x128_on_3_values_256": lambda: tlk(heads=6, kv_heads=3, dim=128, vdim=256, chunk=80, rot_dims=64),
    "talking_8x128_on_8_values_128": lambda: tlk(heads=8, kv_heads=8, dim=128, vdim=128, chunk=80, rot_dims=64),
    "differential_4x32_on_2": lambda: dif(heads=4, kv_heads=2, dim=32, vdim=64, chunk=70),
    "differential_16x16_on_1": lambda: dif(heads=16, kv_heads=1, dim=16, vdim=32, chunk=128),
    "differential_3x56_on_3_values_112": lambda: dif(heads=3, kv_heads=3, dim=56, vdim=112, chunk=100),
    "differential_12x40_on_4_values_56": lambda: dif(heads=12, kv_heads=4, dim=40, vdim=56, chunk=37),
    "differential_10x8_on_2_values_24": lambda: dif(heads=10, kv_heads=2, dim=8, vdim=24, chunk=64),
    "differential_2x128_on_1_values_256": lambda: dif(heads=2, kv_heads=1, dim=128, vdim=256, chunk=90),
    "latent_rows_of_40": lambda: lat(heads=4, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, window=50),
    "latent_rows_of_104": lambda: lat(heads=9, dim=24, rot_dim=24, vdim=32, q_rank=24, kv_rank=80, window=70),
    "latent_rows_of_128": lambda: lat(heads=5, dim=24, rot_dim=16, vdim=24, q_rank=48, kv_rank=112, window=33),
    "latent_rows_of_192": lambda: lat(heads=3, dim=32, rot_dim=64, vdim=32, q_rank=48, kv_rank=128, window=0),
}


@pytest.mark.parametrize("page", [16, 24])
@pytest.mark.parametrize("shape", sorted(SHAPES))
def test_tensor_core_attention_shapes_and_schedules(shape, page):
  """Every instantiation of the tensor-core kernels: prompts in portions that end inside, at and after the key tiles, query tiles
  that start anywhere, several sequences whose tiles sit side by side in one work item, then single tokens."""
  cfg = model([SHAPES[shape]()], width=64, vocab=90)
  n = 150
  toks = tokens_for(cfg, n, seed=len(shape))
  t = _peaky(cfg, len(shape), toks, 1.5)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype="bfloat16", tokens_per_page=page, num_pages=4 * (n // page + 2) + 2, max_len=n + 8)
  assert rms_err(whole(engine, toks), want) < LOOSE
  for cuts in ([63, 1, 1, 30, 33], [64, 64], [65, 5, 58, 9], [31, 2, 31, 33, 7, 25]):
    assert rms_err(in_portions(engine, toks, cuts, decode=12), want[: sum(cuts) + 12]) < LOOSE, cuts
  # sequences side by side: in the middle of a prompt, at its start, decoding
  engine.step([(0, toks[:70], []), (2, toks[:101], []), (3, toks[:5], [])])
  out = engine.step([(0, toks[70:90], list(range(20))), (1, toks[:37], list(range(37))), (2, [toks[101]], [0]), (3, toks[5:7], [0, 1])]).cpu().numpy()
  assert rms_err(out, np.concatenate([want[70:90], want[:37], want[101:102], want[5:7]])) < LOOSE
  # and all of them decoding, at very different positions
  out = engine.step([(0, [toks[90]], [0]), (1, [toks[37]], [0]), (2, [toks[102]], [0]), (3, [toks[7]], [0])]).cpu().numpy()
  assert rms_err(out, np.stack([want[90], want[37], want[102], want[7]])) < 2 * LOOSE


def test_float32_keeps_to_the_oracle_where_scores_are_large():
  """A talking attention whose mixed scores reach tens, in float32: nothing on the way may be rounded to fewer bits."""
  cfg = model([tlk(heads=8, kv_heads=4, dim=96, vdim=64, chunk=60, rot_dims=48), dif(heads=4, kv_heads=2, dim=80, vdim=64, chunk=50)])
  toks = tokens_for(cfg, 100)
  t = _peaky(cfg, 50, toks, 6.0)
  engine = make_engine(cfg, t, tokens_per_page=16, num_pages=20)
  assert rel_err(in_portions(engine, toks, [61], decode=30), ref.forward(cfg, t, toks)[:91]) < 5 * TIGHT


# ---- the framework's entry point: scheduler, sampler -------------------------------------------------------------------------------

def _greedy(cfg, t, prompt, n):
  seq = list(prompt)
  for _ in range(n):
    logits = ref.forward(cfg, t, seq)[-1]
    top2 = np.sort(logits)[-2:]
    assert float(top2[1] - top2[0]) > 1e-4, "near-tie in the test's own model; change the seed"
    seq.append(int(logits.argmax()))
  return seq[len(prompt):]


def test_greedy_generation_through_the_offline_engine():
  from maxtext_indextts2_b200 import offline_engine

  cfg = DEFAULT()
  t = weights(cfg, 17)
  config = pyconfig.from_model_dict(cfg, dtype="float32", per_device_batch_size=2, max_target_length=64, pagedattn_tokens_per_page=4,
                                    pagedattn_num_pages=30, decode_sampling_strategy="greedy")
  eng = offline_engine.OfflineEngine(config, params=as_torch(t))
  prompts = [tokens_for(cfg, n, seed=30 + n) for n in (5, 11, 3, 8, 2)]  # five prompts over two slots: slots and pages are reused
  outs = eng.batch_inference(prompts, max_decode_length=9)
  for prompt, out in zip(prompts, outs):
    assert out.token_ids.tolist() == _greedy(cfg, t, prompt, 9)


# ---- the command lines: prompts in, tokens out; a trace of batched steps replayed through bin/trace_run --------------------------------

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _write_model_dir(path, cfg, t):
  from tests.test_gugidra_host import _write_safetensors

  os.makedirs(path)
  with open(path / "config.json", "w") as f:
    json.dump(cfg, f)
  _write_safetensors(path / "model.safetensors", as_torch(t))


def test_decode_command_line_generates_the_oracles_greedy_tokens(tmp_path):
  cfg = DEFAULT()
  t = weights(cfg, 19)
  _write_model_dir(tmp_path / "model", cfg, t)
  prompts = [tokens_for(cfg, n, seed=50 + n) for n in (7, 3)]
  cmd = [sys.executable, "-m", "maxtext_indextts2_b200.decode", f"model_dir={tmp_path / 'model'}", "dtype=float32", "decode_sampling_strategy=greedy",
         "pagedattn_tokens_per_page=8", "--max-decode", "6"]
  for p in prompts:
    cmd += ["--prompt", ",".join(str(x) for x in p)]
  r = subprocess.run(cmd, capture_output=True, text=True, timeout=600, cwd=ROOT)
  assert r.returncode == 0, r.stderr[-2000:]
  outs = {d["prompt"]: d["tokens"] for d in (json.loads(l) for l in r.stdout.splitlines() if l.startswith("{"))}
  for i, prompt in enumerate(prompts):
    assert outs[i] == _greedy(cfg, t, prompt, 6)


@pytest.mark.parametrize("dtype,tol", [("float32", TIGHT), ("bfloat16", 5e-2)])  # (bfloat16: per step, some of few rows)
def test_trace_runner_replays_a_mixed_schedule(tmp_path, dtype, tol):
  cfg = DEFAULT()
  lens = {"a": 70, "b": 9, "c": 33, "d": 5, "e": 40, "f": 20}
  toks = {k: tokens_for(cfg, n, seed=ord(k)) for k, n in lens.items()}
  t = weights(cfg, 23, sum(toks.values(), []))
  model_dir = tmp_path / "model"
  _write_model_dir(model_dir, cfg, t)
  # four pages of 64 tokens: a, b, c fill them (2 + 1 + 1); d, e and f fit only into what b and c give back, and take their slots
  plan = [[("a", 30), ("b", 2)], [("a", 1), ("b", 7), ("c", 33)], [("a", 35), ("d", 2)], [("a", 1), ("d", 3), ("e", 39)], [("a", 3), ("e", 1), ("f", 20)]]
  at = {k: 0 for k in toks}
  lines, rows = [], []
  for n, step in enumerate(plan):
    entries, end = [], []
    for k, c in step:
      entries.append({"id": k, "tokens": toks[k][at[k] : at[k] + c], "want": list(range(c))})
      rows.append((n, k, at[k], c))
      at[k] += c
      if at[k] == lens[k]:
        end.append(k)
    lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
  out_dir = tmp_path / "out"
  p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype, "--out", str(out_dir), "--max-tokens", "256"],
                     input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
  assert p.returncode == 0, p.stderr[-2000:]
  assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(plan))]
  want = {k: ref.forward(cfg, t, v) for k, v in toks.items()}
  errs = []
  for n in range(len(plan)):
    got = np.fromfile(out_dir / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    exp = np.concatenate([want[k][lo : lo + c] for s, k, lo, c in rows if s == n])
    assert got.shape == exp.shape
    errs.append(rms_err(got, exp))
  assert max(errs) < tol, errs
