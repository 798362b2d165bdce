"""The Zakelorn design on the layered engine against the plain restatement in oracle/zakelorn_ref.py (numpy float64, same weights).

Small configurations with random weights; where random weights would hide a fault (a far key among hundreds, the first tokens, the
sink, a window's edge, a lost state) the configuration is made so that it shows, and the oracle is told to make that fault to prove it.
float32 engines are compared tightly, bfloat16 ones within rounding.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from maxtext_indextts2_b200 import maxengine, pyconfig
from maxtext_indextts2_b200 import zakelorn as zk
from oracle import zakelorn_ref as ref

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


def att(**kw):
  args = dict(heads=4, kv_heads=2, dim=12, vdim=20, window=11, keep_first=3, scale=0.31, rot_dims=8, rot_base=50.0)
  args.update(kw)
  return zk.attention_part(**args)


def lin(**kw):
  args = dict(heads=3, dim=10, vdim=14)
  args.update(kw)
  return zk.lightning_part(**args)


def par(left=None, right=None, mlp=None, left_scale=0.9, right_scale=1.2):
  return zk.parallel_layer(left or att(), right or lin(), left_scale, right_scale, mlp)


def moe(experts=5, top=3, ff=14, identity=3, groups=4, keep=3, shared_ff=22):
  return zk.moe_ff(experts, top, ff, identity, groups, keep, shared_ff)


def model(layers, width=40, vocab=61, embed_scale=3.0):
  return zk.model_dict(width, vocab, layers, eps=1e-5, embed_scale=embed_scale)


def weights(cfg, seed, toks=None):
  """Random weights; of thirty seeds the one whose routers make the least close call on `toks` (no test rests on which of two
  nearly equal experts or groups is chosen)."""
  if toks is None or not any((l.get("mlp") or {}).get("kind") == "moe" for l in cfg["layers"]):
    return ref.random_model(cfg, seed=seed)
  models = [ref.random_model(cfg, seed=s) for s in range(seed, seed + 30)]
  return max(models, key=lambda t: ref.closest_router_gap(cfg, t, toks))


DEFAULT = lambda: model([par(mlp=zk.dense_ff(50)), par(att(window=6, keep_first=2, heads=6, kv_heads=3), lin(heads=2, dim=7, vdim=9), moe()),
                         par(att(window=0, rot_dims=12), lin(), None), par(mlp=moe(6, 2, 10, 0, 1, 1, 0))])

# ---- each mechanism alone ------------------------------------------------------------------------------------------------------

CASES = {
    "attention": lambda: model([par(right_scale=0.0)]),
    "attention_without_rotation": lambda: model([par(att(rot_dims=0), right_scale=0.0)]),
    "attention_without_window": lambda: model([par(att(window=0), right_scale=0.0)]),
    "attention_without_kept_tokens": lambda: model([par(att(keep_first=0), right_scale=0.0)]),
    "window_of_one_and_one_kept_token": lambda: model([par(att(window=1, keep_first=1), right_scale=0.0)]),
    "more_kept_tokens_than_the_window": lambda: model([par(att(window=4, keep_first=9), right_scale=0.0)]),
    "lightning_attention": lambda: model([par(left_scale=0.0)]),
    "lightning_attention_that_forgets_nothing_or_everything": lambda: model([par(right=lin(decay=[1.0, 0.0, 0.5]), left_scale=0.0)]),
    "both_sides": lambda: model([par(left_scale=0.4, right_scale=1.7)]),
    "dense_feed_forward": lambda: model([par(mlp=zk.dense_ff(33))]),
    "experts_alone": lambda: model([par(mlp=moe(6, 2, 12, 0, 1, 1, 0))]),
    "experts_in_groups": lambda: model([par(mlp=moe(6, 2, 12, 0, 3, 2, 0))]),
    "identity_experts": lambda: model([par(mlp=moe(3, 2, 12, 3, 1, 1, 0))]),
    "shared_expert": lambda: model([par(mlp=moe(4, 1, 12, 0, 1, 1, 18))]),
    "routed_feed_forward": lambda: model([par(mlp=moe())]),
    "every_expert_chosen": lambda: model([par(mlp=moe(3, 4, 12, 1, 2, 2))]),
    "all_together": DEFAULT,
}


@DTYPES
@pytest.mark.parametrize("case", sorted(CASES))
def test_each_mechanism_alone(case, dtype, tol):
  cfg = CASES[case]()
  toks = tokens_for(cfg, 37)
  t = weights(cfg, 11, toks)
  want = ref.forward(cfg, t, toks)
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


@DTYPES
@pytest.mark.parametrize("sizes", [[2, 2, 2, 3, 5, 16, 17, 15], [7, 1, 1, 2, 33, 18], [1, 61], [16, 16, 30], [31, 31]])
def test_portions_of_any_size(sizes, dtype, tol):
  cfg = DEFAULT()
  toks = tokens_for(cfg, sum(sizes))
  t = weights(cfg, 2, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=8)
  assert error(dtype)(in_portions(engine, toks, sizes, slot=2), want) < tol


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
  engine = make_engine(cfg, weights(cfg, 3), tokens_per_page=4, num_pages=5, max_len=64)
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


# ---- far keys, edges of windows and of the kept tokens, sinks, the state, page borders -----------------------------------------------
#
# Queries and keys have unit RMS, so a large scale alone makes scores spread widely: single keys (also far ones, also the one at an
# edge) then carry most of a query's weight.


@pytest.mark.parametrize("page", [4, 16, 64])
def test_far_keys_and_page_borders(page):
  peaky = dict(dim=16, vdim=16, scale=1.0)
  cfg = model([par(att(window=0, **peaky), right_scale=0.3), par(att(window=200, keep_first=5, **peaky), mlp=moe()), par(att(window=0, **peaky), lin(decay=[0.99, 0.999, 1.0]))])
  n = 330
  toks = tokens_for(cfg, n)
  t = weights(cfg, 21, toks)
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
  """The check that the test above would see a lost far key, a lost first token or a lost state: the oracle fed only the last 100
  tokens differs clearly, for each of the three ways in which the past can be seen."""
  for layer in (par(att(window=0, dim=16, vdim=16, scale=1.0), right_scale=0.0), par(att(window=5, keep_first=4, dim=16, vdim=16, scale=1.0), right_scale=0.0),
                par(right=lin(decay=[0.99, 0.999, 1.0]), left_scale=0.0)):
    cfg = model([layer])
    toks = tokens_for(cfg, 330)
    t = weights(cfg, 21, toks)
    assert rms_err(ref.forward(cfg, t, toks[230:])[-20:], ref.forward(cfg, t, toks)[-20:]) > 3e-2


@DTYPES
@pytest.mark.parametrize("size,keep", [(1, 0), (1, 1), (2, 3), (7, 2), (16, 1), (16, 16), (33, 4), (64, 5), (70, 9), (5, 37)])
def test_keys_just_inside_and_just_outside_the_window_and_the_kept_tokens(size, keep, dtype, tol):
  """Peaky scores: a query's weight often sits on the oldest key it may see.  The oracle with a window, or with the kept tokens, one
  token longer or shorter gives clearly different logits, so an edge that is one off would show; the engine agrees with the exact one
  over a whole prompt, over portions that end around the edges, and decoding across them."""
  cfg = model([par(att(dim=16, vdim=16, window=size, keep_first=keep, scale=1.2), right_scale=0.2),
               par(att(dim=16, vdim=16, window=size, keep_first=keep, scale=1.2, heads=2, kv_heads=1), right_scale=0.2)])
  n = 3 * max(size, keep) + 40
  toks = tokens_for(cfg, n, seed=size)
  t = weights(cfg, 30 + size, toks)
  want = ref.forward(cfg, t, toks)
  for hook in ({"size": 1}, {"size": -1}, {"first": 1}, {"first": -1}):
    if size + hook.get("size", 0) < 1 or keep + hook.get("first", 0) < 0:
      continue
    bad = ref.forward(cfg, t, toks, hooks={i: {"left": hook} for i in range(2)})
    assert rms_err(bad[size:], want[size:]) > 2 * LOOSE, hook
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=8, num_pages=90, max_len=320)
  err = error(dtype)
  assert err(whole(engine, toks), want) < tol
  for cuts in ([size - 1, 1, 1, size, 2], [size, size + 1, size - 1], [keep - 1, 2, size], [keep, 1, size + keep], [keep + 1, 2 * size - 2, 3]):
    cuts = [c for c in cuts if c > 0]
    d = min(size + 5, n - sum(cuts))
    assert err(in_portions(engine, toks, cuts, decode=d), want[: sum(cuts) + d]) < tol, cuts


@DTYPES
def test_every_part_shows(dtype, tol):
  """The oracle without the sink (or with a scaled one), the kept tokens, the rotation, the unit RMS, the gates, either side, the biases of the norms, the
  layer scale, the identity experts, the groups, the correction, the shared expert's gate, or with renormalised weights is clearly elsewhere."""
  cfg = model([par(att(dim=16, vdim=16, scale=0.5), mlp=moe(5, 3, 14, 3, 4, 2)), par(att(dim=16, vdim=16, scale=0.5))])
  toks = tokens_for(cfg, 70)
  t = weights(cfg, 70, toks)
  t["l0.mix.left.sink"] = np.array([3.0, 2.5, 4.0, 3.5])
  t["l0.ls2"] = t["l0.ls2"] * 2.0
  want = ref.forward(cfg, t, toks)
  for hook in ([{"left": {k: True}} for k in ("no_sink", "scaled_sink", "no_rot", "no_unit", "no_gate")] + [{"left": {"first": -3}}, {"right": {"reset": 60}}]
               + [{k: True} for k in ("no_left", "no_right", "no_bias", "no_ls")]
               + [{"mlp": {k: True}} for k in ("no_identity", "no_shared_gate", "no_groups", "no_correction", "renormalized")]):
    assert rms_err(ref.forward(cfg, t, toks, hooks={0: hook})[60:], want[60:]) > 0.04, hook
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=16, num_pages=20)
  assert error(dtype)(whole(engine, toks), want) < tol
  assert error(dtype)(in_portions(engine, toks, [50], decode=20), want) < tol


@DTYPES
def test_a_sink_that_outweighs_the_keys(dtype, tol):
  cfg = model([par(att(heads=4, kv_heads=1, dim=16, vdim=16, window=40, keep_first=2), right_scale=1e-3)])
  toks = tokens_for(cfg, 60)
  t = weights(cfg, 44, toks)
  t["l0.mix.left.sink"] = np.array([12.0, 9.0, 14.0, 2.0])
  want = ref.forward(cfg, t, toks)
  assert rms_err(ref.forward(cfg, t, toks, hooks={0: {"left": {"no_sink": True}}}), want) > 0.2
  engine = make_engine(cfg, t, dtype=dtype, tokens_per_page=16, num_pages=20)
  assert error(dtype)(whole(engine, toks), want) < 2 * tol
  assert error(dtype)(in_portions(engine, toks, [30], decode=30), want) < 2 * tol


def test_choice_scores_below_zero_still_lose_against_barred_groups():
  """Corrections that push every choice score below zero: a group that is not kept must count as minus infinity, not as zero."""
  cfg = model([par(mlp=moe(6, 3, 12, 2, 4, 2, 0))])
  toks = tokens_for(cfg, 50)
  models = []
  for s in range(60, 68):
    t = ref.random_model(cfg, seed=s)
    t["l0.mlp.correction"] = ref.bf16_values(t["l0.mlp.correction"] - 2.0)
    models.append(t)
  t = max(models, key=lambda t: ref.closest_router_gap(cfg, t, toks))
  want = ref.forward(cfg, t, toks)
  assert rms_err(ref.forward(cfg, t, toks, hooks={0: {"mlp": {"no_groups": True}}}), want) > 0.04
  engine = make_engine(cfg, t)
  assert rel_err(whole(engine, toks), want) < TIGHT


def test_a_slot_that_is_taken_again_starts_from_an_empty_state():
  cfg = model([par(right=lin(decay=[0.99, 1.0, 0.9]), left_scale=0.1)])
  t = weights(cfg, 7)
  engine = make_engine(cfg, t)
  a, b = tokens_for(cfg, 30, seed=1), tokens_for(cfg, 12, seed=2)
  whole(engine, a, slot=0)
  assert rel_err(whole(engine, b, slot=0), ref.forward(cfg, t, b)) < TIGHT
  # ... also when its first step is one decoded token
  assert rel_err(in_portions(engine, b, [], slot=0, decode=12), ref.forward(cfg, t, b)) < TIGHT


@pytest.mark.parametrize("dim,vdim", [(8, 8), (64, 24), (128, 128), (200, 40), (10, 7)])
def test_decayed_sums_in_chunks_and_token_by_token(dim, vdim):
  """bf16 engines: portions take the chunked kernel, single tokens the token walk, both from the same state; decays that keep
  everything, forget everything and anything between, portions that end before, at and after a chunk's edge."""
  cfg = model([par(right=lin(heads=5, dim=dim, vdim=vdim, decay=[1.0, 0.0, 0.999, 0.3, 0.9]), left_scale=0.0)], width=64)
  toks = tokens_for(cfg, 300)
  t = weights(cfg, 8)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype="bfloat16", tokens_per_page=16, num_pages=60, max_len=320)
  assert rms_err(whole(engine, toks), want) < LOOSE / 2
  for cuts, decode in (([63, 65, 64, 4], 5), ([128, 1, 129], 3), ([5, 59, 2, 190], 9), ([], 300)):
    assert rms_err(in_portions(engine, toks, cuts, decode=decode), want[: sum(cuts) + decode]) < LOOSE / 2, cuts


# ---- other sizes ------------------------------------------------------------------------------------------------------------------

SIZES = {
    "odd_width": lambda: model([par(mlp=moe(7, 3, 9, 2, 3, 2, 11)), par(mlp=zk.dense_ff(31))], width=37, vocab=47),
    "one_head_everywhere": lambda: model([par(att(heads=1, kv_heads=1), lin(heads=1), moe())]),
    "heads_with_kv_heads_of_their_own": lambda: model([par(att(kv_heads=4), lin(heads=5))]),
    "many_heads_on_one_key_head": lambda: model([par(att(heads=10, kv_heads=1, dim=8, vdim=8), lin(heads=11, dim=8, vdim=8))]),
    "three_and_five_key_heads": lambda: model([par(att(heads=9, kv_heads=3, dim=16, vdim=16)), par(att(heads=5, kv_heads=5, dim=8, vdim=16)), par(att(heads=10, kv_heads=5, dim=16, vdim=8))]),
    "value_size_over_key_size": lambda: model([par(att(dim=8, vdim=40), lin(dim=6, vdim=33))]),
    "key_size_over_value_size": lambda: model([par(att(dim=40, vdim=8, rot_dims=40), lin(dim=33, vdim=6))]),
    "rotation_of_two_channels": lambda: model([par(att(rot_dims=2))]),
    "rotation_of_every_channel": lambda: model([par(att(rot_dims=12))]),
    "wide_heads": lambda: model([par(att(heads=2, kv_heads=1, dim=72, vdim=200), lin(heads=2, dim=136, vdim=72)), par(att(heads=2, kv_heads=2, dim=256, vdim=256), lin(heads=1, dim=256, vdim=128))], width=64),
    "layers_without_feed_forward": lambda: model([par(), par()]),
    "one_expert_and_one_identity": lambda: model([par(mlp=moe(1, 1, 12, 1, 1, 1, 0)), par(mlp=moe(1, 1, 8, 0, 1, 1, 9)), par(mlp=moe(1, 2, 8, 1, 2, 2, 9))]),
    "groups_of_one": lambda: model([par(mlp=moe(5, 2, 12, 2, 7, 3, 8))]),
    "all_chosen_experts_are_often_identities": lambda: model([par(mlp=moe(2, 2, 12, 10, 3, 3, 8))]),
    "many_experts_top_one": lambda: model([par(mlp=moe(40, 1, 6, 5, 9, 4, 0))]),
    "more_than_64_experts": lambda: model([par(mlp=moe(72, 5, 6, 8, 16, 7, 16)), par(mlp=moe(60, 4, 8, 4, 8, 3, 8))], width=64),
    "window_longer_than_the_sequence": lambda: model([par(att(window=100, keep_first=60)), par(att(window=64, keep_first=4))]),
    "no_scaling_of_the_embedding": lambda: model([par()], embed_scale=1.0),
    "other_scales": lambda: model([par(left_scale=-0.7, right_scale=0.05), par(left_scale=2.5, right_scale=-1.0)], embed_scale=0.25),
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
  cfg = model([par(att(heads=4, kv_heads=2, dim=32, vdim=32, window=24, rot_dims=16), lin(heads=2, dim=64, vdim=64), zk.dense_ff(256)),
               par(att(heads=4, kv_heads=1, dim=64, vdim=64, window=40, keep_first=6, rot_dims=32), lin(heads=4, dim=32, vdim=32), moe(6, 3, 64, 2, 4, 3, 128)),
               par(att(heads=2, kv_heads=2, dim=128, vdim=128, window=33, keep_first=2, rot_dims=64), lin(heads=1, dim=128, vdim=128), moe(8, 2, 128, 0, 1, 1, 64))],
              width=128, vocab=256)
  toks = tokens_for(cfg, 90)
  t = weights(cfg, 15, toks)
  want = ref.forward(cfg, t, toks)
  engine = make_engine(cfg, t, dtype="bfloat16", tokens_per_page=16, num_pages=30)
  assert rms_err(whole(engine, toks), want) < LOOSE
  assert rms_err(in_portions(engine, toks, [70], decode=20), want) < LOOSE


def test_a_prompt_with_many_rows_per_expert():
  """The pipelined grouped products, with identity experts' slot ranges behind them."""
  cfg = model([par(att(dim=16, vdim=16), lin(heads=2, dim=16, vdim=16), moe(3, 3, 64, 2, 1, 1, 64))], width=128, vocab=90)
  toks = tokens_for(cfg, 400)
  t = weights(cfg, 18, toks)
  engine = make_engine(cfg, t, dtype="bfloat16", tokens_per_page=16, num_pages=40, max_len=420)
  assert rms_err(whole(engine, toks), ref.forward(cfg, t, toks)) < LOOSE


# ---- the tensor-core kernels over mixed schedules (bf16) ---------------------------------------------------------------------------

SHAPES = {
    "16_on_2": lambda: par(att(heads=4, kv_heads=2, dim=16, vdim=16, window=70, keep_first=4), lin(heads=2, dim=16, vdim=16)),
    "32_on_1": lambda: par(att(heads=8, kv_heads=1, dim=32, vdim=32, window=100, keep_first=33), lin(heads=3, dim=32, vdim=64)),
    "48_on_3": lambda: par(att(heads=6, kv_heads=3, dim=48, vdim=48, window=37, keep_first=1), lin(heads=2, dim=48, vdim=40)),
    "64_on_2": lambda: par(att(heads=20, kv_heads=2, dim=64, vdim=64, window=64, keep_first=20), lin(heads=2, dim=64, vdim=64)),
    "96_on_1": lambda: par(att(heads=4, kv_heads=1, dim=96, vdim=96, window=90, keep_first=3), lin(heads=1, dim=96, vdim=32)),
    "128_on_2": lambda: par(att(heads=4, kv_heads=2, dim=128, vdim=128, window=65, keep_first=64), lin(heads=2, dim=128, vdim=128)),
    "256_on_1": lambda: par(att(heads=2, kv_heads=1, dim=256, vdim=256, window=50, keep_first=10), lin(heads=1, dim=256, vdim=64)),
    "values_24_keys_40": lambda: par(att(heads=6, kv_heads=2, dim=40, vdim=24, window=33, keep_first=5), lin(heads=3, dim=24, vdim=56)),
    "values_72_keys_16": lambda: par(att(heads=9, kv_heads=3, dim=16, vdim=72, window=80, keep_first=90), lin(heads=2, dim=80, vdim=16)),
    "values_256_keys_128": lambda: par(att(heads=3, kv_heads=1, dim=128, vdim=256, window=48, keep_first=2), lin(heads=1, dim=112, vdim=96)),
}


@pytest.mark.parametrize("page", [16, 24])
@pytest.mark.parametrize("shape", sorted(SHAPES))
def test_tensor_core_shapes_and_schedules(shape, page):
  """Every instantiation of the tensor-core kernels: prompts in portions that end inside, at and after the tiles, query tiles that
  start anywhere, several sequences side by side, then single tokens."""
  cfg = model([SHAPES[shape]()], width=64, vocab=90)
  n = 150
  cfg["layers"][0]["mixer"]["left"]["scale"] = 1.5 * cfg["layers"][0]["mixer"]["left"]["dim"] ** -0.5
  toks = tokens_for(cfg, n, seed=len(shape))
  t = weights(cfg, len(shape), toks)
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
