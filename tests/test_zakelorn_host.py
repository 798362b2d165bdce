"""Host-side pieces of the Zakelorn design: config reading, checks, the plan of layer descriptors, the oracle's own pieces.  No GPU."""

import copy
import json
import math
import os

import numpy as np
import pytest
import torch

from maxtext_indextts2_b200 import params as params_lib, pyconfig
from maxtext_indextts2_b200 import zakelorn as zk
from oracle import zakelorn_ref as ref
from tests.test_gugidra_host import _write_safetensors

KW = dict(per_device_batch_size=2, max_target_length=40, pagedattn_num_pages=9, pagedattn_tokens_per_page=8)


def _model():
  layers = [zk.parallel_layer(zk.attention_part(4, 2, 12, 20, window=9, keep_first=3, scale=0.31, rot_dims=8, rot_base=50.0), zk.lightning_part(3, 10, 14, [0.5, 0.9, 1.0]),
                              0.8, 1.3, zk.dense_ff(26)),
            zk.parallel_layer(zk.attention_part(6, 3, 8, rot_dims=0), zk.lightning_part(2, 6), 1.0, -0.5, zk.moe_ff(5, 3, 14, identity=3, groups=4, keep=2, shared_ff=18)),
            zk.parallel_layer(zk.attention_part(2, 1, 8, window=4), zk.lightning_part(1, 6), mlp=zk.moe_ff(4, 1, 10))]
  return zk.model_dict(40, 61, layers, eps=1e-5, embed_scale=2.5)


def _tensors(cfg, seed=1):
  return {k: torch.from_numpy(v).to(torch.bfloat16) for k, v in ref.random_model(cfg, seed=seed).items()}


def test_model_folder_round_trip_and_plan(tmp_path):
  cfg = _model()
  tensors = _tensors(cfg)
  os.makedirs(tmp_path / "m")
  with open(tmp_path / "m" / "config.json", "w") as f:
    json.dump(cfg, f)
  _write_safetensors(tmp_path / "m" / "model.safetensors", tensors)
  loaded = params_lib.load_model_dir(str(tmp_path / "m"))
  config = pyconfig.from_model_dir(str(tmp_path / "m"), **KW)
  assert config.decoder_block == "zakelorn" and config.emb_dim == 40 and config.vocab_size == 61 and config.num_decoder_layers == 3
  assert config.normalization_layer_epsilon == 1e-5 and config.embedding_scale == 2.5
  plan = zk.model_plan(config, loaded)
  assert plan["head"] is plan["embedding"] and plan["embed_scale"] == 2.5
  assert torch.equal(plan["final_norm"], tensors["final.norm"].float()) and torch.equal(plan["final_norm_b"], tensors["final.norm.b"].float())
  p0, p1, p2 = plan["layers"]
  assert all(p["norm_style"] == "out_layer" and p["mixer"] == "composite" for p in plan["layers"])
  # the layer scale is part of the norms' weights and biases
  for n in ("1", "2"):
    s = tensors["l0.ls" + n].float()
    assert torch.equal(p0[f"norm{n}"], tensors[f"l0.norm{n}"].float() * s) and torch.equal(p0[f"norm{n}b"], tensors[f"l0.norm{n}.b"].float() * s)
  # projections: left q, k, v, gate, then right q, k, v, gate; both output projections side by side, the scales on the activations
  a, r = p0["attn"], p0["rec"]
  assert p0["n_in"] == 48 + 24 + 40 + 80 + 30 + 30 + 42 + 42
  assert torch.equal(p0["w_in"][112:192], tensors["l0.mix.left.g"]) and torch.equal(p0["w_in"][192:222], tensors["l0.mix.right.q"])
  assert torch.equal(p0["w_in"][252:294], tensors["l0.mix.right.v"]) and torch.equal(p0["w_in"][294:], tensors["l0.mix.right.g"])
  assert torch.equal(p0["wo"], torch.cat([tensors["l0.mix.left.o"], tensors["l0.mix.right.o"]], dim=1))
  assert (a["window"], a["keep_first"], a["rot_dims"], a["rot_half"], a["value_gate"], a["scale"], a["out_scale"]) == (9, 3, 8, 0, 1, 0.31, 0.8)
  assert np.allclose(a["rot_freq"].numpy(), ref.frequencies(8, 50.0), rtol=1e-13) and torch.equal(a["sink"], tensors["l0.mix.left.sink"].float())
  assert torch.equal(a["q_norm"], torch.ones(12)) and torch.equal(a["k_norm"], torch.ones(12))
  assert (r["kind"], r["heads"], r["dim"], r["vdim"], r["norm_whole"], r["gate_silu"], r["out_scale"]) == ("decay", 3, 10, 14, 1, 0, 1.3)
  assert torch.equal(r["head_decay"], torch.tensor([0.5, 0.9, 1.0])) and torch.equal(r["out_norm"], tensors["l0.mix.right.norm"].float())
  assert (p0["ff_kind"], p0["ff"]) == ("gelu_up", 26) and torch.equal(p0["w_gate_up"], tensors["l0.mlp.up"]) and torch.equal(p0["w_down"], tensors["l0.mlp.down"])
  # no mask and no rotation: off
  assert (p1["attn"]["window"], p1["attn"]["keep_first"], p1["attn"]["rot_dims"], p1["attn"]["rot_freq"]) == (0, 0, 0, None)
  # routed: identity experts have no weights, the shared expert's gate is one more row of the router
  e = p1["moe"]
  assert (e["experts"], e["identity"], e["top"], e["groups"], e["keep_groups"], e["groups_max"], e["shared_ff"], e["shared_gate"]) == (5, 3, 3, 4, 2, 1, 18, 1)
  assert (e["score_softmax"], e["plain_weights"], e["act_silu"]) == (1, 1, 1) and e["correction"].shape == (8,) and e["w_gate_up"].shape == (5, 28, 40)
  assert torch.equal(e["w_router"], torch.cat([tensors["l1.mlp.router"], tensors["l1.mlp.shared.sg"]]))
  assert torch.equal(e["w_gate_up"][3, 0::2], tensors["l1.mlp.e3.gate"]) and torch.equal(e["shared_gate_up"][1::2], tensors["l1.mlp.shared.up"])
  assert p2["moe"]["w_router"].shape == (4, 40) and p2["moe"]["identity"] == 0 and p2["moe"].get("shared_gate", 0) == 0


def test_input_projection_is_padded_to_whole_tiles_when_the_width_allows():
  cfg = zk.model_dict(64, 50, [zk.parallel_layer(zk.attention_part(2, 1, 8), zk.lightning_part(1, 8))])
  config = pyconfig.from_model_dict(cfg, **KW)
  plan = zk.model_plan(config, zk.random_tensors(config, seed=0))["layers"][0]
  assert plan["n_in"] == 128 and plan["w_in"].shape == (128, 64) and torch.count_nonzero(plan["w_in"][80:]) == 0


def test_optional_parts_may_be_left_out_of_the_config():
  cfg = _model()
  router = cfg["layers"][1]["mlp"]["router"]
  del router["groups"], router["identity"], cfg["layers"][1]["mlp"]["shared"], cfg["embedding"]
  cfg["layers"][0]["mixer"]["left"]["mask"] = None
  cfg["layers"][2]["mlp"] = None
  cfg["layers"][0]["mlp"] = {"ff": 26}
  config = pyconfig.from_model_dict(cfg, **KW)
  plan = zk.model_plan(config, _tensors(cfg))
  e = plan["layers"][1]["moe"]
  assert (e["identity"], e["groups"], e["keep_groups"], e["shared_ff"]) == (0, 1, 1, 0) and plan["embed_scale"] == 1.0
  assert plan["layers"][0]["attn"]["window"] == 0 and plan["layers"][0]["ff_kind"] == "gelu_up" and plan["layers"][2]["moe"] is None and plan["layers"][2]["ff"] == 0


def test_bad_configs_and_tensors_are_refused():
  def bad(change):
    cfg = copy.deepcopy(_model())
    change(cfg["layers"])
    with pytest.raises(ValueError):
      pyconfig.from_model_dict(cfg, **KW)

  bad(lambda l: l[0].update(type="attention"))
  bad(lambda l: l[0]["mixer"]["left"].update(heads=5))
  bad(lambda l: l[0]["mixer"]["left"]["rot"].update(dims=7))
  bad(lambda l: l[0]["mixer"]["left"]["rot"].update(dims=14))
  bad(lambda l: l[0]["mixer"]["left"]["mask"].update(keep_first=-1))
  bad(lambda l: l[0]["mixer"]["right"].update(decay=[0.5]))
  bad(lambda l: l[0]["mixer"].pop("left_scale"))
  bad(lambda l: l[0]["mlp"].update(kind="gated"))
  bad(lambda l: l[1]["mlp"]["router"].update(top=5))      # the kept groups hold four
  bad(lambda l: l[1]["mlp"]["router"].update(identity=2))  # seven outputs do not form four groups
  bad(lambda l: l[1]["mlp"]["router"]["groups"].update(keep=5))
  config = pyconfig.from_model_dict(_model(), **KW)
  tensors = _tensors(_model())
  for name in ("l0.mix.left.sink", "l1.mlp.router", "l0.ls1", "final.norm.b"):
    wrong = dict(tensors, **{name: tensors[name][:-1]})
    with pytest.raises(ValueError, match=name.replace(".", r"\.")):
      zk.model_plan(config, wrong)


def test_mechanism_functions_of_the_oracle_agree_with_closed_forms():
  # (so a shared misreading cannot hide in the oracle and in the engine)
  assert np.allclose(ref.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 5.0]), np.array([0.5, 0.0]), 3.0), [[-0.5, 2.5]])
  assert np.allclose(ref.rms_unit(np.array([3.0, 4.0]), 0.0), np.array([3.0, 4.0]) / math.sqrt(12.5))
  assert ref.visible(9, 3, 2) == [0, 1, 7, 8, 9] and ref.visible(2, 3, 2) == [0, 1, 2] and ref.visible(3, 3, 1) == [0, 1, 2, 3] and ref.visible(4, 0, 0) == [0, 1, 2, 3, 4]
  r = ref.rotate_pairs(np.array([[[1.0, 0.0, 0.0, 2.0, 7.0]]]), np.array([3]), np.array([0.5, 0.25]))
  assert np.allclose(r[0, 0], [math.cos(1.5), math.sin(1.5), -2 * math.sin(0.75), 2 * math.cos(0.75), 7.0])
  # one key of score 1 beside a sink of ln 2: the weight is e / (e + 2), and the sink is not scaled
  o = ref.sink_attention(np.array([[[2.0]]]), np.array([[[1.0]]]), np.array([[[3.0]]]), 0.5, [math.log(2.0)], 4, 0)
  assert np.allclose(o, 3.0 * math.e / (math.e + 2.0))
  # window of one, first token kept: the query at 2 sees the keys 0 and 2
  o = ref.sink_attention(np.ones((3, 1, 1)), np.zeros((3, 1, 1)), np.array([[[1.0]], [[10.0]], [[100.0]]]), 1.0, [0.0], 1, 1)
  assert np.allclose(o[:, 0, 0], [1.0 / 2, 11.0 / 3, 101.0 / 3])
  # decayed sums: the weights of older tokens are powers of the decay
  q, k, v = np.ones((3, 1, 1)), np.array([[[1.0]], [[2.0]], [[3.0]]]), np.ones((3, 1, 1))
  o, S = ref.decayed_sums(q, k, v, np.array([0.5]))
  assert np.allclose(o[:, 0, 0], [1.0, 2.5, 4.25]) and np.allclose(S, 4.25)
  assert np.allclose(ref.decayed_sums(q[2:], k[2:], v[2:], np.array([0.5]), ref.decayed_sums(q[:2], k[:2], v[:2], np.array([0.5]))[1])[0], 4.25)
  # groups by their largest choice score; negative scores of barred groups do not win
  s, c = ref.choice_scores(np.log(np.array([[4.0, 1.0, 3.0, 2.0]])), np.array([-1.0, -1.0, -1.2, -1.0]), 2, 1)
  assert np.allclose(s, [[0.4, 0.1, 0.3, 0.2]]) and np.allclose(c[0, :2], [-0.6, -0.9]) and np.all(np.isinf(c[0, 2:]))
  assert np.allclose(ref.gelu_tanh(np.array([0.0, 10.0, -10.0])), [0.0, 10.0, 0.0])
  # an identity expert returns its input, times its score as it is
  t = {"router": np.array([[0.0], [0.0]]), "correction": np.array([0.0, 1.0]), "e0.gate": np.ones((1, 1)), "e0.up": np.ones((1, 1)), "e0.down": np.ones((1, 1))}
  assert np.allclose(ref.moe_ff(np.array([[6.0]]), t, "", {"kind": "moe", "expert": {"ff": 1}, "router": {"experts": 1, "identity": 1, "top": 1}}), 3.0)


def test_random_tensors_have_the_names_and_shapes_the_plan_reads():
  cfg = _model()
  config = pyconfig.from_model_dict(cfg, **KW)
  t = zk.random_tensors(config, seed=3)
  want = ref.random_model(cfg, seed=0)
  assert set(t) == set(want) and all(tuple(t[k].shape) == want[k].shape for k in t)
  zk.model_plan(config, t)
