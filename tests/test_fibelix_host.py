"""Host-side pieces of the Fibelix design: config reading, checks, the plan of layer descriptors, the oracle's own pieces.  No GPU."""

import json
import math
import os

import numpy as np
import pytest
import torch

from maxtext_indextts2_b200 import fibelix as fx
from maxtext_indextts2_b200 import params as params_lib, pyconfig
from oracle import fibelix_ref as ref
from tests.test_gugidra_host import _write_safetensors

KW = dict(per_device_batch_size=2, max_target_length=40, pagedattn_num_pages=9, pagedattn_tokens_per_page=8)
YARN = {"factor": 3.0, "original": 90, "fast": 8.0, "slow": 0.5}


def _model():
  layers = [fx.differential_layer(4, 2, 12, 20, chunk=9, scale=0.31, diff=0.35, mlp=fx.moe_ff(5, 2, 14)),
            fx.latent_layer(3, 10, 8, 14, 22, 26, window=7, rot_base=70.0, rot_scaling=YARN, scale=0.2, mlp=fx.moe_ff(4, 1, 12)),
            fx.talking_layer(4, 2, 12, 18, chunk=11, scale=0.4, rot_dims=8, rot_base=50.0, rot_factor=5.0),
            fx.differential_layer(6, 2, 12, 20, chunk=6, diff=0.2, kv_from=0, mlp=fx.moe_ff(6, 3, 10))]
  return fx.model_dict(40, 61, layers, eps=1e-5)


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
  assert config.decoder_block == "fibelix" and config.emb_dim == 40 and config.vocab_size == 61 and config.num_decoder_layers == 4
  assert config.normalization_layer_epsilon == 1e-5
  plan = fx.model_plan(config, loaded)
  # weights around zero become 1 + w in fp32; the head is the embedding table itself
  assert plan["head"] is plan["embedding"] and torch.equal(plan["final_norm"], 1.0 + tensors["final.norm"].float())
  p0, p1, p2, p3 = plan["layers"]
  assert all(p["norm_style"] == "pre" and p["conv1"] is None for p in plan["layers"]) and torch.equal(p1["norm1"], 1.0 + tensors["l1.norm1"].float())
  # differential: both maps of q, then of k, then v; no biases
  a = p0["attn"]
  assert p0["n_in"] == 96 + 48 + 40 and torch.equal(p0["w_in"][96:144], tensors["l0.mix.k"]) and torch.equal(p0["w_in"][144:], tensors["l0.mix.v"])
  assert (a["maps"], a["chunk"], a["window"], a["rot_dims"], a["shared_kv"], a["kv_from"]) == (2, 9, 0, 0, 0, None) and "b_in" not in p0
  dot = lambda x, y: float((tensors["l0.mix." + x].double() * tensors["l0.mix." + y].double()).sum())
  assert abs(a["diff_lambda"] - (math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + 0.35)) < 1e-12 and abs(a["diff_scale"] - 0.65) < 1e-12
  # latent: query down-projection, key / value down-projection with the rotated part, head gates
  m = p1["latent"]
  assert p1["n_in"] == 22 + 34 + 3 and torch.equal(p1["w_in"][22:56], tensors["l1.mix.dkv"]) and torch.equal(p1["w_in"][56:], tensors["l1.mix.g"])
  freq, amp = ref.yarn_frequencies(8, 70.0, YARN)
  assert (m["window"], m["rot_half"], m["q_rank"], m["kv_rank"]) == (7, 0, 22, 26) and np.allclose(m["rot_freq"].numpy(), freq, rtol=1e-13)
  assert abs(m["rot_amp"] - amp) < 1e-12 and m["w_uk_t"].shape == (3, 26, 10) and m["w_uv"].shape == (3, 14, 26) and m["sink"] is None
  # talking: biases in the order of the rows, scaled frequencies, a sink whose score is zero
  b = p2["attn"]
  assert p2["n_in"] == 48 + 24 + 36 and torch.equal(p2["b_in"], torch.cat([tensors[f"l2.mix.{n}.b"] for n in "qkv"]).float())
  assert torch.equal(p2["bo"], tensors["l2.mix.o.b"].float()) and (b["maps"], b["chunk"], b["rot_half"], b["rot_dims"]) == (1, 11, 1, 8)
  assert np.allclose(b["rot_freq"].numpy(), ref.linear_frequencies(8, 50.0, 5.0), rtol=1e-13) and b["sink"].tolist() == [0.0] * 4
  assert b["talk"].shape == (4, 4) and torch.equal(b["temp"], tensors["l2.mix.temp"].float()) and p2["moe"] is None
  # a layer that reads another layer's cache projects queries only, with heads of its own
  c = p3["attn"]
  assert p3["n_in"] == 144 and (c["shared_kv"], c["kv_from"], c["chunk"], c["heads"]) == (1, 0, 6, 6)
  # experts: gate and up rows interleaved, stacked; softmax over the chosen logits
  e = p0["moe"]
  assert (e["experts"], e["top"], e["ff"], e["shared_ff"], e["chosen_softmax"], e["act_silu"]) == (5, 2, 14, 0, 1, 1)
  assert torch.equal(e["w_gate_up"][3, 0::2], tensors["l0.mlp.e3.gate"]) and torch.equal(e["w_gate_up"][3, 1::2], tensors["l0.mlp.e3.up"])
  assert torch.equal(e["w_down"][4], tensors["l0.mlp.e4.down"]) and torch.equal(e["router_bias"], tensors["l0.mlp.router.b"].float())


def test_yarn_frequencies_three_regimes():
  # dims 8, base 10000: pair(turns) = 8 ln(original / (2 pi turns)) / (2 ln base); original chosen so that pair(1) = 2.5, pair(4) < 2
  original = 2.0 * math.pi * 10000.0 ** (2.5 * 2 / 8)
  f, amp = fx.yarn_rot_frequencies(8, 10000.0, {"factor": 4.0, "original": original, "fast": 4.0, "slow": 1.0})
  plain = [10000.0 ** (-2 * i / 8) for i in range(4)]
  lo, hi = math.floor(2.5 - 8 * math.log(4.0) / (2 * math.log(10000.0))), 3
  assert lo == 1
  want = [p / 4.0 * r + p * (1 - r) for p, r in zip(plain, [0.0, 0.0, 0.5, 1.0])]
  assert np.allclose(f.numpy(), want, rtol=1e-12) and abs(amp - (0.1 * math.log(4.0) + 1.0)) < 1e-15
  assert np.allclose(ref.yarn_frequencies(8, 10000.0, {"factor": 4.0, "original": original, "fast": 4.0, "slow": 1.0})[0], want, rtol=1e-12)
  f, amp = fx.yarn_rot_frequencies(4, 100.0, None)
  assert np.allclose(f.numpy(), [1.0, 0.1]) and amp == 1.0
  # lo == hi: the ramp is a step; lo clamped at 0, hi at dims - 1
  for s in ({"factor": 2.0, "original": 7.0, "fast": 1.0, "slow": 1.0}, {"factor": 2.0, "original": 1e9, "fast": 1.0, "slow": 0.1}):
    assert np.allclose(fx.yarn_rot_frequencies(10, 30.0, s)[0].numpy(), ref.yarn_frequencies(10, 30.0, s)[0], rtol=1e-13)


def test_mechanism_functions_of_the_oracle_agree_with_closed_forms():
  # (so a shared misreading cannot hide in the oracle and in the engine)
  assert np.allclose(ref.around_zero_norm(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.0), [[3.0 / math.sqrt(12.5), 8.0 / math.sqrt(12.5)]])
  assert list(ref.chunk_visible(9, 5)) == [5, 6, 7, 8, 9] and list(ref.chunk_visible(10, 5)) == [10] and list(ref.chunk_visible(2, 0)) == [0, 1, 2]
  assert list(ref.window_visible(9, 3)) == [7, 8, 9] and list(ref.window_visible(1, 3)) == [0, 1]
  r = ref.rotate_half(np.array([[[1.0, 0.0, 0.0, 2.0, 7.0]]]), np.array([3]), np.array([0.5, 0.25]))
  assert np.allclose(r[0, 0], [math.cos(1.5), -2 * math.sin(0.75), math.sin(1.5), 2 * math.cos(0.75), 7.0])
  r = ref.rotate_pairs(np.array([[[1.0, 0.0, 0.0, 2.0]]]), np.array([3]), np.array([0.5, 0.25]), amp=2.0)
  assert np.allclose(r[0, 0], [2 * math.cos(1.5), 2 * math.sin(1.5), -4 * math.sin(0.75), 4 * math.cos(0.75)])
  # two heads on one key head, one key, scores 2 and 0; head 0 gets 0.5 s_0, head 1 gets -s_0 + s_1; one joins each denominator
  q, k, v = np.array([[[2.0], [0.0]]]), np.array([[[1.0]]]), np.array([[[3.0]]])
  o = ref.talking_attention(q, k, v, 0.5, np.array([2.0, 1.0]), np.array([[0.5, 0.0], [-1.0, 1.0]]), 4)
  assert np.allclose(o[0, :, 0], [3.0 * math.e / (1 + math.e), 3.0 * math.exp(-2.0) / (1 + math.exp(-2.0))])
  # two maps over two values: the first looks at key 0 only, the second at both evenly
  q = np.zeros((2, 1, 2, 1))
  q[1, 0, 0, 0] = 100.0
  k = np.array([[[[1.0], [0.0]]], [[[-1.0], [0.0]]]])
  a = ref.two_map_attention(q, k, np.array([[[2.0]], [[6.0]]]), 1.0, 4)
  assert np.allclose(a[1, 0, :, 0], [2.0, 4.0])
  assert np.allclose(ref.map_difference(np.array([[[[4.0, 0.0], [1.0, 2.0]]]]), 0.5, 0.25, 0.0), np.array([[[3.5, -1.0]]]) / math.sqrt(6.625) * 0.75)
  c, w = ref.route(np.log(np.array([[1.0, 4.0, 3.0, 2.0]])), 2)
  assert c.tolist() == [[1, 2]] and np.allclose(w, [[4 / 7, 3 / 7]])


def test_input_projection_and_bias_are_padded_to_whole_tiles_when_the_width_allows():
  cfg = fx.model_dict(64, 50, [fx.talking_layer(2, 1, 8)])
  config = pyconfig.from_model_dict(cfg, **KW)
  plan = fx.model_plan(config, fx.random_tensors(config, seed=0))["layers"][0]
  assert plan["n_in"] == 128 and float(plan["w_in"][32:].float().abs().max()) == 0.0 and plan["b_in"].shape == (128,) and float(plan["b_in"][32:].abs().max()) == 0.0


@pytest.mark.parametrize("break_it,match", [
    (lambda c: c["layers"][0].update(type="conv"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=24), "geometry"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1), "mask.size"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_bad_configs_are_refused(break_it, match):
  cfg = _model()
  break_it(cfg)
  with pytest.raises(ValueError, match=match):
    pyconfig.from_model_dict(cfg, **KW)


def test_missing_or_misshaped_tensors_are_refused():
  cfg = _model()
  config = pyconfig.from_model_dict(cfg, **KW)
  t = _tensors(cfg)
  for name in ("l2.mix.q.b", "l0.mlp.router.b", "l1.mix.dq.norm", "l2.mix.talk", "l0.mix.lk2"):
    bad = dict(t)
    bad[name] = bad[name][:-1]
    with pytest.raises(ValueError, match=name.replace(".", r"\.")):
      fx.model_plan(config, bad)
    del bad[name]
    with pytest.raises(KeyError):
      fx.model_plan(config, bad)


def test_random_tensors_have_the_names_and_shapes_the_plan_reads():
  cfg = _model()
  config = pyconfig.from_model_dict(cfg, **KW)
  t = fx.random_tensors(config, seed=3)
  want = ref.random_model(cfg, seed=0)
  assert set(t) == set(want) and all(tuple(t[k].shape) == want[k].shape for k in t)
  fx.model_plan(config, t)
