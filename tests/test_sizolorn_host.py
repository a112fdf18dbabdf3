"""CPU checks of the Sizolorn configuration reader, the registry entries, the random checkpoints and the oracle."""
import json
import math

import numpy as np
import pytest
import torch

import sizolorn_oracle as O
from xotorch_support_jetson_b200.model_config import hybrid_model_config, is_hybrid, load_model_config
from xotorch_support_jetson_b200.models import model_cards
from xotorch_support_jetson_b200.synth import random_sizolorn_state, sizolorn_param_shapes, write_random_checkpoint


def test_config_reader_maps_every_constant():
  raw = model_cards["sizolorn-tiny"]["hf_config"]
  cfg = hybrid_model_config(raw)
  assert is_hybrid(cfg) and cfg["block"] == "prenorm" and cfg["norm_kind"] == "layer" and cfg["tied_head"]
  assert cfg["norm_eps"] == raw["norm"]["eps"] and cfg["streams"] == raw["streams"] and cfg["logit_softcap"] == 0.0
  both, fil, uni, again = cfg["layers"]
  m0, m1, m2 = (raw["layers"][i]["mixer"] for i in range(3))
  for lay, m in ((both, m0["left"]), (fil, m1), (uni, m2)):
    assert lay["mixer"] == "softmax" and all(lay[k] == m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
    assert lay["rot_dims"] == m["rot"]["dims"] and lay["rot_base"] == m["rot"]["base"] and lay["rot_mult"] == 1.0
  assert both["window"] == m0["left"]["mask"]["size"] and "chunk" not in both and both["gate"] and not both.get("qkv_bias") and both["rot_pairs"] == "half"
  assert both["second"] == {"mixer": "mlstm", **m0["right"]} and (both["left_scale"], both["right_scale"]) == (m0["left_scale"], m0["right_scale"])
  assert fil["chunk"] == m1["mask"]["size"] and "window" not in fil and fil["taps"] == m1["conv"] and fil["rot_pairs"] == "interleaved"
  assert fil["qkv_bias"] and fil["o_bias"] and fil["qk_norm"] and fil["gate"] and not fil.get("head_norm") and not fil.get("second")
  sc = m1["rot"]["scaling"]
  assert fil["rot_scaling"] == "bands" and (fil["rot_factor"], fil["rot_p0"], fil["rot_p1"], fil["rot_orig"]) == (sc["factor"], sc["low"], sc["high"], sc["original"])
  assert uni["chunk"] == m2["mask"]["size"] and uni["head_norm"] and uni["qkv_bias"] and uni["o_bias"] and not uni.get("gate") and not uni.get("qk_norm")
  assert uni["rot_scaling"] == "none" and uni["rot_pairs"] == "interleaved" and not uni.get("taps")
  r = raw["layers"][0]["mlp"]
  assert both["ff_kind"] == "moe" and both["ff_act"] == "relu2" and both["route_bias"] and both["route_norm"] and both["route_score"] == "softmax"
  assert (both["ff"], both["experts"], both["identity"], both["top"], both["groups"], both["shared_ff"], both["shared_gate"]) == \
         (r["expert"]["ff"], r["router"]["experts"], r["router"]["identity"], r["router"]["top"], 0, r["shared"]["ff"], True)
  assert uni["ff"] == 0 and uni["ff_kind"] == "none"
  assert [l["weights_of"] for l in cfg["layers"]] == [-1, -1, -1, 0]
  assert {k: v for k, v in again.items() if k != "weights_of"} == {k: v for k, v in both.items() if k != "weights_of"}


def test_optional_parts_and_refusals():
  raw = json.loads(json.dumps(model_cards["sizolorn-tiny"]["hf_config"]))
  lean = {**raw, "layers": [json.loads(json.dumps(raw["layers"][1]))]}
  m, f = lean["layers"][0]["mixer"], lean["layers"][0]["mlp"]
  del m["rot"]["scaling"], m["conv"], f["shared"], f["router"]["identity"]
  lay = hybrid_model_config(lean)["layers"][0]
  assert lay["rot_scaling"] == "none" and lay["taps"] == 0 and lay["shared_ff"] == 0 and not lay["shared_gate"] and lay["identity"] == 0
  for bad in ({"type": "convolution"}, {"mlp": {"kind": "dense", "ff": 8}}):
    with pytest.raises(ValueError):
      hybrid_model_config({**raw, "layers": [{**raw["layers"][1], **bad}]})
  wide = json.loads(json.dumps(raw["layers"][1]))
  wide["mixer"]["rot"]["dims"] = wide["mixer"]["dim"] + 2
  with pytest.raises(ValueError):
    hybrid_model_config({**raw, "layers": [wide]})


def test_checkpoint_on_disk_round_trip(tmp_path):
  raw = model_cards["sizolorn-tiny"]["hf_config"]
  p = write_random_checkpoint(tmp_path / "m", raw, seed=1)
  cfg = load_model_config(p / "config.json")
  assert cfg["architecture"] == "Sizolorn" and cfg["num_layers"] == len(raw["layers"])
  sh = sizolorn_param_shapes(raw)
  s, D = raw["streams"], raw["width"]
  assert "head" not in sh and "l2.norm2" not in sh and "l2.hc2.in" not in sh and not any(k.startswith("l3.") for k in sh)
  assert sh["l0.hc1.mix"] == (s, s) and sh["l1.hc2.out"] == (s,) and sh["l0.mlp.router"] == (7, D) and sh["l0.mlp.correction"] == (7,)
  assert sh["l1.mix.v.conv"] == (2 * 24, 4) and sh["l1.mix.q.norm"] == (4 * 32,) and sh["l0.mix.right.norm"] == (3 * 40,) and sh["l0.mix.left.g"] == (6, D)
  assert "l2.mix.g" not in sh and "l0.mix.left.q.b" not in sh and sh["l2.mix.o.b"] == (D,)
  w = random_sizolorn_state(raw, seed=1)
  assert set(w) == set(sh) and all(tuple(w[k].shape) == tuple(v) for k, v in sh.items())
  for mid in ("sizolorn-tiny", "sizolorn-1b"):
    assert hybrid_model_config(model_cards[mid]["hf_config"])["num_layers"] == model_cards[mid]["layers"]


def test_oracle_pieces():
  rng = np.random.default_rng(0)
  # rotation keeps the length of a pair and passes what lies behind; neighbours or halves
  y = rng.standard_normal((3, 2, 8))
  rot = {"base": 1000.0, "dims": 6}
  for neighbours, pairs in ((True, [(0, 1), (2, 3), (4, 5)]), (False, [(0, 3), (1, 4), (2, 5)])):
    z = O.rotate(y, [0, 5, 9], rot, neighbours)
    assert np.allclose(z[..., 6:], y[..., 6:]) and np.allclose(z[0], y[0])
    for i, (a, b) in enumerate(pairs):
      assert np.allclose(z[..., a] ** 2 + z[..., b] ** 2, y[..., a] ** 2 + y[..., b] ** 2)
      ang = 5 * 1000.0 ** (-2 * i / 6)
      assert np.allclose(z[1, :, a], y[1, :, a] * math.cos(ang) - y[1, :, b] * math.sin(ang))
  # band scaling: the fastest pair keeps its frequency, the slowest is divided by the factor
  fr = O.frequencies({"base": 500000.0, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}})
  plain = O.frequencies({"base": 500000.0, "dims": 32})
  assert fr[0] == plain[0] and np.isclose(fr[-1], plain[-1] / 8.0) and ((fr <= plain + 1e-18) & (fr >= plain / 8.0 - 1e-18)).all()
  assert any(f not in (p, p / 8.0) for f, p in zip(fr, plain))
  # filter: the newest tap is the last one, nothing before the start
  u = rng.standard_normal((4, 2))
  w = np.array([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]])
  f = O.short_filter(u, w)
  assert np.allclose(f[:, 0], u[:, 0]) and np.allclose(f[:, 1], [0, 0, u[0, 1], u[1, 1]])
  # masks
  assert O.seen_window(5, 2).sum(1).tolist() == [1, 2, 2, 2, 2] and O.seen_chunk(7, 3).sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1]
  # routing: a correction moves the choice, the weights come from the scores alone
  z = np.array([0.0, 2.0, 1.0, -1.0])
  s = np.exp(z) / np.exp(z).sum()
  p = O.route(z, np.array([0.0, -1.0, 0.0, 0.0]), 2)
  assert sorted(p) == [0, 2] and np.isclose(p[0] / p[2], s[0] / s[2]) and np.isclose(sum(p.values()), 1.0)
  # streams: equal copies, mixing from row to column
  X = rng.standard_normal((2, 3, 4))
  y = rng.standard_normal((2, 4))
  st = {"h.in": torch.tensor([1.0, 0.0, 0.0]), "h.out": torch.tensor([0.0, 2.0, 0.0]), "h.mix": torch.zeros(3, 3)}
  st["h.mix"][0, 2] = 1.0
  Z = O.write_streams(st, "h.", X, y)
  assert np.allclose(Z[:, 0], 0) and np.allclose(Z[:, 1], 2 * y) and np.allclose(Z[:, 2], X[:, 0]) and np.allclose(O.read_streams(st, "h.", X), X[:, 0])
  # layer norm: the mean goes, the rest has unit size
  v = O.layer_norm(rng.standard_normal((3, 50)) + 7.0, np.ones(50), 0.0)
  assert np.allclose(v.mean(1), 0.0) and np.allclose((v ** 2).mean(1), 1.0)


def test_oracle_matrix_memory_in_closed_form():
  """The running maximum is a matter of numerics: memory and normaliser are sums with weights e^(i_s + f_(s+1) + .. + f_t), and the
  denominator is max(|n . q|, 1) in those units."""
  H, n, m, D, T, cap = 2, 3, 4, 5, 6, 4.0
  g = torch.Generator().manual_seed(3)
  st = {f"p.{k}": torch.randn(r, D, generator=g, dtype=torch.float64) for k, r in {"q": H * n, "k": H * n, "v": H * m, "g": H * m, "i": H, "f": H}.items()}
  st.update({"p.i.b": torch.tensor([-3.0, 2.0]), "p.f.b": torch.tensor([3.0, -1.0]), "p.norm": torch.ones(H * m), "p.o": torch.eye(D, H * m, dtype=torch.float64)})
  h = np.random.default_rng(1).standard_normal((T, D))
  q, k, v, gate, zi, zf = (h @ st["p." + x].numpy().T for x in "qkvgif")
  q, k, v = (a.reshape(T, H, -1) for a in (q / math.sqrt(n), k, v))
  li = cap * np.tanh((zi + st["p.i.b"].numpy()) / cap)
  lf = -np.log1p(np.exp(-cap * np.tanh((zf + st["p.f.b"].numpy()) / cap)))
  t = T - 1
  want = []
  for a in range(H):
    wts = [math.exp(li[s, a] + lf[s + 1:t + 1, a].sum()) for s in range(T)]
    S = sum(w * np.outer(k[s, a], v[s, a]) for s, w in enumerate(wts))
    den = max(abs(sum(w * k[s, a] for s, w in enumerate(wts)) @ q[t, a]), 1.0)
    o = S.T @ q[t, a] / den
    want.append(o / math.sqrt((o ** 2).mean()))
  want = np.concatenate(want) * O.sigmoid(gate[t])
  got = O.matrix_memory(st, "p.", {"heads": H, "dim": n, "vdim": m, "gate_cap": cap}, h, 0.0)[t]
  assert np.allclose(got, want[:D], rtol=1e-4)
