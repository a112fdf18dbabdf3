"""CPU checks of the Rurutar configuration reader, the registry entries, the random checkpoints and the oracle."""
import json
import math

import numpy as np
import pytest
import torch

import rurutar_oracle as O
from xotorch_support_jetson_b200.model_config import hybrid_model_config, is_hybrid, load_model_config, resolve_tensor_sizes
from xotorch_support_jetson_b200.models import model_cards
from xotorch_support_jetson_b200.synth import random_rurutar_state, rurutar_param_shapes, write_random_checkpoint


def test_config_reader_maps_every_constant():
  raw = model_cards["rurutar-tiny"]["hf_config"]
  cfg = hybrid_model_config(raw)
  assert is_hybrid(cfg) and cfg["block"] == "prenorm" and cfg["norm_kind"] == "tanh"
  assert cfg["norm_eps"] == raw["norm"]["eps"] and cfg["embed_scale"] == raw["embedding"]["scale"] and cfg["logit_softcap"] == raw["logit_softcap"]
  gla, lat, bare, sharing = cfg["layers"]
  m0, m1, m3 = (raw["layers"][i]["mixer"] for i in (0, 1, 3))
  assert gla["mixer"] == "gla" and (gla["heads"], gla["dim"], gla["vdim"], gla["tau"], gla["rank"]) == (m0["heads"], m0["dim"], m0["vdim"], m0["tau"], m0["rank"])
  assert (gla["ff_kind"], gla["ff_act"], gla["ff"]) == ("glu", "geglu", raw["layers"][0]["mlp"]["ff"])
  assert lat["mixer"] == "latent" and lat["gate"] and lat["kv_from"] == -1 and lat["window"] == m1["mask"]["size"]
  for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale"):
    assert lat[k] == m1[k]
  sc = m1["rot"]["scaling"]
  assert lat["rot_pairs"] == "half" and lat["rot_scaling"] == "ramp" and lat["rot_dims"] == m1["rot"]["dims"] and lat["rot_base"] == m1["rot"]["base"]
  assert (lat["rot_factor"], lat["rot_orig"], lat["rot_p0"], lat["rot_p1"]) == (sc["factor"], sc["original"], sc["fast"], sc["slow"])
  assert abs(lat["rot_mult"] - (0.1 * math.log(sc["factor"]) + 1.0)) < 1e-15
  r1 = raw["layers"][1]["mlp"]
  assert lat["ff_kind"] == "moe" and lat["ff_act"] == "swiglu" and not lat["route_input"] and lat["route_norm"] and lat["route_score"] == "softmax"
  assert (lat["ff"], lat["experts"], lat["top"], lat["groups"], lat["shared_ff"], lat["shared_gate"]) == \
         (r1["expert"]["ff"], r1["router"]["experts"], r1["router"]["top"], 0, r1["shared"]["ff"], True)
  assert bare["ff"] == 0 and bare["ff_kind"] == "none"
  assert sharing["kv_from"] == m3["kv_from"] and sharing["window"] != lat["window"] and sharing["heads"] != lat["heads"]


def test_optional_parts_and_refusals():
  raw = json.loads(json.dumps(model_cards["rurutar-tiny"]["hf_config"]))
  lean = {k: v for k, v in raw.items() if k != "logit_softcap"}
  lean["layers"] = [json.loads(json.dumps(raw["layers"][1]))]
  del lean["layers"][0]["mixer"]["rot"]["scaling"]
  del lean["layers"][0]["mlp"]["shared"]
  cfg = hybrid_model_config(lean)
  lay = cfg["layers"][0]
  assert cfg["logit_softcap"] == 0.0 and lay["rot_scaling"] == "none" and lay["rot_mult"] == 1.0
  assert lay["shared_ff"] == 0 and not lay["shared_gate"]
  for bad in ({"type": "convolution"}, {"mlp": {"kind": "sparse", "ff": 8}}):
    with pytest.raises(ValueError):
      hybrid_model_config({**raw, "layers": [{**raw["layers"][0], **bad}]})
  wide = json.loads(json.dumps(raw["layers"][1]))
  wide["mixer"]["rot"]["dims"] = wide["mixer"]["rot_dim"] + 2
  with pytest.raises(ValueError):
    hybrid_model_config({**raw, "layers": [wide]})


def test_decay_rank_comes_from_the_checkpoint(tmp_path):
  raw = json.loads(json.dumps(model_cards["rurutar-tiny"]["hf_config"]))
  for lc in raw["layers"]:
    lc["mixer"].pop("rank", None)
  cfg = hybrid_model_config(raw)
  assert cfg["layers"][0]["rank"] == 0
  resolve_tensor_sizes(cfg, rurutar_param_shapes(raw, rank=11))
  assert cfg["layers"][0]["rank"] == 11 and cfg["layers"][2]["rank"] == 11
  with pytest.raises(ValueError):
    resolve_tensor_sizes(hybrid_model_config(raw), {})
  p = write_random_checkpoint(tmp_path / "m", raw, seed=1)      # the rank is only in the file's header
  assert load_model_config(p / "config.json")["layers"][0]["rank"] == 16


def test_checkpoint_on_disk_round_trip(tmp_path):
  raw = model_cards["rurutar-tiny"]["hf_config"]
  p = write_random_checkpoint(tmp_path / "m", raw, seed=1)
  cfg = load_model_config(p / "config.json")
  assert cfg["architecture"] == "Rurutar" and cfg["num_layers"] == len(raw["layers"])
  sh = rurutar_param_shapes(raw)
  assert sh["final.norm.alpha"] == () and sh["l0.norm1.b"] == (raw["width"],) and "l2.norm2" not in sh
  assert "l3.mix.dkv" not in sh and "l1.mix.dkv" in sh and sh["l1.mlp.shared.sg"] == (1, raw["width"])
  assert sh["l0.mix.a1"] == (raw["layers"][0]["mixer"]["rank"], raw["width"]) and sh["l0.mix.norm"] == (raw["layers"][0]["mixer"]["vdim"],)
  w = random_rurutar_state(raw, seed=1)
  assert set(w) == set(sh) and all(tuple(w[k].shape) == tuple(v) for k, v in sh.items())
  for mid in ("rurutar-tiny", "rurutar-1b"):
    assert hybrid_model_config(model_cards[mid]["hf_config"])["num_layers"] == model_cards[mid]["layers"]


def test_oracle_pieces():
  rng = np.random.default_rng(0)
  # rotation keeps the length of a pair up to the factor, pairs i with i + dims / 2, and passes what lies behind
  rot = {"base": 1000.0, "dims": 6, "scaling": {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 1.0}}
  y = rng.standard_normal((3, 2, 8))
  z = O.rotate(y, [0, 5, 9], rot)
  mult = 0.1 * math.log(8.0) + 1.0
  assert np.allclose(z[..., 6:], y[..., 6:]) and np.allclose(z[0, :, :6], mult * y[0, :, :6])
  for i in range(3):
    assert np.allclose(z[..., i] ** 2 + z[..., i + 3] ** 2, mult ** 2 * (y[..., i] ** 2 + y[..., i + 3] ** 2))
  fr, m = O.frequencies({"base": 10000.0, "dims": 32, "scaling": {"factor": 16.0, "original": 512, "fast": 32.0, "slow": 1.0}})
  assert m == 0.1 * math.log(16.0) + 1.0 and fr[0] == 1.0 and abs(fr[-1] - 10000.0 ** (-30 / 32) / 16.0) < 1e-18
  assert O.frequencies({"base": 10.0, "dims": 4})[1] == 1.0
  # routing: weights are a softmax among the chosen logits alone
  w = O.route(np.array([0.0, 3.0, 2.0, 2.5]), 2)
  assert sorted(w) == [1, 3] and abs(w[1] / w[3] - math.exp(0.5)) < 1e-12 and abs(sum(w.values()) - 1.0) < 1e-12
  assert O.route(np.array([1.0, 7.0]), 1) == {1: 1.0}
  # the tanh norm looks at one channel at a time
  st = {"n": torch.tensor([2.0, 3.0]), "n.b": torch.tensor([0.5, -1.0]), "n.alpha": torch.tensor(0.7)}
  assert np.allclose(O.squash(st, "n", np.array([[1.0, -2.0]])), [[2.0 * math.tanh(0.7) + 0.5, 3.0 * math.tanh(-1.4) - 1.0]])
  # gated linear attention with a decay that forgets nothing is a plain sum; with one that forgets at once, the last token
  D, H, n, dv = 4, 1, 2, 3
  st = {f"p.{k}": torch.randn(r, D, generator=torch.Generator().manual_seed(i), dtype=torch.float64)
        for i, (k, r) in enumerate([("q", n), ("k", n), ("v", dv), ("g", dv), ("a1", 2)])}
  st.update({"p.a2": torch.zeros(n, 2), "p.norm": torch.ones(dv), "p.o": torch.eye(dv, D, dtype=torch.float64).T.contiguous()})
  mx = {"heads": H, "dim": n, "vdim": dv, "tau": 2.0}
  h = rng.standard_normal((3, D))
  q, k, v, g = (h @ st["p." + x].numpy().T for x in "qkvg")
  for off, last in ((60.0, False), (-400.0, True)):
    st["p.a2.b"] = torch.full((n,), off)
    S = sum(np.outer(k[t], v[t]) for t in range(3)) if not last else np.outer(k[2], v[2])
    o = S.T @ q[2] / math.sqrt(n)
    o = o / math.sqrt((o ** 2).mean()) * O.silu(g[2])
    assert np.allclose(O.gated_linear_attention(st, "p.", mx, h, 0.0)[2, :3], o)
  # a window of one token: every query reads its own value, whatever the scores
  D, R, dr = 5, 3, 2
  gen = torch.Generator().manual_seed(9)
  st = {f"p.{k}": torch.randn(*s, generator=gen, dtype=torch.float64) for k, s in
        {"dq": (4, D), "uq": (2 * 4, 4), "dkv": (R + dr, D), "uk": (2 * 2, R), "uv": (2 * 3, R), "g": (2, D), "o": (D, 6)}.items()}
  st.update({"p.dq.norm": torch.ones(4), "p.dkv.norm": torch.ones(R)})
  mx = {"heads": 2, "dim": 2, "rot_dim": dr, "vdim": 3, "kv_rank": R, "scale": 0.4, "mask": {"size": 1}, "rot": {"base": 100.0, "dims": dr}}
  h = rng.standard_normal((4, D))
  c, kr = O.latent_rows(st, "p.", mx, h, 0.0)
  val = (c @ st["p.uv"].numpy().T).reshape(4, 2, 3) * O.sigmoid(h @ st["p.g"].numpy().T)[:, :, None]
  assert np.allclose(O.latent_attention(st, "p.", mx, h, 0.0, c, kr), val.reshape(4, 6) @ st["p.o"].numpy().T)
