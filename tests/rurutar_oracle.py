"""Rurutar restated from its equations: a plain, slow float64 implementation, one function per mechanism.

It shares no code with the engine.  ``state``: name -> torch tensor (any float type; everything is taken to float64),
``cfg``: the design's ``config.json`` as a dict.  Attention is evaluated with dense ``[T, T]`` score matrices over expanded
keys and values, the linear attention token by token.

Notation.  A layer works on the stream ``x`` [T, D]:

    x <- x + mixer(f1(x)),      x <- x + ff(f2(x)),      f(x) = tanh(a x) * w + b   (a one number; w, b per channel)
"""
import math

import numpy as np
import torch


def _t(state, name):
  return state[name].detach().to(torch.float64).cpu().numpy()


def rms(y, w, eps):
  """Rows divided by their root mean square (eps inside the root), times a plain weight."""
  return y / np.sqrt(np.mean(y * y, axis=-1, keepdims=True) + eps) * w


def squash(state, name, x):
  """The norm of the stream: it looks at one channel at a time."""
  return np.tanh(_t(state, name + ".alpha").reshape(()) * x) * _t(state, name) + _t(state, name + ".b")


def sigmoid(z):
  return 1.0 / (1.0 + np.exp(-z))


def silu(z):
  return z * sigmoid(z)


def gelu_tanh(z):
  return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
  """(frequency per pair, factor on cos and sin) of a rotary part, rescaled along a ramp over the pair index."""
  n, base = int(rot["dims"]), float(rot["base"])
  f = [base ** (-2.0 * i / n) for i in range(n // 2)]
  sc = rot.get("scaling")
  if not sc:
    return np.array(f), 1.0
  fac, orig = float(sc["factor"]), float(sc["original"])
  turns = lambda t: n * math.log(orig / (2.0 * math.pi * t)) / (2.0 * math.log(base))  # noqa: E731
  lo = max(math.floor(turns(float(sc["fast"]))), 0)
  hi = min(math.ceil(turns(float(sc["slow"]))), n - 1)
  out = []
  for i, v in enumerate(f):
    r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
    out.append(v / fac * r + v * (1.0 - r))
  return np.array(out), 0.1 * math.log(fac) + 1.0


def rotate(y, pos, rot):
  """Last axis of y [T, ..., n]: entries i and i + dims/2 turn together by pos * frequency i; entries from dims on pass."""
  fr, mult = frequencies(rot)
  h = len(fr)
  ang = np.asarray(pos, dtype=np.float64)[:, None] * fr
  c, s = np.cos(ang) * mult, np.sin(ang) * mult
  while c.ndim < y.ndim:
    c, s = c[:, None], s[:, None]
  u, v = y[..., :h], y[..., h:2 * h]
  return np.concatenate([u * c - v * s, v * c + u * s, y[..., 2 * h:]], axis=-1)


def gated_linear_attention(state, pre, mx, h, eps):
  """A [dim, vdim] state per head: every key channel fades by its own factor before k v^T is added; the query reads the state
  after its own token has joined it."""
  T = h.shape[0]
  H, n, dv, tau = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"]), float(mx["tau"])
  q = (h @ _t(state, pre + "q").T).reshape(T, H, n) / math.sqrt(n)
  k = (h @ _t(state, pre + "k").T).reshape(T, H, n)
  v = (h @ _t(state, pre + "v").T).reshape(T, H, dv)
  z = (h @ _t(state, pre + "a1").T) @ _t(state, pre + "a2").T + _t(state, pre + "a2.b")
  fade = (sigmoid(z) ** (1.0 / tau)).reshape(T, H, n)
  S = np.zeros((H, n, dv))
  o = np.zeros((T, H, dv))
  for t in range(T):
    S = fade[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
    o[t] = np.einsum("hnv,hn->hv", S, q[t])
  o = rms(o, _t(state, pre + "norm"), eps).reshape(T, H * dv)
  return (o * silu(h @ _t(state, pre + "g").T)) @ _t(state, pre + "o").T


def latent_rows(state, pre, mx, h, eps):
  """What a token leaves for later ones: its normed latent and one rotated key part for all heads."""
  R = int(mx["kv_rank"])
  d = h @ _t(state, pre + "dkv").T
  return rms(d[:, :R], _t(state, pre + "dkv.norm"), eps), rotate(d[:, R:], np.arange(h.shape[0]), mx["rot"])


def latent_attention(state, pre, mx, h, eps, c, kr):
  """Queries through a normed latent of their own; keys and values are per-head images of c (kr: the rotated key part);
  softmax over the last mask.size positions; one sigmoid gate per head."""
  T = h.shape[0]
  H, n, dr, dv = int(mx["heads"]), int(mx["dim"]), int(mx["rot_dim"]), int(mx["vdim"])
  q = rms(h @ _t(state, pre + "dq").T, _t(state, pre + "dq.norm"), eps) @ _t(state, pre + "uq").T
  q = q.reshape(T, H, n + dr)
  qu, qr = q[..., :n], rotate(q[..., n:], np.arange(T), mx["rot"])
  k = (c @ _t(state, pre + "uk").T).reshape(T, H, n)
  v = (c @ _t(state, pre + "uv").T).reshape(T, H, dv)
  i, j = np.arange(T)[:, None], np.arange(T)[None, :]
  seen = (j <= i) & (i - j < int(mx["mask"]["size"]))
  gate = sigmoid(h @ _t(state, pre + "g").T)
  out = np.zeros((T, H, dv))
  for a in range(H):
    s = np.where(seen, (qu[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * float(mx["scale"]), -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    out[:, a] = (e / e.sum(axis=1, keepdims=True)) @ v[:, a] * gate[:, a:a + 1]
  return out.reshape(T, H * dv) @ _t(state, pre + "o").T


def dense(state, pre, h):
  return (gelu_tanh(h @ _t(state, pre + "gate").T) * (h @ _t(state, pre + "up").T)) @ _t(state, pre + "down").T


def expert(state, pre, h):
  return (silu(h @ _t(state, pre + "gate").T) * (h @ _t(state, pre + "up").T)) @ _t(state, pre + "down").T


def route(z, top):
  """Router logits of one token -> {expert: weight}: the largest logits, weights a softmax among the chosen."""
  best = sorted(range(len(z)), key=lambda e: (-z[e], e))[:top]
  w = np.exp(np.array([z[e] for e in best]) - z[best[0]])
  return dict(zip(best, w / w.sum()))


def experts(state, pre, mlp, h):
  E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
  Z = h @ _t(state, pre + "router").T
  picks = [route(z, top) for z in Z]
  y = np.zeros_like(h)
  for e in range(E):
    rows = [t for t in range(h.shape[0]) if e in picks[t]]
    if rows:
      y[rows] += np.array([picks[t][e] for t in rows])[:, None] * expert(state, f"{pre}e{e}.", h[rows])
  if mlp.get("shared"):
    y += sigmoid(h @ _t(state, pre + "shared.sg").T) * expert(state, pre + "shared.", h)
  return y


def forward(state, cfg, tokens, want_layers=False):
  """tokens of ONE sequence from position 0 -> float64 logits [T, vocab] (and the stream after every layer)."""
  eps = float(cfg["norm"]["eps"])
  x = _t(state, "embed")[np.asarray(tokens, dtype=np.int64)] * float(cfg["embedding"]["scale"])
  per_layer, left = [], {}
  for li, lc in enumerate(cfg["layers"]):
    p, mx = f"l{li}.", lc["mixer"]
    h = squash(state, p + "norm1", x)
    if lc["type"] == "gla":
      x = x + gated_linear_attention(state, p + "mix.", mx, h, eps)
    else:
      if mx.get("kv_from") is None:
        left[li] = latent_rows(state, p + "mix.", mx, h, eps)
      x = x + latent_attention(state, p + "mix.", mx, h, eps, *left[li if mx.get("kv_from") is None else int(mx["kv_from"])])
    mlp = lc.get("mlp")
    if mlp is not None:
      h = squash(state, p + "norm2", x)
      x = x + (dense(state, p + "mlp.", h) if mlp["kind"] == "dense" else experts(state, p + "mlp.", mlp, h))
    per_layer.append(x.copy())
  logits = squash(state, "final.norm", x) @ _t(state, "head").T
  cap = float(cfg.get("logit_softcap") or 0.0)
  if cap > 0.0:
    logits = cap * np.tanh(logits / cap)
  return (logits, per_layer) if want_layers else logits
