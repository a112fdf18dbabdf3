"""Sizolorn restated from its equations: a plain, slow float64 implementation, one function per mechanism.

It shares no code with the engine.  ``state``: name -> torch tensor (any float type; everything is taken to float64),
``cfg``: the design's ``config.json`` as a dict.  Attention is evaluated with dense ``[T, T]`` score matrices, the matrix
memory token by token, the experts expert by expert.

Notation.  The stream is s copies X [T, s, D] of one width; for every sublayer (a = read weights [s], b = write weights
[s], M = mixing matrix [from, to]):

    u = sum_i a_i X_i,      y = sublayer(f(u)),      X_j <- sum_i M_ij X_i + b_j y,      f(u) = (u - mean) / std * w
"""
import math

import numpy as np
import torch


def _t(state, name):
  return state[name].detach().to(torch.float64).cpu().numpy()


def layer_norm(y, w, eps):
  """Rows with their mean taken off, divided by the root of (mean squared deviation + eps), times a weight per channel."""
  d = y - y.mean(axis=-1, keepdims=True)
  return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w


def unit_rms(y, eps):
  return y / np.sqrt(np.mean(y * y, axis=-1, keepdims=True) + eps)


def sigmoid(z):
  return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
  return -np.logaddexp(0.0, -z)


# ----------------------------------------------------------------------------- the stream of several copies
def read_streams(state, pre, X):
  return np.einsum("tsd,s->td", X, _t(state, pre + "in"))


def write_streams(state, pre, X, y):
  return np.einsum("tsd,sr->trd", X, _t(state, pre + "mix")) + _t(state, pre + "out")[None, :, None] * y[:, None, :]


# ----------------------------------------------------------------------------- attention
def frequencies(rot):
  """base^(-2i/dims); with band scaling, short wavelengths keep theirs, long ones are divided, between them a blend."""
  n, base = int(rot["dims"]), float(rot["base"])
  sc, out = rot.get("scaling"), []
  for i in range(n // 2):
    f = base ** (-2.0 * i / n)
    if sc:
      wave, fac, orig, low, high = 2.0 * math.pi / f, float(sc["factor"]), float(sc["original"]), float(sc["low"]), float(sc["high"])
      if wave > orig / low:
        f = f / fac
      elif wave >= orig / high:
        s = (orig / wave - low) / (high - low)
        f = (1.0 - s) * f / fac + s * f
    out.append(f)
  return np.array(out)


def rotate(y, pos, rot, neighbours):
  """y [T, heads, n]: pairs (2i, 2i + 1) when neighbours, else (i, i + dims/2), turned by pos * frequency i."""
  if not rot or not int(rot["dims"]):
    return y
  n = int(rot["dims"])
  first = np.arange(0, n, 2) if neighbours else np.arange(n // 2)
  second = first + 1 if neighbours else first + n // 2
  ang = np.asarray(pos, dtype=np.float64)[:, None] * frequencies(rot)
  c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
  out = y.copy()
  out[..., first] = y[..., first] * c - y[..., second] * s
  out[..., second] = y[..., second] * c + y[..., first] * s
  return out


def short_filter(u, w):
  """y_t = sum_j w[:, j] u_(t - taps + 1 + j), nothing before the first row."""
  taps = w.shape[1]
  past = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
  return sum(w[:, j] * past[j:j + u.shape[0]] for j in range(taps))


def seen_window(T, size):
  i, j = np.arange(T)[:, None], np.arange(T)[None, :]
  return (j <= i) & (i - j < size)


def seen_chunk(T, size):
  i, j = np.arange(T)[:, None], np.arange(T)[None, :]
  return (j <= i) & (i // size == j // size)


def weigh_values(q, k, v, seen, scale):
  """Softmax attention: q [T, H, n], k [T, G, n], v [T, G, m]; query head h meets key head h // (H / G)."""
  H, G = q.shape[1], k.shape[1]
  out = np.zeros((q.shape[0], H, v.shape[2]))
  for h in range(H):
    g = h // (H // G)
    s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
  return out


def project(state, name, h):
  y = h @ _t(state, name).T
  return y + _t(state, name + ".b") if name + ".b" in state else y


def attention(state, pre, mx, h, eps, kind):
  """kind: "filtered" (filters, whole-projection norms, neighbour pairs, chunks, head gates), "unit" (neighbour pairs, unit
  heads after the rotation, chunks) or "window" (half-split pairs, a sliding window, head gates)."""
  T = h.shape[0]
  H, G, n, m = (int(mx[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
  q, k, v = (project(state, pre + s, h) for s in "qkv")
  if kind == "filtered":
    if mx.get("conv"):
      q, k, v = (short_filter(a, _t(state, f"{pre}{s}.conv")) for a, s in ((q, "q"), (k, "k"), (v, "v")))
    q, k = unit_rms(q, eps) * _t(state, pre + "q.norm"), unit_rms(k, eps) * _t(state, pre + "k.norm")
  pos = np.arange(T)
  q, k = (rotate(a.reshape(T, x, n), pos, mx.get("rot"), kind != "window") for a, x in ((q, H), (k, G)))
  if kind == "unit":
    q, k = unit_rms(q, eps), unit_rms(k, eps)
  size = int(mx["mask"]["size"])
  o = weigh_values(q, k, v.reshape(T, G, m), seen_window(T, size) if kind == "window" else seen_chunk(T, size), float(mx["scale"]))
  if kind != "unit":
    o = o * sigmoid(h @ _t(state, pre + "g").T)[:, :, None]
  return project(state, pre + "o", o.reshape(T, H * m))


# ----------------------------------------------------------------------------- matrix memory
def matrix_memory(state, pre, mx, h, eps):
  """Per head a [n, m] memory and an [n] normaliser, both kept relative to exp(running maximum); the write strength is
  exp(i), the fade exp(f); the query reads after its own token was written."""
  T = h.shape[0]
  H, n, m, cap = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"]), float(mx["gate_cap"])
  q = (h @ _t(state, pre + "q").T).reshape(T, H, n) / math.sqrt(n)
  k = (h @ _t(state, pre + "k").T).reshape(T, H, n)
  v = (h @ _t(state, pre + "v").T).reshape(T, H, m)
  li = cap * np.tanh(project(state, pre + "i", h) / cap)
  lf = log_sigmoid(cap * np.tanh(project(state, pre + "f", h) / cap))
  S, N, top = np.zeros((H, n, m)), np.zeros((H, n)), np.zeros(H)
  o = np.zeros((T, H, m))
  for t in range(T):
    new = np.maximum(lf[t] + top, li[t])
    fade, write = np.exp(lf[t] + top - new), np.exp(li[t] - new)
    S = fade[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
    N = fade[:, None] * N + write[:, None] * k[t]
    top = new
    size = np.maximum(np.abs(np.einsum("hn,hn->h", N, q[t])), np.exp(-top)) + 1e-6
    o[t] = np.einsum("hnm,hn->hm", S, q[t]) / size[:, None]
  o = unit_rms(o, eps).reshape(T, H * m) * _t(state, pre + "norm") * sigmoid(h @ _t(state, pre + "g").T)
  return o @ _t(state, pre + "o").T


def mixer(state, pre, lc, h, eps):
  mx = lc["mixer"]
  if lc["type"] == "parallel":
    left = attention(state, pre + "left.", mx["left"], h, eps, "window")
    return float(mx["left_scale"]) * left + float(mx["right_scale"]) * matrix_memory(state, pre + "right.", mx["right"], h, eps)
  return attention(state, pre, mx, h, eps, {"attention": "filtered", "attention_2": "unit"}[lc["type"]])


# ----------------------------------------------------------------------------- experts
def expert(state, pre, h):
  return np.maximum(h @ _t(state, pre + "up").T, 0.0) ** 2 @ _t(state, pre + "down").T


def route(z, correction, top):
  """Router logits of one token -> {output: weight}: chosen by softmax score + correction, weighted by the scores alone."""
  s = np.exp(z - z.max())
  s = s / s.sum()
  best = sorted(range(len(z)), key=lambda e: (-(s[e] + correction[e]), e))[:top]
  w = s[best] / (s[best].sum() + 1e-20)
  return dict(zip(best, w))


def experts(state, pre, mlp, h):
  """Router outputs behind the experts hand the input itself on."""
  E, same, top = int(mlp["router"]["experts"]), int(mlp["router"].get("identity", 0)), int(mlp["router"]["top"])
  Z, corr = h @ _t(state, pre + "router").T, _t(state, pre + "correction")
  picks = [route(z, corr, top) for z in Z]
  y = np.zeros_like(h)
  for e in range(E + same):
    rows = [t for t in range(h.shape[0]) if e in picks[t]]
    if rows:
      w = np.array([picks[t][e] for t in rows])[:, None]
      y[rows] += w * (expert(state, f"{pre}e{e}.", h[rows]) if e < E else h[rows])
  if mlp.get("shared"):
    y += sigmoid(h @ _t(state, pre + "shared.sg").T) * expert(state, pre + "shared.", h)
  return y


def forward(state, cfg, tokens, want_layers=False):
  """tokens of ONE sequence from position 0 -> float64 logits [T, vocab] (and the sum of the streams after every layer)."""
  eps = float(cfg["norm"]["eps"])
  emb = _t(state, "embed")
  x = emb[np.asarray(tokens, dtype=np.int64)]
  X = np.repeat(x[:, None, :], int(cfg["streams"]), axis=1)
  per_layer = []
  for li, lc in enumerate(cfg["layers"]):
    p = f"l{li if lc.get('weights_of') is None else int(lc['weights_of'])}."
    y = mixer(state, p + "mix.", lc, layer_norm(read_streams(state, p + "hc1.", X), _t(state, p + "norm1"), eps), eps)
    X = write_streams(state, p + "hc1.", X, y)
    if lc.get("mlp") is not None:
      y = experts(state, p + "mlp.", lc["mlp"], layer_norm(read_streams(state, p + "hc2.", X), _t(state, p + "norm2"), eps))
      X = write_streams(state, p + "hc2.", X, y)
    per_layer.append(X.sum(axis=1))
  logits = layer_norm(X.sum(axis=1), _t(state, "final.norm"), eps) @ emb.T
  return (logits, per_layer) if want_layers else logits
