"""Plain, slow restatement of the Fekanex design in torch (fp32 or fp64, CPU): one function per mechanism, whole sequences at once,
no cache, no batching.  The product path (libxotb200_lm.so) shares no code with this file; the tests compare the two on small
random models.

Notation: T tokens, D width, H query heads, G key/value heads, dk / dv query-key / value head sizes, E experts."""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

Tensor = torch.Tensor

GLU_SLOPE = 1.702          # slope of the sigmoid inside the dense feed-forward's gate


def unit_rms(x: Tensor, eps: float) -> Tensor:
  return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def bigram_rows(tokens: Tensor, b: dict) -> Tensor:
  """row of the bigram table for every token: a hash of (token before it, token); the first token of a sequence has the last row"""
  rows = torch.full_like(tokens, b["buckets"])
  rows[1:] = (tokens[:-1] * b["mul_prev"] + tokens[1:] * b["mul_cur"]) % b["buckets"]
  return rows


def embedding(tokens: Tensor, W: Dict[str, Tensor], e: dict) -> Tensor:
  x = W["embed"][tokens] * e.get("scale", 1.0)
  if e.get("bigram"):
    x = x + W["bigram"][bigram_rows(tokens, e["bigram"])]
  return x


def causal_filter(u: Tensor, w: Tensor) -> Tensor:
  """u [T, C], w [C, taps]: the last tap multiplies the current row, zeros before the first row"""
  taps = w.shape[1]
  padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
  return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def frequencies(rot: dict) -> Tuple[Tensor, float]:
  """(angle per position of every plane, factor of both cosine and sine).  With scaling, planes that turn more than `fast` times over the
  original length keep their frequency, those that turn fewer than `slow` times are slowed by the factor, a linear blend between."""
  d, base = rot["dims"], float(rot["base"])
  i = torch.arange(d // 2, dtype=torch.float64)
  f = base ** (-2.0 * i / d)
  s = rot.get("scaling")
  if not s:
    return f, 1.0
  plane = lambda turns: d * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
  lo, hi = max(math.floor(plane(s["fast"])), 0), min(math.ceil(plane(s["slow"])), d - 1)
  ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
  return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def turn(x: Tensor, rot: Optional[dict]) -> Tensor:
  """x [T, heads, d]: the planes (2i, 2i + 1) among the first rot.dims entries turned by position * frequency"""
  if not rot or rot["dims"] == 0:
    return x
  n = rot["dims"]
  f, mul = frequencies(rot)
  ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
  c, s = (torch.cos(ang) * mul).to(x.dtype), (torch.sin(ang) * mul).to(x.dtype)
  u, v = x[..., 0:n:2], x[..., 1:n:2]
  out = x.clone()
  out[..., 0:n:2] = u * c - v * s
  out[..., 1:n:2] = v * c + u * s
  return out


def visible(T: int, mask: Optional[dict]) -> Tensor:
  """[T, T] bool: row i sees the keys up to i, of those the last `size` and the first `keep_first`"""
  i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
  ok = j <= i
  if mask and mask.get("size"):
    ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
  return ok


def softmax_one_more(scores: Tensor) -> Tensor:
  """exp(s) / (1 + sum exp(s)) over the last dimension"""
  top = scores.max(dim=-1, keepdim=True).values.clamp(min=0.0)
  e = torch.exp(scores - top)
  return e / (e.sum(dim=-1, keepdim=True) + torch.exp(-top))


def projected(h: Tensor, W: Dict[str, Tensor], name: str) -> Tensor:
  u = h @ W[name].T + W[name + ".b"]
  return causal_filter(u, W[name + ".conv"]) if name + ".conv" in W else u


def attention(h: Tensor, W: Dict[str, Tensor], m: dict, eps: float, first_values: Optional[Tensor]) -> Tuple[Tensor, Tensor]:
  """(mixer output, the values before they are mixed).  first_values: those of the first mixing layer; None = no mixing here."""
  T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
  q = unit_rms(turn(projected(h, W, "q").reshape(T, H, dk), m.get("rot")), eps)
  k = unit_rms(turn(projected(h, W, "k").reshape(T, G, dk), m.get("rot")), eps)
  own = projected(h, W, "v").reshape(T, G, dv)
  v = own if first_values is None else (1 - W["vmix"]) * own + W["vmix"] * first_values
  k, v = (t.repeat_interleave(H // G, dim=1) for t in (k, v))
  s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
  p = softmax_one_more(s.masked_fill(~visible(T, m.get("mask")), -math.inf))
  return torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * dv) @ W["o"].T, own


def dense_ff(h: Tensor, W: Dict[str, Tensor], limit: float) -> Tensor:
  g = torch.clamp(h @ W["gate"].T, max=limit)
  u = torch.clamp(h @ W["up"].T, min=-limit, max=limit)
  return (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1.0)) @ W["down"].T


def expert(h: Tensor, W: Dict[str, Tensor]) -> Tensor:
  z = h @ W["gate"].T
  return (z * torch.sigmoid(z) * (h @ W["up"].T)) @ W["down"].T


def route(h: Tensor, W: Dict[str, Tensor], r: dict, gaps: Optional[list] = None) -> Tuple[Tensor, Tensor]:
  """(ids [T, top], weights [T, top]).  `gaps` collects per row the lead of the last chosen expert over the best one left out."""
  z = h @ W["router"].T
  order = torch.sort(z, dim=-1, descending=True, stable=True)
  top = r["top"]
  if gaps is not None:
    gaps.append((order.values[:, top - 1] - order.values[:, top]).double() if top < r["experts"] else torch.full((h.shape[0],), math.inf, dtype=torch.float64))
  return order.indices[:, :top], torch.softmax(order.values[:, :top], dim=-1)


def moe_ff(h: Tensor, W: Dict[str, Tensor], mlp: dict, gaps: Optional[list] = None) -> Tensor:
  ids, w = route(h, W, mlp["router"], gaps)
  out = torch.zeros_like(h)
  for e in range(mlp["router"]["experts"]):
    t, k = torch.where(ids == e)
    if t.numel():
      out[t] += w[t, k][:, None] * expert(h[t], sub(W, f"e{e}."))
  return out


def sub(weights: Dict[str, Tensor], prefix: str) -> Dict[str, Tensor]:
  return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: Dict[str, Tensor], tokens, dtype=torch.float64, gaps: Optional[list] = None) -> Tuple[Tensor, List[Tensor]]:
  """logits [T, vocab] of one whole sequence and the residual stream after every layer"""
  Wt = {k: v.to(dtype) for k, v in weights.items()}
  eps = cfg["norm"]["eps"]
  x = embedding(torch.as_tensor(tokens, dtype=torch.long), Wt, cfg["embedding"])
  trail, first_values, seen_mix = [], None, False
  for i, layer in enumerate(cfg["layers"]):
    p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
    h = unit_rms(x, eps) * Wt[p + "norm1"]
    mixes = bool(m.get("v_mix"))
    y, own = attention(h, sub(Wt, p + "mix."), m, eps, first_values if mixes and seen_mix else None)
    if mixes and not seen_mix:
      first_values, seen_mix = own, True
    if mlp is not None:
      W = sub(Wt, p + "mlp.")
      y = y + (dense_ff(h, W, mlp["limit"]) if mlp["kind"] == "dense" else moe_ff(h, W, mlp, gaps))
    x = x + y
    trail.append(x)
  return unit_rms(x, eps) * Wt["final.norm"] @ Wt["embed"].T * cfg.get("logit_scale", 1.0), trail


# ---- small random models -------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
  D, V = cfg["width"], cfg["vocab"]
  out: Dict[str, Tuple[int, ...]] = {"embed": (V, D), "final.norm": (D,)}
  if cfg["embedding"].get("bigram"):
    out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, D)
  for i, layer in enumerate(cfg["layers"]):
    p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
    out[p + "norm1"] = (D,)
    for name, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
      out.update({p + f"mix.{name}": (n, D), p + f"mix.{name}.b": (n,)})
      if m.get("conv"):
        out[p + f"mix.{name}.conv"] = (n, m["conv"])
    out[p + "mix.o"] = (D, m["heads"] * m["vdim"])
    if m.get("v_mix"):
      out[p + "mix.vmix"] = ()
    if mlp is None:
      continue
    if mlp["kind"] == "dense":
      out.update({p + "mlp.gate": (mlp["ff"], D), p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
    else:
      E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
      out[p + "mlp.router"] = (E, D)
      for e in range(E):
        out.update({p + f"mlp.e{e}.gate": (F, D), p + f"mlp.e{e}.up": (F, D), p + f"mlp.e{e}.down": (D, F)})
  return out


def random_weights(cfg: dict, seed: int) -> Dict[str, Tensor]:
  """bf16-representable random weights (a 16-bit engine and this oracle start from identical numbers)"""
  g = torch.Generator().manual_seed(seed)
  rnd = lambda shape, mean, dev: mean + dev * torch.randn(shape, generator=g)
  out = {}
  for name, shape in tensor_shapes(cfg).items():
    last = name.rsplit(".", 1)[-1]
    if last == "vmix":
      t = rnd(shape, 0.4, 0.15)
    elif last == "b":
      t = rnd(shape, 0.0, 0.3)
    elif last == "conv":
      t = rnd(shape, 0.0, 0.6)
      t[:, -1] += 0.8
    elif "norm" in last:
      t = rnd(shape, 1.0, 0.2)
    elif name in ("embed", "bigram"):
      t = rnd(shape, 0.0, 1.0 if name == "embed" else 0.5)
    elif last in ("gate", "up"):
      t = rnd(shape, 0.0, 1.6 / math.sqrt(shape[1]))  # some entries beyond the clamp
    else:
      t = rnd(shape, 0.0, 1.0 / math.sqrt(shape[1]))
    out[name] = t.to(torch.bfloat16).to(torch.float32)
  return out
