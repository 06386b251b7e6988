"""Plain, slow restatement of the Rinutar design in torch (fp32 or fp64, CPU): one function per mechanism, whole sequences at once,
no cache, no batching.  The product path (libxotb200_lm.so) shares no code with this file; the tests compare the two on small
random models.

Notation: T tokens, D width, H heads, dn / dr unrotated / rotated query-key sizes, dv value size, R latent rank, E experts."""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

Tensor = torch.Tensor

GLU_SLOPE = 1.702          # slope of the sigmoid inside the experts' gate


def dyt(x: Tensor, alpha: Tensor, w: Tensor, b: Tensor) -> Tensor:
  """Dynamic Tanh: no statistic of the row, every entry by itself"""
  return torch.tanh(alpha * x) * w + b


def rms_norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
  return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * w


def turn(x: Tensor, base: float) -> Tensor:
  """x [T, ..., d]: row t turned by the angles t * base^(-2i/d) in the planes (i, i + d/2)"""
  T, d = x.shape[0], x.shape[-1]
  if d == 0:
    return x
  half = d // 2
  f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / d)
  ang = (torch.arange(T, dtype=torch.float64)[:, None] * f[None, :]).reshape([T] + [1] * (x.dim() - 2) + [half])
  c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
  u, v = x[..., :half], x[..., half:]
  return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def softmax_with_sink(scores: Tensor, sink: Tensor) -> Tensor:
  """scores [H, T, T] (minus infinity where a key is not seen), sink [H]: weights exp(s) / (exp(sink) + sum exp(s))"""
  top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink[:, None, None])
  e = torch.exp(scores - top)
  return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def latent_mixer(h: Tensor, W: Dict[str, Tensor], m: dict, eps: float) -> Tensor:
  """Keys and values of every head come out of one normed latent row per token; one more, rotated, key part is shared by the heads."""
  T, H, dn, dr, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
  base = (m.get("rot") or {}).get("base", 10000.0)
  q = (h @ W["q"].T).reshape(T, H, dn + dr)
  down = h @ W["dkv"].T
  c = rms_norm(down[:, :R], W["dkv.norm"], eps)
  shared_key = turn(down[:, R:], base)
  q_rot = turn(q[..., dn:], base)
  k = (c @ W["uk"].T).reshape(T, H, dn)
  v = (c @ W["uv"].T).reshape(T, H, dv)
  s = (torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", q_rot, shared_key)) * m["scale"]
  later = torch.ones(T, T).triu(1).bool()
  p = softmax_with_sink(s.masked_fill(later, -math.inf), W["sink"])
  return torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * dv) @ W["o"].T


def gelu_tanh(z: Tensor) -> Tensor:
  return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h: Tensor, W: Dict[str, Tensor]) -> Tensor:
  return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def expert(h: Tensor, W: Dict[str, Tensor], limit: float) -> Tensor:
  g = torch.clamp(h @ W["gate"].T, max=limit)
  u = torch.clamp(h @ W["up"].T, min=-limit, max=limit)
  return (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1.0)) @ W["down"].T


def route(h: Tensor, W: Dict[str, Tensor], r: dict, gaps: Optional[list] = None) -> Tuple[Tensor, Tensor]:
  """(ids [T, top], weights [T, top]).  `gaps` collects per row the smallest lead of a choice that was made (an expert over the best
  one left out, a kept group over the best one dropped)."""
  E, top = r["experts"], r["top"]
  s = torch.sigmoid(h @ W["router"].T)
  choice = s + W["correction"]
  T = h.shape[0]
  gap = torch.full((T,), math.inf, dtype=torch.float64)
  groups = r.get("groups")
  if groups:
    count, keep = groups["count"], groups["keep"]
    per = E // count
    best = torch.sort(choice.reshape(T, count, per), dim=-1, descending=True).values
    score = best[..., :min(2, per)].sum(-1)
    order = torch.sort(score, dim=-1, descending=True, stable=True)
    if keep < count:
      gap = torch.minimum(gap, (order.values[:, keep - 1] - order.values[:, keep]).double())
    dropped = torch.ones(T, count).bool()
    dropped.scatter_(1, order.indices[:, :keep], False)
    choice = choice.masked_fill(dropped.repeat_interleave(per, dim=1), -math.inf)
  order = torch.sort(choice, dim=-1, descending=True, stable=True)
  ids = order.indices[:, :top]
  if top < E:
    gap = torch.minimum(gap, (order.values[:, top - 1] - order.values[:, top]).double())
  w = torch.gather(s, 1, ids)
  w = w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"]
  if gaps is not None:
    gaps.append(gap)
  return ids, w


def moe_ff(h: Tensor, W: Dict[str, Tensor], mlp: dict, gaps: Optional[list] = None) -> Tensor:
  ids, w = route(h, W, mlp["router"], gaps)
  out = torch.zeros_like(h)
  for e in range(mlp["router"]["experts"]):
    t, k = torch.where(ids == e)
    if t.numel():
      out[t] += w[t, k][:, None] * expert(h[t], sub(W, f"e{e}."), mlp["expert"]["limit"])
  return out


def sub(weights: Dict[str, Tensor], prefix: str) -> Dict[str, Tensor]:
  return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def owner(cfg: dict, i: int) -> int:
  """the layer whose tensors layer i uses"""
  while cfg["layers"][i].get("weights_of") is not None:
    i = cfg["layers"][i]["weights_of"]
  return i


def forward(cfg: dict, weights: Dict[str, Tensor], tokens, dtype=torch.float64, gaps: Optional[list] = None) -> Tuple[Tensor, List[Tensor]]:
  """logits [T, vocab] of one whole sequence and the residual stream after every layer"""
  Wt = {k: v.to(dtype) for k, v in weights.items()}
  eps = cfg["norm"]["eps"]
  norm = lambda name, x: dyt(x, Wt[name + ".alpha"], Wt[name], Wt[name + ".b"])
  x = Wt["embed"][torch.as_tensor(tokens, dtype=torch.long)]
  trail = []
  for i, layer in enumerate(cfg["layers"]):
    p, mlp = f"l{owner(cfg, i)}.", layer.get("mlp")
    x = x + latent_mixer(norm(p + "norm1", x), sub(Wt, p + "mix."), layer["mixer"], eps) * Wt[p + "ls1"]
    if mlp is not None:
      h, W = norm(p + "norm2", x), sub(Wt, p + "mlp.")
      x = x + (dense_ff(h, W) if mlp["kind"] == "dense" else moe_ff(h, W, mlp, gaps)) * Wt[p + "ls2"]
    trail.append(x)
  return norm("final.norm", x) @ Wt["embed"].T, trail


# ---- small random models -------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
  D, V = cfg["width"], cfg["vocab"]
  out: Dict[str, Tuple[int, ...]] = {"embed": (V, D)}
  def norm(name):
    out[name] = out[name + ".b"] = (D,)
    out[name + ".alpha"] = ()
  for i, layer in enumerate(cfg["layers"]):
    if layer.get("weights_of") is not None:
      continue
    p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    norm(p + "norm1")
    out.update({p + "mix.q": (H * (dn + dr), D), p + "mix.dkv": (R + dr, D), p + "mix.dkv.norm": (R,), p + "mix.uk": (H * dn, R),
                p + "mix.uv": (H * dv, R), p + "mix.sink": (H,), p + "mix.o": (D, H * dv), p + "ls1": (D,)})
    if mlp is None:
      continue
    norm(p + "norm2")
    out[p + "ls2"] = (D,)
    if mlp["kind"] == "dense":
      out.update({p + "mlp.gate": (mlp["ff"], D), p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
    else:
      E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
      out.update({p + "mlp.router": (E, D), p + "mlp.correction": (E,)})
      for e in range(E):
        out.update({p + f"mlp.e{e}.gate": (F, D), p + f"mlp.e{e}.up": (F, D), p + f"mlp.e{e}.down": (D, F)})
  norm("final.norm")
  return out


def random_weights(cfg: dict, seed: int) -> Dict[str, Tensor]:
  """bf16-representable random weights (a 16-bit engine and this oracle start from identical numbers)"""
  g = torch.Generator().manual_seed(seed)
  rnd = lambda shape, mean, dev: mean + dev * torch.randn(shape, generator=g)
  out = {}
  for name, shape in tensor_shapes(cfg).items():
    last = name.rsplit(".", 1)[-1]
    if last == "alpha":
      t = rnd(shape, 0.8, 0.15)
    elif last in ("ls1", "ls2"):
      t = rnd(shape, 0.6, 0.2)
    elif last == "correction":
      t = rnd(shape, -0.9, 0.6)                       # most choice scores are negative
    elif last == "b":
      t = rnd(shape, 0.0, 0.2)
    elif "norm" in last:
      t = rnd(shape, 1.0, 0.2)
    elif len(shape) == 1:
      t = rnd(shape, 0.0, 0.7)                        # sinks
    elif name == "embed":
      t = rnd(shape, 0.0, 1.0)
    elif last in ("gate", "up"):
      t = rnd(shape, 0.0, 1.6 / math.sqrt(shape[1]))  # some entries beyond the experts' clamp
    else:
      t = rnd(shape, 0.0, 1.0 / math.sqrt(shape[1]))
    out[name] = t.to(torch.bfloat16).to(torch.float32)
  return out
