"""Helpers of the Rinutar tests: small configurations of the family, the oracle's logits and the rows a 16-bit engine is held to.
Engines, schedules and the error measure come from layered_util."""
from __future__ import annotations

import copy
from typing import List, Optional, Tuple

import numpy as np
import torch

from tests import rinutar_oracle as ro


def dense(ff=36):
  return {"kind": "dense", "ff": ff}


def moe(experts=8, top=3, ff=12, groups: Optional[Tuple[int, int]] = (4, 2), scale=1.3, limit=0.7):
  r = {"experts": experts, "top": top, "scale": float(scale)}
  if groups:
    r["groups"] = {"count": groups[0], "keep": groups[1]}
  return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": float(limit)}}


def attn(heads=3, dim=8, rot_dim=4, vdim=12, kv_rank=20, base=200.0, scale=None, mlp=None, weights_of=None):
  layer = {"type": "latent_attention", "mlp": copy.deepcopy(mlp),
           "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
                     "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)}}
  if weights_of is not None:
    layer["weights_of"] = int(weights_of)
  return layer


def again(layers: List[dict], j: int) -> dict:
  """one more layer that uses layer j's weights"""
  layer = copy.deepcopy(layers[j])
  layer["weights_of"] = j
  return layer


def config(layers: List[dict], width=48, vocab=80, eps=1e-5) -> dict:
  return {"architecture": "Rinutar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}


def oracle_logits(cfg, weights, tokens, dtype=torch.float64):
  with torch.no_grad():
    lg, trail = ro.forward(cfg, weights, tokens, dtype)
  return lg.double().numpy(), [t.double().numpy() for t in trail]


def settled_rows(cfg, weights, tokens, dtype: str, gap=0.015) -> np.ndarray:
  """[T] bool: the rows a test holds to the tolerance.  float32: all.  bfloat16: those where no router choice (an expert over the best
  one left out, a group over the best one dropped) leads by less than `gap`; with the router's input rounded to 16 bits the others may
  legitimately choose otherwise."""
  out = np.ones(len(tokens), dtype=bool)
  if dtype == "float32":
    return out
  gaps: list = []
  with torch.no_grad():
    ro.forward(cfg, weights, tokens, torch.float64, gaps)
  for g in gaps:
    out &= g.numpy() >= gap
  return out
