"""Helpers of the Fekanex tests: small configurations of the family, the oracle's logits and the rows a 16-bit engine is held to.
Engines, schedules and the error measure come from layered_util."""
from __future__ import annotations

import copy
from typing import List, Optional

import numpy as np
import torch

from tests import fekanex_oracle as fo


def dense(ff=36, limit=0.9):
  return {"kind": "dense", "ff": ff, "limit": float(limit)}


def moe(experts=6, top=2, ff=12):
  return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def yarn(factor=8.0, original=40, fast=6.0, slow=0.5):
  return {"factor": float(factor), "original": original, "fast": float(fast), "slow": float(slow)}


def attn(heads=4, kv_heads=2, dim=12, vdim=12, conv: Optional[int] = 3, rot_dims=8, base=100.0, scaling: Optional[dict] = None, size: Optional[int] = 9, keep=2,
         scale=None, v_mix=False, mlp=None):
  """one layer; rot_dims 0 = no rotation, size None = no window"""
  m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": float(scale if scale is not None else dim ** -0.5), "v_mix": bool(v_mix),
       "mask": {"size": size, "keep_first": keep} if size else None, "rot": {"base": float(base), "dims": rot_dims} if rot_dims else None}
  if rot_dims and scaling:
    m["rot"]["scaling"] = dict(scaling)
  return {"type": "attention", "mixer": m, "mlp": copy.deepcopy(mlp)}


def config(layers: List[dict], width=48, vocab=80, eps=1e-5, scale=0.7, buckets: Optional[int] = 53, mul_prev=17, mul_cur=5, logit_scale=0.8) -> dict:
  emb = {"scale": float(scale)}
  if buckets:
    emb["bigram"] = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
  return {"architecture": "Fekanex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": float(logit_scale), "embedding": emb,
          "layers": copy.deepcopy(layers)}


def oracle_logits(cfg, weights, tokens, dtype=torch.float64):
  with torch.no_grad():
    lg, trail = fo.forward(cfg, weights, tokens, dtype)
  return lg.double().numpy(), [t.double().numpy() for t in trail]


def settled_rows(cfg, weights, tokens, dtype: str, gap=0.03) -> np.ndarray:
  """[T] bool: the rows a test holds to the tolerance.  float32: all.  bfloat16: those where no router choice (an expert over the best
  one left out) leads by less than `gap`: with the router's input rounded to 16 bits the others may legitimately choose otherwise."""
  out = np.ones(len(tokens), dtype=bool)
  if dtype == "float32":
    return out
  gaps: list = []
  with torch.no_grad():
    fo.forward(cfg, weights, tokens, torch.float64, gaps)
  for g in gaps:
    out &= g.numpy() >= gap
  return out
