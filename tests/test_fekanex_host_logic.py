"""Host-side logic of the Fekanex family (no GPU): config.json -> layer table, the registry, and self-checks of the plain oracle
that the GPU tests compare the engine with."""
import math

import numpy as np
import pytest
import torch

from tests import fekanex_oracle as fo
from tests.fekanex_util import attn, config, dense, moe, yarn
from xotorch_b200 import _lib
from xotorch_b200.layered import LAYERED_FAMILIES, fekanex_globals, fekanex_layers
from xotorch_b200.models import is_layered, model_summary

F64 = torch.float64


def test_config_becomes_a_layer_table():
  layers = [attn(heads=6, kv_heads=3, dim=10, vdim=7, conv=4, rot_dims=6, base=777.0, scaling=yarn(5.0, 300, 11.0, 2.0), size=21, keep=3, scale=0.4, v_mix=True, mlp=dense(50, 1.5)),
            attn(heads=2, kv_heads=2, conv=None, rot_dims=0, size=None, mlp=moe(12, 4, 24)), attn(rot_dims=4, keep=0, mlp=None)]
  cfg = config(layers, width=40, vocab=91, eps=1e-3, scale=0.3, buckets=19, mul_prev=23, mul_cur=29, logit_scale=1.7)
  a, b, c = fekanex_layers(cfg, {})
  assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.conv_taps, a.kv_from) == (_lib.LM_MIX_ATTENTION, 6, 3, 10, 7, 4, -1)
  assert (a.rot_dims, a.rot_layout, a.rot_base, a.rot_scale_kind) == (6, _lib.LM_ROT_INTERLEAVED, 777.0, _lib.LM_ROT_SCALE_YARN)
  assert (a.rot_scale_factor, a.rot_scale_original, a.rot_scale_high, a.rot_scale_low) == (5.0, 300.0, 11.0, 2.0)
  assert (a.window, a.keep_first, a.scale, a.sink, a.qk_norm, a.proj_bias, a.v_mix) == (21, 3, 0.4, _lib.LM_SINK_ONE, _lib.LM_QKNORM_HEAD_ROTATED, 1, 1)
  assert (a.ff_kind, a.ff, a.expert_limit, a.expert_slope) == (_lib.LM_FF_CLAMPED_GLU, 50, 1.5, 1.702)
  assert (b.conv_taps, b.rot_dims, b.window, b.keep_first, b.v_mix, b.rot_scale_kind) == (0, 0, 0, 0, 0, 0)
  assert (b.ff_kind, b.experts, b.top, b.expert_ff, b.expert_act, b.router_kind, b.router_bias) == \
         (_lib.LM_FF_MOE, 12, 4, 24, _lib.LM_EXPERT_SILU_GATED, _lib.LM_ROUTER_TOPK_SOFTMAX, 0)
  assert (c.ff, c.experts, c.rot_dims, c.rot_scale_factor, c.keep_first) == (0, 0, 4, 0.0, 0)
  g = fekanex_globals(cfg)
  assert (g["width"], g["vocab"], g["norm_eps"], g["block"], g["tied_head"], g["logit_scale"], g["embed_scale"]) == (40, 91, 1e-3, _lib.LM_BLOCK_PARALLEL_RMS, 1, 1.7, 0.3)
  assert (g["bigram_buckets"], g["bigram_mul_prev"], g["bigram_mul_cur"]) == (19, 23, 29)
  assert fekanex_globals(config(layers, buckets=None))["bigram_buckets"] == 0


def test_registry_knows_the_family():
  cfg = config([attn(mlp=dense())], width=24, vocab=33)
  assert "Fekanex" in LAYERED_FAMILIES and is_layered(cfg)
  s = model_summary(cfg)
  assert (s["n_layers"], s["vocab"], s["width"], s["engine"]) == (1, 33, 24, "layered")


def test_unknown_kinds_are_refused():
  bad = config([attn()])
  bad["layers"][0]["type"] = "delta"
  with pytest.raises(ValueError, match="delta"):
    fekanex_layers(bad, {})
  with pytest.raises(ValueError, match="sparse"):
    fekanex_layers(config([attn(mlp={"kind": "sparse", "ff": 8})]), {})


# ---- the oracle's own mechanisms -----------------------------------------------------------------------------------------------
def test_oracle_bigram_rows_and_embedding():
  t = torch.tensor([4, 9, 2])
  assert fo.bigram_rows(t, {"buckets": 10, "mul_prev": 3, "mul_cur": 7}).tolist() == [10, (12 + 63) % 10, (27 + 14) % 10]
  W = {"embed": torch.eye(10, dtype=F64), "bigram": torch.arange(11, dtype=F64)[:, None].repeat(1, 10)}
  x = fo.embedding(t, W, {"scale": 0.5, "bigram": {"buckets": 10, "mul_prev": 3, "mul_cur": 7}})
  assert x[0, 4] == 10.5 and x[0, 0] == 10.0 and x[1, 9] == 5.5 and x[2, 0] == 1.0


def test_oracle_filter_sees_zeros_before_the_start():
  u = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64)
  y = fo.causal_filter(u, torch.tensor([[0.5, 10.0, 1.0]], dtype=F64))
  assert y[:, 0].tolist() == [1.0, 12.0, 24.5]
  assert torch.equal(fo.causal_filter(u, torch.tensor([[3.0]], dtype=F64)), 3 * u)


def test_oracle_frequencies_by_hand():
  rot = {"base": 100.0, "dims": 8}
  f, mul = fo.frequencies(rot)
  assert mul == 1.0 and torch.allclose(f, torch.tensor([1.0, 100 ** -0.25, 0.1, 100 ** -0.75], dtype=F64))
  at = lambda turns: 8 * math.log(40 / (2 * math.pi * turns)) / (2 * math.log(100))
  g, mul = fo.frequencies({**rot, "scaling": yarn(8.0, 40, 6.0, 0.5)})
  lo, hi = max(math.floor(at(6.0)), 0), min(math.ceil(at(0.5)), 7)
  assert (lo, hi) == (0, 3) and abs(mul - (0.1 * math.log(8) + 1)) < 1e-12
  ramp = torch.tensor([0, 1 / 3, 2 / 3, 1], dtype=F64)
  assert torch.allclose(g, f / 8 * ramp + f * (1 - ramp))


def test_oracle_rotation_turns_neighbouring_entries():
  x = torch.zeros(4, 1, 6, dtype=F64)
  x[:, 0, 2] = 1.0
  x[:, 0, 5] = 3.0                                     # beyond the rotated entries
  t, ang = fo.turn(x, {"base": 50.0, "dims": 4})[3, 0], 3 * 50.0 ** -0.5
  assert abs(float(t[2]) - math.cos(ang)) < 1e-12 and abs(float(t[3]) - math.sin(ang)) < 1e-12 and float(t[5]) == 3.0
  s = fo.turn(x, {"base": 50.0, "dims": 4, "scaling": yarn()})[0, 0]
  assert abs(float(s[2]) - (0.1 * math.log(8.0) + 1)) < 1e-12 and float(s[5]) == 3.0, "the factor lengthens the rotated entries only"


def test_oracle_mask_and_softmax():
  ok = fo.visible(6, {"size": 2, "keep_first": 1})
  assert ok.tolist()[5] == [True, False, False, False, True, True] and ok.tolist()[1] == [True, True] + [False] * 4
  assert fo.visible(4, None).tolist()[3] == [True] * 4 and fo.visible(4, {"size": 1, "keep_first": 0}).sum() == 4
  p = fo.softmax_one_more(torch.tensor([1.0, -math.inf, 2.0], dtype=F64))
  den = 1 + math.exp(1) + math.exp(2)
  assert torch.allclose(p, torch.tensor([math.exp(1) / den, 0.0, math.exp(2) / den], dtype=F64))
  p = fo.softmax_one_more(torch.tensor([-30.0], dtype=F64))
  assert abs(float(p) - math.exp(-30)) < 1e-20


def test_oracle_activations_and_routing():
  W = {"gate": torch.eye(3, dtype=F64), "up": torch.diag(torch.tensor([9.0, -9.0, 0.5], dtype=F64)), "down": torch.eye(3, dtype=F64)}
  y = fo.dense_ff(torch.tensor([[5.0, -5.0, 1.0]], dtype=F64), W, 2.0)
  sg = lambda g: g / (1 + math.exp(-1.702 * g))        # the gate is bounded above only, the up value on both sides
  assert torch.allclose(y, torch.tensor([[sg(2.0) * 3.0, sg(-5.0) * 3.0, sg(1.0) * 1.5]], dtype=F64))
  W = {"router": torch.tensor([[0.3], [2.0], [-1.0], [1.0]], dtype=F64)}
  gaps = []
  ids, w = fo.route(torch.ones(1, 1, dtype=F64), W, {"experts": 4, "top": 2}, gaps)
  assert ids.tolist() == [[1, 3]] and abs(float(w[0, 0]) - 1 / (1 + math.exp(-1.0))) < 1e-12 and abs(float(gaps[0]) - 0.7) < 1e-12


def test_oracle_values_mix_with_the_first_mixing_layer():
  """layer 1 is the first mixing layer: layers 2 and 4 take its values, 3 does not, and layer 1's own number is unused"""
  cfg = config([attn(), attn(v_mix=True), attn(v_mix=True), attn(), attn(v_mix=True)])
  W = fo.random_weights(cfg, 3)
  toks = np.random.default_rng(0).integers(0, cfg["vocab"], 20)
  full, _ = fo.forward(cfg, W, toks)
  moved = {name: not torch.allclose(full, fo.forward(cfg, {**W, name: torch.tensor(0.9)}, toks)[0]) for name in W if name.endswith("vmix")}
  assert moved == {"l1.mix.vmix": False, "l2.mix.vmix": True, "l4.mix.vmix": True}
  part, _ = fo.forward(cfg, W, toks[:7])
  assert torch.allclose(full[:7], part, atol=1e-10)
