"""Host-side logic of the Rinutar family (no GPU): config.json -> layer table, the registry, shared weights, and self-checks of the
plain oracle that the GPU tests compare the engine with."""
import math

import numpy as np
import pytest
import torch

from tests import rinutar_oracle as ro
from tests.rinutar_util import again, attn, config, dense, moe
from xotorch_b200 import _lib
from xotorch_b200.layered import LAYERED_FAMILIES, rinutar_globals, rinutar_layers, weight_owner
from xotorch_b200.models import is_layered, model_summary


def test_config_becomes_a_layer_table():
  layers = [attn(heads=5, dim=10, rot_dim=6, vdim=7, kv_rank=33, base=777.0, scale=0.4, mlp=dense(50)),
            attn(heads=2, mlp=moe(12, 4, 24, (6, 3), 2.5, 0.9)), attn(heads=4, dim=9, rot_dim=0, mlp=None)]
  layers += [again(layers, 1), attn(mlp=moe(5, 5, 8, None))]
  cfg = config(layers, width=40, vocab=91, eps=1e-3)
  a, b, c, d, e = rinutar_layers(cfg, {})
  assert (a.mixer, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.rot_dims) == (_lib.LM_MIX_LATENT_ATTN, 5, 10, 6, 7, 33, 0, 6)
  assert (a.rot_layout, a.rot_base, a.scale, a.sink, a.window, a.out_gate, a.weights_of) == (_lib.LM_ROT_HALF, 777.0, 0.4, 1, 0, 0, -1)
  assert (a.ff_kind, a.ff) == (_lib.LM_FF_GELU_GATED, 50)
  assert (b.ff_kind, b.experts, b.top, b.expert_ff, b.groups, b.groups_keep) == (_lib.LM_FF_MOE, 12, 4, 24, 6, 3)
  assert (b.expert_act, b.expert_limit, b.expert_slope) == (_lib.LM_EXPERT_CLAMPED_GLU, 0.9, 1.702)
  assert (b.router_kind, b.router_correction, b.group_best, b.router_scale, b.router_bias, b.shared_ff) == (_lib.LM_ROUTER_SIGMOID_GROUPS, 1, 2, 2.5, 0, 0)
  assert (c.ff, c.ff_kind, c.rot_dims, c.rot_dim) == (0, _lib.LM_FF_GELU_GATED, 0, 0)
  assert d.weights_of == 1 and {k: v for k, v in vars(d).items() if k != "weights_of"} == {k: v for k, v in vars(b).items() if k != "weights_of"}
  assert (e.groups, e.groups_keep) == (1, 1)
  g = rinutar_globals(cfg)
  assert (g["width"], g["vocab"], g["norm_eps"], g["block"], g["layer_scale"], g["tied_head"]) == (40, 91, 1e-3, _lib.LM_BLOCK_PRE_DYT, 1, 1)


def test_registry_knows_the_family():
  cfg = config([attn(mlp=dense())], width=24, vocab=33)
  assert "Rinutar" in LAYERED_FAMILIES and is_layered(cfg)
  s = model_summary(cfg)
  assert (s["n_layers"], s["vocab"], s["width"], s["engine"]) == (1, 33, 24, "layered")


def test_unknown_kinds_and_bad_references_are_refused():
  bad = config([attn()])
  bad["layers"][0]["type"] = "delta"
  with pytest.raises(ValueError, match="delta"):
    rinutar_layers(bad, {})
  bad = config([attn(mlp={"kind": "sparse", "ff": 8})])
  with pytest.raises(ValueError, match="sparse"):
    rinutar_layers(bad, {})
  chain = [attn(), attn(weights_of=0), attn(weights_of=1)]
  assert [weight_owner(chain, i) for i in range(3)] == [0, 0, 0]
  for layers in ([attn(weights_of=0)], [attn(weights_of=1), attn(weights_of=0)], [attn(weights_of=5)]):
    with pytest.raises(ValueError, match="weights_of"):
      rinutar_layers(config(layers), {})


# ---- the oracle's own mechanisms -----------------------------------------------------------------------------------------------
def test_oracle_dynamic_tanh_looks_at_every_entry_by_itself():
  x = torch.tensor([[0.5, -40.0, 0.0]], dtype=torch.float64)
  y = ro.dyt(x, torch.tensor(2.0), torch.tensor([1.0, 3.0, 5.0], dtype=torch.float64), torch.tensor([0.0, 0.25, -1.0], dtype=torch.float64))
  assert torch.allclose(y, torch.tensor([[math.tanh(1.0), -2.75, -1.0]], dtype=torch.float64))


def test_oracle_rotation_depends_on_the_distance():
  v, w = torch.randn(1, 6, dtype=torch.float64), torch.randn(1, 6, dtype=torch.float64)
  a, b = ro.turn(v.repeat(9, 1), 50.0), ro.turn(w.repeat(9, 1), 50.0)
  assert torch.allclose(a[7] @ b[4], a[3] @ b[0]) and torch.allclose(a[0], v[0])
  e = torch.zeros(4, 6, dtype=torch.float64)
  e[:, 1] = 1.0                                         # the plane of entry 1 is (1, 4), turned by p * 50^(-2/6)
  t, ang = ro.turn(e, 50.0)[3], 3 * 50.0 ** (-2 / 6)
  assert abs(float(t[1]) - math.cos(ang)) < 1e-12 and abs(float(t[4]) - math.sin(ang)) < 1e-12


def test_oracle_sink_counts_once_and_is_not_scaled():
  s = torch.tensor([[[1.0, -math.inf], [0.5, 2.0]]], dtype=torch.float64)
  p = ro.softmax_with_sink(s, torch.tensor([1.5], dtype=torch.float64))
  assert abs(float(p[0, 0, 0]) - math.exp(1.0) / (math.exp(1.0) + math.exp(1.5))) < 1e-12 and float(p[0, 0, 1]) == 0.0
  assert abs(float(p[0, 1].sum()) - (math.exp(0.5) + math.exp(2.0)) / (math.exp(0.5) + math.exp(2.0) + math.exp(1.5))) < 1e-12


def test_oracle_activations():
  z = torch.tensor([1.0, -2.0], dtype=torch.float64)
  want = [0.5 * v * (1 + math.tanh(math.sqrt(2 / math.pi) * (v + 0.044715 * v ** 3))) for v in (1.0, -2.0)]
  assert torch.allclose(ro.gelu_tanh(z), torch.tensor(want, dtype=torch.float64))
  W = {"gate": torch.eye(3, dtype=torch.float64), "up": torch.diag(torch.tensor([9.0, -9.0, 0.5], dtype=torch.float64)), "down": torch.eye(3, dtype=torch.float64)}
  y = ro.expert(torch.tensor([[5.0, -5.0, 1.0]], dtype=torch.float64), W, 2.0)
  sg = lambda g: g / (1 + math.exp(-1.702 * g))        # the gate is bounded above only, the up value on both sides
  assert torch.allclose(y, torch.tensor([[sg(2.0) * 3.0, sg(-5.0) * 3.0, sg(1.0) * 1.5]], dtype=torch.float64))


def test_oracle_routing_by_hand():
  logit = lambda s: math.log(s / (1 - s))
  s = [0.9, 0.1, 0.6, 0.5, 0.2, 0.7]
  W = {"router": torch.tensor([[logit(v)] for v in s], dtype=torch.float64), "correction": torch.tensor([-1.0, -1.0, -0.8, -0.8, -1.0, -1.0], dtype=torch.float64)}
  h = torch.ones(1, 1, dtype=torch.float64)
  # choice scores -0.1 -0.9 | -0.2 -0.3 | -0.8 -0.3; groups -1.0, -0.5, -1.1: the group with the single best expert comes second
  r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 1.5}
  ids, w = ro.route(h, W, r)
  assert ids.tolist() == [[2, 3]] and torch.allclose(w, torch.tensor([[0.6, 0.5]], dtype=torch.float64) / 1.1 * 1.5)
  ids, w = ro.route(h, W, {**r, "groups": {"count": 3, "keep": 2}})
  assert ids.tolist() == [[0, 2]] and torch.allclose(w, torch.tensor([[0.9, 0.6]], dtype=torch.float64) / 1.5 * 1.5)
  ids, _ = ro.route(h, W, {"experts": 6, "top": 4, "scale": 1.0})
  assert ids.tolist() == [[0, 2, 3, 5]] or sorted(ids.tolist()[0]) == [0, 2, 3, 5]


def test_oracle_prefixes_agree_and_shared_weights_are_the_owners():
  layers = [attn(mlp=dense()), attn(heads=2, mlp=moe())]
  cfg = config(layers + [again(layers, 0), again(layers, 1)])
  W = ro.random_weights(cfg, 3)
  assert not [k for k in W if k.startswith(("l2.", "l3."))]
  toks = np.random.default_rng(0).integers(0, cfg["vocab"], 30)
  full, _ = ro.forward(cfg, W, toks)
  part, _ = ro.forward(cfg, W, toks[:11])
  assert torch.allclose(full[:11], part, atol=1e-10)
  spelled = config(layers + layers)
  for j in (0, 1):
    W.update({f"l{j + 2}." + k[len(f"l{j}."):]: v for k, v in W.items() if k.startswith(f"l{j}.")})
  again_full, _ = ro.forward(spelled, W, toks)
  assert torch.allclose(full, again_full, atol=1e-10)
