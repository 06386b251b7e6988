"""The Rinutar family on the layered engine (libxotb200_lm.so) against the plain oracle (tests/rinutar_oracle.py) on small random
models (-m gpu).  The float32 engine is held to the oracle in float64 tightly, the bfloat16 engine loosely; tests ask for the logits of
EVERY row unless they say otherwise, so a wrong key, sink, expert or weight at any place shows."""
import json
import struct

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from tests import rinutar_oracle as ro
from tests.layered_util import TOL, bf16_bits, make_engine, rand_tokens, row_err, run_cut
from tests.rinutar_util import again, attn, config, dense, moe, oracle_logits, settled_rows

DTYPES = ["float32", "bfloat16"]

# layers of different shapes, dense / expert / no feed-forward, three layers that use earlier layers' weights (two of one owner)
_BASE = [attn(heads=3, dim=8, rot_dim=4, vdim=12, kv_rank=20, mlp=dense(36)),
         attn(heads=4, dim=6, rot_dim=6, vdim=5, kv_rank=13, base=30.0, mlp=moe(8, 3, 12, (4, 2))),
         attn(heads=2, dim=10, rot_dim=2, vdim=9, kv_rank=24, mlp=None)]
MIXED = _BASE + [again(_BASE, 1), again(_BASE, 0), attn(heads=1, dim=12, rot_dim=8, vdim=16, kv_rank=10, mlp=moe(5, 2, 9, None, 2.0, 1.1)), again(_BASE, 1)]


def check(native, cfg, W, tokens, cuts, dtype, slot=0, tol=None):
  ref, _ = oracle_logits(cfg, W, tokens)
  got = run_cut(native, slot, tokens, cuts)
  ok = settled_rows(cfg, W, tokens, dtype)
  assert ok.mean() > 0.5, "too many rows with a close call between experts: the test would not say much"
  e = row_err(got[ok], ref[ok])
  assert e < (tol or TOL[dtype]), f"{dtype}: rows differ from the oracle, worst relative error {e:.3e}"
  return got


# ---- each mechanism alone ------------------------------------------------------------------------------------------------
SINGLE = {
  "attention": [attn()],
  "attention_one_head": [attn(heads=1)],
  "attention_many_heads": [attn(heads=40, dim=4, rot_dim=2, vdim=4)],
  "attention_33_heads": [attn(heads=33, dim=4, rot_dim=2, vdim=3)],
  "attention_nothing_rotated": [attn(rot_dim=0)],
  "attention_rotated_part_larger": [attn(dim=4, rot_dim=16)],
  "attention_odd_sizes": [attn(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=11)],
  "attention_rank_1": [attn(kv_rank=1)],
  "attention_rank_70": [attn(kv_rank=70)],
  "attention_rank_130": [attn(kv_rank=130)],
  "attention_rank_260": [attn(kv_rank=260)],
  "attention_wide_values": [attn(vdim=140)],
  "attention_wide_heads": [attn(heads=2, dim=250, rot_dim=20)],
  "attention_unit_sizes": [attn(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1)],
  "dense": [attn(mlp=dense(36))],
  "dense_aligned": [attn(mlp=dense(64))],
  "dense_odd": [attn(mlp=dense(29))],
  "experts": [attn(mlp=moe())],
  "experts_aligned": [attn(mlp=moe(8, 2, 16))],
  "experts_odd_sizes": [attn(mlp=moe(6, 2, 9, (3, 2)))],
  "experts_no_groups": [attn(mlp=moe(7, 3, 12, None))],
  "experts_one_group": [attn(mlp=moe(6, 2, 12, (1, 1)))],
  "experts_all_groups_kept": [attn(mlp=moe(8, 2, 12, (4, 4)))],
  "experts_one_group_kept": [attn(mlp=moe(12, 3, 8, (3, 1)))],
  "experts_groups_of_one": [attn(mlp=moe(6, 2, 12, (6, 3)))],
  "experts_whole_groups_chosen": [attn(mlp=moe(8, 4, 12, (4, 2)))],
  "experts_top_1": [attn(mlp=moe(8, 1, 12, (2, 1)))],
  "experts_all_chosen": [attn(mlp=moe(5, 5, 8, None))],
  "one_expert": [attn(mlp=moe(1, 1, 24, None))],
  "many_experts": [attn(mlp=moe(72, 6, 8, (36, 5)))],
  "experts_tight_limit": [attn(mlp=moe(limit=0.1))],
  "experts_wide_limit": [attn(mlp=moe(limit=50.0, scale=1.0))],
  "no_feed_forward_anywhere": [attn(), attn(heads=2, dim=6)],
  "shared_weights": [attn(mlp=dense(36)), attn(mlp=dense(36), weights_of=0)],
  "shared_weights_twice": [attn(mlp=moe()), attn(mlp=moe(), weights_of=0), attn(mlp=moe(), weights_of=1)],
  "shared_weights_of_a_later_layer": [attn(heads=2, weights_of=1), attn(heads=2)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_mechanism_models(name, dtype):
  cfg = config(SINGLE[name], width=37 if "odd" in name else 48)
  W = ro.random_weights(cfg, 11)
  n = make_engine(cfg, W, dtype)
  toks = rand_tokens(cfg["vocab"], 41, 3)
  n.set_trace(True)
  ref, trail = oracle_logits(cfg, W, toks)
  ok = settled_rows(cfg, W, toks, dtype)
  assert ok.mean() > 0.5
  got, _ = n.step([0], [toks], want=list(range(len(toks))))
  x = n.read_trace(len(toks))
  for i, t in enumerate(trail):
    assert np.abs(x[i] - t)[ok].max() / np.abs(t).max() < (1e-5 if dtype == "float32" else 0.03), f"residual stream after layer {i} differs"
  assert row_err(got[ok], ref[ok]) < TOL[dtype]
  n.set_trace(False)
  cut = run_cut(n, 1, toks, [7, 5, 2, 1])            # short portions and single rows: the cache carried between steps
  assert row_err(cut[ok], ref[ok]) < TOL[dtype]
  n.close()


def test_eps_belongs_to_the_latent_norm_alone():
  """a large eps changes the latents' norm; the block norms, which have no statistic, do not know it"""
  for eps in (1e-5, 0.5):
    cfg = config([attn(mlp=dense())], eps=eps)
    W = ro.random_weights(cfg, 3)
    n = make_engine(cfg, W, "float32")
    check(n, cfg, W, rand_tokens(cfg["vocab"], 15, 1), [9, 1], "float32")
    n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_strong_norm_scalars(dtype):
  """alphas of both signs and of different sizes at every norm: a norm that takes a neighbour's scalar, or norms before the layer scale,
  shows"""
  layers = [attn(mlp=dense()), attn(heads=2, mlp=moe())]
  cfg = config(layers + [again(layers, 0)])
  W = ro.random_weights(cfg, 5)
  for i, (k, v) in enumerate({"l0.norm1": 0.3, "l0.norm2": -2.0, "l1.norm1": 1.5, "l1.norm2": 0.7, "final.norm": -0.4}.items()):
    W[k + ".alpha"] = torch.tensor(v).to(torch.bfloat16).float()
  W["l0.ls1"][::3] = -1.5
  W["l1.ls2"][::2] = 0.0
  n = make_engine(cfg, W, dtype)
  check(n, cfg, W, rand_tokens(cfg["vocab"], 33, 1), [20, 1], dtype)
  n.close()


# ---- prefill / decoding / portions -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [17, 1], [5, 2, 9, 1], [64]])
def test_portions_equal_the_whole_prompt(cuts, dtype):
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 2)
  n = make_engine(cfg, W, dtype, page_size=4)
  toks = rand_tokens(cfg["vocab"], 37, 8)
  got = check(n, cfg, W, toks, cuts, dtype)
  n.clear_request(0)
  whole = run_cut(n, 0, toks, [len(toks)])
  ok = settled_rows(cfg, W, toks, dtype)
  assert row_err(got[ok], whole.astype(np.float64)[ok]) < (2e-5 if dtype == "float32" else 0.05), "cutting the prompt changes rounding only"
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
  """300 tokens, all but six decoded one by one: the keys of a decode step are cut into runs (the sink must join once, where the runs are
  merged), pages fill up, a layer with another's weights keeps its own keys"""
  layers = [attn(heads=2, mlp=dense(24)), attn(heads=5, dim=6, rot_dim=4, vdim=8, mlp=moe(4, 2, 8, (2, 1)))]
  cfg = config(layers + [again(layers, 0)], width=32)
  W = ro.random_weights(cfg, 21)
  n = make_engine(cfg, W, dtype, max_tokens=400, page_size=16)
  check(n, cfg, W, rand_tokens(cfg["vocab"], 300, 4), [6, 1], dtype)
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(dtype):
  """the first token sees itself and the sink"""
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 9)
  n = make_engine(cfg, W, dtype)
  for length in (1, 2, 3, 5):
    toks = rand_tokens(cfg["vocab"], length, 30 + length)
    ref, ok = oracle_logits(cfg, W, toks)[0], settled_rows(cfg, W, toks, dtype)
    for cuts in ([1], [length]):
      n.clear_request(0)
      got = run_cut(n, 0, toks, cuts)
      assert not ok.any() or row_err(got[ok], ref[ok]) < TOL[dtype]
  n.close()


# ---- batches ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_equal_each_alone(dtype):
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 4)
  n = make_engine(cfg, W, dtype, max_tokens=256, max_requests=5, page_size=4)
  lens = [1, 13, 30, 2, 8]
  seqs = [rand_tokens(cfg["vocab"], L + 6, 50 + i) for i, L in enumerate(lens)]
  refs = [oracle_logits(cfg, W, s)[0] for s in seqs]
  oks = [settled_rows(cfg, W, s, dtype) for s in seqs]
  slots = [3, 0, 4, 1, 2]
  lg, _ = n.step(slots, [s[:L] for s, L in zip(seqs, lens)], want=list(range(sum(lens))))
  at = 0
  for i, L in enumerate(lens):
    ok = oks[i][:L]
    assert not ok.any() or row_err(lg[at:at + L][ok], refs[i][:L][ok]) < TOL[dtype], f"prompt of request {i}"
    at += L
  live = list(range(len(lens)))
  for t in range(6):
    if t == 2:
      live.remove(0)
      n.clear_request(slots[0])
    if t == 4:
      live.remove(3)
      n.clear_request(slots[3])
    lg, am = n.step([slots[i] for i in live], [seqs[i][lens[i] + t:lens[i] + t + 1] for i in live])
    for k, i in enumerate(live):
      if oks[i][lens[i] + t]:
        assert row_err(lg[k:k + 1], refs[i][lens[i] + t:lens[i] + t + 1]) < TOL[dtype], f"request {i}, decoded token {t}"
      assert am[k] == int(np.argmax(lg[k]))
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_requests_in_one_step(dtype):
  """more than a thousand rows (a count that is no multiple of four) in one step: the router then takes several rows per block"""
  cfg = config([attn(heads=2, mlp=moe(8, 3, 16, (4, 2))), attn(mlp=moe(6, 2, 9, (3, 2)))], width=48)
  W = ro.random_weights(cfg, 14)
  seqs = [rand_tokens(cfg["vocab"], 101, 200 + i) for i in range(13)]
  n = make_engine(cfg, W, dtype, max_tokens=1400, max_requests=13, page_size=16)
  lg, _ = n.step(list(range(13)), seqs, want=list(range(1313)))
  for i in (0, 6, 12):
    ok = settled_rows(cfg, W, seqs[i], dtype)
    assert ok.mean() > 0.5 and row_err(lg[101 * i:101 * (i + 1)][ok], oracle_logits(cfg, W, seqs[i])[0][ok]) < TOL[dtype]
  n.close()


def test_mixed_batch_of_portions_and_decoded_rows():
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 6)
  n = make_engine(cfg, W, "float32", page_size=4)
  a, b = rand_tokens(cfg["vocab"], 20, 1), rand_tokens(cfg["vocab"], 26, 2)
  ra, rb = oracle_logits(cfg, W, a)[0], oracle_logits(cfg, W, b)[0]
  n.step([0], [a[:15]])
  lg, _ = n.step([0, 1], [a[15:16], b[:11]], want=list(range(12)))
  assert row_err(lg[:1], ra[15:16]) < TOL["float32"] and row_err(lg[1:], rb[:11]) < TOL["float32"]
  lg, _ = n.step([1, 0], [b[11:26], a[16:17]], want=list(range(16)))
  assert row_err(lg[:15], rb[11:26]) < TOL["float32"] and row_err(lg[15:], ra[16:17]) < TOL["float32"]
  n.close()


def test_long_and_short_requests_in_one_bfloat16_step():
  """a prompt for the tensor-core attention, a short prompt and a decoded row in ONE step: the two attention forms share its buffers"""
  cfg = config([attn(heads=4, dim=16, rot_dim=8, vdim=24, kv_rank=40, mlp=dense(64)), attn(heads=2, dim=9, rot_dim=6, vdim=10, kv_rank=21)], width=64)
  W = ro.random_weights(cfg, 16)
  n = make_engine(cfg, W, "bfloat16", max_tokens=600, page_size=8)
  a, b, c = rand_tokens(cfg["vocab"], 90, 1), rand_tokens(cfg["vocab"], 7, 2), rand_tokens(cfg["vocab"], 41, 3)
  ra, rb, rc = (oracle_logits(cfg, W, t)[0] for t in (a, b, c))
  n.step([2], [c[:40]])
  lg, _ = n.step([1, 2, 0], [b, c[40:41], a], want=list(range(98)))
  assert row_err(lg[:7], rb) < TOL["bfloat16"] and row_err(lg[7:8], rc[40:]) < TOL["bfloat16"] and row_err(lg[8:], ra) < TOL["bfloat16"]
  n.close()


# ---- pages and slots that are given back and used again ----------------------------------------------------------------------
def test_freed_pages_and_slots_are_clean_for_the_next_request():
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 13)
  n = make_engine(cfg, W, "float32", max_tokens=64, max_requests=2, page_size=4)
  total = n.cache_stats()["pages_total"]
  a, b, c = (rand_tokens(cfg["vocab"], L, s) for L, s in ((29, 1), (18, 2), (31, 3)))
  check(n, cfg, W, a, [9, 1], "float32", slot=0)
  check(n, cfg, W, b, [18], "float32", slot=1)
  assert n.cache_stats()["pages_free"] == total - 8 - 5
  n.clear_request(0)                                  # a's pages go back ...
  assert n.cache_stats()["pages_free"] == total - 5 and n.request_len(0) == 0
  check(n, cfg, W, c, [5, 3, 1], "float32", slot=0)   # ... and c starts clean on them, next to the live b
  lg, _ = n.step([1], [a[:3]], want=[0, 1, 2])        # b goes on undisturbed
  ref = oracle_logits(cfg, W, np.concatenate([b, a[:3]]))[0]
  assert row_err(lg, ref[18:]) < TOL["float32"]
  n.clear_request(0)
  n.clear_request(1)
  assert n.cache_stats()["pages_free"] == total
  with pytest.raises(Exception, match="cache"):
    n.step([0], [rand_tokens(cfg["vocab"], 200, 1)])
  assert n.cache_stats()["pages_free"] == total and n.request_len(0) == 0
  n.close()


# ---- keys and sinks made to stand out ----------------------------------------------------------------------------------------
def plant(cfg, W):
  """The last token of the vocabulary gets an embedding whose queries are the keys of the last but one: the first norm and the query
  projection are inverted for it (the rotated query part is aimed at zero, so that the distance does not matter).  The other
  tokens' embeddings are small: their own queries stay dull whatever the score scale.  Returns (key token, query token)."""
  m, V = cfg["layers"][0]["mixer"], cfg["vocab"]
  H, dn, dr, R = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
  W["embed"][:V - 2] *= 0.25
  W["l0.norm1.b"] *= 0.25
  W["l0.mix.o"] *= 4.0
  D64 = {k: v.double() for k, v in W.items()}
  alpha, w, b = D64["l0.norm1.alpha"], D64["l0.norm1"], D64["l0.norm1.b"]
  hk = ro.dyt(D64["embed"][V - 2], alpha, w, b)
  c = ro.rms_norm((D64["l0.mix.dkv"] @ hk)[:R], D64["l0.mix.dkv.norm"], cfg["norm"]["eps"])
  want = torch.zeros(H, dn + dr, dtype=torch.float64)
  want[:, :dn] = (D64["l0.mix.uk"] @ c).reshape(H, dn)
  want = want / want.norm()
  null = torch.linalg.pinv(D64["l0.mix.q"])
  lo, hi = 0.0, 100.0
  for _ in range(50):                                   # the largest multiple whose operand the norm can produce
    mid = (lo + hi) / 2
    z = (null @ (mid * want).reshape(-1) - b) / w
    lo, hi = (mid, hi) if z.abs().max() < 0.95 else (lo, mid)
  z = (null @ (lo * want).reshape(-1) - b) / w
  W["embed"][V - 1] = (torch.atanh(z) / alpha).float()
  W["embed"] = W["embed"].to(torch.bfloat16).to(torch.float32)
  return V - 2, V - 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
def test_far_keys_and_page_borders(decode, dtype):
  """One key made to take much of the weight of the last row (sharp scores, planted embeddings): far away, and on either side of a page
  border.  Losing it, or reading a neighbour for it, moves the logits by far more than the tolerance.  The last 40 rows are decoded
  one by one when `decode`."""
  V, n_tok = 40, 150
  for name, pos, page in (("far", 3, 16), ("first", 0, 16), ("page_first", 64, 64), ("page_last", 63, 64), ("second_token", 1, 8), ("last_page_full", 143, 16), ("newest_but_one", 148, 8)):
    cfg = config([attn(heads=2, dim=12, rot_dim=4, vdim=12, kv_rank=24, scale=12.0)], vocab=V, width=64)
    W = ro.random_weights(cfg, 17)
    key_tok, query_tok = plant(cfg, W)
    seq = rand_tokens(V - 2, n_tok, 5)
    seq[-1] = query_tok
    without = oracle_logits(cfg, W, seq)[0]
    seq[pos] = key_tok
    ref = oracle_logits(cfg, W, seq)[0]
    gain = row_err(without[-1:], ref[-1:])
    assert gain > 3 * TOL["bfloat16"], f"{name}: the planted key does not stand out ({gain})"
    n = make_engine(cfg, W, dtype, max_tokens=256, page_size=page)
    got = run_cut(n, 0, seq, [n_tok - 40, 1] if decode else [n_tok])
    e = row_err(got[-1:], ref[-1:])
    assert e < TOL[dtype], f"{name} ({'decoded' if decode else 'prompt'}): {e:.3e}"
    assert row_err(got, ref) < TOL[dtype]
    n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_of_every_size(dtype):
  """head 0 has a sink that takes nearly everything, head 1 one that takes nearly nothing, head 2 an ordinary one: a sink that is left
  out, scaled or counted per key run shows on one head or another (prompt in both attention forms, and decoding over several key runs)"""
  cfg = config([attn(heads=3, vdim=8, scale=0.1)], width=32)
  W = ro.random_weights(cfg, 29)
  W["l0.mix.sink"] = torch.tensor([9.0, -9.0, 4.5])
  W["l0.mix.o"] *= 4.0
  toks = rand_tokens(cfg["vocab"], 200, 7)
  for wrong in (torch.full((3,), -80.0), torch.tensor([9.0, -9.0, 4.5]) * 0.1, torch.tensor([9.0, -9.0, 1.0])):
    other = dict(W)
    other["l0.mix.sink"] = wrong
    assert row_err(oracle_logits(cfg, other, toks)[0], oracle_logits(cfg, W, toks)[0]) > 2 * TOL["bfloat16"], "the sinks must matter"
  n = make_engine(cfg, W, dtype, max_tokens=1024, page_size=16)
  check(n, cfg, W, toks, [len(toks)], dtype, slot=0)
  check(n, cfg, W, toks, [150, 1], dtype, slot=1)
  n.set_attention_mode(1)
  check(n, cfg, W, toks, [len(toks)], dtype, slot=2)
  n.close()


def test_rotation_follows_the_position_not_the_portion():
  """scores that rest on the rotated part alone, low base: a portion that starts at position 13 must turn its queries and keys by the
  positions in the sequence"""
  cfg = config([attn(heads=2, dim=1, rot_dim=8, base=8.0, scale=2.0)], width=32)
  W = ro.random_weights(cfg, 31)
  toks = rand_tokens(cfg["vocab"], 60, 9)
  flat = config([attn(heads=2, dim=1, rot_dim=8, base=1e30, scale=2.0)], width=32)
  assert row_err(oracle_logits(flat, W, toks)[0], oracle_logits(cfg, W, toks)[0]) > 0.05, "the rotation must matter"
  n = make_engine(cfg, W, "float32", page_size=8)
  check(n, cfg, W, toks, [13, 20, 1], "float32")
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_choice_scores_and_weights_are_different_things(dtype):
  """corrections so strong that they alone choose: the chosen experts' WEIGHTS still come from the uncorrected scores; every choice score
  is negative, so a dropped group that counted as zero would win"""
  cfg = config([attn(mlp=moe(8, 3, 12, (4, 2), 2.0))])
  W = ro.random_weights(cfg, 8)
  W["l0.mlp.correction"] = torch.tensor([-19.0, -3.0, -17.0, -5.0, -5.0, -8.0, -6.5, -11.0])
  toks = rand_tokens(cfg["vocab"], 30, 2)
  W["l0.mlp.router"] *= 0.5
  # groups (-19, -3) (-17, -5) (-5, -8) (-6.5, -11), each plus scores in 0..1: the last two are kept, of them 4, 6 and 5 chosen
  ids, w = ro.route(torch.randn(50, 48, dtype=torch.float64, generator=torch.Generator().manual_seed(1)), ro.sub({k: v.double() for k, v in W.items()}, "l0.mlp."), cfg["layers"][0]["mlp"]["router"])
  assert all(set(row) == {4, 5, 6} for row in ids.tolist()) and (w.std(-1) > 0.003).all()
  n = make_engine(cfg, W, dtype)
  check(n, cfg, W, toks, [30], dtype, slot=0)
  check(n, cfg, W, toks, [11, 2, 1], dtype, slot=1)
  n.close()


def test_shared_weights_have_their_own_cache():
  """the second use of the weights sees other inputs, so its keys differ: with one cache for both the logits would differ"""
  layers = [attn(heads=2, scale=1.5, mlp=dense())]
  cfg = config(layers + [again(layers, 0), again(layers, 0)])
  W = ro.random_weights(cfg, 5)
  n = make_engine(cfg, W, "float32", page_size=4)
  once = make_engine(config(layers), W, "float32", page_size=4)
  assert n.weight_bytes() == once.weight_bytes(), "shared weights are held once"
  once.close()
  check(n, cfg, W, rand_tokens(cfg["vocab"], 45, 2), [19, 1], "float32")
  n.close()


# ---- several shards ----------------------------------------------------------------------------------------------------------
def shard_weights(W, keep):
  return {k: v for k, v in W.items() if keep(k)}


@pytest.mark.parametrize("split", [1, 3, 5])
def test_two_shards_hand_over_the_residual_stream(split):
  """a shard that uses the weights of a layer outside it, and a last shard without the first layer, hold their own copies of those
  tensors and of the embedding table"""
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 31)
  n_layers = len(MIXED)
  a = make_engine(cfg, W, "float32", start=0, end=split - 1)
  b = make_engine(cfg, W, "float32", start=split, end=n_layers - 1)
  toks = rand_tokens(cfg["vocab"], 19, 7)
  ref = oracle_logits(cfg, W, toks)[0]
  hid = a.step([0], [toks[:12]])
  lg, _ = b.step([0], [hid], want=list(range(12)))
  assert row_err(lg, ref[:12]) < TOL["float32"]
  hid = a.step([0], [toks[12:]])
  lg, _ = b.step([0], [hid], want=list(range(7)))
  assert row_err(lg, ref[12:]) < TOL["float32"]
  a.close()
  b.close()


# ---- the loader and the entry points -----------------------------------------------------------------------------------------
def write_model_dir(path, cfg, W):
  hdr, blobs, at = {}, [], 0
  for k, t in W.items():
    raw = bf16_bits(t).tobytes()
    hdr[k] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
    blobs.append(raw)
    at += len(raw)
  h = json.dumps(hdr).encode()
  with open(path / "model.safetensors", "wb") as f:
    f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
  with open(path / "config.json", "w") as f:
    json.dump(cfg, f)


def test_model_directory_loader_is_strict(tmp_path):
  from xotorch_b200.models import load_model_config, make_native
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 3)
  write_model_dir(tmp_path, cfg, W)
  n = make_native(load_model_config(tmp_path), 0, "float32")
  n.load_dir(tmp_path)
  n.begin_pool(64, 1, 8)
  check(n, cfg, W, rand_tokens(cfg["vocab"], 12, 1), [12], "float32")
  n.close()
  for missing in ("l0.mix.sink", "l1.mlp.e3.up", "l1.mlp.correction", "l0.mlp.gate", "l2.ls1", "l1.norm2.alpha", "final.norm.b", "final.norm.alpha", "l5.mix.dkv.norm"):
    bad = dict(W)
    del bad[missing]
    write_model_dir(tmp_path, cfg, bad)
    with pytest.raises(Exception, match=missing.replace(".", r"\.")):
      make_native(load_model_config(tmp_path), 0, "float32").load_dir(tmp_path)
  for extra, shape in (("l3.mix.q", (48, 48)), ("l1.mlp.router.b", (8,)), ("l2.ls2", (48,)), ("head", (80, 48)), ("l0.mix.g", (3, 48))):
    bad = dict(W)
    bad[extra] = torch.zeros(*shape)                   # tensors of a layer that uses another's, a bias, a scale without a sublayer, a head, a gate
    write_model_dir(tmp_path, cfg, bad)
    with pytest.raises(Exception, match=extra.replace(".", r"\.")):
      make_native(load_model_config(tmp_path), 0, "float32").load_dir(tmp_path)
  write_model_dir(tmp_path, cfg, W)
  bad = config(MIXED)
  bad["layers"][3]["mixer"]["scale"] *= 2              # a layer that uses another's weights but not its constants
  with pytest.raises(Exception, match="weights of layer 1"):
    make_native(bad, 0, "float32").load_dir(tmp_path)


def oracle_greedy(cfg, W, prompt, n_new):
  seq, ids, gaps = list(prompt), [], []
  for _ in range(n_new):
    lg = oracle_logits(cfg, W, np.array(seq))[0][-1]
    top = np.sort(lg)[-2:]
    ids.append(int(np.argmax(lg)))
    gaps.append(float((top[1] - top[0]) / lg.std()))
    seq.append(ids[-1])
  return ids, gaps


@pytest.mark.parametrize("dtype,budget", [("float32", 2048), ("bfloat16", 7)])
def test_greedy_generation_through_the_batch_scheduler(dtype, budget):
  from xotorch_b200.scheduler import ContinuousBatch
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 8)
  n = make_engine(cfg, W, dtype)
  events = []
  sched = ContinuousBatch(n, max_requests=3, max_tokens=160, page_size=8, token_budget=budget,
                          on_token=lambda rid, toks, fin: events.append((rid, list(toks), fin)))
  reqs = [(f"r{i}", rand_tokens(cfg["vocab"], L, 70 + i), g) for i, (L, g) in enumerate([(5, 9), (17, 4), (1, 12), (26, 6), (3, 1)])]
  for rid, p, g in reqs[:3]:
    sched.submit(rid, p, g)
  sched.step()
  for rid, p, g in reqs[3:]:
    sched.submit(rid, p, g)                           # joins while others are running
  out = sched.run_until_idle()
  for rid, p, g in reqs:
    ids, gaps = oracle_greedy(cfg, W, p, g)
    assert len(out[rid]) == g
    if out[rid] != ids:                               # after a near tie the continuations differ legitimately
      d = next(i for i in range(g) if out[rid][i] != ids[i])
      close = not settled_rows(cfg, W, np.concatenate([p, ids[:d]]).astype(np.int32), dtype).all()
      assert close or gaps[d] < (1e-3 if dtype == "float32" else 0.15), f"{rid}: ids leave the oracle's at step {d} with a clear gap {gaps[d]}"
    assert [e[1][0] for e in events if e[0] == rid] == out[rid]
  st = n.cache_stats()
  assert st["pages_free"] == st["pages_total"], "finished requests must give their pages back"
  n.close()


def test_command_line_generates_from_a_model_directory(tmp_path, capsys):
  from xotorch_b200.cli import main
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 8)
  write_model_dir(tmp_path, cfg, W)
  prompts = [rand_tokens(cfg["vocab"], 6, 1), rand_tokens(cfg["vocab"], 11, 2)]
  arg = ";".join(",".join(str(int(t)) for t in p) for p in prompts)
  assert main(["generate", "--model", str(tmp_path), "--prompt-ids", arg, "--max-tokens", "5", "--dtype", "float32"]) == 0
  lines = [json.loads(l) for l in capsys.readouterr().out.strip().splitlines()]
  for p, line in zip(prompts, lines):
    ids, gaps = oracle_greedy(cfg, W, p, 5)
    if line["ids"] != ids:
      d = next(i for i in range(5) if line["ids"][i] != ids[i])
      assert gaps[d] < 1e-3


def test_trace_replay_of_a_model_directory(tmp_path):
  """the token-trace replayer on a model directory: prompts in one batch, then decoding together, one request ending early"""
  from xotorch_b200.trace_replay import TraceReplayer
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 15)
  model, out = tmp_path / "m", tmp_path / "o"
  model.mkdir()
  write_model_dir(model, cfg, W)
  a, b = rand_tokens(cfg["vocab"], 22, 1), rand_tokens(cfg["vocab"], 9, 2)
  ra, rb = oracle_logits(cfg, W, a)[0], oracle_logits(cfg, W, b)[0]
  rp = TraceReplayer(model, "float32", out, max_tokens=64)
  rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": a[:18].tolist(), "want": [0, 17]}, {"id": "b", "tokens": b[:8].tolist(), "want": [7]}], "end": []})
  rp.run_step({"step": 1, "entries": [{"id": "a", "tokens": [int(a[18])], "want": [0]}, {"id": "b", "tokens": [int(b[8])], "want": [0]}], "end": ["b"]})
  rp.run_step({"step": 2, "entries": [{"id": "a", "tokens": a[19:22].tolist(), "want": []}], "end": ["a"]})
  V = cfg["vocab"]
  s0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V)
  s1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(-1, V)
  assert row_err(s0, np.stack([ra[0], ra[17], rb[7]])) < TOL["float32"]
  assert row_err(s1, np.stack([ra[18], rb[8]])) < TOL["float32"]
  assert not (out / "2.f32").exists()
  rp.close()


def test_inference_engine_serves_a_model_directory(tmp_path):
  """`B200ShardInferenceEngine` (the engine interface the node drives) on a model split over two shards, two request ids
  interleaved: ensure_shard -> registry -> LayeredShard, the position protocol of infer_tensor, sample(temp 0)"""
  import asyncio
  from xotorch_b200.inference.b200_engine import B200ShardInferenceEngine, LocalDirDownloader
  from xotorch_b200.inference.shard import Shard
  layers = [attn(mlp=dense(36)), attn(heads=2, dim=10, rot_dim=2)]
  cfg = config(layers + [again(layers, 0), again(layers, 1)])
  W = ro.random_weights(cfg, 27)
  write_model_dir(tmp_path, cfg, W)
  n = len(cfg["layers"])
  first, last = Shard("m", 0, 1, n), Shard("m", 2, n - 1, n)
  prompts = {"a": rand_tokens(cfg["vocab"], 9, 1), "b": rand_tokens(cfg["vocab"], 21, 2)}

  async def run():
    e1 = B200ShardInferenceEngine(LocalDirDownloader({"m": tmp_path}), device=0, max_concurrent_requests=2, max_total_len=64)
    e2 = B200ShardInferenceEngine(LocalDirDownloader({"m": tmp_path}), device=0, max_concurrent_requests=2, max_total_len=64)
    out, state, data = {r: [] for r in prompts}, {r: None for r in prompts}, {r: p.reshape(1, -1).astype(np.int64) for r, p in prompts.items()}
    for _ in range(4):
      for r in prompts:                               # the two requests take turns, token by token
        hid, st = await e1.infer_tensor(r, first, data[r], state[r])
        assert hid.ndim == 3 and hid.shape[2] == cfg["width"]
        logits, st2 = await e2.infer_tensor(r, last, hid, state[r])
        tok = await e2.sample(logits, temp=0.0)
        out[r].append(int(tok[0, 0]))
        state[r] = st2
        data[r] = tok.reshape(1, 1).astype(np.int64)
    return out

  out = asyncio.run(run())
  for r, p in prompts.items():
    ids, gaps = oracle_greedy(cfg, W, p, 4)
    if out[r] != ids:
      d = next(i for i in range(4) if out[r][i] != ids[i])
      assert gaps[d] < 0.15, f"{r}: ids leave the oracle's at step {d} with a clear gap"


# ---- decode steps replayed from CUDA graphs ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_graph_replay_of_decode_steps_changes_nothing(dtype):
  cfg = config(MIXED)
  W = ro.random_weights(cfg, 19)
  seqs = [rand_tokens(cfg["vocab"], 300, 40 + i) for i in range(3)]
  starts = [240, 3, 17]

  def run(graphs):
    n = make_engine(cfg, W, dtype, max_tokens=1000, max_requests=3, page_size=8)
    n.set_graphs(graphs)
    n.step([0, 1, 2], [s[:k] for s, k in zip(seqs, starts)])
    out, live = [], [0, 1, 2]
    for t in range(40):
      if t == 25:
        live = [0, 2]
        n.clear_request(1)
      lg, _ = n.step(live, [seqs[i][starts[i] + t:starts[i] + t + 1] for i in live])
      out.append(lg)
    replays = n.graph_replays()
    n.close()
    return out, replays

  plain, r0 = run(False)
  replayed, r1 = run(True)
  assert r0 == 0 and r1 >= 30
  for a, b in zip(plain, replayed):
    assert np.array_equal(a, b)
  ref = oracle_logits(cfg, W, seqs[0][:280])[0]
  ok = settled_rows(cfg, W, seqs[0][:280], dtype)[240:280]
  got = np.stack([x[0] for x in replayed])
  assert row_err(got[ok], ref[240:280][ok]) < TOL[dtype]


# ---- sizes the tensor-core paths take ----------------------------------------------------------------------------------------
def test_prompt_kernels_on_aligned_sizes_equal_the_plain_ones():
  """sizes that are multiples of 8 and prompts of hundreds of rows: the bf16 engine runs its products (gated and closing epilogues), its
  prompt attention (with the sink folded in at the end) and its experts on the tensor cores there; the results must agree with the
  plain kernels on the same 16-bit operands and with the oracle"""
  layers = [attn(heads=4, dim=16, rot_dim=8, vdim=24, kv_rank=40, mlp=dense(104)),
            attn(heads=2, dim=32, rot_dim=16, vdim=72, kv_rank=64, mlp=moe(8, 2, 32, (4, 3)))]
  cfg = config(layers + [again(layers, 0), again(layers, 1)], width=72, vocab=136)
  W = ro.random_weights(cfg, 12)
  n = make_engine(cfg, W, "bfloat16", max_tokens=1400, max_requests=3, page_size=32)
  a, b = rand_tokens(cfg["vocab"], 300, 9), rand_tokens(cfg["vocab"], 150, 10)
  ra, rb = oracle_logits(cfg, W, a)[0], oracle_logits(cfg, W, b)[0]
  before, flash_before = n.tensor_core_launches(), n.prompt_attention_launches()
  lg1, _ = n.step([0, 1], [a[:200], b], want=list(range(350)))          # a's first 200 rows and all of b in one batch
  lg2, _ = n.step([0], [a[200:]], want=list(range(100)))               # the rest of a starts far inside the sequence
  assert n.tensor_core_launches() > before and n.prompt_attention_launches() > flash_before
  tc_a = np.concatenate([lg1[:200], lg2])
  oka, okb = settled_rows(cfg, W, a, "bfloat16"), settled_rows(cfg, W, b, "bfloat16")
  assert oka.mean() > 0.6 and okb.mean() > 0.6
  assert row_err(tc_a[oka], ra[oka]) < TOL["bfloat16"] and row_err(lg1[200:][okb], rb[okb]) < TOL["bfloat16"]
  # three requests decode together: grouped expert products inside decode steps that are captured and replayed as CUDA graphs
  c = rand_tokens(cfg["vocab"], 12, 11)
  n.step([2], [c[:4]])
  a2, b2 = np.concatenate([a, a[:8]]), np.concatenate([b, b[:8]])
  ra2, rb2, rc = oracle_logits(cfg, W, a2)[0], oracle_logits(cfg, W, b2)[0], oracle_logits(cfg, W, c)[0]
  ok2 = [settled_rows(cfg, W, s, "bfloat16") for s in (a2, b2, c)]
  replays = n.graph_replays()
  for t in range(8):
    lg, _ = n.step([0, 1, 2], [a2[300 + t:301 + t], b2[150 + t:151 + t], c[4 + t:5 + t]])
    keep = np.array([ok2[0][300 + t], ok2[1][150 + t], ok2[2][4 + t]])
    if keep.any():
      assert row_err(lg[keep], np.stack([ra2[300 + t], rb2[150 + t], rc[4 + t]])[keep]) < TOL["bfloat16"], f"decoded token {t}"
  assert n.graph_replays() - replays >= 5
  n.clear_request(2)
  n.set_gemm_mode(1)
  n.set_attention_mode(1)
  fma = run_cut(n, 2, a, [200, 100])
  assert row_err(fma[oka], ra[oka]) < TOL["bfloat16"]
  assert row_err(tc_a[oka], fma.astype(np.float64)[oka]) < 0.05, "16-bit operands and fp32 accumulation in both"
  n.close()


# ---- other shapes, drawn at random ---------------------------------------------------------------------------------------------
def random_model(seed):
  """a model whose sizes, layer order and routing are drawn from ranges that include multiples of 8 (tensor-core kernels) and odd values
  (plain kernels); layers that use another's weights point at any earlier owner, several may share one"""
  r = np.random.default_rng(seed)
  pick = lambda *xs: xs[int(r.integers(len(xs)))]
  aligned = seed % 2 == 0
  width = pick(64, 96, 160) if aligned else pick(41, 52, 100)
  layers = []
  for i in range(int(r.integers(3, 7))):
    if layers and r.random() < 0.35:
      layers.append(again(layers, int(r.integers(len(layers)))))
      continue
    kind = pick(None, "dense", "dense", "moe", "moe")
    mlp = None
    if kind == "dense":
      mlp = dense(pick(40, 96) if aligned else pick(29, 60))
    elif kind == "moe":
      count, per = pick(1, 2, 3, 5), pick(1, 2, 4)
      keep = int(r.integers(1, count + 1))
      mlp = moe(count * per, int(r.integers(1, min(4, keep * per) + 1)), pick(16, 40) if aligned else pick(9, 20), (count, keep), pick(1.0, 1.7), pick(0.4, 1.5))
    dims = dict(dim=pick(16, 40), rot_dim=pick(8, 16), vdim=pick(8, 24, 96), kv_rank=pick(32, 72, 136)) if aligned else \
           dict(dim=pick(5, 12, 33), rot_dim=pick(2, 6, 14), vdim=pick(3, 10, 20), kv_rank=pick(7, 19, 50))
    layers.append(attn(heads=pick(1, 2, 3, 6), base=pick(50.0, 1e4), mlp=mlp, **dims))
  return config(layers, width=width, vocab=pick(50, 131), eps=pick(1e-6, 1e-3))


def row_errors(got, ref):
  d = got.astype(np.float64) - ref
  d = d - d.mean(axis=-1, keepdims=True)
  r = ref - ref.mean(axis=-1, keepdims=True)
  return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1) + 1e-30)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(10))
def test_models_drawn_at_random(seed, dtype):
  """whole prompts (one long enough for the tensor-core kernels next to a short one), then decoding together, then a portion"""
  cfg = random_model(seed)
  W = ro.random_weights(cfg, 100 + seed)
  n = make_engine(cfg, W, dtype, max_tokens=800, max_requests=3, page_size=16)
  a, b = rand_tokens(cfg["vocab"], 180, seed), rand_tokens(cfg["vocab"], 30, seed + 50)
  ra, rb = oracle_logits(cfg, W, a)[0], oracle_logits(cfg, W, b)[0]
  oka, okb = settled_rows(cfg, W, a, dtype), settled_rows(cfg, W, b, dtype)
  errs, keep = [], []
  lg, _ = n.step([2, 0], [a[:140], b[:9]], want=list(range(149)))
  errs += [row_errors(lg[:140], ra[:140]), row_errors(lg[140:], rb[:9])]
  keep += [oka[:140], okb[:9]]
  for t in range(21):
    lg, _ = n.step([0, 2], [b[9 + t:10 + t], a[140 + t:141 + t]])
    errs += [row_errors(lg[:1], rb[9 + t:10 + t]), row_errors(lg[1:], ra[140 + t:141 + t])]
    keep += [okb[9 + t:10 + t], oka[140 + t:141 + t]]
  lg, _ = n.step([2], [a[161:]], want=list(range(19)))               # a portion of 19 rows after decoding
  errs.append(row_errors(lg, ra[161:]))
  keep.append(oka[161:])
  e, keep = np.concatenate(errs), np.concatenate(keep)
  n.close()
  assert keep.mean() > 0.3, "too many close calls between experts: the test would not say much"
  assert e[keep].max() < TOL[dtype], f"worst {e[keep].max():.2e}: " + json.dumps(cfg["layers"])
  assert np.median(e) < 0.5 * TOL[dtype]
