"""The Fekanex family on the layered engine (libxotb200_lm.so) against the plain oracle (tests/fekanex_oracle.py) on small random
models (-m gpu).  The float32 engine is held to the oracle in float64 tightly, the bfloat16 engine loosely; tests ask for the logits of
EVERY row unless they say otherwise, so a wrong key, window edge, filter input, pair row or expert at any place shows."""
import json
import struct

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from tests import fekanex_oracle as fo
from tests.fekanex_util import attn, config, dense, moe, oracle_logits, settled_rows, yarn
from tests.layered_util import TOL, bf16_bits, make_engine, rand_tokens, row_err, run_cut

DTYPES = ["float32", "bfloat16"]

# layers of different shapes, windows, filters and rotations; dense / expert / no feed-forward; values mixed in layers 1, 2 and 4
MIXED = [attn(heads=3, kv_heads=3, dim=8, vdim=12, conv=2, rot_dims=4, size=6, keep=1, mlp=dense(36)),
         attn(heads=4, kv_heads=2, dim=12, vdim=10, conv=3, rot_dims=12, scaling=yarn(), size=9, keep=3, v_mix=True, mlp=moe(6, 2, 12)),
         attn(heads=6, kv_heads=2, dim=6, vdim=10, conv=4, rot_dims=2, base=30.0, size=None, v_mix=True, mlp=None),
         attn(heads=2, kv_heads=1, dim=10, vdim=9, conv=None, rot_dims=0, size=4, keep=0, mlp=moe(5, 3, 9)),
         attn(heads=2, kv_heads=2, dim=16, vdim=10, conv=5, rot_dims=8, scaling=yarn(3.0, 500, 20.0, 1.0), size=20, keep=4, v_mix=True, mlp=dense(29, 0.6))]


def check(native, cfg, W, tokens, cuts, dtype, slot=0, tol=None):
  ref, _ = oracle_logits(cfg, W, tokens)
  got = run_cut(native, slot, tokens, cuts)
  ok = settled_rows(cfg, W, tokens, dtype)
  assert ok.mean() > 0.4, "too many rows with a close call between experts: the test would not say much"
  e = row_err(got[ok], ref[ok])
  assert e < (tol or TOL[dtype]), f"{dtype}: rows differ from the oracle, worst relative error {e:.3e}"
  return got


# ---- each mechanism alone ------------------------------------------------------------------------------------------------
SINGLE = {
  "attention": ([attn()], {}),
  "one_head": ([attn(heads=1, kv_heads=1)], {}),
  "one_kv_head": ([attn(heads=6, kv_heads=1)], {}),
  "as_many_kv_heads": ([attn(heads=5, kv_heads=5)], {}),
  "many_heads": ([attn(heads=40, kv_heads=20, dim=4, vdim=4, rot_dims=4)], {}),
  "odd_sizes": ([attn(heads=3, kv_heads=3, dim=5, vdim=7, rot_dims=4)], {"width": 37}),
  "unit_sizes": ([attn(heads=1, kv_heads=1, dim=1, vdim=1, rot_dims=0)], {}),
  "heads_beyond_128": ([attn(heads=2, kv_heads=1, dim=200, vdim=140, rot_dims=150, base=1e4, scaling=yarn()), attn(heads=1, kv_heads=1, dim=132, vdim=8, conv=4)], {}),
  "wide_heads": ([attn(heads=2, kv_heads=1, dim=272, vdim=140, rot_dims=200, base=1e4)], {}),
  "wide_values": ([attn(heads=2, kv_heads=1, vdim=300)], {}),
  "no_filter": ([attn(conv=None)], {}),
  "filter_1": ([attn(conv=1)], {}),
  "filter_2": ([attn(conv=2)], {}),
  "filter_4": ([attn(conv=4)], {}),
  "filter_8": ([attn(conv=8)], {}),
  "filter_beyond_registers": ([attn(conv=11)], {}),
  "no_rotation": ([attn(rot_dims=0)], {}),
  "whole_head_rotated": ([attn(rot_dims=12)], {}),
  "yarn": ([attn(dim=20, rot_dims=16, scaling=yarn())], {}),
  "yarn_all_slowed": ([attn(rot_dims=8, scaling=yarn(4.0, 7, 30.0, 20.0))], {}),
  "yarn_none_slowed": ([attn(rot_dims=8, base=3.0, scaling=yarn(4.0, 100000, 32.0, 1.0))], {}),
  "yarn_narrow_ramp": ([attn(rot_dims=8, scaling=yarn(16.0, 60, 2.0, 1.9))], {}),
  "yarn_of_factor_1": ([attn(rot_dims=8, scaling=yarn(1.0))], {}),
  "window_1": ([attn(size=1, keep=1)], {}),
  "window_without_kept_tokens": ([attn(size=5, keep=0)], {}),
  "kept_tokens_beyond_window": ([attn(size=3, keep=8)], {}),
  "window_beyond_prompt": ([attn(size=500, keep=2)], {}),
  "no_window": ([attn(size=None)], {}),
  # head sizes that are no multiple of 4 take the preparation kernel for any size, the others mostly the one in fours
  "plain_filter": ([attn(vdim=10)], {}),
  "plain_no_filter": ([attn(vdim=10, conv=None)], {}),
  "plain_filter_2": ([attn(dim=10, conv=2)], {}),
  "plain_yarn": ([attn(vdim=9, rot_dims=12, scaling=yarn())], {}),
  "plain_values_mixed": ([attn(vdim=10, v_mix=True), attn(vdim=10, v_mix=True)], {}),
  "rotated_part_no_multiple_of_4": ([attn(rot_dims=6), attn(rot_dims=10, scaling=yarn()), attn(rot_dims=2)], {}),
  "values_mixed": ([attn(v_mix=True), attn(v_mix=True)], {}),
  "values_mixed_later": ([attn(vdim=8), attn(v_mix=True), attn(kv_heads=1), attn(heads=2, dim=8, v_mix=True)], {}),
  "dense": ([attn(mlp=dense(36))], {}),
  "dense_aligned": ([attn(mlp=dense(64))], {}),
  "dense_odd": ([attn(mlp=dense(29))], {}),
  "dense_tight_limit": ([attn(mlp=dense(40, 0.1))], {}),
  "dense_wide_limit": ([attn(mlp=dense(40, 50.0))], {}),
  "experts": ([attn(mlp=moe())], {}),
  "experts_aligned": ([attn(mlp=moe(8, 3, 16))], {}),
  "experts_odd_sizes": ([attn(mlp=moe(7, 2, 9))], {}),
  "experts_top_1": ([attn(mlp=moe(8, 1, 12))], {}),
  "experts_all_chosen": ([attn(mlp=moe(5, 5, 8))], {}),
  "one_expert": ([attn(mlp=moe(1, 1, 24))], {}),
  "many_experts": ([attn(mlp=moe(72, 6, 8))], {}),
  "no_pair_table": ([attn(mlp=dense())], {"buckets": None}),
  "one_bucket": ([attn()], {"buckets": 1}),
  "large_pair_factors": ([attn()], {"buckets": 1009, "mul_prev": 2 ** 33 + 5, "mul_cur": 10 ** 9 + 7}),
  "embedding_not_scaled": ([attn()], {"scale": 1.0}),
  "large_eps": ([attn(mlp=dense())], {"eps": 0.5}),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_mechanism_models(name, dtype):
  layers, extra = SINGLE[name]
  cfg = config(layers, **extra)
  W = fo.random_weights(cfg, 11)
  n = make_engine(cfg, W, dtype)
  toks = rand_tokens(cfg["vocab"], 41, 3)
  n.set_trace(True)
  ref, trail = oracle_logits(cfg, W, toks)
  ok = settled_rows(cfg, W, toks, dtype)
  assert ok.mean() > 0.4
  got, _ = n.step([0], [toks], want=list(range(len(toks))))
  x = n.read_trace(len(toks))
  for i, t in enumerate(trail):
    assert np.abs(x[i] - t)[ok].max() / np.abs(t).max() < (1e-5 if dtype == "float32" else 0.03), f"residual stream after layer {i} differs"
  assert row_err(got[ok], ref[ok]) < TOL[dtype]
  n.set_trace(False)
  cut = run_cut(n, 1, toks, [7, 5, 2, 1])            # short portions and single rows: cache, filter inputs and previous token carried
  assert row_err(cut[ok], ref[ok]) < TOL[dtype]
  n.close()


# ---- prefill / decoding / portions -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[1], [2], [3], [17, 1], [5, 2, 9, 1], [64]])
def test_portions_equal_the_whole_prompt(cuts, dtype):
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 2)
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
  """300 tokens, all but six decoded one by one: windows pass over decoded tokens, the keys of a layer without a window are cut into runs
  (the sink must join once, where the runs are merged), pages fill up"""
  layers = [attn(heads=2, kv_heads=1, size=50, keep=4, v_mix=True, mlp=dense(24)), attn(heads=4, kv_heads=2, vdim=10, size=None, scaling=yarn(), mlp=moe(4, 2, 8)),
            attn(heads=3, kv_heads=1, size=100, keep=1, v_mix=True)]
  cfg = config(layers, width=32)
  W = fo.random_weights(cfg, 21)
  n = make_engine(cfg, W, dtype, max_tokens=400, page_size=16)
  check(n, cfg, W, rand_tokens(cfg["vocab"], 300, 4), [6, 1], dtype)
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(dtype):
  """the first token sees itself and the sink, has the last row of the pair table and filters that reach before the start"""
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 9)
  W["bigram"][-1] *= 4.0
  n = make_engine(cfg, W, dtype)
  for length in (1, 2, 3, 5):
    toks = rand_tokens(cfg["vocab"], length, 30 + length)
    ref, ok = oracle_logits(cfg, W, toks)[0], settled_rows(cfg, W, toks, dtype)
    for cuts in ([1], [length]):
      n.clear_request(0)
      got = run_cut(n, 0, toks, cuts)
      assert not ok.any() or row_err(got[ok], ref[ok]) < TOL[dtype]
  n.close()


# ---- state between steps made to stand out -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vdim", [8, 9])
@pytest.mark.parametrize("taps", [2, 4, 10])
def test_filters_that_only_see_the_oldest_input(taps, vdim, dtype):
  """every filter is a pure delay by taps - 1 tokens, so a token's queries, keys and values come wholly from earlier steps' inputs when it
  is decoded; portions shorter than the filter move part of the inputs on"""
  cfg = config([attn(vdim=vdim, conv=taps, v_mix=True), attn(vdim=vdim, conv=taps, v_mix=True)])
  W = fo.random_weights(cfg, 6)
  for k in W:
    if k.endswith(".conv"):
      W[k][:] = 0.0
      W[k][:, 0] = 1.0
  toks = rand_tokens(cfg["vocab"], 45, 2)
  n = make_engine(cfg, W, dtype, page_size=4)
  for slot, cuts in enumerate(([45], [1], [2], [13, 1, 2, 3])):
    check(n, cfg, W, toks, cuts, dtype, slot=slot)
  n.close()


def test_biases_enter_before_the_filter():
  """large biases: the filter reaches before the start, where it must see zeros and not biases, and sums the bias once per tap elsewhere"""
  cfg = config([attn(conv=4, size=None)])
  W = fo.random_weights(cfg, 6)
  for t in "qkv":
    W[f"l0.mix.{t}.b"] *= 8.0
  toks = rand_tokens(cfg["vocab"], 20, 2)
  n = make_engine(cfg, W, "float32", page_size=4)
  check(n, cfg, W, toks, [20], "float32", slot=0)
  check(n, cfg, W, toks, [1], "float32", slot=1)
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_previous_token_is_carried_between_steps_and_requests(dtype):
  """a pair table that outweighs the embedding: a wrong previous token — across a step border, from a neighbour in the batch, from the
  slot's last owner — changes the row by far more than the tolerance"""
  cfg = config([attn(mlp=dense())], buckets=211, mul_prev=89, mul_cur=3)
  W = fo.random_weights(cfg, 4)
  W["bigram"] *= 8.0
  a, b, c = (rand_tokens(cfg["vocab"], L, s) for L, s in ((19, 1), (14, 2), (9, 3)))
  ra, rb, rc = (oracle_logits(cfg, W, t)[0] for t in (a, b, c))
  n = make_engine(cfg, W, dtype, page_size=4, max_requests=2)
  lg, _ = n.step([1, 0], [a[:11], b[:5]], want=list(range(16)))
  assert row_err(lg[:11], ra[:11]) < TOL[dtype] and row_err(lg[11:], rb[:5]) < TOL[dtype]
  for t in range(8):
    lg, _ = n.step([0, 1], [b[5 + t:6 + t], a[11 + t:12 + t]])
    assert row_err(lg[:1], rb[5 + t:6 + t]) < TOL[dtype] and row_err(lg[1:], ra[11 + t:12 + t]) < TOL[dtype]
  n.clear_request(1)
  lg, _ = n.step([1, 0], [c, b[13:]], want=list(range(10)))
  assert row_err(lg[:9], rc) < TOL[dtype] and row_err(lg[9:], rb[13:]) < TOL[dtype]
  n.close()


# ---- batches ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_equal_each_alone(dtype):
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 4)
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
  """more than a thousand rows in one step and many heads: the preparation launch then takes several heads per block"""
  cfg = config([attn(heads=24, kv_heads=12, dim=6, vdim=5, rot_dims=4, v_mix=True, mlp=moe(8, 3, 16)), attn(heads=24, kv_heads=12, dim=5, vdim=5, rot_dims=0, v_mix=True, mlp=moe(6, 2, 9))])
  W = fo.random_weights(cfg, 14)
  seqs = [rand_tokens(cfg["vocab"], 101, 200 + i) for i in range(13)]
  n = make_engine(cfg, W, dtype, max_tokens=1400, max_requests=13, page_size=16)
  lg, _ = n.step(list(range(13)), seqs, want=list(range(1313)))
  for i in (0, 6, 12):
    ok = settled_rows(cfg, W, seqs[i], dtype)
    assert ok.mean() > 0.4 and row_err(lg[101 * i:101 * (i + 1)][ok], oracle_logits(cfg, W, seqs[i])[0][ok]) < TOL[dtype]
  n.close()


def test_mixed_batch_of_portions_and_decoded_rows():
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 6)
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
  """a prompt for the tensor-core attention, a short prompt and a decoded row in ONE step"""
  cfg = config([attn(heads=4, kv_heads=2, dim=16, vdim=24, size=33, keep=5, v_mix=True, mlp=dense(64)), attn(heads=2, kv_heads=2, dim=24, vdim=24, v_mix=True)], width=64)
  W = fo.random_weights(cfg, 16)
  n = make_engine(cfg, W, "bfloat16", max_tokens=600, page_size=8)
  a, b, c = rand_tokens(cfg["vocab"], 90, 1), rand_tokens(cfg["vocab"], 7, 2), rand_tokens(cfg["vocab"], 41, 3)
  ra, rb, rc = (oracle_logits(cfg, W, t)[0] for t in (a, b, c))
  n.step([2], [c[:40]])
  lg, _ = n.step([1, 2, 0], [b, c[40:41], a], want=list(range(98)))
  assert row_err(lg[:7], rb) < TOL["bfloat16"] and row_err(lg[7:8], rc[40:]) < TOL["bfloat16"] and row_err(lg[8:], ra) < TOL["bfloat16"]
  assert n.prompt_attention_launches() > 0
  n.close()


# ---- pages and slots that are given back and used again ----------------------------------------------------------------------
def test_freed_pages_and_slots_are_clean_for_the_next_request():
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 13)
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
def plant(cfg, W, gain=2.0):
  """The last two tokens of the vocabulary get embeddings made for each other: the key of the first and every query of the second
  point along one sign vector on the head entries that are not rotated (the first layer's norm weight and projections are inverted for
  it), so that this pair's score stands out whatever the distance.  Filters of queries and keys pass the current token only, their
  biases and the pair table are off, values keep their filters.  Returns (key token, query token)."""
  m, V, D = cfg["layers"][0]["mixer"], cfg["vocab"], cfg["width"]
  rot = (m.get("rot") or {}).get("dims", 0)
  u = torch.zeros(m["dim"], dtype=torch.float64)
  u[rot:] = torch.tensor([1.0, -1.0] * m["dim"], dtype=torch.float64)[:m["dim"] - rot]
  W["bigram"] *= 0.0
  for t in "qk":
    W[f"l0.mix.{t}.b"] *= 0.0
    W[f"l0.mix.{t}.conv"][:, :-1] = 0.0
    W[f"l0.mix.{t}.conv"][:, -1] = 1.0
  W["l0.mix.o"] *= gain
  for tok, t, heads in ((V - 2, "k", m["kv_heads"]), (V - 1, "q", m["heads"])):
    d = torch.linalg.pinv(W[f"l0.mix.{t}"].double() * W["l0.norm1"].double()) @ u.repeat(heads)
    W["embed"][tok] = (d / d.norm() * D ** 0.5).to(torch.bfloat16).float()
  return V - 2, V - 1


# (window, kept, sequence length, position of the planted key, does the last row see it)
EDGES = {"window_oldest": (60, 3, 150, 90, True), "window_just_out": (60, 3, 150, 89, False), "last_kept": (60, 3, 150, 2, True), "first_not_kept": (60, 3, 150, 3, False),
         "first": (60, 3, 150, 0, True), "first_none_kept": (60, 0, 150, 0, False), "far_no_window": (None, 0, 150, 5, True), "page_last": (100, 1, 150, 63, True),
         "page_first": (100, 1, 150, 64, True), "tile_edge": (64, 4, 192, 128, True), "tile_edge_out": (64, 4, 192, 127, False), "newest_but_one": (2, 0, 100, 98, True),
         "window_1": (1, 0, 100, 98, False), "kept_in_later_page": (20, 70, 150, 69, True), "not_kept_in_later_page": (20, 70, 150, 70, False)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("name", sorted(EDGES))
def test_window_edges_kept_tokens_and_page_borders(name, decode, dtype):
  """One key made to take most of the weight of the last row.  Where the row must see it, the key moves the logits by far more than the
  tolerance; where it must not, a mask that is one token off would.  The last 40 rows are decoded one by one when `decode`; sizes of
  the tensor-core attention."""
  size, keep, n_tok, pos, seen = EDGES[name]
  V = 40
  layer = attn(heads=2, kv_heads=1, dim=32, vdim=16, rot_dims=8, size=size, keep=keep, scale=1.0)
  cfg = config([layer], vocab=V, width=96)
  W = fo.random_weights(cfg, 17)
  key_tok, query_tok = plant(cfg, W)
  seq = rand_tokens(V - 2, n_tok, 5)
  seq[-1] = query_tok
  without = oracle_logits(cfg, W, seq)[0]
  seq[pos] = key_tok
  ref = oracle_logits(cfg, W, seq)[0]
  open_cfg = config([attn(heads=2, kv_heads=1, dim=32, vdim=16, rot_dims=8, size=None, scale=1.0)], vocab=V, width=96)
  gain = row_err(without[-1:], ref[-1:]) if seen else row_err(oracle_logits(open_cfg, W, seq)[0][-1:], ref[-1:])
  assert gain > 3 * TOL["bfloat16"], f"{name}: the planted key does not stand out ({gain})"
  n = make_engine(cfg, W, dtype, max_tokens=256, page_size=64 if name.startswith("page") else 16)
  got = run_cut(n, 0, seq, [n_tok - 40, 1] if decode else [n_tok])
  e = row_err(got[-1:], ref[-1:])
  assert e < TOL[dtype], f"{name} ({'decoded' if decode else 'prompt'}): {e:.3e} (the key moves the row by {gain:.2e})"
  assert row_err(got, ref) < TOL[dtype]
  if dtype == "bfloat16":
    assert n.prompt_attention_launches() > 0
  n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_takes_its_share(dtype):
  """tiny scores: the sink weighs as much as one key, and its share falls as keys come in (prompt in both attention forms, and decoding
  over several key runs); larger scores, most below zero, leave nearly everything to it"""
  for scale in (0.01, 0.25, 1.0):
    cfg = config([attn(heads=3, kv_heads=3, dim=16, vdim=8, size=None, scale=scale)], width=32)
    W = fo.random_weights(cfg, 29)
    W["l0.mix.o"] *= 4.0
    W["l0.mix.q.b"] *= 8.0
    W["l0.mix.k.b"] = -W["l0.mix.q.b"]                 # scores below zero on average
    toks = rand_tokens(cfg["vocab"], 200, 7)
    ref = oracle_logits(cfg, W, toks)[0]
    n = make_engine(cfg, W, dtype, max_tokens=1024, page_size=16)
    for slot, cuts in enumerate(([200], [150, 1])):
      assert row_err(run_cut(n, slot, toks, cuts), ref) < TOL[dtype]
    n.set_attention_mode(1)
    assert row_err(run_cut(n, 2, toks, [200]), ref) < TOL[dtype]
    n.close()
  one = fo.softmax_one_more
  fo.softmax_one_more = lambda s: torch.softmax(s, dim=-1)     # a mistake planted in the oracle: no sink
  try:
    assert row_err(oracle_logits(cfg, W, toks)[0], ref) > 2 * TOL["bfloat16"], "the sink must matter"
  finally:
    fo.softmax_one_more = one


def test_rotation_follows_the_position_not_the_portion():
  """scores that rest on the rotated entries alone, low base: a portion that starts at position 13 must turn its queries and keys by the
  positions in the sequence; without a window a kept token's rotation is its own position's"""
  for layer in (attn(heads=2, dim=8, rot_dims=8, base=8.0, size=None, scale=1.5), attn(heads=2, dim=8, rot_dims=8, base=8.0, size=7, keep=3, scale=1.5, scaling=yarn(4.0, 30, 4.0, 0.5))):
    cfg = config([layer], width=32)
    W = fo.random_weights(cfg, 31)
    W["l0.mix.o"] *= 4.0
    toks = rand_tokens(cfg["vocab"], 60, 9)
    flat = config([layer], width=32)
    flat["layers"][0]["mixer"]["rot"] = None
    assert row_err(oracle_logits(flat, W, toks)[0], oracle_logits(cfg, W, toks)[0]) > 0.05, "the rotation must matter"
    n = make_engine(cfg, W, "float32", page_size=8)
    check(n, cfg, W, toks, [13, 20, 1], "float32")
    n.close()


def test_norm_comes_after_the_rotation_with_its_factor():
  """a large YaRN factor lengthens the rotated entries against the others before the head is normed: norming first, or leaving the factor
  out of the norm, gives other scores"""
  cfg = config([attn(heads=2, dim=16, rot_dims=4, size=None, scale=1.0, scaling=yarn(5000.0, 40, 6.0, 0.5))], width=32)
  W = fo.random_weights(cfg, 31)
  W["l0.mix.o"] *= 4.0
  toks = rand_tokens(cfg["vocab"], 40, 9)
  plain = config([attn(heads=2, dim=16, rot_dims=4, size=None, scale=1.0)], width=32)
  assert row_err(oracle_logits(plain, W, toks)[0], oracle_logits(cfg, W, toks)[0]) > 0.05
  for dtype in DTYPES:
    n = make_engine(cfg, W, dtype, page_size=8)
    check(n, cfg, W, toks, [30, 1], dtype)
    n.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_values_are_what_is_cached(dtype):
  """mixing numbers of 1 (nothing of the layer's own values), 0 (nothing of the first's), beyond 1 and below 0; the first mixing layer's
  own number is wild and must not matter; values of decoded tokens come from the step that brought the token"""
  layers = [attn(v_mix=False, kv_heads=1), attn(v_mix=True)] + [attn(v_mix=True) for _ in range(4)]
  cfg = config(layers, width=40)
  W = fo.random_weights(cfg, 31)
  for i, v in zip(range(1, 6), (77.0, 1.0, 0.0, 1.75, -0.5)):
    W[f"l{i}.mix.vmix"] = torch.tensor(v)
  toks = rand_tokens(cfg["vocab"], 40, 9)
  n = make_engine(cfg, W, dtype, page_size=8)
  for slot, cuts in enumerate(([40], [25, 1], [3])):
    check(n, cfg, W, toks, cuts, dtype, slot=slot)
  n.close()


# ---- several shards ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("split", [1, 2, 3, 4])
def test_two_shards_hand_over_the_stream_and_the_first_values(split):
  """the first mixing layer is layer 1: from split 2 on its values cross the border row by row behind the stream; the last shard holds
  its own copy of the embedding table and no pair table"""
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 31)
  n_layers = len(MIXED)
  a = make_engine(cfg, W, "float32", start=0, end=split - 1)
  b = make_engine(cfg, W, "float32", start=split, end=n_layers - 1)
  extra = 2 * 10 if split >= 2 else 0
  assert (a.hidden_out, b.hidden_in) == (cfg["width"] + extra, cfg["width"] + extra)
  toks = rand_tokens(cfg["vocab"], 19, 7)
  ref = oracle_logits(cfg, W, toks)[0]
  for lo, hi in ((0, 12), (12, 18), (18, 19)):
    hid = a.step([0], [toks[lo:hi]])
    assert hid.shape == (hi - lo, cfg["width"] + extra)
    lg, _ = b.step([0], [hid], want=list(range(hi - lo)))
    assert row_err(lg, ref[lo:hi]) < TOL["float32"]
  a.close()
  b.close()


def test_a_middle_shard_passes_the_first_values_on():
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 32)
  parts = [make_engine(cfg, W, "float32", start=s, end=e) for s, e in ((0, 1), (2, 3), (4, 4))]
  toks = rand_tokens(cfg["vocab"], 15, 7)
  hid = parts[0].step([0], [toks])
  hid = parts[1].step([0], [hid])
  lg, _ = parts[2].step([0], [hid], want=list(range(15)))
  assert row_err(lg, oracle_logits(cfg, W, toks)[0]) < TOL["float32"]
  for p in parts:
    p.close()


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
  W = fo.random_weights(cfg, 3)
  write_model_dir(tmp_path, cfg, W)
  n = make_native(load_model_config(tmp_path), 0, "float32")
  n.load_dir(tmp_path)
  n.begin_pool(64, 1, 8)
  check(n, cfg, W, rand_tokens(cfg["vocab"], 12, 1), [12], "float32")
  n.close()
  for missing in ("bigram", "l0.mix.q.b", "l1.mlp.e3.up", "l1.mix.vmix", "l0.mlp.gate", "l2.mix.v.conv", "l1.norm1", "final.norm", "l3.mlp.router"):
    bad = dict(W)
    del bad[missing]
    write_model_dir(tmp_path, cfg, bad)
    with pytest.raises(Exception, match=missing.replace(".", r"\.")):
      make_native(load_model_config(tmp_path), 0, "float32").load_dir(tmp_path)
  for extra, shape in (("l0.norm2", (48,)), ("l1.mlp.router.b", (6,)), ("l3.mix.q.conv", (20, 3)), ("head", (80, 48)), ("l0.mix.sink", (3,)), ("l0.mix.vmix", (1,)), ("l0.mix.o.b", (48,))):
    bad = dict(W)
    bad[extra] = torch.zeros(*shape)                   # a second norm, a bias, filters of a layer without them, a head, a learned sink, an unmixed layer's number
    write_model_dir(tmp_path, cfg, bad)
    with pytest.raises(Exception, match=extra.replace(".", r"\.")):
      make_native(load_model_config(tmp_path), 0, "float32").load_dir(tmp_path)
  write_model_dir(tmp_path, cfg, W)
  bad = config(MIXED)
  bad["layers"][4]["mixer"]["vdim"] = 12               # values of another size cannot be mixed with the first's
  with pytest.raises(Exception, match="other sizes"):
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
  W = fo.random_weights(cfg, 8)
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
  W = fo.random_weights(cfg, 8)
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
  W = fo.random_weights(cfg, 15)
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
  interleaved; the hidden state that crosses carries the first mixing layer's values"""
  import asyncio
  from xotorch_b200.inference.b200_engine import B200ShardInferenceEngine, LocalDirDownloader
  from xotorch_b200.inference.shard import Shard
  cfg = config([attn(vdim=10, v_mix=True, mlp=dense(36)), attn(heads=2, dim=10, v_mix=False), attn(vdim=10, v_mix=True, mlp=dense(20))])
  W = fo.random_weights(cfg, 27)
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
        assert hid.ndim == 3 and hid.shape[2] == cfg["width"] + 2 * 10
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
  """the two branches of a parallel layer are branches of the captured graph; pair rows and filter inputs are read from what each step
  stages, not from what was captured"""
  cfg = config(MIXED)
  W = fo.random_weights(cfg, 19)
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
  """sizes that are multiples of 8 and prompts of hundreds of rows: the bf16 engine runs its products, prompt attention and experts on the
  tensor cores there; the results must agree with the plain kernels on the same 16-bit operands and with the oracle"""
  layers = [attn(heads=4, kv_heads=2, dim=40, vdim=24, conv=4, rot_dims=16, base=1e4, scaling=yarn(4.0, 128, 16.0, 1.0), size=70, keep=3, v_mix=True, mlp=dense(104)),
            attn(heads=6, kv_heads=2, dim=64, vdim=24, conv=3, rot_dims=64, base=1e4, size=130, keep=9, v_mix=True, mlp=moe(8, 3, 32)),
            attn(heads=2, kv_heads=1, dim=24, vdim=72, conv=2, rot_dims=8, size=None, mlp=moe(4, 2, 16))]
  cfg = config(layers, width=72, vocab=136)
  W = fo.random_weights(cfg, 12)
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
  """a model whose sizes, masks, filters, rotations and layer order are drawn from ranges that include multiples of 8 (tensor-core
  kernels) and odd values (plain kernels)"""
  r = np.random.default_rng(seed)
  pick = lambda *xs: xs[int(r.integers(len(xs)))]
  aligned = seed % 2 == 0
  width = pick(64, 96, 160) if aligned else pick(41, 52, 100)
  mix_kv, mix_v = pick(1, 2, 3), pick(8, 24, 40) if aligned else pick(3, 10, 21)
  layers = []
  for i in range(int(r.integers(2, 6))):
    mixes = r.random() < 0.6
    kv = mix_kv if mixes else pick(1, 2, 4)
    dim = pick(16, 40, 96) if aligned else pick(6, 12, 33)
    rot_dims = pick(0, 4, dim // 4 * 2, dim // 2 * 2)
    kind = pick(None, "dense", "dense", "moe", "moe")
    mlp = None
    if kind == "dense":
      mlp = dense(pick(40, 96) if aligned else pick(29, 60), pick(0.4, 1.5))
    elif kind == "moe":
      E = pick(2, 5, 8)
      mlp = moe(E, int(r.integers(1, min(4, E) + 1)), pick(16, 40) if aligned else pick(9, 20))
    layers.append(attn(heads=kv * pick(1, 2, 3), kv_heads=kv, dim=dim, vdim=mix_v if mixes else (pick(8, 24) if aligned else pick(5, 14)), conv=pick(None, 2, 3, 4, 6), rot_dims=rot_dims,
                       base=pick(50.0, 1e4), scaling=pick(None, yarn(pick(2.0, 8.0), pick(30, 300), pick(8.0, 32.0), 1.0)), size=pick(None, 7, 40, 64), keep=pick(0, 1, 5), v_mix=mixes,
                       scale=pick(0.1, 0.25), mlp=mlp))
  return config(layers, width=width, vocab=pick(50, 131), eps=pick(1e-6, 1e-3), scale=pick(0.3, 1.0), buckets=pick(None, 31, 97), logit_scale=pick(0.5, 1.0))


def row_errors(got, ref):
  d = got.astype(np.float64) - ref
  d = d - d.mean(axis=-1, keepdims=True)
  r = ref - ref.mean(axis=-1, keepdims=True)
  return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1) + 1e-30)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(12))
def test_models_drawn_at_random(seed, dtype):
  """whole prompts (one long enough for the tensor-core kernels next to a short one), then decoding together, then a portion"""
  cfg = random_model(seed)
  W = fo.random_weights(cfg, 100 + seed)
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
