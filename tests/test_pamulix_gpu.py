"""Pamulix on the layer-list decoder against the float64 restatement (tests/pamulix_oracle.py): every mechanism alone, prefill against
token-by-token decoding, portions, mixed batches, pages and slots used again, far keys and keys on both sides of a block's edge in prompts and
in decoding, values shared between layers, other sizes, greedy generation through the scheduler, the command lines.  All configurations
are made here, small, with random weights whose values are exact in bfloat16."""
import importlib
import json
import math
import os
import struct
import subprocess
import sys

import numpy as np
import pytest
import torch

import pamulix_oracle as ref
from util import b200

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _models():
    return importlib.import_module("llm-inference-engine_b200.models.pamulix")


def _serving():
    return importlib.import_module("llm-inference-engine_b200.serving")


def session(config, packed, dtype="float32", pool_tokens=512, max_seqs=4, max_batch_tokens=512):
    model = _models().PamulixModel(config, packed, dtype=dtype, device=DEV, max_tokens=max_batch_tokens, max_seqs=max_seqs,
                                   max_pages_per_seq=(pool_tokens + 63) // 64)
    return _serving().Session(model, pool_tokens, max_seqs=max_seqs, max_batch_tokens=max_batch_tokens, poison=True)


def tokens_of(config, n, seed):
    return np.random.default_rng(seed).integers(0, config["vocab"], n).tolist()


def replay(sess, requests, schedule):
    """schedule: list of steps, each a list of (name, n) -- the next n tokens of that request, all positions wanted.
    Returns name -> logits [len(tokens), vocab] (numpy)."""
    fed = {k: 0 for k in requests}
    rid, got = {}, {k: [] for k in requests}
    for step in schedule:
        entries = []
        for name, n in step:
            if name not in rid:
                rid[name] = sess.open()
            toks = requests[name][fed[name]:fed[name] + n]
            assert len(toks) == n
            entries.append((rid[name], toks, list(range(n))))
            fed[name] += n
        out = sess.feed(entries).cpu().numpy()
        at = 0
        for name, n in step:
            got[name].append(out[at:at + n])
            at += n
        for name, _ in step:
            if fed[name] == len(requests[name]) and name in rid:
                sess.close(rid.pop(name))
    return {k: np.concatenate(v) for k, v in got.items() if v}


def want_logits(config, W, tokens):
    return ref.forward(config, W, tokens).numpy()


def per_position(got, want):
    return np.linalg.norm(got - want, axis=-1) / np.linalg.norm(want, axis=-1)


def check_all(got, config, W, requests, tol):
    for name, lg in got.items():
        assert not np.isnan(lg).any(), name
        err = per_position(lg, want_logits(config, W, requests[name]))
        assert err.max() < tol, (name, int(err.argmax()), float(err.max()))


# both mixers, experts and none; layers that share values with others between them, a layer that shares none, odd sizes, three block lengths
MIXED = [ref.attention(v_mix=False, heads=3, kv_heads=1, dim=7, vdim=5, chunk=17, mlp=ref.moe()), ref.attention(mlp=ref.moe()),
         ref.latent(mlp=ref.moe(experts=3, top=1, ff=10)), ref.attention(heads=6, dim=9, chunk=70, scale=0.5),
         ref.latent(heads=2, dim=7, rot_dim=6, vdim=9, kv_rank=11, q_rank=5, factor=None), ref.attention(heads=2, chunk=64, mlp=ref.moe(experts=4, top=4))]


# ------------------------------------------------------------------ each mechanism alone (one- and two-layer models, residual stream compared)
@pytest.mark.parametrize("layer,kw", [
    (ref.attention(v_mix=False), {}),
    (ref.attention(heads=1, kv_heads=1, dim=33, vdim=5), {}),                        # one head, nothing a multiple of 4
    (ref.attention(heads=6, kv_heads=6, dim=16, vdim=24, chunk=1), {}),              # a block of a single position
    (ref.attention(heads=8, kv_heads=2, dim=16, vdim=16, chunk=64, scale=0.9), {}),  # blocks that are pages
    (ref.attention(heads=12, kv_heads=3, dim=40, vdim=8, chunk=149), {}),            # head rows that are no power of two of pieces
    (ref.attention(heads=16, kv_heads=1, dim=64, vdim=96, chunk=1000), {}),          # one block longer than the sequence
    (ref.attention(heads=5, kv_heads=5, dim=4, vdim=4, scale=1e-4), {}),             # flat scores: the one in the denominator shows
    (ref.attention(), dict(eps=0.3)),                                                # an epsilon that counts, in every norm
    (ref.latent(), {}),
    (ref.latent(heads=1, dim=33, rot_dim=2, vdim=5, kv_rank=7, q_rank=3), {}),
    (ref.latent(heads=6, dim=16, rot_dim=16, vdim=24, kv_rank=32, q_rank=48, scale=0.31), {}),          # query rank above the width
    (ref.latent(heads=18, dim=4, rot_dim=12, vdim=4, kv_rank=16, q_rank=1), {}),                        # a query rank of one
    (ref.latent(factor=None), {}),                                                                      # plain frequencies
    (ref.latent(rot_dim=32, base=50.0, factor=16.0, original=1000, fast=30.0, slow=2.0), {}),           # the blend spans most pairs
    (ref.latent(rot_dim=16, base=1e6, factor=2.5, original=40, fast=1.0, slow=1.0), {}),                # the band has one pair or none
    (ref.latent(rot_dim=4, base=10.0, factor=3.0, original=100000, fast=4.0, slow=0.5), {}),            # every pair is fast
    (ref.latent(kv_rank=200, rot_dim=24), dict(eps=0.3)),
    (ref.latent(kv_rank=1020, rot_dim=16, heads=2), {}),                                                # a cached row longer than a CTA holds in one piece each
    (ref.attention(mlp=ref.moe()), {}),
    (ref.latent(mlp=ref.moe(experts=1, top=1, ff=7)), {}),
    (ref.attention(mlp=ref.moe(experts=4, top=4, ff=16)), {}),
    (ref.latent(mlp=ref.moe(experts=70, top=5, ff=8)), {}),                                             # more experts than a warp
    (ref.attention(mlp=ref.moe()), dict(width=37, mult=1.0)),
    (ref.latent(mlp=ref.moe()), dict(width=31, mult=2.5)),
    (ref.attention(mlp=ref.moe(ff=16)), dict(width=5000, vocab=11)),
], ids=["attn", "attn_one_head", "attn_chunk1", "attn_page", "attn_dim40", "attn_one_chunk", "attn_flat", "attn_eps", "latent", "latent_odd", "latent_wide_q", "latent_q1",
        "latent_plain", "yarn_wide_band", "yarn_no_band", "yarn_all_fast", "latent_eps", "latent_long_row", "moe", "moe_one", "moe_all", "moe_many", "width37", "width31",
        "wide"])
def test_one_layer_residual_stream(layer, kw):
    config = ref.make_config([layer], **kw)
    W, packed = ref.make_weights(config, seed=3)
    toks = tokens_of(config, 150, 1)
    sess = session(config, packed)
    logits, trace = sess.feed([(sess.open(), toks, [0, 1, 149])], trace=True)
    res = []
    want = ref.forward(config, W, toks, res).numpy()
    assert per_position(trace[0].cpu().numpy(), res[0].numpy()).max() < 2e-5
    assert ref.rel_err(logits.cpu().numpy(), want[[0, 1, 149]]) < 2e-5
    # and token by token: the forms that decode
    r, steps = sess.open(), []
    for t in toks[:24]:
        steps.append(sess.feed([(r, [t], [])], trace=True)[1][0].cpu().numpy())
    assert per_position(np.concatenate(steps), res[0].numpy()[:24]).max() < 2e-5


def test_every_constant_does_something_and_is_followed():
    mk = lambda a={}, l={}, **kw: ref.make_config([ref.attention(mlp=ref.moe()), ref.latent(**l), ref.attention(**dict(dict(chunk=30), **a))], **kw)
    base = mk(mult=1.0)
    W, packed = ref.make_weights(base, seed=5)
    toks = tokens_of(base, 110, 3)
    want = want_logits(base, W, toks)
    for config in (mk(mult=0.5), mk(mult=1.0, eps=0.2), mk(dict(scale=0.8), mult=1.0), mk(dict(chunk=31), mult=1.0), mk(dict(chunk=110), mult=1.0), mk(dict(v_mix=False), mult=1.0),
                   mk(l=dict(scale=0.6), mult=1.0), mk(l=dict(base=300.0), mult=1.0), mk(l=dict(factor=16.0), mult=1.0), mk(l=dict(factor=None), mult=1.0),
                   mk(l=dict(original=512), mult=1.0), mk(l=dict(fast=0.6), mult=1.0), mk(l=dict(slow=0.1), mult=1.0)):
        w = want_logits(config, W, toks)
        assert ref.rel_err(w, want) > 1e-4, config
        sess = session(config, packed)
        assert ref.rel_err(sess.feed([(sess.open(), toks, list(range(110)))]).cpu().numpy(), w) < 2e-5


def test_null_or_absent_mask_is_plain_causal_and_absent_value_mixing_is_none():
    config = ref.make_config([ref.attention(chunk=1000, v_mix=False), ref.attention(chunk=1000, v_mix=False)])
    W, packed = ref.make_weights(config, seed=6)
    bare = json.loads(json.dumps(config))
    bare["layers"][0]["mixer"]["mask"] = None
    for layer in bare["layers"]:
        del layer["mixer"]["v_mix"]
    del bare["layers"][1]["mixer"]["mask"]
    req = {"a": tokens_of(config, 150, 2)}
    check_all(replay(session(bare, packed), req, [[("a", 100)]] + [[("a", 1)]] * 50), config, W, req, 3e-5)


@pytest.mark.parametrize("cuts", [[90], [1] * 90, [40, 2, 1, 47]], ids=["whole", "single", "cut"])
def test_shared_values_come_from_the_first_sharing_layer_of_the_same_token(cuts):
    """The mixing layer takes nearly everything from the first sharing layer; a layer before it shares nothing, one between does as well (its own
    values must not be the ones that travel on)."""
    config = ref.make_config([ref.attention(v_mix=False), ref.attention(), ref.attention(heads=2), ref.latent(), ref.attention(heads=6)])
    W, packed = ref.make_weights(config, seed=7)
    for i, lam in ((1, 0.25), (2, 0.125), (4, 0.96875)):
        packed[f"l{i}.mix.vmix"] = torch.tensor(lam, dtype=torch.bfloat16)
        W[f"l{i}.mix.vmix"] = packed[f"l{i}.mix.vmix"].double()
    req = {"a": tokens_of(config, 90, 4)}
    check_all(replay(session(config, packed), req, [[("a", n)] for n in cuts]), config, W, req, 3e-5)
    other = dict(W, **{"l1.mix.vmix": torch.tensor(0.9, dtype=torch.float64)})
    assert ref.rel_err(want_logits(config, other, req["a"]), want_logits(config, W, req["a"])) == 0.0     # the first layer's number is unused
    for name in ("l2.mix.vmix", "l4.mix.vmix"):
        other = dict(W, **{name: torch.tensor(0.5, dtype=torch.float64)})
        assert ref.rel_err(want_logits(config, other, req["a"]), want_logits(config, W, req["a"])) > 1e-2


def test_router_bias_and_weights_of_far_apart_logits():
    """Logits hundreds apart: the choice still follows the logits where every score but one underflows, and the bias decides."""
    config = ref.make_config([ref.attention(mlp=ref.moe(experts=6, top=3))])
    W, packed = ref.make_weights(config, seed=8)
    for name, v in (("l0.mlp.router", 40.0 * W["l0.mlp.router"]), ("l0.mlp.router.b", torch.tensor([-300.0, 250, 0, 100, -50, 20], dtype=torch.float64))):
        packed[name] = v.to(torch.bfloat16)
        W[name] = packed[name].double()
    req = {"a": tokens_of(config, 60, 5)}
    check_all(replay(session(config, packed), req, [[("a", 40)]] + [[("a", 1)]] * 20), config, W, req, 3e-5)


ALL_EXPERTS = [ref.attention(heads=4, kv_heads=2, dim=16, vdim=24, chunk=50, mlp=ref.moe(experts=3, top=3)),
               ref.latent(heads=3, dim=16, rot_dim=16, vdim=24, kv_rank=32, q_rank=24, mlp=ref.moe(experts=2, top=2, ff=16)),
               ref.attention(heads=2, kv_heads=2, dim=32, vdim=24, chunk=33), ref.latent(heads=20, dim=8, rot_dim=16, vdim=8, kv_rank=32, q_rank=16)]


def test_whole_model_every_layer_fp32_and_16_bit():
    # every expert is chosen in this configuration, so that 16-bit rounding cannot flip a close choice
    config = ref.make_config(ALL_EXPERTS, width=48)
    W, packed = ref.make_weights(config, seed=9)
    toks = tokens_of(config, 200, 2)
    res = []
    want = ref.forward(config, W, toks, res).numpy()
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 2e-2), ("float16", 3e-3)):
        sess = session(config, packed, dtype=dtype)
        logits, trace = sess.feed([(sess.open(), toks, list(range(200)))], trace=True)
        for i, got in enumerate(list(trace.cpu().numpy()) + [logits.cpu().numpy()]):
            err = per_position(got, res[i].numpy() if i < len(ALL_EXPERTS) else want)
            assert np.median(err) < tol and err.max() < 4 * tol, (dtype, i, float(np.median(err)), float(err.max()))


def test_positions_far_from_the_start():
    """Rotation angles, distances and block numbers at thousands are formed in enough bits."""
    config = ref.make_config([ref.latent(heads=2, rot_dim=16, base=20.0, factor=8.0, original=100), ref.attention(heads=2, kv_heads=1, chunk=999)], width=32)
    W, packed = ref.make_weights(config, seed=10)
    toks = tokens_of(config, 4100, 4)
    want = want_logits(config, W, toks)
    sess = session(config, packed, pool_tokens=4160, max_seqs=1, max_batch_tokens=4100)
    at = [0, 1, 998, 999, 3995, 3996, 4095, 4098]
    r = sess.open()
    got = sess.feed([(r, toks[:4099], at)]).cpu().numpy()
    assert per_position(got, want[at]).max() < 3e-5
    assert per_position(sess.feed([(r, toks[4099:], [0])]).cpu().numpy(), want[4099:]).max() < 3e-5


# ------------------------------------------------------------------ schedules
def test_prefill_equals_token_by_token_decoding_and_first_tokens():
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=11)
    req = {"a": tokens_of(config, 90, 3)}
    whole = replay(session(config, packed), req, [[("a", 90)]])
    single = replay(session(config, packed), req, [[("a", 1)] for _ in range(90)])
    check_all(whole, config, W, req, 5e-5)
    check_all(single, config, W, req, 5e-5)  # includes positions 0, 1, 2 decoded one by one
    assert ref.rel_err(single["a"], whole["a"]) < 2e-5


@pytest.mark.parametrize("cuts", [[2] * 60, [1, 2, 3, 5, 8, 13, 21, 34, 33], [63, 1, 1, 55], [64, 6, 50], [69, 1, 1, 2, 67], [16, 1, 2, 101], [128, 2, 7, 1], [7, 113], [8, 7, 8, 9, 64, 65], [130]],
                         ids=["twos", "growing", "page_edge", "page_then_short", "block_edge", "small_block_edge", "two_pages", "long_tail", "around_the_short_form", "whole"])
def test_portions(cuts):
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=12)
    req = {"a": tokens_of(config, sum(cuts), 4)}
    check_all(replay(session(config, packed), req, [[("a", n)] for n in cuts]), config, W, req, 5e-5)


def test_long_decoding():
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=13)
    req = {"a": tokens_of(config, 330, 5)}
    check_all(replay(session(config, packed), req, [[("a", 10)]] + [[("a", 1)] for _ in range(320)]), config, W, req, 1e-4)


def test_mixed_batches_equal_each_request_alone_and_reuse_pages_and_slots():
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=14)
    req = {"a": tokens_of(config, 130, 11), "b": tokens_of(config, 3, 12), "c": tokens_of(config, 75, 13), "d": tokens_of(config, 64, 14),
           "e": tokens_of(config, 100, 15), "f": tokens_of(config, 1, 16), "g": tokens_of(config, 66, 17)}
    # at most 4 alive and 6 pages held at any time, 12 pages and 7 slots asked for over the run: pages and slots come back and go out again
    schedule = [
        [("a", 60), ("b", 1), ("c", 2)],
        [("a", 1), ("b", 2), ("c", 70), ("d", 5)],          # b ends: its slot and page return
        [("a", 4), ("c", 1), ("d", 58), ("f", 1)],          # f takes b's slot, lives for one step
        [("a", 1), ("c", 1), ("d", 1)],                     # a batch of decoded tokens; d ends at a page's last position
        [("a", 64), ("c", 1), ("e", 30)],                   # a and c end; e took d's page and slot
        [("g", 2)],                                         # e is left out of this step
        [("e", 70), ("g", 62)],
        [("g", 1)], [("g", 1)],
    ]
    sess = session(config, packed, pool_tokens=6 * 64, max_seqs=4)
    got = replay(sess, req, schedule)
    check_all(got, config, W, req, 5e-5)
    assert sess.batcher.free_pages() == 6 and sess.batcher.free_slots() == 4
    for name in req:  # and each alone, on a fresh engine: the same numbers up to summation order
        alone = replay(session(config, packed), {name: req[name]}, [[(name, len(req[name]))]])
        assert ref.rel_err(got[name], alone[name]) < 2e-5, name


@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
def test_sixteen_bit_logits_do_not_depend_on_the_schedule(dtype):
    config = ref.make_config(ALL_EXPERTS, width=48)
    W, packed = ref.make_weights(config, seed=15)
    req = {"a": tokens_of(config, 140, 6), "b": tokens_of(config, 73, 7)}
    whole = replay(session(config, packed, dtype=dtype), req, [[("a", 140)], [("b", 73)]])
    cut = replay(session(config, packed, dtype=dtype), req, [[("a", 3)], [("a", 70), ("b", 1)], [("b", 70), ("a", 2)]] + [[("a", 1), ("b", 1)]] * 2 + [[("a", 1)]] * 63)
    for name in req:
        assert ref.rel_err(cut[name], whole[name]) < (1e-2 if dtype == "bfloat16" else 2e-3), name


def test_pages_used_again_carry_nothing_over():
    config = ref.make_config([ref.attention(chunk=100), ref.latent(), ref.attention(chunk=9)])
    W, packed = ref.make_weights(config, seed=16)
    sess = session(config, packed, pool_tokens=128, max_seqs=1)
    for seed, cuts in ((1, [100, 1, 1]), (2, [1] * 9), (3, [2, 3, 90]), (4, [5])):
        req = {"a": tokens_of(config, sum(cuts), seed)}
        check_all(replay(sess, req, [[("a", n)] for n in cuts]), config, W, req, 3e-5)


def test_pool_exhaustion_is_refused_not_overwritten():
    config = ref.make_config([ref.latent(), ref.attention()])
    W, packed = ref.make_weights(config, seed=1)
    sess = session(config, packed, pool_tokens=128, max_seqs=2)
    a, b = sess.open(), sess.open()
    sess.feed([(a, tokens_of(config, 100, 1), [])])
    with pytest.raises(b200().B200Error):
        sess.feed([(b, tokens_of(config, 10, 2), [])])   # both pages are a's
    sess.close(a)
    got = sess.feed([(b, tokens_of(config, 10, 2), [9])]).cpu().numpy()
    assert ref.rel_err(got, want_logits(config, W, tokens_of(config, 10, 2))[[9]]) < 5e-5


# ------------------------------------------------------------------ one key that takes the whole softmax
def _feed_query(sess, tokens, decode):
    """The logits of the last token, which arrives with its whole prompt or alone."""
    r = sess.open()
    if decode:
        sess.feed([(r, tokens[:-1], [])])
        return sess.feed([(r, tokens[-1:], [0])]).cpu().numpy()[0]
    return sess.feed([(r, tokens, [len(tokens) - 1])]).cpu().numpy()[0]


def _marked_tokens(config, query_pos, key_pos):
    """Token 1 at the query, token 0 at the key and nowhere else."""
    tokens = [2 + t % (config["vocab"] - 2) for t in tokens_of(config, query_pos + 1, query_pos * 1000 + key_pos)]
    tokens[key_pos], tokens[query_pos] = 0, 1
    return tokens


def _block_pointing(chunk, seed, heads=2, kv_heads=1, dim=48, vdim=20):
    """One attention layer in which the query of token 1 points, in every head, at the key of token 0 (score 72 before the distance bias; the
    others' are below half of that)."""
    config = ref.make_config([ref.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, chunk=chunk, scale=72.0 / dim)], width=64, mult=1.0)
    W, packed = ref.make_weights(config, seed=seed)
    e = W["embed"]
    wq = W["l0.mix.q"].clone().view(heads, dim, -1)
    for a in range(heads):
        k = (W["l0.mix.k"] @ e[0]).view(kv_heads, dim)[a // (heads // kv_heads)]
        wq[a] += torch.outer(20.0 * k / k.norm() - wq[a] @ e[1], e[1] / (e[1] @ e[1]))
    one = torch.ones(dim, dtype=torch.float64)
    for name, v in (("l0.mix.q", wq.reshape(heads * dim, -1)), ("l0.mix.q.norm", one), ("l0.mix.k.norm", one)):
        packed[name] = v.to(torch.bfloat16)
        W[name] = packed[name].double()
    return config, W, packed


# (chunk, query, key): first / last positions of a block, pages inside and across, several blocks on; just inside and just outside
EDGES = [(20, 39, 20), (20, 39, 19), (20, 40, 39), (20, 40, 20), (64, 127, 64), (64, 127, 63), (64, 128, 127), (100, 199, 100), (100, 199, 99), (100, 250, 200), (100, 250, 199),
         (300, 299, 0), (300, 300, 299), (300, 420, 300), (300, 420, 299), (257, 300, 257), (257, 300, 256), (400, 330, 10), (400, 330, 64), (400, 330, 63)]


@pytest.mark.parametrize("dtype,shape", [("float32", {}), ("bfloat16", dict(dim=64, vdim=32)), ("bfloat16", dict(dim=48, vdim=20)), ("float16", dict(heads=8, kv_heads=2, dim=128, vdim=64))],
                         ids=["fp32", "bf16_tiles", "bf16_per_token", "fp16_tiles"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("chunk,query_pos,key_pos", EDGES, ids=lambda v: str(v))
def test_key_on_both_sides_of_a_blocks_edge(chunk, query_pos, key_pos, decode, dtype, shape):
    config, W, packed = _block_pointing(chunk, seed=chunk + query_pos, **shape)
    tokens = _marked_tokens(config, query_pos, key_pos)
    other = list(tokens)
    other[key_pos] = 5
    want, want_other = want_logits(config, W, tokens)[-1], want_logits(config, W, other)[-1]
    seen = query_pos // chunk == key_pos // chunk
    assert (ref.rel_err(want_other, want) > 5e-2) == seen
    for sequence, expect in ((tokens, want), (other, want_other)) if dtype == "float32" else ((tokens, want),):
        got = _feed_query(session(config, packed, dtype=dtype), sequence, decode)
        # (outside the block several keys share the weight, with scores whose 16-bit rounding counts)
        tol = 3e-5 if dtype == "float32" else (2.5e-2 if seen else 1.5e-1)
        assert ref.rel_err(got, expect) < tol, ref.rel_err(got, expect)


def _latent_pointing(seed, heads=2, dim=48, rot_dim=8, kv_rank=48, q_rank=20):
    """A latent layer in which the query of token 1 points, in every head, to where the key of token 0 stands out most among all tokens' keys."""
    scale = 0.25
    config = ref.make_config([ref.latent(heads=heads, dim=dim, rot_dim=rot_dim, vdim=16, kv_rank=kv_rank, q_rank=q_rank, scale=scale)], width=64, mult=1.0)
    W, packed = ref.make_weights(config, seed=seed)
    eps, p, e = config["norm"]["eps"], "l0.mix.", W["embed"]
    c = ref.rms((e @ W[p + "dkv"].T)[:, :kv_rank], W[p + "dkv.norm"], eps)
    keys = (c @ W[p + "uk"].T).view(-1, heads, dim)
    c_q = ref.rms(e[1] @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    wq = 0.1 * W[p + "uq"].clone().view(heads, dim + rot_dim, -1)
    for a in range(heads):
        k = keys[:, a]
        u = torch.linalg.solve(k.T @ k + 0.05 * torch.trace(k.T @ k) / dim * torch.eye(dim, dtype=torch.float64), k[0])
        wq[a, :dim] += (70.0 / scale / (u @ k[0])) * u[:, None] * (c_q / (c_q @ c_q))[None, :]
    packed[p + "uq"] = wq.reshape(heads * (dim + rot_dim), -1).to(torch.bfloat16)
    W[p + "uq"] = packed[p + "uq"].double()
    return config, W, packed


FAR = [(100, 0), (100, 1), (63, 0), (64, 0), (128, 63), (128, 64), (127, 64), (190, 66), (310, 0), (310, 10), (420, 2), (420, 128)]


@pytest.mark.parametrize("dtype,shape", [("float32", {}), ("bfloat16", {}), ("bfloat16", dict(heads=20, kv_rank=64, rot_dim=16)), ("bfloat16", dict(heads=3, dim=64, kv_rank=256, rot_dim=32))],
                         ids=["fp32", "few_heads", "many_heads", "rank_256"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("query_pos,key_pos", FAR, ids=lambda v: str(v))
def test_far_key_of_the_latent_attention(query_pos, key_pos, decode, dtype, shape):
    config, W, packed = _latent_pointing(seed=query_pos + key_pos, **shape)
    tokens = _marked_tokens(config, query_pos, key_pos)
    other = list(tokens)
    other[key_pos] = 5
    want, want_other = want_logits(config, W, tokens)[-1], want_logits(config, W, other)[-1]
    assert ref.rel_err(want_other, want) > 5e-2
    for sequence, expect, tol in ((tokens, want, 3e-5), (other, want_other, 2e-4)) if dtype == "float32" else ((tokens, want, 2.5e-2),):
        got = _feed_query(session(config, packed, dtype=dtype), sequence, decode)
        assert ref.rel_err(got, expect) < tol, ref.rel_err(got, expect)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("back", [1, 2, 63, 64, 65, 200])
def test_rotated_part_alone_finds_its_distance(back, decode, dtype):
    """Only the rotated part scores (the un-rotated query is zero) and all tokens are the same but two: the query's phase is set so that exactly
    the key `back` places earlier is in phase in every pair."""
    n = 32
    rot = dict(base=3.0, factor=2.0, original=200, fast=20.0, slow=4.0)
    config = ref.make_config([ref.latent(heads=2, dim=8, rot_dim=n, vdim=12, kv_rank=16, q_rank=64, scale=1.6, **rot), ref.attention()], width=64, mult=1.0)
    W, packed = ref.make_weights(config, seed=60 + back)
    tokens = [2] * 260
    tokens[-1], tokens[259 - back] = 1, 0
    freq, amp = ref.pair_frequencies(config["layers"][0]["mixer"]["rot"])
    p, eps, e = "l0.mix.", config["norm"]["eps"], W["embed"]
    # every token's rotated key part is the same vector (the weights see a direction all embeddings share)
    for t in range(e.shape[0]):
        e[t, 0] = 4.0
    down = W[p + "dkv"]
    down[16:] = 0.0
    down[16:, 0] = 0.25 * torch.tensor([1.0, 0.0] * (n // 2), dtype=torch.float64)
    for name, v in (("embed", e), (p + "dkv", down)):
        packed[name] = v.to(torch.bfloat16)
        W[name] = packed[name].double()
    c_q = ref.rms(e[1] @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    target = torch.zeros(2, 8 + n, dtype=torch.float64)
    for i, f in enumerate(freq):   # unit pairs turned back by the distance: q at position 259 and k at 259 - back then point the same way
        target[:, 8 + 2 * i], target[:, 8 + 2 * i + 1] = math.cos(-back * f), math.sin(-back * f)
    wq = 2.0 * target.reshape(-1, 1) * (c_q / (c_q @ c_q))[None, :]
    packed[p + "uq"] = wq.to(torch.bfloat16)
    W[p + "uq"] = packed[p + "uq"].double()
    want = want_logits(config, W, tokens)[-1]
    moved = list(tokens)
    moved[259 - back], moved[258 - back] = 2, 0
    assert ref.rel_err(want_logits(config, W, moved)[-1], want) > 2e-2   # the neighbour is out of phase
    got = _feed_query(session(config, packed, dtype=dtype), tokens, decode)
    assert ref.rel_err(got, want) < (3e-5 if dtype == "float32" else 3e-2), ref.rel_err(got, want)


# ------------------------------------------------------------------ the tensor-core kernels of 16-bit engines
@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
def test_tensor_core_paths_against_the_oracle_and_against_single_tokens(dtype):
    """Sizes every tensor-core path takes: tiles of prompt tokens in blocks that end inside a tile and inside a page, one-token tiles over 20
    heads, a rank of 256, head products and experts on 128-row tiles (a prompt of 300 tokens), 16-byte pieces everywhere."""
    layers = [ref.attention(heads=6, kv_heads=3, dim=64, vdim=32, chunk=90, mlp=ref.moe(experts=4, top=4, ff=64)),
              ref.latent(heads=5, dim=64, rot_dim=16, vdim=48, kv_rank=80, q_rank=64, mlp=ref.moe(experts=4, top=4, ff=64)),
              ref.attention(heads=9, kv_heads=3, dim=128, vdim=32, chunk=37),
              ref.latent(heads=20, dim=64, rot_dim=32, vdim=64, kv_rank=80, q_rank=96),
              ref.attention(heads=3, kv_heads=3, dim=32, vdim=32, chunk=350),
              ref.latent(heads=2, dim=64, rot_dim=16, vdim=24, kv_rank=256, q_rank=64, scale=0.1)]
    config = ref.make_config(layers, width=64)
    W, packed = ref.make_weights(config, seed=41)
    req = {"a": tokens_of(config, 420, 9)}
    want = want_logits(config, W, req["a"])
    tol = 2e-2 if dtype == "bfloat16" else 3e-3
    runs = {}
    for name, schedule in (("whole", [[("a", 420)]]), ("cut", [[("a", 300)], [("a", 37)], [("a", 70)], [("a", 3)]] + [[("a", 1)]] * 10)):
        runs[name] = replay(session(config, packed, dtype=dtype, pool_tokens=448, max_batch_tokens=448), req, schedule)["a"]
        err = per_position(runs[name], want)
        assert np.median(err) < tol and err.max() < 4 * tol, (name, float(np.median(err)), float(err.max()))
    assert ref.rel_err(runs["cut"], runs["whole"]) < tol


# ------------------------------------------------------------------ the scheduler's own entry point, the registry, the command line
@pytest.mark.parametrize("chunk", [0, 5])
def test_greedy_generation_through_the_scheduler(chunk):
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=30)
    prompts = [tokens_of(config, n, 40 + n) for n in (1, 9, 70, 23, 2, 65)]   # six requests over four slots
    sess = session(config, packed, pool_tokens=6 * 64, max_seqs=4, max_batch_tokens=128)
    out = sess.generate(prompts, 12, chunk=chunk)
    for p, ids in zip(prompts, out):
        assert ids == ref.greedy(config, W, p, 12)
    assert sess.batcher.free_pages() == 6 and sess.batcher.free_slots() == 4


def _write_checkpoint(folder, config, packed):
    header, blob = {}, b""
    for k, v in packed.items():
        raw = v.contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    hj = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + blob)
    (folder / "config.json").write_text(json.dumps(config))


def test_registry_loads_a_checkpoint_folder(tmp_path):
    config = ref.make_config(MIXED[:2])
    W, packed = ref.make_weights(config, seed=33)
    _write_checkpoint(tmp_path, config, packed)
    model = importlib.import_module("llm-inference-engine_b200.models").load_model(str(tmp_path), dtype="float32", device=DEV, max_tokens=128, max_seqs=2)
    sess = _serving().Session(model, 128, max_seqs=2)
    toks = tokens_of(config, 20, 1)
    got = sess.feed([(sess.open(), toks, [19])]).cpu().numpy()
    assert ref.rel_err(got, want_logits(config, W, toks)[[19]]) < 5e-5


def test_command_lines_replay_a_schedule_and_generate(tmp_path):
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=34)
    _write_checkpoint(tmp_path, config, packed)
    a, b = tokens_of(config, 80, 1), tokens_of(config, 5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:72], "want": []}, {"id": "b", "tokens": b[:4], "want": [3]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:], "want": [0]}, {"id": "a", "tokens": a[72:], "want": [7]}], "end": ["a", "b"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = want_logits(config, W, a), want_logits(config, W, b)
    got0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    got1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    got2 = np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1)
    assert ref.rel_err(got0, wa[[0, 69]]) < 5e-5 and ref.rel_err(got1, wb[[3]]) < 5e-5 and ref.rel_err(got2, np.stack([wb[4], wa[79]])) < 5e-5
    g = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "b200_generate"), "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6",
                        "--prompt", ",".join(map(str, a[:9])), "--prompt", ",".join(map(str, b))], capture_output=True, text=True, timeout=600)
    assert g.returncode == 0, g.stderr[-2000:]
    lines = [json.loads(l) for l in g.stdout.splitlines() if l.startswith("{")]
    assert [l["generated"] for l in lines] == [ref.greedy(config, W, a[:9], 6), ref.greedy(config, W, b, 6)]
