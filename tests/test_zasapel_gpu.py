"""Zasapel on the layer-list decoder against the float64 restatement (tests/zasapel_oracle.py): every mechanism alone, prefill against
token-by-token decoding, portions, mixed batches, pages and slots used again, far keys and far state in prompts and in decoding, page and
chunk borders, other sizes, greedy generation through the scheduler, the command line, the mechanisms' own launchers.  All configurations
are made here, small, with random weights whose values are exact in bfloat16."""
import importlib
import json
import os
import struct
import subprocess
import sys

import numpy as np
import pytest
import torch

import zasapel_oracle as ref
from util import b200

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _models():
    return importlib.import_module("llm-inference-engine_b200.models.zasapel")


def _serving():
    return importlib.import_module("llm-inference-engine_b200.serving")


def session(config, packed, dtype="float32", pool_tokens=512, max_seqs=4, max_batch_tokens=512):
    model = _models().ZasapelModel(config, packed, dtype=dtype, device=DEV, max_tokens=max_batch_tokens, max_seqs=max_seqs,
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


# both mixers, every kind of feed-forward and none, rows borrowed from an earlier layer with other heads and sizes, odd sizes
MIXED = [ref.mingru(width=20, mlp=ref.dense()), ref.latent(mlp=ref.moe()), ref.latent(heads=2, dim=7, vdim=9, kv_rank=16, q_rank=11, scale=0.5, kv_from=1),
         ref.mingru(width=33, mlp=ref.moe(experts=3, top=1, ff=10, limit=0.5)), ref.latent(heads=5, dim=8, vdim=6, kv_rank=20, q_rank=8, mlp=ref.dense(ff=13))]


# ------------------------------------------------------------------ each mechanism alone (one-layer models, residual stream compared)
@pytest.mark.parametrize("layer,kw", [
    (ref.mingru(), {}),
    (ref.mingru(width=1), {}),                                          # a single channel
    (ref.mingru(width=200), {}),                                        # wider than the model, several channel blocks of one thread each
    (ref.mingru(width=640), dict(width=64)),                            # four channels per thread, two channel blocks
    (ref.latent(), {}),
    (ref.latent(heads=1, dim=33, vdim=5, kv_rank=7, q_rank=3), {}),     # one head, nothing a multiple of 4
    (ref.latent(heads=6, dim=16, vdim=24, kv_rank=32, q_rank=48, scale=0.31), {}),   # query rank above the width
    (ref.latent(heads=18, dim=4, vdim=4, kv_rank=16, q_rank=1), {}),    # a query rank of one
    (ref.mingru(mlp=ref.dense()), {}),
    (ref.mingru(mlp=ref.dense(ff=1)), dict(eps=0.1)),                   # the norm of a single value
    (ref.mingru(mlp=ref.dense(ff=9000)), {}),                           # longer than a thread block holds in registers
    (ref.mingru(mlp=ref.dense(ff=9001)), {}),
    (ref.mingru(mlp=ref.moe()), {}),
    (ref.mingru(mlp=ref.moe(experts=1, top=1, ff=7)), {}),
    (ref.mingru(mlp=ref.moe(experts=4, top=4, ff=16, limit=0.2)), {}),  # every expert chosen, a limit that binds nearly everywhere
    (ref.mingru(mlp=ref.moe(experts=70, top=5, ff=8, limit=50.0)), {}), # more experts than a warp; a limit that never binds
    (ref.mingru(mlp=ref.dense()), dict(taps=1)),
    (ref.mingru(mlp=ref.dense()), dict(taps=2)),
    (ref.mingru(mlp=ref.dense()), dict(taps=4)),
    (ref.mingru(mlp=ref.dense()), dict(taps=5)),
    (ref.mingru(mlp=ref.moe()), dict(taps=9, width=37)),
    (ref.latent(mlp=ref.moe()), dict(taps=4, width=31, alpha=0.5)),
    (ref.latent(mlp=ref.moe(ff=16)), dict(taps=3, width=5000, vocab=11)),   # a row longer than a thread block holds in registers (fp32)
    (ref.mingru(mlp=ref.dense()), dict(alpha=1.0, eps=0.3)),            # an epsilon that counts, in every norm
], ids=["mingru", "mingru_1", "mingru_200", "mingru_640", "latent", "latent_odd", "latent_wide_q", "latent_q1", "dense", "dense_ff1", "dense_long", "dense_long_odd",
        "moe", "moe_one", "moe_all", "moe_many", "taps1", "taps2", "taps4", "taps5", "taps9_odd", "odd_width", "wide_row", "eps"])
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
    for t in toks[:12]:
        steps.append(sess.feed([(r, [t], [])], trace=True)[1][0].cpu().numpy())
    assert per_position(np.concatenate(steps), res[0].numpy()[:12]).max() < 2e-5


def test_without_input_convolution_the_sublayers_read_the_stream_itself():
    config = ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe())])
    W, packed = ref.make_weights(config, seed=4)
    for k in W:
        if ".canon" in k:
            W[k] = torch.zeros_like(W[k])
    bare = dict(config)
    del bare["canon"]
    packed = {k: v for k, v in packed.items() if ".canon" not in k}
    req = {"a": tokens_of(config, 40, 2)}
    for schedule in ([[("a", 40)]], [[("a", 20)]] + [[("a", 1)]] * 20):
        check_all(replay(session(bare, packed), req, schedule), config, W, req, 3e-5)


def test_constants_that_are_one_or_equal_elsewhere():
    """alpha, limit, the four activation numbers and the epsilon each do something: another value gives another model, and the engine follows."""
    base = ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe(limit=1.0))], alpha=1.0)
    W, packed = ref.make_weights(base, seed=5)
    toks = tokens_of(base, 50, 3)
    want = want_logits(base, W, toks)
    others = [ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe(limit=1.0))], alpha=3.0),
              ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe(limit=0.25))], alpha=1.0),
              ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe(limit=1.0), scale=0.9)], alpha=1.0),
              ref.make_config([ref.mingru(mlp=ref.dense()), ref.latent(mlp=ref.moe(limit=1.0))], alpha=1.0, eps=0.2)]
    for config in others:
        w = want_logits(config, W, toks)
        assert ref.rel_err(w, want) > 5e-3
        sess = session(config, packed)
        assert ref.rel_err(sess.feed([(sess.open(), toks, list(range(50)))]).cpu().numpy(), w) < 3e-5


def test_whole_model_every_layer_fp32_and_16_bit():
    # every expert is chosen in this configuration, so that 16-bit rounding cannot flip a close choice
    layers = [ref.mingru(width=24, mlp=ref.dense()), ref.latent(heads=3, dim=16, vdim=24, kv_rank=32, q_rank=24, mlp=ref.moe(experts=3, top=3)),
              ref.latent(heads=2, dim=24, vdim=8, kv_rank=32, q_rank=16, kv_from=1, mlp=ref.moe(experts=2, top=2, ff=16)), ref.mingru(width=40)]
    config = ref.make_config(layers, width=48)
    W, packed = ref.make_weights(config, seed=6)
    toks = tokens_of(config, 200, 2)
    res = []
    want = ref.forward(config, W, toks, res).numpy()
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 3e-2), ("float16", 5e-3)):
        sess = session(config, packed, dtype=dtype)
        logits, trace = sess.feed([(sess.open(), toks, list(range(200)))], trace=True)
        for i, got in enumerate(list(trace.cpu().numpy()) + [logits.cpu().numpy()]):
            err = per_position(got, res[i].numpy() if i < len(layers) else want)
            assert np.median(err) < tol and err.max() < 4 * tol, (dtype, i, float(np.median(err)), float(err.max()))


def test_positions_far_from_the_start():
    """The position vector at thousands: angles are formed in enough bits."""
    config = ref.make_config([ref.mingru(width=16)], width=64, taps=2)
    W, packed = ref.make_weights(config, seed=7)
    toks = tokens_of(config, 6000, 4)
    want = want_logits(config, W, toks)
    sess = session(config, packed, pool_tokens=6016, max_seqs=1, max_batch_tokens=6000)
    got = sess.feed([(sess.open(), toks, [0, 1, 4095, 4096, 5000, 5999])]).cpu().numpy()   # one portion of more than 64 x 64 tokens: longer chunks
    assert per_position(got, want[[0, 1, 4095, 4096, 5000, 5999]]).max() < 3e-5
    r = sess.open() if sess.batcher.free_slots() else None
    assert r is None


# ------------------------------------------------------------------ schedules
def test_prefill_equals_token_by_token_decoding_and_first_tokens():
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=8)
    req = {"a": tokens_of(config, 90, 3)}
    whole = replay(session(config, packed), req, [[("a", 90)]])
    single = replay(session(config, packed), req, [[("a", 1)] for _ in range(90)])
    check_all(whole, config, W, req, 5e-5)
    check_all(single, config, W, req, 5e-5)  # includes positions 0, 1, 2 decoded one by one
    assert ref.rel_err(single["a"], whole["a"]) < 2e-5


@pytest.mark.parametrize("taps", [2, 4, 7])
@pytest.mark.parametrize("cuts", [[2] * 60, [1, 2, 3, 5, 8, 13, 21, 34, 33], [63, 1, 1, 55], [64, 6, 50], [128, 2, 7, 1], [7, 113], [8, 7, 8, 9, 64, 65], [130]],
                         ids=["twos", "growing", "page_edge", "page_then_short", "two_chunks", "long_tail", "around_the_short_form", "whole"])
def test_portions(cuts, taps):
    config = ref.make_config(MIXED, taps=taps)
    W, packed = ref.make_weights(config, seed=9)
    req = {"a": tokens_of(config, sum(cuts), 4)}
    got = replay(session(config, packed), req, [[("a", n)] for n in cuts])
    check_all(got, config, W, req, 5e-5)


def test_long_decoding():
    config = ref.make_config(MIXED)
    W, packed = ref.make_weights(config, seed=10)
    req = {"a": tokens_of(config, 330, 5)}
    got = replay(session(config, packed), req, [[("a", 10)]] + [[("a", 1)] for _ in range(320)])
    check_all(got, config, W, req, 1e-4)


def test_mixed_batches_equal_each_request_alone_and_reuse_pages_and_slots():
    config = ref.make_config(MIXED, taps=4)
    W, packed = ref.make_weights(config, seed=11)
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
    layers = [ref.mingru(width=24, mlp=ref.dense()), ref.latent(heads=3, dim=16, vdim=24, kv_rank=32, q_rank=24, mlp=ref.moe(experts=3, top=3)),
              ref.latent(heads=20, dim=8, vdim=8, kv_rank=32, q_rank=16, kv_from=1)]
    config = ref.make_config(layers, width=48, taps=4)
    W, packed = ref.make_weights(config, seed=12)
    req = {"a": tokens_of(config, 140, 6)}
    whole = replay(session(config, packed, dtype=dtype), req, [[("a", 140)]])["a"]
    cut = replay(session(config, packed, dtype=dtype), req, [[("a", 3)], [("a", 70)], [("a", 2)]] + [[("a", 1)]] * 65)["a"]
    assert ref.rel_err(cut, whole) < (1e-2 if dtype == "bfloat16" else 2e-3)


def test_a_slot_used_again_starts_from_nothing():
    """State of a finished sequence -- recurrent state, ring of convolution inputs -- must not reach the next one in its slot."""
    config = ref.make_config([ref.mingru(mlp=ref.moe()), ref.latent()], taps=6)
    W, packed = ref.make_weights(config, seed=13)
    sess = session(config, packed, max_seqs=1)
    for seed, cuts in ((1, [40, 1, 1]), (2, [1] * 9), (3, [2, 3, 30]), (4, [5])):
        req = {"a": tokens_of(config, sum(cuts), seed)}
        check_all(replay(sess, req, [[("a", n)] for n in cuts]), config, W, req, 3e-5)


def test_pool_exhaustion_is_refused_not_overwritten():
    config = ref.make_config([ref.latent(), ref.mingru()])
    W, packed = ref.make_weights(config, seed=1)
    sess = session(config, packed, pool_tokens=128, max_seqs=2)
    a, b = sess.open(), sess.open()
    sess.feed([(a, tokens_of(config, 100, 1), [])])
    with pytest.raises(b200().B200Error):
        sess.feed([(b, tokens_of(config, 10, 2), [])])   # both pages are a's
    sess.close(a)
    got = sess.feed([(b, tokens_of(config, 10, 2), [9])]).cpu().numpy()
    assert ref.rel_err(got, want_logits(config, W, tokens_of(config, 10, 2))[[9]]) < 5e-5


# ------------------------------------------------------------------ a far key that takes the whole softmax
def _pointing_model(tokens, query_pos, key_pos, seed, heads=2, dim=48, kv_rank=48, q_rank=20):
    """Two latent layers (the second reads the first's rows) whose first layer's query at query_pos is bent, in every head, to the direction in
    which the key of key_pos stands out most among the prompt's keys: that key takes (nearly) the whole softmax."""
    scale = 0.25
    mk = lambda **kw: ref.latent(heads=heads, dim=dim, vdim=16, kv_rank=kv_rank, q_rank=q_rank, scale=scale, **kw)
    config = ref.make_config([mk(), mk(kv_from=0)], width=64)
    W, packed = ref.make_weights(config, seed=seed)
    eps, p = config["norm"]["eps"], "l0.mix."
    x = W["embed"][torch.as_tensor(tokens)] + ref.position_vector(len(tokens), config["width"])
    h = ref.with_conv(x[:query_pos + 1], W["l0.canon1"])
    keys = (ref.latent_rows(h, W, p, eps) @ W[p + "uk"].T).view(query_pos + 1, heads, dim)
    c_q = (ref.rms_unit(h[query_pos] @ W[p + "dq"].T, eps) * W[p + "dq.norm"])
    wq = 0.1 * W[p + "uq"].clone().view(heads, dim, -1)
    for a in range(heads):
        k = keys[:, a]
        u = torch.linalg.solve(k.T @ k + 0.05 * torch.trace(k.T @ k) / dim * torch.eye(dim, dtype=torch.float64), k[key_pos])
        wq[a] += (70.0 / scale / (u @ k[key_pos])) * u[:, None] * (c_q / (c_q @ c_q))[None, :]   # a score of 70
    packed[p + "uq"] = wq.reshape(heads * dim, -1).to(torch.bfloat16)
    W[p + "uq"] = packed[p + "uq"].double()
    return config, W, packed


FAR = [(100, 0), (100, 1), (63, 0), (64, 0), (128, 63), (128, 64), (127, 64), (190, 66), (310, 0), (310, 10), (420, 2), (420, 128)]


@pytest.mark.parametrize("dtype,shape", [("float32", {}), ("bfloat16", {}), ("bfloat16", dict(heads=20, dim=48, kv_rank=64)), ("bfloat16", dict(heads=3, dim=64, kv_rank=256))],
                         ids=["fp32", "few_heads", "many_heads", "rank_256"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("query_pos,key_pos", FAR, ids=lambda v: str(v))
def test_far_key_that_dominates(query_pos, key_pos, decode, dtype, shape):
    probe = ref.make_config([ref.latent()], width=64)
    tokens = tokens_of(probe, query_pos + 1, query_pos * 1000 + key_pos)
    config, W, packed = _pointing_model(tokens, query_pos, key_pos, seed=query_pos + key_pos + 1, **shape)
    other = list(tokens)
    other[key_pos] = (tokens[key_pos] + 7) % config["vocab"]
    want, want_other = want_logits(config, W, tokens)[query_pos], want_logits(config, W, other)[query_pos]
    assert ref.rel_err(want_other, want) > 5e-2   # the far key shows
    cases = [(tokens, want, 3e-5 if dtype == "float32" else 2.5e-2)]
    if dtype == "float32":   # without that key nothing stands out, and large scores lie close together: too close for 16 bits
        cases.append((other, want_other, 2e-4))
    for sequence, expect, tol in cases:
        sess = session(config, packed, dtype=dtype)
        r = sess.open()
        if decode:   # everything before the query is in the pool already; it arrives alone
            sess.feed([(r, sequence[:query_pos], [])])
            got = sess.feed([(r, sequence[query_pos:], [0])]).cpu().numpy()[0]
        else:
            got = sess.feed([(r, sequence, [query_pos])]).cpu().numpy()[0]
        assert ref.rel_err(got, expect) < tol, ref.rel_err(got, expect)


# ------------------------------------------------------------------ a far token that only the recurrent state carries
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("query_pos,key_pos", [(20, 0), (63, 0), (64, 0), (64, 63), (128, 63), (200, 64), (300, 1), (300, 130), (330, 7), (330, 320)], ids=lambda v: str(v))
def test_far_token_in_the_recurrent_state(query_pos, key_pos, decode, dtype):
    """The gate is shut (z next to 0) except at key_pos, where it is bent open: the state hundreds of tokens later is that token's."""
    config = ref.make_config([ref.mingru(width=48)], width=64, taps=3)
    W, packed = ref.make_weights(config, seed=query_pos + 3 * key_pos)
    tokens = tokens_of(config, query_pos + 1, query_pos * 1000 + key_pos)
    x = W["embed"][torch.as_tensor(tokens)] + ref.position_vector(len(tokens), config["width"])
    h = ref.with_conv(x, W["l0.canon1"])
    u = torch.linalg.solve(h.T @ h + 0.002 * torch.trace(h.T @ h) / 64 * torch.eye(64, dtype=torch.float64), h[key_pos])   # where this token stands out most
    wz = 0.02 * W["l0.mix.z"] + 60.0 * torch.ones(48, 1, dtype=torch.float64) * (u / (u @ h[key_pos]))[None, :]
    for name, v in (("l0.mix.z", wz), ("l0.mix.z.b", torch.full((48,), -36.0, dtype=torch.float64))):
        packed[name] = v.to(torch.bfloat16)
        W[name] = packed[name].double()
    other = list(tokens)
    other[key_pos] = (tokens[key_pos] + 7) % config["vocab"]
    want, want_other = want_logits(config, W, tokens)[query_pos], want_logits(config, W, other)[query_pos]
    assert ref.rel_err(want_other, want) > 5e-2
    tol = 3e-5 if dtype == "float32" else 2e-2
    for sequence, expect in ((tokens, want), (other, want_other)) if dtype == "float32" else ((tokens, want),):
        sess = session(config, packed, dtype=dtype)
        r = sess.open()
        if decode:
            sess.feed([(r, sequence[:query_pos], [])])
            got = sess.feed([(r, sequence[query_pos:], [0])]).cpu().numpy()[0]
        else:
            got = sess.feed([(r, sequence, [query_pos])]).cpu().numpy()[0]
        assert ref.rel_err(got, expect) < tol, ref.rel_err(got, expect)


@pytest.mark.parametrize("back", range(0, 6))
@pytest.mark.parametrize("cut", [1, 2, 3, 30])
def test_a_single_tap_reaches_exactly_its_token(back, cut):
    """One tap of the input convolution is the whole convolution: the token `back` places earlier, through the ring when it lies in an earlier
    portion, and nothing before the sequence's start."""
    config = ref.make_config([ref.mingru(mlp=ref.dense())], taps=6)
    W, packed = ref.make_weights(config, seed=20 + back)
    for k in ("l0.canon1", "l0.canon2"):
        w = torch.zeros(config["width"], 6)
        w[:, 5 - back] = 3.0
        packed[k] = w.to(torch.bfloat16)
        W[k] = packed[k].double()
    req = {"a": tokens_of(config, 30, back)}
    check_all(replay(session(config, packed), req, [[("a", min(cut, 30 - i))] for i in range(0, 30, cut)]), config, W, req, 3e-5)


# ------------------------------------------------------------------ the tensor-core kernels of 16-bit engines
@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
def test_tensor_core_paths_against_the_oracle_and_against_single_tokens(dtype):
    """Sizes every tensor-core path takes: tiles of prompt tokens, one-token tiles over 20 heads, a rank of 256, head products and experts on
    128-row tiles (a prompt of 300 tokens), 16-byte pieces everywhere."""
    layers = [ref.mingru(width=128, mlp=ref.dense(ff=192)),
              ref.latent(heads=6, dim=64, vdim=48, kv_rank=80, q_rank=64, mlp=ref.moe(experts=4, top=4, ff=64)),
              ref.latent(heads=20, dim=64, vdim=64, kv_rank=80, q_rank=96, kv_from=1, mlp=ref.moe(experts=4, top=4, ff=64, limit=0.4)),
              ref.latent(heads=2, dim=64, vdim=24, kv_rank=256, q_rank=64, scale=0.1)]
    config = ref.make_config(layers, width=64, taps=4)
    W, packed = ref.make_weights(config, seed=41)
    req = {"a": tokens_of(config, 420, 9)}
    want = want_logits(config, W, req["a"])
    tol = 3e-2 if dtype == "bfloat16" else 5e-3
    runs = {}
    for name, schedule in (("whole", [[("a", 420)]]), ("cut", [[("a", 300)], [("a", 37)], [("a", 70)], [("a", 3)]] + [[("a", 1)]] * 10)):
        runs[name] = replay(session(config, packed, dtype=dtype, pool_tokens=448, max_batch_tokens=448), req, schedule)["a"]
        err = per_position(runs[name], want)
        assert np.median(err) < tol and err.max() < 4 * tol, (name, float(np.median(err)), float(err.max()))
    assert ref.rel_err(runs["cut"], runs["whole"]) < tol / 2


# ------------------------------------------------------------------ the mechanisms' own launchers
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16], ids=["f32", "bf16", "f16"])
@pytest.mark.parametrize("rows,cols", [(1, 1), (3, 7), (5, 64), (4, 4096), (2, 8200), (2, 20000), (3, 9001)])
def test_poly_norm_launcher(rows, cols, dtype):
    m = b200()
    g = torch.Generator().manual_seed(cols)
    x = (1.5 * torch.randn(rows, cols, generator=g)).to(dtype).to(DEV)
    coef = torch.tensor([0.7, -1.1, 0.4, 0.25], device=DEV)
    want = ref.poly_norm(x.cpu().double(), coef.cpu().double(), 1e-3)
    m.poly_norm(x, coef, 1e-3)
    tol = 2e-6 if dtype == torch.float32 else (1e-2 if dtype == torch.bfloat16 else 2e-3)
    assert (x.cpu().double() - want).abs().max().item() < tol * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("cols", [3, 64, 520])
def test_mingru_launcher(cols, dtype):
    """Five portions in one call -- many chunks, two chunks, one short chunk, a few tokens, one token -- some continuing from a state, against a
    plain loop; slots in another order than the sequences, the unused slot untouched."""
    m = b200()
    lens, pos0, slots = [300, 70, 9, 5, 1], [0, 13, 0, 4, 0], [4, 2, 0, 5, 1]
    g = torch.Generator().manual_seed(cols)
    T, ld = sum(lens), 3 * cols + 5
    proj = torch.randn(T, ld, generator=g).to(dtype).to(DEV)
    bias = torch.randn(2 * cols, generator=g).to(DEV)
    state = torch.randn(6, cols, generator=g).to(DEV)
    before = state.cpu().double()
    starts = np.concatenate([[0], np.cumsum(lens)]).tolist()
    out = m.mingru(proj, bias, state, starts, pos0, slots, cols, chunk_tokens=32)
    p, b = proj.cpu().double(), bias.cpu().double()
    for s in range(5):
        S = before[slots[s]].clone() if pos0[s] else torch.zeros(cols, dtype=torch.float64)
        for t in range(starts[s], starts[s + 1]):
            z = torch.sigmoid(p[t, :cols] + b[:cols])
            u = p[t, cols:2 * cols] + b[cols:]
            S = (1 - z) * S + z * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
            gt = p[t, 2 * cols:3 * cols]
            want = S * gt * torch.sigmoid(gt)
            tol = 2e-6 if dtype == torch.float32 else 8e-3
            assert (out[t].cpu().double() - want).abs().max().item() < tol * max(1.0, want.abs().max().item()), (s, t)
        assert torch.allclose(state[slots[s]].cpu().double(), S, rtol=1e-5, atol=1e-6), s
    assert torch.equal(state[3].cpu().double(), before[3])


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
