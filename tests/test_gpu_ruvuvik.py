"""Ruvuvik (layer-list family) on the GPU against the float64 oracle of tests/ref_ruvuvik.py: every mechanism alone, prompts against
token-by-token decoding, prompt portions, ragged batches, slot reuse, one position that decides the output far back and just inside /
outside a chunk's edge (in prompts and decoded), sinks that swallow a head, a token felt hundreds of steps later through the recurrent state,
the edges of the kernels' tiles, the first tokens, long decoding, borrowed weights, odd sizes, greedy generation through the scheduler, the
directory loader and the command-line replay.  Small configurations made here; weights are random but exactly representable in bf16, so the
float32 engine and the oracle see the same numbers and the comparison is sharp."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ref_ruvuvik as R

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4     # relative rms error of a logits row, float32 engine vs float64 oracle
BF16_TOL = 6e-2


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def att(heads=4, kv_heads=2, dim=16, vdim=12, chunk=29, rot=12, base=5000.0, scale=0.4, softcap=6.0, ff=40):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "attention", "mixer": m, "mlp": dense(ff)}


def lat(heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=24, base=20000.0, scale=0.3, ff=40):
    return {"type": "latent_attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def wkv(heads=3, dim=12, ff=40):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": dense(ff)}


def again(layer, of):
    return dict(copy.deepcopy(layer), weights_of=of)


def config(layers, width=64, vocab=131, eps=1e-5):
    return {"architecture": "Ruvuvik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def mixed_config():
    a, b, c, d = att(), wkv(), lat(), att(heads=6, kv_heads=1, dim=10, vdim=20, chunk=11, rot=6, ff=0)
    return config([b, a, c, d, again(a, 1), again(b, 0), wkv(heads=2, dim=20, ff=24), again(c, 2), again(b, 0)])


def load(pkg, cfg, bits, dtype="float32", n_ctx=512, n_seq=8):
    m = pkg.Model.from_config(cfg, dtype=dtype, n_ctx=n_ctx, n_seq=n_seq)
    for name, b in bits.items():
        m.set_tensor(name, pkg.TYPES["bf16"], b)
    m.finalize()
    return m


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def run_whole(m, toks, want=None):
    s = m.seq_alloc()
    lg, _ = m.batch_step([(s, toks, list(range(len(toks))) if want is None else want)])
    m.seq_free(s)
    return lg


def run_rest(m, s, toks, first):
    rows = [m.batch_step([(s, toks[:first], list(range(first)))])[0]]
    for t in toks[first:]:
        rows.append(m.batch_step([(s, [t], [0])])[0])
    return np.concatenate(rows)


def run_decoded(m, toks, first):
    """The first `first` tokens as a prompt, the rest one by one; logits of every position."""
    s = m.seq_alloc()
    out = run_rest(m, s, toks, first)
    m.seq_free(s)
    return out


def check(got, want, tol):
    e = R.rel_err(np.asarray(got, dtype=np.float64), want)
    assert e.max() < tol, f"worst row {int(e.argmax())}: {e.max():.3e} (tolerance {tol})"


def edited(layers, edits=None, **kw):
    return config(layers, **kw), edits or {}


MECHANISMS = {
    "chunked_attention": lambda: edited([att()]),
    "latent_attention": lambda: edited([lat()]),
    "wkv": lambda: edited([wkv()]),
    "one_key_head": lambda: edited([att(heads=5, kv_heads=1, dim=12, vdim=12, chunk=500)]),
    "every_head_its_own": lambda: edited([att(heads=3, kv_heads=3, dim=16, vdim=8, chunk=7)]),
    "whole_head_rotates": lambda: edited([att(rot=16)]),
    "nothing_rotates": lambda: edited([att(rot=0)]),
    "no_chunks": lambda: edited([att(chunk=0)]),
    "chunk_of_one": lambda: edited([att(chunk=1)]),
    "no_softcap": lambda: edited([att(softcap=0.0)]),
    "tight_softcap": lambda: edited([att(softcap=0.7, scale=2.0)]),
    "temperatures_far_apart": lambda: edited([att()], {"l0.mix.temp": lambda a: np.array([-2.0, 0.0, 0.25, 6.0])}),
    "norm_weights_far_apart": lambda: edited([att()], {"l0.mix.q.norm": lambda a: np.linspace(-3.0, 4.0, a.size), "l0.mix.k.norm": lambda a: np.linspace(2.0, -2.0, a.size)}),
    "strong_and_weak_sinks": lambda: edited([lat()], {"l0.mix.sink": lambda a: np.array([9.0, -9.0, 1.0])}),
    "scores_far_below_the_sink": lambda: edited([lat()], {"l0.mix.sink": lambda a: np.array([40.0, 0.0, -40.0])}),
    "large_latent_norm": lambda: edited([lat()], {"l0.mix.dkv.norm": lambda a: 8.0 * a}),
    "fast_and_slow_decays": lambda: edited([wkv()], {"l0.mix.w0": lambda a: np.linspace(-9.0, 3.0, a.size)}),
    "blends_differ_between_inputs": lambda: edited([wkv()], {f"l0.mix.mu.{s}": (lambda a, v=v: 0 * a + v) for s, v in zip("rkvgw", (-0.5, 0.0, 1.0, 0.3, 1.5))}),
    "no_bonus": lambda: edited([wkv()], {"l0.mix.u": lambda a: 0 * a}),
    "strong_bonus": lambda: edited([wkv()], {"l0.mix.u": lambda a: 6.0 * a}),
    "decay_follows_the_token": lambda: edited([wkv()], {"l0.mix.w1": lambda a: 4.0 * a, "l0.mix.w2": lambda a: 2.0 * a}),
    "xielu_numbers": lambda: edited([lat(ff=96)], {"l0.mlp.act": lambda a: np.array([3.0, -4.0])}),
    "no_feed_forward": lambda: edited([att(ff=0), wkv(ff=0), lat(ff=0)]),
    "norms_near_minus_one": lambda: edited([att(), wkv()], {"l0.norm1": lambda a: a - 0.9, "embed.norm": lambda a: a - 0.8, "final.norm": lambda a: a + 2.0}),
    "borrowed_weights": lambda: edited([att(), lat(), wkv(), again(wkv(), 2), again(att(), 0), again(lat(), 1)]),
    "borrowed_from_a_later_layer_and_twice": lambda: edited([again(wkv(), 2), again(lat(), 3), wkv(), lat(), again(wkv(), 0)]),
    "nine_layers": lambda: (mixed_config(), {}),
}


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
@pytest.mark.parametrize("which", sorted(MECHANISMS))
def test_each_mechanism_alone(pkg, cuda, which, dtype, tol):
    cfg, edits = MECHANISMS[which]()
    bits, W = R.random_weights(cfg, seed=3)
    for name, f in edits.items():
        R.set_weight(bits, W, name, f(W[name]))
    toks = tokens_for(cfg, 41, 1)
    want, taps = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    m.tap_layers(True)
    got = run_whole(m, toks)
    got_taps = m.debug_read("layers", taps.size).reshape(taps.shape)
    m.tap_layers(False)
    dec = run_decoded(m, toks, 30)
    m.close()
    check(got, want, tol)
    check(dec, want, tol)
    assert np.abs(got_taps - taps).max() < (1e-4 if dtype == "float32" else 8e-2) * np.abs(taps).max()


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_prompt_and_decoding_agree_with_the_oracle(pkg, cuda, dtype, tol):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=5)
    toks = tokens_for(cfg, 90, 2)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    check(run_whole(m, toks), want, tol)
    check(run_decoded(m, toks, 1), want, tol)    # everything after the first token through the decode path
    check(run_decoded(m, toks, 41), want, tol)
    m.close()


def test_prompt_portions_of_several_sizes(pkg, cuda):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=6)
    toks = tokens_for(cfg, 61, 3)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    for cuts in ([2, 2, 2, 55], [17, 16, 1, 27], [33, 2, 26], [60, 1], [1, 3, 57], [29, 29, 3], [11, 22, 28]):
        s = m.seq_alloc()
        rows, at = [], 0
        for n in cuts:
            rows.append(m.batch_step([(s, toks[at:at + n], list(range(n)))])[0])
            at += n
        m.seq_free(s)
        check(np.concatenate(rows), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ragged_batch_equals_each_request_alone(pkg, cuda, dtype):
    # 1 to 9 live requests: the weight-streaming products of a few tokens and the tiled ones of many
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=7)
    m = load(pkg, cfg, bits, dtype, n_seq=9)
    lens = [1, 70, 9, 33, 18, 2, 29, 30, 58]
    reqs = [tokens_for(cfg, n + 6, 10 + i) for i, n in enumerate(lens)]
    alone = [run_decoded(m, r, n) for r, n in zip(reqs, lens)]
    slots = [m.seq_alloc() for _ in reqs]
    lg, _ = m.batch_step([(s, r[:n], list(range(n))) for s, r, n in zip(slots, reqs, lens)])
    got = [[] for _ in reqs]
    at = 0
    for i, n in enumerate(lens):
        got[i].append(lg[at:at + n])
        at += n
    live = list(range(len(reqs)))
    for k in range(6):
        live = live[:(9, 9, 6, 4, 3, 1)[k]]                    # requests end one after the other
        lg, _ = m.batch_step([(slots[i], [reqs[i][lens[i] + k]], [0]) for i in live])
        for j, i in enumerate(live):
            got[i].append(lg[j:j + 1])
    for i, r in enumerate(reqs):
        g = np.concatenate(got[i])
        assert np.abs(g - alone[i][:len(g)]).max() < (5e-5 if dtype == "float32" else 6e-2) * np.abs(alone[i]).max()
        want, _ = R.forward(cfg, W, r[:len(g)])
        check(g, want, F32_TOL if dtype == "float32" else BF16_TOL)
    m.close()


def test_slots_are_clean_when_handed_out_again(pkg, cuda):
    # caches, recurrent states and the token before the next one must all start empty in a slot that is used again
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=8)
    m = load(pkg, cfg, bits, n_seq=2)
    a, b = tokens_for(cfg, 80, 20), tokens_for(cfg, 23, 21)     # the longer one fills every chunk's rows several times over
    wa, _ = R.forward(cfg, W, a)
    wb, _ = R.forward(cfg, W, b)
    for _ in range(3):                                          # the same two slots over and over, in changing roles
        s0, s1 = m.seq_alloc(), m.seq_alloc()
        lg, _ = m.batch_step([(s0, a, list(range(len(a)))), (s1, b, list(range(len(b))))])
        check(lg[:len(a)], wa, F32_TOL)
        check(lg[len(a):], wb, F32_TOL)
        m.seq_free(s0)
        s2 = m.seq_alloc()
        assert s2 == s0
        check(run_rest(m, s2, b, 5), wb, F32_TOL)
        m.seq_free(s1)
        m.seq_free(s2)
        a, b, wa, wb = b, a, wb, wa
    m.close()


def loud_position_case(layer, T, where, vocab=97, width=48, eps=1e-5):
    """One layer that carries one loud position: token B (only at `where`) has an embedding along a direction that no other token has, and the
    layer's value (or latent) answers that direction far louder than any other; so whoever sees position `where` gets a result far from
    whoever does not."""
    cfg = config([layer], width=width, vocab=vocab, eps=eps)
    bits, W = R.random_weights(cfg, seed=11)
    B = 5
    emb = W["embed"].copy()
    emb[:, 0] = 0.0
    emb[B, :] = 0.0
    emb[B, 0] = 4.0
    R.set_weight(bits, W, "embed", emb)
    toks = [t if t != B else B + 1 for t in tokens_for(cfg, T, 4)]
    toks[where] = B
    return cfg, bits, W, toks


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("chunk", [1000, 59, 60])
def test_one_position_at_a_chunk_edge_decides_the_output(pkg, cuda, chunk, decoded):
    # the loud position is 295 = 5 * 59: the first of its chunk of 59, in the same chunk of 1000, and the last but four of its chunk of 60 that
    # ends before 300.  Queries 296 .. 353 see it under 59 and 1000; under 60 those from 300 on do not.
    cfg, bits, W, toks = loud_position_case(att(heads=2, kv_heads=1, dim=16, vdim=16, chunk=chunk, rot=16, scale=0.05, ff=0), 356, 295)
    wv = W["l0.mix.v"].copy()
    wv[:, 0] = 50.0 * np.sign(wv[:, 1] + 1e-9)
    R.set_weight(bits, W, "l0.mix.v", wv)
    want, _ = R.forward(cfg, W, toks)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["mask"]["size"] = {1000: 60, 59: 60, 60: 59}[chunk]
    moved, _ = R.forward(other, W, toks)
    assert R.rel_err(moved[300:354], want[300:354]).min() > 0.05   # the test is blind unless that one position decides the answers
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 290) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_one_position_far_back_in_latent_attention(pkg, cuda, decoded):
    # position 3 of 400 must still be seen by the last query: every token's query has one large entry, and only the loud token's latent (its
    # first entry, along the loud direction) has a key entry to meet it, so that one score among 400 stands out
    cfg, bits, W, toks = loud_position_case(lat(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, scale=0.2, ff=0), 400, 3)
    emb = W["embed"].copy()
    emb[:, 1] = 2.0
    R.set_weight(bits, W, "embed", emb)
    q, dkv, uk = W["l0.mix.q"].copy(), W["l0.mix.dkv"].copy(), W["l0.mix.uk"].copy()
    dkv[:24, 0] = 0.0
    dkv[0, :] = 0.0
    dkv[0, 0] = 10.0
    for h in range(2):
        q[h * 24, :] = 0.0
        q[h * 24, 1] = 5.0
        uk[h * 16, :] = 0.0
        uk[h * 16, 0] = 1.0
    for name, v in (("l0.mix.q", q), ("l0.mix.dkv", dkv), ("l0.mix.uk", uk)):
        R.set_weight(bits, W, name, v)
    want, _ = R.forward(cfg, W, toks)
    changed = list(toks)
    changed[3] = 6
    moved, _ = R.forward(cfg, W, changed)
    assert R.rel_err(moved[-1:], want[-1:])[0] > 0.1
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 370) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_a_position_turns_by_its_place(pkg, cuda, decoded):
    # all weight of the score on the rotated parts: a key read at another position than its own, or pairs laid out otherwise, answer differently
    cfg = config([lat(heads=2, dim=4, rot_dim=16, vdim=16, kv_rank=24, base=300.0, scale=1.5, ff=0), att(heads=2, kv_heads=2, dim=16, vdim=16, chunk=200, rot=16,
                                                                                                        base=300.0, scale=1.5, softcap=50.0, ff=0)])
    bits, W = R.random_weights(cfg, seed=23)
    R.set_weight(bits, W, "l0.mix.uk", 0 * W["l0.mix.uk"])
    toks = tokens_for(cfg, 150, 4)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 70) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_a_sink_takes_its_share(pkg, cuda, decoded):
    # scores near zero and a sink near ln(number of keys): without it, or with it scaled or counted once per key, the head's result is another
    cfg = config([lat(heads=3, scale=0.02, ff=0)])
    bits, W = R.random_weights(cfg, seed=24)
    R.set_weight(bits, W, "l0.mix.sink", np.array([4.6, 5.5, 3.0]))
    toks = tokens_for(cfg, 180, 4)
    want, _ = R.forward(cfg, W, toks)
    for other in (np.array([-60.0] * 3), np.array([0.0] * 3), np.array([0.1, 0.1, 0.06])):
        W2 = dict(W)
        W2["l0.mix.sink"] = other
        moved, _ = R.forward(cfg, W2, toks)
        assert R.rel_err(moved[-1:], want[-1:])[0] > 50 * F32_TOL
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 120) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


def test_a_token_is_felt_hundreds_of_steps_later_through_the_state(pkg, cuda):
    # with slow decays the first token still moves the last logits 350 positions later, in a prompt and decoded
    cfg = config([wkv(heads=2, dim=24)])
    bits, W = R.random_weights(cfg, seed=12)
    R.set_weight(bits, W, "l0.mix.w0", 0 * W["l0.mix.w0"] - 9.0)
    toks = tokens_for(cfg, 350, 6)
    want, _ = R.forward(cfg, W, toks)
    changed = list(toks)
    changed[0] = (toks[0] + 1) % cfg["vocab"]
    moved, _ = R.forward(cfg, W, changed)
    assert R.rel_err(moved[-1:], want[-1:])[0] > 10 * F32_TOL
    m = load(pkg, cfg, bits)
    check(run_whole(m, toks), want, F32_TOL)
    check(run_decoded(m, toks, 300), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("decoded", [1, 2, 5])
def test_the_previous_token_reaches_every_input(pkg, cuda, decoded):
    # blends of one: every input of the WKV mixer is the token BEFORE the current one (zeros at the start), through prompt cuts too
    cfg = config([wkv(heads=2, dim=8), again(wkv(heads=2, dim=8), 0)])
    bits, W = R.random_weights(cfg, seed=25)
    for s in "rkvgw":
        R.set_weight(bits, W, f"l0.mix.mu.{s}", 0 * W[f"l0.mix.mu.{s}"] + 1.0)
    toks = tokens_for(cfg, 12, 6)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    check(run_whole(m, toks), want, F32_TOL)
    check(run_decoded(m, toks, decoded), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_chunks_pass_over_decoded_tokens_many_times(pkg, cuda, dtype, tol):
    # chunks of 1, 2, 5 and 17 rows: decoding starts each of them anew many times
    cfg = config([att(chunk=17), att(heads=2, kv_heads=2, dim=8, vdim=8, chunk=1, rot=8), att(heads=2, kv_heads=1, dim=12, vdim=20, chunk=2, rot=6),
                  att(heads=3, kv_heads=1, dim=8, vdim=8, chunk=5, rot=8)])
    bits, W = R.random_weights(cfg, seed=13)
    toks = tokens_for(cfg, 170, 5)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    check(run_decoded(m, toks, 20), want, tol)
    check(run_decoded(m, toks, 3), want, tol)                   # the prompt is shorter than a chunk
    check(run_decoded(m, toks, 34), want, tol)                  # the prompt ends with a chunk
    m.close()


@pytest.mark.parametrize("chunk", [128, 200, 300])
def test_chunks_whose_rows_are_split_over_ctas(pkg, cuda, chunk):
    # 128 rows and more: a decode step splits the chunk's rows, most splits are empty right after a chunk has begun
    cfg = config([att(heads=2, kv_heads=1, dim=16, vdim=16, chunk=chunk, rot=8, ff=0)], vocab=53)
    bits, W = R.random_weights(cfg, seed=26)
    toks = tokens_for(cfg, 330, 5)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    check(run_decoded(m, toks, 120), want, F32_TOL)
    check(run_whole(m, toks), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("n", [1, 2, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 130, 200])
def test_lengths_and_chunks_around_the_edges_of_tiles(pkg, cuda, n):
    # prompt attention walks 32 or 64 keys per tile and 4 or 64 queries per CTA, decode attention 128 cache rows per pass, the recurrence and
    # the decay's map 16 tokens: a prompt that ends just before, at and just after an edge, chunks that end there too, then two decoded tokens
    cfg = config([att(heads=2, kv_heads=1, dim=8, vdim=16, chunk=64, rot=8), lat(heads=2, dim=8, vdim=12), wkv(heads=2, dim=16),
                  att(heads=2, kv_heads=1, dim=8, vdim=8, chunk=max(n - 1, 1), rot=8), att(heads=2, kv_heads=2, dim=8, vdim=8, chunk=n + 1, rot=8)], width=32, vocab=53)
    bits, W = R.random_weights(cfg, seed=14)
    toks = tokens_for(cfg, n + 3, n)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    check(run_decoded(m, toks, n), want, F32_TOL)
    m.close()


def test_first_tokens_of_a_sequence(pkg, cuda):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=15)
    m = load(pkg, cfg, bits)
    for tok in (0, 7, cfg["vocab"] - 1):
        want, _ = R.forward(cfg, W, [tok])
        check(run_whole(m, [tok]), want, F32_TOL)
    toks = tokens_for(cfg, 6, 9)
    want, _ = R.forward(cfg, W, toks)
    check(run_decoded(m, toks, 1), want, F32_TOL)
    check(run_decoded(m, toks, 2), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_long_decoding(pkg, cuda, dtype, tol):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=16)
    toks = tokens_for(cfg, 260, 6)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    check(run_decoded(m, toks, 4), want, tol)
    m.close()


ODD = {   # configuration, inner size of the decay's map
    "one_of_everything": lambda: (config([att(heads=1, kv_heads=1, dim=2, vdim=1, chunk=1, rot=2, ff=1), lat(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, ff=1),
                                          wkv(heads=1, dim=1, ff=1)], width=16, vocab=11), 1),
    "odd_sizes": lambda: (config([att(heads=6, kv_heads=3, dim=10, vdim=14, chunk=6, rot=6, ff=50), wkv(heads=5, dim=7, ff=18), lat(heads=5, dim=9, rot_dim=6, vdim=13, kv_rank=35, ff=33),
                                  wkv(heads=2, dim=33, ff=0)], width=30, vocab=67), {1: 5, 3: 19}),
    "values_wider_than_keys": lambda: (config([att(heads=2, kv_heads=2, dim=8, vdim=72, chunk=30, rot=8), lat(heads=2, dim=6, rot_dim=2, vdim=72, kv_rank=40)], vocab=31), 8),
    "wide_heads": lambda: (config([att(heads=2, kv_heads=1, dim=136, vdim=264, chunk=30, rot=64), lat(heads=2, dim=130, rot_dim=64, vdim=136, kv_rank=260),
                                   wkv(heads=1, dim=136)], vocab=31), 70),
    "many_heads": lambda: (config([att(heads=20, kv_heads=4, dim=8, vdim=8, chunk=16, rot=4), lat(heads=35, dim=4, rot_dim=4, vdim=4, kv_rank=16), wkv(heads=17, dim=8)], vocab=31), 130),
    "tensor_core_shapes": lambda: (config([att(heads=4, kv_heads=2, dim=32, vdim=32, chunk=24, rot=32, ff=256), wkv(heads=4, dim=32, ff=128),
                                           lat(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, ff=128), again(wkv(heads=4, dim=32, ff=128), 1)], width=128, vocab=128), 24),
    "state_of_64": lambda: (config([wkv(heads=3, dim=64), wkv(heads=1, dim=64)], vocab=31), 8),
    "state_of_128": lambda: (config([wkv(heads=2, dim=128)], vocab=31), 12),
    "state_of_256": lambda: (config([wkv(heads=1, dim=256)], vocab=31), 8),
    "state_in_shared_memory": lambda: (config([wkv(heads=2, dim=264)], vocab=31), 3),
    "chunk_longer_than_the_context": lambda: (config([att(chunk=100000), lat()]), 8),
    "kv_heads_not_given": lambda: (config([{"type": "attention", "mlp": None, "mixer": {"heads": 3, "dim": 8, "scale": 0.3, "softcap": 9.0, "mask": {"size": 9}, "rot": {"base": 50.0, "dims": 4}}}]), 8),
}


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
@pytest.mark.parametrize("which", sorted(ODD))
def test_other_sizes(pkg, cuda, which, dtype, tol):
    cfg, rank = ODD[which]()
    bits, W = R.random_weights(cfg, seed=17, rank=rank)
    toks = tokens_for(cfg, 45, 7)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    check(run_whole(m, toks), want, tol)
    check(run_decoded(m, toks, 20), want, tol)
    m.close()


@pytest.mark.parametrize("dim", [32, 64, 128, 256])
def test_recurrence_across_its_chunks(pkg, cuda, dim):
    # the recurrence takes 16 tokens at a time: whole chunks, a rest of every kind, cuts inside a chunk, and several entries at once
    cfg = config([wkv(heads=2, dim=dim, ff=0)], width=32, vocab=31)
    bits, W = R.random_weights(cfg, seed=28)
    m = load(pkg, cfg, bits, n_seq=6)
    reqs = [tokens_for(cfg, n, n) for n in (48, 31, 17, 1, 65)]
    wants = [R.forward(cfg, W, r)[0] for r in reqs]
    slots = [m.seq_alloc() for _ in reqs]
    lg, _ = m.batch_step([(s, r, list(range(len(r)))) for s, r in zip(slots, reqs)])
    at = 0
    for r, w in zip(reqs, wants):
        check(lg[at:at + len(r)], w, F32_TOL)
        at += len(r)
    for s in slots:
        m.seq_free(s)
    for first in (16, 33, 40):
        check(run_decoded(m, reqs[0], first), wants[0], F32_TOL)
    m.close()


def test_a_prompt_of_more_than_a_thousand_tokens(pkg, cuda):
    # wide token tiles everywhere; two requests, the shorter one ends inside a tile
    cfg = config([wkv(heads=2, dim=32, ff=64), att(heads=2, kv_heads=1, dim=16, vdim=16, chunk=300, rot=16, ff=0), lat(heads=2, dim=16, rot_dim=8, vdim=16, ff=64)], width=64, vocab=53)
    bits, W = R.random_weights(cfg, seed=29)
    a, b = tokens_for(cfg, 1100, 1), tokens_for(cfg, 333, 2)
    wa, wb = R.forward(cfg, W, a)[0], R.forward(cfg, W, b)[0]
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        m = load(pkg, cfg, bits, dtype, n_ctx=1200, n_seq=2)
        s, t = m.seq_alloc(), m.seq_alloc()
        lg, _ = m.batch_step([(s, a, list(range(1100))), (t, b, list(range(333)))])
        check(lg[:1100], wa, tol)
        check(lg[1100:], wb, tol)
        m.close()


def test_tensors_arrive_in_any_order(pkg, cuda):
    # the inner size of the decay's map is nowhere in the configuration: whichever of its two tensors comes first tells it
    cfg = config([wkv(heads=2, dim=8)])
    bits, W = R.random_weights(cfg, seed=27, rank=13)
    toks = tokens_for(cfg, 20, 7)
    want, _ = R.forward(cfg, W, toks)
    for order in (list(bits), list(bits)[::-1]):
        m = load(pkg, cfg, {k: bits[k] for k in order})
        check(run_whole(m, toks), want, F32_TOL)
        m.close()
    m = pkg.Model.from_config(cfg, dtype="float32", n_ctx=64, n_seq=2)
    m.set_tensor("l0.mix.w1", pkg.TYPES["bf16"], bits["l0.mix.w1"])
    with pytest.raises(Exception):                              # the two disagree
        m.set_tensor("l0.mix.w2", pkg.TYPES["bf16"], np.zeros((16, 12), dtype=np.uint16))
    with pytest.raises(Exception):
        m.finalize()
    m.close()


def test_greedy_generation_through_the_scheduler(pkg, cuda):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=20, gain=1.5)
    m = load(pkg, cfg, bits, n_seq=2)                           # fewer slots than requests: two batches
    prompts = [tokens_for(cfg, n, 30 + n) for n in (5, 19, 11)]
    outs = pkg.BatchScheduler(m).generate(prompts, 6)
    for p, o in zip(prompts, outs):
        assert len(o) == 6
        seq = list(p)
        for tok in o:
            lg, _ = R.forward(cfg, W, seq)
            top2 = np.sort(lg[-1])[-2:]
            if top2[1] - top2[0] > 1e-3 * np.abs(lg[-1]).max():   # a clear winner must be the engine's choice
                assert int(np.argmax(lg[-1])) == tok
            seq.append(tok)
    m.close()


def test_directory_loader_and_command_line(pkg, cuda, tmp_path):
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=21, rank={0: 9, 6: 5})
    shapes = R.tensor_shapes(cfg, {0: 9, 6: 5})
    d = tmp_path / "model"
    R.write_model_dir(str(d), cfg, bits, shapes)
    toks = tokens_for(cfg, 30, 4)
    want, _ = R.forward(cfg, W, toks)
    m = pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    check(run_whole(m, toks), want, F32_TOL)
    m.close()
    for gone in ("l1.mix.temp", "l0.mix.mu.g", "l0.mix.w1", "l2.mix.sink", "l2.mix.uv", "l0.mix.r", "l6.mlp.act", "l0.norm2", "embed.norm"):
        R.write_model_dir(str(d), cfg, {k: v for k, v in bits.items() if k != gone}, shapes)
        with pytest.raises(Exception):
            pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    # the command-line replay: a prompt of two requests, then one decoded token each
    R.write_model_dir(str(d), cfg, bits, shapes)
    a, b = toks[:20], tokens_for(cfg, 8, 5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:19], "want": [0, 18]}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}, {"id": "b", "tokens": b[7:], "want": [0]}], "end": ["a", "b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    wa, _ = R.forward(cfg, W, a)
    wb, _ = R.forward(cfg, W, b)
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert "done 0" in p.stdout and "done 1" in p.stdout
    g0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(3, -1)
    g1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1)
    check(g0, np.stack([wa[0], wa[18], wb[6]]), F32_TOL)
    check(g1, np.stack([wa[19], wb[7]]), F32_TOL)
    # greedy generation from the command line against the scheduler in this process
    m = pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    mine = pkg.BatchScheduler(m).generate([a, b], 5)
    m.close()
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "generate"), "--model", str(d), "--dtype", "float32", "--prompt", ",".join(map(str, a)), "--prompt",
                        ",".join(map(str, b)), "--max-new", "5", "--n-ctx", "64"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in p.stdout.split()] == mine


def test_fused_and_single_step_kernels_agree(pkg, cuda, tmp_path):
    # the recurrence's own kernel against the one every gated recurrence shares (PB200_WKV_PLAIN), xIELU in the up product's epilogue against a
    # kernel of its own (PB200_FF_UNFUSED), through the command-line replay: a prompt of two requests, then decoded tokens
    cfg = config([wkv(heads=2, dim=32, ff=72), lat(ff=33), wkv(heads=1, dim=64, ff=40)])
    bits, W = R.random_weights(cfg, seed=22)
    d = tmp_path / "model"
    R.write_model_dir(str(d), cfg, bits, R.tensor_shapes(cfg))
    a, b = tokens_for(cfg, 40, 6), tokens_for(cfg, 9, 7)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:36], "want": list(range(36))}, {"id": "b", "tokens": b[:5], "want": [0, 4]}], "end": []}]
    for k in range(4):
        steps.append({"step": k + 1, "entries": [{"id": "a", "tokens": [a[36 + k]], "want": [0]}, {"id": "b", "tokens": [b[5 + k]], "want": [0]}], "end": ["a", "b"] if k == 3 else []})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    rows = {}
    for mode in ("fused", "single"):
        env = {k: v for k, v in os.environ.items() if k not in ("PB200_WKV_PLAIN", "PB200_FF_UNFUSED")}
        if mode == "single":
            env["PB200_WKV_PLAIN"] = env["PB200_FF_UNFUSED"] = "1"
        out = tmp_path / mode
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600, env=env)
        assert p.returncode == 0, p.stderr[-2000:]
        rows[mode] = np.concatenate([np.fromfile(out / f"{k}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for k in range(5)])
    wa, _ = R.forward(cfg, W, a)
    wb, _ = R.forward(cfg, W, b)
    want = np.concatenate([wa[:36], wb[[0, 4]]] + [np.stack([wa[36 + k], wb[5 + k]]) for k in range(4)])
    check(rows["fused"], want, F32_TOL)
    check(rows["single"], want, F32_TOL)
    assert np.abs(rows["fused"] - rows["single"]).max() < 2e-5 * np.abs(want).max()
