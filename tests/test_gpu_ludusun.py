"""Ludusun (layer-list family) on the GPU against the float64 oracle of tests/ref_ludusun.py: every mechanism alone, prompts against
token-by-token decoding, prompt portions, ragged batches, slot reuse, one position that decides the output far back and just inside / outside a
window's edge (in prompts and decoded), layers that read another layer's keys and values, sinks, the steps of the query temperature, a token felt
hundreds of steps later through the recurrent state, the edges of the kernels' tiles, the first tokens, long decoding, odd sizes, greedy generation
through the scheduler, the directory loader and the command-line replay.  Small configurations made here; weights are random but exactly
representable in bf16, so the float32 engine and the oracle see the same numbers and the comparison is sharp."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ref_ludusun as R

pytestmark = pytest.mark.gpu

F32_TOL = 5e-5     # relative rms error of a logits row, float32 engine vs float64 oracle
BF16_TOL = 6e-2
YARN = {"factor": 8.0, "original": 96, "fast": 6.0, "slow": 0.5}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def att(heads=4, kv_heads=2, dim=16, vdim=12, rot=12, base=3000.0, yarn=YARN, scale=0.4, ff=40, of=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if yarn:
            m["rot"]["scaling"] = dict(yarn)
    if of is not None:
        m["kv_from"] = of
    return {"type": "attention", "mixer": m, "mlp": dense(ff)}


def lat(heads=3, dim=12, vdim=10, kv_rank=24, q_rank=20, window=29, scale=0.3, ff=40):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": dense(ff)}


def par(heads=4, kv_heads=2, dim=10, scale=0.3, coef=0.6, every=9, r_heads=4, r_kv=2, r_dim=12, r_vdim=8, taps=4, left=0.7, right=1.3, ff=40):
    m = {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale},
         "right": {"heads": r_heads, "kv_heads": r_kv, "dim": r_dim, "vdim": r_vdim, "conv": taps}, "left_scale": left, "right_scale": right}
    if every:
        m["left"]["q_temp"] = {"coef": coef, "every": every}
    return {"type": "parallel", "mixer": m, "mlp": dense(ff)}


def config(layers, width=64, vocab=131, eps=1e-5, scale=8.0, cap=12.0):
    c = {"architecture": "Ludusun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if cap:
        c["logit_softcap"] = cap
    return c


def mixed_config():
    return config([par(), att(), lat(), att(of=1, scale=0.7, ff=0), par(heads=3, kv_heads=1, dim=14, every=4, r_heads=2, r_kv=2, r_dim=32, r_vdim=20, taps=2, ff=0),
                   lat(heads=5, dim=6, vdim=20, kv_rank=9, q_rank=11, window=11), att(heads=6, kv_heads=3, dim=10, vdim=20, rot=6, yarn=None), att(of=1), att(heads=6, kv_heads=3, dim=10, vdim=20, rot=6, yarn=None, of=6, ff=24)])


def load(pkg, cfg, bits, dtype="float32", n_ctx=512, n_seq=8):
    m = pkg.Model.from_config(cfg, dtype=dtype, n_ctx=n_ctx, n_seq=n_seq)
    for name, b in bits.items():
        m.set_tensor(name, pkg.TYPES["bf16"], b)
    m.finalize()
    return m


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def run_whole(m, toks):
    s = m.seq_alloc()
    lg, _ = m.batch_step([(s, toks, list(range(len(toks))))])
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


def silenced(bits, W, cfg, i, side):
    """One branch of a parallel mixer out of action."""
    name = f"l{i}.mix.{side}.o"
    R.set_weight(bits, W, name, 0 * W[name])


MECHANISMS = {
    "attention": lambda: edited([att()]),
    "latent_attention": lambda: edited([lat()]),
    "parallel": lambda: edited([par()]),
    "one_key_head": lambda: edited([att(heads=5, kv_heads=1, dim=12, vdim=12), par(heads=5, kv_heads=1, r_heads=5, r_kv=1)]),
    "every_head_its_own": lambda: edited([att(heads=3, kv_heads=3, dim=16, vdim=8), par(heads=3, kv_heads=3, r_heads=3, r_kv=3)]),
    "whole_head_rotates": lambda: edited([att(rot=16)]),
    "nothing_rotates": lambda: edited([att(rot=0)]),
    "plain_frequencies": lambda: edited([att(yarn=None)]),
    "blend_over_all_pairs": lambda: edited([att(rot=16, base=30.0, yarn={"factor": 30.0, "original": 60, "fast": 9.0, "slow": 0.02})]),
    "blend_in_one_step": lambda: edited([att(rot=16, base=1e6, yarn={"factor": 3.0, "original": 8, "fast": 4.0, "slow": 2.0})]),
    "magnitude_against_unrotated_entries": lambda: edited([att(dim=20, rot=8, yarn={"factor": 4000.0, "original": 64, "fast": 4.0, "slow": 1.0}, scale=1.0)]),
    "large_eps": lambda: edited([att(), par(), lat()], eps=0.3),
    "strong_and_weak_sinks": lambda: edited([att()], {"l0.mix.sink": lambda a: np.array([9.0, -9.0, 1.0, 4.0])}),
    "scores_far_below_the_sink": lambda: edited([att()], {"l0.mix.sink": lambda a: np.array([40.0, 0.0, -40.0, 88.0])}),
    "reads_the_layer_before": lambda: edited([att(), att(of=0, scale=0.9)]),
    "two_readers_and_layers_between": lambda: edited([lat(), att(), par(), att(of=1), att(heads=8, kv_heads=2, dim=16, vdim=12, of=1), att(), att(of=5)]),
    "no_window": lambda: edited([lat(window=0)]),
    "window_of_one": lambda: edited([lat(window=1)]),
    "large_latent_norms": lambda: edited([lat()], {"l0.mix.dkv.norm": lambda a: 6.0 * a, "l0.mix.dq.norm": lambda a: -3.0 * a}),
    "head_gates_far_apart": lambda: edited([lat()], {"l0.mix.g": lambda a: a * np.array([[0.0], [9.0], [-9.0]])}),
    "biases_lead": lambda: edited([par()], {"l0.mix.left.q.b": lambda a: 4.0 * a, "l0.mix.left.k.b": lambda a: 3.0 * a}),
    "no_query_temperature": lambda: edited([par(every=0)]),
    "temperature_at_every_position": lambda: edited([par(every=1, coef=1.5)]),
    "temperature_falls": lambda: edited([par(every=3, coef=-0.4)]),
    "one_tap": lambda: edited([par(taps=1)]),
    "seven_taps": lambda: edited([par(taps=7)]),
    "left_only": lambda: edited([par(right=0.0)]),
    "right_only": lambda: edited([par(left=0.0)]),
    "fast_and_slow_decays": lambda: edited([par()], {"l0.mix.right.A_log": lambda a: np.array([-8.0, -2.0, 1.0, 3.0])}),
    "decay_follows_the_token": lambda: edited([par()], {"l0.mix.right.a1": lambda a: 3.0 * a, "l0.mix.right.a2": lambda a: 3.0 * a}),
    "decay_differs_by_channel": lambda: edited([par()], {"l0.mix.right.dt_bias": lambda a: np.linspace(-9.0, 6.0, a.size)}),
    "steps_near_zero_and_one": lambda: edited([par()], {"l0.mix.right.b": lambda a: 9.0 * a}),
    "recurrence_gate_wide_open": lambda: edited([par()], {"l0.mix.right.g1": lambda a: 4.0 * a}),
    "no_feed_forward": lambda: edited([att(ff=0), par(ff=0), lat(ff=0)]),
    "no_softcap": lambda: edited([lat()], cap=0.0),
    "tight_softcap": lambda: edited([lat()], cap=0.8),
    "plain_embedding": lambda: edited([att()], scale=1.0),
    "norms_near_minus_one": lambda: edited([att(), par()], {"l0.norm1": lambda a: a - 0.9, "l1.norm2": lambda a: a - 0.8, "final.norm": lambda a: a + 2.0}),
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
    assert np.abs(got_taps - taps).max() < (5e-5 if dtype == "float32" else 8e-2) * np.abs(taps).max()


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
    # caches, convolution inputs and recurrent states must all start empty in a slot that is used again
    cfg = mixed_config()
    bits, W = R.random_weights(cfg, seed=8)
    m = load(pkg, cfg, bits, n_seq=2)
    a, b = tokens_for(cfg, 80, 20), tokens_for(cfg, 23, 21)     # the longer one fills every window's rows several times over
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


LOUD = 5


def loud_case(layers, T, where, vocab=97, width=48):
    """Token LOUD, which occurs at `where` alone, has an embedding along a direction that no other token has."""
    cfg = config(layers, width=width, vocab=vocab, scale=2.0)
    bits, W = R.random_weights(cfg, seed=11)
    emb = W["embed"] * np.sqrt(width)
    emb[:, 0] = 0.0
    emb[LOUD, :] = 0.0
    emb[LOUD, 0] = 4.0
    R.set_weight(bits, W, "embed", emb)
    toks = [t if t != LOUD else LOUD + 1 for t in tokens_for(cfg, T, 4)]
    toks[where] = LOUD
    return cfg, bits, W, toks


def loud_column(bits, W, name, gain):
    w = W[name].copy()
    w[:, 0] = gain * np.sign(w[:, 1] + 1e-9)
    R.set_weight(bits, W, name, w)


@pytest.mark.parametrize("decoded", [0, 290, 340])
@pytest.mark.parametrize("window", [49, 50, 51, 160])
def test_one_position_at_a_windows_edge_decides_the_output(pkg, cuda, window, decoded):
    # the loud position is 295: query 344 is the last one that sees it through a window of 50, 343 through one of 49, 345 through one of 51
    cfg, bits, W, toks = loud_case([lat(heads=2, dim=16, vdim=16, kv_rank=24, q_rank=16, window=window, scale=0.05, ff=0)], 350 if window < 100 else 470, 295)
    dkv, uv = W["l0.mix.dkv"].copy(), W["l0.mix.uv"].copy()
    dkv[:, 0], dkv[0, :], dkv[0, 0] = 0.0, 0.0, 10.0             # the loud token's latent is its first entry, no other token's has one
    uv[:, 0] = 30.0 * np.sign(uv[:, 1] + 1e-9)
    R.set_weight(bits, W, "l0.mix.dkv", dkv)
    R.set_weight(bits, W, "l0.mix.uv", uv)
    want, _ = R.forward(cfg, W, toks)
    last = 295 + window - 1                                      # the last query that sees it
    for other in (window - 1, window + 1):
        c2 = copy.deepcopy(cfg)
        c2["layers"][0]["mixer"]["mask"]["size"] = other
        moved, _ = R.forward(c2, W, toks)
        assert R.rel_err(moved[last:last + 2], want[last:last + 2]).max() > 0.05   # the test is blind unless that one position decides the answers
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, decoded) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_one_position_far_back_decides_the_output(pkg, cuda, decoded):
    # position 3 of 400 in the causal layers: through a layer's own keys and through another layer's, each with one loud value; the reader alone
    # (the source's result silenced) as well
    for silence in (None, 0, 1):
        layers = [att(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, scale=0.05, ff=0), att(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, scale=0.05, ff=0, of=0)]
        cfg, bits, W, toks = loud_case(layers, 400, 3)
        loud_column(bits, W, "l0.mix.v", 60.0)
        if silence is not None:
            R.set_weight(bits, W, f"l{silence}.mix.o", 0 * W[f"l{silence}.mix.o"])
        want, _ = R.forward(cfg, W, toks)
        moved, _ = R.forward(cfg, W, toks[:3] + [LOUD + 1] + toks[4:])
        assert R.rel_err(moved[-1:], want[-1:])[0] > 0.05
        m = load(pkg, cfg, bits)
        got = run_decoded(m, toks, 370) if decoded else run_whole(m, toks)
        m.close()
        check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("where", [0, 3, 200])
def test_one_loud_key_that_is_its_own_value(pkg, cuda, where, decoded):
    # left branch alone: one score of 300 stands out, and what it brings is the key itself
    cfg, bits, W, toks = loud_case([par(heads=4, kv_heads=2, dim=16, scale=0.02, every=50, coef=0.5, ff=0)], 300, where)
    silenced(bits, W, cfg, 0, "right")
    loud_column(bits, W, "l0.mix.left.k", 14.0)
    R.set_weight(bits, W, "l0.mix.left.q.b", 2.0 * np.sign(W["l0.mix.left.q.b"]))
    want, _ = R.forward(cfg, W, toks)
    moved, _ = R.forward(cfg, W, toks[:where] + [LOUD + 1] + toks[where + 1:])
    assert R.rel_err(moved[-1:], want[-1:])[0] > 0.05
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 270) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [1, 30, 0])
@pytest.mark.parametrize("every", [1, 7, 10])
def test_the_query_temperature_steps_where_it_should(pkg, cuda, every, decoded):
    # a strong coefficient: positions every - 1, 2 every - 1, .. are the first ones with the next temperature
    cfg = config([par(heads=2, kv_heads=2, dim=16, scale=0.5, every=every, coef=2.0, ff=0)], width=48, vocab=61)
    bits, W = R.random_weights(cfg, seed=31)
    silenced(bits, W, cfg, 0, "right")
    toks = tokens_for(cfg, 45, 4)
    want, _ = R.forward(cfg, W, toks)
    c2 = copy.deepcopy(cfg)
    c2["layers"][0]["mixer"]["left"]["q_temp"]["every"] = every + 1
    moved, _ = R.forward(c2, W, toks)
    assert R.rel_err(moved, want)[every - 1 if every > 1 else 1] > 100 * F32_TOL
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, decoded) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_a_position_turns_by_its_place(pkg, cuda, decoded):
    # sharp scores: a key read at another position than its own, pairs laid out otherwise or frequencies blended otherwise answer differently
    cfg = config([att(heads=2, kv_heads=2, dim=16, vdim=16, rot=16, base=300.0, scale=1.5, ff=0), att(heads=4, kv_heads=2, dim=16, vdim=16, rot=16, base=300.0, scale=1.5, ff=0, of=0)])
    bits, W = R.random_weights(cfg, seed=23)
    toks = tokens_for(cfg, 150, 4)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 70) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


@pytest.mark.parametrize("decoded", [False, True])
def test_a_sink_takes_its_share(pkg, cuda, decoded):
    # scores near zero and a sink near ln(number of keys): without it, or with it scaled or counted once per key, the head's result is another
    cfg = config([att(heads=4, scale=0.02, ff=0), att(heads=4, scale=0.02, ff=0, of=0)])
    bits, W = R.random_weights(cfg, seed=24)
    R.set_weight(bits, W, "l0.mix.sink", np.array([4.6, 5.5, 3.0, 5.0]))
    R.set_weight(bits, W, "l1.mix.sink", np.array([5.0, 3.5, 4.0, 6.0]))
    toks = tokens_for(cfg, 180, 4)
    want, _ = R.forward(cfg, W, toks)
    for name in ("l0.mix.sink", "l1.mix.sink"):
        for factor in (-10.0, 0.0, 0.02):
            W2 = dict(W)
            W2[name] = factor * W[name]
            moved, _ = R.forward(cfg, W2, toks)
            assert R.rel_err(moved[-1:], want[-1:])[0] > 50 * F32_TOL
    m = load(pkg, cfg, bits)
    got = run_decoded(m, toks, 120) if decoded else run_whole(m, toks)
    m.close()
    check(got, want, F32_TOL)


def test_a_token_is_felt_hundreds_of_steps_later_through_the_state(pkg, cuda):
    # with slow decays the first token still moves the last logits 350 positions later (left branch silenced), in a prompt and decoded
    cfg = config([par(r_heads=2, r_kv=1, r_dim=32, r_vdim=24, ff=0)])
    bits, W = R.random_weights(cfg, seed=12)
    silenced(bits, W, cfg, 0, "left")
    R.set_weight(bits, W, "l0.mix.right.A_log", 0 * W["l0.mix.right.A_log"] - 12.0)
    R.set_weight(bits, W, "l0.mix.right.b", 0 * W["l0.mix.right.b"])
    emb = W["embed"].copy()
    emb[7, 0] = 3.0                                                # only the first token (7) writes along the first direction ..
    emb[np.arange(cfg["vocab"]) != 7, 0] = 0.0
    R.set_weight(bits, W, "embed", emb)
    toks = [t if t != 7 else 8 for t in tokens_for(cfg, 350, 6)]
    toks[0] = 7
    loud_column(bits, W, "l0.mix.right.v", 6.0)                    # .. a value far above the others
    want, _ = R.forward(cfg, W, toks)
    moved, _ = R.forward(cfg, W, [8] + toks[1:])
    assert R.rel_err(moved[-1:], want[-1:])[0] > 10 * F32_TOL
    m = load(pkg, cfg, bits)
    check(run_whole(m, toks), want, F32_TOL)
    check(run_decoded(m, toks, 300), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("taps", [1, 2, 3, 6])
def test_the_convolution_reaches_back_through_cuts(pkg, cuda, taps):
    # the oldest tap leads: every input of the recurrence is the token taps - 1 positions back (zeros before the start), through prompt cuts too
    cfg = config([par(r_heads=2, r_kv=2, r_dim=8, r_vdim=12, taps=taps, ff=0)])
    bits, W = R.random_weights(cfg, seed=25)
    silenced(bits, W, cfg, 0, "left")
    for s in "qkv":
        w = 0.1 * W[f"l0.mix.right.{s}.conv"]
        w[:, 0] += 1.0
        R.set_weight(bits, W, f"l0.mix.right.{s}.conv", w)
    toks = tokens_for(cfg, 24, 6)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    check(run_whole(m, toks), want, F32_TOL)
    for first in (1, 2, 3, 5, 8):
        check(run_decoded(m, toks, first), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_windows_pass_over_decoded_tokens_many_times(pkg, cuda, dtype, tol):
    # windows of 1, 2, 5 and 17 rows: decoding wraps each of them many times
    cfg = config([lat(window=17), lat(heads=2, dim=8, vdim=8, kv_rank=16, window=1), lat(heads=2, dim=12, vdim=20, kv_rank=7, window=2), lat(window=5)])
    bits, W = R.random_weights(cfg, seed=13)
    toks = tokens_for(cfg, 170, 5)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits, dtype)
    check(run_decoded(m, toks, 20), want, tol)
    check(run_decoded(m, toks, 3), want, tol)                   # the prompt is shorter than a window
    check(run_decoded(m, toks, 34), want, tol)                  # the prompt ends with a full ring
    m.close()


@pytest.mark.parametrize("window", [64, 128, 200, 300])
def test_windows_whose_rows_are_split_over_ctas(pkg, cuda, window):
    # 64 rows and more: a decode step splits the ring's rows
    cfg = config([lat(heads=2, dim=16, vdim=16, kv_rank=16, window=window, ff=0)], vocab=53)
    bits, W = R.random_weights(cfg, seed=26)
    toks = tokens_for(cfg, 330, 5)
    want, _ = R.forward(cfg, W, toks)
    m = load(pkg, cfg, bits)
    check(run_decoded(m, toks, 120), want, F32_TOL)
    check(run_decoded(m, toks, window), want, F32_TOL)
    check(run_whole(m, toks), want, F32_TOL)
    m.close()


@pytest.mark.parametrize("n", [1, 2, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 130, 200])
def test_lengths_and_windows_around_the_edges_of_tiles(pkg, cuda, n):
    # prompt attention walks 32 or 64 keys per tile and 4 or 64 queries per CTA, decode attention 64 rows per split, the recurrence and its maps 16
    # tokens: a prompt that ends just before, at and just after an edge, windows that end there too, then three decoded tokens
    cfg = config([att(heads=2, kv_heads=1, dim=8, vdim=16, rot=8), lat(heads=2, dim=8, vdim=12, window=64), par(r_heads=2, r_kv=1, r_dim=32, r_vdim=16),
                  lat(heads=2, dim=8, vdim=8, window=max(n - 1, 1)), lat(heads=2, dim=8, vdim=8, window=n + 1), att(heads=2, kv_heads=1, dim=8, vdim=16, rot=8, of=0)], width=32, vocab=53)
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


ODD = {   # configuration, inner sizes of the two low-rank maps
    "one_of_everything": lambda: (config([att(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, ff=1), att(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, ff=1, of=0),
                                          lat(heads=1, dim=1, vdim=1, kv_rank=1, q_rank=1, window=1, ff=1),
                                          par(heads=1, kv_heads=1, dim=1, every=1, r_heads=1, r_kv=1, r_dim=1, r_vdim=1, taps=1, ff=1)], width=16, vocab=11), 1),
    "odd_sizes": lambda: (config([att(heads=6, kv_heads=3, dim=10, vdim=14, rot=6, ff=50), par(heads=5, kv_heads=5, dim=7, r_heads=6, r_kv=2, r_dim=9, r_vdim=13, taps=3, ff=18),
                                  lat(heads=5, dim=9, vdim=13, kv_rank=35, q_rank=17, window=19, ff=33), par(heads=2, kv_heads=1, dim=33, r_heads=2, r_kv=1, r_dim=33, r_vdim=5, ff=0)],
                                 width=30, vocab=67), {1: (5, 3), 3: (19, 66)}),
    "values_wider_than_keys": lambda: (config([att(heads=2, kv_heads=2, dim=8, vdim=72, rot=8), lat(heads=2, dim=6, vdim=72, kv_rank=40), par(r_dim=16, r_vdim=72)], vocab=31), 8),
    "wide_heads": lambda: (config([att(heads=2, kv_heads=1, dim=136, vdim=264, rot=64), lat(heads=2, dim=130, vdim=136, kv_rank=260, q_rank=300),
                                   par(heads=2, kv_heads=1, dim=136, r_heads=1, r_kv=1, r_dim=136, r_vdim=264)], vocab=31), (70, 130)),
    "many_heads": lambda: (config([att(heads=20, kv_heads=4, dim=8, vdim=8, rot=4), lat(heads=35, dim=4, vdim=4, kv_rank=16), par(heads=20, kv_heads=5, dim=4, r_heads=34, r_kv=17, r_dim=8, r_vdim=4)], vocab=31), 130),
    "tensor_core_shapes": lambda: (config([att(heads=4, kv_heads=2, dim=32, vdim=32, rot=32, ff=256), lat(heads=4, dim=32, vdim=32, kv_rank=64, q_rank=64, window=24, ff=128),
                                           par(heads=4, kv_heads=2, dim=32, r_heads=4, r_kv=2, r_dim=32, r_vdim=32, ff=128), att(heads=4, kv_heads=2, dim=32, vdim=32, rot=32, ff=256, of=0)], width=128, vocab=128), (32, 16)),
    "recurrence_of_32": lambda: (config([par(r_heads=3, r_kv=1, r_dim=32, r_vdim=20)], vocab=31), 8),
    "recurrence_of_64": lambda: (config([par(r_heads=3, r_kv=3, r_dim=64, r_vdim=64), par(r_heads=2, r_kv=1, r_dim=64, r_vdim=4)], vocab=31), 8),
    "recurrence_of_128": lambda: (config([par(r_heads=2, r_kv=1, r_dim=128, r_vdim=36)], vocab=31), (12, 65)),
    "recurrence_of_256": lambda: (config([par(r_heads=2, r_kv=2, r_dim=256, r_vdim=16)], vocab=31), 8),
    "recurrence_with_ragged_values": lambda: (config([par(r_heads=2, r_kv=1, r_dim=64, r_vdim=18), par(r_heads=2, r_kv=1, r_dim=20, r_vdim=17)], vocab=31), 8),
    "state_in_shared_memory": lambda: (config([par(r_heads=2, r_kv=1, r_dim=264, r_vdim=70)], vocab=31), 3),
    "window_longer_than_the_context": lambda: (config([lat(window=100000), att()]), 8),
    "sizes_not_given": lambda: (config([{"type": "attention", "mlp": None, "mixer": {"heads": 3, "dim": 8, "scale": 0.3, "rot": {"base": 50.0, "dims": 4}}},
                                        {"type": "parallel", "mlp": None, "mixer": {"left": {"heads": 2, "dim": 8, "scale": 0.3}, "right": {"heads": 3, "dim": 8, "conv": 2}}}]), 8),
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


@pytest.mark.parametrize("dim", [24, 32, 64, 128, 256])
def test_recurrence_across_its_chunks(pkg, cuda, dim):
    # the recurrence takes 16 tokens at a time: whole chunks, a rest of every kind, cuts inside a chunk, and several entries at once
    cfg = config([par(r_heads=2, r_kv=1, r_dim=dim, r_vdim=24, ff=0)], width=32, vocab=31)
    bits, W = R.random_weights(cfg, seed=28)
    silenced(bits, W, cfg, 0, "left")
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
    cfg = config([par(heads=2, kv_heads=1, dim=16, every=100, r_heads=2, r_kv=1, r_dim=32, r_vdim=32, ff=64), att(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, ff=0),
                  lat(heads=2, dim=16, vdim=16, window=300, ff=64), att(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, ff=0, of=1)], width=64, vocab=53)
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
    # the inner sizes of the low-rank maps are nowhere in the configuration: whichever of a map's two tensors comes first tells it
    cfg = config([par(), par(taps=2)])
    bits, W = R.random_weights(cfg, seed=27, rank={0: (13, 5), 1: (2, 21)})
    toks = tokens_for(cfg, 20, 7)
    want, _ = R.forward(cfg, W, toks)
    for order in (list(bits), list(bits)[::-1]):
        m = load(pkg, cfg, {k: bits[k] for k in order})
        check(run_whole(m, toks), want, F32_TOL)
        m.close()
    for first, second, size in (("l0.mix.right.a1", "l0.mix.right.a2", 48 * 12), ("l0.mix.right.g2", "l0.mix.right.g1", 64 * 6)):
        m = pkg.Model.from_config(cfg, dtype="float32", n_ctx=64, n_seq=2)
        m.set_tensor(first, pkg.TYPES["bf16"], bits[first])
        with pytest.raises(Exception):                          # the two disagree
            m.set_tensor(second, pkg.TYPES["bf16"], np.zeros(size, dtype=np.uint16))
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


ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def replay(d, out, steps, env=None):
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600, env=env)
    assert p.returncode == 0, p.stderr[-2000:]
    return p.stdout


def test_directory_loader_and_command_line(pkg, cuda, tmp_path):
    cfg = mixed_config()
    rank = {0: (9, 4), 4: (5, 20)}
    bits, W = R.random_weights(cfg, seed=21, rank=rank)
    shapes = R.tensor_shapes(cfg, rank)
    d = tmp_path / "model"
    R.write_model_dir(str(d), cfg, bits, shapes)
    toks = tokens_for(cfg, 30, 4)
    want, _ = R.forward(cfg, W, toks)
    m = pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    check(run_whole(m, toks), want, F32_TOL)
    m.close()
    for gone in ("embed", "l0.mix.left.q.b", "l0.mix.left.g", "l0.mix.right.a1", "l0.mix.right.g2", "l0.mix.right.k.conv", "l0.mix.right.dt_bias", "l1.mix.sink", "l3.mix.sink",
                 "l2.mix.uv", "l2.mix.dq.norm", "l4.mix.right.o", "l1.mlp.up", "l0.norm2", "final.norm"):
        R.write_model_dir(str(d), cfg, {k: v for k, v in bits.items() if k != gone}, shapes)
        with pytest.raises(Exception):
            pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    # the command-line replay: a prompt of two requests, then one decoded token each
    R.write_model_dir(str(d), cfg, bits, shapes)
    a, b = toks[:20], tokens_for(cfg, 8, 5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:19], "want": [0, 18]}, {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}, {"id": "b", "tokens": b[7:], "want": [0]}], "end": ["a", "b"]}]
    out = tmp_path / "out"
    wa, _ = R.forward(cfg, W, a)
    wb, _ = R.forward(cfg, W, b)
    said = replay(d, out, steps)
    assert "done 0" in said and "done 1" in said
    check(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, -1), np.stack([wa[0], wa[18], wb[6]]), F32_TOL)
    check(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1), np.stack([wa[19], wb[7]]), F32_TOL)
    # greedy generation from the command line against the scheduler in this process
    m = pkg.Model.from_dir(str(d), dtype="float32", n_ctx=64, n_seq=2)
    mine = pkg.BatchScheduler(m).generate([a, b], 5)
    m.close()
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", str(d), "--dtype", "float32", "--prompt", ",".join(map(str, a)), "--prompt",
                        ",".join(map(str, b)), "--max-new", "5", "--n-ctx", "64"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in p.stdout.split()] == mine


SINGLE = ("PB200_DELTA_PLAIN", "PB200_FF_UNFUSED", "PB200_DUAL_UNFUSED", "PB200_ONE_STREAM")


def test_fused_and_single_step_kernels_agree(pkg, cuda, tmp_path):
    # the recurrence's own kernel against the one every gated recurrence shares, the feed-forward's activation in the product's epilogue and the
    # token preparation of both branches in one launch against kernels of their own, two streams against one; through the command-line replay
    cfg = config([par(r_heads=2, r_kv=1, r_dim=32, r_vdim=16, ff=72), lat(ff=33), att(ff=1), par(r_heads=1, r_kv=1, r_dim=64, r_vdim=32, ff=40), att(of=2, ff=100)])
    bits, W = R.random_weights(cfg, seed=22)
    d = tmp_path / "model"
    R.write_model_dir(str(d), cfg, bits, R.tensor_shapes(cfg))
    a, b = tokens_for(cfg, 40, 6), tokens_for(cfg, 9, 7)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:36], "want": list(range(36))}, {"id": "b", "tokens": b[:5], "want": [0, 4]}], "end": []}]
    for k in range(4):
        steps.append({"step": k + 1, "entries": [{"id": "a", "tokens": [a[36 + k]], "want": [0]}, {"id": "b", "tokens": [b[5 + k]], "want": [0]}], "end": ["a", "b"] if k == 3 else []})
    rows = {}
    for mode in ("fused", "single"):
        env = {k: v for k, v in os.environ.items() if k not in SINGLE}
        if mode == "single":
            env.update({k: "1" for k in SINGLE})
        out = tmp_path / mode
        replay(d, out, steps, env)
        rows[mode] = np.concatenate([np.fromfile(out / f"{k}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for k in range(5)])
    wa, _ = R.forward(cfg, W, a)
    wb, _ = R.forward(cfg, W, b)
    want = np.concatenate([wa[:36], wb[[0, 4]]] + [np.stack([wa[36 + k], wb[5 + k]]) for k in range(4)])
    check(rows["fused"], want, F32_TOL)
    check(rows["single"], want, F32_TOL)
    assert np.abs(rows["fused"] - rows["single"]).max() < 2e-5 * np.abs(want).max()
