"""CPU-side tests of the Ludusun design: its place in the architecture table, configurations the reader refuses, and the float64 oracle's own
invariants (the GPU tests compare the engine with that oracle)."""
import json

import numpy as np

import ref_ludusun as R


def att(heads=2, kv_heads=1, dim=4, vdim=4, rot=4, of=None, **more):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 0.5, "rot": {"base": 100.0, "dims": rot}, **more}
    if of is not None:
        m["kv_from"] = of
    return {"type": "attention", "mlp": {"kind": "dense", "ff": 8}, "mixer": m}


def lat(heads=2, dim=4, vdim=4, kv_rank=6, q_rank=5, window=5):
    return {"type": "latent_attention", "mlp": None, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": 0.5, "mask": {"size": window}}}


def par(heads=2, kv_heads=1, dim=4, vdim=4, r_heads=2, r_kv=1, r_dim=3, taps=3, every=4):
    return {"type": "parallel", "mlp": None,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 0.5, "q_temp": {"coef": 0.5, "every": every}},
                      "right": {"heads": r_heads, "kv_heads": r_kv, "dim": r_dim, "vdim": 5, "conv": taps}, "left_scale": 0.5, "right_scale": 2.0}}


def tiny(layers, width=16, vocab=8):
    return {"architecture": "Ludusun", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0}, "logit_softcap": 5.0, "layers": layers}


def test_architecture_table(lib):
    names = [lib.c.pb200_arch_name(i).decode() for i in range(lib.c.pb200_arch_count())]
    assert "Ludusun" in names
    assert lib.c.pb200_arch_family(b"Ludusun") == 1


def test_bad_configurations_are_refused_before_any_device_work(lib):
    mk = lib.c.pb200_model_create_from_config

    def refused(cfg):
        return not mk(json.dumps(cfg).encode(), 30, 0, 64, 1)
    assert refused(tiny([]))
    assert refused(tiny([{"type": "wkv", "mixer": {"heads": 2, "dim": 4}}]))           # another design's layer
    assert refused(tiny([{"type": "attention"}]))                                      # no mixer
    assert refused(tiny([att(heads=3, kv_heads=2)]))                                   # query heads per key head
    assert refused(tiny([att(rot=6)]))                                                 # more rotated entries than a head has
    assert refused(tiny([att(rot=3)]))                                                 # pairs need an even count
    assert refused(tiny([att(mask={"size": 4})]))                                      # these layers are causal without a mask
    assert refused(tiny([att(of=0)]))                                                  # a layer cannot read its own keys as another's
    assert refused(tiny([att(), att(of=2)]))                                           # nor a later layer's
    assert refused(tiny([lat(), att(of=0)]))                                           # nor a latent layer's
    assert refused(tiny([att(), att(of=0), att(of=1)]))                                # nor those of a layer that has none
    assert refused(tiny([att(), att(heads=2, kv_heads=2, of=0)]))                      # nor keys of another shape
    assert refused(tiny([att(), att(vdim=3, of=0)]))
    assert refused(tiny([lat(q_rank=0)]))
    assert refused(tiny([lat(kv_rank=0)]))
    assert refused(tiny([par(vdim=3)]))                                                # a key is its own value
    assert refused(tiny([par(r_heads=3, r_kv=2)]))
    assert refused(tiny([par(taps=0)]))
    assert refused(tiny([par(every=0)]))
    assert refused(tiny([dict(lat(), mlp={"kind": "moe"})]))                           # unknown feed-forward
    assert refused(tiny([{"type": "parallel", "mixer": {"left": par()["mixer"]["left"]}}]))


def test_norm_is_stored_around_zero():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((5, 12)) * 3 + 2
    assert np.allclose((R.zero_centred_norm(x, np.zeros(12), 0.0) ** 2).mean(-1), 1.0)
    assert np.allclose(R.zero_centred_norm(x, np.full(12, -1.0), 0.0), 0.0)
    assert np.allclose(R.rms_unit(np.full((1, 4), 2.0), 12.0), 0.5)                    # eps inside the root: 2 / sqrt(4 + 12)


def test_rotation_pairs_the_halves():
    e = np.zeros((1, 1, 6))
    e[0, 0, 1] = 1.0
    a = 5 * 100.0 ** (-2.0 / 4)                                                        # pair 1 of four rotated entries is (1, 3)
    assert np.allclose(R.rotate(e, [5], {"base": 100.0, "dims": 4})[0, 0], [0, np.cos(a), 0, np.sin(a), 0, 0])
    x = np.random.default_rng(2).standard_normal((7, 2, 8))
    y = R.rotate(x, np.arange(7) + 3, {"base": 50.0, "dims": 6})
    assert np.allclose(y[..., 6:], x[..., 6:]) and np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1))
    sc = {"factor": 4.0, "original": 100, "fast": 8.0, "slow": 1.0}
    y = R.rotate(x, np.arange(7), {"base": 50.0, "dims": 8, "scaling": sc})
    assert np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1) * (0.1 * np.log(4.0) + 1.0) ** 2)


def test_frequency_blend_keeps_fast_pairs_and_slows_slow_ones():
    rot = {"base": 1e4, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    f, mag = R.frequencies(rot)
    g, one = R.frequencies({"base": 1e4, "dims": 64})
    assert one == 1.0 and np.isclose(mag, 1.0 + 0.1 * np.log(8.0))
    r = f / g
    assert r[0] == 1.0 and np.isclose(r[-1], 1 / 8) and (np.diff(r) <= 1e-12).all() and ((r > 0.2) & (r < 0.9)).any()


def test_window_and_sink():
    see = R.visible(np.arange(40)[:, None], np.arange(40)[None, :], 7)
    assert see[13].nonzero()[0].tolist() == list(range(7, 14)) and see[0].sum() == 1 and (see.sum(0)[:33] == 7).all()
    rng = np.random.default_rng(3)
    s, see = rng.standard_normal((6, 6)), np.tril(np.ones((6, 6), dtype=bool))
    w = R.softmax_heads(s, see, 0.7)
    extra = R.softmax_heads(np.concatenate([np.full((6, 1), 0.7), s], 1), np.concatenate([np.ones((6, 1), dtype=bool), see], 1))
    assert np.allclose(w, extra[:, 1:])
    assert np.allclose(R.softmax_heads(s, see, -800.0), R.softmax_heads(s, see)) and (R.softmax_heads(s, see, 800.0) < 1e-200).all()


def test_query_temperature_steps():
    t = R.query_temperature(np.arange(20), 2.0, 5)
    assert np.allclose(t[:4], 1.0) and np.allclose(t[4:9], 1 + 2 * np.log(2)) and np.allclose(t[9:14], 1 + 2 * np.log(3))


def test_convolution_against_its_sum():
    rng = np.random.default_rng(4)
    u, w = rng.standard_normal((6, 3)), rng.standard_normal((3, 4))
    y = R.causal_conv(u, w)
    for t in range(6):
        assert np.allclose(y[t], sum(w[:, 3 - d] * u[t - d] for d in range(4) if t >= d))


def test_delta_recurrence():
    rng = np.random.default_rng(5)
    T, H, d, dv = 9, 2, 3, 4
    q, k, v = rng.standard_normal((T, H, d)), R.unit_vector(rng.standard_normal((T, H, d))), rng.standard_normal((T, H, dv))
    g, beta = rng.uniform(0.1, 0.99, (T, H, d)), rng.uniform(0, 1, (T, H))
    o, S = R.delta_recurrence(q, k, v, g, beta)
    o1, S1 = R.delta_recurrence(q[:4], k[:4], v[:4], g[:4], beta[:4])
    o2, S2 = R.delta_recurrence(q[4:], k[4:], v[4:], g[4:], beta[4:], S1)              # carried across a cut
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # a step of one answers the key it has just written with its value; a step of zero writes nothing
    o3, S3 = R.delta_recurrence(k, k, v, g, np.ones((T, H)))
    assert np.allclose(o3, v, atol=1e-5)
    o4, S4 = R.delta_recurrence(q, k, v, g, np.zeros((T, H)))
    assert np.allclose(S4, 0) and np.allclose(o4, 0)
    # without earlier writes to meet, every write fades by its own channels' decays
    kk = np.zeros((3, 1, 3))
    kk[0, 0, 0] = kk[1, 0, 1] = kk[2, 0, 2] = 1.0
    _, S5 = R.delta_recurrence(kk, kk, np.ones((3, 1, 1)), g[:3, :1], np.ones((3, 1)))
    assert np.allclose(S5[0, :, 0], [g[1, 0, 0] * g[2, 0, 0], g[2, 0, 1], 1.0])


def test_a_reader_with_the_sources_queries_repeats_its_result():
    cfg = tiny([att(), att(of=0)])
    _, W = R.random_weights(cfg, seed=6)
    assert "l1.mix.k" not in W and "l1.mix.v" not in W and "l1.mix.sink" in W
    h, kept = np.random.default_rng(1).standard_normal((7, 16)), {}
    a = R.attention(cfg, cfg["layers"][0]["mixer"], W, "l0.mix.", h, np.arange(7), kept, 0)
    W2 = {n.replace("l0.", "l1."): v for n, v in W.items() if n.startswith("l0.")}
    assert np.allclose(R.attention(cfg, cfg["layers"][1]["mixer"], W2, "l1.mix.", h, np.arange(7), kept, 1), a)
    assert not np.allclose(R.attention(cfg, cfg["layers"][1]["mixer"], W2, "l1.mix.", h, np.arange(7), {0: (kept[0][0], 2 * kept[0][1])}, 1), a)


def test_model_is_causal_and_soft_capped():
    cfg = tiny([att(), par(), lat(), att(of=0)])
    _, W = R.random_weights(cfg, seed=5)
    toks = [1, 5, 2, 7, 0, 3, 3, 6]
    full, taps = R.forward(cfg, W, toks)
    part, _ = R.forward(cfg, W, toks[:5])
    assert np.allclose(full[:5], part) and np.abs(full).max() < 5.0 and taps.shape == (4, 8, 16)
    cfg["logit_softcap"] = 0.0
    assert np.allclose(5.0 * np.tanh(R.forward(cfg, W, toks)[0] / 5.0), full)
