"""CPU-side tests of the Ruvuvik design: its place in the architecture table, configurations the reader refuses, and the float64 oracle's own
invariants (the GPU tests compare the engine with that oracle)."""
import copy
import json

import numpy as np

import ref_ruvuvik as R


def att(heads=2, kv_heads=1, dim=4, vdim=4, chunk=5, rot=4):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": 8},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 0.5, "softcap": 5.0, "mask": {"size": chunk}, "rot": {"base": 100.0, "dims": rot}}}


def lat(heads=2, dim=4, rot_dim=4, vdim=4, kv_rank=6, rot=4):
    return {"type": "latent_attention", "mlp": None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": 0.5, "rot": {"base": 100.0, "dims": rot}}}


def wkv(heads=2, dim=4):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": None}


def tiny(layers, width=16, vocab=8):
    return {"architecture": "Ruvuvik", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "layers": layers}


def test_architecture_table(lib):
    names = [lib.c.pb200_arch_name(i).decode() for i in range(lib.c.pb200_arch_count())]
    assert "Ruvuvik" in names
    assert lib.c.pb200_arch_family(b"Ruvuvik") == 1


def test_bad_configurations_are_refused_before_any_device_work(lib):
    mk = lib.c.pb200_model_create_from_config

    def refused(cfg):
        return not mk(json.dumps(cfg).encode(), 30, 0, 64, 1)
    assert refused(tiny([]))
    assert refused(tiny([{"type": "mamba2", "mixer": {"heads": 2, "vdim": 4}}]))       # another design's layer
    assert refused(tiny([{"type": "wkv"}]))                                            # no mixer
    assert refused(tiny([att(heads=3, kv_heads=2)]))                                   # query heads per key head
    assert refused(tiny([att(rot=6)]))                                                 # more rotated entries than a head has
    assert refused(tiny([att(rot=3)]))                                                 # pairs need an even count
    assert refused(tiny([lat(rot=6)]))
    assert refused(tiny([lat(kv_rank=0)]))
    assert refused(tiny([wkv(dim=0)]))
    assert refused(tiny([dict(wkv(), mlp={"kind": "moe"})]))                           # unknown feed-forward
    assert refused(tiny([wkv(), dict(wkv(), weights_of=2)]))                           # no such layer
    assert refused(tiny([dict(wkv(), weights_of=0)]))                                  # a layer cannot borrow its own tensors
    assert refused(tiny([dict(wkv(), weights_of=1), dict(wkv(), weights_of=0)]))       # nor two each other's


def test_norm_is_stored_around_zero():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((5, 12)) * 3 + 2
    assert np.allclose((R.zero_centred_norm(x, np.zeros(12), 0.0) ** 2).mean(-1), 1.0)
    assert np.allclose(R.zero_centred_norm(x, np.full(12, -1.0), 0.0), 0.0)
    assert np.allclose(R.rms_unit(np.full((1, 4), 2.0), 12.0), 0.5)                    # eps inside the root: 2 / sqrt(4 + 12)


def test_xielu():
    z = np.linspace(-4, 4, 801)
    y = R.xielu(z, 0.3, -0.7)
    assert y[400] == 0.0
    d = np.diff(y) / np.diff(z)
    assert abs(d[399] - 0.5) < 0.02 and abs(d[400] - 0.5) < 0.02                       # slope 1/2 on both sides of zero
    assert np.isclose(R.xielu(np.array([2.0]), 0.3, -0.7)[0], np.log1p(np.exp(0.3)) * 4 + 1.0)
    want = (0.5 + np.log1p(np.exp(-0.7))) * (np.exp(-3.0) - 1 + 3.0) - 1.5
    assert np.isclose(R.xielu(np.array([-3.0]), 0.3, -0.7)[0], want)


def test_rotation_pairs_neighbours():
    rng = np.random.default_rng(2)
    x = rng.standard_normal((7, 2, 8))
    y = R.rotate(x, np.arange(7) + 3, 6, 50.0)
    assert np.allclose(y[..., 6:], x[..., 6:]) and np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1))
    e = np.zeros((1, 1, 4))
    e[0, 0, 2] = 1.0
    a = 5 * 100.0 ** (-2.0 / 4)                                                        # pair 1 is (2, 3)
    assert np.allclose(R.rotate(e, [5], 4, 100.0)[0, 0], [0, 0, np.cos(a), np.sin(a)])


def test_chunks_count_from_the_sequence_start():
    see = R.visible(np.arange(40)[:, None], np.arange(40)[None, :], 7)
    assert see[13].nonzero()[0].tolist() == list(range(7, 14)) and see[14].nonzero()[0].tolist() == [14]
    assert see[0].sum() == 1 and not see[6, 7]
    assert R.visible(39, 0, None) and not R.visible(0, 1, None)


def test_sink_is_a_key_without_a_value():
    rng = np.random.default_rng(3)
    s, see = rng.standard_normal((6, 6)), np.tril(np.ones((6, 6), dtype=bool))
    w = R.softmax_heads(s, see, 0.7)
    extra = R.softmax_heads(np.concatenate([np.full((6, 1), 0.7), s], 1), np.concatenate([np.ones((6, 1), dtype=bool), see], 1))
    assert np.allclose(w, extra[:, 1:])
    assert np.allclose(R.softmax_heads(s, see, -800.0), R.softmax_heads(s, see)) and (R.softmax_heads(s, see, 800.0) < 1e-200).all()


def test_wkv_recurrence_against_the_unrolled_sum():
    rng = np.random.default_rng(4)
    T, H, d = 9, 2, 3
    r, k, v = (rng.standard_normal((T, H, d)) for _ in range(3))
    w, u = rng.uniform(0.1, 0.99, (T, H, d)), rng.standard_normal((H, d))
    o, S = R.wkv_recurrence(r, k, v, w, u)
    for h in range(H):
        for t in range(T):
            want = (r[t, h] * u[h] * k[t, h]).sum() * v[t, h]
            for j in range(t):                                                         # the current token's decay is not in it yet
                want = want + (r[t, h] * np.prod(w[j + 1:t, h], axis=0) * k[j, h]).sum() * v[j, h]
            assert np.allclose(o[t, h], want)
    o1, S1 = R.wkv_recurrence(r[:4], k[:4], v[:4], w[:4], u)
    o2, S2 = R.wkv_recurrence(r[4:], k[4:], v[4:], w[4:], u, S1)                       # carried across a cut
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)


def test_token_mix():
    h = np.arange(12.0).reshape(4, 3)
    assert np.allclose(R.token_mix(h, np.zeros(3)), h)
    assert np.allclose(R.token_mix(h, np.ones(3)), np.concatenate([np.zeros((1, 3)), h[:-1]]))
    assert np.allclose(R.token_mix(h[2:], np.full(3, 0.5), h[1])[0], 0.5 * (h[1] + h[2]))


def test_model_is_causal_and_borrowed_layers_repeat_their_weights():
    cfg = tiny([att(), wkv(), lat(), dict(wkv(), weights_of=1), dict(att(), weights_of=0)])
    _, W = R.random_weights(cfg, seed=5)
    assert not any(n.startswith(("l3.", "l4.")) for n in W)
    toks = [1, 5, 2, 7, 0, 3, 3, 6]
    full, _ = R.forward(cfg, W, toks)
    part, _ = R.forward(cfg, W, toks[:5])
    assert np.allclose(full[:5], part)
    own = copy.deepcopy(cfg)
    for i in (3, 4):
        del own["layers"][i]["weights_of"]
    W2 = dict(W)
    for name in W:
        for a, b in (("l1.", "l3."), ("l0.", "l4.")):
            if name.startswith(a):
                W2[b + name[len(a):]] = W[name]
    assert np.allclose(R.forward(own, W2, toks)[0], full)
