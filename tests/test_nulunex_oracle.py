"""The plain Nulunex implementation against itself and against brute force, and the parts of the product that need no GPU:
configuration, registry, weight packing and sharing, cache."""
import json

import numpy as np
import pytest
import torch

import nulunex_builders as nb
from oracle import nulunex


@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_whole_sequence_equals_pieces(name):
    cfg = nb.CONFIGS[name]
    w, ids = nb.weights(cfg, 1), nb.tokens(cfg, 90, 2)
    whole = nulunex.forward(w, cfg, ids)
    for sizes in ([1] * 90, [2, 3, 2, 30, 2, 51], [64, 26]):
        st, at, out = nulunex.State(len(cfg["layers"])), 0, []
        for n in sizes:
            out.append(nulunex.forward(w, cfg, ids[at : at + n], st))
            at += n
        assert at == 90 and np.abs(np.concatenate(out) - whole).max() < 1e-9


def test_visibility_is_the_rule_itself():
    for size in (1, 2, 5, 30, 40):
        chunk, window = nulunex.chunk_visible(np.arange(30), np.arange(30), size), nulunex.window_visible(np.arange(30), np.arange(30), size)
        for i in range(30):
            for j in range(30):
                assert chunk[i, j] == (j <= i and j >= i - i % size), (i, j, size)
                assert window[i, j] == (i - size < j <= i), (i, j, size)


def test_sink_is_one_more_key_without_a_value():
    rs = np.random.default_rng(0)
    s = rs.standard_normal((4, 7)) * 3
    s[1, 3:] = -np.inf
    for sink in (0.0, -2.5, 40.0):
        full = np.exp(np.concatenate([s, np.full((4, 1), sink)], axis=1))
        assert np.allclose(nulunex.softmax_with_sink(s, sink), (full / full.sum(1, keepdims=True))[:, :-1])


def test_rotations_keep_relative_positions_and_the_tail_and_differ_by_a_permutation():
    rs = np.random.default_rng(4)
    x, y = rs.standard_normal((1, 1, 12)), rs.standard_normal((1, 1, 12))
    for rotate in (nulunex.rotate_halves, nulunex.rotate_neighbours):
        a = [float((rotate(x, [p + 7], 8, 900.0) * rotate(y, [p], 8, 900.0)).sum()) for p in (0, 5, 400)]
        assert np.ptp(a) < 1e-9 and (rotate(x, [9], 8, 900.0)[..., 8:] == x[..., 8:]).all()
        assert np.isclose((rotate(x, [9], 8, 900.0) ** 2).sum(), (x ** 2).sum())
    order = [0, 2, 4, 6, 1, 3, 5, 7]  # neighbours put into halves
    assert np.allclose(nulunex.rotate_neighbours(x[..., :8], [5], 8, 900.0)[..., order], nulunex.rotate_halves(x[..., :8][..., order], [5], 8, 900.0))


def test_clamped_unit():
    g, u = np.array([-3.0, 0.5, 2.0, 9.0]), np.array([-4.0, 0.25, 1.0, 4.0])
    want = [-3.0 / (1 + np.exp(1.702 * 3.0)) * (1 - 1.5), 0.5 / (1 + np.exp(-0.851)) * 1.25, 1.5 / (1 + np.exp(-1.702 * 1.5)) * 2.0,
            1.5 / (1 + np.exp(-1.702 * 1.5)) * 2.5]
    assert np.allclose(nulunex.clamped_glu(g, u, 1.5), want)


def test_latent_attention_is_ordinary_attention_over_projected_keys():
    """One head, one query: the score and the value written out."""
    mix = nb.latent(heads=1, dim=4, rot_dim=2, vdim=3, rank=5, window=3, ff=None)["mixer"]
    cfg = nb.config([nb.latent(heads=1, dim=4, rot_dim=2, vdim=3, rank=5, window=3, ff=None)], width=6)
    w = {k[len("l0.mix."):]: v.astype(np.float64) for k, v in nb.weights(cfg, 3).items() if k.startswith("l0.mix.")}
    x = np.random.default_rng(1).standard_normal((5, 6))
    got, _ = nulunex.latent_mixer(x, w, mix, 1e-3)
    y = x @ w["dkv"].T
    c = y[:, :5] / np.sqrt((y[:, :5] ** 2).mean(1, keepdims=True) + 1e-3) * w["dkv.norm"]
    q, p = (x @ w["q"].T)[4], []

    def turn(v, pos):
        return np.array([v[0] * np.cos(pos) - v[1] * np.sin(pos), v[1] * np.cos(pos) + v[0] * np.sin(pos)])

    for j in (2, 3, 4):
        p.append(np.exp((q[:4] @ (w["uk"] @ c[j]) + turn(q[4:], 4) @ turn(y[j, 5:], j)) * mix["scale"]))
    z = sum(p) + np.exp(w["sink"][0])
    want = w["o"] @ sum(e / z * (w["uv"] @ c[j]) for e, j in zip(p, (2, 3, 4)))
    assert np.allclose(got[4], want)


# ------------------------------------------------------------------------------------------ product, host side
@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_configuration_and_weights_round_trip(name, tmp_path):
    from recurrent_drafting import configuration_nulunex, registry

    cfg = nb.CONFIGS[name]
    c = configuration_nulunex.NulunexConfig.from_dict(cfg)
    assert c.to_dict() == cfg and c.num_hidden_layers == len(cfg["layers"]) and c.vocab_size == cfg["vocab"]
    w = nb.weights(cfg, 6)
    llm = nb.build(cfg, w, torch.float32, device="cpu")
    back = llm.checkpoint_state_dict()
    assert set(back) == set(w) and all(np.array_equal(back[k].numpy(), w[k]) for k in w)
    llm.save_pretrained(str(tmp_path))
    assert json.loads((tmp_path / "config.json").read_text()) == cfg
    again = registry.load_model(str(tmp_path), torch.float32, device="cpu")
    assert type(again).__name__ == "NulunexForCausalLM"
    assert all(torch.equal(a, b) for a, b in zip(again.checkpoint_state_dict().values(), back.values()))
    own = nb.build(cfg, w, torch.float32, device="cpu")
    own.init_random(seed=3)
    own.load_state_dict(llm.state_dict())  # the module's own layout
    assert all(torch.equal(a, b) for a, b in zip(own.checkpoint_state_dict().values(), back.values()))
    with pytest.raises(KeyError):
        llm.load_state_dict({**{k: torch.from_numpy(v) for k, v in w.items()}, "l0.mix.extra": torch.zeros(1)})


def test_shared_layers_are_one_object_with_a_cache_each():
    from recurrent_drafting import configuration_nulunex, kv_cache, modeling_nulunex, registry

    a, l = nb.attention(), nb.latent()
    cfg = nb.config([nb.shared(a, 2), l, a, nb.shared(a, 0), nb.shared(l, 1)])  # also of a later layer, and of one that shares itself
    c = configuration_nulunex.NulunexConfig.from_dict(cfg)
    assert [c.owner(i) for i in range(5)] == [2, 1, 2, 2, 1]
    llm = modeling_nulunex.NulunexForCausalLM(c).to(torch.bfloat16)
    assert llm.layers[0] is llm.layers[2] is llm.layers[3] and llm.layers[1] is llm.layers[4]
    assert {n.split(".")[0] for n in llm.checkpoint_state_dict()} == {"embed", "head", "final", "l1", "l2"}
    cache = llm.new_cache(2, 50)
    assert [type(x) for x in cache.layers] == [kv_cache.LayerKeyValues, kv_cache.LayerLatents, kv_cache.LayerKeyValues, kv_cache.LayerKeyValues,
                                               kv_cache.LayerLatents]
    assert len({x.keys.data_ptr() if hasattr(x, "keys") else x.rows.data_ptr() for x in cache.layers}) == 5
    assert cache.layers[0].keys.shape == cache.layers[0].values.shape == (2, 2, 50, 32) and cache.layers[1].rows.shape == (2, 1, 50, 48)
    assert cache.bytes_per_token() == 2 * (3 * 2 * 2 * 32 + 2 * 48)
    assert "Nulunex" in registry.architectures()


def test_refusals():
    from recurrent_drafting.configuration_nulunex import NulunexConfig

    a, l = nb.attention(), nb.latent()
    for layers in ([{**a, "type": "mlstm"}], [{**a, "mlp": {"kind": "moe", "ff": 8, "limit": 1.0}}], [{**a, "mixer": {**a["mixer"], "vdim": 8}}],
                   [{**a, "mixer": {**a["mixer"], "kv_heads": 3}}], [a, nb.shared(l, 0)], [a, nb.shared(nb.attention(chunk=21), 0)],
                   [nb.shared(a, 0)], [nb.shared(a, 1), nb.shared(a, 0)], [a, nb.shared(a, 7)]):
        with pytest.raises(ValueError):
            NulunexConfig.from_dict(nb.config(layers))
