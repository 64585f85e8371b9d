"""The plain Dilavik implementation against itself and against brute force, and the parts of the product that need no
GPU: configuration, registry, weight packing, command line."""
import json

import numpy as np
import pytest
import torch

import dilavik_builders as db
from oracle import dilavik


@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_whole_sequence_equals_pieces(name):
    cfg = db.CONFIGS[name]
    w, ids = db.weights(cfg, 1), db.tokens(cfg, 90, 2)
    whole = dilavik.forward(w, cfg, ids)
    for sizes in ([1] * 90, [2, 3, 2, 30, 2, 51], [64, 26]):
        st, at, out = dilavik.State(len(cfg["layers"])), 0, []
        for n in sizes:
            out.append(dilavik.forward(w, cfg, ids[at : at + n], st))
            at += n
        assert at == 90 and np.abs(np.concatenate(out) - whole).max() < 1e-9


def test_window_visibility_is_the_rule_itself():
    for size, keep in ((1, 0), (1, 1), (5, 0), (5, 3), (4, 4), (3, 9), (40, 2)):
        vis = dilavik.window_visible(np.arange(30), np.arange(30), size, keep)
        for i in range(30):
            for j in range(30):
                assert vis[i, j] == (j <= i and (i - j < size or j < keep)), (i, j, size, keep)


def test_recurrence_equals_its_closed_form():
    """num_t = sum_j e^(F_t - F_j + i_j - m_t) (q_t . k_j) v_j with m_t from the running maximum that starts at 0."""
    rs = np.random.default_rng(3)
    T, d, dv = 25, 6, 5
    q, k, v = rs.standard_normal((T, 1, d)), rs.standard_normal((T, 1, d)), rs.standard_normal((T, 1, dv))
    i, f = 3 * rs.standard_normal((T, 1)), -np.abs(rs.standard_normal((T, 1)))
    st = dilavik.mlstm_zero_state(1, d, dv)
    F = np.cumsum(f[:, 0])
    for t in range(T):
        st, o = dilavik.mlstm_step(st, q[t], k[t], v[t], i[t], f[t])
        m = max([F[t]] + [F[t] - F[j] + i[j, 0] for j in range(t + 1)])
        assert abs(m - st[2][0]) < 1e-12
        p = np.array([np.exp(F[t] - F[j] + i[j, 0] - m) * (q[t, 0] @ k[j, 0]) for j in range(t + 1)])
        want = p @ v[: t + 1, 0] / (max(abs(p.sum()), np.exp(-m)) + 1e-6)
        assert np.abs(o[0] - want).max() < 1e-10


def test_rotation_keeps_relative_positions_and_the_tail():
    rs = np.random.default_rng(4)
    x, y = rs.standard_normal((1, 1, 12)), rs.standard_normal((1, 1, 12))
    a = [float((dilavik.partial_rotary(x, [p + 7], 8, 900.0) * dilavik.partial_rotary(y, [p], 8, 900.0)).sum()) for p in (0, 5, 400)]
    assert np.ptp(a) < 1e-9
    assert (dilavik.partial_rotary(x, [9], 8, 900.0)[..., 8:] == x[..., 8:]).all()


def test_grouped_norm_and_depth_average():
    rs = np.random.default_rng(5)
    x, w = rs.standard_normal((3, 12)), rs.standard_normal(12)
    y = dilavik.grouped_rms_norm(x, w, 3, 1e-2)
    for g in range(3):
        part = x[:, 4 * g : 4 * g + 4]
        assert np.allclose(y[:, 4 * g : 4 * g + 4], part / np.sqrt((part ** 2).sum(1, keepdims=True) / 4 + 1e-2) * w[4 * g : 4 * g + 4])
    h = [rs.standard_normal((2, 4)) for _ in range(3)]
    assert np.allclose(dilavik.depth_average([0.5, -1.0, 2.0], h), 0.5 * h[0] - h[1] + 2 * h[2])


def test_xielu_is_smooth_at_zero_and_matches_both_branches():
    p, q = 0.4, -0.9
    z = np.array([-3.0, -1e-7, 0.0, 1e-7, 2.5])
    y = dilavik.xielu(z, p, q)
    assert np.allclose(y[0], (0.5 + np.log1p(np.exp(q))) * (np.exp(-3.0) - 1 + 3.0) - 1.5)
    assert np.allclose(y[4], np.log1p(np.exp(p)) * 6.25 + 1.25)
    assert np.allclose(y[1:4], z[1:4] / 2, atol=1e-12)


# ------------------------------------------------------------------------------------------ product, host side
@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_configuration_and_weights_round_trip(name, tmp_path):
    from recurrent_drafting import configuration_dilavik, registry

    cfg = db.CONFIGS[name]
    c = configuration_dilavik.DilavikConfig.from_dict(cfg)
    assert c.to_dict() == cfg and c.num_hidden_layers == len(cfg["layers"]) and c.vocab_size == cfg["vocab"]
    w = db.weights(cfg, 6)
    llm = db.build(cfg, w, torch.float32, device="cpu")
    back = llm.checkpoint_state_dict()
    assert set(back) == set(w) and all(np.array_equal(back[k].numpy(), w[k]) for k in w)
    llm.save_pretrained(str(tmp_path))
    assert json.loads((tmp_path / "config.json").read_text()) == cfg
    again = registry.load_model(str(tmp_path), torch.float32, device="cpu")
    assert type(again).__name__ == "DilavikForCausalLM"
    assert all(torch.equal(a, b) for a, b in zip(again.checkpoint_state_dict().values(), back.values()))
    with pytest.raises(KeyError):
        llm.load_state_dict({**{k: torch.from_numpy(v) for k, v in w.items()}, "l0.mix.extra": torch.zeros(1)})


def test_registry_names_and_refusals(tmp_path):
    from recurrent_drafting import configuration_dilavik, modeling_llama, registry

    assert {"Dilavik", "LlamaForCausalLM"} <= set(registry.architectures())
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "llama"}))
    assert registry.model_class_of(str(tmp_path)) is modeling_llama.LlamaForCausalLM
    with pytest.raises(ValueError):
        registry.architecture_of({"architecture": "SomethingElse"})
    for broken in ({"type": "conv"}, {"mlp": {"kind": "moe", "ff": 8}}):
        layer = {**db.attention(), **broken}
        with pytest.raises(ValueError):
            configuration_dilavik.DilavikConfig.from_dict(db.config([layer]))
    with pytest.raises(ValueError):
        configuration_dilavik.DilavikConfig.from_dict(db.config([db.attention()], width=100, groups=3))


def test_cache_holds_what_each_layer_needs():
    from recurrent_drafting import configuration_dilavik, kv_cache, modeling_dilavik

    cfg = db.CONFIGS["mixed"]
    llm = modeling_dilavik.DilavikForCausalLM(configuration_dilavik.DilavikConfig.from_dict(cfg)).to(torch.bfloat16)
    cache = llm.new_cache(2, 50, draft_tokens=6)
    kinds = [type(l) for l in cache.layers]
    assert kinds == [kv_cache.LayerMatrixState, kv_cache.LayerKeyValues] * 2
    assert cache.layers[1].keys.shape == (2, 2, 50, 32) and cache.layers[1].values.shape == (2, 2, 50, 24)
    assert cache.layers[0].S.shape == (2, 3, 16, 40) and cache.layers[0].S.dtype == torch.float32
    assert cache.layers[0].draft_gates.shape == (6, 6) and cache.bytes_per_token() == 2 * (2 * 56 + 4 * 56)
