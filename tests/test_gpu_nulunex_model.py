"""The Nulunex decoder in the framework: prefill, decoding, portions, batches and generation against the plain
implementation, through the session, the decode loops and the command lines."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import nulunex_builders as nb
from oracle import nulunex
from session_helpers import feed, padded, run

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
TOL = {"fp32": 3e-5, "bf16": 6e-2}


def pair(name, dt, seed=0):
    """(configuration, weights the model holds, model)."""
    cfg = nb.CONFIGS[name] if isinstance(name, str) else name
    w = nb.weights(cfg, seed)
    return cfg, (nb.bf16(w) if dt == "bf16" else w), nb.build(cfg, w, DTYPES[dt])


def greedy(w, cfg, prompt, n):
    st, ids = nulunex.State(len(cfg["layers"])), list(prompt)
    logits = nulunex.forward(w, cfg, prompt, st)[-1]
    for _ in range(n):
        ids.append(int(np.argmax(logits)))
        logits = nulunex.forward(w, cfg, ids[-1:], st)[-1]
    return ids


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_prompt_and_every_layer(name, dt):
    from recurrent_drafting import _lib
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = nb.tokens(cfg, 140, 1)
    layers = []
    want = nulunex.forward(w, cfg, ids, layer_outputs=layers)
    s = Session(llm, 1, 160)
    got_layers, plain = [], llm.backbone
    llm.backbone = lambda *a, **k: plain(*a, layer_outputs=got_layers, **k)
    got = run(s, [ids])[0]
    for i, (a, b) in enumerate(zip(got_layers, layers)):
        err = np.abs(a.cpu().numpy() - b).max() / np.abs(b).max()
        assert err < (1e-5 if dt == "fp32" else 4e-2), (i, err)
    assert len(got_layers) == len(layers) and nb.error(got, want) < TOL[dt]
    assert _lib.launches > 0


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_portions_down_to_single_tokens_equal_the_prompt(name, dt):
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = nb.tokens(cfg, 150, 2)
    want = nulunex.forward(w, cfg, ids)
    s = Session(llm, 2, 160)
    for k, sizes in enumerate(([110] + [1] * 40, [2, 3, 2, 60, 2, 64, 17], [64, 64, 22], [1] * 30 + [120], [33] * 4 + [18], [32, 33, 85])):
        got = feed(s, k % 2, ids, sizes)
        assert nb.error(got, want) < TOL[dt], sizes
        s.release(k % 2)  # the next round starts a new sequence in the same slots


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_unequal_rows_together_equal_each_alone(name, dt):
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = [nb.tokens(cfg, n, 10 + n) for n in (100, 37, 3, 111)]
    want = [nulunex.forward(w, cfg, x) for x in ids]
    s = Session(llm, 4, 128)
    rounds = [(60, 1, 2, 0), (1, 30, 1, 70), (0, 5, 0, 1), (39, 1, 0, 40)]
    at, got = [0] * 4, [[] for _ in range(4)]
    for counts in rounds:
        for r, part in enumerate(run(s, [ids[r][at[r] : at[r] + counts[r]] for r in range(4)])):
            got[r].append(part)
            at[r] += counts[r]
    assert at == [len(x) for x in ids]
    for r in range(4):
        assert nb.error(np.concatenate(got[r]), want[r]) < TOL[dt], r
    # rows given back and used again while the others go on
    s.release(1)
    s.release(3)
    again = [nb.tokens(cfg, n, 50 + n) for n in (20, 66, 9, 12)]
    parts = run(s, again)
    for r in range(4):
        whole = np.concatenate([ids[r], again[r]]) if r in (0, 2) else again[r]
        assert nb.error(parts[r], nulunex.forward(w, cfg, whole)[-len(again[r]) :]) < TOL[dt], r


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("layer", ["attention", "latent", "attention128", "latent128"])
def test_edges_of_the_window_and_the_chunk_move_the_logits(dt, decode, layer):
    """Changing one token changes a position's logits exactly when the plain model says so: one mixer only, so that nothing
    else carries the token over."""
    from recurrent_drafting.session import Session

    size, T = 40, 130
    one = {"attention": nb.attention(chunk=size, scale=0.05, ff=None), "latent": nb.latent(window=size, scale=0.05, ff=None),
           "attention128": nb.attention(dim=128, rot=64, chunk=size, scale=0.02, ff=None),
           "latent128": nb.latent(dim=128, rot_dim=64, vdim=128, rank=72, window=size, scale=0.02, ff=None)}[layer]
    cfg, w, llm = pair(nb.config([one], vocab=64), dt)
    ids = nb.tokens(cfg, T, 3)
    q = 118  # not the last position of its chunk
    first = q // size * size if "attention" in layer else q - size + 1
    s = Session(llm, 1, 140)
    sizes = [T - 20] + [1] * 20 if decode else [T]
    base = feed(s, 0, ids, sizes)[q]
    for j in (0, first - 1, first, first + 1, first - 2, q - 1, q + 1, 63, 64):
        other = ids.copy()
        other[j] = 3 + (ids[j] - 3 + 17) % 60
        s.release(0)
        moved = np.abs(feed(s, 0, other, sizes)[q] - base).max()
        expect = np.abs(nulunex.forward(w, cfg, other)[q] - nulunex.forward(w, cfg, ids)[q]).max()
        seen = first <= j <= q
        assert (expect > 1e-9) == seen and (expect == 0 or expect > 0.01), (j, expect)
        assert (moved > 0) == seen, (j, moved)
        assert abs(moved - expect) < (1e-3 if dt == "fp32" else 0.5) * expect + 1e-9


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
def test_long_decoding_past_many_windows_and_chunks(dt):
    from recurrent_drafting.session import Session

    cfg, w, llm = pair("mixed", dt)
    ids = nb.tokens(cfg, 600, 4)
    got = feed(Session(llm, 1, 600), 0, ids, [100] + [1] * 500)
    # the worst of 600 positions
    assert nb.error(got, nulunex.forward(w, cfg, ids)) < (1 if dt == "fp32" else 1.5) * TOL[dt]


def test_far_positions_keep_their_angles():
    """Thousands of tokens: angles of the fast pairs have turned hundreds of times."""
    from recurrent_drafting.session import Session

    cfg = nb.config([nb.attention(chunk=300, base=20.0, ff=None), nb.latent(window=200, base=30.0, ff=None)], width=64, vocab=50)
    cfg, w, llm = pair(cfg, "fp32")
    ids = nb.tokens(cfg, 3000, 5)
    want = nulunex.forward(w, cfg, ids)[-150:]
    s = Session(llm, 1, 3000)
    assert nb.error(feed(s, 0, ids, [2850, 100] + [1] * 50)[-150:], want) < 2e-4


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", sorted(nb.CONFIGS))
def test_greedy_generation_of_a_padded_batch(name, graphs):
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "fp32")
    prompts = [nb.tokens(cfg, n, 20 + n) for n in (21, 5, 40)]
    L = 40 + 30
    outs = list(rd.autoregressive.generate(llm, padded(prompts), L, rd.SpecialTokens(0, None), cuda_graphs=graphs))
    assert [o.shape[1] for o in outs] == list(range(41, L + 1))
    for r, p in enumerate(prompts):
        assert outs[-1][r, 40 - len(p) :].tolist() == greedy(w, cfg, p, 30), r


@pytest.mark.parametrize("name", ["wide", "latents"])
def test_graphs_and_ordinary_launches_agree_in_bf16_and_sampling_draws_from_the_model(name):
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "bf16")
    batch = padded([nb.tokens(cfg, n, n) for n in (50, 12)])
    runs = [torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 80, rd.SpecialTokens(0, None), cuda_graphs=g)])
            for g in (False, True)]
    assert torch.equal(runs[0], runs[1])
    torch.manual_seed(1)  # a cold distribution is the arg-max
    cold = torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 80, rd.SpecialTokens(0, None), rd.SamplingArgs(1e-4, False))])
    assert torch.equal(cold, runs[0])
    warm = []
    for g in (False, True):
        torch.manual_seed(7)
        warm.append(torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 80, rd.SpecialTokens(0, None), rd.SamplingArgs(2.0, False),
                                                                              cuda_graphs=g)]))
    assert torch.equal(warm[0], warm[1]) and not torch.equal(warm[0], runs[0])


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_speculative_decoding_yields_the_greedy_tokens(name, graphs):
    """Draft, verify over the packed tree, accept, commit keys and latents: the stream is the greedy one."""
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "fp32")
    with torch.device("cuda"):
        drafter = rd.modeling_drafter.Drafter(rd.configuration_drafter.DrafterConfig(
            vocab_size=cfg["vocab"], hidden_size=cfg["width"], exit_dim=2 * cfg["width"], num_draft_layers=1, rnn=True)).to(torch.float32)
    model = rd.RecurrentDrafting(llm, drafter.init_random(0.05, seed=5) or drafter, cuda_graphs=graphs)
    prompts = [nb.tokens(cfg, n, 20 + n) for n in (21, 5, 40)]
    last = None
    for last in model.generate(rd.stats.Ledger(), padded(prompts), 70, rd.modeling_drafter.BeamShape(4, 3), rd.SamplingArgs(1.0, True),
                               rd.SpecialTokens(0, None)):
        pass
    for r, p in enumerate(prompts):
        row = last[r].tolist()
        while row and row[0] == 0:
            row.pop(0)
        assert row == greedy(w, cfg, p, len(row) - len(p)), r


class PlantedDrafter(torch.nn.Module):
    """Stands in for a drafter: its beams follow the model's own greedy continuation for a while, so that paths of every
    length are accepted."""

    def __init__(self, cfg, rows, width, length):
        super().__init__()
        self.cfg, self.rows, self.W, self.L, self.steps, self.at = cfg, rows, width, length, 0, []

    def beam_search_sparse(self, ctx, init_tok, embeddings, beam_shape):
        B, W, L = len(self.rows), self.W, self.L
        beams = torch.zeros(B, W, L, dtype=torch.int64)
        for b in range(B):
            true = (self.rows[b][self.at[b] : self.at[b] + L] + [3] * L)[:L]
            for i in range(W):
                hit = 1 + (self.steps + b) % L  # the longest right prefix of this step, in beam 1; shorter ones elsewhere
                hit = hit if i == 1 else max(1, hit - 1 - i)
                beams[b, i] = torch.tensor(true[:hit] + [3 + (7 * i + self.steps + k) % (self.cfg["vocab"] - 3) for k in range(L - hit)])
        self.steps += 1
        draft = type("Draft", (), {})()
        draft.beams = beams.cuda()
        return draft


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
def test_accepted_paths_of_every_length_are_committed(dt):
    import recurrent_drafting as rd

    cfg, w, llm = pair("mixed", dt)
    prompts = [nb.tokens(cfg, n, 20 + n) for n in (21, 5)]
    W, L = 3, 4
    if dt == "fp32":
        rows = [greedy(w, cfg, p, 60) for p in prompts]
    else:  # the bf16 model's own stream
        out = None
        for out in rd.autoregressive.generate(llm, padded(prompts), 21 + 60, rd.SpecialTokens(0, None)):
            pass
        rows = [out[r, 21 - len(p) :].tolist() for r, p in enumerate(prompts)]
    planted = PlantedDrafter(cfg, rows, W, L)
    planted.at = [len(p) for p in prompts]
    model = rd.RecurrentDrafting(llm, planted, cuda_graphs=False)
    accepted, last = set(), None
    for last in model.generate(rd.stats.Ledger(), padded(prompts), 60, rd.modeling_drafter.BeamShape(W, L), rd.SamplingArgs(1.0, True),
                               rd.SpecialTokens(0, None)):
        st = model.last_state
        accepted |= set(st.n_accepted.tolist())
        planted.at = st.kv_len.tolist()
    assert accepted == set(range(L)), accepted
    n = st.kv_len.tolist()
    for r in range(2):
        row = last[r].tolist()
        while row[0] == 0:
            row.pop(0)
        assert row == rows[r][: len(row)], r
        # what the cache holds is what a plain run over the same tokens leaves
        plain = nulunex.State(len(cfg["layers"]))
        nulunex.forward(w, cfg, rows[r][: n[r]], plain)
        for layer, mine in zip(model.last_cache.layers, plain.layer):
            if hasattr(layer, "rows"):
                held = [(layer.rows[r, 0, : n[r]], np.concatenate(mine, axis=1))]
            else:
                held = [(x[r, :, : n[r]].transpose(0, 1), y) for x, y in zip((layer.keys, layer.values), mine)]
            for x, y in held:
                assert np.abs(x.float().cpu().numpy() - y).max() < (1e-3 if dt == "fp32" else 0.1) * np.abs(y).max()


# ------------------------------------------------------------------------------------------ command lines
def test_generate_command_line(tmp_path, capsys):
    from recurrent_drafting.cmd import generate as cli

    cfg, w, llm = pair("mixed", "fp32")
    llm.save_pretrained(str(tmp_path))
    prompts = [nb.tokens(cfg, n, n) for n in (9, 14)]
    (tmp_path / "prompts.txt").write_text("\n".join(" ".join(str(int(t)) for t in p) for p in prompts))
    common = ["--hf_llm", str(tmp_path), "--prompt_token_ids", str(tmp_path / "prompts.txt"), "--batch_size", "2", "--dtype", "fp32",
              "--max_prompt_length", "20", "--max_generation_length", "10", "--greedy_search"]
    assert cli.main(common + ["--autoregression"]) == 0
    rows = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    for r, p in enumerate(prompts):
        assert rows[r][14 - len(p) :] == greedy(w, cfg, p, 30 - 14)
    assert cli.main(common + ["--hf_drafter", "random:1", "--beam_width", "3", "--beam_length", "3"]) == 0
    assert "Tokens/second" in capsys.readouterr().out
    assert cli.main(["--hf_llm", "random:nulunex-tiny", "--autoregression", "--greedy_search", "--max_prompt_length", "40",
                     "--max_generation_length", "20"]) == 0


def test_trace_replay(tmp_path):
    cfg, w, llm = pair("mixed", "fp32")
    llm.save_pretrained(str(tmp_path))
    out = tmp_path / "out"
    out.mkdir()
    a, b = nb.tokens(cfg, 80, 1), nb.tokens(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50].tolist(), "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:].tolist(), "want": []}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "b", "tokens": b.tolist(), "want": [0, 11]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "96"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 5"]
    got = [np.fromfile(out / f, dtype="<f4").reshape(2, -1) for f in ("0.f32", "5.f32")]
    assert nb.error(got[0], nulunex.forward(w, cfg, a)[[49, 3]]) < 3e-5
    assert nb.error(got[1], nulunex.forward(w, cfg, b)[[0, 11]]) < 3e-5
