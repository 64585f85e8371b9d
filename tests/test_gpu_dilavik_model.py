"""The Dilavik decoder in the framework: prefill, decoding, portions, batches and generation against the plain
implementation, through the session, the decode loops and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import dilavik_builders as db
from oracle import dilavik

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}
TOL = {"fp32": 3e-5, "bf16": 6e-2}


def pair(name, dt, seed=0):
    """(configuration, weights the model holds, model)."""
    cfg = db.CONFIGS[name] if isinstance(name, str) else name
    w = db.weights(cfg, seed)
    return cfg, (db.bf16(w) if dt == "bf16" else w), db.build(cfg, w, DTYPES[dt])


def run(session, portions):
    """portions: token array per row (may be empty).  Logits of all of them, per row."""
    flat = np.concatenate([np.asarray(p, dtype=np.int64) for p in portions])
    hidden = session.extend(torch.from_numpy(flat).cuda(), [len(p) for p in portions])
    logits = session.logits(hidden[: len(flat)]).double().cpu().numpy()
    session.check()
    out, at = [], 0
    for p in portions:
        out.append(logits[at : at + len(p)])
        at += len(p)
    return out


def feed(session, row, ids, sizes):
    """One row's tokens in portions; the logits of all of them."""
    out, at = [], 0
    for n in sizes:
        portions = [[] for _ in range(session.batch)]
        portions[row] = ids[at : at + n]
        out.append(run(session, portions)[row])
        at += n
    assert at == len(ids)
    return np.concatenate(out)


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_prompt_and_every_layer(name, dt):
    from recurrent_drafting import _lib
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = db.tokens(cfg, 140, 1)
    layers = []
    want = dilavik.forward(w, cfg, ids, layer_outputs=layers)
    s = Session(llm, 1, 160)
    got_layers, plain = [], llm.backbone
    llm.backbone = lambda *a, **k: plain(*a, layer_outputs=got_layers, **k)
    got = run(s, [ids])[0]
    for i, (a, b) in enumerate(zip(got_layers, layers)):
        err = np.abs(a.cpu().numpy() - b).max() / np.abs(b).max()
        assert err < (1e-5 if dt == "fp32" else 4e-2), (i, err)
    assert len(got_layers) == len(layers) and db.error(got, want) < TOL[dt]
    assert _lib.launches > 0


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_portions_down_to_single_tokens_equal_the_prompt(name, dt):
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = db.tokens(cfg, 150, 2)
    want = dilavik.forward(w, cfg, ids)
    s = Session(llm, 2, 160)
    for k, sizes in enumerate(([110] + [1] * 40, [2, 3, 2, 60, 2, 64, 17], [64, 64, 22], [1] * 30 + [120], [33] * 4 + [18])):
        got = feed(s, k % 2, ids, sizes)
        assert db.error(got, want) < TOL[dt], sizes
        s.release(k % 2)  # the next round starts a new sequence in the same slots


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_unequal_rows_together_equal_each_alone(name, dt):
    from recurrent_drafting.session import Session

    cfg, w, llm = pair(name, dt)
    ids = [db.tokens(cfg, n, 10 + n) for n in (100, 37, 3, 71)]
    want = [dilavik.forward(w, cfg, x) for x in ids]
    s = Session(llm, 4, 128)
    rounds = [(60, 1, 2, 0), (1, 30, 1, 70), (0, 5, 0, 1), (39, 1, 0, 0)]
    at, got = [0] * 4, [[] for _ in range(4)]
    for counts in rounds:
        for r, part in enumerate(run(s, [ids[r][at[r] : at[r] + counts[r]] for r in range(4)])):
            got[r].append(part)
            at[r] += counts[r]
    assert at == [len(x) for x in ids]
    for r in range(4):
        assert db.error(np.concatenate(got[r]), want[r]) < TOL[dt], r
    # rows given back and used again while the others go on
    s.release(1)
    s.release(3)
    again = [db.tokens(cfg, n, 50 + n) for n in (20, 66, 9, 12)]
    parts = run(s, again)
    for r in range(4):
        whole = np.concatenate([ids[r], again[r]]) if r in (0, 2) else again[r]
        assert db.error(parts[r], dilavik.forward(w, cfg, whole)[-len(again[r]) :]) < TOL[dt], r


def test_a_row_that_would_outgrow_the_cache_is_refused():
    from recurrent_drafting import _lib
    from recurrent_drafting.session import Session

    cfg, w, llm = pair("odd", "fp32")
    s = Session(llm, 1, 16)
    run(s, [db.tokens(cfg, 10, 0)])
    with pytest.raises(_lib.RedrafterError):
        run(s, [db.tokens(cfg, 7, 0)])


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("decode", [False, True])
def test_edges_of_the_window_and_the_first_tokens_move_the_logits(dt, decode):
    """Changing one token far back changes a position's logits exactly when the plain model says so: one attention
    layer only, so that nothing else carries the token over."""
    from recurrent_drafting.session import Session

    keep, size, T = 3, 40, 130
    cfg = db.config([db.attention(4, 2, 32, 24, 16, 5000.0, 0.05, size, keep, ff=None)], vocab=64)
    cfg, w, llm = pair(cfg, dt)
    ids = db.tokens(cfg, T, 3)
    q = T - 1
    s = Session(llm, 1, 140)
    sizes = [T - 20] + [1] * 20 if decode else [T]
    base = feed(s, 0, ids, sizes)[q]
    for j in (0, keep - 1, keep, keep + 1, q - size - 1, q - size, q - size + 1, q - 1, 64, 63):
        other = ids.copy()
        other[j] = 3 + (ids[j] - 3 + 17) % 60
        s.release(0)
        moved = np.abs(feed(s, 0, other, sizes)[q] - base).max()
        expect = np.abs(dilavik.forward(w, cfg, other)[q] - dilavik.forward(w, cfg, ids)[q]).max()
        seen = j < keep or q - j < size
        assert (expect > 1e-9) == seen
        assert expect == 0 or expect > 0.02
        assert (moved > 0) == seen, (j, moved)
        assert abs(moved - expect) < (1e-3 if dt == "fp32" else 0.5) * expect + 1e-9


def test_long_decoding_stays_on_the_plain_recurrence():
    from recurrent_drafting.session import Session

    cfg, w, llm = pair("mixed", "fp32")
    ids = db.tokens(cfg, 700, 4)
    got = feed(Session(llm, 1, 700), 0, ids, [100] + [1] * 600)
    assert db.error(got, dilavik.forward(w, cfg, ids)) < 3e-5
    cfg, w, llm = pair("mixed", "bf16")
    got = feed(Session(llm, 1, 700), 0, ids, [100] + [1] * 600)
    assert db.error(got, dilavik.forward(w, cfg, ids)) < 1.5 * TOL["bf16"]  # the worst of 700 positions


# ------------------------------------------------------------------------------------------ generation
def padded(prompts):
    n = max(len(p) for p in prompts)
    return torch.from_numpy(np.stack([np.concatenate([np.zeros(n - len(p), np.int64), p]) for p in prompts])).cuda()


def greedy(w, cfg, prompt, n):
    st, ids = dilavik.State(len(cfg["layers"])), list(prompt)
    logits = dilavik.forward(w, cfg, prompt, st)[-1]
    for _ in range(n):
        ids.append(int(np.argmax(logits)))
        logits = dilavik.forward(w, cfg, ids[-1:], st)[-1]
    return ids


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", sorted(db.CONFIGS))
def test_greedy_generation_of_a_padded_batch(name, graphs):
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "fp32")
    prompts = [db.tokens(cfg, n, 20 + n) for n in (21, 5, 40)]
    L = 40 + 30
    outs = list(rd.autoregressive.generate(llm, padded(prompts), L, rd.SpecialTokens(0, None), cuda_graphs=graphs))
    assert [o.shape[1] for o in outs] == list(range(41, L + 1))
    for r, p in enumerate(prompts):
        assert outs[-1][r, 40 - len(p) :].tolist() == greedy(w, cfg, p, 30), r


def test_graphs_and_ordinary_launches_agree_in_bf16_and_sampling_draws_from_the_model():
    import recurrent_drafting as rd

    cfg, w, llm = pair("wide", "bf16")
    batch = padded([db.tokens(cfg, n, n) for n in (30, 12)])
    runs = [torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 60, rd.SpecialTokens(0, None), cuda_graphs=g)])
            for g in (False, True)]
    assert torch.equal(runs[0], runs[1])
    # a cold distribution is the arg-max
    torch.manual_seed(1)
    cold = torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 60, rd.SpecialTokens(0, None), rd.SamplingArgs(1e-4, False))])
    assert torch.equal(cold, runs[0])
    warm = []
    for g in (False, True):
        torch.manual_seed(7)
        warm.append(torch.stack([o[:, -1] for o in rd.autoregressive.generate(llm, batch, 60, rd.SpecialTokens(0, None), rd.SamplingArgs(2.0, False),
                                                                              cuda_graphs=g)]))
    assert torch.equal(warm[0], warm[1]) and not torch.equal(warm[0], runs[0])


def drafted(llm, cfg, dtype, seed=5):
    import recurrent_drafting as rd

    with torch.device("cuda"):
        dr = rd.modeling_drafter.Drafter(rd.configuration_drafter.DrafterConfig(
            vocab_size=cfg["vocab"], hidden_size=cfg["width"], exit_dim=2 * cfg["width"], num_draft_layers=1, rnn=True)).to(dtype)
    dr.init_random(0.05, seed=seed)
    return rd.RecurrentDrafting(llm, dr)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["mixed", "plain", "wide"])
def test_speculative_decoding_yields_the_greedy_tokens(name, graphs):
    """Draft, verify over the packed tree, accept, commit keys and recurrent states: the stream is the greedy one."""
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "fp32")
    model = drafted(llm, cfg, torch.float32)
    model.cuda_graphs = graphs
    prompts = [db.tokens(cfg, n, 20 + n) for n in (21, 5, 40)]
    last = None
    for last in model.generate(rd.stats.Ledger(), padded(prompts), 70, rd.modeling_drafter.BeamShape(4, 3), rd.SamplingArgs(1.0, True),
                               rd.SpecialTokens(0, None)):
        pass
    for r, p in enumerate(prompts):
        row = [t for t in last[r].tolist()]
        while row and row[0] == 0:
            row.pop(0)
        assert row[: len(p)] == p.tolist()
        want = greedy(w, cfg, p, len(row) - len(p))
        assert row == want, r


class PlantedDrafter(torch.nn.Module):
    """Stands in for a drafter: its beams follow the model's own greedy continuation for a while, so that paths of every
    length are accepted."""

    def __init__(self, cfg, w, prompts, width, length):
        super().__init__()
        self.cfg, self.w, self.W, self.L = cfg, w, width, length
        self.rows = [greedy(w, cfg, p, 60) for p in prompts]
        self.steps = 0

    def beam_search_sparse(self, ctx, init_tok, embeddings, beam_shape):
        B, W, L = len(self.rows), self.W, self.L
        beams = torch.zeros(B, W, L, dtype=torch.int64)
        for b in range(B):
            at = self.at[b]
            true = (self.rows[b][at : at + L] + [3] * L)[:L]
            assert int(init_tok[b]) == true[0]
            for i in range(W):
                hit = 1 + (self.steps + b) % L  # the longest right prefix of this step, in beam 1; shorter ones elsewhere
                hit = hit if i == 1 else max(1, hit - 1 - i)
                beams[b, i] = torch.tensor(true[:hit] + [3 + (7 * i + self.steps + k) % (self.cfg["vocab"] - 3) for k in range(L - hit)])
        self.steps += 1

        class Draft:
            pass

        d = Draft()
        d.beams = beams.cuda()
        return d


@pytest.mark.parametrize("name", ["mixed", "plain"])
def test_accepted_paths_of_every_length_are_committed(name):
    import recurrent_drafting as rd

    cfg, w, llm = pair(name, "fp32")
    prompts = [db.tokens(cfg, n, 20 + n) for n in (21, 5)]
    W, L = 3, 4
    planted = PlantedDrafter(cfg, w, prompts, W, L)
    planted.at = [len(p) for p in prompts]
    model = rd.RecurrentDrafting(llm, planted, cuda_graphs=False)
    accepted, last = set(), None
    for last in model.generate(rd.stats.Ledger(), padded(prompts), 60, rd.modeling_drafter.BeamShape(W, L), rd.SamplingArgs(1.0, True),
                               rd.SpecialTokens(0, None)):
        st = model.last_state
        accepted |= set(st.n_accepted.tolist())
        planted.at = st.kv_len.tolist()
    assert accepted == set(range(L)), accepted
    for r, p in enumerate(prompts):
        row = last[r].tolist()
        while row[0] == 0:
            row.pop(0)
        assert row == planted.rows[r][: len(row)], r
    # the committed states are those of the plain recurrence over the same tokens
    n = st.kv_len.tolist()
    for r in range(2):
        plain = dilavik.State(len(cfg["layers"]))
        dilavik.forward(w, cfg, planted.rows[r][: n[r]], plain)
        for layer, mine in zip(model.last_cache.layers, plain.layer):
            if hasattr(layer, "S"):
                assert np.abs(layer.S[r].cpu().numpy() - mine[0]).max() < 1e-3 * np.abs(mine[0]).max()
            else:
                keys = layer.keys[r, :, : n[r]].cpu().numpy()
                assert np.abs(keys - mine[0].transpose(1, 0, 2)).max() < 1e-3 * np.abs(mine[0]).max()


# ------------------------------------------------------------------------------------------ command lines
def test_generate_command_line(tmp_path, capsys):
    from recurrent_drafting.cmd import generate as cli

    cfg, w, llm = pair("mixed", "fp32")
    llm.save_pretrained(str(tmp_path))
    prompts = [db.tokens(cfg, n, n) for n in (9, 14)]
    (tmp_path / "prompts.txt").write_text("\n".join(" ".join(str(int(t)) for t in p) for p in prompts))
    common = ["--hf_llm", str(tmp_path), "--prompt_token_ids", str(tmp_path / "prompts.txt"), "--batch_size", "2", "--dtype", "fp32",
              "--max_prompt_length", "20", "--max_generation_length", "10", "--greedy_search"]
    assert cli.main(common + ["--autoregression"]) == 0
    rows = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    for r, p in enumerate(prompts):
        assert rows[r][14 - len(p) :] == greedy(w, cfg, p, 30 - 14)
    assert cli.main(common + ["--hf_drafter", "random:1", "--beam_width", "3", "--beam_length", "3"]) == 0
    assert "Tokens/second" in capsys.readouterr().out


def test_trace_replay(tmp_path):
    cfg, w, llm = pair("mixed", "fp32")
    llm.save_pretrained(str(tmp_path))
    out = tmp_path / "out"
    out.mkdir()
    a, b = db.tokens(cfg, 40, 1), db.tokens(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30].tolist(), "want": [29, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:].tolist(), "want": []}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "b", "tokens": b.tolist(), "want": [0, 11]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 5"]
    assert sorted(os.listdir(out)) == ["0.f32", "5.f32"]
    got = [np.fromfile(out / f, dtype="<f4").reshape(2, -1) for f in ("0.f32", "5.f32")]
    assert db.error(got[0], dilavik.forward(w, cfg, a)[[29, 3]]) < 3e-5
    assert db.error(got[1], dilavik.forward(w, cfg, b)[[0, 11]]) < 3e-5
