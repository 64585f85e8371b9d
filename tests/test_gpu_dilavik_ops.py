"""Each mechanism of the Dilavik decoder alone: the CUDA kernels against the plain implementation."""
import numpy as np
import pytest
import torch

import dilavik_builders as db
from oracle import dilavik

pytestmark = pytest.mark.gpu

_alive = []


def ptr(t):
    """Device pointer of a tensor that stays alive until the test ends."""
    from recurrent_drafting import _lib

    _alive.append(t)
    return _lib.ptr(t)


@pytest.fixture(autouse=True)
def _release():
    yield
    torch.cuda.synchronize()
    _alive.clear()


DTYPES = {"fp32": torch.float32, "bf16": torch.bfloat16}


def dev(x, dtype=None):
    t = torch.from_numpy(np.ascontiguousarray(x)).cuda()
    return t if dtype is None else t.to(dtype)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def rounded(x, dtype):
    return torch.from_numpy(np.ascontiguousarray(x)).to(dtype).double().numpy()


def close(got, want, dtype, tol32=2e-5, tol16=1e-2):
    """Every element within tol of (the array's RMS + the element's own size)."""
    got = got.double().cpu().numpy()
    scale = np.sqrt((want ** 2).mean()) + 1e-30
    err = (np.abs(got - want) / (scale + np.abs(want))).max()
    assert err < (tol32 if dtype == torch.float32 else tol16), err


# ------------------------------------------------------------------------------------------ stream, norm, activation
@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("H,groups", [(128, 1), (128, 4), (60, 5), (4096, 8), (192, 64)])
def test_scaled_embedding_depth_average_and_grouped_norm(dt, H, groups):
    from recurrent_drafting import _lib

    dtype, rs = DTYPES[dt], np.random.default_rng(H + groups)
    M, n = 5, 4
    table, w = rs.standard_normal((11, H)).astype(np.float32), rs.standard_normal(H).astype(np.float32)
    ids, eps = np.array([3, 0, 10, 7, 3]), 3e-3
    hist = (rs.standard_normal((n, M, H)) * 10.0 ** rs.integers(-3, 2, (n, M, 1))).astype(np.float32)
    coeff = rs.standard_normal(n).astype(np.float32)
    t_w, code, st = dev(w, dtype), _lib.dtype_code(dtype), _lib.stream()
    w_ = rounded(w, dtype)
    x, y = torch.empty(M, H, device="cuda"), torch.empty(M, H, dtype=dtype, device="cuda")
    t_table, t_ids, t_hist, t_coeff = dev(table, dtype), dev(ids), dev(hist), dev(coeff)
    _lib.call("rd_stream_norm", code, ptr(t_table), ptr(t_ids), 2.5, None, 0, None, 0, ptr(x), ptr(t_w), ptr(y), M,
              None, H, groups, eps, st)
    want = dilavik.embed(rounded(table, dtype), ids, 2.5)
    close(x, want, torch.float32)
    close(y, dilavik.grouped_rms_norm(want, w_, groups, eps), dtype)
    _lib.call("rd_stream_norm", code, None, None, 0.0, ptr(t_hist), M * H, ptr(t_coeff), n, ptr(x), ptr(t_w), ptr(y),
              M, None, H, groups, eps, st)
    want = dilavik.depth_average(coeff.astype(np.float64), hist.astype(np.float64))
    close(x, want, torch.float32)
    close(y, dilavik.grouped_rms_norm(want, w_, groups, eps), dtype)
    _lib.call("rd_stream_norm", code, None, None, 0.0, ptr(t_hist[1]), M * H, None, 1, None, ptr(t_w), ptr(y), M, None, H, groups,
              eps, st)
    close(y, dilavik.grouped_rms_norm(hist[1].astype(np.float64), w_, groups, eps), dtype)


@pytest.mark.parametrize("dt,M,N,K", [("fp32", 7, 50, 60), ("bf16", 7, 50, 60), ("bf16", 130, 320, 128), ("bf16", 9, 96, 72), ("bf16", 300, 512, 200)])
def test_linear_layers_with_xielu_and_with_unrounded_features(dt, M, N, K):
    from recurrent_drafting import modeling_common

    dtype, rs = DTYPES[dt], np.random.default_rng(M + N)
    a, w = rs.standard_normal((M, K)).astype(np.float32), (rs.standard_normal((N, K)) / np.sqrt(K)).astype(np.float32)
    z = rounded(a, dtype) @ rounded(w, dtype).T
    lin = modeling_common.Linear(dev(w, dtype))
    c = torch.empty(M, (N + 7) // 8 * 8, dtype=dtype, device="cuda")
    p, q = 0.3, -0.8
    lin.xielu(dev(a, dtype), c, float(dilavik.softplus(p)), float(0.5 + dilavik.softplus(q)))
    close(c[:, :N], dilavik.xielu(z, p, q), dtype)
    hi = torch.zeros(M, N - 32, device="cuda")
    lin.split(dev(a, dtype), c, hi, 32)
    close(c[:, :32], z[:, :32], dtype)
    close(hi, z[:, 32:], torch.float32)  # products of bf16 values, accumulated and stored in fp32


# ------------------------------------------------------------------------------------------ attention
def run_attention(mix, rows, dtype, tree=None, boost=None):
    """rows: (cached, new) tokens of every batch row.  Random q, k, v, gates through rd_rotary_append and
    rd_attention_window; returns (got [M, H, dv] list per row, the same from the plain implementation).
    boost: (row, query token, key token, factor): the key is set to factor times the query of its head group, so that
    its score stands out."""
    from recurrent_drafting import _lib, mixers

    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    size, keep, rot, base = mix["mask"]["size"], mix["mask"]["keep_first"], mix["rot"]["dims"], mix["rot"]["base"]
    rs = np.random.default_rng(sum(a * 7 + b for a, b in rows) + size)
    B, max_len = len(rows), max(a + b for a, b in rows) + 3
    begin = [b % 2 for b in range(B)]  # a row need not start at slot 0
    max_len += 1
    kc = torch.full((B, G, max_len, d), 7.0, dtype=dtype, device="cuda")
    vc = torch.full((B, G, max_len, dv), 7.0, dtype=dtype, device="cuda")
    code, st = _lib.dtype_code(dtype), _lib.stream()
    cos, sin = mixers.RotaryTables().get(rot, base, max_len + 8, "cuda")
    data = []
    for r, (cached, new) in enumerate(rows):
        T = cached + new
        q, k, v, g = (rounded(rs.standard_normal((T, n)) * s, dtype) for n, s in ((H * d, 1.5), (G * d, 1.5), (G * dv, 1.0), (H, 1.0)))
        pos = np.arange(T)
        if tree is not None:
            pos[cached:] = cached + tree[r][1]
        if boost is not None and boost[0] == r:
            _, qi, kj, f = boost
            # undo the rotation of the distance, so that the rotated score is f |q|^2 whatever the positions
            turned = dilavik.partial_rotary(q[qi].reshape(1, H, d), [pos[qi] - pos[kj]], rot, base) if rot else q[qi].reshape(1, H, d)
            k[kj] = rounded((f * turned[0, :: H // G]).reshape(-1), dtype)
        data.append((q, k, v, g, pos))

    width = (H + G) * d + G * dv + H
    ld = (width + 7) // 8 * 8

    def append(pick):
        """rotary + append for the picked tokens of every row; returns the projection buffer."""
        parts = [np.concatenate([x[pick(*rows[r])] for x in data[r][:4]], axis=1) for r in range(B)]
        flat = np.concatenate(parts)
        proj = torch.zeros(len(flat), ld, dtype=dtype, device="cuda")
        proj[:, :width] = dev(flat, dtype)
        tok_row = i32([r for r in range(B) for _ in range(len(parts[r]))])
        posn = np.concatenate([data[r][4][pick(*rows[r])] for r in range(B)])
        slot = np.concatenate([np.arange(sum(rows[r]))[pick(*rows[r])] + begin[r] for r in range(B)])
        if len(flat):
            _lib.call("rd_rotary_append", code, ptr(proj), ld, ptr(kc), ptr(vc), ptr(tok_row), ptr(i32(posn.tolist())),
                      ptr(i32(slot.tolist())), ptr(cos), ptr(sin), max_len + 8, len(flat), None, H, G, d, dv, rot, max_len, st)
            torch.cuda.synchronize()
        return proj, i32(posn.tolist())

    append(lambda c, n: slice(0, c))
    proj, tok_pos = append(lambda c, n: slice(c, c + n))
    M = proj.shape[0]
    out = torch.full((M, H * dv), 9.0, dtype=dtype, device="cuda")
    starts = np.concatenate([[0], np.cumsum([n for _, n in rows])])
    mode, mask, words = (_lib.ATTN_CAUSAL, None, 0)
    if tree is not None:
        mode, words = _lib.ATTN_TREE, (max(n for _, n in rows) + 31) // 32
        bits = np.zeros((M, words), dtype=np.uint32)
        for r in range(B):
            for i, row in enumerate(tree[r][0]):
                for j in np.nonzero(row)[0]:
                    bits[starts[r] + i, j >> 5] |= np.uint32(1) << np.uint32(j & 31)
        mask = dev(bits.view(np.int32))
    gate = proj[:, (H + G) * d + G * dv :]
    _lib.call("rd_attention_window", code, ptr(proj), ld, ptr(kc), ptr(vc), ptr(gate), ld, ptr(out), ptr(i32(starts.tolist())),
              ptr(i32(begin)), ptr(i32([c for c, _ in rows])), B, H, G, d, dv, max_len, max(n for _, n in rows), mode, ptr(tok_pos),
              ptr(mask), words, mix["scale"], size, keep, max_len, st)
    got = out.double().cpu().numpy().reshape(M, H, dv)
    res = []
    for r, (cached, new) in enumerate(rows):
        q, k, v, g, pos = data[r]
        T = cached + new
        if new == 0:
            continue
        qr = rounded(dilavik.partial_rotary(q.reshape(T, H, d), pos, rot, base) if rot else q.reshape(T, H, d), dtype)
        kr = rounded(dilavik.partial_rotary(k.reshape(T, G, d), pos, rot, base) if rot else k.reshape(T, G, d), dtype)
        vis = dilavik.window_visible(pos[cached:], pos, size, keep)
        if tree is not None:
            vis[:, cached:] &= tree[r][0].astype(bool)
        want = dilavik.softmax_attention(qr[cached:], kr, v.reshape(T, G, dv), vis, mix["scale"]) * dilavik.sigmoid(g[cached:])[:, :, None]
        res.append((got[starts[r] : starts[r + 1]], want))
    return res


def check_attention(res, dtype):
    for got, want in res:
        assert np.abs(got - want).max() < (3e-5 if dtype == torch.float32 else 3e-2), np.abs(got - want).max()


SIZES = [(32, 24, 16, 4, 2), (64, 56, 24, 6, 2), (128, 128, 128, 4, 1), (128, 64, 20, 2, 2), (40, 120, 40, 3, 1), (200, 256, 64, 2, 1),
         (10, 14, 6, 3, 3), (12, 5, 0, 6, 2)]


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("d,dv,rot,H,G", SIZES)
@pytest.mark.parametrize("window,keep", [(1, 0), (20, 3), (64, 64), (65, 0), (500, 2)])
def test_window_attention(dt, d, dv, rot, H, G, window, keep):
    mix = db.attention(H, G, d, dv, rot, 3000.0, 1.3 / np.sqrt(d), window, keep)["mixer"]
    for rows in ([(0, 150), (0, 1), (37, 70)], [(300, 1), (5, 1), (0, 1)], [(129, 2), (64, 3), (0, 0)]):
        check_attention(run_attention(mix, rows, DTYPES[dt]), DTYPES[dt])


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("cached,new", [(0, 200), (140, 60), (199, 1), (196, 4)])
@pytest.mark.parametrize("window,keep", [(50, 4), (64, 0), (63, 2)])
def test_one_key_at_every_edge_of_the_window(dt, cached, new, window, keep):
    """A key that outweighs all others sits just inside or just outside the window, or among or behind the kept tokens:
    the output is its value, or is not moved by it."""
    mix = db.attention(4, 2, 64, 56, 24, 3000.0, 0.125, window, keep)["mixer"]
    q = 199
    for key in (q - window + 1, q - window, q - window - 1, 0, max(keep - 1, 0), keep, keep + 1, 64, 63, 128, q, q - 1):
        res = run_attention(mix, [(cached, new)], DTYPES[dt], boost=(0, q, key, 4.0))
        check_attention(res, DTYPES[dt])


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("d,dv,H,G", [(32, 24, 4, 2), (128, 128, 4, 1), (10, 14, 3, 3)])
@pytest.mark.parametrize("window,keep,cached", [(3, 0, 40), (1, 4, 2), (30, 5, 100), (2, 6, 3)])
def test_window_attention_over_a_draft_tree(dt, d, dv, H, G, window, keep, cached):
    parent = [-1, 0, 0, 1, 1, 2, 5, 3, 0, 8]
    anc, depth = np.zeros((10, 10), dtype=np.uint8), np.zeros(10, dtype=np.int64)
    for i, p in enumerate(parent):
        anc[i] = anc[p] if p >= 0 else 0
        anc[i, i] = 1
        depth[i] = depth[p] + 1 if p >= 0 else 0
    mix = db.attention(H, G, d, dv, 8 if d > 10 else 6, 3000.0, 1.3 / np.sqrt(d), window, keep)["mixer"]
    rows = [(cached, 10), (0, 10), (cached + 1, 10)]
    check_attention(run_attention(mix, rows, DTYPES[dt], tree=[(anc, depth)] * 3), DTYPES[dt])


# ------------------------------------------------------------------------------------------ matrix memory
def mlstm_inputs(mix, T, dtype, seed, extreme=False):
    rs = np.random.default_rng(seed)
    H, d, dv = mix["heads"], mix["dim"], mix["vdim"]
    q, k, v, g = (rounded(rs.standard_normal((T, n)), dtype) for n in (H * d, H * d, H * dv, H * dv))
    zi, zf = rs.standard_normal((T, H)) * (8 if extreme else 2), rs.standard_normal((T, H)) * (8 if extreme else 2)
    return q, k, v, g, zi.astype(np.float32).astype(np.float64), zf.astype(np.float32).astype(np.float64)


class Memory:
    """The recurrence of several rows on the device, fed in portions by a chosen kernel, and the plain one beside it."""

    def __init__(self, mix, B, dtype, seed=0):
        rs = np.random.default_rng(seed)
        self.mix, self.B, self.dtype = mix, B, dtype
        H, d, dv = mix["heads"], mix["dim"], mix["vdim"]
        self.bias = rs.standard_normal((2, H)).astype(np.float32) + np.array([[0.0], [3.0]], np.float32)
        self.norm = rs.standard_normal(H * dv).astype(np.float32)
        # garbage: a row of length 0 must not see it
        self.S, self.n, self.m = (torch.full(s, 5.0, device="cuda") for s in ((B, H, d, dv), (B, H, d), (B, H)))
        self.state = [dilavik.mlstm_zero_state(H, d, dv) for _ in range(B)]
        self.length = [0] * B
        self.eps = 1e-3

    def plain(self, r, data, upto=None):
        q, k, v, g, zi, zf = data
        m, T = self.mix, len(q)
        H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
        i = cap * np.tanh((zi + self.bias[0]) / cap)
        f = dilavik.log_sigmoid(cap * np.tanh((zf + self.bias[1]) / cap))
        st, o = self.state[r], np.zeros((T, H, dv))
        for t in range(T):
            st, o[t] = dilavik.mlstm_step(st, q[t].reshape(H, d) * d ** -0.5, k[t].reshape(H, d), v[t].reshape(H, dv), i[t], f[t])
        return st, dilavik.rms(o, self.eps).reshape(T, H * dv) * rounded(self.norm, self.dtype) * dilavik.sigmoid(g)

    def pack(self, portions):
        m = self.mix
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        width = 2 * H * (d + dv)
        ld = (width + 7) // 8 * 8
        M = sum(len(p[0]) for p in portions)
        proj = torch.zeros(M, ld, dtype=self.dtype, device="cuda")
        proj[:, :width] = dev(np.concatenate([np.concatenate(p[:4], axis=1) for p in portions]), self.dtype)
        gates = dev(np.concatenate([np.concatenate(p[4:], axis=1) for p in portions]).astype(np.float32))
        starts = np.concatenate([[0], np.cumsum([len(p[0]) for p in portions])])
        self.t_bias, self.t_norm = dev(self.bias), dev(self.norm, self.dtype)
        out = torch.full((M, H * dv), 9.0, dtype=self.dtype, device="cuda")
        return proj, gates, starts, out

    def args(self, _lib, proj, gates, starts, out):
        m = self.mix
        keep = (i32(starts.tolist()), i32(self.length))
        return keep, (ptr(proj), proj.stride(0), ptr(gates), gates.stride(0), ptr(self.t_bias[0]), ptr(self.t_bias[1]), m["gate_cap"],
                      ptr(self.t_norm), self.eps, ptr(out), ptr(self.S), ptr(self.n), ptr(self.m), ptr(keep[0]),
                      ptr(keep[1]), self.B, m["heads"], m["dim"], m["vdim"])

    def feed(self, portions, kernel):
        from recurrent_drafting import _lib

        m = self.mix
        proj, gates, starts, out = self.pack(portions)
        M, st = proj.shape[0], _lib.stream()
        keep, common = self.args(_lib, proj, gates, starts, out)
        if kernel == "scan":
            _lib.call("rd_mlstm_scan", _lib.dtype_code(self.dtype), *common, max(len(p[0]) for p in portions), None, 0, 0, None, None, st)
        else:
            need = _lib.load().rd_mlstm_chunk_workspace_bytes(M, self.B, m["heads"], m["dim"], m["vdim"])
            ws, status = torch.empty(need, dtype=torch.uint8, device="cuda"), i32([0])
            _lib.call("rd_mlstm_chunk", *common, M, max(len(p[0]) for p in portions), ptr(ws), need, ptr(status), st)
            assert int(status.item()) == 0
        for r in range(self.B):
            if len(portions[r][0]):
                self.state[r], want = self.plain(r, portions[r])
                self.length[r] += len(portions[r][0])
                close(out[starts[r] : starts[r + 1]], want, self.dtype, 1e-4, 4e-2)
        self.check_state()

    def check_state(self):
        for r in range(self.B):
            if self.length[r]:
                for got, want in zip((self.S[r], self.n[r], self.m[r]), self.state[r]):
                    close(got, want, torch.float32, 2e-4)


MEMORY_SIZES = [(2, 32, 72), (1, 256, 96), (3, 16, 40), (2, 64, 32), (1, 128, 200), (2, 72, 8), (1, 200, 512)]


@pytest.mark.parametrize("dt,kernel", [("fp32", "scan"), ("bf16", "scan"), ("bf16", "chunk")])
@pytest.mark.parametrize("heads,d,dv", MEMORY_SIZES)
def test_matrix_memory_in_portions(dt, kernel, heads, d, dv):
    mix = db.mlstm(heads, d, dv, 5.0)["mixer"]
    mem = Memory(mix, 3, DTYPES[dt])
    seed = 0
    for counts in ((70, 1, 128), (2, 0, 127), (1, 260, 2), (65, 129, 0)):
        seed += 1
        mem.feed([mlstm_inputs(mix, n, mem.dtype, 100 * seed + r) for r, n in enumerate(counts)], kernel)
    # rows 0 and 2 are given back: their next tokens start from zero, row 1 goes on
    for r in (0, 2):
        mem.length[r] = 0
        mem.state[r] = dilavik.mlstm_zero_state(heads, d, dv)
    mem.feed([mlstm_inputs(mix, n, mem.dtype, 900 + n) for n in (5, 9, 70)], kernel)


@pytest.mark.parametrize("heads,d,dv", [(2, 5, 7), (1, 30, 66), (2, 6, 500)])
def test_matrix_memory_of_any_size(heads, d, dv):
    mix = db.mlstm(heads, d, dv, 5.0)["mixer"]
    for dtype in DTYPES.values():
        mem = Memory(mix, 2, dtype)
        mem.feed([mlstm_inputs(mix, n, dtype, n) for n in (17, 1)], "scan")
        mem.feed([mlstm_inputs(mix, n, dtype, n) for n in (1, 6)], "scan")


@pytest.mark.parametrize("dt,kernel", [("fp32", "scan"), ("bf16", "chunk")])
def test_matrix_memory_with_gates_wide_open_and_shut(dt, kernel):
    """Input gates up to e^15 and forget gates near 0 and near 1: the running maximum carries the scale."""
    mix = db.mlstm(2, 32, 32, 15.0)["mixer"]
    mem = Memory(mix, 2, DTYPES[dt])
    for k in range(3):
        mem.feed([mlstm_inputs(mix, n, mem.dtype, 31 * k + n, extreme=True) for n in (90, 64)], kernel)


def test_matrix_memory_of_many_unequal_rows():
    mix = db.mlstm(8, 16, 64, 5.0)["mixer"]
    mem = Memory(mix, 20, torch.bfloat16)
    mem.feed([mlstm_inputs(mix, 20 + 5 * r, mem.dtype, r) for r in range(20)], "chunk")
    mem.feed([mlstm_inputs(mix, 3 * r, mem.dtype, 50 + r) for r in range(20)], "chunk")


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("heads,d,dv", [(2, 24, 64), (1, 256, 96), (2, 6, 10)])
def test_matrix_memory_over_a_draft_tree_and_its_commit(dt, heads, d, dv):
    from recurrent_drafting import _lib

    dtype = DTYPES[dt]
    mix = db.mlstm(heads, d, dv, 5.0)["mixer"]
    mem = Memory(mix, 2, dtype)
    mem.feed([mlstm_inputs(mix, n, dtype, n) for n in (21, 40)], "scan")
    # row r: packed tokens, parents before children
    parents = [[-1, 0, 0, 1, 3, 2], [-1, 0, 1, 1, 2, 0, 5, 6]]
    portions = [mlstm_inputs(mix, len(p), dtype, 70 + i) for i, p in enumerate(parents)]
    paths = []
    for p in parents:
        mine = []
        for i in range(len(p)):
            mine.append((mine[p[i]] if p[i] >= 0 else []) + [i])
        paths.append(mine)
    proj, gates, starts, out = mem.pack(portions)
    keep, common = mem.args(_lib, proj, gates, starts, out)
    bits = np.zeros((len(proj), 1), dtype=np.uint32)
    for r in range(2):
        for i, path in enumerate(paths[r]):
            bits[starts[r] + i, 0] = sum(1 << j for j in path)
    M, ws, mask, st = len(proj), torch.empty(len(proj) * heads * dv, device="cuda"), dev(bits.view(np.int32)), _lib.stream()
    _lib.call("rd_mlstm_tree", _lib.dtype_code(dtype), *common, M, ptr(mask), 1, ptr(ws), ws.numel() * 4, st)
    for r in range(2):
        for i, path in enumerate(paths[r]):
            _, want = mem.plain(r, tuple(x[path] for x in portions[r]))
            close(out[starts[r] + i], want[-1], dtype, 1e-4, 4e-2)
    mem.check_state()  # verification left the states alone
    # commit: beam `seq` of two, its first count + 1 tokens
    Lb = 4
    unpacker = i32([[paths[0][4][:4], [0, 2, 5, 5]], [[0, 1, 2, 4], [0, 5, 6, 7]]])
    seq, count = [0, 1], [3, 1]
    _lib.call("rd_mlstm_scan", _lib.dtype_code(dtype), *common, Lb, ptr(unpacker), 2, Lb, ptr(i32(seq)), ptr(i32(count)), st)
    for r in range(2):
        path = unpacker[r, seq[r], : count[r] + 1].tolist()
        mem.state[r], _ = mem.plain(r, tuple(x[path] for x in portions[r]))
    mem.check_state()


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
def test_cache_rows_of_an_accepted_path(dt):
    from recurrent_drafting import _lib

    dtype, rs = DTYPES[dt], np.random.default_rng(0)
    B, G, L, d = 2, 3, 20, 10
    plane = rs.standard_normal((B, G, L, d)).astype(np.float32)
    t = dev(plane, dtype)
    want = t.clone()
    begin, base, n, seq = [0, 2], [5, 9], [3, 0], [1, 0]
    unp = [[[0, 1, 2, 3], [0, 2, 4, 7]], [[0, 3, 5, 6], [0, 1, 2, 3]]]
    for b in range(B):
        for j in range(n[b] + 1):
            want[b, :, begin[b] + base[b] + j] = dev(plane, dtype)[b, :, begin[b] + base[b] + unp[b][seq[b]][j]]
    _lib.call("rd_cache_commit", _lib.dtype_code(dtype), ptr(t), B, G, L, d, ptr(i32(begin)), ptr(i32(base)), ptr(i32(unp)), 2, 4,
              ptr(i32(n)), ptr(i32(seq)), _lib.stream())
    assert torch.equal(t, want)
