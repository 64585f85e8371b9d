"""Each mechanism of the Nulunex decoder alone: the CUDA kernels against the plain implementation."""
import ctypes

import numpy as np
import pytest
import torch

from oracle import nulunex

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


ROTATE = {0: nulunex.rotate_halves, 1: nulunex.rotate_neighbours}


def table(rot, base, n_pos):
    from recurrent_drafting import mixers

    return mixers.RotaryTables().get(rot, base, n_pos, "cuda")


# ------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dt,M,ff,K", [("fp32", 7, 25, 60), ("bf16", 7, 25, 60), ("bf16", 130, 304, 128), ("bf16", 9, 44, 72), ("bf16", 300, 33, 200)])
@pytest.mark.parametrize("limit,alpha", [(0.4, 1.702), (50.0, 0.6)])
def test_clamped_gated_unit(dt, M, ff, K, limit, alpha):
    from recurrent_drafting import modeling_common

    dtype, rs = DTYPES[dt], np.random.default_rng(M + ff)
    a = rs.standard_normal((M, K)).astype(np.float32)
    gate, up = ((rs.standard_normal((ff, K)) / np.sqrt(K)).astype(np.float32) for _ in range(2))
    lin = modeling_common.Linear(dev(np.stack([gate, up], axis=1).reshape(2 * ff, K), dtype))
    c = torch.empty(M, (ff + 7) // 8 * 8, dtype=dtype, device="cuda")
    lin.clamped_glu(dev(a, dtype), c, limit, alpha)
    x = rounded(a, dtype)
    close(c[:, :ff], nulunex.clamped_glu(x @ rounded(gate, dtype).T, x @ rounded(up, dtype).T, limit, alpha), dtype)


# ------------------------------------------------------------------------------------------ heads: rotation, norm, append
@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("neighbours", [0, 1])
@pytest.mark.parametrize("H,G,d,dv,rot,eps", [(4, 2, 32, 0, 16, 1e-2), (3, 1, 10, 0, 10, 1e-5), (2, 2, 128, 0, 64, 3e-1), (2, 1, 40, 24, 8, 1e-3),
                                             (2, 1, 24, 0, 24, None), (3, 3, 16, 8, 0, 0.0)])
def test_rotation_head_norm_and_append(dt, neighbours, H, G, d, dv, rot, eps):
    from recurrent_drafting import _lib

    dtype, rs = DTYPES[dt], np.random.default_rng(d + H)
    M, B, max_len = 9, 3, 40
    width = (H + G) * d + G * dv
    ld = width + 3
    proj = rounded(rs.standard_normal((M, ld)) * np.exp(rs.standard_normal((M, 1))), dtype)
    pos, row, slot = rs.integers(0, 300, M), rs.integers(0, B, M), rs.permutation(max_len)[:M]
    cos, sin = table(rot, 700.0, 300)
    vd = dv or d
    kc, vc = torch.full((B, G, max_len, d), 7.0, dtype=dtype, device="cuda"), torch.full((B, G, max_len, vd), 7.0, dtype=dtype, device="cuda")
    p = dev(proj, dtype)
    _lib.call("rd_rotary_norm_append", _lib.dtype_code(dtype), ptr(p), ld, ptr(kc), ptr(vc), ptr(i32(row.tolist())), ptr(i32(pos.tolist())),
              ptr(i32(slot.tolist())), ptr(cos), ptr(sin), 300, M, None, H, G, d, dv, rot, neighbours, -1.0 if eps is None else eps, max_len,
              _lib.stream())
    heads = proj[:, : (H + G) * d].reshape(M, H + G, d)
    turned = ROTATE[neighbours](heads, pos, rot, 700.0) if rot else heads
    if eps is not None:
        turned = nulunex.unit_rms(turned, eps)
    close(p[:, : H * d], turned[:, :H].reshape(M, -1), dtype)
    assert torch.equal(p[:, width:].double().cpu(), torch.from_numpy(proj[:, width:]))
    values = proj[:, (H + G) * d : width].reshape(M, G, dv) if dv else heads[:, H:]
    touched = np.zeros((B, max_len), bool)
    for t in range(M):
        close(kc[row[t], :, slot[t]], turned[t, H:], dtype)
        close(vc[row[t], :, slot[t]], values[t], dtype)
        touched[row[t], slot[t]] = True
    for c in (kc, vc):
        assert (c.permute(0, 2, 1, 3)[torch.from_numpy(~touched).cuda()] == 7).all()


@pytest.mark.parametrize("M,H,G,rot,K", [(5, 2, 1, 64, 128), (140, 4, 2, 128, 192), (300, 3, 2, 16, 256), (33, 1, 1, 0, 64)])
def test_projection_with_rotation_head_norm_and_append_in_its_epilogue(M, H, G, rot, K):
    from recurrent_drafting import mixers, modeling_common

    rs = np.random.default_rng(M)
    B, max_len, eps = 3, 2 * M, 2e-2
    a, w = rounded(rs.standard_normal((M, K)), torch.bfloat16), rounded(rs.standard_normal(((H + G) * 128, K)) / np.sqrt(K), torch.bfloat16)
    pos, row, slot = rs.integers(0, 500, M), rs.integers(0, B, M), rs.permutation(max_len)[:M]
    cos, sin = mixers.RotaryTables().get(rot, 5e4, 500, "cuda", head=128)
    kc, vc = (torch.full((B, G, max_len, 128), 7.0, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    q, status = torch.empty(M, H * 128, dtype=torch.bfloat16, device="cuda"), i32([0])
    lin = modeling_common.Linear(dev(w, torch.bfloat16))
    meta = [i32(x.tolist()) for x in (row, pos, slot)]
    lin.qk_rope_norm(dev(a, torch.bfloat16), q, kc, vc, *meta, cos, sin, H, G, rot, eps, None, M, status)
    torch.cuda.synchronize()
    assert int(status) == 0
    heads = (a @ w.T).reshape(M, H + G, 128)
    turned = nulunex.unit_rms(nulunex.rotate_halves(heads, pos, rot, 5e4) if rot else heads, eps)
    close(q, turned[:, :H].reshape(M, -1), torch.bfloat16)
    touched = np.zeros((B, max_len), bool)
    touched[row, slot] = True
    for cache, want in ((kc, turned[:, H:]), (vc, heads[:, H:])):
        by_slot = cache.permute(0, 2, 1, 3)
        close(by_slot[torch.from_numpy(row).cuda(), torch.from_numpy(slot).cuda()], want, torch.bfloat16)
        assert (by_slot[torch.from_numpy(~touched).cuda()] == 7).all()


# ------------------------------------------------------------------------------------------ latents
@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("H,d,r,rot,rank,neighbours", [(3, 24, 8, 8, 40, 1), (2, 6, 4, 4, 14, 1), (4, 128, 64, 64, 512, 1), (2, 16, 12, 6, 33, 0),
                                                      (1, 8, 5, 0, 700, 1)])
@pytest.mark.parametrize("in_place", [False, True])
def test_latent_norm_rotation_and_append(dt, H, d, r, rot, rank, neighbours, in_place):
    from recurrent_drafting import _lib

    dtype, rs = DTYPES[dt], np.random.default_rng(rank)
    M, B, max_len, eps = 6, 2, 30, 5e-2
    ldq, ldd = H * (d + r) + 5, rank + r + 2
    q, dkv = rounded(rs.standard_normal((M, ldq)), dtype), rs.standard_normal((M, ldd)).astype(np.float32)
    w = rounded(1 + 0.3 * rs.standard_normal(rank), dtype)
    pos, row, slot = rs.integers(0, 200, M), rs.integers(0, B, M), rs.permutation(max_len)[:M]
    cos, sin = table(rot, 300.0, 200)
    cache = torch.full((B, max_len, rank + r), 7.0, dtype=dtype, device="cuda")
    t_q = dev(q, dtype)
    wide = torch.full((M, H * (rank + r)), 3.0, dtype=dtype, device="cuda")
    to, ld_to, head = (t_q[:, d:], ldq, d + r) if in_place else (wide[:, rank:], wide.stride(0), rank + r)
    _lib.call("rd_latent_append", _lib.dtype_code(dtype), ptr(t_q), ldq, ptr(to), ld_to, head, ptr(dev(dkv)), ldd, ptr(dev(w, dtype)), eps, ptr(cache),
              ptr(i32(row.tolist())), ptr(i32(pos.tolist())), ptr(i32(slot.tolist())), ptr(cos), ptr(sin), 200, M, None, H, d, r, rot, neighbours, rank,
              max_len, _lib.stream())

    def turn(x):
        return ROTATE[neighbours](x, pos, rot, 300.0) if rot else x

    heads = q[:, : H * (d + r)].reshape(M, H, d + r)
    turned = turn(heads[..., d:])
    if in_place:
        got = t_q[:, : H * (d + r)].reshape(M, H, d + r)
        assert torch.equal(got[..., :d].double().cpu(), torch.from_numpy(heads[..., :d]))
        close(got[..., d:], turned, dtype)
    else:
        got = wide.reshape(M, H, rank + r)
        assert (got[..., :rank] == 3).all()
        close(got[..., rank:], turned, dtype)
        assert torch.equal(t_q.double().cpu(), torch.from_numpy(q))
    c = nulunex.rms_norm(dkv[:, :rank].astype(np.float64), w, eps)
    k = turn(dkv[:, None, rank : rank + r].astype(np.float64))[:, 0]
    touched = np.zeros((B, max_len), bool)
    touched[row, slot] = True
    close(cache[torch.from_numpy(row).cuda(), torch.from_numpy(slot).cuda()], np.concatenate([c, k], axis=1), dtype)
    assert (cache[torch.from_numpy(~touched).cuda()] == 7).all()


@pytest.mark.parametrize("dt,width", [("fp32", 48), ("bf16", 48), ("bf16", 14), ("bf16", 21)])
@pytest.mark.parametrize("kind,size", [(0, 1), (0, 70), (0, 64), (1, 50), (1, 64)])
def test_gathered_rows_are_those_that_the_new_tokens_see(dt, width, kind, size):
    from recurrent_drafting import _lib

    dtype, max_len, B = DTYPES[dt], 400, 4
    cache = torch.arange(B * max_len, device="cuda").view(B, max_len, 1).repeat(1, 1, width).to(torch.float32)
    cache = (cache % 251).to(dtype).contiguous()
    base, new, begin = [0, 200, 133, 64], [70, 3, 0, 100], [0, 2, 1, 0]
    starts = np.concatenate([[0], np.cumsum(new)]).tolist()
    first = [max(0, b - size + 1 if kind == 0 else b // size * size) // 64 * 64 for b in base]
    counts = [b + n - f if n else 0 for b, n, f in zip(base, new, first)]
    total = sum(counts)
    out = torch.full((total + 80, width), 9.0, dtype=dtype, device="cuda")
    out_begin, n_out = i32([-1] * B), i32([-1])
    _lib.call("rd_latent_gather", _lib.dtype_code(dtype), ptr(cache), width, max_len, ptr(i32(starts)), ptr(i32(begin)), ptr(i32(base)), B, kind, size,
              ptr(out), total + 80, ptr(out_begin), ptr(n_out), _lib.stream())
    assert int(n_out) == total + 63
    at = 0
    for b in range(B):
        assert int(out_begin[b]) == at - first[b]
        assert torch.equal(out[at : at + counts[b]], cache[b, begin[b] + first[b] : begin[b] + first[b] + counts[b]])
        at += counts[b]
    assert (out[total : total + 63] == 0).all() and (out[total + 63 :] == 9).all()


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 40, 24), (37, 2, 512, 128), (5, 4, 128, 512), (70, 3, 17, 9), (33, 1, 64, 200)])
def test_one_product_per_head(dt, M, H, N, K):
    from recurrent_drafting import _lib

    dtype, rs = DTYPES[dt], np.random.default_rng(M * N)
    pad = 8
    a, w = rounded(rs.standard_normal((M, H, K + pad)), dtype), rounded(rs.standard_normal((H, N, K)) / np.sqrt(K), dtype)
    c = torch.full((M, H, N + pad), 9.0, dtype=dtype, device="cuda")
    live = torch.tensor([max(M - 2, 1)], dtype=torch.int32, device="cuda")
    _lib.call("rd_head_gemm", _lib.dtype_code(dtype), ptr(dev(a, dtype)), H * (K + pad), K + pad, ptr(dev(w, dtype)), ptr(c), H * (N + pad), N + pad, M,
              ptr(live), H, N, K, _lib.stream())
    n = int(live)
    close(c[:n, :, :N], np.einsum("mhk,hnk->mhn", a[:n, :, :K], w), dtype)
    assert (c[n:] == 9).all() and (c[:, :, N:] == 9).all()


# ------------------------------------------------------------------------------------------ attention
TREE_PARENT = [-1, 0, 0, 1, 1, 2, 5, 3, 0, 8]


def draft_tree():
    anc, depth = np.zeros((10, 10), dtype=np.uint8), np.zeros(10, dtype=np.int64)
    for i, p in enumerate(TREE_PARENT):
        anc[i] = anc[p] if p >= 0 else 0
        anc[i, i] = 1
        depth[i] = depth[p] + 1 if p >= 0 else 0
    return anc, depth


def run_attention(form, kind, size, rows, dtype, H, G, d, dv, tail=0, scale=None, sink=None, tree=False, boost=None):
    """rows: (cached, new) tokens of every batch row.  Random queries, keys and values already in the cache, through one of
    the kernels: form "cache" (rd_attention_masked over per-head caches), "umma" (the tcgen05 kernel over them), "latent"
    (values are the first dv features of the one key), "tail" (packed rows, last `tail` key features shared), "umma-tail".
    boost: (row, query, key, factor): the key becomes factor times the query.  Returns (got, want) per row."""
    from recurrent_drafting import _lib

    rs = np.random.default_rng(sum(a * 7 + b for a, b in rows) + size)
    scale = 1.3 / np.sqrt(d) if scale is None else scale
    B, max_len = len(rows), max(a + b for a, b in rows) + 4
    sinks = None if sink is None else (rs.standard_normal(H) + sink).astype(np.float32)
    begin = [b % 2 for b in range(B)]
    packed = form in ("tail", "umma-tail")
    k = rounded(rs.standard_normal((B, G, max_len, d)) * 1.2, dtype)
    v = k[..., :dv] if form == "latent" else rounded(rs.standard_normal((B, G, max_len, dv)), dtype)
    q = [rounded(rs.standard_normal((n, H, d)) * 1.2, dtype) for _, n in rows]
    if boost is not None:
        r, qi, kj, f = boost
        k[r, :, kj] = rounded(f * q[r][qi - rows[r][0], :: H // G], dtype)
        if form == "latent":
            v = k[..., :dv]
    if tail:
        k[..., d - tail :] = k[:, :1, :, d - tail :]
    starts = np.concatenate([[0], np.cumsum([n for _, n in rows])])
    M = int(starts[-1])
    flat = np.concatenate(q).reshape(M, H * d)
    out = torch.full((M, H * dv), 9.0, dtype=dtype, device="cuda")
    anc, depth = draft_tree()
    mode, mask, words, tok_pos = _lib.ATTN_CAUSAL, None, 0, None
    if tree:
        mode, words = _lib.ATTN_TREE, 1
        mask = dev(np.concatenate([(anc.astype(np.int64) << np.arange(10)[None, :]).sum(1) for _ in rows]).astype(np.int32).reshape(M, 1))
        tok_pos = i32(np.concatenate([c + depth for c, _ in rows]).tolist())
    status = i32([0])
    common = dict(row_start=ptr(i32(starts.tolist())), base_len=ptr(i32([c for c, _ in rows])), tok_pos=ptr(tok_pos) if tree else None,
                  tree_mask=ptr(mask) if tree else None)
    t_sink = dev(sinks) if sink is not None else None
    p_sink = ptr(t_sink) if sink is not None else None
    max_new = max(n for _, n in rows)
    if packed:
        # rows back to back, from the tile that holds the first visible key on; a row's key 0 may lie before the buffer
        first = [max(0, c - size + 1 if kind == 0 else c // size * size) // 64 * 64 for c, _ in rows]
        parts = [k[r, :, first[r] : sum(rows[r])] for r in range(B)]
        vals = [v[r, :, first[r] : sum(rows[r])] for r in range(B)]
        at = np.concatenate([[0], np.cumsum([x.shape[1] for x in parts])])
        kb = np.concatenate(parts, axis=1).transpose(1, 0, 2)  # [N, H, d]
        vb = np.concatenate(vals, axis=1).transpose(1, 0, 2)
        N = kb.shape[0] + 63
        zeros = np.zeros((63, H, 1))
        kb, vb = (np.concatenate([x, np.repeat(zeros, x.shape[2], axis=2)]) for x in (kb, vb))
        own, shared = dev(kb[..., : d - tail].reshape(N, -1), dtype), dev(kb[:, 0, d - tail :], dtype)
        values = dev(vb.reshape(N, -1), dtype)
        kv_begin = ptr(i32([int(at[r]) - first[r] for r in range(B)]))
    else:
        def shifted(x):
            y = np.full(x.shape, 5.0)
            for b in range(B):
                y[b, :, begin[b] :] = x[b, :, : max_len - begin[b]]
            return dev(y, dtype)

        kc = shifted(k)
        vc = kc if form == "latent" else shifted(v)
        kv_begin = ptr(i32(begin))
    tq = dev(flat, dtype)
    if form in ("umma", "umma-tail"):
        lib = _lib.load()
        if packed:
            plan = lib.rd_attention_tail_plan_create(ptr(tq), H * d, M, ptr(own), own.shape[1], ptr(shared), tail, ptr(values), values.shape[1], N, B, H, tail)
        else:
            plan = lib.rd_attention_plan_create(ptr(tq), M, ptr(kc), ptr(vc), B, H, G, 128, max_len)
        assert plan
        _lib.call("rd_attention_tc_masked", plan, ptr(out), common["row_start"], kv_begin, common["base_len"], max_new, mode, common["tok_pos"],
                  common["tree_mask"], words, scale, kind, size, 0, None, 0, p_sink, ptr(status), _lib.stream())
        torch.cuda.synchronize()
        lib.rd_attention_plan_destroy(plan)
        assert int(status) == 0
    else:
        desc = _lib.AttentionDesc(q=ptr(tq), ldq=H * d, out=ptr(out), kv_begin=kv_begin, sink=p_sink, dtype=_lib.dtype_code(dtype), B=B, nh=H, nkv=G, dim=d,
                                  vdim=dv, max_new=max_new, max_kv=max_len, mode=mode, mask_words=words, mask_kind=kind, window=size, scale=scale, **common)
        if packed:
            desc.k, desc.k_row, desc.k_head, desc.v, desc.v_row, desc.v_head = ptr(own), own.shape[1], d - tail, ptr(values), values.shape[1], dv
            desc.k_tail, desc.tail_row, desc.tail_dim = ptr(shared), tail, tail
        else:
            desc.k, desc.k_batch, desc.k_head, desc.k_row = ptr(kc), *kc.stride()[:3]
            desc.v, desc.v_batch, desc.v_head, desc.v_row = ptr(vc), *vc.stride()[:3]
        if form == "latent" and dtype == torch.bfloat16 and d % 8 == 0:
            lib = _lib.load()
            plan = lib.rd_attention_latent_plan_create(ptr(tq), M * H, ptr(kc), B * max_len, d)
            assert plan
            _lib.call("rd_attention_latent", plan, ctypes.byref(desc), ptr(status), _lib.stream())
            torch.cuda.synchronize()
            lib.rd_attention_latent_plan_destroy(plan)
            assert int(status) == 0
        else:
            _lib.attention_masked(desc)
        torch.cuda.synchronize()
    got = out.double().cpu().numpy().reshape(M, H, dv)
    visible = (nulunex.window_visible, nulunex.chunk_visible)[kind]
    res = []
    for r, (cached, new) in enumerate(rows):
        if new == 0:
            continue
        pos = np.arange(cached + new)
        if tree:
            pos[cached:] = cached + depth
        vis = visible(pos[cached:], pos, size)
        if tree:
            vis[:, cached:] &= anc.astype(bool)
        kr, vr = (x[r, :, : cached + new].transpose(1, 0, 2) for x in (k, v))
        # a softmax without a sink is one with a sink that weighs nothing
        want = nulunex.attend(q[r], kr, vr, vis, scale, np.full(H, -1e30) if sinks is None else sinks.astype(np.float64))
        res.append((got[starts[r] : starts[r + 1]], want))
    return res


def check_attention(res, dtype, tol16=3e-2):
    for got, want in res:
        err = np.abs(got - want).max()
        assert err < (3e-5 if dtype == torch.float32 else tol16), err


ROWS = ([(0, 150), (0, 1), (37, 70)], [(300, 1), (5, 1), (0, 1)], [(129, 2), (64, 3), (0, 0)])
MASKS = [(1, 1), (1, 20), (1, 64), (1, 100), (1, 500), (0, 1), (0, 33), (0, 500)]


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("kind,size", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 32, 32), (4, 1, 128, 128), (6, 3, 96, 40), (3, 3, 10, 14), (2, 1, 200, 256)])
def test_masked_attention(dt, kind, size, H, G, d, dv):
    for rows, sink in zip(ROWS, (0.0, None, 2.0)):
        check_attention(run_attention("cache", kind, size, rows, DTYPES[dt], H, G, d, dv, sink=sink), DTYPES[dt])


@pytest.mark.parametrize("kind,size", MASKS)
@pytest.mark.parametrize("H,G", [(4, 2), (3, 1)])
def test_masked_attention_on_tcgen05(kind, size, H, G):
    for rows, sink in zip(ROWS + ([(190, 200), (70, 10)],), (0.0, None, 3.0, 1.0)):
        check_attention(run_attention("umma", kind, size, rows, torch.bfloat16, H, G, 128, 128, sink=sink), torch.bfloat16)


@pytest.mark.parametrize("kind,size", MASKS)
@pytest.mark.parametrize("form,H,d,dv,tail", [("tail", 4, 32, 24, 8), ("tail", 2, 112, 128, 16), ("umma-tail", 4, 192, 128, 64), ("umma-tail", 3, 160, 128, 32)])
def test_attention_with_shared_key_features_over_packed_rows(kind, size, form, H, d, dv, tail):
    for rows, sink in (([(0, 150), (0, 40), (137, 70)], 1.0), ([(200, 64), (0, 33), (77, 0), (64, 129)], None), ([(300, 257)], 3.0)):
        check_attention(run_attention(form, kind, size, rows, torch.bfloat16, H, H, d, dv, tail=tail, sink=sink), torch.bfloat16)


LATENT_SIZES = [(3, 48, 40), (20, 120, 104), (32, 128, 128), (5, 232, 200), (4, 320, 256), (8, 576, 512), (32, 544, 512), (2, 36, 30), (2, 21, 14)]


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("kind,size", [(0, 1), (0, 33), (0, 64), (0, 500), (1, 50)])
@pytest.mark.parametrize("H,d,dv", LATENT_SIZES)
def test_attention_whose_values_are_a_part_of_the_shared_key(dt, kind, size, H, d, dv):
    for rows, sink in (([(300, 1), (5, 1), (0, 1)], 1.0), ([(129, 2), (64, 9), (0, 0)], 2.5), ([(0, 40), (90, 30)], None)):
        check_attention(run_attention("latent", kind, size, rows, DTYPES[dt], H, 1, d, dv, sink=sink), DTYPES[dt])


@pytest.mark.parametrize("kind,size", [(0, 50), (0, 64), (1, 50), (1, 64), (1, 40)])
@pytest.mark.parametrize("dt,form,H,G,d,dv,tail", [
    ("fp32", "cache", 4, 2, 64, 56, 0), ("bf16", "cache", 4, 2, 64, 56, 0), ("bf16", "umma", 4, 2, 128, 128, 0), ("fp32", "latent", 4, 1, 72, 64, 0),
    ("bf16", "latent", 4, 1, 72, 64, 0), ("bf16", "tail", 2, 2, 40, 32, 8), ("bf16", "umma-tail", 2, 2, 192, 128, 64)])
def test_one_key_at_every_edge_stands_out(dt, kind, size, form, H, G, d, dv, tail):
    """A key that outweighs all others sits just inside or just outside the window or the chunk, or at a tile's border: the
    output is its value, or is not moved by it."""
    q = 199
    first = q - size + 1 if kind == 0 else q // size * size
    for cached, new in ((0, 200), (140, 60), (199, 1), (196, 4)):
        if form == "tail" and new <= 32:
            continue
        for key in (first, first - 1, first + 1, 0, 64, 63, 127, 128, q, q - 1):
            for sink in (None, 4.0):
                res = run_attention(form, kind, size, [(cached, new)], DTYPES[dt], H, G, d, dv, tail=tail, sink=sink, scale=0.25 / np.sqrt(d / 64),
                                    boost=(0, q, key, 3.0))
                check_attention(res, DTYPES[dt], tol16=4e-2)


@pytest.mark.parametrize("dt", ["fp32", "bf16"])
@pytest.mark.parametrize("kind,size,cached", [(0, 3, 40), (0, 1, 2), (0, 30, 100), (1, 42, 40), (1, 2, 5), (1, 64, 126)])
@pytest.mark.parametrize("form,H,G,d,dv", [("cache", 4, 2, 32, 24), ("cache", 8, 1, 128, 128), ("cache", 3, 3, 10, 14), ("latent", 6, 1, 48, 40),
                                          ("latent", 3, 1, 21, 14)])
def test_attention_over_a_draft_tree(dt, kind, size, cached, form, H, G, d, dv):
    rows = [(cached, 10), (0, 10), (cached + 1, 10)]
    check_attention(run_attention(form, kind, size, rows, DTYPES[dt], H, G, d, dv, sink=1.0, tree=True), DTYPES[dt])


def test_sink_far_above_and_far_below_the_scores():
    for form, d, dv in (("cache", 64, 64), ("umma", 128, 128), ("latent", 72, 64)):
        G = 1 if form == "latent" else 2
        for sink in (60.0, -60.0):
            check_attention(run_attention(form, 0, 40, [(0, 100), (30, 40)], torch.bfloat16, 4, G, d, dv, sink=sink), torch.bfloat16)
