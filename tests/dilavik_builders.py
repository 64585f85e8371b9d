"""Small Dilavik configurations and random weights for the tests.  Scales are chosen so that attention is peaked, gates
open and close and every layer's result matters: a wrong key, a lost state or a skipped layer then changes the logits."""
import numpy as np


def attention(heads=4, kv_heads=2, dim=32, vdim=24, rot=16, base=5000.0, scale=0.25, window=20, keep=3, ff=96):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base},
                      "scale": scale, "mask": {"size": window, "keep_first": keep}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mlstm(heads=3, dim=16, vdim=40, cap=7.0, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=160, width=128, groups=2, eps=1e-4, scale=1.7):
    return {"architecture": "Dilavik", "vocab": vocab, "width": width, "embedding": {"scale": scale},
            "norm": {"eps": eps, "groups": groups}, "layers": layers}


CONFIGS = {
    # recurrent layer first, one with a feed-forward, attention without one; unequal layers
    "mixed": config([mlstm(ff=72), attention(ff=None), mlstm(heads=2, dim=48, vdim=32), attention(window=9, keep=0, kv_heads=4)]),
    # every key/value head its own query head, full rotation, one norm group, no kept token, keys larger than values
    "plain": config([attention(heads=2, kv_heads=2, dim=64, vdim=64, rot=64, window=33, keep=0), mlstm(heads=1, dim=64, vdim=64)],
                    width=64, groups=1, vocab=96),
    # head size 128 on both sides, one key/value head, matrix memory at its largest tile
    "wide": config([attention(heads=4, kv_heads=1, dim=128, vdim=128, rot=32, window=70, keep=5, ff=128),
                    mlstm(heads=1, dim=256, vdim=96, ff=64), attention(heads=2, kv_heads=1, dim=96, vdim=128, rot=96, window=64, keep=64)],
                   width=192, groups=3, vocab=224),
    # sizes that no vector path takes: the general kernels serve these
    "odd": config([attention(heads=3, kv_heads=3, dim=10, vdim=14, rot=6, window=11, keep=2, ff=50), mlstm(heads=2, dim=6, vdim=10, cap=3.0),
                   attention(heads=6, kv_heads=2, dim=12, vdim=5, rot=0, window=1, keep=1, ff=30)], width=60, groups=5, vocab=77),
}


def weights(cfg, seed):
    """fp32 arrays under the checkpoint's names."""
    rs = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return (rs.standard_normal((n, k)) * gain / np.sqrt(k)).astype(np.float32)

    def vec(n, mean=1.0, std=0.3):
        return (mean + std * rs.standard_normal(n)).astype(np.float32)

    w = {"embed": (rs.standard_normal((V, W)) * 0.8).astype(np.float32), "head": mat(V, W, 1.5), "final.norm": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        w[pre + "norm1"] = vec(W)
        dwa = 0.25 * rs.standard_normal(i + 2)
        dwa[-1] += 0.9
        w[pre + "dwa"] = dwa.astype(np.float32)
        p = pre + "mix."
        if layer["type"] == "attention":
            w[p + "q"], w[p + "k"] = mat(m["heads"] * m["dim"], W, 1.6), mat(m["kv_heads"] * m["dim"], W, 1.6)
            w[p + "v"], w[p + "g"] = mat(m["kv_heads"] * m["vdim"], W, 1.2), mat(m["heads"], W)
        else:
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            w[p + "q"], w[p + "k"] = mat(H * d, W, 1.5), mat(H * d, W, 1.5)
            w[p + "v"], w[p + "g"] = mat(H * dv, W, 1.2), mat(H * dv, W)
            w[p + "i"], w[p + "f"] = mat(H, W, 1.5), mat(H, W, 1.5)
            w[p + "i.b"], w[p + "f.b"] = vec(H, 0.0, 0.7), vec(H, 4.0, 1.0)
            w[p + "norm"] = vec(H * dv)
        w[p + "o"] = mat(W, m["heads"] * m["vdim"], 1.2)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[pre + "norm2"] = vec(W)
            w[pre + "mlp.up"], w[pre + "mlp.down"] = mat(ff, W), mat(W, ff, 0.7)
            w[pre + "mlp.act"] = vec(2, 0.0, 0.8)
    return w


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(3, cfg["vocab"], n).astype(np.int64)


def bf16(w):
    """The values a bf16 model holds."""
    import torch

    return {k: torch.from_numpy(v).to(torch.bfloat16).float().numpy() for k, v in w.items()}


def build(cfg, w, dtype, device="cuda"):
    import torch
    from recurrent_drafting import configuration_dilavik, modeling_dilavik

    with torch.device(device):
        llm = modeling_dilavik.DilavikForCausalLM(configuration_dilavik.DilavikConfig.from_dict(cfg)).to(dtype)
    llm.load_state_dict({k: torch.from_numpy(v) for k, v in w.items()})
    return llm


def error(got, want):
    """RMS over the vocabulary of the centred difference, in units of the wanted logits' own RMS; the worst row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    scale = np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())
    return float(np.sqrt((d ** 2).mean(-1)).max() / scale)
