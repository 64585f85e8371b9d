"""Small Nulunex configurations and random weights for the tests.  Scales are chosen so that attention is peaked, sinks take
a share that matters, feed-forward inputs reach their limit and every layer moves the stream: a wrong key, a lost sink or
a wrong weight owner then changes the logits."""
import numpy as np

from dilavik_builders import bf16, error, tokens  # noqa: F401


def attention(heads=4, kv_heads=2, dim=32, rot=16, base=5000.0, scale=0.25, chunk=20, ff=72, limit=1.3):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"dims": rot, "base": base}, "scale": scale,
                      "mask": {"size": chunk}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def latent(heads=3, dim=24, rot_dim=8, vdim=16, rank=40, base=900.0, scale=0.3, window=17, ff=88, limit=0.7):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                      "rot": {"dims": rot_dim, "base": base}, "scale": scale, "mask": {"size": window}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def shared(layer, of):
    return {**layer, "weights_of": of}


def config(layers, vocab=160, width=128, eps=1e-4):
    return {"architecture": "Nulunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_A, _B, _L = attention(), attention(heads=4, kv_heads=2, dim=128, rot=64, scale=0.08, chunk=70, ff=128), latent()

CONFIGS = {
    # both mixers, a shared layer of each kind, layers with and without a feed-forward
    "mixed": config([_A, _L, latent(heads=5, dim=16, rot_dim=16, vdim=40, rank=72, window=33, ff=None), shared(_A, 0), shared(_L, 1),
                     attention(heads=6, kv_heads=1, dim=64, rot=64, scale=0.13, chunk=64, ff=None)]),
    # the sizes of the tcgen05 kernels: heads of 128, latent heads of 128 + 64 and of 128 + 32
    "wide": config([_B, latent(heads=2, dim=128, rot_dim=64, vdim=128, rank=192, window=90, scale=0.09), shared(_B, 0),
                    latent(heads=3, dim=128, rot_dim=32, vdim=128, rank=96, window=64, scale=0.1),
                    attention(heads=3, kv_heads=3, dim=128, rot=128, scale=0.1, chunk=33)], width=192, vocab=224),
    # large latents: the largest tiles of the kernels that read the latents themselves
    "latents": config([latent(heads=4, dim=64, rot_dim=32, vdim=48, rank=512, window=130, scale=0.1),
                       latent(heads=20, dim=16, rot_dim=24, vdim=24, rank=200, window=40, scale=0.2)], width=256, vocab=96),
    # sizes that no vector path takes: the general kernels serve these
    "odd": config([attention(heads=3, kv_heads=3, dim=10, rot=6, chunk=11, scale=0.6, ff=50), latent(heads=2, dim=6, rot_dim=4, vdim=5, rank=14, window=1, ff=30),
                   attention(heads=6, kv_heads=2, dim=12, rot=2, chunk=1, ff=None), latent(heads=3, dim=9, rot_dim=2, vdim=7, rank=21, window=23, scale=0.5)],
                  width=60, vocab=77),
}


def weights(cfg, seed):
    """fp32 arrays under the checkpoint's names."""
    rs = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return (rs.standard_normal((n, k)) * gain / np.sqrt(k)).astype(np.float32)

    def vec(n, mean=1.0, std=0.3):
        return (mean + std * rs.standard_normal(n)).astype(np.float32)

    w = {"embed": (rs.standard_normal((V, W)) * 1.2).astype(np.float32), "head": mat(V, W, 1.5), "final.norm": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        pre, m = f"l{i}.", layer["mixer"]
        p = pre + "mix."
        w[pre + "norm1"] = vec(W)
        if layer["type"] == "attention":
            w[p + "q"], w[p + "k"] = mat(m["heads"] * m["dim"], W), mat(m["kv_heads"] * m["dim"], W, 1.4)
        else:
            H, r = m["heads"], m["kv_rank"]
            w[p + "q"] = mat(H * (m["dim"] + m["rot_dim"]), W, 1.5)
            w[p + "dkv"], w[p + "dkv.norm"] = mat(r + m["rot_dim"], W, 1.3), vec(r)
            w[p + "uk"], w[p + "uv"] = mat(H * m["dim"], r, 1.3), mat(H * m["vdim"], r, 1.3)
            w[p + "sink"] = vec(H, 1.5, 1.0)
        w[p + "o"] = mat(W, m["heads"] * m["vdim"], 1.2)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[pre + "norm2"] = vec(W)
            w[pre + "mlp.gate"], w[pre + "mlp.up"], w[pre + "mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff, 1.2)
    return w


def build(cfg, w, dtype, device="cuda"):
    import torch
    from recurrent_drafting import configuration_nulunex, modeling_nulunex

    with torch.device(device):
        llm = modeling_nulunex.NulunexForCausalLM(configuration_nulunex.NulunexConfig.from_dict(cfg)).to(dtype)
    llm.load_state_dict({k: torch.from_numpy(v) for k, v in w.items()})
    return llm
