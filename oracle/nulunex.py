"""Plain restatement of the Nulunex decoder in numpy float64, one function per mechanism.

Every function works on ONE sequence: x is [T, width], token t sits at position pos0 + t.  Nothing here
is fast and nothing is shared with the product code.  A weight dictionary maps tensor names to arrays,
a configuration is the parsed config.json.

`State` holds what earlier tokens of a sequence left behind (normed rotated keys and raw values of the
grouped attention, latents and rotated key parts of the latent attention), so that a sequence can also be
fed in pieces, down to one token at a time.
"""
import numpy as np


# ------------------------------------------------------------------------------------------ small pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def clamped_glu(gate, up, limit, alpha=1.702):
    """Gate cut from above, up cut on both sides; g sigmoid(alpha g) (u + 1)."""
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(alpha * g) * (u + 1.0)


def feed_forward(x, gate, up, down, limit):
    return clamped_glu(x @ gate.T, x @ up.T, limit) @ down.T


# ------------------------------------------------------------------------------------------ rotation
def rotation_angles(positions, dims, base):
    """[T, dims/2]: position times base^(-2i/dims)."""
    return np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)[None, :]


def rotate_halves(x, positions, dims, base):
    """x [T, heads, d]: feature i turns with feature i + dims/2; features past dims stay."""
    a = rotation_angles(positions, dims, base)[:, None, :]
    h = dims // 2
    u, v = x[..., :h], x[..., h:dims]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., dims:]], axis=-1)


def rotate_neighbours(x, positions, dims, base):
    """x [T, heads, d]: feature 2i turns with feature 2i + 1; features past dims stay."""
    a = rotation_angles(positions, dims, base)[:, None, :]
    y = np.array(x, dtype=np.float64)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return y


# ------------------------------------------------------------------------------------------ visibility, softmax
def chunk_visible(qpos, kpos, size):
    """[Q, K] bool: not in the future and in the query's own chunk of `size` positions."""
    i, j = np.asarray(qpos)[:, None], np.asarray(kpos)[None, :]
    return (j <= i) & (i // size == j // size)


def window_visible(qpos, kpos, size):
    """[Q, K] bool: the query itself and the size - 1 positions before it."""
    i, j = np.asarray(qpos)[:, None], np.asarray(kpos)[None, :]
    return (j <= i) & (i - j < size)


def softmax_with_sink(s, sink):
    """Softmax along the last axis with exp(sink) added to the denominator; -inf scores weigh nothing."""
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    p = np.exp(s - m)
    return p / (p.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def attend(q, k, v, visible, scale, sink):
    """q [Q, H, d], k [K, G, d], v [K, G, dv], visible [Q, K], sink [H] -> [Q, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = np.empty((q.shape[0], H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(visible, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        out[:, h] = softmax_with_sink(s, sink[h]) @ v[:, g]
    return out


# ------------------------------------------------------------------------------------------ mixers
def attention_mixer(x, w, mix, eps, pos0=0, kv=None):
    """Chunked grouped attention whose values are the raw keys.  Returns (output [T, width], (keys, values) including
    what was cached before)."""
    T = x.shape[0]
    H, G, d = mix["heads"], mix["kv_heads"], mix["dim"]
    pos = pos0 + np.arange(T)
    v = (x @ w["k"].T).reshape(T, G, d)
    q = unit_rms(rotate_halves((x @ w["q"].T).reshape(T, H, d), pos, mix["rot"]["dims"], mix["rot"]["base"]), eps)
    k = unit_rms(rotate_halves(v, pos, mix["rot"]["dims"], mix["rot"]["base"]), eps)
    if kv is not None:
        k, v = np.concatenate([kv[0], k]), np.concatenate([kv[1], v])
    vis = chunk_visible(pos, np.arange(k.shape[0]), mix["mask"]["size"])
    out = attend(q, k, v, vis, mix["scale"], np.zeros(H))
    return out.reshape(T, H * d) @ w["o"].T, (k, v)


def latents(x, w, mix, eps, pos):
    """(c [T, rank] normed, shared rotated key part [T, rot_dim])."""
    r = mix["kv_rank"]
    y = x @ w["dkv"].T
    rot = rotate_neighbours(y[:, None, r:], pos, mix["rot"]["dims"], mix["rot"]["base"])[:, 0]
    return rms_norm(y[:, :r], w["dkv.norm"], eps), rot


def latent_mixer(x, w, mix, eps, pos0=0, cached=None):
    """Window attention over keys and values that are projections of one latent per token.  Returns (output [T, width],
    (latents, rotated key parts) including what was cached before)."""
    T = x.shape[0]
    H, d, r, dv = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    pos = pos0 + np.arange(T)
    q = (x @ w["q"].T).reshape(T, H, d + r)
    q = np.concatenate([q[..., :d], rotate_neighbours(q[..., d:], pos, mix["rot"]["dims"], mix["rot"]["base"])], axis=-1)
    c, kr = latents(x, w, mix, eps, pos)
    if cached is not None:
        c, kr = np.concatenate([cached[0], c]), np.concatenate([cached[1], kr])
    K = c.shape[0]
    k = np.concatenate([(c @ w["uk"].T).reshape(K, H, d), np.broadcast_to(kr[:, None, :], (K, H, r))], axis=-1)
    v = (c @ w["uv"].T).reshape(K, H, dv)
    out = attend(q, k, v, window_visible(pos, np.arange(K), mix["mask"]["size"]), mix["scale"], w["sink"])
    return out.reshape(T, H * dv) @ w["o"].T, (c, kr)


# ------------------------------------------------------------------------------------------ the model
class State:
    """What a sequence carries from piece to piece."""

    def __init__(self, n_layers):
        self.length = 0
        self.layer = [None] * n_layers


def owner(cfg, l):
    """The layer whose tensors layer l uses."""
    while cfg["layers"][l].get("weights_of") is not None:
        l = cfg["layers"][l]["weights_of"]
    return l


def mixer_weights(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(w, cfg, ids, state=None, layer_outputs=None):
    """Logits [T, vocab] of the tokens `ids`, continuing `state` (updated in place) when one is given.
    layer_outputs, a list, receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    state = State(len(cfg["layers"])) if state is None else state
    x = w["embed"][np.asarray(ids)]
    mixers = {"attention": attention_mixer, "latent_attention": latent_mixer}
    for l, layer in enumerate(cfg["layers"]):
        pre = f"l{owner(cfg, l)}."
        h = rms_norm(x, w[pre + "norm1"], eps)
        y, state.layer[l] = mixers[layer["type"]](h, mixer_weights(w, pre + "mix."), layer["mixer"], eps, state.length, state.layer[l])
        x = x + y
        mlp = layer["mlp"]
        if mlp is not None:
            h = rms_norm(x, w[pre + "norm2"], eps)
            x = x + feed_forward(h, w[pre + "mlp.gate"], w[pre + "mlp.up"], w[pre + "mlp.down"], mlp["limit"])
        if layer_outputs is not None:
            layer_outputs.append(x)
    state.length += len(ids)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
