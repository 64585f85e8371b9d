"""Plain restatement of the Dilavik decoder in numpy float64, one function per mechanism.

Every function works on ONE sequence: x is [T, width], token t sits at position pos0 + t.  Nothing here
is fast and nothing is shared with the product code.  A weight dictionary maps tensor names to arrays,
a configuration is the parsed config.json.

The whole-sequence forms take no state.  `State` holds what earlier tokens of a sequence left behind
(rotated keys and values of the attention layers; S, n, m of the recurrent ones), so that a sequence can
also be fed in pieces, down to one token at a time.
"""
import numpy as np


# ------------------------------------------------------------------------------------------ small pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def grouped_rms_norm(x, w, groups, eps):
    """RMS norm whose mean square is taken over each of `groups` consecutive parts of the row."""
    T, H = x.shape
    return rms(x.reshape(T, groups, H // groups), eps).reshape(T, H) * w


def embed(table, ids, scale):
    return table[np.asarray(ids)] * scale


def depth_average(coeff, history):
    """sum_j coeff[j] * history[j]: history = [embedding output, result of layer 0, ...]."""
    assert len(coeff) == len(history)
    return sum(c * x for c, x in zip(coeff, history))


def xielu(z, p, q):
    """softplus(p) z^2 + z/2 above zero; (1/2 + softplus(q)) (e^z - 1 - z) + z/2 elsewhere."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z + z / 2, (0.5 + softplus(q)) * (np.expm1(neg) - neg) + z / 2)


def dense_feed_forward(x, up, down, act):
    return xielu(x @ up.T, act[0], act[1]) @ down.T


# ------------------------------------------------------------------------------------------ attention
def partial_rotary(x, positions, dims, base):
    """Rotates the pairs (i, i + dims/2) of the first `dims` features of x [T, heads, dim]."""
    half = dims // 2
    freq = base ** (-2.0 * np.arange(half) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def window_visible(qpos, kpos, size, keep_first):
    """[Q, K] bool: not in the future, and within the window or among the sequence's first tokens."""
    i, j = np.asarray(qpos)[:, None], np.asarray(kpos)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_attention(q, k, v, visible, scale):
    """q [Q, H, d], k [K, G, d], v [K, G, dv], visible [Q, K] -> [Q, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = np.empty((q.shape[0], H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = np.where(visible, s, -np.inf)
        p = np.exp(s - s.max(axis=-1, keepdims=True))
        out[:, h] = (p / p.sum(axis=-1, keepdims=True)) @ v[:, g]
    return out


def head_gate(out, x, wg):
    """out [T, H, dv] times one sigmoid per head, formed from the mixer's input."""
    return out * sigmoid(x @ wg.T)[:, :, None]


def attention_mixer(x, w, mix, pos0=0, kv=None):
    """Returns (output [T, width], (keys, values) including what was cached before)."""
    T = x.shape[0]
    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    pos = pos0 + np.arange(T)
    q = partial_rotary((x @ w["q"].T).reshape(T, H, d), pos, mix["rot"]["dims"], mix["rot"]["base"])
    k = partial_rotary((x @ w["k"].T).reshape(T, G, d), pos, mix["rot"]["dims"], mix["rot"]["base"])
    v = (x @ w["v"].T).reshape(T, G, dv)
    if kv is not None:
        k, v = np.concatenate([kv[0], k]), np.concatenate([kv[1], v])
    vis = window_visible(pos, np.arange(k.shape[0]), mix["mask"]["size"], mix["mask"]["keep_first"])
    out = head_gate(softmax_attention(q, k, v, vis, mix["scale"]), x, w["g"])
    return out.reshape(T, H * dv) @ w["o"].T, (k, v)


# ------------------------------------------------------------------------------------------ matrix memory
def mlstm_gates(x, w, cap):
    """(log input gate, log forget gate), each [T, heads]."""
    i = cap * np.tanh((x @ w["i"].T + w["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((x @ w["f"].T + w["f.b"]) / cap))
    return i, f


def mlstm_zero_state(heads, dim, vdim):
    return np.zeros((heads, dim, vdim)), np.zeros((heads, dim)), np.zeros(heads)


def mlstm_step(state, q, k, v, i, f):
    """One token of all heads: q, k [heads, dim], v [heads, vdim], i, f [heads]."""
    S, n, m = state
    m_new = np.maximum(f + m, i)
    a, b = np.exp(f + m - m_new), np.exp(i - m_new)
    S = a[:, None, None] * S + b[:, None, None] * k[:, :, None] * v[:, None, :]
    n = a[:, None] * n + b[:, None] * k
    den = np.maximum(np.abs((n * q).sum(-1)), np.exp(-m_new)) + 1e-6
    o = np.einsum("hdv,hd->hv", S, q) / den[:, None]
    return (S, n, m_new), o


def mlstm_mixer(x, w, mix, eps, state=None):
    """Returns (output [T, width], state after the last token)."""
    T = x.shape[0]
    nh, d, dv = mix["heads"], mix["dim"], mix["vdim"]
    q = (x @ w["q"].T).reshape(T, nh, d) * d ** -0.5
    k = (x @ w["k"].T).reshape(T, nh, d)
    v = (x @ w["v"].T).reshape(T, nh, dv)
    i, f = mlstm_gates(x, w, mix["gate_cap"])
    state = mlstm_zero_state(nh, d, dv) if state is None else state
    o = np.empty((T, nh, dv))
    for t in range(T):
        state, o[t] = mlstm_step(state, q[t], k[t], v[t], i[t], f[t])
    o = rms(o, eps).reshape(T, nh * dv) * w["norm"] * sigmoid(x @ w["g"].T)
    return o @ w["o"].T, state


# ------------------------------------------------------------------------------------------ the model
class State:
    """What a sequence carries from piece to piece."""

    def __init__(self, n_layers):
        self.length = 0
        self.layer = [None] * n_layers


def mixer_weights(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(w, cfg, ids, state=None, layer_outputs=None):
    """Logits [T, vocab] of the tokens `ids`, continuing `state` (updated in place) when one is given.
    layer_outputs, a list, receives the residual stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    groups, eps = cfg["norm"]["groups"], cfg["norm"]["eps"]
    state = State(len(cfg["layers"])) if state is None else state
    x = embed(w["embed"], ids, cfg["embedding"]["scale"])
    history = [x]
    for l, layer in enumerate(cfg["layers"]):
        pre = f"l{l}."
        mw = mixer_weights(w, pre + "mix.")
        h = grouped_rms_norm(x, w[pre + "norm1"], groups, eps)
        if layer["type"] == "attention":
            y, state.layer[l] = attention_mixer(h, mw, layer["mixer"], state.length, state.layer[l])
        elif layer["type"] == "mlstm":
            y, state.layer[l] = mlstm_mixer(h, mw, layer["mixer"], eps, state.layer[l])
        else:
            raise ValueError(layer["type"])
        x = x + y
        if layer["mlp"] is not None:
            h = grouped_rms_norm(x, w[pre + "norm2"], groups, eps)
            x = x + dense_feed_forward(h, w[pre + "mlp.up"], w[pre + "mlp.down"], w[pre + "mlp.act"])
        history.append(x)
        x = depth_average(w[pre + "dwa"], history)
        if layer_outputs is not None:
            layer_outputs.append(x)
    state.length += len(ids)
    return grouped_rms_norm(x, w["final.norm"], groups, eps) @ w["head"].T
