"""A plain, slow implementation of the Pivinex decoder, one function per mechanism, written
from the design's equations in float64.  It is the oracle of the tests: it shares no code with
the package, processes a whole sequence at once, forms keys and values per head and keeps no
cache.

Notation: ``h`` is a [T, width] block of rows, matrices are stored [out, in] and applied as
``h @ W.T``; ``w`` maps tensor names to float64 tensors and ``pre`` is the prefix of a part's
tensors.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def prepare(raw, round_to=None):
    """float64 copies of the stored tensors; ``round_to`` rounds matrices to that type first,
    as a model bound for it holds them (the router stays 32-bit)."""
    out = {}
    for name, t in raw.items():
        if round_to is not None and t.dim() >= 2 and not name.endswith(".router"):
            t = t.to(round_to)
        out[name] = t.to(F64)
    return out


# ---------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------

def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def rotate_pairs(vec, position, base):
    """All numbers of ``vec`` in neighbouring pairs; pair i turns by position * base^(-2i/n)."""
    out = vec.clone()
    n = vec.shape[0]
    for i in range(n // 2):
        a = position * base ** (-2.0 * i / n)
        u, v = vec[2 * i], vec[2 * i + 1]
        out[2 * i] = u * math.cos(a) - v * math.sin(a)
        out[2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


# ---------------------------------------------------------------------------------------
# the mixer
# ---------------------------------------------------------------------------------------

def visible(i, j, window):
    """Whether position i sees position j: itself and the window - 1 positions before it."""
    return 0 <= i - j and i - j < window


def queries(h, w, pre, m, eps):
    """Queries through a latent of their own: [T, heads, dim + rot_dim], the last rot_dim turned."""
    H, D, P = m["heads"], m["dim"], m["rot_dim"]
    T = h.shape[0]
    c = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (c @ w[pre + "uq"].T).view(T, H, D + P).clone()
    for t in range(T):
        for hd in range(H):
            q[t, hd, D:] = rotate_pairs(q[t, hd, D:], t, m["rot"]["base"])
    return q


def latent_rows(h, w, pre, m, eps):
    """(latent [T, kv_rank], shared turned key part [T, rot_dim])."""
    R = m["kv_rank"]
    d = h @ w[pre + "dkv"].T
    c = rms_norm(d[:, :R], w[pre + "dkv.norm"], eps)
    kr = torch.stack([rotate_pairs(d[t, R:], t, m["rot"]["base"]) for t in range(h.shape[0])])
    return c, kr


def window_softmax(q, k, v, scale, window):
    """q, k [T, H, n], v [T, H, V]: softmax over the visible positions, head by head."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        js = torch.tensor([j for j in range(max(0, i - window - 2), i + 1) if visible(i, j, window)])
        for hd in range(H):
            s = (k[js, hd] @ q[i, hd]) * scale
            out[i, hd] = torch.softmax(s, 0) @ v[js, hd]
    return out


def latent_attention(h, w, pre, m, eps):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = queries(h, w, pre, m, eps)
    c, kr = latent_rows(h, w, pre, m, eps)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D),
                   kr[:, None, :].expand(T, H, kr.shape[1])], dim=2)
    v = (c @ w[pre + "uv"].T).view(T, H, V)
    o = window_softmax(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(T, H * V) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------

def dense_ff(h, w, pre):
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, correction, top, scale):
    """One token's choice from its logits: (experts, weights).  The choice looks at the softmax
    plus the correction, the weights at the softmax alone; nothing is renormalised."""
    s = torch.softmax(z, 0)
    chosen = torch.argsort(s + correction, descending=True, stable=True)[:top]
    return chosen, s[chosen] * scale


def expert(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def routed_ff(h, w, pre, mlp):
    """Experts with matrices come first; the router's last outputs pass the input through."""
    r = mlp["router"]
    z = h @ w[pre + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, wts = route(z[t], w[pre + "correction"], r["top"], r["scale"])
        for e, a in zip(chosen.tolist(), wts):
            y = h[t] if e >= r["experts"] else expert(h[t:t + 1], w, f"{pre}e{e}.")[0]
            out[t] += a * y
    return out


# ---------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------

def layer_runs(cfg):
    """[(layer, whether the embedding output is added before it)] in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for p in range(loop["times"]):
        runs += [(i, p > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` (a list) receives the stream after
    every layer run."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = layer_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    x = x0
    for i, again in layer_runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        if again:
            x = x + x0
        h = layer_norm(x, w[p + "norm1"], eps)
        y = latent_attention(h, w, p + "mix.", layer["mixer"], eps) * w[p + "ls1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            f = dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp)
            y = y + f * w[p + "ls2"]
        x = x + mult * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
