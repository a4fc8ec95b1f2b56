"""A plain, slow implementation of the Nukodra decoder, one function per mechanism, written from
the design's equations in float64.  It is the oracle of the tests: it shares no code with the
package, processes a whole sequence at once, forms keys and values per head, walks recurrences
token by token and keeps no cache.

Notation: ``h`` is a [T, width] block of rows, matrices are stored [out, in] and applied as
``h @ W.T``; ``w`` maps tensor names to float64 tensors and ``pre`` is the prefix of a part's
tensors.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def prepare(raw, round_to=None):
    """float64 copies of the stored tensors; ``round_to`` rounds matrices to that type first, as a
    model bound for it holds them (what stays 32-bit there stays so here)."""
    out = {}
    for name, t in raw.items():
        stays = name.endswith(".conv") or ".hc" in name
        if round_to is not None and t.dim() >= 2 and not stays:
            t = t.to(round_to)
        out[name] = t.to(F64)
    return out


# ---------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_rms(x, weight, eps):
    """The norm in front of a sublayer and of the head: its weight is an offset from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def rotate_halves(vec, position, base, dims):
    """The first ``dims`` numbers turn: number i with number i + dims/2, by position * base^(-2i/dims)."""
    out = vec.clone()
    half = dims // 2
    for i in range(half):
        a = position * base ** (-2.0 * i / dims)
        u, v = vec[i], vec[i + half]
        out[i] = u * math.cos(a) - v * math.sin(a)
        out[i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def rotate_rows(x, rot):
    """x [T, n, d]: every vector of row t turned by position t (``rot`` None: none)."""
    if not rot or not rot["dims"]:
        return x
    out = x.clone()
    for t in range(x.shape[0]):
        for k in range(x.shape[1]):
            out[t, k] = rotate_halves(x[t, k], t, rot["base"], rot["dims"])
    return out


def visible(i, j, window):
    """Whether position i sees position j: itself and what is before it, with a window only the
    window - 1 nearest of those."""
    return j <= i and (not window or i - j < window)


def softmax_over_visible(q, k, v, scale, window=0, cap=0.0, sink=None):
    """q [T, H, n], k [T, H, n], v [T, H, V], head by head.  ``cap``: scores bent by
    cap * tanh(s / cap); ``sink`` [H]: one more logit in the denominator, without a value."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        js = torch.tensor([j for j in range(i + 1) if visible(i, j, window)])
        s = torch.einsum("jhn,hn->hj", k[js], q[i]) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        if sink is not None:
            s = torch.cat([s, sink[:, None]], dim=1)
        p = torch.softmax(s, 1)[:, :len(js)]
        out[i] = torch.einsum("hj,jhv->hv", p, v[js])
    return out


# ---------------------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------------------

def latent_rows(h, w, pre, m, eps):
    """(latent [T, kv_rank], turned key part of all heads [T, rot_dim])."""
    R = m["kv_rank"]
    d = h @ w[pre + "dkv"].T
    c = unit_rms(d[:, :R], eps) * w[pre + "dkv.norm"]
    return c, rotate_rows(d[:, None, R:], m.get("rot"))[:, 0]


def latent_attention(h, w, pre, m, rows):
    """``rows``: the latent and the key part this layer attends to, its own or another layer's."""
    H, D, P, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    T = h.shape[0]
    c, kr = rows
    q = (h @ w[pre + "q"].T).view(T, H, D + P)
    q = torch.cat([q[..., :D], rotate_rows(q[..., D:], m.get("rot"))], dim=2)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D), kr[:, None, :].expand(T, H, P)], dim=2)
    v = (c @ w[pre + "uv"].T).view(T, H, V)
    o = softmax_over_visible(q, k, v, m["scale"], (m.get("mask") or {}).get("size", 0))
    o = o.reshape(T, H * V) * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def window_attention(h, w, pre, m, eps):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (h @ w[pre + n].T + w[pre + n + ".b"] for n in ("q", "k", "v"))
    q = unit_rms(q, eps) * w[pre + "q.norm"]            # over all heads at once
    k = unit_rms(k, eps) * w[pre + "k.norm"]
    q = rotate_rows(q.view(T, H, D), m.get("rot"))
    k = rotate_rows(k.view(T, G, D), m.get("rot"))
    of = torch.tensor([hd // (H // G) for hd in range(H)])
    o = softmax_over_visible(q, k[:, of], v.view(T, G, V)[:, of], m["scale"],
                             (m.get("mask") or {}).get("size", 0), m.get("softcap", 0.0),
                             w[pre + "sink"])
    o = o.reshape(T, H * V) * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def short_conv(x, taps_w, bias):
    """Causal, per channel: the last column of ``taps_w`` [channels, taps] meets the current row."""
    T, taps = x.shape[0], taps_w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        acc = bias.clone()
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                acc = acc + taps_w[:, j] * x[s]
        out[t] = acc
    return out


def state_space(x, B, C, dt, a_log, D, group_of, state=None):
    """x [T, H, V], B and C [T, G, N], dt [T, H]: per head S <- exp(-exp(a_log) dt) S + dt B x^T,
    y = S^T C + D x, token after token.  Returns (y [T, H, V], the state [H, N, V])."""
    T, H, V = x.shape
    S = torch.zeros(H, B.shape[2], V, dtype=F64) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        b, c = B[t, group_of], C[t, group_of]
        S = torch.exp(-torch.exp(a_log) * dt[t])[:, None, None] * S \
            + (dt[t][:, None] * b)[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, c) + D[:, None] * x[t]
    return y, S


def mamba2(h, w, pre, m, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    T, inner = h.shape[0], H * V
    z, xbc, dt = torch.split(h @ w[pre + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"], threshold=1e9)
    group_of = torch.tensor([hd // (H // G) for hd in range(H)])
    y, _ = state_space(x.view(T, H, V), B.view(T, G, N), C.view(T, G, N), dt, w[pre + "A_log"],
                       w[pre + "D"], group_of)
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = unit_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def dense_ff(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


# ---------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------

def connect(X, w, pre, sublayer):
    """One sublayer under hyper-connections: X [streams, T, width]."""
    u = torch.einsum("s,stw->tw", w[pre + "in"], X)
    y = sublayer(u)
    return torch.einsum("st,snw->tnw", w[pre + "mix"], X) + w[pre + "out"][:, None, None] * y


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` (a list) receives the sum of the
    streams after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = x[None].repeat(cfg["streams"], 1, 1) if cfg.get("streams") else x
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]

        def mixer(u):
            h = layer_rms(u, w[p + "norm1"], eps)
            if kind == "latent_attention":
                if m.get("kv_from") is None:
                    latents[i] = latent_rows(h, w, p + "mix.", m, eps)
                return latent_attention(h, w, p + "mix.", m, latents[m.get("kv_from", i)])
            if kind == "attention":
                return window_attention(h, w, p + "mix.", m, eps)
            return mamba2(h, w, p + "mix.", m, eps)

        def feed_forward(u):
            return dense_ff(layer_rms(u, w[p + "norm2"], eps), w, p + "mlp.")

        for q, sublayer in ((1, mixer), (2, feed_forward if layer.get("mlp") else None)):
            if sublayer is not None:
                X = connect(X, w, f"{p}hc{q}.", sublayer) if cfg.get("streams") else X + sublayer(X)
        if layers_out is not None:
            layers_out.append(X.sum(0) if cfg.get("streams") else X.clone())
    x = X.sum(0) if cfg.get("streams") else X
    return layer_rms(x, w["final.norm"], eps) @ w["embed"].T
