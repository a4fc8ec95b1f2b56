"""Nukodra: a decoder whose layers are listed one by one in config.json.  The residual stream
exists in several copies (hyper-connections): every sublayer reads a learned combination of them
through an RMS norm whose weights are kept as offsets from one, and writes its output and a learned mixture
of the copies back; the head reads their sum.  A layer is a mixer followed by a dense gated
feed-forward (``W_down (silu(W_gate h) * (W_up h))``), or a mixer alone.  Three mixers:

* attention over a shared latent, causal, with an output gate; a layer may read the latents another
  layer wrote (``kv_from``) with its own queries and expansions;
* grouped attention inside a sliding window: biases, queries and keys normed over their whole
  projections and turned in halves, capped scores, a sink per head, an output gate;
* a state-space recurrence (Mamba-2) with short convolutions and a gated norm in parts.

The token table is also the head.  config.json::

    {"architecture": "Nukodra", "vocab": V, "width": W, "streams": s   (absent: one plain stream),
     "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
                           "rot": {"base", "dims"}, "kv_from": j   (optional)}}
              | {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap"   (optional),
                           "mask": {"size"}   (optional), "rot": {"base", "dims"}}}
              | {"type": "mamba2",
                 "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"}},
                each with "mlp": {"kind": "dense", "ff"} | null, ...]}

Tensors: ``embed``; per layer ``l<i>.norm1``, ``l<i>.hc1.{in, mix, out}`` and, with a feed-forward,
``l<i>.norm2``, ``l<i>.hc2.{in, mix, out}`` and ``l<i>.mlp.{gate, up, down}``; the mixers'
``l<i>.mix.{q, dkv, dkv.norm, uk, uv, g, o}``, ``l<i>.mix.{q, k, v}`` each with ``.b``,
``l<i>.mix.{q.norm, k.norm, sink, g, o}`` or ``l<i>.mix.{in, conv, conv.b, dt_bias, A_log, D, norm,
o}``; ``final.norm``.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Any, Mapping

import torch

from ..config.model_config import (Architecture, ConfigError, need, positive_int,
                                   register_architecture)
from ..parts.hyper_connection import MAX_STREAMS
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

LAYER_TYPES = ("latent_attention", "attention", "mamba2")


def _number(name: str, v: Any, positive: bool = False) -> float:
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"{name} must be a{' positive' if positive else ''} number, got {v!r}")
    return float(v)


def _section(raw: Mapping, key: str, where: str) -> Mapping:
    v = raw.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where} needs an object {key!r}")
    return v


def _check_rot(where: str, m: Mapping, extent: int) -> None:
    if m.get("rot") is None:
        return
    rot = _section(m, "rot", where)
    _number(f"{where}.rot.base", need(rot, "base"), positive=True)
    dims = need(rot, "dims")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims % 2 or not 0 <= dims <= extent:
        raise ConfigError(f"{where}.rot.dims must be an even number up to {extent}, got {dims!r}")


def _check_layer(i: int, layer, layers) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, Mapping) or layer.get("type") not in LAYER_TYPES:
        raise ConfigError(f"{where}.type must be one of {LAYER_TYPES}")
    m, kind = _section(layer, "mixer", where), layer["type"]
    wm = where + ".mixer"
    sizes = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank"),
             "attention": ("heads", "kv_heads", "dim", "vdim"),
             "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups")}[kind]
    for key in sizes:
        positive_int(f"{wm}.{key}", need(m, key))
    if kind == "mamba2":
        if m["heads"] % m["groups"]:
            raise ConfigError(f"{wm}.heads is not a multiple of groups")
        if m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ConfigError(f"{wm}.norm_groups does not divide heads * vdim")
    else:
        _number(f"{wm}.scale", need(m, "scale"))
        _check_rot(wm, m, m["rot_dim"] if kind == "latent_attention" else m["dim"])
        if m.get("mask") is not None:
            positive_int(f"{wm}.mask.size", need(_section(m, "mask", wm), "size"))
    if kind == "attention":
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{wm}.heads is not a multiple of kv_heads")
        if m.get("softcap") is not None:
            _number(f"{wm}.softcap", m["softcap"], positive=True)
    src = m.get("kv_from")
    if kind == "latent_attention" and src is not None:
        ok = isinstance(src, int) and not isinstance(src, bool) and 0 <= src < i \
            and layers[src].get("type") == "latent_attention" \
            and layers[src]["mixer"].get("kv_from") is None
        if not ok:
            raise ConfigError(f"{wm}.kv_from must name an earlier latent_attention layer that has "
                              f"a latent of its own, got {src!r}")
        if any(layers[src]["mixer"].get(k) != m.get(k) for k in ("kv_rank", "rot_dim", "rot")):
            raise ConfigError(f"{wm}: kv_rank, rot_dim and rot must equal those of layer {src}, "
                              f"whose cache it reads")
    mlp = layer.get("mlp")
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
            raise ConfigError(f"{where}.mlp must be null or an object of kind 'dense'")
        positive_int(f"{where}.mlp.ff", need(mlp, "ff"))


@dataclass(frozen=True)
class NukodraConfig:
    vocab: int
    width: int
    streams: int | None                 # None: one stream without connections
    norm_eps: float
    layers: tuple                       # the layer entries of config.json, as they stand
    architectures: tuple[str, ...] = ("Nukodra",)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NukodraConfig":
        vocab = positive_int("vocab", need(raw, "vocab"))
        width = positive_int("width", need(raw, "width"))
        streams = raw.get("streams")
        if streams is not None and positive_int("streams", streams) > MAX_STREAMS:
            raise ConfigError(f"streams: at most {MAX_STREAMS}, got {streams}")
        eps = _number("norm.eps", need(_section(raw, "norm", "config.json"), "eps"), positive=True)
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        for i, layer in enumerate(layers):
            _check_layer(i, layer, layers)
        return cls(vocab, width, streams, eps, tuple(copy.deepcopy(list(layers))))

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": "Nukodra", "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.streams is not None:
            out["streams"] = self.streams
        return out

    def num_parameters(self) -> int:
        return sum(math.prod(t.shape) for t in init_weights(self, 0, shapes_only=True).values())


def _norm_spec(name: str, cfg: NukodraConfig) -> PartSpec:
    return PartSpec("rms_norm", dict(width=cfg.width, eps=cfg.norm_eps, weight=name, one_plus=True))


def _connection_spec(p: str, cfg: NukodraConfig) -> PartSpec:
    return PartSpec("hyper_connection", dict(streams=cfg.streams, read=p + "in", mix=p + "mix",
                                             write=p + "out"))


def _mixer_spec(p: str, kind: str, m: Mapping, cfg: NukodraConfig) -> PartSpec:
    W, eps = cfg.width, cfg.norm_eps
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    window = (m.get("mask") or {}).get("size", 0)
    if kind == "latent_attention":
        own = m.get("kv_from") is None
        return PartSpec("latent_attention", dict(
            width=W, n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
            kv_rank=m["kv_rank"], scale=m["scale"], rot_base=rot["base"], rot_dims=rot["dims"],
            rot_pairing="halves", eps=eps, q_weight=p + "q",
            latent_weight=p + "dkv" if own else None,
            latent_norm=p + "dkv.norm" if own else None, key_up=p + "uk", value_up=p + "uv",
            sink=None, gate=p + "g", out_weight=p + "o", shares_cache=not own, window=window))
    if kind == "attention":
        return PartSpec("span_attention", dict(
            width=W, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
            value_dim=m["vdim"], scale=m["scale"], prefix=p, window=window, qk_norm="rows", eps=eps,
            gate=True, biases=True, rot_base=rot["base"], rot_dims=rot["dims"],
            softcap=m.get("softcap") or 0.0, sink=True))
    return PartSpec("state_space", dict(
        width=W, n_heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"],
        taps=m["conv"], norm_groups=m["norm_groups"], eps=eps, prefix=p))


def build_spec(cfg: NukodraConfig) -> ModelSpec:
    layers, schedule = [], []
    entry_of: dict[int, int] = {}          # layer -> the cache entry it owns
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        parts = dict(norm1=_norm_spec(p + "norm1", cfg),
                     mixer=_mixer_spec(p + "mix.", layer["type"], m, cfg))
        mlp = layer.get("mlp")
        if mlp is not None:
            parts["norm2"] = _norm_spec(p + "norm2", cfg)
            parts["feed_forward"] = PartSpec("gated", dict(
                width=cfg.width, inner=mlp["ff"], activation="silu", gate_weight=p + "mlp.gate",
                up_weight=p + "mlp.up", down_weight=p + "mlp.down"))
        if cfg.streams is not None:
            parts["connect1"] = _connection_spec(p + "hc1.", cfg)
            if mlp is not None:
                parts["connect2"] = _connection_spec(p + "hc2.", cfg)
        layers.append(LayerSpec("pre_norm" if cfg.streams is None else "hyper_connected", parts))
        src = m.get("kv_from") if layer["type"] == "latent_attention" else None
        if src is None:
            entry_of[i] = len(entry_of)
        schedule.append(LayerCall(i, entry_of[i if src is None else src], src is None))
    return ModelSpec(
        name="Nukodra", vocab_size=cfg.vocab, width=cfg.width, max_positions=None,
        embedding=PartSpec("token_table", dict(vocab_size=cfg.vocab, width=cfg.width,
                                               table="embed")),
        position=PartSpec("none", {}), layers=tuple(layers), schedule=tuple(schedule),
        final_norm=_norm_spec("final.norm", cfg),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, width=cfg.width, weight="embed")),
        eos_token_id=None)


def init_weights(cfg: NukodraConfig, seed: int, shapes_only: bool = False):
    """Seeded random float32 weights under the checkpoint's names, drawn from one CPU generator
    in the order the names are listed here.  Matrices ~ N(0, 1/sqrt(in)); norm weights around 0
    where they are offsets and around 1 elsewhere; connections near reading the mean of the
    copies, keeping each and writing to all, spread enough that an exchanged index shows."""
    gen = torch.Generator(device="cpu")
    gen.manual_seed(int(seed))
    w: dict[str, torch.Tensor] = {}

    def put(name, shape, std=None, mean=0.0):
        if shapes_only:
            w[name] = torch.empty(shape, device="meta")
            return
        if std is None:
            std = 1.0 / math.sqrt(shape[-1])
        w[name] = torch.randn(shape, generator=gen, dtype=torch.float32) * std + mean

    def connect(name):
        S = cfg.streams
        if S is None:
            return
        put(name + "in", (S,), 0.3, 1.0 / S)
        put(name + "mix", (S, S), 0.15)
        if not shapes_only:
            w[name + "mix"] += 0.85 * torch.eye(S)
        put(name + "out", (S,), 0.3, 1.0)

    W = cfg.width
    put("embed", (cfg.vocab, W), 0.5)
    for i, layer in enumerate(cfg.layers):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        a = p + "mix."
        put(p + "norm1", (W,), 0.1)
        connect(p + "hc1.")
        H, V = m["heads"], m["vdim"]
        if kind == "latent_attention":
            D, P, R = m["dim"], m["rot_dim"], m["kv_rank"]
            put(a + "q", (H * (D + P), W), 1.5 / math.sqrt(W))
            if m.get("kv_from") is None:
                put(a + "dkv", (R + P, W))
                put(a + "dkv.norm", (R,), 0.1, 1.0)
            put(a + "uk", (H * D, R), 1.5 / math.sqrt(R))
            put(a + "uv", (H * V, R))
        elif kind == "attention":
            D, G = m["dim"], m["kv_heads"]
            for name, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
                put(a + name, (rows, W))
                put(a + name + ".b", (rows,), 0.2)
            put(a + "q.norm", (H * D,), 0.2, 1.5)
            put(a + "k.norm", (G * D,), 0.2, 1.5)
            put(a + "sink", (H,), 1.0, 1.0)
        else:
            N, G = m["state"], m["groups"]
            C = H * V + 2 * G * N
            put(a + "in", (H * V + C + H, W))
            put(a + "conv", (C, m["conv"]), 0.5)
            put(a + "conv.b", (C,), 0.2)
            put(a + "dt_bias", (H,), 0.7, -1.0)
            put(a + "A_log", (H,), 0.7, 0.0)
            put(a + "D", (H,), 0.3, 1.0)
            put(a + "norm", (H * V,), 0.1, 1.0)
        if kind != "mamba2":
            put(a + "g", (H * V, W))
        put(a + "o", (W, H * V))
        mlp = layer.get("mlp")
        if mlp is not None:
            put(p + "norm2", (W,), 0.1)
            connect(p + "hc2.")
            put(p + "mlp.gate", (mlp["ff"], W), 1.5 / math.sqrt(W))
            put(p + "mlp.up", (mlp["ff"], W))
            put(p + "mlp.down", (W, mlp["ff"]))
    put("final.norm", (W,), 0.1)
    return w


def _latent(heads, dim, rot_dim, vdim, kv_rank, base=10000.0, kv_from=None):
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
           "scale": 1.0 / math.sqrt(dim + rot_dim), "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def _attention(heads, kv_heads, dim, window, base=100000.0, softcap=30.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
            "scale": 1.0 / math.sqrt(dim), "softcap": softcap, "mask": {"size": window},
            "rot": {"base": base, "dims": dim}}


def _mamba2(heads, vdim, state, groups, conv=4, norm_groups=None):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
            "norm_groups": norm_groups or groups}


def _preset(vocab, width, streams, latent, attention, mamba2, ff, eps=1e-6):
    """Four layers: a recurrence, a latent layer, windowed attention, and a latent layer that
    reads the first one's rows."""
    mlp = {"kind": "dense", "ff": ff}
    layers = [{"type": "mamba2", "mixer": mamba2, "mlp": None},
              {"type": "latent_attention", "mixer": latent, "mlp": dict(mlp)},
              {"type": "attention", "mixer": attention, "mlp": dict(mlp)},
              {"type": "latent_attention", "mixer": dict(copy.deepcopy(latent), kv_from=1),
               "mlp": dict(mlp)}]
    return {"architecture": "Nukodra", "vocab": vocab, "width": width, "streams": streams,
            "norm": {"eps": eps}, "layers": layers}


PRESETS: dict[str, dict] = {
    # a few hundred thousand parameters: for demonstrations and smoke runs
    "nukodra-tiny": _preset(384, 96, 3, _latent(4, 16, 8, 24, 40), _attention(4, 2, 24, 40),
                            _mamba2(6, 20, 24, 2), 160),
    # layer sizes of a small and a mid-sized production model, few layers: for measurements
    "nukodra-1k": _preset(32768, 1024, 2, _latent(8, 128, 64, 128, 256),
                          _attention(16, 4, 64, 256), _mamba2(32, 64, 128, 2), 4096),
    "nukodra-2k": _preset(32768, 2048, 4, _latent(16, 128, 64, 128, 512),
                          _attention(16, 4, 128, 256), _mamba2(64, 64, 128, 4), 8192),
}

NUKODRA = Architecture(name="Nukodra", config_cls=NukodraConfig, build_spec=build_spec,
                       init_weights=init_weights, model_types=("nukodra",), presets=PRESETS,
                       preset_aliases={})
register_architecture(NUKODRA, replace=True)
