"""Pivinex: a decoder whose layers are listed one by one in config.json and of which a stretch
may run several times in a row with the same weights (every pass with a cache entry of its own;
the embedding's output is added to the stream before each pass but the first).  The token rows
are layer-normed at the input.  Every layer is a parallel block under one layer norm (a weight,
no bias) whose sublayers' outputs are scaled per channel and by a constant of the model,

    h = norm1(x);   x += m * (ls1 * mixer(h) + ls2 * feed_forward(h))

The mixer is attention over a shared latent inside a sliding window, whose queries come through
a latent of their own (each latent RMS-normed).  The feed-forward is dense
(``W_down (gelu_tanh(W_gate h) * (W_up h))``), a mixture of experts
(``W_down (silu(W_gate h) * (W_up h))``) chosen by corrected softmax scores, some of whose choices
pass the input through, or absent.  The head is a table of its own.

config.json::

    {"architecture": "Pivinex", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "loop": {"start": a, "stop": b, "times": n}   (optional: layers a .. b-1 run n times),
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale",
                           "mask": {"size"}, "rot": {"base", "dims"}},
                 "mlp": {"kind": "dense", "ff"}
                      | {"kind": "moe", "expert": {"ff"},
                         "router": {"experts", "top", "identity", "scale"}} | null}, ...]}

Tensors: ``embed``, ``embed.norm``; per layer ``l<i>.norm1``, ``l<i>.mix.{dq, dq.norm, uq, dkv,
dkv.norm, uk, uv, o}``, ``l<i>.ls1`` and, with a feed-forward, ``l<i>.ls2`` and
``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.{router, correction}`` and
``l<i>.mlp.e<k>.{gate, up, down}``; ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Any, Mapping

import torch

from ..config.model_config import (Architecture, ConfigError, need, positive_int,
                                   register_architecture)
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

LAYER_TYPES = ("latent_attention",)
FEED_FORWARDS = ("dense", "moe")


def _number(name: str, v: Any, positive: bool = False) -> float:
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and not v > 0):
        raise ConfigError(f"{name} must be a{' positive' if positive else ''} number, got {v!r}")
    return float(v)


def _section(raw: Mapping, key: str, where: str) -> Mapping:
    v = raw.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"{where} needs an object {key!r}")
    return v


def _check_mlp(where: str, mlp) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, Mapping) or mlp.get("kind") not in FEED_FORWARDS:
        raise ConfigError(f"{where} must be null or an object whose kind is one of {FEED_FORWARDS}")
    if mlp["kind"] == "dense":
        positive_int(f"{where}.ff", need(mlp, "ff"))
        return
    ex, ro = _section(mlp, "expert", where), _section(mlp, "router", where)
    positive_int(f"{where}.expert.ff", need(ex, "ff"))
    experts = positive_int(f"{where}.router.experts", need(ro, "experts"))
    top = positive_int(f"{where}.router.top", need(ro, "top"))
    identity = ro.get("identity", 0)
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f"{where}.router.identity must be a number of experts, got {identity!r}")
    if top > experts + identity:
        raise ConfigError(f"{where}.router: {experts} + {identity} outputs and {top} chosen ones "
                          f"do not fit together")
    _number(f"{where}.router.scale", ro.get("scale", 1.0))


def _check_layer(i: int, layer) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, Mapping) or layer.get("type") not in LAYER_TYPES:
        raise ConfigError(f"{where}.type must be one of {LAYER_TYPES}")
    m = _section(layer, "mixer", where)
    wm = where + ".mixer"
    for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"):
        positive_int(f"{wm}.{key}", need(m, key))
    _number(f"{wm}.scale", need(m, "scale"))
    positive_int(f"{wm}.mask.size", need(_section(m, "mask", wm), "size"))
    rot = _section(m, "rot", wm)
    _number(f"{wm}.rot.base", need(rot, "base"), positive=True)
    dims = need(rot, "dims")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims % 2 or \
            not 0 <= dims <= m["rot_dim"]:
        raise ConfigError(f"{wm}.rot.dims must be an even number up to rot_dim, got {dims!r}")
    _check_mlp(where + ".mlp", layer.get("mlp"))


@dataclass(frozen=True)
class PivinexConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    loop: tuple | None              # (start, stop, times)
    layers: tuple                   # the layer entries of config.json, as they stand
    architectures: tuple[str, ...] = ("Pivinex",)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "PivinexConfig":
        vocab = positive_int("vocab", need(raw, "vocab"))
        width = positive_int("width", need(raw, "width"))
        eps = _number("norm.eps", need(_section(raw, "norm", "config.json"), "eps"), positive=True)
        mult = _number("residual_mult", raw.get("residual_mult", 1.0))
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        for i, layer in enumerate(layers):
            _check_layer(i, layer)
        loop = raw.get("loop")
        if loop is not None:
            if not isinstance(loop, Mapping):
                raise ConfigError("'loop' must be an object with start, stop and times")
            a, b, n = (need(loop, "start"), need(loop, "stop"),
                       positive_int("loop.times", need(loop, "times")))
            if not all(isinstance(v, int) and not isinstance(v, bool) for v in (a, b)) \
                    or not 0 <= a <= b <= len(layers):
                raise ConfigError(f"loop: start..stop must lie inside the {len(layers)} layers")
            loop = (a, b, n)
        return cls(vocab, width, eps, mult, loop, tuple(copy.deepcopy(list(layers))))

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": "Pivinex", "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
               "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def layer_calls(self) -> tuple[LayerCall, ...]:
        """The layers in the order they run; every run has a cache entry of its own, and the
        first layer of each pass but the first has the embedding's output added before it."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(LayerCall(i) for i in range(n))
        a, b, times = self.loop
        calls = [LayerCall(i) for i in range(a)]
        for p in range(times):
            calls += [LayerCall(i, adds_embedding=p > 0 and i == a) for i in range(a, b)]
        return tuple(calls + [LayerCall(i) for i in range(b, n)])

    def num_parameters(self) -> int:
        return sum(math.prod(t.shape) for t in init_weights(self, 0, shapes_only=True).values())


def _norm_spec(name: str, width: int, eps: float) -> PartSpec:
    return PartSpec("layernorm", dict(width=width, eps=eps, weight=name, bias=None))


def _feed_forward_spec(p: str, width: int, mlp) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated", dict(
            width=width, inner=mlp["ff"], activation="gelu_tanh", gate_weight=p + "mlp.gate",
            up_weight=p + "mlp.up", down_weight=p + "mlp.down"))
    r = mlp["router"]
    return PartSpec("routed_experts", dict(
        width=width, ff=mlp["expert"]["ff"], experts=r["experts"], top=r["top"],
        scoring="softmax_corrected", activation="silu", router=p + "mlp.router",
        correction=p + "mlp.correction", weight_scale=float(r.get("scale", 1.0)),
        identity=r.get("identity", 0), expert_prefix=p + "mlp.e"))


def build_spec(cfg: PivinexConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        parts = dict(
            norm1=_norm_spec(p + "norm1", W, eps),
            mixer=PartSpec("latent_attention", dict(
                width=W, n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                kv_rank=m["kv_rank"], scale=m["scale"], rot_base=m["rot"]["base"],
                rot_dims=m["rot"]["dims"], eps=eps, q_weight=p + "mix.uq", q_rank=m["q_rank"],
                q_down=p + "mix.dq", q_down_norm=p + "mix.dq.norm", latent_weight=p + "mix.dkv",
                latent_norm=p + "mix.dkv.norm", key_up=p + "mix.uk", value_up=p + "mix.uv",
                sink=None, out_weight=p + "mix.o", window=m["mask"]["size"])),
            scale1=PartSpec("channel_scale", dict(width=W, weight=p + "ls1",
                                                  multiplier=cfg.residual_mult)))
        mlp = layer.get("mlp")
        if mlp is not None:
            parts["feed_forward"] = _feed_forward_spec(p, W, mlp)
            parts["scale2"] = PartSpec("channel_scale", dict(width=W, weight=p + "ls2",
                                                             multiplier=cfg.residual_mult))
        else:
            unused.append(rf"l{i}\.ls2")     # a factor without a sublayer may be in the file
        layers.append(LayerSpec("scaled_parallel", parts))
    return ModelSpec(
        name="Pivinex", vocab_size=cfg.vocab, width=W, max_positions=None,
        embedding=PartSpec("normed_token_table", dict(
            vocab_size=cfg.vocab, width=W, table="embed", eps=eps, norm_weight="embed.norm")),
        position=PartSpec("none", {}),
        layers=tuple(layers), schedule=cfg.layer_calls(),
        final_norm=_norm_spec("final.norm", W, eps),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, width=W, weight="head")),
        eos_token_id=None, ignore_tensors=tuple(unused))


def init_weights(cfg: PivinexConfig, seed: int, shapes_only: bool = False):
    """Seeded random float32 weights under the checkpoint's names, drawn from one CPU generator
    in the order the names are listed here.  Matrices ~ N(0, 1/sqrt(in)); norm weights and layer
    scales near 1; corrections of the size of the scores' differences."""
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

    W = cfg.width
    put("embed", (cfg.vocab, W), 0.5)
    put("embed.norm", (W,), 0.1, 1.0)
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        H, D, P, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        R, Q = m["kv_rank"], m["q_rank"]
        put(p + "norm1", (W,), 0.1, 1.0)
        a = p + "mix."
        put(a + "dq", (Q, W))
        put(a + "dq.norm", (Q,), 0.1, 1.0)
        put(a + "uq", (H * (D + P), Q), 1.5 / math.sqrt(Q))
        put(a + "dkv", (R + P, W))
        put(a + "dkv.norm", (R,), 0.1, 1.0)
        put(a + "uk", (H * D, R), 1.5 / math.sqrt(R))
        put(a + "uv", (H * V, R))
        put(a + "o", (W, H * V))
        put(p + "ls1", (W,), 0.2, 1.0)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        f = p + "mlp."
        if mlp["kind"] == "dense":
            put(f + "gate", (mlp["ff"], W), 1.5 / math.sqrt(W))
            put(f + "up", (mlp["ff"], W))
            put(f + "down", (W, mlp["ff"]))
        else:
            ff, r = mlp["expert"]["ff"], mlp["router"]
            n = r["experts"] + r.get("identity", 0)
            for e in range(r["experts"]):
                put(f"{f}e{e}.gate", (ff, W), 1.5 / math.sqrt(W))
                put(f"{f}e{e}.up", (ff, W))
                put(f"{f}e{e}.down", (W, ff))
            put(f + "router", (n, W), 1.5 / math.sqrt(W))
            put(f + "correction", (n,), 0.3 / n)
        put(p + "ls2", (W,), 0.2, 1.0)
    put("final.norm", (W,), 0.1, 1.0)
    put("head", (cfg.vocab, W))
    return w


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
            "q_rank": q_rank, "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim),
            "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}


def _moe(ff, experts, top, identity, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale}}


def _layers(n, mixer, dense, moe):
    """n layers: dense and routed feed-forwards in turn."""
    return [{"type": "latent_attention", "mixer": copy.deepcopy(mixer),
             "mlp": copy.deepcopy(dense if i % 2 == 0 else moe)} for i in range(n)]


def _preset(vocab, width, layers, loop=None, eps=1e-6, mult=0.5):
    out = {"architecture": "Pivinex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "residual_mult": mult, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


PRESETS: dict[str, dict] = {
    # a few hundred thousand parameters: for demonstrations and smoke runs
    "pivinex-tiny": _preset(384, 96, _layers(
        3, _latent(4, 16, 8, 24, 40, 48, 40), {"kind": "dense", "ff": 160}, _moe(48, 6, 2, 1, 1.5)),
        loop=(1, 3, 2)),
    # layer sizes of a small and a mid-sized production model, few layers: for measurements
    "pivinex-1k": _preset(32768, 1024, _layers(
        4, _latent(8, 128, 64, 128, 256, 512, 256), {"kind": "dense", "ff": 4096},
        _moe(512, 32, 4, 4, 2.0))),
    "pivinex-2k": _preset(32768, 2048, _layers(
        4, _latent(16, 128, 64, 128, 512, 1024, 256), {"kind": "dense", "ff": 8192},
        _moe(1024, 64, 6, 8, 2.0))),
}

PIVINEX = Architecture(name="Pivinex", config_cls=PivinexConfig, build_spec=build_spec,
                       init_weights=init_weights, model_types=("pivinex",), presets=PRESETS,
                       preset_aliases={})
register_architecture(PIVINEX, replace=True)
