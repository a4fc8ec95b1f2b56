"""Small Nukodra configurations for the tests, with random weights written to temporary folders,
and the plain implementation's view of the same weights."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch

import plain_nukodra


def _lat(heads, dim, rot, vdim, kv_rank, base=10000.0, scale=None, kv_from=None, rot_dims=None,
         window=None):
    out = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank,
           "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot),
           "rot": {"base": base, "dims": rot if rot_dims is None else rot_dims}}
    if kv_from is not None:
        out["kv_from"] = kv_from
    if window is not None:
        out["mask"] = {"size": window}
    return out


def _att(heads, kv_heads, dim, vdim, window, rot_dims, base=5000.0, softcap=15.0, scale=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
           "scale": scale if scale is not None else 1.0 / math.sqrt(dim),
           "rot": {"base": base, "dims": rot_dims}}
    if softcap is not None:
        out["softcap"] = softcap
    if window is not None:
        out["mask"] = {"size": window}
    return out


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
            "norm_groups": norm_groups}


def _layer(mixer, ff=None):
    kind = "mamba2" if "state" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _model(vocab, width, eps, layers, streams):
    out = {"architecture": "Nukodra", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": layers}
    if streams is not None:
        out["streams"] = streams
    return out


# sizes that are no multiple of a page (16), of 8 or of each other and differ from layer to layer;
# two readers of one layer's latents with other sizes of their own, a window that ends inside a
# page and none, values of another size than the keys, partly and wholly turned heads, grouped and
# shared state inputs, every mixer with a feed-forward and without
CASE_A = _model(307, 44, 1e-5, [
    _layer(_ssm(6, 10, 14, 2, 3, 4)),
    _layer(_lat(3, 12, 6, 20, 28, base=300.0), 52),
    _layer(_att(4, 2, 26, 18, 21, 14), 36),
    _layer(_lat(5, 10, 6, 7, 28, base=300.0, kv_from=1, scale=0.4)),
    _layer(_ssm(5, 7, 9, 1, 5, 1), 60),
    _layer(_lat(2, 14, 10, 26, 18, base=5e5, rot_dims=4), 28),
    _layer(_att(6, 1, 11, 9, None, 10, base=80.0, softcap=None)),
    _layer(_lat(4, 12, 6, 16, 28, base=300.0, kv_from=1), 40),
], 3)
# what the first case keeps apart is equal or 1 here, or absent: one copy of the stream, one head,
# equal sizes, windows of one token and of two, one tap, a state of one number, a group per head
# and a norm over the whole row, a cap and scales of 1
CASE_B = _model(257, 40, 1e-6, [
    _layer(_att(1, 1, 8, 8, 1, 8, softcap=1.0, scale=1.0), 40),
    _layer(_ssm(4, 8, 8, 4, 1, 1), 40),
    _layer(_lat(1, 8, 8, 8, 8, scale=1.0)),
    _layer(_ssm(1, 8, 1, 1, 2, 1)),
    _layer(_att(2, 2, 8, 8, 2, 2), 8),
    _layer(_lat(2, 8, 8, 8, 8, kv_from=2), 24),
], 1)
# sizes the tile kernels take, stored in bfloat16; windows on both sides of the key tiles
CASE_C = _model(512, 128, 1e-6, [
    _layer(_ssm(8, 32, 64, 2, 4, 2), 192),
    _layer(_lat(4, 64, 32, 64, 64, base=2000.0), 256),
    _layer(_att(8, 2, 64, 64, 48, 64)),
    _layer(_lat(2, 72, 32, 104, 64, base=2000.0, kv_from=1)),
    _layer(_att(4, 4, 96, 96, 200, 64, softcap=8.0), 192),
    _layer(_ssm(3, 64, 128, 1, 4, 3)),
    _layer(_lat(3, 128, 16, 128, 128, base=500.0), 128),
    _layer(_att(6, 2, 48, 48, 129, 48, softcap=None), 64),
    _layer(_lat(16, 32, 32, 32, 64, base=2000.0, kv_from=1)),
], 4)
# a plain stream without copies; a latent layer inside a window
CASE_D = _model(190, 56, 1e-5, [
    _layer(_lat(3, 16, 8, 24, 32, window=19), 48),
    _layer(_ssm(4, 12, 16, 2, 4, 3)),
    _layer(_att(4, 2, 16, 16, 37, 8), 64),
], None)

CASES = {"case_a": (CASE_A, 81), "case_b": (CASE_B, 82), "case_c": (CASE_C, 83),
         "case_d": (CASE_D, 84)}


class Case:
    def __init__(self, name, folder, config, seed):
        from hetero_serve_b200.weights import read_safetensors
        self.name, self.dir, self.config, self.seed = name, str(folder), config, seed
        self.raw = read_safetensors(Path(folder) / "model.safetensors")
        self.plain = plain_nukodra.prepare(self.raw)
        self.plain_bf16 = plain_nukodra.prepare(self.raw, round_to=torch.bfloat16)
        self.vocab = config["vocab"]
        self._memo = {}

    def logits(self, tokens, dtype="float32"):
        key = (tuple(tokens), dtype)
        if key not in self._memo:
            w = self.plain_bf16 if dtype == "bfloat16" else self.plain
            self._memo[key] = plain_nukodra.forward(self.config, w, tokens)
        return self._memo[key]

    def tokens(self, n, seed):
        g = torch.Generator().manual_seed(seed)
        return torch.randint(0, self.vocab, (n,), generator=g).tolist()


def case_of(config, folder, seed=1, dtype="float32", name="case"):
    from hetero_serve_b200.weights import write_model_dir
    write_model_dir(folder, config, seed, dtype)
    return Case(name, folder, json.loads((Path(folder) / "config.json").read_text()), seed)


def make_cases(tmp_path_factory):
    return {name: case_of(cfg, tmp_path_factory.mktemp("nukodra_" + name), seed,
                          "bfloat16" if name == "case_c" else "float32", name)
            for name, (cfg, seed) in CASES.items()}


# -- models in which ONE earlier token stands out ----------------------------------------------
# In the attention models token ASK's query and token MARK's key meet in one number of each head
# and nowhere else: every other pair scores 0 there, so an ASK query gives most of its softmax to
# an earlier MARK it can see, and a window that is one position off, a lost far key, a missing sink
# or a missing cap changes the logits by far more than any tolerance.  In the model of a recurrence
# the state hardly decays, so that a MARK hundreds of tokens back still shows.  One mixer each.
MARK, ASK = 7, 11
PLANTED = {
    # a narrow window; sizes no tile kernel takes
    "narrow": _model(97, 32, 1e-5, [_layer(_att(4, 2, 13, 9, 13, 6, softcap=20.0, scale=12 / 13.0), 40)], 2),
    # windows around the tiles of 128 keys, sizes the tile kernels take
    "wide": _model(97, 32, 1e-5, [_layer(_att(4, 1, 64, 64, 150, 32, softcap=20.0, scale=12 / 64.0), 40)], 3),
    # no window: keys far away
    "latent_odd": _model(97, 32, 1e-5, [_layer(_lat(2, 13, 6, 9, 15), 40)], 2),
    "latent": _model(97, 32, 1e-5, [_layer(_lat(2, 16, 8, 24, 32), 40)], 2),
    "memory": _model(97, 32, 1e-5, [_layer(_ssm(4, 16, 24, 2, 4, 2), 40)], 2),
}


def planted_weights(which):
    from hetero_serve_b200.config.model_config import architecture_of
    raw = PLANTED[which]
    arch = architecture_of(raw)
    cfg = arch.config_cls.from_dict(raw)
    w = arch.init_weights(cfg, 61)
    W, m, kind = raw["width"], raw["layers"][0]["mixer"], raw["layers"][0]["type"]
    w["embed"][:, :2] = 0.0                      # number 0 is MARK's alone, number 1 ASK's
    w["embed"][MARK, 0] = w["embed"][ASK, 1] = 3.0
    w["l0.norm1"] = torch.zeros(W)
    w["l0.hc1.in"].fill_(1.0 / raw["streams"])
    a = "l0.mix."
    if kind == "attention":
        D = m["dim"]
        for name, heads, number in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
            mat, bias = w[a + name].zero_(), w[a + name + ".b"].zero_()
            for hd in range(heads):
                mat[hd * D + D - 1, number] = 40.0
                bias[hd * D + D - 2 - number] = 0.3     # what every other token's vector is made of
            w[a + name + ".norm"].fill_(1.0)
        w[a + "sink"] = torch.linspace(7.0, 9.0, m["heads"])
    elif kind == "latent_attention":
        w[a + "dkv"][:, :2] = 0.0
        w[a + "dkv"][0] = 0.0
        w[a + "dkv"][0, 0] = 6.0
        w[a + "dkv.norm"].fill_(1.0)
        w[a + "q"].zero_()
        w[a + "uk"].zero_()
        strength = math.sqrt(9.0 / (m["scale"] * math.sqrt(m["kv_rank"])))
        for hd in range(m["heads"]):
            w[a + "q"][hd * (m["dim"] + m["rot_dim"]) + m["dim"] - 1, 1] = strength
            w[a + "uk"][hd * m["dim"] + m["dim"] - 1, 0] = strength
    else:
        w[a + "A_log"].fill_(-7.0)
    return cfg, w


def planted_case(tmp_path_factory, which):
    from hetero_serve_b200.weights import write_safetensors
    cfg, w = planted_weights(which)
    folder = tmp_path_factory.mktemp("nukodra_planted_" + which)
    (folder / "config.json").write_text(json.dumps(cfg.to_dict(), indent=2) + "\n")
    write_safetensors(folder / "model.safetensors", w, {"format": "pt"})
    return Case("planted_" + which, folder, json.loads((folder / "config.json").read_text()), 61)


def planted_tokens(case, mark_at, length, seed):
    """Random tokens without MARK and ASK, then MARK at ``mark_at`` and ASK as the last token."""
    t = [x if x not in (MARK, ASK) else MARK + 1 for x in case.tokens(length, seed)]
    t[mark_at] = MARK
    t[-1] = ASK
    return t


def rms_error(got, want):
    """Root mean square of the difference with its mean taken off, over the root mean square
    of the wanted row."""
    d = got.double() - want.double()
    d = d - d.mean()
    return math.sqrt(float((d * d).mean())) / max(1e-12, math.sqrt(float((want.double() ** 2).mean())))
