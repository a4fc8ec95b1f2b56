"""Small Pivinex configurations for the tests, with random weights written to temporary
folders, and the plain implementation's view of the same weights."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch

import plain_pivinex


def _lat(heads, dim, rot, vdim, kv_rank, q_rank, window, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank,
            "q_rank": q_rank, "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot),
            "mask": {"size": window}, "rot": {"base": base, "dims": rot}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, identity, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale}}


def _layer(mixer, mlp):
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def _model(vocab, width, eps, layers, mult, loop=None):
    out = {"architecture": "Pivinex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "residual_mult": mult, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# sizes that are no multiple of a page (16), of 8 or of each other and differ from layer to layer;
# every layer another window; three passes of a stretch in the middle; all feed-forwards and none
CASE_A = _model(307, 44, 1e-5, [
    _layer(_lat(3, 12, 6, 20, 28, 36, 21, base=300.0), _moe(28, 5, 2, 3, scale=1.7)),
    _layer(_lat(5, 10, 4, 7, 18, 22, 9, base=5e5, scale=0.4), _dense(52)),
    _layer(_lat(2, 14, 10, 26, 33, 19, 40), None),
    _layer(_lat(3, 12, 6, 20, 28, 36, 17, scale=0.3), _moe(20, 7, 4, 1, scale=0.6)),
], 0.8, loop=(1, 3, 3))
# what the first case keeps apart is equal or 1 here, or absent: one head, equal sizes, a window of
# one token and one of two, one expert chosen of one, every output chosen, no identity choice,
# factors of 1, a stretch from the first layer to the last that runs twice
CASE_B = _model(257, 40, 1e-6, [
    _layer(_lat(1, 8, 8, 8, 8, 8, 1, scale=1.0), _moe(24, 1, 1, 0)),
    _layer(_lat(2, 2, 2, 2, 16, 16, 2), _dense(40)),
    _layer(_lat(4, 8, 2, 8, 8, 8, 16), _moe(16, 2, 3, 1)),
], 1.0, loop=(0, 3, 2))
# sizes the wide kernels take (head parts in multiples of 8), stored in bfloat16; windows on both
# sides of a tile of 128, one wider than most portions; a stretch that is listed but runs once
CASE_C = _model(512, 128, 1e-6, [
    _layer(_lat(4, 64, 32, 64, 64, 96, 48), _moe(64, 8, 3, 2, scale=2.5)),
    _layer(_lat(2, 72, 64, 104, 96, 64, 200, base=500.0), _dense(256)),
    _layer(_lat(4, 24, 8, 40, 64, 64, 129), _moe(64, 8, 2, 0)),
    _layer(_lat(3, 128, 16, 128, 128, 128, 128), _dense(192)),
], 0.6, loop=(1, 2, 1))

CASES = {"case_a": (CASE_A, 71), "case_b": (CASE_B, 72), "case_c": (CASE_C, 73)}


class Case:
    def __init__(self, name, folder, config, seed):
        from hetero_serve_b200.weights import read_safetensors
        self.name, self.dir, self.config, self.seed = name, str(folder), config, seed
        self.raw = read_safetensors(Path(folder) / "model.safetensors")
        self.plain = plain_pivinex.prepare(self.raw)
        self.plain_bf16 = plain_pivinex.prepare(self.raw, round_to=torch.bfloat16)
        self.vocab = config["vocab"]
        self._memo = {}

    def logits(self, tokens, dtype="float32"):
        key = (tuple(tokens), dtype)
        if key not in self._memo:
            w = self.plain_bf16 if dtype == "bfloat16" else self.plain
            self._memo[key] = plain_pivinex.forward(self.config, w, tokens)
        return self._memo[key]

    def tokens(self, n, seed):
        g = torch.Generator().manual_seed(seed)
        return torch.randint(0, self.vocab, (n,), generator=g).tolist()


def case_of(config, folder, seed=1, dtype="float32", name="case"):
    from hetero_serve_b200.weights import write_model_dir
    write_model_dir(folder, config, seed, dtype)
    return Case(name, folder, json.loads((Path(folder) / "config.json").read_text()), seed)


def make_cases(tmp_path_factory):
    return {name: case_of(cfg, tmp_path_factory.mktemp("pivinex_" + name), seed,
                          "bfloat16" if name == "case_c" else "float32", name)
            for name, (cfg, seed) in CASES.items()}


# -- models in which ONE key stands out -------------------------------------------------------
# Token ASK's query and token MARK's key meet in one number of each head and nowhere else: every
# other pair of tokens scores 0 there, so an ASK query gives nearly all of its softmax to an
# earlier MARK it can see, and a window that is one position off changes the logits by far more
# than any tolerance.  One layer each: a MARK that is not visible changes nothing at all.
MARK, ASK = 7, 11
PLANTED = {
    # a narrow window; head sizes no tile kernel takes
    "narrow": _model(97, 32, 1e-5, [_layer(_lat(2, 13, 6, 9, 15, 11, 13), _dense(40))], 0.9),
    # windows around the key tiles of 128, with sizes the tile kernels take
    "wide": _model(97, 32, 1e-5, [_layer(_lat(2, 16, 8, 24, 32, 24, 150), _dense(40))], 0.9),
}


def planted_case(tmp_path_factory, which):
    from hetero_serve_b200.config.model_config import architecture_of
    from hetero_serve_b200.weights import write_safetensors
    raw = PLANTED[which]
    arch = architecture_of(raw)
    cfg = arch.config_cls.from_dict(raw)
    w = arch.init_weights(cfg, 61)
    W, m = raw["width"], raw["layers"][0]["mixer"]
    w["embed"][:, :4] = 0.0
    w["embed"][MARK, 0], w["embed"][MARK, 1] = 3.0, -3.0
    w["embed"][ASK, 2], w["embed"][ASK, 3] = 3.0, -3.0
    w["embed.norm"], w["l0.norm1"] = torch.ones(W), torch.ones(W)
    probe = torch.zeros(2, W)                       # rows that sum to 0: the norms' mean drops out
    probe[0, 0], probe[0, 1] = 1.0, -1.0
    probe[1, 2], probe[1, 3] = 1.0, -1.0
    a = "l0.mix."
    # number 0 of the query latent is there for ASK alone, number 0 of the key latent for MARK alone
    for name, row in (("dq", probe[1]), ("dkv", probe[0])):
        w[a + name][:, :4] = 0.0
        w[a + name][0] = row * 3.0
        w[a + name + ".norm"] = torch.ones_like(w[a + name + ".norm"])
    # every head's query and unrotated key look at those two numbers and at nothing else
    strength = math.sqrt(30.0 / (m["scale"] * math.sqrt(m["q_rank"] * m["kv_rank"])))
    w[a + "uq"].zero_()
    w[a + "uk"].zero_()
    for hd in range(m["heads"]):
        w[a + "uq"][hd * (m["dim"] + m["rot_dim"]) + m["dim"] - 1, 0] = strength
        w[a + "uk"][hd * m["dim"] + m["dim"] - 1, 0] = strength
    folder = tmp_path_factory.mktemp("pivinex_planted_" + which)
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
