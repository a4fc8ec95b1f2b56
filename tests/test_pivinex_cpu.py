"""Pivinex without a GPU: the configuration, the spec, the plain implementation's own sanity, and
the engine (step function, cache manager) driven with the plain twins of the kernels against the
plain model."""

import copy
import dataclasses
import io
import math

import pytest
import torch

import pivinex_cases as pc
import plain_ops
import plain_pivinex
import traces
from hetero_serve_b200.config import ConfigError
from hetero_serve_b200.config.model_config import architecture_of
from hetero_serve_b200.engine.loading import load_model
from hetero_serve_b200.engine.replay import replay
from hetero_serve_b200.engine.step import Runner, StepEntry
from hetero_serve_b200.parts import LayerCall, LayerSpec, Model, PartSpec

TOL = 1e-4          # float32 rows between the twins; logits of these models reach 3 to 5
F64 = torch.float64


def _replay(case, steps, tmp_path, max_tokens, **kw):
    out = tmp_path / "out"
    out.mkdir(exist_ok=True)
    assert replay(model_dir=case.dir, dtype="float32", out_dir=out, max_tokens=max_tokens,
                  lines=traces.lines_of(steps), report=io.StringIO(), device="cpu",
                  ops=plain_ops.PlainOps(), **kw) == 0
    return out


def _worst(case, out, index, reqs):
    got = traces.collect(out, index, case.vocab)
    return traces.worst_error(got, {r: case.logits(t) for r, t in reqs.items()})


def _runner(case, pages, slots=1):
    model, _ = load_model(case.dir, "float32", "cpu")
    return Runner(model, num_pages=pages, page_size=16, max_requests=slots, dtype=torch.float32,
                  device="cpu", ops=plain_ops.PlainOps())


# -- configuration and spec -----------------------------------------------------------------
def test_config_is_read_and_written_back(pivinex_case):
    arch = architecture_of(pivinex_case.config)
    cfg = arch.config_cls.from_dict(pivinex_case.config)
    assert arch.name == "Pivinex"
    assert arch.config_cls.from_dict(cfg.to_dict()) == cfg
    assert cfg.width == pivinex_case.config["width"]


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "do not fit"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.update(residual_mult="a"), "residual_mult"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_errors(change, message):
    cfg = copy.deepcopy(pc.CASE_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_of(cfg).config_cls.from_dict(cfg)


def test_calls_and_cache_entries_of_the_spec(pivinex_cases):
    case = pivinex_cases["case_a"]
    arch = architecture_of(case.config)
    model = Model(arch.build_spec(arch.config_cls.from_dict(case.config)))
    calls = model.schedule
    assert [c.layer for c in calls] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [c.adds_embedding for c in calls] == [False] * 3 + [True, False, True, False, False]
    assert len({c.cache for c in calls}) == 8 and model.keeps_embedding
    # one shared row a token: one head, one plane; a group per row size and window
    groups = {(g.kv_heads, g.planes, g.head_dim, g.window): len(g.entries) for g in model.cache_groups}
    assert groups == {(1, 1, 34, 21): 1, (1, 1, 22, 9): 3, (1, 1, 43, 40): 3, (1, 1, 34, 17): 1}
    assert model.state_shapes == {} and model.spec.max_positions is None
    names = model.tensor_requests()
    assert names["l0.mlp.router"].shape == (8, 44) and names["l0.mlp.router"].role == "float32"
    assert "l0.mlp.e4.up" in names and "l0.mlp.e5.up" not in names
    assert "l2.ls1" in names and "l2.ls2" not in names and "l2.mlp.gate" not in names
    assert set(names) == set(case.raw)


def test_a_checkpoint_that_does_not_fit(pivinex_cases, tmp_path):
    from pathlib import Path
    from hetero_serve_b200.weights import WeightError, write_safetensors
    case = pivinex_cases["case_a"]
    raw = {n: t for n, t in case.raw.items() if n != "l0.mlp.correction"}
    raw["l1.mix.sink"] = torch.zeros(5)
    raw["l2.ls2"] = torch.ones(44)              # a factor without its sublayer: ignored
    (tmp_path / "config.json").write_text((Path(case.dir) / "config.json").read_text())
    write_safetensors(tmp_path / "model.safetensors", raw, {"format": "pt"})
    with pytest.raises(WeightError) as err:
        load_model(tmp_path, "float32", "cpu")
    assert "l0.mlp.correction" in str(err.value) and "l1.mix.sink" in str(err.value)
    assert "l2.ls2" not in str(err.value)


# -- the plain implementation's own sanity ----------------------------------------------------
def test_plain_prefix_property(pivinex_case):
    toks = pivinex_case.tokens(70, 5)
    full, part = pivinex_case.logits(toks), pivinex_case.logits(toks[:23])
    assert (full[:23] - part).abs().max() < 1e-9


def test_plain_window_rule():
    assert [j for j in range(12) if plain_pivinex.visible(9, j, 4)] == [6, 7, 8, 9]
    assert [j for j in range(12) if plain_pivinex.visible(2, j, 4)] == [0, 1, 2]
    assert [j for j in range(12) if plain_pivinex.visible(5, j, 1)] == [5]


def test_plain_layer_runs():
    cfg = {"layers": [None] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert plain_pivinex.layer_runs(cfg) == [(0, False), (1, False), (2, False), (1, True),
                                             (2, False), (3, False)]
    assert plain_pivinex.layer_runs({"layers": [None] * 2}) == [(0, False), (1, False)]


def test_plain_rotation_keeps_lengths_and_turns_by_the_difference():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(6, generator=g, dtype=F64), torch.randn(6, generator=g, dtype=F64)
    turn = lambda v, p: plain_pivinex.rotate_pairs(v, p, 100.0)
    assert abs(float(turn(q, 9) @ turn(k, 4) - turn(q, 25) @ turn(k, 20))) < 1e-12
    assert abs(float(turn(q, 9).norm() - q.norm())) < 1e-12
    a = 3 * 100.0 ** (-2 / 6)                     # neighbours are a pair: numbers 2 and 3
    want = q[2] * math.cos(a) - q[3] * math.sin(a)
    assert abs(float(turn(q, 3)[2] - want)) < 1e-12


def test_plain_route_chooses_by_corrected_and_weighs_by_plain_scores():
    z = torch.tensor([2.0, 1.0, 0.0, -1.0], dtype=F64)
    s = torch.softmax(z, 0)
    c = torch.tensor([-0.7, 0.0, 0.0, 0.5], dtype=F64)
    chosen, wts = plain_pivinex.route(z, c, 2, 1.5)
    assert chosen.tolist() == [3, 1] and (wts - 1.5 * s[[3, 1]]).abs().max() < 1e-12


def test_plain_identity_experts_pass_the_input_through():
    g = torch.Generator().manual_seed(2)
    h = torch.randn(3, 5, generator=g, dtype=F64)
    w = {"m.router": torch.zeros(3, 5, dtype=F64), "m.correction": torch.tensor([0.0, 1.0, 2.0], dtype=F64),
         "m.e0.gate": torch.ones(4, 5, dtype=F64), "m.e0.up": torch.ones(4, 5, dtype=F64),
         "m.e0.down": torch.ones(5, 4, dtype=F64)}
    mlp = {"router": {"experts": 1, "identity": 2, "top": 2, "scale": 3.0}}
    # both choices pass the input through, each with a third of the softmax
    assert (plain_pivinex.routed_ff(h, w, "m.", mlp) - 2 * h).abs().max() < 1e-12


@pytest.mark.parametrize("which", ["narrow", "wide"])
def test_plain_visibility_of_one_key(pivinex_planted, which):
    case = pivinex_planted[which]
    size = case.config["layers"][0]["mixer"]["mask"]["size"]
    for d in (1, 2, size - 2, size - 1, size, size + 1):
        t = pc.planted_tokens(case, 3, 3 + d + 1, 3)
        blank = list(t)
        blank[3] = pc.MARK + 1
        change = float((case.logits(t)[-1] - case.logits(blank)[-1]).abs().max())
        if d < size:
            assert change > 0.5, d
        else:
            assert change == 0.0, d


# -- the engine with plain kernels -------------------------------------------------------------
@pytest.mark.parametrize("driver", ["whole", "tail", "portions"])
def test_cuts_agree_with_the_plain_model(pivinex_case, tmp_path, driver):
    reqs = {f"r{i}": pivinex_case.tokens(n, 50 + i) for i, n in enumerate((1, 2, 19, 83))}
    if driver == "whole":
        steps, index = traces.whole(reqs)
    elif driver == "tail":
        steps, index = traces.tail_one_by_one(reqs, tail=45)
    else:
        steps, index = traces.portions(reqs, sizes=(7, 2, 16, 3, 2, 5, 21))
    out = _replay(pivinex_case, steps, tmp_path, max_tokens=128)
    err, where = _worst(pivinex_case, out, index, reqs)
    assert err < TOL, (err, where)


def test_mixed_batches_reuse_pages(pivinex_case, tmp_path):
    reqs = {f"r{i}": pivinex_case.tokens(n, 70 + i) for i, n in enumerate((47, 5, 18, 66, 3, 26))}
    steps, index, peak = traces.mixed(reqs, seed=3, max_live=3, sizes=(1, 2, 5, 1, 17, 3, 1, 9))
    out = _replay(pivinex_case, steps, tmp_path, max_tokens=peak, max_requests=3)
    err, where = _worst(pivinex_case, out, index, reqs)
    assert sum(len(v) for v in index.values()) > 20 and err < TOL, (err, where)


def test_pages_behind_the_window_are_given_back(pivinex_planted):
    """A request far longer than the pool holds runs in portions: the window's pages go back to
    the pool as it advances."""
    case = pivinex_planted["narrow"]
    rn = _runner(case, pages=4)
    toks = pc.planted_tokens(case, 190, 200, 17)
    want, at = case.logits(toks), 0
    for n in (20, 13, 2, 19, 1, 1, 20, 7, 20, 20, 3, 20, 1, 20, 20, 2, 10, 1):
        res = rn.step([StepEntry("a", toks[at:at + n], want=[n - 1])])
        assert (res.logits[0].double() - want[at + n - 1]).abs().max() < TOL, at
        at += n
        assert rn.manager.pages_free(0) >= 1
    assert at == 200
    rn.manager.check()
    rn.close("a")
    assert rn.manager.pages_free(0) == rn.manager.pools[0].num_pages


@pytest.mark.parametrize("how", ["whole", "alone", "portions"])
def test_the_edges_of_the_window(pivinex_planted, how):
    """One key that takes nearly all of the softmax when it is visible, asked for from every
    distance around the window's edge and from far away: in a prompt, decoded alone, and at the
    end of a portion of two."""
    case = pivinex_planted["narrow"]
    for at in (0, 1, 15, 16):                      # a page's last and first row among them
        for d in (1, 11, 12, 13, 14, 15, 16, 17, 33, 90):
            t = pc.planted_tokens(case, at, at + d + 1, 100 + d)
            rn = _runner(case, pages=12)
            n = len(t)
            if how == "whole":
                res = rn.step([StepEntry("a", t, want=[n - 1])])
            elif how == "alone":
                rn.step([StepEntry("a", t[:-1])])
                res = rn.step([StepEntry("a", t[-1:], want=[0])])
            else:
                cut = max(1, n - 2)
                for a in range(0, cut, 7):
                    rn.step([StepEntry("a", t[a:min(cut, a + 7)])])
                res = rn.step([StepEntry("a", t[cut:], want=[n - cut - 1])])
            err = float((res.logits[-1].double() - case.logits(t)[-1]).abs().max())
            assert err < TOL, (at, d, err)


def test_long_decoding(pivinex_cases):
    case = pivinex_cases["case_b"]
    t = case.tokens(120, 9)
    rn = _runner(case, pages=12)
    rn.step([StepEntry("d", t[:3])])
    want = case.logits(t)
    for i in range(3, 120):
        res = rn.step([StepEntry("d", [t[i]], want=[0])])
        assert (res.logits[0].double() - want[i]).abs().max() < TOL, i


def test_the_parts_in_other_arrangements(pivinex_cases):
    """The same mixers and feed-forwards under one unscaled norm (each adds into the stream
    itself), a token table without a norm, and the embedding's output added again before a block
    that knows nothing of it."""
    case = pivinex_cases["case_a"]
    arch = architecture_of(case.config)
    spec = arch.build_spec(arch.config_cls.from_dict(case.config))
    layers = []
    for i in (0, 1):
        parts = {k: v for k, v in spec.layers[i].parts.items() if not k.startswith("scale")}
        layers.append(LayerSpec("parallel", parts))
    layers.append(spec.layers[3])                # a scaled block behind an unscaled one
    spec = dataclasses.replace(
        spec, layers=tuple(layers),
        embedding=PartSpec("token_table", dict(vocab_size=case.vocab, width=44, table="embed")),
        schedule=(LayerCall(0), LayerCall(1, adds_embedding=True), LayerCall(2),
                  LayerCall(2, adds_embedding=True), LayerCall(0)))
    model = Model(spec)
    model.bind({n: case.raw[n] for n in model.tensor_requests()}, torch.float32, "cpu")
    rn = Runner(model, num_pages=8, page_size=16, max_requests=1, dtype=torch.float32,
                device="cpu", ops=plain_ops.PlainOps())
    toks = case.tokens(60, 3)
    rn.step([StepEntry("a", toks[:13])])
    got = rn.step([StepEntry("a", toks[13:], want=[0, 46])]).logits.double()
    w, cfg, P = case.plain, case.config, plain_pivinex
    eps, mult, L = cfg["norm"]["eps"], cfg["residual_mult"], cfg["layers"]
    x0 = w["embed"][torch.tensor(toks)]

    def unscaled(x, i):
        h = P.layer_norm(x, w[f"l{i}.norm1"], eps)
        ff = P.dense_ff(h, w, "l1.mlp.") if i == 1 else P.routed_ff(h, w, "l0.mlp.", L[0]["mlp"])
        return x + P.latent_attention(h, w, f"l{i}.mix.", L[i]["mixer"], eps) + ff

    def scaled(x):
        h = P.layer_norm(x, w["l3.norm1"], eps)
        return x + mult * (P.latent_attention(h, w, "l3.mix.", L[3]["mixer"], eps) * w["l3.ls1"]
                           + P.routed_ff(h, w, "l3.mlp.", L[3]["mlp"]) * w["l3.ls2"])

    x = scaled(scaled(unscaled(unscaled(x0, 0) + x0, 1)) + x0)
    x = unscaled(x, 0)
    want = P.layer_norm(x, w["final.norm"], eps) @ w["head"].T
    assert (got - want[[13, 59]]).abs().max() < TOL


ORDERS = {
    "no loop": ([pc._layer(pc._lat(2, 8, 4, 6, 12, 10, 7), pc._moe(16, 3, 2, 1)),
                 pc._layer(pc._lat(2, 8, 4, 6, 12, 10, 7), pc._dense(24))], None),
    "no feed-forward anywhere": ([pc._layer(pc._lat(2, 8, 4, 6, 12, 10, 30), None)] * 2, (0, 1, 3)),
    "an empty stretch": ([pc._layer(pc._lat(1, 8, 4, 6, 12, 10, 5), pc._dense(24))] * 2, (1, 1, 4)),
    "the last layer loops": ([pc._layer(pc._lat(1, 8, 4, 6, 12, 10, 5), pc._dense(24)),
                              pc._layer(pc._lat(3, 4, 2, 10, 6, 14, 64), pc._moe(16, 2, 1, 5))], (1, 2, 4)),
    "one layer": ([pc._layer(pc._lat(2, 8, 4, 6, 12, 10, 1000), pc._dense(24))], None),
}


@pytest.mark.parametrize("which", ORDERS)
def test_other_orders_of_layers(which, tmp_path):
    layers, loop = ORDERS[which]
    folder = tmp_path / "model"
    folder.mkdir()
    case = pc.case_of(pc._model(90, 48, 1e-6, layers, 1.3, loop), folder, name=which)
    reqs = {f"r{i}": case.tokens(n, 20 + i) for i, n in enumerate((70, 9, 33))}
    steps, index, peak = traces.mixed(reqs, seed=1, max_live=2, sizes=(1, 2, 5, 1, 17, 3))
    out = _replay(case, steps, tmp_path, max_tokens=peak, max_requests=2)
    err, where = _worst(case, out, index, reqs)
    assert err < TOL, (err, where)
