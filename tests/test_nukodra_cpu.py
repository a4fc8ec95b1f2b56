"""Nukodra without a GPU: the configuration, the spec, the plain implementation's own sanity, and
the engine (step function, cache manager) driven with the plain twins of the kernels against the
plain model."""

import copy
import dataclasses
import io
import math

import pytest
import torch

import nukodra_cases as nc
import plain_nukodra as P
import plain_ops
import traces
from hetero_serve_b200.config import ConfigError
from hetero_serve_b200.config.model_config import architecture_of
from hetero_serve_b200.engine.loading import load_model
from hetero_serve_b200.engine.replay import replay
from hetero_serve_b200.engine.step import Runner, StepEntry
from hetero_serve_b200.parts import LayerCall, LayerSpec, Model, PartSpec

TOL = 1e-4          # float32 rows between the twins; logits of these models reach 5 to 20
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
@pytest.mark.parametrize("name", nc.CASES)
def test_config_is_read_and_written_back(nukodra_cases, name):
    config = nukodra_cases[name].config
    arch = architecture_of(config)
    cfg = arch.config_cls.from_dict(config)
    assert arch.name == "Nukodra"
    assert arch.config_cls.from_dict(cfg.to_dict()) == cfg
    assert all(config[k] == v for k, v in cfg.to_dict().items())
    assert cfg.width == config["width"] and cfg.streams == config.get("streams")
    assert cfg.num_parameters() == sum(t.numel() for t in nukodra_cases[name].raw.values())


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=28), "rot.dims"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][7]["mixer"].update(kv_from=5), "must equal"),
    (lambda c: c["layers"][7]["mixer"]["rot"].update(base=10.0), "must equal"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "dense"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(streams=99), "streams"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_config_errors(change, message):
    cfg = copy.deepcopy(nc.CASE_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        architecture_of(cfg).config_cls.from_dict(cfg)


def test_calls_and_cache_entries_of_the_spec(nukodra_cases):
    case = nukodra_cases["case_a"]
    arch = architecture_of(case.config)
    model = Model(arch.build_spec(arch.config_cls.from_dict(case.config)))
    calls = model.schedule
    assert [c.layer for c in calls] == list(range(8))
    assert [c.writes_cache for c in calls] == [True, True, True, False, True, True, True, False]
    assert calls[3].cache == calls[1].cache == calls[7].cache
    groups = {(g.kv_heads, g.planes, g.head_dim, g.window): len(g.entries) for g in model.cache_groups}
    assert groups == {(1, 1, 34, 0): 1, (2, 1, 44, 21): 1, (1, 1, 28, 0): 1, (1, 1, 20, 0): 1}
    # states and, behind them, a ring of the convolutions' inputs
    assert model.state_shapes == {0: (6 * 14 * 10 + 3 * (60 + 56),), 4: (5 * 9 * 7 + 5 * (35 + 18),)}
    assert set(model.tensor_requests()) == set(case.raw)
    assert model.tensor_requests()["l0.mix.conv"].role == "float32"
    assert model.counts_prompt_rows


def test_a_checkpoint_that_does_not_fit(nukodra_cases, tmp_path):
    from pathlib import Path
    from hetero_serve_b200.weights import WeightError, write_safetensors
    case = nukodra_cases["case_a"]
    raw = {n: t for n, t in case.raw.items() if n not in ("l2.mix.sink", "l1.hc2.mix")}
    raw["l3.mix.dkv"] = torch.zeros(34, 44)            # a layer that reads another's latents
    raw["l0.mix.conv"] = raw["l0.mix.conv"][:, :2].contiguous()
    (tmp_path / "config.json").write_text((Path(case.dir) / "config.json").read_text())
    write_safetensors(tmp_path / "model.safetensors", raw, {"format": "pt"})
    with pytest.raises(WeightError) as err:
        load_model(tmp_path, "float32", "cpu")
    for name in ("l2.mix.sink", "l1.hc2.mix", "l3.mix.dkv", "l0.mix.conv"):
        assert name in str(err.value)


# -- the plain implementation's own sanity ----------------------------------------------------
def test_plain_prefix_property(nukodra_case):
    toks = nukodra_case.tokens(70, 5)
    full, part = nukodra_case.logits(toks), nukodra_case.logits(toks[:23])
    assert (full[:23] - part).abs().max() < 1e-9


def test_plain_window_rule():
    assert [j for j in range(12) if P.visible(9, j, 4)] == [6, 7, 8, 9]
    assert [j for j in range(12) if P.visible(2, j, 4)] == [0, 1, 2]
    assert [j for j in range(12) if P.visible(5, j, 1)] == [5]
    assert [j for j in range(12) if P.visible(3, j, 0)] == [0, 1, 2, 3]


def test_plain_rotation_turns_by_the_difference_and_pairs_halves():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(9, generator=g, dtype=F64), torch.randn(9, generator=g, dtype=F64)
    turn = lambda v, p: P.rotate_halves(v, p, 100.0, 6)
    assert abs(float(turn(q, 9) @ turn(k, 4) - turn(q, 25) @ turn(k, 20))) < 1e-12
    a = 3 * 100.0 ** (-2 / 6)                     # number 1 is paired with number 4
    assert abs(float(turn(q, 3)[1] - (q[1] * math.cos(a) - q[4] * math.sin(a)))) < 1e-12
    assert torch.equal(turn(q, 3)[6:], q[6:])


def test_plain_cap_and_sink():
    """Two visible keys of equal score: each weighs 1 / (2 + e^(sink - score)), the score capped
    and the sink not."""
    q, k = torch.full((2, 1, 1), 2.0, dtype=F64), torch.ones(2, 1, 1, dtype=F64)
    v = torch.tensor([[[1.0]], [[3.0]]], dtype=F64)
    s = 1.5 * math.tanh(6.0 / 1.5)
    out = P.softmax_over_visible(q, k, v, 3.0, 0, 1.5, torch.tensor([2.0], dtype=F64))
    assert abs(float(out[1, 0, 0]) - 4.0 / (2.0 + math.exp(2.0 - s))) < 1e-12
    assert abs(float(P.softmax_over_visible(q, k, v, 3.0)[1, 0, 0]) - 2.0) < 1e-12


def test_plain_row_norm_is_over_all_heads():
    w = {"p.q": torch.eye(4, dtype=F64), "p.k": torch.eye(4, dtype=F64)[:2]}
    h = torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=F64)
    u = P.unit_rms(h, 0.0)
    assert abs(float(u[0, 1]) - 4.0 / 2.5) < 1e-12 and w["p.q"].shape == (4, 4)


def test_plain_state_space_is_a_decaying_sum():
    g = torch.Generator().manual_seed(3)
    T, H, V, G, N = 7, 4, 3, 2, 5
    x, B, C = (torch.randn(T, n, d, generator=g, dtype=F64) for n, d in ((H, V), (G, N), (G, N)))
    dt, a_log = torch.rand(T, H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64)
    D = torch.randn(H, generator=g, dtype=F64)
    y, S = P.state_space(x, B, C, dt, a_log, D, torch.tensor([0, 0, 1, 1]))
    t, h = 6, 2
    want = D[h] * x[t, h]
    for s in range(t + 1):
        decay = math.exp(-math.exp(float(a_log[h])) * float(dt[s + 1:t + 1, h].sum()))
        want = want + decay * dt[s, h] * float(B[s, 1] @ C[t, 1]) * x[s, h]
    assert (y[t, h] - want).abs().max() < 1e-12
    y2, S2 = P.state_space(x[4:], B[4:], C[4:], dt[4:], a_log, D, torch.tensor([0, 0, 1, 1]),
                           P.state_space(x[:4], B[:4], C[:4], dt[:4], a_log, D,
                                         torch.tensor([0, 0, 1, 1]))[1])
    assert (y2 - y[4:]).abs().max() < 1e-12 and (S2 - S).abs().max() < 1e-12


def test_plain_short_conv():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    out = P.short_conv(x, torch.tensor([[3.0, 2.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert out[:, 0].tolist() == [2.5, 23.5, 230.5]


def test_plain_connection_mixes_from_the_old_copies():
    X = torch.tensor([1.0, 10.0], dtype=F64).view(2, 1, 1)
    w = {"c.in": torch.tensor([2.0, 0.1], dtype=F64), "c.out": torch.tensor([1.0, -1.0], dtype=F64),
         "c.mix": torch.tensor([[0.0, 5.0], [1.0, 0.0]], dtype=F64)}      # [from, to]
    out = P.connect(X, w, "c.", lambda u: u * 100)
    assert out.view(-1).tolist() == [10.0 + 300.0, 5.0 - 300.0]


@pytest.mark.parametrize("which", ["narrow", "wide", "latent", "latent_odd", "memory"])
def test_plain_visibility_of_one_token(nukodra_planted, which):
    case = nukodra_planted[which]
    size = case.config["layers"][0]["mixer"].get("mask", {}).get("size", 10 ** 9)
    for d in (1, 2, 11, 12, 13, 14, 148, 149, 150, 151, 400):
        t = nc.planted_tokens(case, 3, 3 + d + 1, 3)
        blank = list(t)
        blank[3] = nc.MARK + 1
        change = float((case.logits(t)[-1] - case.logits(blank)[-1]).abs().max())
        if d < size:
            assert change > 0.02, (d, change)
        else:
            assert change == 0.0, d


# -- the engine with plain kernels -------------------------------------------------------------
@pytest.mark.parametrize("driver", ["whole", "tail", "portions"])
def test_cuts_agree_with_the_plain_model(nukodra_case, tmp_path, driver):
    reqs = {f"r{i}": nukodra_case.tokens(n, 50 + i) for i, n in enumerate((1, 2, 19, 83))}
    if driver == "whole":
        steps, index = traces.whole(reqs)
    elif driver == "tail":
        steps, index = traces.tail_one_by_one(reqs, tail=45)
    else:
        steps, index = traces.portions(reqs, sizes=(7, 2, 16, 3, 2, 5, 21))
    out = _replay(nukodra_case, steps, tmp_path, max_tokens=128)
    err, where = _worst(nukodra_case, out, index, reqs)
    assert err < TOL, (err, where)


def test_mixed_batches_reuse_pages_and_slots(nukodra_case, tmp_path):
    reqs = {f"r{i}": nukodra_case.tokens(n, 70 + i) for i, n in enumerate((47, 5, 18, 66, 3, 26))}
    steps, index, peak = traces.mixed(reqs, seed=3, max_live=3, sizes=(1, 2, 5, 1, 17, 3, 1, 9))
    out = _replay(nukodra_case, steps, tmp_path, max_tokens=peak, max_requests=3)
    err, where = _worst(nukodra_case, out, index, reqs)
    assert sum(len(v) for v in index.values()) > 20 and err < TOL, (err, where)


def test_a_slot_is_cleared_for_its_next_owner(nukodra_planted):
    """The recurrence hardly forgets here: a state or convolution input left by the request before
    would show."""
    case = nukodra_planted["memory"]
    rn = _runner(case, pages=8)
    for seed, n in ((4, 30), (5, 2), (6, 41)):
        t = nc.planted_tokens(case, n // 2, n, seed)
        rn.step([StepEntry("x", t[:n - 1])])
        res = rn.step([StepEntry("x", t[n - 1:], want=[0])])
        assert (res.logits[0].double() - case.logits(t)[-1]).abs().max() < TOL, seed
        rn.close("x")
    rn.manager.check()


def test_pages_behind_the_window_are_given_back(nukodra_planted):
    """A request far longer than the pool holds runs in portions: the window's pages go back to
    the pool as it advances."""
    case = nukodra_planted["narrow"]
    rn = _runner(case, pages=4)
    toks = nc.planted_tokens(case, 190, 200, 17)
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
@pytest.mark.parametrize("which", ["narrow", "latent_odd", "memory"])
def test_one_token_from_every_distance(nukodra_planted, which, how):
    """One token that takes most of what a query sees when it is visible, asked for from every
    distance around the window's edge and from far away: in a prompt, decoded alone, and at the
    end of a portion of two."""
    case = nukodra_planted[which]
    for at in (0, 1, 15, 16):                      # a page's last and first row among them
        for d in (1, 11, 12, 13, 14, 15, 16, 17, 33, 90):
            t = nc.planted_tokens(case, at, at + d + 1, 100 + d)
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


def test_long_decoding(nukodra_cases):
    case = nukodra_cases["case_b"]
    t = case.tokens(120, 9)
    rn = _runner(case, pages=12)
    rn.step([StepEntry("d", t[:3])])
    want = case.logits(t)
    for i in range(3, 120):
        res = rn.step([StepEntry("d", [t[i]], want=[0])])
        assert (res.logits[0].double() - want[i]).abs().max() < TOL, i


def test_the_parts_in_other_arrangements(nukodra_cases):
    """Copies of the stream that live for a stretch of layers only: connected blocks between plain
    ones, the embedding's output added again in the middle of a stretch, a norm whose rows the
    connecting launch does not form, and mixers that add into the stream themselves."""
    case = nukodra_cases["case_a"]
    arch = architecture_of(case.config)
    spec = arch.build_spec(arch.config_cls.from_dict(case.config))
    L = spec.layers
    plain = lambda i: LayerSpec("pre_norm", {k: v for k, v in L[i].parts.items()
                                             if not k.startswith("connect")})
    layernorm = PartSpec("layernorm", dict(width=44, eps=1e-5, weight="l5.norm1", bias=None))
    other = LayerSpec("hyper_connected", dict(L[5].parts, norm1=layernorm))
    spec = dataclasses.replace(
        spec, layers=(plain(2), L[0], L[1], plain(4), other),
        schedule=(LayerCall(0), LayerCall(1), LayerCall(2), LayerCall(4), LayerCall(3),
                  LayerCall(4), LayerCall(1, adds_embedding=True), LayerCall(2)))
    model = Model(spec)
    model.bind({n: case.raw[n] for n in model.tensor_requests()}, torch.float32, "cpu")
    rn = Runner(model, num_pages=20, page_size=16, max_requests=1, dtype=torch.float32,
                device="cpu", ops=plain_ops.PlainOps())
    toks = case.tokens(40, 3)
    rn.step([StepEntry("a", toks[:13])])
    got = rn.step([StepEntry("a", toks[13:], want=[0, 26])]).logits.double()
    w, cfg = case.plain, case.config
    eps, layers = cfg["norm"]["eps"], cfg["layers"]

    def sublayers(i, norm1=P.layer_rms):
        p, m, kind = f"l{i}.", layers[i]["mixer"], layers[i]["type"]

        def mixer(u):
            h = norm1(u, w[p + "norm1"], eps)
            if kind == "latent_attention":
                return P.latent_attention(h, w, p + "mix.", m, P.latent_rows(h, w, p + "mix.", m, eps))
            return (P.window_attention if kind == "attention" else P.mamba2)(h, w, p + "mix.", m, eps)
        yield "hc1.", mixer
        if layers[i]["mlp"]:
            yield "hc2.", lambda u: P.dense_ff(P.layer_rms(u, w[p + "norm2"], eps), w, p + "mlp.")

    def ln(u, weight, e):
        d = u - u.mean(-1, keepdim=True)
        return d / torch.sqrt((d * d).mean(-1, keepdim=True) + 1e-5) * weight

    def stretch(x, *runs):
        X = x[None].repeat(3, 1, 1)
        for i in runs:
            for q, f in sublayers(i, ln if i == 5 else P.layer_rms):
                X = P.connect(X, w, f"l{i}.{q}", f)
        return X.sum(0)

    def unconnected(x, i):
        for _q, f in sublayers(i):
            x = x + f(x)
        return x

    x0 = w["embed"][torch.tensor(toks)]
    x = stretch(unconnected(x0, 2), 0, 1, 5)
    x = stretch(unconnected(x, 4), 5) + x0
    x = stretch(x, 0, 1)
    want = P.layer_rms(x, w["final.norm"], eps) @ w["embed"].T
    assert (got - want[[13, 39]]).abs().max() < TOL


ORDERS = {
    "recurrences alone": ([nc._layer(nc._ssm(4, 8, 12, 2, 4, 2)), nc._layer(nc._ssm(2, 10, 6, 1, 2, 4), 24)], 5),
    "latents alone": ([nc._layer(nc._lat(2, 8, 4, 6, 12)), nc._layer(nc._lat(3, 6, 4, 10, 12, kv_from=0), 24),
                       nc._layer(nc._lat(1, 4, 4, 5, 12, kv_from=0))], 2),
    "windows alone": ([nc._layer(nc._att(2, 1, 8, 6, 7, 4), 16), nc._layer(nc._att(2, 2, 8, 6, 30, 8)),
                       nc._layer(nc._att(4, 2, 6, 10, 1000, 0))], 3),
    "a plain stream": ([nc._layer(nc._ssm(4, 8, 12, 2, 4, 2), 24), nc._layer(nc._lat(2, 8, 4, 6, 12)),
                        nc._layer(nc._lat(2, 8, 4, 6, 12, kv_from=1))], None),
    "one layer": ([nc._layer(nc._att(2, 1, 8, 6, 5, 4))], 16),
}


@pytest.mark.parametrize("which", ORDERS)
def test_other_orders_of_layers(which, tmp_path):
    layers, streams = ORDERS[which]
    folder = tmp_path / "model"
    folder.mkdir()
    case = nc.case_of(nc._model(90, 48, 1e-6, layers, streams), folder, name=which)
    reqs = {f"r{i}": case.tokens(n, 20 + i) for i, n in enumerate((70, 9, 33))}
    steps, index, peak = traces.mixed(reqs, seed=1, max_live=2, sizes=(1, 2, 5, 1, 17, 3))
    out = _replay(case, steps, tmp_path, max_tokens=peak, max_requests=2)
    err, where = _worst(case, out, index, reqs)
    assert err < TOL, (err, where)
