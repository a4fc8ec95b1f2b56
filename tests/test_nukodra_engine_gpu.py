"""Nukodra through the engine on the GPU: the step function, the paged cache with latents that
several layers read and windowed groups, per-request states and the CUDA kernels against the plain
implementation (tests/plain_nukodra.py), in both precisions; then greedy generation through the
Python entry point and its scheduler."""

import io
import subprocess
import sys

import pytest
import torch

import nukodra_cases as nc
import plain_nukodra
import traces
from hetero_serve_b200.engine.loading import load_model
from hetero_serve_b200.engine.replay import replay
from hetero_serve_b200.engine.step import Runner, StepEntry

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
# relative root-mean-square error of a row of logits: float32 sums of a few hundred terms;
# bfloat16 rounds the rows the projections read and the cache rows to 8 bits, which these small
# deep models amplify (the plain twins, rounding at the same places, are as far off)
TOL = {"float32": 5e-5, "bfloat16": 8e-2}


def _bound(errs, dtype):
    """float32: the largest error.  bfloat16: nineteen rows in twenty and twice the median (single
    rows whose stream nearly cancels are far off while nothing is wrong)."""
    errs = sorted(errs)
    if dtype == "float32":
        return errs[-1]
    return max(errs[int(0.95 * (len(errs) - 1))], 2 * errs[len(errs) // 2]) if len(errs) > 4 \
        else errs[len(errs) // 2]


def _replay(case, dtype, steps, tmp_path, max_tokens, **kw):
    out = tmp_path / f"out_{dtype}"
    out.mkdir(exist_ok=True)
    assert replay(model_dir=case.dir, dtype=dtype, out_dir=out, max_tokens=max_tokens,
                  lines=traces.lines_of(steps), report=io.StringIO(), device=DEV, **kw) == 0
    return out


def _worst(case, dtype, out, index, reqs):
    got = traces.collect(out, index, case.vocab)
    errs = sorted(((nc.rms_error(torch.as_tensor(row), case.logits(reqs[rid], dtype)[p]),
                    (rid, p)) for (rid, p), row in got.items()), reverse=True)
    return _bound([e for e, _ in errs], dtype), errs[0][1], len(errs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("driver", ["whole", "tail", "portions"])
def test_cuts_agree_with_the_plain_model(nukodra_case, tmp_path, dtype, driver):
    reqs = {f"r{i}": nukodra_case.tokens(n, 150 + i) for i, n in enumerate((1, 2, 23, 70, 131))}
    if driver == "whole":
        steps, index = traces.whole(reqs)
    elif driver == "tail":
        steps, index = traces.tail_one_by_one(reqs, tail=50)
    else:
        steps, index = traces.portions(reqs, sizes=(24, 7, 2, 16, 3, 2, 31, 5, 2, 9))
    out = _replay(nukodra_case, dtype, steps, tmp_path, max_tokens=192)
    err, where, n = _worst(nukodra_case, dtype, out, index, reqs)
    assert n > 4 and err < TOL[dtype], (err, where)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages_and_slots(nukodra_case, tmp_path, dtype):
    reqs = {f"r{i}": nukodra_case.tokens(n, 170 + i) for i, n in
            enumerate((90, 9, 64, 23, 70, 3, 55, 31, 2))}
    steps, index, peak = traces.mixed(reqs, seed=2)
    out = _replay(nukodra_case, dtype, steps, tmp_path, max_tokens=peak, max_requests=4)
    err, where, n = _worst(nukodra_case, dtype, out, index, reqs)
    assert n > 40 and err < TOL[dtype], (err, where)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_wide_sizes_and_long_prompts(nukodra_cases, tmp_path, dtype):
    """Sizes the tensor-core kernels take, prompts and portions longer and shorter than the
    windows, the tiles and the recurrence's chunks, stored in bfloat16; then portions beside
    single tokens of others."""
    case = nukodra_cases["case_c"]
    reqs = {"a": case.tokens(400, 301), "b": case.tokens(150, 302), "c": case.tokens(9, 303)}
    steps, index = traces.whole(reqs)
    out = _replay(case, dtype, steps, tmp_path, max_tokens=448)
    err, where, n = _worst(case, dtype, out, index, reqs)
    assert n > 200 and err < TOL[dtype], (err, where)
    steps, index = traces.portions(reqs, sizes=(70, 2, 133, 1, 17))
    out = _replay(case, dtype, steps, tmp_path, max_tokens=448)
    err, where, n = _worst(case, dtype, out, index, reqs)
    assert err < TOL[dtype], (err, where)
    steps, index, peak = traces.mixed(reqs, seed=5, sizes=(1, 90, 2, 1, 130, 5, 1, 3, 64))
    out = _replay(case, dtype, steps, tmp_path, max_tokens=peak)
    err, where, n = _worst(case, dtype, out, index, reqs)
    assert err < TOL[dtype], (err, where)


def _runner(case, dtype="float32", pages=16, slots=4, **kw):
    model, _ = load_model(case.dir, dtype, DEV)
    return Runner(model, num_pages=pages, page_size=16, max_requests=slots, dtype=model.dtype,
                  device=DEV, **kw)


def test_a_request_alone_and_in_a_batch(nukodra_case):
    """The logits of a request do not depend on its neighbours in the batch, nor on the slot and
    pages it got.  (In float32 to the order of additions: a step of few tokens splits each
    token's keys over more blocks.)"""
    case = nukodra_case
    a, b, c = case.tokens(45, 1), case.tokens(20, 2), case.tokens(33, 3)
    alone = _runner(case)
    want = alone.step([StepEntry("a", a[:30], want=[29])]).logits.clone()
    want2 = alone.step([StepEntry("a", a[30:], want=[0, 14])]).logits.clone()
    rn = _runner(case)
    rn.step([StepEntry("c", c)])                  # takes the first slot and pages
    got = rn.step([StepEntry("b", b[:7]), StepEntry("a", a[:30], want=[29]),
                   StepEntry("c", [5])]).logits.clone()
    rn.close("c")
    got2 = rn.step([StepEntry("a", a[30:], want=[0, 14]), StepEntry("b", b[7:])]).logits
    for x, y in ((got[0], want[0]), (got2[0], want2[0]), (got2[1], want2[1])):
        assert nc.rms_error(x.cpu(), y.cpu()) < 5e-6
    assert nc.rms_error(got2[1].cpu(), case.logits(a)[44]) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["case_a", "memory"])
def test_freed_pages_and_slots_start_clean(nukodra_cases, nukodra_planted, name, dtype):
    case = nukodra_cases.get(name) or nukodra_planted[name]
    rn = _runner(case, dtype, pages=8, slots=1)
    for seed, n in ((4, 100), (5, 41), (6, 3), (7, 110)):
        t = case.tokens(n, seed)
        rn.step([StepEntry("x", t[:n // 2])])
        res = rn.step([StepEntry("x", t[n // 2:], want=[n - n // 2 - 1])])
        assert nc.rms_error(res.logits[0].cpu(), case.logits(t, dtype)[n - 1]) < TOL[dtype], seed
        rn.close("x")
    rn.manager.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "alone", "portions"])
@pytest.mark.parametrize("which", ["narrow", "wide", "latent", "latent_odd", "memory"])
def test_one_token_from_every_distance(nukodra_planted, which, dtype, how):
    """One token that takes most of what a query sees when it is visible, asked for from every
    distance around the window's edge and from far away, on a page's last and first row and on a
    tile's."""
    case = nukodra_planted[which]
    size = case.config["layers"][0]["mixer"].get("mask", {}).get("size", 64)
    rn = _runner(case, dtype, pages=64, slots=2)
    k = 0
    for at in (0, 15, 16, 120):
        for d in (1, 5, size - 2, size - 1, size, size + 1, size + 2, 127, 128, 129, 400):
            t = nc.planted_tokens(case, at, at + d + 1, 100 + d)
            n, rid = len(t), f"q{k}"
            k += 1
            if how == "whole":
                res = rn.step([StepEntry(rid, t, want=[n - 1])])
            elif how == "alone":
                rn.step([StepEntry(rid, t[:-1])])
                res = rn.step([StepEntry(rid, t[-1:], want=[0])])
            else:
                cut = max(1, n - 2 - 5 * (k % 2))         # a portion of two, or of seven
                for a in range(0, cut, 70):
                    rn.step([StepEntry(rid, t[a:min(cut, a + 70)])])
                res = rn.step([StepEntry(rid, t[cut:], want=[n - cut - 1])])
            rn.close(rid)
            err = nc.rms_error(res.logits[-1].cpu(), case.logits(t, dtype)[-1])
            assert err < TOL[dtype], (at, d, err)
    rn.manager.check()


@pytest.mark.parametrize("name, dtype", [("case_a", "float32"), ("case_c", "bfloat16"),
                                         ("memory", "bfloat16")])
def test_long_decoding(nukodra_cases, nukodra_planted, name, dtype):
    """Single-token steps across many window and page borders, the pages behind the windows
    going back to the pool."""
    case = nukodra_cases.get(name) or nukodra_planted[name]
    n = 280
    t = case.tokens(n, 9)
    rn = _runner(case, dtype, pages=20, slots=1)
    rn.step([StepEntry("d", t[:12])])
    want = case.logits(t, dtype)
    errs = []
    for i in range(12, n):
        res = rn.step([StepEntry("d", [t[i]], want=[0])])
        if i % 5 in (0, 4) or i % 16 == 0 or i > 270:
            errs.append(nc.rms_error(res.logits[0].cpu(), want[i]))
    assert _bound(errs, dtype) < TOL[dtype]
    rn.manager.check()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_captured_steps_equal_eager_steps(nukodra_cases, dtype):
    """The same steps through CUDA graphs (sizes rounded up to a class, padding rows, states set
    back after the run that precedes a capture) and launched one by one."""
    case = nukodra_cases["case_c"]
    a, b = case.tokens(340, 401), case.tokens(30, 402)
    eager, graphs = _runner(case, dtype, pages=64), _runner(case, dtype, pages=64, cuda_graphs=True)
    plan = [[("a", a[:100], [99])], [("a", a[100:120], [0, 19]), ("b", b[:1], [0])],
            [("a", a[120:121], [0]), ("b", b[1:2], [0])], [("a", a[121:122], [0]), ("b", b[2:3], [0])],
            [("a", a[122:340], [17, 217]), ("b", b[3:4], [0])], [("a2", a[:100], [99])]]
    for step in plan:
        want = eager.step([StepEntry(r, t, w) for r, t, w in step]).logits.clone()
        got = graphs.step([StepEntry(r, t, w) for r, t, w in step]).logits.clone()
        for i in range(want.shape[0]):
            assert nc.rms_error(got[i].cpu(), want[i].cpu()) < (2e-2 if dtype == "bfloat16" else 1e-5), step[0][0]
    assert nc.rms_error(want[0].cpu(), case.logits(a, dtype)[99]) < TOL[dtype]


def _greedy(case, prompt, n):
    toks, out, margins = list(prompt), [], []
    for _ in range(n):
        row = plain_nukodra.forward(case.config, case.plain, toks)[-1]
        top = torch.topk(row, 2).values
        margins.append(float(top[0] - top[1]))
        out.append(int(row.argmax()))
        toks.append(out[-1])
    return out, margins


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_entry_point(nukodra_case, graphs):
    """Prompts of unequal length, cut into portions by a small token budget, decoded side by
    side by the scheduler; the tokens are the plain model's greedy tokens."""
    from hetero_serve_b200 import LLMEngine
    case = nukodra_case
    prompts = [case.tokens(n, 200 + n) for n in (37, 5, 18)]
    eng = LLMEngine(case.dir, dtype="float32", num_blocks=24, max_batch=4, max_prefill_tokens=16,
                    policy="mixed", cuda_graphs=graphs, device=DEV)
    got = eng.generate(prompts, max_new_tokens=12)
    for p, g in zip(prompts, got):
        want, margins = _greedy(case, p, 12)
        for i, (a, b, m) in enumerate(zip(g, want, margins)):
            if m < 1e-3:
                break                                         # a close call: stop comparing
            assert a == b, (len(p), i, g, want)
    eng.runner.manager.check()


def test_command_line_runs_a_preset():
    out = subprocess.run([sys.executable, "-m", "hetero_serve_b200", "--model", "nukodra-tiny",
                          "--random-prompts", "2:12", "--max-new-tokens", "4"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]


ORDERS = {
    "recurrences alone": ([nc._layer(nc._ssm(4, 32, 64, 2, 4, 2), 96), nc._layer(nc._ssm(2, 96, 16, 1, 2, 4))], 5),
    "latents alone": ([nc._layer(nc._lat(2, 16, 8, 24, 32)), nc._layer(nc._lat(3, 24, 8, 40, 32, kv_from=0), 64),
                       nc._layer(nc._lat(17, 8, 8, 8, 32, kv_from=0))], 2),
    "windows alone": ([nc._layer(nc._att(4, 1, 32, 32, 9, 32), 64), nc._layer(nc._att(2, 2, 128, 64, 130, 64)),
                       nc._layer(nc._att(20, 1, 64, 64, None, 0))], 3),
    "a plain stream": ([nc._layer(nc._ssm(4, 32, 48, 4, 4, 1), 64), nc._layer(nc._lat(2, 16, 8, 24, 32)),
                        nc._layer(nc._lat(2, 16, 8, 24, 32, kv_from=1))], None),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ORDERS)
def test_other_orders_of_layers(which, dtype, tmp_path):
    layers, streams = ORDERS[which]
    folder = tmp_path / "model"
    folder.mkdir()
    case = nc.case_of(nc._model(90, 64, 1e-6, layers, streams), folder, name=which)
    reqs = {f"r{i}": case.tokens(n, 20 + i) for i, n in enumerate((70, 9, 33, 150))}
    steps, index, peak = traces.mixed(reqs, seed=1, max_live=3)
    out = _replay(case, dtype, steps, tmp_path, max_tokens=peak, max_requests=3)
    err, where, n = _worst(case, dtype, out, index, reqs)
    assert n > 10 and err < TOL[dtype], (err, where)
