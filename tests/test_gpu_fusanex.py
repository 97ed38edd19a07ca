"""Fusanex on the device against its plain statement (tests/plain_fusanex.py, float64, whole sequences).

Whole models: the residual after every layer; every way of cutting the work (whole prompts, a tail decoded token by token,
portions down to two tokens and one, mixed batches whose pages and state slots are used again), bit for bit against one
another in 32-bit; long decoding; decoding from captured graphs; batches of unequal requests against each alone; one key far back
or at a page's border that decides the logits; greedy generation through the scheduler; the trace runner.  Mechanisms alone: norms in
groups of one residual with several branches folded in, head norms with gains and a temperature, the gated recurrence (all
forms of its gates and of its walk, a write far back read much later), blends of neighbouring tokens and their products,
the recurrence with a bonus, the router's correction and renormalised weights, identity experts.
"""
import copy
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_fusanex as plain
import traces
from fusanex_configs import CONFIGS, shaped_weights, write_folder, write_tensors
from helpers import folder_weights, max_diff

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def runner_for(folder, dtype, page_size, pages, slots=4, poison=True):
    from wllm_b200.config import EngineConfig
    from wllm_b200.engine import build_model, build_runner
    eng = EngineConfig(dtype=dtype, block_size=page_size, max_num_seqs=slots)
    return build_runner(build_model(folder, eng.dtype, eng.device), eng, num_pages=pages, poison_pages=poison)


def plain_rows(folder, name, reqs):
    w = {k: v.double() for k, v in folder_weights(folder).items()}
    return {(rid, p): row.float() for rid, toks in reqs.items() for p, row in enumerate(plain.forward(CONFIGS[name], w, toks))}


def close_enough(rows, ref, dtype, what=""):
    """32-bit: every logit within 2e-4 of the logits' scale.  bfloat16: every row's root-mean-square difference against the
    rows' scale: the typical row within 1.5 %, 97 of 100 rows within 6 % (where two experts' scores nearly tie, the rounded
    input may choose the other one, in any implementation: single rows far off, about one in a hundred with these weights)."""
    assert set(rows) == set(ref)
    scale = max(1.0, max(float(r.abs().max()) for r in ref.values()))
    if dtype == torch.float32:
        assert max_diff(rows, ref) < 2e-4 * scale, what
        return
    rms = math.sqrt(sum(float(r.double().pow(2).mean()) for r in ref.values()) / len(ref))
    rel = sorted(float((rows[k].double() - ref[k].double()).pow(2).mean().sqrt()) / rms for k in ref)
    assert rel[len(rel) // 2] < 0.015 and rel[int(0.97 * len(rel))] < 0.06, (what, rel[len(rel) // 2], rel[int(0.97 * len(rel))], rel[-1])


def requests_of(name, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


@pytest.fixture(scope="module")
def setups(tmp_path_factory):
    out = {}
    for name in CONFIGS:
        folder = write_folder(str(tmp_path_factory.mktemp("fusanex") / name), name)
        reqs = requests_of(name, (5, 64, 31, 90, 2, 47, 70, 25, 1, 113, 17), seed=3)
        out[name] = (folder, reqs, plain_rows(folder, name, reqs))
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_residual_after_every_layer(setups, name, dtype):
    from wllm_b200.engine import StepEntry
    folder, reqs, _ = setups[name]
    toks = reqs["r3"]
    w = {k: v.double() for k, v in folder_weights(folder).items()}
    want = []
    plain.forward(CONFIGS[name], w, toks, want)
    runner = runner_for(folder, dtype, 16, 8)
    model, got = runner.model, []

    class Watched:
        def __init__(self, block):
            self.block = block

        def __getattr__(self, key):
            return getattr(self.block, key)

        def __call__(self, residual, ctx, cache):
            self.block(residual, ctx, cache)
            got.append((residual.stream + residual.pending.materialize(ctx, "watched_branch")).double().cpu())
    blocks = model.blocks
    model.blocks = [Watched(b) for b in blocks]
    rc = runner.cache.open("x")
    runner.step([StepEntry(rc, toks, [0])])
    model.blocks = blocks
    assert len(got) == len(CONFIGS[name]["layers"])
    for run, (a, b) in enumerate(zip(got, want)):
        tol = (2e-5 if dtype == torch.float32 else 0.03) * float(b.abs().max())
        worst = (a - b).abs().amax(-1).sort().values
        # (bfloat16 is judged by rows: where two experts' scores nearly tie, the rounded input may choose the other one)
        at = len(worst) - 1 if dtype == torch.float32 else int(0.9 * len(worst))
        assert worst[at] < tol, (run, float(worst[at]), float(worst[-1]), tol)


CUTS = (("whole", traces.whole), ("tail", lambda r: traces.tail_singly(r, 16)), ("portions", traces.portions),
        ("mixed", lambda r: traces.mixed(r, seed=5)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cut_matches_the_plain_statement(setups, name, dtype):
    folder, reqs, ref = setups[name]
    first = None
    for cut, make in CUTS:
        steps = make(reqs)
        pages = -(-traces.peak_tokens(steps) // 16)
        runner = runner_for(folder, dtype, 16, pages)       # four state slots for eleven requests: slots are used again
        rows = traces.run_in_process(runner, steps)
        close_enough(rows, ref, dtype, cut)
        assert all(f == pages for f in runner.cache.free_pages())
        if cut == "mixed":      # pages were used again
            assert all(g.pool.takes > pages for g in runner.cache.groups if g.spec.window is None) and len(reqs) > 4
        if dtype == torch.float32:
            if first is None:
                first = rows
            else:
                bad = sorted(k for k in first if not torch.equal(first[k], rows[k]))
                assert not bad, f"{cut}: first differing (request, position) {bad[0]}"


@pytest.mark.parametrize("page", [32, 64])
def test_other_page_sizes_give_the_same_rows(setups, page):
    folder, reqs, ref = setups["mixed"]
    steps = traces.mixed(reqs, seed=9)
    runner = runner_for(folder, torch.float32, page, -(-traces.peak_tokens(steps, page if page > 64 else 64) // page))
    close_enough(traces.run_in_process(runner, steps), ref, torch.float32, f"pages of {page}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_long_prompts_and_long_decoding(setups, name, dtype):
    """A prompt long enough for segments and runs side by side, in one step and in portions; and most of it decoded token by token."""
    from wllm_b200.kernels import ops
    folder = setups[name][0]
    reqs = requests_of(name, (330,), seed=8)
    assert 330 >= 2 * ops.RGLRU_RUNS_FROM and ops.linattn_segment_plan(330, 1, 2, 64)[1] > 2
    ref = plain_rows(folder, name, reqs)
    for cut, steps in (("whole", traces.whole(reqs)), ("portions", traces.portions(reqs, sizes=(140, 2, 131, 1, 37))), ("decoded", traces.tail_singly(reqs, 190))):
        runner = runner_for(folder, dtype, 16, 21)
        close_enough(traces.run_in_process(runner, steps), ref, dtype, cut)
        assert all(f == 21 for f in runner.cache.free_pages())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_batch_of_unequal_requests_gives_each_its_own_rows(setups, dtype):
    """Single tokens of some beside a long and two short portions, then all of them decoding together, against each alone."""
    from wllm_b200.engine import StepEntry
    folder = setups["heads64"][0]
    reqs = requests_of("heads64", (40, 170, 3, 66), seed=12)
    ref = plain_rows(folder, "heads64", reqs)
    runner = runner_for(folder, dtype, 16, 40)
    rc = {k: runner.cache.open(k) for k in reqs}
    plan = [{"r0": 30}, {"r0": 1, "r1": 150, "r2": 2, "r3": 60}, {"r0": 1, "r1": 1, "r2": 1, "r3": 1}] + [{"r0": 1, "r1": 1, "r3": 1}] * 5 + \
        [{"r0": 2, "r1": 10}, {"r1": 3}]
    rows, pos = {}, dict.fromkeys(reqs, 0)
    for step in plan:
        logits = runner.step([StepEntry(rc[k], reqs[k][pos[k]:pos[k] + c], list(range(c))) for k, c in step.items()]).float().cpu()
        at = 0
        for k, c in step.items():
            rows.update({(k, pos[k] + i): logits[at + i] for i in range(c)})
            at, pos[k] = at + c, pos[k] + c
    close_enough(rows, {k: v for k, v in ref.items() if k in rows}, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "heads64"])
def test_a_far_key_decides(tmp_path, name, dtype):
    """One token's key is made to lie along one other token's query, with a score scale that gives it all the weight: where it stands
    (at the start, at page and chunk borders, far back, just before) the last token's logits follow it, in a prompt and decoded alone.
    The gated recurrences and the time mixing keep what they are; only the attention of the first pair of mixers is shaped."""
    from wllm_b200.engine import StepEntry
    cfg = copy.deepcopy(CONFIGS[name])
    tensors = shaped_weights(cfg, 77)
    at = next(i for i, l in enumerate(cfg["layers"]) if l["type"] == "parallel")
    cfg["layers"] = [cfg["layers"][at]]
    tensors = {k.replace(f"l{at}.", "l0."): v for k, v in tensors.items() if k.startswith(f"l{at}.") or not k.startswith("l")}
    left = cfg["layers"][0]["mixer"]["left"]
    left["scale"] = 2.0
    W, V, D = cfg["width"], cfg["vocab"], left["dim"]
    marked, asking = 7, 11
    g = torch.Generator().manual_seed(3)
    tensors["embed"] = torch.randn(V, W, generator=g) * 0.1
    tensors["embed"][:, :2] = 0.0
    tensors["embed"][marked] = 0.0
    tensors["embed"][marked, 0] = 3.0
    tensors["embed"][asking] = 0.0
    tensors["embed"][asking, 1] = 3.0
    tensors["l0.norm1"] = torch.ones(W)
    direction = torch.randn(D, generator=g)
    tensors["l0.mix.left.q"][:, 1] = direction.repeat(left["heads"]) * 3
    tensors["l0.mix.left.k"][:, 0] = direction.repeat(left.get("kv_heads", left["heads"])) * 3
    for k in ("l0.mix.left.q.norm", "l0.mix.left.k.norm"):
        tensors[k] = torch.ones(D)
    folder = write_tensors(str(tmp_path / "m"), cfg, tensors)
    w = {k: v.double() for k, v in folder_weights(folder).items()}
    n = 200
    base = torch.randint(20, V, (n,), generator=g).tolist()
    base[-1] = asking
    plain_base = plain.forward(cfg, w, base)[-1]
    runner = runner_for(folder, dtype, 16, 14)
    tol = 2e-4 if dtype == torch.float32 else 0.05
    decided = 0
    for place in (0, 1, 15, 16, 17, 63, 64, 127, 128, 191, 192, n - 2):
        toks = list(base)
        toks[place] = marked
        want = plain.forward(cfg, w, toks)[-1]
        decided += int((want - plain_base).abs().max() > 0.2 * float(plain_base.abs().max()))
        scale = max(1.0, float(want.abs().max()))
        for cuts in ([n], [n - 1, 1], [place + 1, n - 1 - place], [70, 2, n - 73, 1]):
            rc = runner.cache.open("x")
            pos = 0
            for c in cuts:
                last = runner.step([StepEntry(rc, toks[pos:pos + c], [c - 1])])
                pos += c
            runner.cache.close(rc)
            assert (last[0].double().cpu() - want).abs().max() < tol * scale, (place, cuts)
    assert decided >= 10


def test_decoding_from_captured_graphs_gives_the_eager_rows(setups):
    folder, reqs, ref = setups["mixed"]
    some = {k: reqs[k] for k in ("r1", "r2", "r5")}
    steps = traces.tail_singly(some, 30)
    rows = {}
    for graphs in (False, True):
        runner = runner_for(folder, torch.float32, 16, -(-traces.peak_tokens(steps) // 16), poison=False)
        assert runner.model.graph_safe
        if graphs:
            runner.enable_graphs()
        rows[graphs] = traces.run_in_process(runner, steps)
        assert (runner.graph_launches > 0) == graphs
        close_enough(rows[graphs], {k: v for k, v in ref.items() if k[0] in some}, torch.float32)
    bad = sorted(k for k in rows[False] if not torch.equal(rows[False][k], rows[True][k]))
    assert not bad, f"first differing (request, position) {bad[0]}"


def test_greedy_generation_through_the_scheduler(setups):
    from wllm_b200 import LLM, SamplingParams
    folder, reqs, _ = setups["mixed"]
    w = {k: v.double() for k, v in folder_weights(folder).items()}
    prompts = [reqs["r0"], reqs["r2"], reqs["r3"][:40], reqs["r8"]]
    llm = LLM(folder, dtype="float32", block_size=16, num_blocks=12, chunked_prefill_tokens=24, max_num_seqs=3)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True))
    for prompt, o in zip(prompts, outs):
        toks = list(prompt)
        for _ in range(30):
            toks.append(int(plain.forward(CONFIGS["mixed"], w, toks)[-1].argmax()))
        assert o.token_ids == toks[len(prompt):]
    assert all(f == 12 for f in llm.runner.cache.free_pages())
    bf = LLM(folder, dtype="bfloat16", block_size=16, num_blocks=12, chunked_prefill_tokens=24, max_num_seqs=3, cuda_graphs=True)
    assert [len(o.token_ids) for o in bf.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))] == [10] * 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_trace_runner_replays_a_mixed_trace(setups, tmp_path, dtype):
    folder, reqs, ref = setups["heads64"]
    steps = traces.mixed(reqs, seed=11)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                           "--max-tokens", str(traces.peak_tokens(steps))], input="".join(json.dumps(s) + "\n" for s in steps),
                          capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    rows, pos = {}, {}
    V = CONFIGS["heads64"]["vocab"]
    for s in steps:
        keys = []
        for e in s["entries"]:
            p = pos.get(e["id"], 0)
            keys += [(e["id"], p + w) for w in e["want"]]
            pos[e["id"]] = p + len(e["tokens"])
        data = np.fromfile(str(out / f"{s['step']}.f32"), dtype="<f4").reshape(len(keys), V)
        rows.update({k: torch.from_numpy(r.copy()) for k, r in zip(keys, data)})
    close_enough(rows, ref, torch.float32 if dtype == "float32" else torch.bfloat16)


# ------------------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------------------
def step_arrays(lens, slots, first):
    """The step's index arrays for requests that bring `lens` tokens, hold `slots` and stand at positions `first`."""
    ints = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    return SimpleNamespace(positions=ints([p + i for n, p in zip(lens, first) for i in range(n)]),
                           token_req=ints([r for r, n in enumerate(lens) for _ in range(n)]),
                           req_q_start=ints([sum(lens[:i]) for i in range(len(lens))]), req_q_len=ints(lens), req_slot=ints(slots))


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,groups", [(64, 4), (50, 5), (2048, 1), (4096, 8), (90, 90), (6144, 3)])
def test_norms_in_groups_with_branches_folded_in(H, groups, out_dtype):
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(H)
    n, eps = 21, 1e-5
    resid = torch.randn(n, H, generator=g) * torch.logspace(-2, 2, groups).repeat_interleave(H // groups)[torch.randperm(H, generator=g)]
    a, b = torch.randn(n, H, generator=g).to(out_dtype), torch.randn(5, n, H, generator=g)
    c = torch.randn(n, H, generator=g)
    w1, w2 = (1 + 0.3 * torch.randn(H, generator=g)).to(torch.bfloat16), (1 + 0.3 * torch.randn(H, generator=g)).to(torch.bfloat16)
    terms = [(a, 0, 0.6), (b, 5, -0.5), (c, 0, 1.0)]
    sums = [a.double(), b.double().sum(0), c.double()]
    rows = torch.tensor([20, 0, 7], dtype=torch.int32)
    for count in (0, 1, 2, 3):
        want = resid.double() + sum(f * t for (_, _, f), t in zip(terms[:count], sums[:count]))
        r = resid.clone().to(DEV)
        outs = [torch.empty(n, H, dtype=out_dtype, device=DEV) for _ in range(2)]
        dev = [(t.to(DEV), p, f) for t, p, f in terms[:count]]
        picked = torch.empty(3, H, dtype=out_dtype, device=DEV)
        ops.fold_norm(r, dev, [w1.to(DEV)], eps, [picked], groups=groups, rows=rows.to(DEV))
        assert torch.equal(r.cpu(), resid)                      # read at some rows: nothing is written back
        ops.fold_norm(r, dev, [w1.to(DEV), w2.to(DEV)], eps, outs, groups=groups)
        assert (r.cpu().double() - want).abs().max() < 1e-5 * float(want.abs().max())
        for o, w in zip(outs, (w1, w2)):
            ref = plain.group_norm(want, w.double(), groups, eps)
            assert (o.cpu().double() - ref).abs().max() < (5e-5 if out_dtype == torch.float32 else 1e-2) * float(ref.abs().max())
        assert torch.equal(picked.cpu(), outs[0].cpu()[rows.long()])
        only = resid.clone().to(DEV)
        ops.fold_norm(only, dev, [], 0.0, [], groups=1)
        assert torch.equal(only, r)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 0), (5, 1, 10, 6, 0), (2, 2, 64, 64, 32), (3, 1, 96, 96, 0), (2, 1, 256, 128, 64)])
def test_head_norms_with_gains_and_a_temperature(sizes, dtype):
    """Gains in front of the turn, values divided by their root mean square, queries times the factor of their position at both sides of
    every step of it; few tokens and many (the 16-byte path), partial sums, heads held with zeros behind them."""
    from wllm_b200.kernels import ops
    nq, nkv, hd_file, vd_file, rot = sizes
    hd, vd = -(-hd_file // 8) * 8, -(-vd_file // 8) * 8
    g = torch.Generator().manual_seed(hd_file)
    n, ps, eps, every, coef = 300, 16, 1e-5, 7, 0.8
    def padded(x, heads, size, to):
        out = x.new_zeros((x.shape[0], heads, to))
        out[:, :, :size] = x.view(x.shape[0], heads, size)
        return out.view(x.shape[0], heads * to)
    qf, kf, vf = torch.randn(n, nq * hd_file, generator=g), torch.randn(n, nkv * hd_file, generator=g), torch.randn(n, nkv * vd_file, generator=g) * 3
    gq, gk = (1 + 0.3 * torch.randn(hd_file, generator=g)).to(dtype), (1 + 0.3 * torch.randn(hd_file, generator=g)).to(dtype)
    fused = torch.cat([padded(qf, nq, hd_file, hd), padded(kf, nkv, hd_file, hd), padded(vf, nkv, vd_file, vd)], 1)
    positions = torch.arange(n) + 3
    inv = torch.tensor([50.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)])
    slots = torch.randperm(n + 20, generator=g)[:n].int()
    gains = [padded(x[None], 1, hd_file, hd)[0].contiguous().to(DEV) for x in (gq, gk)]
    def turned(x):                       # [n, heads, size], pairs (j, j + rot / 2)
        if not rot:
            return x
        ang = positions.double()[:, None, None] * inv.double()
        a, b, rest = x[..., :rot // 2], x[..., rot // 2:rot], x[..., rot:]
        return torch.cat([a * ang.cos() - b * ang.sin(), b * ang.cos() + a * ang.sin(), rest], -1)
    for parts, m in ((0, n), (3, n), (0, 40)):
        src = fused.to(dtype) if not parts else torch.randn(parts, n, fused.shape[1], generator=g)
        if parts:
            src[-1] = fused - src[:-1].sum(0)
        exact = (src.double() if not parts else src.double().sum(0))[:m]
        q, k, v = exact[:, :nq * hd], exact[:, nq * hd:(nq + nkv) * hd], exact[:, (nq + nkv) * hd:]
        pos_m = positions[:m]
        unpad = lambda x, heads, size, to: x.reshape(m, heads, to)[..., :size]
        temp = plain.temperature(pos_m, every, coef, torch.float64)[:, None, None]
        save, positions = positions, pos_m
        want_q = turned(plain.rms(unpad(q, nq, hd_file, hd), eps) * gq.double()) * temp
        want_k = turned(plain.rms(unpad(k, nkv, hd_file, hd), eps) * gk.double())
        want_v = plain.rms(unpad(v, nkv, vd_file, vd), eps)
        positions = save
        pages = -(-(n + 20) // ps)
        kp, vp = torch.zeros(pages, nkv, ps, hd, dtype=dtype, device=DEV), torch.zeros(pages, nkv, ps, vd, dtype=dtype, device=DEV)
        qo = torch.empty(m, nq * hd, dtype=dtype, device=DEV)
        dev = src[..., :m, :].contiguous().to(DEV)
        ops.rope_head_norm_kv_write(dev, qo, pos_m.int().to(DEV), slots[:m].to(DEV), inv.to(DEV), kp, vp, nq, nkv, hd, rot, ps, eps, *gains,
                                    hd_file, vd_file, True, coef, every, in_splits=parts, vd=vd)
        tol = (1e-5 if rot else 3e-6) if dtype == torch.float32 else 0.01         # (angles of some hundred radians are 32-bit)
        got_q = qo.cpu().double().view(m, nq, hd)
        assert (got_q[..., :hd_file] - want_q).abs().max() < tol * float(want_q.abs().max()) and float(got_q[..., hd_file:].abs().sum()) == 0.0
        at = slots[:m].long()
        got_k, got_v = (x.cpu().double()[at // ps, :, at % ps] for x in (kp, vp))
        assert (got_k[..., :hd_file] - want_k).abs().max() < tol * float(want_k.abs().max())
        assert (got_v[..., :vd_file] - want_v).abs().max() < tol * float(want_v.abs().max())
        # without gains, temperature and normed values: the plain unit norm
        ops.rope_head_norm_kv_write(dev, qo, pos_m.int().to(DEV), slots[:m].to(DEV), inv.to(DEV), kp, vp, nq, nkv, hd, rot, ps, eps, None, None,
                                    hd_file, vd_file, False, 0.0, 0, in_splits=parts, vd=vd)
        save, positions = positions, pos_m
        bare = turned(plain.rms(unpad(q, nq, hd_file, hd), eps))
        positions = save
        assert (qo.cpu().double().view(m, nq, hd)[..., :hd_file] - bare).abs().max() < tol * float(bare.abs().max())
        got_v = vp.cpu().double()[at // ps, :, at % ps]
        assert (got_v - v.reshape(m, nkv, vd)).abs().max() < tol * float(v.abs().max())


def lru_unit(W, B, T, g, dtype):
    """Weights of a gated recurrence, and the same for the kernels."""
    s = W // B
    w = {"conv": torch.randn(W, T, generator=g) * 0.5, "conv.b": torch.randn(W, generator=g) * 0.3, "x.b": torch.randn(W, generator=g) * 0.3,
         "y.b": torch.randn(W, generator=g) * 0.3, "ra": torch.randn(B, s, s, generator=g) / s ** 0.5, "ri": torch.randn(B, s, s, generator=g) / s ** 0.5,
         "ra.b": torch.randn(B, s, generator=g), "ri.b": torch.randn(B, s, generator=g), "lam": torch.rand(W, generator=g) * 7 - 8}
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    dev = lambda k: w[k].reshape(-1).contiguous().to(DEV)
    unit = dict(x_bias=dev("x.b"), y_bias=dev("y.b"), conv_bias=dev("conv.b"), taps=w["conv"].t().contiguous().to(DEV))
    maps = torch.cat([w["ra"], w["ri"]], 1)
    gates = dict(maps=(torch.cat([maps, maps], 2) if dtype == torch.bfloat16 else maps).to(dtype).contiguous().to(DEV), ra_bias=dev("ra.b"),
                 ri_bias=dev("ri.b"), rate=(8.0 * torch.nn.functional.softplus(w["lam"].double())).float().to(DEV))
    return w, unit, gates


def plain_lru(w, y, x):
    """What the output projection reads, and the state behind every token: [n, W] each."""
    w = {k: v.double() for k, v in w.items()}
    u = plain.short_conv(x + w["x.b"], w["conv"], w["conv.b"])
    S = plain.lru(u, plain.block_gate(u, w["ra"], w["ra.b"]), plain.block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return S * plain.gelu_tanh(y + w["y.b"]), S


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,B,T", [(48, 3, 4), (30, 3, 2), (21, 1, 5), (160, 1, 1), (256, 2, 4), (144, 2, 3)])
def test_the_gated_recurrence_across_portions_and_slots(W, B, T, dtype):
    """Three requests in slots of a pool of six, in steps that cut them anywhere: portions shorter than the taps, single tokens (the one
    kernel for them, and those for portions, which must agree), the gates' maps on the grouped product, long portions as runs side by side.  One early input is a hundred
    times the others and the slowest channels forget a few thousandths of their state in a hundred tokens, so it still shows at the end.
    The slots of nobody stay as they were."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(W * T)
    w, unit, gates = lru_unit(W, B, T, g, dtype)
    off = -(-W // 8) * 8
    unit.update(y_off=0, x_off=off)
    total = [330, 150, 9]
    inputs = [torch.randn(n, 2 * off, generator=g) for n in total]
    inputs[0][3, off:] *= 100
    inputs = [x.to(dtype) for x in inputs]
    want = [plain_lru(w, x.double()[:, :W], x.double()[:, off:off + W]) for x in inputs]
    tame = inputs[0].double().clone()
    tame[3, off:] /= 100
    without = plain_lru(w, tame[:, :W], tame[:, off:off + W])[1][-1]
    assert float((want[0][1][-1] - without).abs().max()) > 0.1                    # the early write still shows at the end
    slots = [4, 0, 2]
    results = {}
    for cut, calls in (("portions", [(5, 2, 1), (1, 1, 0), (2, 3, 2), (150, 130, 0), (1, 1, 1), (130, 2, 3), (1, 11, 1), (40, 0, 1)]),
                       ("singly", [(300, 140, 1)] + [(1, 1, 1)] * 8 + [(1, 1, 0)] * 2 + [(20, 0, 0)])):
        ring, state = torch.zeros(6, T, W, device=DEV), torch.zeros(6, W, device=DEV)
        ring[[1, 3, 5]] = float("nan")
        state[[1, 3, 5]] = float("nan")
        pos = [0, 0, 0]
        outs = [[] for _ in total]
        for lens in calls:
            lens = [min(n, t - p) for n, t, p in zip(lens, total, pos)]
            live = [r for r in range(3) if lens[r] > 0]
            ctx = step_arrays([lens[r] for r in live], [slots[r] for r in live], [pos[r] for r in live])
            rows = torch.cat([inputs[r][pos[r]:pos[r] + lens[r]] for r in live])
            n = rows.shape[0]
            forms = [(rows.to(DEV), 0)]
            parts = torch.randn(3, n, 2 * off, generator=g)
            parts[-1] = rows.float() - parts[:-1].sum(0)
            forms.append((parts.to(DEV), 3))
            answers = []
            for fused, p in forms:
                ways = ["pairs"] + (["step"] if max(lens) == 1 and ops.rglru_step_ok(gates, fused, off) else []) + \
                    (["grouped"] if ops.rglru_grouped_ok(gates, fused, off) else [])
                for way in ways:
                    for long in {max(lens) >= ops.RGLRU_RUNS_FROM, way == "grouped"}:
                        rg, st, out = ring.clone(), state.clone(), torch.empty(n, W, dtype=dtype, device=DEV)
                        if way == "step":
                            ops.rglru_step(fused, p, unit, gates, ctx, rg, st, out)
                        elif way == "pairs":
                            ab = torch.empty(n, W, 2, device=DEV)
                            ops.rglru_gates(fused, p, unit, gates, ctx, rg, ab)
                            ops.rglru_scan(fused, p, unit, gates, ctx, rg, ab, st, out, long)
                        else:
                            uv, z = torch.empty(B * n, 2 * W // B, dtype=dtype, device=DEV), torch.empty(B * n, 2 * W // B, device=DEV)
                            ops.rglru_gate_sums(fused, p, unit, gates, ctx, rg, uv, torch.empty(1 + 3 * ops.moe_row_tiles(B * n, B), dtype=torch.int32, device=DEV), z)
                            ops.rglru_scan(fused, p, unit, gates, ctx, rg, (z, uv), st, out, long)
                        answers.append((out, rg, st))
            for out, rg, st in answers[1:]:
                tol = 2e-4 if dtype == torch.float32 else 0.02
                big = max(1.0, float(answers[0][0].abs().max()))
                assert (out.float() - answers[0][0].float()).abs().max() < tol * big
                assert (st[slots] - answers[0][2][slots]).abs().max() < 1e-3 * max(1.0, float(answers[0][2][slots].abs().max()))
            out, ring, state = answers[0]
            at = 0
            for r in live:
                outs[r].append(out[at:at + lens[r]].cpu().double())
                at += lens[r]
                pos[r] += lens[r]
        for r in range(3):
            got = torch.cat(outs[r])
            ref, S = want[r][0][:got.shape[0]], want[r][1][:got.shape[0]]
            tol = 2e-5 if dtype == torch.float32 else 0.01
            assert (got - ref).abs().max() < tol * max(1.0, float(ref.abs().max())), (cut, r)
            assert (state[slots[r]].cpu().double() - S[-1]).abs().max() < (2e-5 if dtype == torch.float32 else 1e-3) * max(1.0, float(S.abs().max()))
        assert pos[0] > 300 and bool(torch.isnan(ring[[1, 3, 5]]).all()) and bool(torch.isnan(state[[1, 3, 5]]).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H", [64, 50, 1032])
def test_blends_of_neighbouring_tokens_across_portions(H, dtype):
    """Portions of one, two and more tokens, both parities, slots of a pool, a request that rests for a step; the table of row tiles."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(H)
    mu = torch.rand(5, H, generator=g)
    total, slots = [60, 41, 10], [3, 1, 0]
    rows = [torch.randn(n, H, generator=g).to(dtype) for n in total]
    want = [[x.double() + (torch.cat([torch.zeros(1, H), x.float()[:-1]]).double() - x.double()) * mu[s].double() for s in range(5)] for x in rows]
    kept = torch.full((5, 2, H), float("nan"), dtype=dtype, device=DEV)
    pos = [0, 0, 0]
    for lens in [(1, 4, 0), (2, 1, 1), (0, 2, 2), (17, 1, 1), (1, 1, 1), (2, 30, 0), (1, 0, 3), (30, 2, 2), (3, 0, 0)]:
        lens = [min(n, t - p) for n, t, p in zip(lens, total, pos)]
        live = [r for r in range(3) if lens[r] > 0]
        ctx = step_arrays([lens[r] for r in live], [slots[r] for r in live], [pos[r] for r in live])
        h = torch.cat([rows[r][pos[r]:pos[r] + lens[r]] for r in live]).to(DEV)
        n = h.shape[0]
        out = torch.empty(5, n, H, dtype=dtype, device=DEV)
        tiles = torch.empty(1 + 3 * 4 * -(-n // 128), dtype=torch.int32, device=DEV)
        before = kept.clone()
        ops.token_blend(h, mu.to(DEV), ctx, kept, out, tiles, 4)
        assert tiles.tolist() == [4] + [v for s in range(4) for v in (s, s * n, n)]
        if dtype == torch.bfloat16 and max(lens) == 1 and H % 8 == 0:
            # the products of a step of single tokens: segments of any number of rows, one of them on the row itself
            segments = [(37, -1), (64, 0), (5, 3), (33, 4)]
            w = torch.randn(sum(r for r, _ in segments), H, generator=g).to(dtype)
            fused, also = torch.empty(n, w.shape[0], device=DEV), before
            ops.blended_product(h, mu.to(DEV), w.to(DEV), segments, ctx, also, fused)
            assert torch.equal(torch.nan_to_num(also), torch.nan_to_num(kept))
            at = 0
            for r, s in segments:
                x = h if s < 0 else out[s]
                ref = x.cpu().double() @ w[at:at + r].double().T
                assert (fused[:, at:at + r].cpu().double() - ref).abs().max() < 1e-4 * max(1.0, float(ref.abs().max()))
                at += r
        at = 0
        for r in live:
            for s in range(5):
                d = (out[s, at:at + lens[r]].cpu().double() - want[r][s][pos[r]:pos[r] + lens[r]]).abs().max()
                assert d < (1e-6 if dtype == torch.float32 else 0.02), (lens, r, s)
            at += lens[r]
            pos[r] += lens[r]
    assert bool(torch.isnan(kept[[2, 4]].float()).all())            # slots of nobody


@pytest.mark.parametrize("n,H", [(1, 256), (8, 2048), (9, 1032), (16, 64), (17, 3000), (32, 4096), (32, 8)])
def test_products_of_blends_of_many_sizes(n, H):
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    mu = torch.rand(5, H, generator=g)
    h, kept = torch.randn(n, H, generator=g).bfloat16(), torch.randn(n + 2, 2, H, generator=g).bfloat16()
    first = [int(v) for v in torch.randint(0, 4, (n,), generator=g)]
    slots = torch.randperm(n + 2, generator=g)[:n].tolist()
    ctx = step_arrays([1] * n, slots, first)
    ctx.req_q_len[n // 2] = 0 if n > 1 else 1              # a padded request of a captured step: it leaves no trace
    segments = [(40, -1), (96, 0), (96, 1), (31, 4)]
    w = torch.randn(sum(r for r, _ in segments), H, generator=g).bfloat16()
    fused, kd = torch.empty(n, w.shape[0], device=DEV), kept.clone().to(DEV)
    ops.blended_product(h.to(DEV), mu.to(DEV), w.to(DEV), segments, ctx, kd, fused)
    before = torch.stack([kept[s, (p - 1) & 1] if p > 0 else torch.zeros(H).bfloat16() for s, p in zip(slots, first)]).double()
    at = 0
    live = [i for i in range(n) if n == 1 or i != n // 2]
    for r, s in segments:
        x = h.double() if s < 0 else (h.double() + (before - h.double()) * mu[s].double()).bfloat16().double()
        ref = x @ w[at:at + r].double().T
        err = (fused[:, at:at + r].cpu().double() - ref)[live].abs().max()
        assert err < 0.02 * max(1.0, float(ref.abs().max())), (r, s, float(err))
        at += r
    want = kept.clone()
    for i in live:
        want[slots[i], first[i] & 1] = h[i]
    assert torch.equal(kd.cpu(), want)


@pytest.mark.parametrize("H,D", [(2, 24), (3, 10), (1, 64), (2, 128)])
def test_the_recurrence_with_a_bonus(H, D):
    """Across steps and as segments side by side, on columns of wider rows; a large write far back through a channel that forgets slowly;
    the bonus large enough to tell a token's own key and value from the others."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(D)
    n, wide = 260, 3 * H * D + 8
    rows = torch.randn(n, wide, generator=g)
    rows[2, H * D:2 * H * D] *= 30
    r, k, v = (rows[:, i * H * D:(i + 1) * H * D] for i in range(3))
    rank = {24: 9, 10: 5, 64: 16, 128: 64}[D]
    low = torch.randn(n, rank + 3, generator=g)
    w2, b2 = torch.randn(H * D, rank, generator=g) * (9 / rank) ** 0.5, torch.rand(H * D, generator=g) * 8 - 8
    bonus = torch.randn(H * D, generator=g) * 4
    decay = torch.exp(-torch.exp(torch.tanh(low[:, 2:2 + rank].double()) @ w2.double().T + b2.double()))
    shaped = lambda t: t.double().view(n, H, D)
    want = plain.time_mix(shaped(r), shaped(k), shaped(v), shaped(decay), bonus.double().view(H, D)).reshape(n, H * D)
    dev = rows.to(DEV)
    rd, kd, vd = (dev[:, i * H * D:(i + 1) * H * D] for i in range(3))
    dd = ops.linattn_decay(low.to(DEV), 0, 2, w2.to(DEV), b2.to(DEV), H, D, torch.empty(n, H * D, device=DEV))
    assert (dd.cpu().double() + 1 - decay).abs().max() < 1e-6
    if rank % 8 == 0:          # many tokens, bfloat16 maps: the tensor-core form, from one tensor and from partial sums
        wb, bb = w2.bfloat16(), b2.bfloat16()
        ref = torch.expm1(-torch.exp(torch.tanh(low[:, 2:2 + rank].double()) @ wb.double().T + bb.double()))
        slabs = torch.randn(3, n, rank + 3, generator=g)
        slabs[-1] = low - slabs[:-1].sum(0)
        for src, parts in ((low, 0), (slabs, 3)):
            for m in (n, 70, 20):
                got = ops.linattn_decay(src[..., :m, :].contiguous().to(DEV), parts, 2, wb.to(DEV), bb.to(DEV), H, D, torch.empty(m, H * D, device=DEV))
                assert ((got.cpu().double() - ref[:m]) / ref[:m]).abs().max() < 2e-3, (parts, m)
    small = decay > 0.999
    assert bool(small.any()) and ((dd.cpu().double() - (decay - 1))[small] / (decay - 1)[small]).abs().max() < 1e-5     # relative to itself
    for cuts, seg in (([n], 0), ([n], 32), ([100, 1, 2, 157], 0), ([130, 130], 48)):
        state, o = torch.zeros(3, H, D, D, device=DEV), torch.empty(n, H * D, device=DEV)
        at = 0
        for c in cuts:
            ctx = step_arrays([c], [1], [at])
            max_seg = -(-c // seg) if seg else 1
            ops.linattn_scan(rd[at:at + c], kd[at:at + c], vd[at:at + c], dd[at:at + c].contiguous(), None, state, o[at:at + c], ctx.req_q_start, ctx.req_q_len,
                             ctx.req_slot, H, D, D, seg if max_seg > 1 else 0, max_seg, torch.empty(max_seg * H * D * D, device=DEV),
                             torch.empty(max_seg * H * D, device=DEV), bonus=bonus.to(DEV))
            at += c
        assert (o.cpu().double() - want).abs().max() < 2e-5 * float(want.abs().max()), cuts
        assert float(state[[0, 2]].abs().max()) == 0.0


def test_head_norm_and_gate_with_a_gain_of_the_whole_row():
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    n, H, V = 19, 3, 20
    o, gate, w = torch.randn(n, H * V, generator=g), torch.randn(n, 5 + H * V, generator=g), torch.randn(H * V, generator=g)
    wide = torch.full((n, H * V + 12), 7.0, device=DEV)
    ops.head_gate_norm(o.to(DEV), gate.to(DEV), 0, 5, w.to(DEV), 1e-6, wide[:, 4:4 + H * V], H, V, -1.5)
    ref = plain.rms(o.double().view(n, H, V), 1e-6).reshape(n, H * V) * w.double() * plain.silu(gate[:, 5:].double()) * -1.5
    assert (wide[:, 4:4 + H * V].cpu().double() - ref).abs().max() < 1e-5
    assert bool((wide[:, :4] == 7).all()) and bool((wide[:, 4 + H * V:] == 7).all())


@pytest.mark.parametrize("n", [1, 37, 1100])
def test_the_router_with_a_correction_and_weights_over_their_sum(n):
    """Corrections that reorder the choice (also to scores below zero and above one), weights of the uncorrected scores over their sum; with
    groups of experts too."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    H, E, top = 96, 12, 3
    x, wr = torch.randn(n, H, generator=g), torch.randn(E, H, generator=g) * 0.2
    corr = torch.randn(E, generator=g) * 0.7
    s = torch.softmax(x.double() @ wr.double().T, -1)
    for groups, kept in ((1, 1), (4, 2)):
        c = s + corr.double()
        if kept < groups:
            best = c.view(n, groups, -1).max(-1).values
            keep = torch.zeros(n, groups, dtype=torch.bool).scatter(1, best.topk(kept).indices, True)
            c = c.masked_fill(~keep.repeat_interleave(E // groups, 1), float("-inf"))
        idx = c.topk(top).indices
        val = torch.gather(s, 1, idx)
        val = val / (val.sum(-1, keepdim=True) + 1e-20)
        assert not torch.equal(idx, s.topk(top).indices)
        chosen, weights = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
        ops.moe_route(x.to(DEV), wr.to(DEV), None, chosen, weights, None, groups, kept, correction=corr.to(DEV), renorm_eps=1e-20)
        assert torch.equal(chosen.cpu().long(), idx) and (weights.cpu().double() - val).abs().max() < 1e-5
        ops.moe_route(x.to(DEV), wr.to(DEV), None, chosen, weights, None, groups, kept, correction=corr.to(DEV))
        assert (weights.cpu().double() - torch.gather(s, 1, idx)).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 5, 60, 700])
def test_experts_with_identity_experts_and_a_shared_one(n, dtype):
    """The whole part on few rows and on many (the grouped tensor-memory products): tokens whose every expert is an identity expert, tokens
    with none, and an expert that nobody chose."""
    from wllm_b200.parts import FEED_FORWARDS
    from wllm_b200.models.fusanex import _feed_forward
    g = torch.Generator().manual_seed(n + 5)
    H, E, I = 64, 5, 48
    mlp = {"kind": "moe", "expert": {"ff": I, "limit": 0.9}, "router": {"experts": E, "top": 2, "identity": 3}, "shared": {"ff": 24, "limit": 0.6}}
    part = FEED_FORWARDS.build(_feed_forward("m.", mlp), hidden_size=H, model_dtype=dtype)
    w = {ps.name: torch.randn(ps.shape, generator=g) * (0.3 if ps.kind == "matrix" else 0.02) for ps in part.param_specs()}
    w["m.correction"][1] = -5.0                                  # nobody chooses expert 1
    w = {k: v.to(dtype).to(torch.float64) for k, v in w.items()}
    part.load(lambda name: w[name].to(dtype).to(DEV))
    x = torch.randn(n, H, generator=g).to(dtype)
    bufs = {}
    ctx = SimpleNamespace(buffer=lambda name, shape, dt: bufs.setdefault((name, tuple(shape), dt), torch.full(tuple(shape), -7, dtype=dt, device=DEV)
                                                                         if not dt.is_floating_point else torch.full(tuple(shape), float("nan"), dtype=dt, device=DEV)))
    got = part(x.to(DEV), ctx).cpu().double()
    idx, _ = plain.route(mlp, w, "m.", x.double())
    ref = plain.experts_ff(mlp, w, "m.", x.double())
    assert n < 60 or (bool((idx >= E).all(-1).any()) and bool((idx < E).all(-1).any()) and not bool((idx == 1).any()))
    worst = (got - ref).abs().amax(-1).sort().values
    tol = 1e-5 if dtype == torch.float32 else 0.02
    assert worst[int(0.98 * (n - 1))] < tol * max(1.0, float(ref.abs().max())), (float(worst[-1]), float(ref.abs().max()))
    if dtype == torch.float32:
        assert worst[-1] < tol * max(1.0, float(ref.abs().max()))
