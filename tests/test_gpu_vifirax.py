"""Vifirax on the device against its plain statement (tests/plain_vifirax.py, float64, whole sequences).

Whole models: the residual after every layer; every way of cutting the work (whole prompts, a tail decoded token by token,
portions down to two tokens and one, mixed batches whose pages and state slots are used again), bit for bit against one
another in 32-bit; long prompts and long decoding; batches of unequal requests; one key far back that decides, also for a layer
that reads another's keys; decoding from captured graphs; greedy generation through the scheduler; the trace runner; a model without any
attention.  Mechanisms alone: the turn with a factor, row norms and biases with and without keys of the mixer's own, a one in the softmax's
denominator, one gate per head, a bias on a branch, low-rank maps and the decays made of them, the state space and the delta rule with decays per
key channel across portions, chunks, segments and slots (a write far back read much later), the router's softmax over the chosen logits, experts of
SiLU units (few rows and many).
"""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch
from safetensors.torch import save_file

import plain_vifirax as plain
import traces
from helpers import folder_weights, max_diff
from test_gpu_gudarax import Scratch, paged
from vifirax_configs import CONFIGS, NEAR, write_folder

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
    rows' scale: the typical row within 1.5 %, nine of ten within 6 % (where two experts' logits nearly tie, the rounded input may choose
    the other one, in any implementation, and the recurrences behind it carry that on: a few rows in a hundred with these weights)."""
    assert set(rows) == set(ref)
    scale = max(1.0, max(float(r.abs().max()) for r in ref.values()))
    if dtype == torch.float32:
        assert max_diff(rows, ref) < 2e-4 * scale, what
        return
    rms = math.sqrt(sum(float(r.double().pow(2).mean()) for r in ref.values()) / len(ref))
    rel = sorted(float((rows[k].double() - ref[k].double()).pow(2).mean().sqrt()) / rms for k in ref)
    assert rel[len(rel) // 2] < 0.015 and rel[int(0.9 * len(rel))] < 0.06, (what, rel[len(rel) // 2], rel[int(0.9 * len(rel))], rel[-1])


def requests_of(name, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


@pytest.fixture(scope="module")
def setups(tmp_path_factory):
    out = {}
    for name in CONFIGS:
        folder = write_folder(str(tmp_path_factory.mktemp("vifirax") / name), name)
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
            p = residual.pending
            if hasattr(p, "materialize"):
                add = p.materialize(ctx, "watched_branch")
            else:
                add = p.tensor.sum(0) if hasattr(p, "tensor") else p
            got.append((residual.stream + add.float()).double().cpu())
    blocks = model.blocks
    model.blocks = [Watched(b) for b in blocks]
    rc = runner.cache.open("x")
    runner.step([StepEntry(rc, toks, [0])])
    model.blocks = blocks
    assert len(got) == len(CONFIGS[name]["layers"])
    for run, (a, b) in enumerate(zip(got, want)):
        tol = (2e-5 if dtype == torch.float32 else 0.03) * float(b.abs().max())
        worst = (a - b).abs().amax(-1).sort().values
        # (bfloat16 is judged by rows: where two experts' logits nearly tie, the rounded input may choose the other one)
        at = len(worst) - 1 if dtype == torch.float32 else int(0.8 * len(worst))
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
        if cut == "mixed":      # pages and slots were used again
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
@pytest.mark.parametrize("name", ["mixed", "odd", "heads64", "recurrent"])
def test_long_prompts_and_long_decoding(setups, name, dtype):
    """A prompt long enough for segments side by side and for the convolution's tiles of tokens, in one step and in portions; and most of
    it decoded token by token."""
    from wllm_b200.kernels import ops
    folder = setups[name][0]
    reqs = requests_of(name, (330,), seed=8)
    assert ops.linattn_segment_plan(330, 1, 4, 64)[1] > 2
    ref = plain_rows(folder, name, reqs)
    for cut, steps in (("whole", traces.whole(reqs)), ("portions", traces.portions(reqs, sizes=(140, 2, 131, 1, 37))), ("decoded", traces.tail_singly(reqs, 190))):
        runner = runner_for(folder, dtype, 16, 21)
        close_enough(traces.run_in_process(runner, steps), ref, dtype, cut)
        assert all(f == 21 for f in runner.cache.free_pages())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "heads64"])
def test_a_batch_of_unequal_requests_gives_each_its_own_rows(setups, name, dtype):
    """Single tokens of some beside a long and two short portions, then all of them decoding together, against each alone."""
    from wllm_b200.engine import StepEntry
    folder = setups[name][0]
    reqs = requests_of(name, (40, 330, 3, 66), seed=12)
    ref = plain_rows(folder, name, reqs)
    runner = runner_for(folder, dtype, 16, 40)
    rc = {k: runner.cache.open(k) for k in reqs}
    plan = [{"r0": 30}, {"r0": 1, "r1": 300, "r2": 2, "r3": 60}, {"r0": 1, "r1": 1, "r2": 1, "r3": 1}] + [{"r0": 1, "r1": 1, "r3": 1}] * 5 + \
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
@pytest.mark.parametrize("dim,vdim", [(32, 24), (64, 64)])
def test_a_far_key_decides(tmp_path, dim, vdim, dtype):
    """Two attention layers, the second on the first one's keys and values.  One token's key is made to lie along one other token's query (in
    the part of the head that does not turn), with a score scale that gives it all the weight: where it stands (at the start, at page and
    chunk borders, far back, just before) the last token's logits follow it, in a prompt and decoded alone."""
    from wllm_b200.engine import StepEntry
    from wllm_b200.weights import random_tensors
    att = {"heads": 4, "kv_heads": 2, "dim": dim, "vdim": vdim, "scale": 1.5, "rot": NEAR}
    V, W = 90, 48
    cfg = {"architecture": "Vifirax", "vocab": V, "width": W, "norm": {"eps": 1e-5},
           "layers": [{"type": "attention", "mixer": att, "mlp": None}, {"type": "attention", "mixer": {**att, "kv_from": 0}, "mlp": None}]}
    tensors = random_tensors(cfg, 5, dtype=torch.float32, std=0.1, vector_std=0.05)
    marked, asking = 7, 11
    g = torch.Generator().manual_seed(3)
    tensors["embed"] = torch.randn(V, W, generator=g) * 0.1
    tensors["embed"][:, :2] = 0.0
    tensors["embed"][marked] = 0.0
    tensors["embed"][marked, 0] = 3.0
    tensors["embed"][asking] = 0.0
    tensors["embed"][asking, 1] = 3.0
    direction = torch.randn(dim, generator=g)
    direction[:NEAR["dims"]] = 0.0
    for i in (0, 1):
        tensors[f"l{i}.mix.q"][:, 1] = direction.repeat(4) * 3
        tensors[f"l{i}.mix.q.norm"] = torch.ones(4 * dim)
    tensors["l0.mix.k"][:, 0] = direction.repeat(2) * 3
    tensors["l0.mix.k.norm"] = torch.ones(2 * dim)
    tensors["l0.mix.v"] *= 10.0
    folder = str(tmp_path / "m")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    save_file({k: t.to(torch.bfloat16).contiguous() for k, t in tensors.items()}, os.path.join(folder, "model.safetensors"))
    w = {k: t.double() for k, t in folder_weights(folder).items()}
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


@pytest.mark.parametrize("name", ["mixed", "recurrent"])
def test_decoding_from_captured_graphs_gives_the_eager_rows(setups, name):
    folder, reqs, ref = setups[name]
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


@pytest.mark.parametrize("name", ["mixed", "recurrent"])
def test_greedy_generation_through_the_scheduler(setups, name):
    from wllm_b200 import LLM, SamplingParams
    folder, reqs, _ = setups[name]
    w = {k: v.double() for k, v in folder_weights(folder).items()}
    prompts = [reqs["r0"], reqs["r2"], reqs["r3"][:40], reqs["r8"]]
    llm = LLM(folder, dtype="float32", block_size=16, num_blocks=12, chunked_prefill_tokens=24, max_num_seqs=3)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True))
    for prompt, o in zip(prompts, outs):
        toks = list(prompt)
        for _ in range(30):
            toks.append(int(plain.forward(CONFIGS[name], w, toks)[-1].argmax()))
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
def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def padded(x, heads, size, to):          # [n, heads * size] -> [n, heads * to], zeros behind every head
    out = x.new_zeros((x.shape[0], heads, to))
    out[:, :, :size] = x.view(x.shape[0], heads, size)
    return out.view(x.shape[0], heads * to)


def turned(x, positions, rot):
    """The plain turn at given positions: x [n, heads, dim]."""
    far = x.new_zeros((int(max(positions)) + 1,) + tuple(x.shape[1:]))
    out = torch.empty_like(x)
    for i, p in enumerate(positions):
        far[p] = x[i]
        out[i] = plain.turn(far, rot)[p]
    return out


def position_of(rot, dim):
    from wllm_b200.parts import POSITIONS, spec
    return POSITIONS.build(spec("rope", theta=rot["base"], head_dim=dim, rotary_dim=rot["dims"], exact_table=True, scaling=rot.get("scaling"))).to(DEV)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("own", [True, False])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 8), (5, 1, 10, 6, 6), (2, 2, 64, 64, 64), (6, 3, 32, 16, 12)])
def test_row_norms_biases_and_a_scaled_turn(sizes, own, dtype):
    """q | k | v (or q alone, for a mixer on another's keys) from a product, as one tensor and as 32-bit partial sums: a bias row, norms of
    the whole rows, the turn with its factor; what lands in q_out and in the pages, against the formulas."""
    from wllm_b200.kernels import ops
    nq, nkv, hd_file, vd_file, dims = sizes
    hd, vd = -(-hd_file // 8) * 8, -(-vd_file // 8) * 8
    g = torch.Generator().manual_seed(nq * 100 + hd_file)
    n, ps, eps = 37, 16, 1e-5
    rot = {**NEAR, "dims": dims}
    pos = position_of(rot, hd)
    assert pos.turn_scale > 1.05
    heads = [("q", nq, hd_file, hd)] + ([("k", nkv, hd_file, hd), ("v", nkv, vd_file, vd)] if own else [])
    rows = {k: torch.randn(n, h * s, generator=g) for k, h, s, _ in heads}
    bias = {k: torch.randn(1, h * s, generator=g) for k, h, s, _ in heads}
    gain = {k: 1 + 0.3 * torch.randn(1, h * s, generator=g) for k, h, s, _ in heads if k != "v"}
    fused = torch.cat([padded(rows[k], h, s, to) for k, h, s, to in heads] + [torch.randn(n, 8, generator=g)], 1)     # the gate's columns behind
    bias_row = torch.cat([padded(bias[k], h, s, to) for k, h, s, to in heads], 1)[0].contiguous().to(DEV)
    gains = {k: padded(gain[k], h, s, to)[0].to(dtype).contiguous() for k, h, s, to in heads if k != "v"}
    positions = torch.arange(3, 3 + 5 * n, 5)
    slots = torch.randperm(4 * ps, generator=g)[:n].to(torch.int32).to(DEV)
    for parts in (0, 3):
        if parts:
            cut = torch.randn(parts, n, fused.shape[1], generator=g)
            cut[0] += fused - cut.sum(0)
            x, src = cut.to(DEV), cut.double().sum(0)
        else:
            x = fused.to(dtype).to(DEV)
            src = x.double().cpu()
        want, c = {}, 0
        for k, h, s, to in heads:
            y = src[:, c:c + h * to].view(n, h, to)[:, :, :s].reshape(n, h * s) + bias[k].double()
            c += h * to
            if k != "v":
                y = plain.gain_norm(y, gains[k].view(h, to)[:, :s].reshape(-1).double(), eps).view(n, h, s)
                y = turned(y, positions.tolist(), rot).reshape(n, h * s)
            want[k] = padded(y, h, s, to)
        q_out = torch.empty(n, nq * hd, dtype=dtype, device=DEV)
        kp, vp = (torch.zeros(4, nkv, ps, d, dtype=dtype, device=DEV) for d in (hd, vd))
        ops.rope_row_norm_kv_write(x, q_out, positions.to(torch.int32).to(DEV), slots if own else None, pos.inv_freq, kp, vp, nq, nkv if own else 0, hd,
                                   dims, ps, gains["q"].to(DEV), gains["k"].to(DEV) if own else None, eps, nq * hd_file, nkv * hd_file if own else 0,
                                   in_splits=parts, vd=vd, bias=bias_row, turn_scale=pos.turn_scale)
        sl = slots.long().cpu()
        got = {"q": q_out.cpu(), "k": kp.cpu()[sl // ps, :, sl % ps].reshape(n, nkv * hd), "v": vp.cpu()[sl // ps, :, sl % ps].reshape(n, nkv * vd)}
        tol = 2e-5 if dtype == torch.float32 else 0.02
        for k in want:
            assert (got[k].double() - want[k]).abs().max() < tol * float(want[k].abs().max()), (parts, k)
        if not own:
            assert (kp == 0).all() and (vp == 0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [5, 300, 1030])
@pytest.mark.parametrize("pairing", ["half", "interleaved"])
def test_a_scaled_turn_without_norms(n, pairing, dtype):
    """The plain rotary kernels (few tokens, many in bfloat16 with 16-byte accesses, a CTA a token) with a factor on sines and cosines."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    nq, nkv, hd, dims, ps = 3, 1, 32, 16, 16
    rot = {**NEAR, "dims": dims}
    pos = position_of(rot, hd)
    x = torch.randn(n, (nq + 2 * nkv) * hd, generator=g).to(dtype)
    positions = (torch.arange(n) * 7 % 501).to(torch.int32)
    pages = -(-n // ps)
    kp, vp = (torch.zeros(pages, nkv, ps, hd, dtype=dtype, device=DEV) for _ in range(2))
    q_out = torch.empty(n, nq * hd, dtype=dtype, device=DEV)
    ops.rope_kv_write(x.to(DEV), q_out, positions.to(DEV), torch.arange(n, dtype=torch.int32, device=DEV), pos.inv_freq, kp, vp, nq, nkv, hd, dims, ps,
                      pairing=pairing, turn_scale=pos.turn_scale)
    f, m = plain.frequencies(rot)
    a = positions.double()[:, None] * torch.tensor(f, dtype=torch.float64)[None]
    c, s = torch.cos(a)[:, None] * m, torch.sin(a)[:, None] * m
    y = x.double()[:, :(nq + nkv) * hd].view(n, nq + nkv, hd).clone()
    ia = torch.arange(0, dims, 2) if pairing == "interleaved" else torch.arange(dims // 2)
    ib = ia + 1 if pairing == "interleaved" else ia + dims // 2
    u, v = y[..., ia].clone(), y[..., ib].clone()
    y[..., ia], y[..., ib] = u * c - v * s, v * c + u * s
    tol = 5e-5 if dtype == torch.float32 else 0.02
    assert (q_out.double().cpu() - y[:, :nq].reshape(n, -1)).abs().max() < tol * 4
    got_k = kp.cpu().permute(0, 2, 1, 3).reshape(-1, nkv * hd)[:n].double()
    assert (got_k - y[:, nq:].reshape(n, -1)).abs().max() < tol * 4
    assert torch.equal(vp.cpu().permute(0, 2, 1, 3).reshape(-1, nkv * hd)[:n], x[:, (nq + nkv) * hd:])


def plain_sink_rows(q, k, v, positions, scale):
    H, G = q.shape[1], k.shape[1]
    out = []
    for a in range(H):
        s = (q[:, a].double() @ k[:, a // (H // G)].double().T) * scale
        seen = torch.arange(k.shape[0])[None, :] <= torch.tensor(positions)[:, None]
        out.append(plain.sink_softmax(s, seen) @ v[:, a // (H // G)].double())
    return torch.cat(out, dim=-1)


@pytest.mark.parametrize("dtype,d,dv", [(torch.float32, 16, 24), (torch.float32, 64, 64), (torch.bfloat16, 16, 24), (torch.bfloat16, 64, 64), (torch.bfloat16, 128, 128)])
@pytest.mark.parametrize("shift", [-30.0, 0.0, 30.0])
def test_attention_with_a_one_in_the_denominator(shift, dtype, d, dv):
    """Scores all far below zero (the one takes everything: next to no output), around zero, and far above (the usual softmax), with one key
    that stands out at page and chunk borders and far back; rows of a portion and decoded rows, every kernel the part may choose, pages in
    scrambled order."""
    from wllm_b200.kernels import ops
    from wllm_b200.parts import MIXERS, spec
    g = torch.Generator().manual_seed(d + int(shift))
    H, G, ps, L, n0 = 4, 2, 16, 300, 236
    scale = 0.3 * (16 / d) ** 0.5
    part = MIXERS.build(spec("attention", num_heads=H, num_kv_heads=G, head_dim=d, value_dim=dv, scale=scale, sink_score=0.0, q_proj="q", k_proj="k",
                             v_proj="v", o_proj="o", position=spec("rope", theta=1.0, head_dim=d, rotary_dim=0)), hidden_size=8, model_dtype=dtype)
    w = {"q": torch.zeros(H * d, 8), "k": torch.zeros(G * d, 8), "v": torch.zeros(G * dv, 8), "o": torch.zeros(8, H * dv)}
    part.load(lambda name: w[name].to(dtype).to(DEV))
    assert part.sinks.tolist() == [0.0] * H
    k, v = torch.randn(L, G, d, generator=g), torch.randn(L, G, dv, generator=g).to(dtype)
    k[:, :, 0] = shift / scale / 4
    q = torch.randn(L - n0, H, d, generator=g)
    q[:, :, 0] = 4.0
    q, positions, strengths = q.to(dtype), list(range(n0, L)), []
    for edge in (0, 15, 16, 63, 64, 128, n0, L - 2):
        k2 = k.clone()
        k2[edge] += 40.0 / (scale * d) * torch.sign(q[-1, 0].float())[None]
        k2 = k2.to(dtype)
        want = plain_sink_rows(q, k2, v, positions, scale)
        strengths.append(float(want[:-1].abs().median()))
        kp, vp, table = paged(k2, v, ps, edge + 5)
        group = type("G", (), {"page_size": ps})()
        cache = type("C", (), {"page_size": ps, "groups": [group]})()
        for rows, single in ((slice(None), False), (slice(-1, None), True)):
            qd = q[rows].reshape(-1, H * d).contiguous().to(DEV)
            n = qd.shape[0]
            out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
            ctx = Scratch(cache=cache, group_tables=[table], token_req=i32([0] * n), positions=i32(positions[rows]), req_q_start=i32([0]), req_q_len=i32([n]),
                          req_ctx_len=i32([L]), num_single=int(single), num_multi=int(not single), max_q_len=n, max_ctx=L, n_requests=1,
                          host={"req_q_len": np.array([n]), "req_ctx_len": np.array([L])})
            part.attend(qd, out, kp, vp, ctx, 0)
            tol = 2e-5 if dtype == torch.float32 else 0.03
            assert (out.double().cpu() - want[rows]).abs().max() < tol * max(1.0, float(want.abs().max())), (edge, single)
    assert (max(strengths) < 1e-6) if shift < 0 else (min(strengths) > 0.01)
    assert dtype == torch.float32 or ops.tc_gemm_status(DEV) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_gate_per_head_and_a_bias_on_the_branch(dtype):
    """Every head's output times the sigmoid of its one number, from a tensor's columns and from partial sums; a branch with its projection's
    bias through the norm behind the sublayer (inside that norm's kernel, and alone), as a tensor and as partial sums."""
    from wllm_b200.kernels import ops
    from wllm_b200.parts import NORMS, BiasedBranch, NormedBranch, Partials, Residual, spec
    g = torch.Generator().manual_seed(4)
    for n, H, V in ((3, 5, 24), (70, 4, 64), (1, 16, 8)):
        x = torch.randn(n, H * V, generator=g).to(dtype)
        fused = torch.randn(n, 40, generator=g).to(dtype)
        want = (x.double().view(n, H, V) * torch.sigmoid(fused.double()[:, 13:13 + H])[..., None]).view(n, H * V)
        got = ops.sigmoid_gate(x.to(DEV).clone(), fused.to(DEV), 0, 13, per=V)
        tol = 1e-6 if dtype == torch.float32 else 0.01
        assert (got.double().cpu() - want).abs().max() < tol * float(want.abs().max())
        cut = torch.randn(3, n, 40, generator=g)
        cut[0] += fused.float() - cut.sum(0)
        got = ops.sigmoid_gate(x.to(DEV).clone(), cut.to(DEV), 3, 13, per=V)
        assert (got.double().cpu() - want).abs().max() < max(tol, 5e-6) * float(want.abs().max())
    W, n, eps = 72, 9, 1e-5
    gain = (torch.randn(W, generator=g) * 0.3).to(dtype)
    norm = NORMS.build(spec("rmsnorm", weight="w", eps=eps, unit_offset=True), hidden_size=W, model_dtype=dtype)
    norm.load(lambda name: gain.to(DEV))
    reader = NORMS.build(spec("identity"), hidden_size=W, model_dtype=dtype)
    bias, start = torch.randn(W, generator=g), torch.randn(n, W, generator=g)
    for parts in (0, 3):
        branch = torch.randn(*((parts, n, W) if parts else (n, W)), generator=g)
        if not parts:
            branch = branch.to(dtype)
        total = branch.double().sum(0) if parts else branch.double()
        added = plain.layer_norm(total + bias.double(), gain.double(), eps)
        dev = branch.to(DEV)
        pending = NormedBranch(BiasedBranch(Partials(dev) if parts else dev, bias.to(DEV)), norm)
        residual = Residual(start.clone().to(DEV))
        residual.pending = pending
        out = reader(residual, Scratch())
        assert (residual.stream.double().cpu() - (start.double() + added)).abs().max() < 1e-5
        assert (out.double().cpu() - (start.double() + added)).abs().max() < (1e-5 if dtype == torch.float32 else 0.02)
        assert (pending.materialize(Scratch()).double().cpu() - added).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,H,D,rank", [(1, 2, 16, 8), (7, 3, 10, 24), (70, 4, 32, 16), (64, 5, 10, 8), (300, 3, 130, 40), (65, 1, 7, 8)])
def test_low_rank_maps_and_the_decays_made_of_them(n, H, D, rank, dtype):
    """up (columns of a wider product) with and without a bias, and as a decay per key channel, minus one: few rows and many (the tensor
    cores), from a tensor and from partial sums.  Channels that forget next to nothing are right relative to themselves."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(n * 7 + rank)
    low = torch.randn(n, rank + 24, generator=g).to(dtype)
    up = (torch.randn(H * D, rank, generator=g) * 0.3).to(dtype)
    bias = (torch.randn(H * D, generator=g) - 2).to(dtype)
    bias[::3] -= 8.0
    log = torch.linspace(-6, 1, H).to(dtype)
    for parts in (0, 3):
        if parts:
            cut = torch.randn(parts, n, rank + 24, generator=g)
            cut[0] += low.float() - cut.sum(0)
            x, src = cut.to(DEV), cut.double().sum(0)
        else:
            x, src = low.to(DEV), low.double()
        z = src[:, 16:16 + rank] @ up.double().T
        got = ops.lowrank_map(x, parts, 16, up.to(DEV), H, D, torch.empty(n, H * D, device=DEV))
        assert (got.double().cpu() - z).abs().max() < 1e-4 * max(1.0, float(z.abs().max()))
        z = z + bias.double()
        less = torch.expm1(-torch.exp(log.double()).repeat_interleave(D) * plain.softplus(z))
        got = ops.lowrank_map(x, parts, 16, up.to(DEV), H, D, torch.empty(n, H * D, device=DEV), bias.to(DEV), log.to(DEV))
        rel = (got.double().cpu() - less).abs() / less.abs()
        assert less.abs().min() < 1e-4 and rel.max() < 2e-3 * (1 if dtype == torch.bfloat16 else 0.05), (parts, float(rel.max()))


def run_portions(part, names, tensors, hs, cuts, dtype, width):
    """Two requests through a part in one batch a step, cut in the given ways, in slots 3 and 1 of 5: their output rows, the slots' tensors."""
    from wllm_b200.parts import CacheRef
    need = part.cache_need().tensors
    states = {name: torch.full((5,) + tuple(shape), float("nan"), dtype=dt, device=DEV) for name, shape, dt in need}
    use = (3, 1)
    for t in states.values():
        for s in use:
            t[s].zero_()
    cache = CacheRef(state_names={name: name for name in states})
    outs, pos = [[], []], [0, 0]
    for it in range(max(len(c) for c in cuts)):
        rows, starts, lens, slot_ids, who = [], [], [], [], []
        for r in (0, 1):
            if it < len(cuts[r]):
                c = cuts[r][it]
                starts.append(sum(lens))
                lens.append(c)
                slot_ids.append(use[r])
                rows.append(hs[r][pos[r]:pos[r] + c])
                who.append(r)
                pos[r] += c
        x = torch.cat(rows).to(dtype).contiguous().to(DEV)
        ctx = Scratch(token_req=i32([j for j, c in enumerate(lens) for _ in range(c)]), req_q_start=i32(starts), req_q_len=i32(lens), req_slot=i32(slot_ids),
                      num_single=sum(c == 1 for c in lens), num_multi=sum(c > 1 for c in lens), max_q_len=max(lens), n_requests=len(lens),
                      state=lambda name: states[name])
        y = part(x, ctx, cache)
        y = y.tensor.sum(0) if hasattr(y, "tensor") else y
        for j, r in enumerate(who):
            outs[r].append(y[starts[j]:starts[j] + lens[j]].float().cpu())
    assert [sum(c) for c in cuts] == pos
    for t in states.values():
        assert all(torch.isnan(t[s]).all() for s in (0, 2, 4))          # slots of nobody are left alone
    return [torch.cat(x) for x in outs]


def check_portions(part, names, tensors, want, hs, dtype):
    """Every way of cutting against the plain rows; in 32-bit the cuts shorter than segments give the same bits."""
    a, b = len(hs[0]), len(hs[1])
    ways = (((a,), (b,)), ((1, 2, 3, 60, 1, 1, 82, a - 150), (40, 1, 1, b - 42)), ((2,) * (a // 2) + (1,) * (a % 2), (b,)), ((a - 1, 1), (1,) * b),
            ((127, 127, a - 254) if a > 254 else (a - 7, 7), (b - 2, 2)))
    first = None
    for cuts in ways:
        got = run_portions(part, names, tensors, hs, cuts, dtype, None)
        for r in (0, 1):
            worst = (got[r].double() - want[r]).abs().amax(-1) / max(1e-3, float(want[r].abs().max()))
            assert float(worst.max()) < (1e-4 if dtype == torch.float32 else 0.04), (cuts, r, float(worst.max()))
        if dtype == torch.float32 and max(max(c) for c in cuts) < 128:
            if first is None:
                first = got
            else:
                assert torch.equal(first[0], got[0]) and torch.equal(first[1], got[1]), cuts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 24, 16, 2, 4, 3), (3, 10, 7, 1, 2, 2), (2, 64, 128, 1, 4, 1), (6, 8, 256, 3, 3, 6), (2, 80, 24, 2, 1, 5), (1, 16, 16, 1, 7, 1), (4, 40, 48, 2, 4, 2)])
def test_the_state_space_across_portions_segments_and_slots(sizes, dtype):
    """heads, values, state rows, groups, taps, norm groups of widely different sizes against the plain statement on whole sequences; an early
    token's large value still read three hundred tokens later through a head that forgets next to nothing."""
    from wllm_b200.parts import MIXERS, spec
    H, V, N, G, T, parts = sizes
    W, inner = 40, H * V
    g = torch.Generator().manual_seed(H * 31 + N)
    C = inner + 2 * G * N
    t = {"in": torch.randn(2 * inner + 2 * G * N + H, W, generator=g) * 0.25, "conv": torch.randn(C, T, generator=g) * 0.6, "conv.b": torch.randn(C, generator=g) * 0.3,
         "dt_bias": torch.rand(H, generator=g) * 3 - 3, "A_log": torch.rand(H, generator=g) * 2 - 1, "D": 1 + 0.3 * torch.randn(H, generator=g),
         "norm": 1 + 0.3 * torch.randn(inner, generator=g), "o": torch.randn(W, inner, generator=g) * 0.2}
    t["A_log"][0] = -7.0                              # head 0 forgets next to nothing ...
    t["in"][-H] = 0.0                                 # ... and takes steps of one size
    t = {k: v.to(dtype) for k, v in t.items()}
    part = MIXERS.build(spec("state_space", num_heads=H, groups=G, state_dim=N, value_dim=V, conv_taps=T, norm_groups=parts, eps=1e-5, in_proj="in",
                             conv="conv", conv_bias="conv.b", decay_log="A_log", step_bias="dt_bias", skip="D", norm_weight="norm", o_proj="o"),
                        hidden_size=W, model_dtype=dtype)
    part.load(lambda name: t[name].to(DEV))
    hs = [torch.randn(n, W, generator=g) for n in (330, 47)]
    hs[0][3] *= 12.0
    hs = [h.to(dtype) for h in hs]
    m = {"heads": H, "vdim": V, "state": N, "groups": G, "conv": T, "norm_groups": parts}
    wd = {k: v.double() for k, v in t.items()}
    want = [plain.mamba2(m, wd, "", h.double(), 1e-5) for h in hs]
    quiet = hs[0].double().clone()
    quiet[3] = 0.0
    assert (plain.mamba2(m, wd, "", quiet, 1e-5)[-1] - want[0][-1]).abs().max() > 0.02 * float(want[0].abs().max())
    check_portions(part, None, None, want, hs, dtype)


@pytest.mark.parametrize("H,G,N,V", [(2, 1, 16, 8), (4, 2, 128, 64), (3, 3, 48, 40), (2, 2, 112, 24), (6, 2, 64, 72), (1, 1, 80, 32)])
def test_the_state_space_in_chunks(H, G, N, V):
    """The chunked kernel alone on given rows: requests whose lengths lie around a chunk's border, in one batch, in two steps that carry the state;
    for pairs of places at both sides of the borders the row B of one and the row C of the other are made to agree, so that one write decides one
    read; heads that forget within a token and heads that forget next to nothing."""
    from wllm_b200.kernels import ops
    g = torch.Generator().manual_seed(H * 100 + N)
    lengths = (1, 2, 63, 64, 65, 129, 200, 128)
    slots = list(range(len(lengths)))[::-1]
    C = H * V + 2 * G * N
    state = torch.full((len(lengths) + 1, H, N, V), float("nan"), device=DEV)
    state[:len(lengths)] = 0.0
    rate = torch.logspace(-6, 0.5, H, dtype=torch.float64) if H > 1 else torch.tensor([1e-3], dtype=torch.float64)
    parts = {i: [] for i in range(len(lengths))}
    got = {i: [] for i in range(len(lengths))}
    for step in range(2):
        lens = list(lengths if step == 0 else lengths[::-1])
        n = sum(lens)
        xbc = torch.randn(n, C, generator=g) * 0.3
        starts = [sum(lens[:i]) for i in range(len(lens))]
        b, c = H * V, H * V + G * N
        for t0, L in zip(starts, lens):
            for s, t in ((0, L - 1), (62, 63), (63, 64), (0, 64), (64, 127), (63, 128), (1, 199)):
                if s <= t < L:
                    v = torch.randn(G * N, generator=g)
                    xbc[t0 + s, b:b + G * N], xbc[t0 + t, c:c + G * N] = v, v
        xbc = xbc.to(torch.bfloat16)
        dt = torch.rand(n, H, generator=g).double() + 0.05
        pairs = torch.stack([-rate * dt, dt], dim=-1).float().contiguous()
        out = torch.full((n, H * V), float("nan"), device=DEV)
        ops.ssd_chunks(xbc.to(DEV), pairs.to(DEV), state, out, i32(starts), i32(lens), i32(slots), H, H // G, N, V)
        for i, (t0, L) in enumerate(zip(starts, lens)):
            parts[i].append((xbc[t0:t0 + L].double(), dt[t0:t0 + L]))
            got[i].append(out[t0:t0 + L].double().cpu())
    for i in parts:
        x = torch.cat([p[0] for p in parts[i]])
        n = x.shape[0]
        want = plain.ssd(x[:, :H * V].reshape(n, H, V), x[:, H * V:H * V + G * N].reshape(n, G, N), x[:, H * V + G * N:].reshape(n, G, N),
                         torch.cat([p[1] for p in parts[i]]), -rate, torch.zeros(H, dtype=torch.float64)).reshape(n, H * V)
        scale = want.abs().view(n, H, V).amax(dim=(0, 2)).repeat_interleave(V).clamp(min=1e-3)
        assert ((torch.cat(got[i]) - want).abs() / scale).max() < 2e-4, (i, lengths[i])
    assert torch.isnan(state[-1]).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 3, 8, 16), (3, 1, 10, 6, 2, 5, 3), (2, 1, 64, 64, 4, 16, 8), (2, 2, 128, 40, 1, 8, 24), (1, 1, 200, 130, 3, 40, 8)])
def test_the_delta_rule_with_a_decay_per_key_channel(sizes, dtype):
    """heads, query/key heads, sizes, taps and the ranks of both low-rank maps of widely different sizes, against the plain statement on whole
    sequences; an early token's large value along a channel that forgets next to nothing still shows in rows far behind."""
    from wllm_b200.parts import MIXERS, spec
    H, G, D, V, T, ra, rg = sizes
    W = 40
    g = torch.Generator().manual_seed(H * 31 + D)
    rnd = lambda *shape: torch.randn(*shape, generator=g)
    t = {"q": rnd(G * D, W) * 0.25, "k": rnd(G * D, W) * 0.25, "v": rnd(H * V, W) * 0.25, "q.conv": rnd(G * D, T) * 0.7, "k.conv": rnd(G * D, T) * 0.7,
         "v.conv": rnd(H * V, T) * 0.7, "b": rnd(H, W) * 0.3, "A_log": torch.rand(H, generator=g) * 2 - 1, "norm": 1 + 0.3 * rnd(V), "a1": rnd(ra, W) * 0.3,
         "a2": rnd(H * D, ra) * 0.3, "dt_bias": torch.rand(H * D, generator=g) * 4 - 5, "g1": rnd(rg, W) * 0.3, "g2": rnd(H * V, rg) * 0.4, "o": rnd(W, H * V) * 0.2}
    t["A_log"][0] = -8.0
    t = {k: v.to(dtype) for k, v in t.items()}
    part = MIXERS.build(spec("delta_rule", num_heads=H, num_kv_heads=G, key_dim=D, value_dim=V, conv_taps=T, eps=1e-5, unit_norm_eps=1e-6, q_scale=D ** -0.5,
                             q_proj="q", k_proj="k", v_proj="v", q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", beta_proj="b", decay_log="A_log",
                             decay_bias="dt_bias", decay_maps={"down": "a1", "up": "a2"}, gate_maps={"down": "g1", "up": "g2"}, head_norm_weight="norm",
                             o_proj="o"), hidden_size=W, model_dtype=dtype)
    part.load(lambda name: t[name].to(DEV))
    hs = [rnd(n, W) for n in (330, 47)]
    hs[0][3] *= 20.0
    hs = [h.to(dtype) for h in hs]
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "conv": T}
    wd = {k: v.double() for k, v in t.items()}
    want = [plain.channel_delta(m, wd, "", h.double(), 1e-5) for h in hs]
    quiet = hs[0].double().clone()
    quiet[3] = 0.0
    assert (plain.channel_delta(m, wd, "", quiet, 1e-5)[40:] - want[0][40:]).abs().max() > 0.02 * float(want[0].abs().max())
    check_portions(part, None, None, want, hs, dtype)


def expert_part(E, top, H, I, dtype, seed):
    from wllm_b200.parts import FEED_FORWARDS, spec
    g = torch.Generator().manual_seed(seed)
    w = {"router": torch.randn(E, H, generator=g) * 0.5, "router.b": torch.randn(E, generator=g) * 2.0}
    for j in range(E):
        w[f"e{j}.gate"], w[f"e{j}.up"], w[f"e{j}.down"] = torch.randn(I, H, generator=g) * 0.3, torch.randn(I, H, generator=g) * 0.3, torch.randn(H, I, generator=g) * 0.2
    w = {k: v.to(dtype) for k, v in w.items()}
    part = FEED_FORWARDS.build(spec("routed_experts", num_experts=E, top=top, router="router", router_bias="router.b", expert_prefix="e", intermediate_size=I,
                                    activation="silu", scores="softmax_chosen"), hidden_size=H, model_dtype=dtype)
    part.load(lambda name: w[name].to(DEV))
    return part, {k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(6, 2, 64, 40, 9), (3, 1, 50, 14, 70), (4, 4, 64, 32, 33), (8, 2, 128, 96, 700), (40, 5, 64, 24, 300)])
def test_experts_of_silu_units_weighted_by_the_softmax_over_the_chosen(sizes, dtype):
    """The chosen experts (the largest logits with their bias), their weights, and the weighted sum of their outputs: few rows (products that
    gather rows on the fly) and many (the tensor-memory product over rows copied into sorted order)."""
    from wllm_b200.kernels import ops
    E, top, H, I, n = sizes
    part, w = expert_part(E, top, H, I, dtype, seed=E * 10 + n)
    g = torch.Generator().manual_seed(n)
    x = torch.randn(n, H, generator=g).to(dtype)
    mlp = {"router": {"experts": E, "top": top}}
    idx, val = plain.route(mlp, w, "", x.double())
    ctx = Scratch()
    out = part(x.to(DEV), ctx)
    chosen = ctx.bufs[("moe_chosen", (n, top), torch.int32)].cpu().long()
    weights = ctx.bufs[("moe_weights", (n, top), torch.float32)].cpu()
    z = (x.double() @ w["router"].T + w["router.b"]).sort(-1, descending=True).values
    gaps = (z[:, :top] - z[:, 1:top + 1]).abs() if top < E else (z[:, :-1] - z[:, 1:]).abs()
    clear = (gaps > 1e-4).all(-1)
    assert clear.sum() > 0.9 * n and torch.equal(chosen[clear], idx[clear]) and (weights[clear].double() - val[clear]).abs().max() < 1e-5
    if top < E:       # the bias decides some of the choices
        assert (plain.route(mlp, {**w, "router.b": w["router.b"] * 0}, "", x.double())[0] != idx).any()
    want = plain.experts_ff(mlp, w, "", x.double())
    tol = 2e-5 if dtype == torch.float32 else 0.03
    assert (out.double().cpu()[clear] - want[clear]).abs().max() < tol * float(want.abs().max())
    assert n * top < part.TC_FROM_PAIRS or dtype == torch.float32 or ops.tc_grouped_ok(x.to(DEV), part.w_gu)


def test_the_router_chooses_far_apart_logits_by_their_order():
    """Logits hundreds apart: the softmax over all experts would round all but one score to nothing; the choice still follows the
    logits, and the weights are finite and sum to one."""
    from wllm_b200.kernels import ops
    n, H, E, top = 5, 32, 7, 4
    x = torch.zeros(n, H)
    x[:, 0] = 1.0
    w = torch.zeros(E, H)
    bias = torch.tensor([-700.0, 300.0, -200.0, 299.5, 10.0, -900.0, 0.0])
    chosen = torch.empty(n, top, dtype=torch.int32, device=DEV)
    weights = torch.empty(n, top, device=DEV)
    ops.moe_route(x.to(DEV), w.to(DEV), None, chosen, weights, None, scores="softmax_chosen", bias=bias.to(DEV))
    assert chosen.cpu().tolist() == [[1, 3, 4, 6]] * n
    assert torch.allclose(weights.cpu().double(), torch.softmax(torch.tensor([300.0, 299.5, 10.0, 0.0], dtype=torch.float64), 0).expand(n, top), atol=1e-6)
