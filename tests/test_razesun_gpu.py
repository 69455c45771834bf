"""The Razesun model on the framework's own step, state and generation paths against the plain oracle: whole prompts,
portions of several sizes down to two tokens, decoding, states that are used again, batches, greedy generation, and the
trace program.  Error measure: root mean square of the difference over the vocabulary, relative to the logits' spread."""
import json
import os
import subprocess
import sys

import pytest
import torch

import razesun_models as M
from conftest import ROOT
from oracle import razesun_oracle as R

pytestmark = pytest.mark.gpu

TOL = {torch.float32: 2e-5, torch.bfloat16: 4e-2}
NAMES = sorted(M.configs())


def build(name, dtype, seed=0):
    from based_b200 import registry, weights
    cfg = M.configs()[name]
    t = M.tensors(cfg, seed)
    m = registry.build_model(cfg, device="cuda", dtype=dtype).eval()
    m.load_tensors(weights.TensorDict(t))
    return cfg, {k: v.double() for k, v in t.items()}, m


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed))


def err(got, ref):
    d = got.double().cpu() - ref
    return float((d.pow(2).mean(-1).sqrt() / ref.std()).max())


def run(m, ids, portions, pool=None, request="r"):
    """Logits of every token of one request, fed in the given portions (the last one repeats)."""
    from based_b200.generation import StatePool
    out, at, n = [], 0, 0
    with torch.inference_mode():
        pool = pool or StatePool(m, max_seqlen=len(ids))
        ip = pool.acquire(request)
        while at < len(ids):
            k = portions[min(n, len(portions) - 1)]
            out.append(m.advance(ids[None, at:at + k].cuda(), ip)[0])
            at += k
            n += 1
        pool.release(request)
    return torch.cat(out)


@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_portions_and_decoding(name, dtype):
    cfg, w, m = build(name, dtype)
    ids = tokens(cfg, 333)
    ref = R.forward(cfg, w, ids)
    whole = run(m, ids, [len(ids)])
    assert err(whole, ref) < TOL[dtype]
    for portions in ([64], [2], [1], [128, 1, 127, 3, 65, 2], [7, 200, 1], [300, 1]):
        got = run(m, ids, portions)
        assert err(got, ref) < TOL[dtype], portions
        assert err(got, whole.double().cpu()) < TOL[dtype], portions
    from based_b200 import ops
    ops.check_status()


@pytest.mark.parametrize("name", NAMES)
def test_residual_stream_after_every_layer(name):
    cfg, w, m = build(name, torch.float32, seed=3)
    ids = tokens(cfg, 50)
    _, ref = R.forward(cfg, w, ids, want_layers=True)
    got = []
    with torch.inference_mode():
        m(ids[None].cuda(), stream_hook=lambda i, s: got.append(s[0].clone()))
    assert len(got) == len(cfg["layers"])
    for a, b in zip(got, ref):
        assert float((a.double().cpu() - b).abs().max() / b.abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_mixer_alone(dtype):
    """One-layer stacks without an MLP: the mixer is all there is."""
    from based_b200 import registry, weights
    for layer in (M.delta(4, 2, 64, 32, 4), M.delta(2, 2, 128, 64, 3), M.latent(4, 32, 16, 48, 56, 80, 0.3, 2000.0), M.rglru(128, 1, 4),
                  M.rglru(256, 1, 3), M.rglru(96, 4, 2)):
        cfg = M.config(96, 101, [layer], [None], mult=1.0)
        t = M.tensors(cfg, 5)
        m = registry.build_model(cfg, device="cuda", dtype=dtype).eval()
        m.load_tensors(weights.TensorDict(t))
        ids = tokens(cfg, 200)
        ref = R.forward(cfg, {k: v.double() for k, v in t.items()}, ids)
        for portions in ([200], [65, 2, 64, 1], [1]):
            assert err(run(m, ids, portions), ref) < TOL[dtype], (layer, portions)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_prompt_and_long_decoding(dtype):
    cfg, w, m = build("mixed", dtype, seed=2)
    ids = tokens(cfg, 1400)
    ref = R.forward(cfg, w, ids)
    assert err(run(m, ids, [1400]), ref) < TOL[dtype]
    assert err(run(m, ids, [900, 1]), ref) < TOL[dtype]
    assert err(run(m, ids, [255, 513, 257, 128]), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_states_are_used_again_and_requests_do_not_mix(dtype):
    """Unequal requests interleaved over one pool, more requests than states, against each alone."""
    from based_b200.generation import StatePool
    cfg, w, m = build("order", dtype)
    reqs = {r: tokens(cfg, n, seed=n) for r, n in (("a", 90), ("b", 1), ("c", 131), ("d", 17), ("e", 64))}
    refs = {r: R.forward(cfg, w, ids) for r, ids in reqs.items()}
    at, out = {}, {r: [] for r in reqs}
    waiting, live = list(reqs), []
    g = torch.Generator().manual_seed(0)
    with torch.inference_mode():
        pool = StatePool(m, max_seqlen=131)
        while waiting or live:
            while waiting and len(live) < 2:
                live.append(waiting.pop(0))
                pool.acquire(live[-1])
                at[live[-1]] = 0
            for r in list(live):
                n = int(torch.randint(1, 40, (1,), generator=g))
                ids = reqs[r][at[r]:at[r] + n]
                out[r].append(m.advance(ids[None].cuda(), pool.live[r])[0])
                at[r] += len(ids)
                if at[r] == len(reqs[r]):
                    pool.release(r)
                    live.remove(r)
        assert len(pool.free) == 2      # two states served five requests
        for r in reqs:
            assert err(torch.cat(out[r]), refs[r]) < TOL[dtype], r
        with pytest.raises(ValueError, match="fit"):
            m.advance(torch.zeros(1, 200, dtype=torch.int64).cuda(), pool.acquire("f"))


def test_batch_rows_are_independent():
    cfg, w, m = build("mixed", torch.bfloat16)
    rows = torch.stack([tokens(cfg, 100, seed=s) for s in range(3)])
    with torch.inference_mode():
        got = m(rows.cuda())
        ip = m.new_inference_params(3, 100)
        parts = [m.advance(rows[:, a:b].cuda(), ip) for a, b in ((0, 70), (70, 72), (72, 98), (98, 99), (99, 100))]
    for i in range(3):
        ref = R.forward(cfg, w, rows[i])
        assert err(got[i], ref) < TOL[torch.bfloat16]
        assert err(torch.cat([p[i] for p in parts]), ref) < TOL[torch.bfloat16]


@pytest.mark.parametrize("name", ["mixed", "order", "odd"])
def test_greedy_generation(name):
    """generate(): eager, CUDA graph and portions give the oracle's greedy continuation (fp32; ties are not expected)."""
    cfg, w, m = build(name, torch.float32, seed=4)
    prompt = torch.stack([tokens(cfg, 37, seed=8), tokens(cfg, 37, seed=9)])
    want = prompt
    for _ in range(12):
        nxt = torch.stack([R.forward(cfg, w, row)[-1].argmax() for row in want])
        want = torch.cat([want, nxt[:, None]], 1)
    eager = m.generate(prompt.cuda(), max_new_tokens=12)
    assert torch.equal(eager.cpu(), want)
    assert torch.equal(m.generate(prompt.cuda(), max_new_tokens=12, cg=True).cpu(), want)
    assert torch.equal(m.generate(prompt.cuda(), max_new_tokens=12, portion=10).cpu(), want)
    b16 = build(name, torch.bfloat16, seed=4)[2]
    t = {}
    a = b16.generate(prompt.cuda(), max_new_tokens=12, timings=t)
    assert torch.equal(a, b16.generate(prompt.cuda(), max_new_tokens=12, cg=True)) and t["decode_ms"] >= t["steps_ms"] > 0
    s = b16.generate(prompt.cuda(), max_new_tokens=6, top_k=5, temperature=0.7)
    assert s.shape == (2, 43) and int(s.max()) < cfg["vocab"]


def test_trace_program(tmp_path):
    """bin/trace_run on a written model folder: wanted places, portions, requests that follow one another."""
    import numpy as np
    cfg = M.configs()["odd"]
    t = M.tensors(cfg)
    M.write_folder(str(tmp_path / "m"), cfg, t)
    (tmp_path / "out").mkdir()
    ids = {r: tokens(cfg, n, seed=n).tolist() for r, n in (("a", 40), ("b", 9))}
    plan = [("a", 0, 30, [29, 3], []), ("a", 30, 32, [], []), ("a", 32, 33, [0], []), ("a", 33, 40, [6], ["a"]), ("b", 0, 9, [8, 0], ["b"])]
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": ids[r][a:b], "want": want}], "end": end})
             for i, (r, a, b, want, end) in enumerate(plan)]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "64"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300,
                       env={**os.environ, "PATH": os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"]})
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(plan))]
    w = {k: v.double() for k, v in t.items()}
    refs = {r: R.forward(cfg, w, torch.tensor(x)) for r, x in ids.items()}
    for i, (r, a, b, want, end) in enumerate(plan):
        f = tmp_path / "out" / f"{i}.f32"
        assert f.exists() == bool(want)
        if want:
            got = torch.from_numpy(np.fromfile(f, dtype="<f4").reshape(len(want), -1))
            assert err(got, refs[r][[a + x for x in want]]) < TOL[torch.float32]
