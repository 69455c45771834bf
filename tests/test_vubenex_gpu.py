"""The Vubenex model on the framework's own step, state and generation paths against the plain oracle: whole prompts,
portions of several sizes down to two tokens, decoding, states that are used again, batches, greedy generation, and the
trace program.  Error measure: root mean square of the difference over the vocabulary, relative to the logits' spread."""
import json
import os
import subprocess
import sys

import pytest
import torch

import vubenex_models as M
from conftest import ROOT
from oracle import vubenex_oracle as V

pytestmark = pytest.mark.gpu

# bf16: rounding alone gives a median of 0.5e-2 and, where a small vector is normed, single positions of 4e-2
TOL = {torch.float32: 2e-5, torch.bfloat16: 8e-2}
MEDIAN = {torch.float32: 1e-5, torch.bfloat16: 1e-2}
NAMES = sorted(M.configs())


def build(cfg, dtype, seed=0):
    from based_b200 import registry, weights
    t = M.tensors(cfg, seed)
    m = registry.build_model(cfg, device="cuda", dtype=dtype).eval()
    m.load_tensors(weights.TensorDict(t))
    return {k: v.double() for k, v in t.items()}, m


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed))


def err(got, ref):
    d = got.double().cpu() - ref
    return float((d.pow(2).mean(-1).sqrt() / ref.std()).max())


def median_err(got, ref):
    d = got.double().cpu() - ref
    return float((d.pow(2).mean(-1).sqrt() / ref.std()).median())


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
    cfg = M.configs()[name]
    w, m = build(cfg, dtype)
    ids = tokens(cfg, 333)
    ref = V.forward(cfg, w, ids)
    whole = run(m, ids, [len(ids)])
    assert err(whole, ref) < TOL[dtype]
    for portions in ([64], [2], [1], [128, 1, 127, 3, 65, 2], [7, 200, 1], [300, 1], [129, 17]):
        got = run(m, ids, portions)
        assert err(got, ref) < TOL[dtype] and median_err(got, ref) < MEDIAN[dtype], portions
        assert err(got, whole.double().cpu()) < TOL[dtype], portions
    from based_b200 import ops
    ops.check_status()


@pytest.mark.parametrize("name", NAMES)
def test_residual_stream_after_every_layer(name):
    cfg = M.configs()[name]
    w, m = build(cfg, torch.float32, seed=3)
    ids = tokens(cfg, 50)
    _, ref = V.forward(cfg, w, ids, want_layers=True)
    got = []
    with torch.inference_mode():
        m(ids[None].cuda(), stream_hook=lambda i, s: got.append(s[0].clone()))
    assert len(got) == len(cfg["layers"])
    for a, b in zip(got, ref):
        assert float((a.double().cpu() - b).abs().max() / b.abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_mixer_alone(dtype):
    """One-layer stacks without an MLP: the mixer and the token input are all there is."""
    for layer in (M.attention(6, 3, 64, 0.2, 0.5, 40), M.attention(2, 1, 128, 0.1, 0.0, 1), M.attention(16, 1, 80, 0.2, 0.3, 20),
                  M.lightning(64, 48, 0.9, 0.999, 0.2, 0.97), M.lightning(128, 64, 0.99)):
        cfg = M.config(96, 101, [layer], [None], 12, positions=300)
        w, m = build(cfg, dtype, seed=5)
        ids = tokens(cfg, 300)
        ref = V.forward(cfg, w, ids)
        for portions in ([300], [65, 2, 64, 1], [130, 40]):
            assert err(run(m, ids, portions), ref) < TOL[dtype], (layer, portions)


@pytest.mark.parametrize("name", ["mixed", "wide"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_prompt_and_long_decoding(name, dtype):
    cfg = M.configs()[name]
    w, m = build(cfg, dtype, seed=2)
    ids = tokens(cfg, 1400)
    ref = V.forward(cfg, w, ids)
    for portions in ([1400], [900, 1], [255, 513, 257, 128]):
        got = run(m, ids, portions)
        assert err(got, ref) < TOL[dtype] and median_err(got, ref) < MEDIAN[dtype], portions


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_states_are_used_again_and_requests_do_not_mix(dtype):
    """Unequal requests interleaved over one pool, more requests than states, against each alone."""
    from based_b200.generation import StatePool
    cfg = M.configs()["order"]
    w, m = build(cfg, dtype)
    reqs = {r: tokens(cfg, n, seed=n) for r, n in (("a", 90), ("b", 1), ("c", 131), ("d", 17), ("e", 64))}
    refs = {r: V.forward(cfg, w, ids) for r, ids in reqs.items()}
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
    cfg = M.configs()["mixed"]
    w, m = build(cfg, torch.bfloat16)
    rows = torch.stack([tokens(cfg, 200, seed=s) for s in range(3)])
    with torch.inference_mode():
        got = m(rows.cuda())
        ip = m.new_inference_params(3, 200)
        parts = [m.advance(rows[:, a:b].cuda(), ip) for a, b in ((0, 170), (170, 172), (172, 198), (198, 199), (199, 200))]
    for i in range(3):
        ref = V.forward(cfg, w, rows[i])
        assert err(got[i], ref) < TOL[torch.bfloat16]
        assert err(torch.cat([p[i] for p in parts]), ref) < TOL[torch.bfloat16]


@pytest.mark.parametrize("name", ["mixed", "order", "odd"])
def test_greedy_generation(name):
    """generate(): eager, CUDA graph and portions give the oracle's greedy continuation (fp32; ties are not expected)."""
    cfg = M.configs()[name]
    w, m = build(cfg, torch.float32, seed=4)
    prompt = torch.stack([tokens(cfg, 37, seed=8), tokens(cfg, 37, seed=9)])
    want = prompt
    for _ in range(12):
        nxt = torch.stack([V.forward(cfg, w, row)[-1].argmax() for row in want])
        want = torch.cat([want, nxt[:, None]], 1)
    eager = m.generate(prompt.cuda(), max_new_tokens=12)
    assert torch.equal(eager.cpu(), want)
    assert torch.equal(m.generate(prompt.cuda(), max_new_tokens=12, cg=True).cpu(), want)
    assert torch.equal(m.generate(prompt.cuda(), max_new_tokens=12, portion=10).cpu(), want)
    _, b16 = build(cfg, torch.bfloat16, seed=4)
    t = {}
    a = b16.generate(prompt.cuda(), max_new_tokens=12, timings=t)
    assert torch.equal(a, b16.generate(prompt.cuda(), max_new_tokens=12, cg=True)) and t["decode_ms"] >= t["steps_ms"] > 0
    s = b16.generate(prompt.cuda(), max_new_tokens=6, top_k=5, temperature=0.7)
    assert s.shape == (2, 43) and int(s.max()) < cfg["vocab"]


def test_positions_end_where_the_table_ends():
    cfg = M.config(64, 64, [M.attention(2, 1, 32, 0.2, 0.3, 4)], [None], 8, positions=20)
    w, m = build(cfg, torch.float32)
    ids = tokens(cfg, 21)
    assert err(run(m, ids[:20], [7]), V.forward(cfg, w, ids[:20])) < TOL[torch.float32]
    with pytest.raises(ValueError, match="positions"):
        run(m, ids, [20, 1])
    assert m.generate(ids[None, :15].cuda(), max_new_tokens=6).shape == (1, 21)    # the last token is not fed back
    with pytest.raises(ValueError, match="positions"):
        m.generate(ids[None, :15].cuda(), max_new_tokens=7)


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
    refs = {r: V.forward(cfg, w, torch.tensor(x)) for r, x in ids.items()}
    for i, (r, a, b, want, end) in enumerate(plan):
        f = tmp_path / "out" / f"{i}.f32"
        assert f.exists() == bool(want)
        if want:
            got = torch.from_numpy(np.fromfile(f, dtype="<f4").reshape(len(want), -1))
            assert err(got, refs[r][[a + x for x in want]]) < TOL[torch.float32]
