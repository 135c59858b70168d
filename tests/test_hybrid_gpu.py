"""Layer-list decoders on the GPU against the plain oracle (oracle/hybrid.py, float64): every mechanism
alone, whole prompts, portions, single tokens, sequences on used state, chunk edges, strong decays,
generation through the framework's entry points. fp32 models are held to fp32 rounding; bf16 models to
the rounding of bfloat16 products."""
import copy
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from emberlm_b200 import build, lib
from oracle import hybrid as oh
from tests import hybrid_cases as hc

pytestmark = pytest.mark.gpu
LIMIT = {"fp32": 3e-5, "bf16": 4e-2}
DTYPES = ["fp32", "bf16"]


def decoder(cfg, w, dtype, max_seq=256, max_portion=256):
    from emberlm_b200 import engine as E
    d = E.HybridDecoder(E.HybridModel(cfg, w, dtype), max_seq, max_portion)
    d.load_parameters(w)
    return d


def portions(dec, t, sizes):
    """Logits of every position, the tokens cut into `sizes` (repeated until the tokens are used up)."""
    out, at, i = [], 0, 0
    while at < len(t):
        n = min(sizes[i % len(sizes)], len(t) - at)
        out.append(dec.extend(t[at:at + n], range(n)).cpu().numpy())
        at, i = at + n, i + 1
    return np.concatenate(out)


def muted(cfg, w, keep):
    """One layer with everything but `keep` taken out of the residual."""
    w = dict(w)
    lay = cfg["layers"][0]
    if keep == "mlp":
        w["l0.norm1b"] = np.zeros_like(w["l0.norm1b"])
    elif lay["mlp"]:
        w["l0.norm2b"] = np.zeros_like(w["l0.norm2b"])
    if keep == "attention":
        w["l0.mix.right.out"] = np.zeros_like(w["l0.mix.right.out"])
    if keep == "lightning":
        w["l0.mix.left.out"] = np.zeros_like(w["l0.mix.left.out"])
    return w


MECHANISMS = [
    ("attention", hc.parallel(hc.attention(4, 2, 36, 24, 16, scaling=(4.0, 1.0, 4.0, 64)), hc.lightning(1, 8, 8))),
    ("attention", hc.parallel(hc.attention(6, 1, 64, 130, 64), hc.lightning(1, 8, 8))),
    ("attention", hc.parallel(hc.attention(2, 2, 128, 64, 2), hc.lightning(1, 8, 8))),
    ("attention", hc.parallel(hc.attention(2, 1, 50, 1, 50), hc.lightning(1, 8, 8))),
    ("attention", hc.parallel(hc.attention(3, 3, 200, 50, 100), hc.lightning(1, 8, 8))),
    ("lightning", hc.parallel(hc.attention(1, 1, 8, 8, 8), hc.lightning(3, 40, 24))),
    ("lightning", hc.parallel(hc.attention(1, 1, 8, 8, 8), hc.lightning(1, 128, 65, [0.999]))),
    ("lightning", hc.parallel(hc.attention(1, 1, 8, 8, 8), hc.lightning(2, 30, 100, [0.0, 1.0]))),
    ("lightning", hc.parallel(hc.attention(1, 1, 8, 8, 8), hc.lightning(2, 200, 33))),
    ("delta", hc.delta(6, 3, 48, 20, 4)),
    ("delta", hc.delta(2, 1, 100, 70, 2)),
    ("delta", hc.delta(1, 1, 64, 128, 4)),
    ("delta", hc.delta(2, 2, 130, 31, 5)),
    ("delta", hc.delta(3, 1, 17, 9, 1)),
    ("mlp", hc.delta(1, 1, 8, 8, 2, hc.mlp(150, 0.8))),
    ("mlp", hc.delta(1, 1, 8, 8, 2, hc.mlp(9, 7.0))),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(MECHANISMS)), ids=lambda i: f"{MECHANISMS[i][0]}{i}")
def test_each_mechanism_alone(case, dtype):
    keep, layer = MECHANISMS[case]
    cfg = hc.model(50, 72, [layer])
    w = muted(cfg, hc.weights(cfg, 10 + case, rank=(9, 33)), keep)
    t = hc.tokens(cfg, 150, case)
    want_layers = []
    want = oh.forward(cfg, w, t, want_layers)
    dec = decoder(cfg, w, dtype)
    trace = torch.zeros(1, len(t), cfg["width"], device="cuda")
    dec.trace_layers(trace)
    got = dec.extend(t, range(len(t))).cpu().numpy()
    dec.trace_layers(None)
    x0 = oh.rms_norm(w["embed"][t].astype(np.float64), w["embed.norm"], cfg["norm"]["eps"])
    # the mechanism's own share of the residual, not the embedding it rides on
    assert hc.error(trace[0].cpu().numpy() - x0, want_layers[0] - x0) <= LIMIT[dtype]
    assert hc.error(got, want) <= LIMIT[dtype]
    dec.reset()
    assert hc.error(portions(dec, t, [100, 1]), want) <= LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(hc.CONFIGS))
def test_whole_prompt_portions_and_tokens_agree_with_the_oracle(name, dtype):
    cfg = hc.CONFIGS[name]
    w = hc.weights(cfg, 21)
    t = hc.tokens(cfg, 140, 22)
    want = oh.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype)
    runs = {"whole": [140], "tokens": [1], "pairs": [2], "odd": [37, 2, 3, 1, 23], "halves": [64, 63, 65], "prompt, then tokens": [97] + [1] * 43}
    for label, sizes in runs.items():
        dec.reset()      # on the cache and state of the run before
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], label


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_portion_are_cut_inside(dtype):
    cfg, w = hc.GROUPED, hc.weights(hc.GROUPED, 31)
    t = hc.tokens(cfg, 130, 32)
    want = oh.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype, max_portion=33)
    rows = [0, 32, 33, 34, 65, 66, 98, 99, 129]
    assert hc.error(dec.extend(t, rows).cpu().numpy(), want[rows]) <= LIMIT[dtype]
    rows = [129, 5, 5, 40]      # any order, also twice
    dec.reset()
    assert hc.error(dec.extend(t, rows).cpu().numpy(), want[rows]) <= LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_after_one_another_do_not_see_each_other(dtype):
    cfg, w = hc.GROUPED, hc.weights(hc.GROUPED, 41)
    dec = decoder(cfg, w, dtype)
    for i, n in enumerate([90, 1, 2, 3, 25, 120, 4]):
        t = hc.tokens(cfg, n, 50 + i)
        dec.reset()
        got = portions(dec, t, [[n], [1], [2, 1], [50, 1]][i % 4])
        assert hc.error(got, oh.forward(cfg, w, t)) <= LIMIT[dtype], n


@pytest.mark.parametrize("dtype", DTYPES)
def test_chunk_edges_stand_out(dtype):
    """Sharp attention (one key wins), chunks of several sizes: rows at both sides of every edge. The
    oracle with a chunk one longer or shorter, counted from elsewhere, or with rotated values must be far
    outside the limit, so a window that is off by one cannot pass."""
    layer = hc.parallel(hc.attention(2, 1, 32, 24, 32), hc.lightning(1, 8, 8))
    cfg = hc.model(61, 64, [layer])
    w = muted(cfg, hc.weights(cfg, 61), "attention")
    layer["mixer"]["left"]["scale"] = 1.5
    t = hc.tokens(cfg, 110, 62)
    want = oh.forward(cfg, w, t)
    for size in (23, 25, 1000):
        wrong = copy.deepcopy(cfg)
        wrong["layers"][0]["mixer"]["left"]["mask"]["size"] = size
        bad = oh.forward(wrong, w, t)
        rows = [i for e in (24, 48, 72, 96) for i in (e - 1, e)]
        assert hc.error(bad[rows], want[rows]) > 5 * LIMIT[dtype]
    dec = decoder(cfg, w, dtype)
    for sizes in ([110], [1], [23, 1, 1, 23], [24], [25], [2], [47, 2, 61], [30, 1, 17, 1, 61]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_memory_of_the_recurrences_is_carried(dtype):
    """Slow decays, so that what was written long ago still counts; the oracle that forgets at a portion's
    start is far outside the limit."""
    layers = [hc.parallel(hc.attention(1, 1, 8, 8, 8), hc.lightning(2, 24, 24, [0.999, 0.98])), hc.delta(2, 1, 32, 24, 4)]
    cfg = hc.model(40, 48, layers)
    w = hc.weights(cfg, 71)
    w["l1.mix.A_log"] = np.full_like(w["l1.mix.A_log"], -6.0)
    t = hc.tokens(cfg, 200, 72)
    want = oh.forward(cfg, w, t)
    for cut in (64, 150):
        assert hc.error(oh.forward(cfg, w, t[cut:]), want[cut:]) > 3 * LIMIT[dtype]
    dec = decoder(cfg, w, dtype)
    for sizes in ([200], [64, 1], [150, 50], [16], [15], [17, 47, 63, 65]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("a_log,dt", [(4.0, 3.0), (-9.0, -4.0), (1.5, 0.0)])
def test_delta_rule_with_strong_and_weak_decays(a_log, dt, dtype):
    """Decays that wipe a channel within a token (e^-160) or hardly move it: nothing overflows. A wiped state
    leaves o = (q . k) u, which the norm over the head divides by |q . k|: the large eps keeps tokens whose
    q and k happen to be orthogonal from magnifying their own rounding."""
    cfg = hc.model(40, 48, [hc.delta(2, 1, 64, 40, 4), hc.delta(1, 1, 20, 20, 3)], eps=1e-2)
    w = hc.weights(cfg, 81)
    for i in (0, 1):
        w[f"l{i}.mix.A_log"] = hc.bf16(w[f"l{i}.mix.A_log"] + a_log)
        w[f"l{i}.mix.dt_bias"] = hc.bf16(w[f"l{i}.mix.dt_bias"] + dt)
    t = hc.tokens(cfg, 170, 82)
    want = oh.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype)
    for sizes in ([170], [1], [33, 2]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


def test_short_convolution_reaches_back_over_portions():
    cfg = hc.model(40, 48, [hc.delta(1, 1, 16, 16, 5)])
    w = hc.weights(cfg, 91)
    for n in ("q", "k", "v"):      # only the oldest tap: a lost input shows in full
        w[f"l0.mix.{n}.conv"][:, 1:] = 0.0
        w[f"l0.mix.{n}.conv"][:, 0] = 1.5
    t = hc.tokens(cfg, 40, 92)
    want = oh.forward(cfg, w, t)
    dec = decoder(cfg, w, "fp32")
    for sizes in ([40], [1], [2], [3], [4, 1], [5], [20, 1, 2]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT["fp32"], sizes


def agrees_with_greedy(cfg, w, prompt, got, margin):
    """Every generated token is the oracle's arg-max of its prefix, up to near ties."""
    seq = np.concatenate([prompt, got])
    z = oh.forward(cfg, w, seq)[len(prompt) - 1:-1]
    best = z.max(axis=1)
    return all(best[i] - z[i, got[i]] <= margin for i in range(len(got)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["grouped", "single"])
def test_greedy_generation(name, dtype):
    cfg = hc.CONFIGS[name]
    w = hc.weights(cfg, 101)
    prompt = hc.tokens(cfg, 19, 102)
    dec = decoder(cfg, w, dtype, max_seq=200)
    got = dec.generate(prompt, 500).cpu().numpy()      # up to the end of the cache, in one burst
    assert len(got) == 200 - 19 + 1
    margin = 1e-3 if dtype == "fp32" else 0.3
    assert agrees_with_greedy(cfg, w, prompt, got, margin)
    z = dec.last_logits().cpu().numpy()
    full = oh.forward(cfg, w, np.concatenate([prompt, got[:-1]]))[-1]
    assert hc.error(z[None], full[None]) <= LIMIT[dtype] * 2
    assert dec.generate(prompt[:1], 5).cpu().numpy().shape == (5,)
    with pytest.raises(RuntimeError):
        dec.generate([], 3)
    with pytest.raises(RuntimeError):
        dec.generate(np.zeros(200, np.int64), 1)


def test_chosen_tokens_and_misuse():
    cfg, w = hc.SINGLE, hc.weights(hc.SINGLE, 111)
    t = hc.tokens(cfg, 30, 112)
    want = oh.forward(cfg, w, t)
    dec = decoder(cfg, w, "fp32", max_seq=30)
    dec.extend(t[:21], [])
    got = [dec.step(x).cpu().numpy() for x in t[21:25]]
    got += list(portions(dec, t[25:], [3, 1]))
    assert hc.error(np.array(got), want[21:]) <= LIMIT["fp32"]
    with pytest.raises(lib.CtdkError):
        dec.step(1)                       # the cache is full
    with pytest.raises(lib.CtdkError):
        dec.extend([1], [])
    dec.reset()
    with pytest.raises(lib.CtdkError):
        dec.extend([1, 2], [2])           # not a row of the portion
    with pytest.raises(lib.CtdkError):
        dec.step(1)                       # no prompt yet


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    path = tmp_path_factory.mktemp("hybrid") / "m"
    w = hc.weights(hc.GROUPED, 121)
    hc.save_folder(path, hc.GROUPED, w)
    build.build()
    return path, w


@pytest.mark.parametrize("precision", ["bf16", "fp32"])
def test_command_line_generation(folder, precision):
    """ctd_generate on a model folder: greedy, and the same tokens from the sampler with top_k 1."""
    path, w = folder
    prompt = hc.tokens(hc.GROUPED, 33, 122)
    exe = Path(build.HERE) / "ctd_generate"

    def run(**req):
        r = subprocess.run([str(exe), "--model", str(path), "--precision", precision], capture_output=True, text=True, timeout=300,
                           input=json.dumps(dict(input_ids=prompt.tolist(), max_new_tokens=40, max_seq_len=128, seed=3, **req)))
        assert r.returncode == 0, r.stderr
        lines = [json.loads(x) for x in r.stdout.splitlines()]
        assert lines[-1]["done"] and lines[-1]["generated_tokens"] == 40
        return np.array([x["token"] for x in lines[:-1]])

    greedy = run(temperature=0.0)
    assert agrees_with_greedy(hc.GROUPED, w, prompt, greedy, 1e-3 if precision == "fp32" else 0.3)
    assert np.array_equal(run(temperature=1.0, top_k=1), greedy)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(folder, tmp_path, dtype):
    path, w = folder
    a, b = hc.tokens(hc.GROUPED, 50, 131), hc.tokens(hc.GROUPED, 20, 132)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:41].tolist(), want=[0, 40])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[41:42].tolist(), want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[42:].tolist(), want=[7, 1])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=b[:3].tolist(), want=[2])], end=[]),
             dict(step=4, entries=[dict(id="b", tokens=b[3:].tolist(), want=[16])], end=["b"])]
    r = subprocess.run([sys.executable, str(Path(build.HERE).parent / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "64"], capture_output=True, text=True, timeout=600,
                       input="".join(json.dumps(s) + "\n" for s in steps), env=dict(os.environ))
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not (tmp_path / "1.f32").exists()
    V = hc.GROUPED["vocab"]
    za, zb = oh.forward(hc.GROUPED, w, a), oh.forward(hc.GROUPED, w, b)
    lim = LIMIT["fp32" if dtype == "float32" else "bf16"]
    for step, want in ((0, za[[0, 40]]), (2, za[[49, 43]]), (3, zb[[2]]), (4, zb[[19]])):
        got = np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(-1, V)
        assert hc.error(got, want) <= lim, step


@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (2, 1000, 24), (130, 136, 72), (257, 512, 64), (300, 260, 1000), (512, 1024, 4096), (1000, 72, 136), (1000, 64, 2048)])
def test_bf16_product(M, N, K):
    """Small integers are exact in bfloat16 and in the fp32 sums: any misplaced tile shows as a wrong integer."""
    gen = torch.Generator(device="cuda").manual_seed(M + N + K)
    ld = (K + 7) // 8 * 8
    A = torch.full((M, ld), 9.0, device="cuda", dtype=torch.bfloat16)
    B = torch.full((N, ld), 9.0, device="cuda", dtype=torch.bfloat16)
    A[:, :K] = torch.randint(-3, 4, (M, K), generator=gen, device="cuda").to(torch.bfloat16)
    B[:, :K] = torch.randint(-3, 4, (N, K), generator=gen, device="cuda").to(torch.bfloat16)
    out = torch.full((M, N + 4), -7.0, device="cuda")
    lib.call("ctdk_gemm_bf16", A.data_ptr(), B.data_ptr(), out.data_ptr(), M, N, K, ld, ld, N + 4, torch.cuda.current_stream().cuda_stream)
    torch.cuda.synchronize()
    want = (A[:, :K].double() @ B[:, :K].double().T).float()
    assert torch.equal(out[:, :N], want)
    assert (out[:, N:] == -7.0).all()
