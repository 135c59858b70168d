"""Detatar decoders on the GPU against the plain oracle (oracle/detatar.py, float64): every mechanism alone,
whole prompts, portions, single tokens, sequences on used state, far keys, first tokens, long decoding,
generation through the framework's entry points. fp32 models are held to fp32 rounding; bf16 models to the
rounding of bfloat16 products."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from emberlm_b200 import build, lib
from oracle import detatar as od
from tests import detatar_cases as dc
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


def share(cfg, w, dec, t):
    """What the only layer adds to the residual: (framework's, oracle's)."""
    trace = torch.zeros(1, len(t), cfg["width"], device="cuda")
    dec.trace_layers(trace)
    dec.extend(t)
    dec.trace_layers(None)
    dec.reset()
    layers = []
    od.forward(cfg, w, t, layers)
    x0 = w["embed"][t].astype(np.float64) * cfg["embedding"]["scale"]
    return trace[0].cpu().numpy() - x0, layers[0] - x0


def close(w, gate):
    """The sublayer behind l0.rg1 / l0.rg2 contributes nothing."""
    w[f"l0.{gate}.b"] = np.full_like(w[f"l0.{gate}.b"], -200.0)
    return w


MIXERS = [dc.latent(4, 36, 16, 24, 40, 28), dc.latent(6, 64, 64, 64, 128, 96), dc.latent(2, 128, 64, 128, 512, 64), dc.latent(3, 96, 32, 64, 72, 200),
          dc.latent(1, 8, 8, 8, 8, 8), dc.latent(17, 16, 8, 8, 24, 16), dc.latent(3, 5, 2, 3, 11, 7), dc.latent(2, 200, 40, 130, 600, 33),
          dc.latent(2, 16, 32, 256, 64, 48), dc.latent(1, 64, 128, 40, 1000, 8),
          dc.wkv(3, 40), dc.wkv(6, 64), dc.wkv(2, 128), dc.wkv(1, 17), dc.wkv(1, 200), dc.wkv(9, 1), dc.wkv(2, 32), dc.wkv(2, 100)]
FFS = [dc.dense(150), dc.dense(9), dc.dense(256), dc.moe(5, 2, 36), dc.moe(8, 8, 16, shared=24), dc.moe(6, 3, 64, identity=3, groups=(3, 2), shared=9),
       dc.moe(30, 6, 128, identity=2, groups=(8, 3)), dc.moe(1, 1, 20, identity=1), dc.moe(40, 1, 8, groups=(40, 1)), dc.moe(270, 3, 8, identity=2, groups=(16, 4)), dc.moe(100, 5, 16, shared=8), dc.moe(2, 2, 300, identity=2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(MIXERS)))
def test_each_mixer_alone(case, dtype):
    # a norm over a single column is its sign: the large eps keeps it from magnifying rounding
    eps = 1e-1 if MIXERS[case]["mixer"]["dim"] == 1 else 1e-5
    cfg = dc.model(50, 72, [dict(MIXERS[case], mlp=dc.dense(8))], groups=[1, 2, 9][case % 3], eps=eps)
    w = close(dc.weights(cfg, 10 + case, rank=[9, 32, 64][case % 3]), "rg2")
    t = hc.tokens(cfg, 150, case)
    dec = decoder(cfg, w, dtype)
    got, want = share(cfg, w, dec, t)
    assert hc.error(got, want) <= LIMIT[dtype]
    want = od.forward(cfg, w, t)
    for sizes in ([150], [100, 1], [1], [2], [31, 33]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(FFS)))
def test_each_feed_forward_alone(case, dtype):
    """Free routing: tokens whose choice is close are left out in bfloat16 (their layer input is rounded)."""
    f = FFS[case]
    cfg = dc.model(300, [72, 264, 41][case % 3], [dict(dc.wkv(1, 8), mlp=f)], groups=1)
    w = close(dc.weights(cfg, 30 + case, clear_choice=False), "rg1")
    t = hc.tokens(cfg, 250, case)
    keep = np.ones(len(t), bool)
    if f["kind"] == "moe":
        h = od.grouped_rms_norm(w["embed"][t].astype(float) * cfg["embedding"]["scale"], w["l0.norm1"], cfg["norm"]["eps"], 1)
        r = f["router"]
        gap = np.array([od.route_margin(w["l0.mlp.router"].astype(float) @ x, w["l0.mlp.correction"].astype(float), r["top"], r.get("groups"))
                        for x in h])
        keep = gap > ((1e-2 if r["experts"] < 64 else 2e-3) if dtype == "bf16" else 1e-5)   # scores shrink with their number
        assert keep.sum() > 100
    dec = decoder(cfg, w, dtype)
    got, want = share(cfg, w, dec, t)
    assert hc.error(got[keep], want[keep]) <= LIMIT[dtype]
    want = od.forward(cfg, w, t)
    for sizes in ([250], [1], [3]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes)[keep], want[keep]) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(dc.CONFIGS))
def test_whole_prompt_portions_and_tokens_agree_with_the_oracle(name, dtype):
    cfg = dc.CONFIGS[name]
    w = dc.weights(cfg, 21)
    t = hc.tokens(cfg, 140, 22)
    want = od.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype)
    runs = {"whole": [140], "tokens": [1], "pairs": [2], "odd": [37, 2, 3, 1, 23], "halves": [64, 63, 65], "prompt, then tokens": [97] + [1] * 43}
    for label, sizes in runs.items():
        dec.reset()      # on the cache and state of the run before
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], label


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_longer_than_a_portion_are_cut_inside(dtype):
    cfg, w = dc.EVEN, dc.weights(dc.EVEN, 31)
    t = hc.tokens(cfg, 130, 32)
    want = od.forward(cfg, w, t)
    for part in (33, 32):      # both parities of the shift state's slots
        dec = decoder(cfg, w, dtype, max_portion=part)
        rows = [0, part - 1, part, part + 1, 2 * part, 3 * part - 1, 129]
        assert hc.error(dec.extend(t, rows).cpu().numpy(), want[rows]) <= LIMIT[dtype]
        rows = [129, 5, 5, 40]      # any order, also twice
        dec.reset()
        assert hc.error(dec.extend(t, rows).cpu().numpy(), want[rows]) <= LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_after_one_another_do_not_see_each_other(dtype):
    cfg, w = dc.ODD, dc.weights(dc.ODD, 41)
    dec = decoder(cfg, w, dtype)
    for i, n in enumerate([90, 1, 2, 3, 25, 120, 4]):
        t = hc.tokens(cfg, n, 50 + i)
        dec.reset()
        got = portions(dec, t, [[n], [1], [2, 1], [50, 1]][i % 4])
        assert hc.error(got, od.forward(cfg, w, t)) <= LIMIT[dtype], n


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(dtype):
    """A missing previous row is zero, not the row itself: shift and mixes of one (the previous row alone)."""
    cfg = dc.model(50, 48, [dc.wkv(2, 24, dc.dense(40)), dc.latent(2, 16, 8, 16, 24, 16)], groups=2)
    w = dc.weights(cfg, 51)
    for n in w:
        if n.endswith(".shift") or ".mu." in n:
            w[n] = hc.bf16(np.full_like(w[n], 0.95))
    t = hc.tokens(cfg, 9, 52)
    want = od.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype)
    for sizes in ([9], [1], [2], [3], [1, 8], [2, 7], [5, 4]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes
        dec.reset()
        assert hc.error(portions(dec, t[::-1].copy(), sizes), od.forward(cfg, w, t[::-1])) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_stands_out(dtype):
    """One token's key answers one token's query so strongly that a single position decides, near the start and
    at both sides of the tiles' edges. The oracle without that position, or with a rotation one off, is far
    outside the limit."""
    cfg = dc.model(40, 64, [dc.latent(2, 32, 16, 32, 48, 32, base=1e5)], groups=1)
    w = dc.weights(cfg, 61)
    w["l0.shift"] = np.zeros_like(w["l0.shift"])
    cfg["layers"][0]["mixer"]["scale"] = 0.9
    T = 300
    rng = np.random.default_rng(62)
    h = od.grouped_rms_norm(w["embed"].astype(float), w["l0.norm1"], cfg["norm"]["eps"], 1)
    # the pair (asking token, answering token) whose unrotated score stands out most among all answers
    eps, p, m = cfg["norm"]["eps"], "l0.mix.", cfg["layers"][0]["mixer"]
    q = (od.rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(40, 2, 48)[:, :, :32]
    k = (od.rms_norm((h @ w[p + "dkv"].T)[:, :48], w[p + "dkv.norm"], eps) @ w[p + "uk"].T).reshape(40, 2, 32)
    s = np.einsum("ahd,bhd->hab", q, k)
    two = -np.sort(-s, axis=2)[:, :, :2]
    head, ask = np.unravel_index(np.argmax(two[:, :, 0] - two[:, :, 1]), two.shape[:2])
    answer = int(np.argmax(s[head, ask]))
    others = np.array([x for x in range(40) if x not in (ask, answer)])
    dec = decoder(cfg, w, dtype, max_seq=T)
    for far in (0, 1, 31, 32, 63, 64, 127, 128, 129, 255):
        t = rng.choice(others, size=T)
        t[far] = answer
        t[[far + 20, 280, 298, 299]] = ask
        rows = [far + 20, 280, 298, 299]
        want = od.forward(cfg, w, t)[rows]
        lost = t.copy()
        lost[far] = others[0]
        assert hc.error(od.forward(cfg, w, lost)[rows], want) > 2.5 * LIMIT[dtype]
        for sizes in ([T], [far + 1, T], [290] + [1] * 10, [far + 20, 1, T]):
            dec.reset()
            assert hc.error(portions(dec, t, sizes)[rows], want) <= LIMIT[dtype], (far, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_memory_of_the_recurrence_is_carried(dtype):
    """Slow decays, so that what was written long ago still counts; the oracle that forgets at a portion's
    start is far outside the limit. A layer that runs a second time has a memory of its own."""
    layers = [dc.wkv(2, 32), dc.wkv(1, 64, dc.dense(40))]
    cfg = dc.model(40, 48, layers + [dc.again(layers, 0)])
    w = dc.weights(cfg, 71)
    for i in (0, 1):
        w[f"l{i}.mix.w0"] = hc.bf16(w[f"l{i}.mix.w0"] * 0.2 - 6.0)
    t = hc.tokens(cfg, 200, 72)
    want = od.forward(cfg, w, t)
    for cut in (64, 150):
        assert hc.error(od.forward(cfg, w, t[cut:]), want[cut:]) > 3 * LIMIT[dtype]
    dec = decoder(cfg, w, dtype)
    for sizes in ([200], [64, 1], [150, 50], [16], [15], [17, 47, 63, 65], [128, 72], [65, 2]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("w0,bonus", [(5.0, 1.0), (-9.0, 0.0), (0.0, 3.0), (2.5, 0.3)])
def test_time_mixing_with_strong_and_weak_decays(w0, bonus, dtype):
    """Decays that wipe a channel within a token (e^-148) or hardly move it: nothing overflows. The large eps
    keeps heads whose output is small from magnifying their own rounding."""
    cfg = dc.model(40, 48, [dc.wkv(2, 64), dc.wkv(1, 20), dc.wkv(1, 128)], eps=0.3)
    w = dc.weights(cfg, 81)
    for i in range(3):
        w[f"l{i}.mix.w0"] = hc.bf16(w[f"l{i}.mix.w0"] * 0.3 + w0)
        w[f"l{i}.mix.u"] = hc.bf16(w[f"l{i}.mix.u"] * bonus + 0.5)
    t = hc.tokens(cfg, 170, 82)
    want = od.forward(cfg, w, t)
    dec = decoder(cfg, w, dtype)
    for sizes in ([170], [1], [33, 2], [64, 106]):
        dec.reset()
        assert hc.error(portions(dec, t, sizes), want) <= LIMIT[dtype], sizes


def test_many_rows_per_expert():
    """Several tiles for one expert, none for another, wide and narrow products."""
    for width, ff, experts in ((328, 296, 3), (64, 24, 12)):
        cfg = dc.model(50, width, [dict(dc.wkv(1, 8), mlp=dc.moe(experts, 2, ff, identity=1, shared=16))], groups=2)
        w = dc.weights(cfg, 91)
        t = hc.tokens(cfg, 600, 92)
        want = od.forward(cfg, w, t)
        for dtype in DTYPES:
            dec = decoder(cfg, w, dtype, max_seq=600, max_portion=600)
            assert hc.error(portions(dec, t, [600]), want) <= LIMIT[dtype]
            dec.reset()
            assert hc.error(portions(dec, t, [300, 299, 1]), want) <= LIMIT[dtype]


def agrees_with_greedy(cfg, w, prompt, got, margin):
    """Every generated token is the oracle's arg-max of its prefix, up to near ties."""
    seq = np.concatenate([prompt, got])
    z = od.forward(cfg, w, seq)[len(prompt) - 1:-1]
    best = z.max(axis=1)
    return all(best[i] - z[i, got[i]] <= margin for i in range(len(got)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even"])
def test_greedy_generation(name, dtype):
    cfg = dc.CONFIGS[name]
    w = dc.weights(cfg, 101)
    prompt = hc.tokens(cfg, 19, 102)
    dec = decoder(cfg, w, dtype, max_seq=400)
    got = dec.generate(prompt, 500).cpu().numpy()      # up to the end of the cache, in one burst
    assert len(got) == 400 - 19 + 1
    margin = 1e-3 if dtype == "fp32" else 0.3
    assert agrees_with_greedy(cfg, w, prompt, got, margin)
    z = dec.last_logits().cpu().numpy()
    full = od.forward(cfg, w, np.concatenate([prompt, got[:-1]]))[-1]
    assert hc.error(z[None], full[None]) <= LIMIT[dtype] * 2
    assert dec.generate(prompt[:1], 5).cpu().numpy().shape == (5,)


def test_two_sequences_of_one_model():
    """Two live sequences share the weights and nothing else."""
    from emberlm_b200 import engine as E
    cfg, w = dc.ODD, dc.weights(dc.ODD, 111)
    model = E.HybridModel(cfg, w, "fp32")
    one = E.HybridDecoder(model, 64, 64)
    one.load_parameters(w)
    two = E.HybridDecoder(model, 64, 64, params=one.params)
    a, b = hc.tokens(cfg, 40, 112), hc.tokens(cfg, 33, 113)
    za, zb = [], []
    for i in range(0, 40, 3):
        za.append(portions(one, a[i:i + 3], [3]))
        if i < 33:
            zb.append(portions(two, b[i:i + 3], [1, 2]))
    assert hc.error(np.concatenate(za), od.forward(cfg, w, a)) <= LIMIT["fp32"]
    assert hc.error(np.concatenate(zb), od.forward(cfg, w, b)) <= LIMIT["fp32"]


def test_chosen_tokens_and_misuse():
    cfg, w = dc.EVEN, dc.weights(dc.EVEN, 121)
    t = hc.tokens(cfg, 30, 122)
    want = od.forward(cfg, w, t)
    dec = decoder(cfg, w, "fp32", max_seq=30)
    dec.extend(t[:21], [])
    got = [dec.step(x).cpu().numpy() for x in t[21:25]]
    got += list(portions(dec, t[25:], [3, 1]))
    assert hc.error(np.array(got), want[21:]) <= LIMIT["fp32"]
    with pytest.raises(lib.CtdkError):
        dec.step(1)                       # the cache is full
    with pytest.raises(lib.CtdkError):
        dec.extend([1], [])


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    path = tmp_path_factory.mktemp("detatar") / "m"
    w = dc.weights(dc.ODD, 131)
    hc.save_folder(path, dc.ODD, w)
    build.build()
    return path, w


@pytest.mark.parametrize("precision", ["bf16", "fp32"])
def test_command_line_generation(folder, precision):
    """ctd_generate on a model folder: greedy, and the same tokens from the sampler with top_k 1."""
    path, w = folder
    prompt = hc.tokens(dc.ODD, 33, 132)
    exe = Path(build.HERE) / "ctd_generate"

    def run(**req):
        r = subprocess.run([str(exe), "--model", str(path), "--precision", precision], capture_output=True, text=True, timeout=300,
                           input=json.dumps(dict(input_ids=prompt.tolist(), max_new_tokens=40, max_seq_len=128, seed=3, **req)))
        assert r.returncode == 0, r.stderr
        lines = [json.loads(x) for x in r.stdout.splitlines()]
        assert lines[-1]["done"] and lines[-1]["generated_tokens"] == 40
        return np.array([x["token"] for x in lines[:-1]])

    greedy = run(temperature=0.0)
    assert agrees_with_greedy(dc.ODD, w, prompt, greedy, 1e-3 if precision == "fp32" else 0.3)
    assert np.array_equal(run(temperature=1.0, top_k=1), greedy)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(folder, tmp_path, dtype):
    path, w = folder
    a, b = hc.tokens(dc.ODD, 50, 141), hc.tokens(dc.ODD, 20, 142)
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
    V = dc.ODD["vocab"]
    za, zb = od.forward(dc.ODD, w, a), od.forward(dc.ODD, w, b)
    lim = LIMIT["fp32" if dtype == "float32" else "bf16"]
    for step, want in ((0, za[[0, 40]]), (2, za[[49, 43]]), (3, zb[[2]]), (4, zb[[19]])):
        got = np.fromfile(tmp_path / f"{step}.f32", np.float32).reshape(-1, V)
        assert hc.error(got, want) <= lim, step
