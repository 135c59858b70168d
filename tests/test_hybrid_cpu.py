"""Layer-list models without a GPU: the description read from config.json, the arena layout, refusals,
weight files, and properties of the oracle that the GPU tests lean on."""
import copy
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

from emberlm_b200 import build, lib, safetensors_io
from oracle import hybrid as oh
from tests import hybrid_cases as hc


def open_model(cfg, w, dtype="bf16"):
    from emberlm_b200 import engine as E
    return E.HybridModel(cfg, w, dtype)


@pytest.mark.parametrize("name", sorted(hc.CONFIGS))
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
def test_layout_covers_every_tensor_without_overlap(name, dtype):
    cfg = hc.CONFIGS[name]
    w = hc.weights(cfg, 1)
    m = open_model(cfg, w, dtype)
    assert m.vocab == cfg["vocab"]
    infos = {t.name.decode(): t for t in m.tensors}
    assert set(infos) == set(w)
    spans = []
    for n, t in infos.items():
        want = w[n].shape if w[n].ndim == 2 else (1,) + w[n].shape
        assert (t.rows, t.cols) == want
        assert t.ld >= t.cols and (not t.is_matrix or t.ld % 8 == 0) and t.offset % 16 == 0
        spans.append((t.offset, t.offset + t.rows * t.ld * (2 if t.is_matrix and dtype == "bf16" else 4)))
    spans.sort()
    assert all(a[1] <= b[0] for a, b in zip(spans, spans[1:])) and spans[-1][1] <= m.arena_bytes
    # one stacked operand per layer: q, k, gate and the second branch's rows share a pitch and follow one another
    q, k = infos["l0.mix.q" if "l0.mix.q" in infos else "l0.mix.left.q"], infos["l0.mix.k" if "l0.mix.q" in infos else "l0.mix.left.k"]
    assert k.offset == q.offset + (q.rows + 7) // 8 * 8 * q.ld * (2 if dtype == "bf16" else 4)


@pytest.mark.parametrize("edit,message", [
    (lambda c, w: c.update(architecture="Other"), "unknown architecture"),
    (lambda c, w: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c, w: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c, w: c["layers"][1]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c, w: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "one value per head"),
    (lambda c, w: c["layers"][0]["mixer"]["left"]["rot"].update(dims=15), "even"),
    (lambda c, w: c["layers"][0]["mixer"]["left"].update(vdim=12), "vdim == dim"),
    (lambda c, w: w.pop("l1.mix.a2"), "missing"),
    (lambda c, w: w.update({"l1.mix.q": w["l1.mix.q"][:-1]}), "does not fit the config"),
    (lambda c, w: c.pop("width"), "'width' not found"),
])
def test_bad_descriptions_are_refused(edit, message):
    cfg, w = copy.deepcopy(hc.GROUPED), hc.weights(hc.GROUPED, 1)
    edit(cfg, w)
    with pytest.raises(lib.CtdkError, match=message):
        open_model(cfg, w)


def test_optional_parts_of_the_config():
    cfg = copy.deepcopy(hc.GROUPED)
    cfg["layers"][0]["mixer"]["left"]["rot"]["scaling"] = None
    cfg["layers"][0]["mixer"]["left"]["mask"] = None      # every earlier position
    del cfg["layers"][1]["mlp"]
    open_model(cfg, hc.weights(hc.GROUPED, 1))


def test_bf16_files_round_trip(tmp_path):
    from emberlm_b200 import engine as E
    w = hc.weights(hc.SINGLE, 3)
    hc.save_folder(tmp_path / "m", hc.SINGLE, w)
    back = safetensors_io.load_safetensors(tmp_path / "m" / "model.safetensors")
    assert set(back) == set(w) and all(np.array_equal(back[k], w[k]) for k in w)
    m, loaded = E.HybridModel.from_folder(tmp_path / "m")
    assert m.vocab == hc.SINGLE["vocab"] and set(loaded) == set(w)


def test_rope_bands_of_the_oracle():
    s = dict(factor=4.0, low=1.0, high=4.0, original=64)
    f0, f1 = oh.rope_frequencies(16, 1e4), oh.rope_frequencies(16, 1e4, s)
    wl = 2 * np.pi / f0
    assert np.array_equal(f1[wl < 16], f0[wl < 16]) and (wl < 16).any()
    assert np.allclose(f1[wl > 64], f0[wl > 64] / 4) and (wl > 64).any()
    mid = (wl >= 16) & (wl <= 64)
    assert mid.any() and (f1[mid] < f0[mid]).all() and (f1[mid] > f0[mid] / 4).all()


def test_oracle_rows_depend_on_earlier_rows_only():
    cfg, w = hc.GROUPED, hc.weights(hc.GROUPED, 5)
    t = hc.tokens(cfg, 60, 6)
    full = oh.forward(cfg, w, t)
    assert np.allclose(full[:33], oh.forward(cfg, w, t[:33]), rtol=0, atol=1e-10)
    other = t.copy()
    other[40:] = (other[40:] + 1) % cfg["vocab"]
    assert np.allclose(full[:40], oh.forward(cfg, w, other)[:40], rtol=0, atol=1e-10)


def test_delta_rule_overwrites_what_a_key_held():
    """With beta 1, no decay and a repeated unit key, the second write replaces the first."""
    k = np.zeros((3, 1, 4))
    k[:, 0, 0] = 1.0
    v = np.array([[[1.0, 2.0]], [[5.0, -1.0]], [[7.0, 7.0]]])
    o = oh.channel_delta_rule(k, k, v, np.ones_like(k), np.ones((3, 1)))
    assert np.allclose(o[:, 0], v[:, 0])


def test_token_by_token_recurrence_equals_its_chunked_form():
    """The identity the prompt kernels use: inside a chunk U = T V - T K e^b S with the triangular T."""
    rng = np.random.default_rng(0)
    n, d, dv = 9, 5, 3
    q, k, v = rng.normal(size=(n, 1, d)), oh.unit(rng.normal(size=(n, 1, d))), rng.normal(size=(n, 1, dv))
    g, beta = rng.uniform(0.3, 1.0, size=(n, 1, d)), rng.uniform(size=(n, 1))
    want = oh.channel_delta_rule(q, k, v, g, beta)[:, 0]
    b = np.cumsum(np.log(g[:, 0]), axis=0)
    A = np.array([[(k[i, 0] * k[j, 0] * np.exp(b[i] - b[j])).sum() if j < i else 0.0 for j in range(n)] for i in range(n)])
    B = np.array([[(q[i, 0] * k[j, 0] * np.exp(b[i] - b[j])).sum() if j <= i else 0.0 for j in range(n)] for i in range(n)])
    T = np.linalg.inv(np.eye(n) + beta * A) * beta[:, 0]
    assert np.allclose(B @ (T @ v[:, 0]), want)


def test_tools_report_usage_and_bad_models(tmp_path):
    build.build()
    exe = Path(build.HERE) / "ctd_trace"
    assert subprocess.run([str(exe)], capture_output=True).returncode == 2
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Zutalix"}))
    (tmp_path / "model.safetensors").write_bytes((2).to_bytes(8, "little") + b"{}")
    r = subprocess.run([str(exe), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path)], capture_output=True,
                       text=True, input="")
    assert r.returncode == 1 and "not found" in r.stderr
