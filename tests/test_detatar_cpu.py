"""Detatar models without a GPU: the description read from config.json, the arena layout, refusals, and
properties of the oracle that the GPU tests lean on."""
import copy

import numpy as np
import pytest

from emberlm_b200 import lib
from oracle import detatar as od
from oracle.hybrid import rms_norm
from tests import detatar_cases as dc
from tests import hybrid_cases as hc


def open_model(cfg, w, dtype="bf16"):
    from emberlm_b200 import engine as E
    return E.HybridModel(cfg, w, dtype)


@pytest.mark.parametrize("name", sorted(dc.CONFIGS))
@pytest.mark.parametrize("dtype", ["bf16", "fp32"])
def test_layout_covers_every_tensor_without_overlap(name, dtype):
    cfg = dc.CONFIGS[name]
    w = dc.weights(cfg, 1)
    m = open_model(cfg, w, dtype)
    infos = {t.name.decode(): t for t in m.tensors}
    assert m.vocab == cfg["vocab"] and set(infos) == set(w)
    spans = []
    for n, t in infos.items():
        assert (t.rows, t.cols) == (w[n].shape if w[n].ndim == 2 else (1,) + w[n].shape)
        assert t.ld >= t.cols and (not t.is_matrix or t.ld % 8 == 0) and t.offset % 16 == 0
        spans.append((t.offset, t.offset + t.rows * t.ld * (2 if t.is_matrix and dtype == "bf16" else 4)))
    spans.sort()
    assert all(a[1] <= b[0] for a, b in zip(spans, spans[1:])) and spans[-1][1] <= m.arena_bytes
    # the experts of a layer stand at equal distances
    for i, lay in enumerate(cfg["layers"]):
        if lay["mlp"] and lay["mlp"]["kind"] == "moe" and "weights_of" not in lay:
            for part in ("gate", "up", "down"):
                at = [infos[f"l{i}.mlp.e{e}.{part}"].offset for e in range(lay["mlp"]["router"]["experts"])]
                assert len(set(np.diff(at))) <= 1


def set_router(c, **kw):
    c["layers"][0]["mlp"]["router"].update(kw)


@pytest.mark.parametrize("edit,message", [
    (lambda c, w: c["layers"][0].update(type="conv"), "unknown mixer type"),
    (lambda c, w: c["layers"][1]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c, w: c["norm"].update(groups=7), "divide the width"),
    (lambda c, w: c["layers"][4].update(weights_of=11), "must name a layer"),
    (lambda c, w: c["layers"][4].update(weights_of=6), "weights of its own"),
    (lambda c, w: set_router(c, groups={"count": 4, "keep": 1}), "equal groups"),
    (lambda c, w: set_router(c, groups={"count": 3, "keep": 1}, top=3), "fewer outputs"),
    (lambda c, w: c["layers"][1]["mixer"]["rot"].update(dims=4), "all of rot_dim"),
    (lambda c, w: w.pop("l0.mlp.e3.up"), "missing"),
    (lambda c, w: w.pop("l2.rg2"), "missing"),
    (lambda c, w: w.update({"l1.mix.uk": w["l1.mix.uk"][:-1]}), "does not fit the config"),
    (lambda c, w: c.pop("embedding"), "'embedding' not found"),
])
def test_bad_descriptions_are_refused(edit, message):
    cfg, w = copy.deepcopy(dc.ODD), dc.weights(dc.ODD, 1)
    edit(cfg, w)
    with pytest.raises(lib.CtdkError, match=message):
        open_model(cfg, w)


def test_optional_parts_of_the_config():
    cfg = copy.deepcopy(dc.ODD)
    del cfg["layers"][3]["mlp"]
    cfg["layers"][3]["weights_of"] = None
    cfg["layers"][2]["mlp"]["shared"] = None
    del cfg["layers"][7]["mlp"]
    cfg["layers"][7]["mlp"] = dc.dense(17)
    open_model(cfg, dc.weights(dc.ODD, 1))


def test_routing_by_hand():
    z = np.log(np.array([0.4, 0.1, 0.2, 0.05, 0.15, 0.1]))
    i, a = od.route(z, np.zeros(6), 2)
    assert list(i) == [0, 2] and np.allclose(a, [2 / 3, 1 / 3])
    # the correction decides who is chosen and leaves the weights alone
    i, a = od.route(z, np.array([-0.5, 0, 0, 0, 0.2, 0]), 2)
    assert list(i) == [4, 2] and np.allclose(a, [3 / 7, 4 / 7])
    # groups of two by their best: {0.4, 0.1} and {0.2, 0.05} stay, 0.15 may not be chosen
    i, a = od.route(z, np.zeros(6), 3, {"count": 3, "keep": 2})
    assert list(i) == [0, 2, 1] and np.allclose(a, np.array([4, 2, 1]) / 7)
    # negative choice scores of a kept group still beat a refused group
    i, _ = od.route(z, np.array([-2, -2, -2, -2, -0.1, -2]), 2, {"count": 3, "keep": 1})
    assert list(i) == [4, 5]
    assert np.isclose(od.route_margin(z, np.zeros(6), 2), 0.05)


def test_grouped_norm_and_token_mix():
    x = np.array([[3.0, 4.0, 0.5, 0.5]])
    y = od.grouped_rms_norm(x, np.ones(4), 0.0, 2)
    assert np.allclose(y, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 1, 1]])
    assert np.allclose(od.grouped_rms_norm(x, 2 * np.ones(4), 1e-3, 1), 2 * rms_norm(x, None, 1e-3))
    h = np.array([[1.0, 1.0], [2.0, 4.0], [0.0, 8.0]])
    assert np.allclose(od.token_mix(h, np.array([0.5, 1.0])), [[0.5, 0.0], [1.5, 1.0], [1.0, 4.0]])


def test_latent_form_equals_the_attention_over_cached_latents():
    """The identity the token kernel uses: W_uk^T q against the latents, W_uv of the mean latent."""
    rng = np.random.default_rng(0)
    T, H, d, dv, R = 7, 3, 4, 5, 6
    q, c = rng.normal(size=(T, H, d)), rng.normal(size=(T, R))
    uk, uv = rng.normal(size=(H, d, R)), rng.normal(size=(H, dv, R))
    want = od.causal_attention(q, np.einsum("hdr,tr->thd", uk, c), np.einsum("hdr,tr->thd", uv, c), 0.3)
    lat = np.repeat(c[:, None], H, axis=1)
    got = np.einsum("hvr,thr->thv", uv, od.causal_attention(np.einsum("thd,hdr->thr", q, uk), lat, lat, 0.3))
    assert np.allclose(got, want)


def test_time_mixing_equals_its_chunked_form():
    """The identity the prompt kernels use: with b the running sum of the log decays, o_i = (r_i e^(b_(i-1)))^T S
    plus, for j < i, (r_i . k_j e^(b_(i-1) - b_j)) v_j, plus the bonus term."""
    rng = np.random.default_rng(1)
    n, d = 11, 4
    r, k, v = (rng.normal(size=(n, 1, d)) for _ in range(3))
    w, u = rng.uniform(0.2, 1.0, size=(n, 1, d)), rng.normal(size=(1, d))
    want = od.wkv_recurrence(r, k, v, w, u)[:, 0]
    cut = 4
    S = np.zeros((d, d))
    for t in range(cut):
        S = w[t, 0][:, None] * S + np.outer(k[t, 0], v[t, 0])
    b = np.cumsum(np.log(w[cut:, 0]), axis=0)
    before = np.concatenate([np.zeros((1, d)), b[:-1]])
    R, K, V = r[cut:, 0], k[cut:, 0], v[cut:, 0]
    A = np.array([[(R[i] * K[j] * np.exp(before[i] - b[j])).sum() if j < i else (R[i] * u[0] * K[i]).sum() * (j == i)
                   for j in range(n - cut)] for i in range(n - cut)])
    assert np.allclose((R * np.exp(before)) @ S + A @ V, want[cut:])


def test_oracle_rows_depend_on_earlier_rows_only():
    cfg, w = dc.ODD, dc.weights(dc.ODD, 5)
    t = hc.tokens(cfg, 30, 6)
    full = od.forward(cfg, w, t)
    assert np.allclose(full[:17], od.forward(cfg, w, t[:17]), rtol=0, atol=1e-10)
    other = t.copy()
    other[20:] = (other[20:] + 1) % cfg["vocab"]
    assert np.allclose(full[:20], od.forward(cfg, w, other)[:20], rtol=0, atol=1e-10)
    assert not np.allclose(full[20:], od.forward(cfg, w, other)[20:])
