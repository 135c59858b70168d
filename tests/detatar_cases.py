"""Small Detatar models for the tests: configurations and random weights (rounded to bfloat16, as the weight
files hold them). Files, tokens and the error measure come from hybrid_cases."""
import numpy as np

from tests.hybrid_cases import bf16


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=1e4, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def wkv(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, groups=None, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def again(layers, j):
    """Layer j's weights once more."""
    return dict(layers[j], weights_of=j)


def model(vocab, width, layers, groups=1, eps=1e-5, scale=1.0):
    return {"architecture": "Detatar", "vocab": vocab, "width": width, "embedding": {"scale": scale},
            "norm": {"eps": eps, "groups": groups}, "layers": layers}


# Sizes that are no multiples of anything, three norm groups, every kind of feed-forward on each mixer, a layer
# of each kind used twice.
_odd = [
    wkv(3, 20, moe(5, 2, 36, identity=1, groups=(3, 2), shared=20)),
    latent(3, 20, 6, 12, 28, 20, base=700.0, scale=0.5, mlp=dense(50)),
    latent(5, 12, 10, 28, 44, 36, scale=0.4, mlp=moe(6, 3, 24, identity=2, groups=(4, 3))),
    wkv(2, 44),
]
ODD = model(130, 60, _odd + [again(_odd, 0), latent(1, 7, 2, 5, 9, 3), again(_odd, 2), wkv(1, 9, dense(17))], groups=3, eps=1e-3, scale=3.0)
# Sizes of the tensor-core kernels; one group, top 1, all outputs chosen, many groups with one kept.
_even = [
    latent(2, 64, 64, 64, 128, 64, base=5e5, mlp=moe(4, 1, 64, shared=64)),
    wkv(2, 64, dense(128)),
    latent(4, 32, 16, 48, 64, 96, mlp=moe(3, 4, 32, identity=1)),
    wkv(1, 128, moe(14, 2, 40, identity=2, groups=(8, 1))),
    latent(3, 128, 64, 128, 256, 128),
]
EVEN = model(96, 128, _even + [again(_even, 3)], groups=4)
# Head sizes above the tile kernels', more norm groups than warps, a wide latent, one-wide heads.
WIDE = model(72, 48, [
    latent(2, 136, 72, 144, 520, 40, mlp=moe(2, 1, 8, groups=(2, 1))),
    wkv(1, 136),
    latent(9, 1, 2, 1, 6, 5),
    wkv(5, 1, moe(1, 1, 16, identity=1, shared=8)),
], groups=12, eps=1e-2, scale=0.7)
CONFIGS = {"odd": ODD, "even": EVEN, "wide": WIDE}


def weights(cfg, seed, rank=12, clear_choice=True):
    """Random weights by tensor name. clear_choice: the routers' corrections are so far apart that rounding
    cannot change a choice (the weights still vary); otherwise they only tilt it."""
    rng = np.random.default_rng(seed)
    W, out = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        out[name] = rng.normal(0.0, gain / np.sqrt(k), (n, k))

    def norm(name, n):
        out[name] = 1.0 + 0.2 * rng.normal(size=n)

    def glu(p, ff):
        mat(p + "gate", ff, W, 1.5)
        mat(p + "up", ff, W, 1.5)
        mat(p + "down", W, ff)

    out["embed"] = rng.normal(size=(cfg["vocab"], W)) / cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        if "weights_of" in lay:
            continue
        p, m, f = f"l{i}.", lay["mixer"], lay["mlp"]
        q, H = p + "mix.", m["heads"]
        norm(p + "norm1", W)
        out[p + "shift"] = rng.uniform(size=W)
        for g in ("rg1", "rg2") if f else ("rg1",):
            mat(p + g, W, W)
            out[p + g + ".b"] = 1.0 + 0.5 * rng.normal(size=W)
        if lay["type"] == "latent_attention":
            mat(q + "dq", m["q_rank"], W)
            norm(q + "dq.norm", m["q_rank"])
            mat(q + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.7)
            mat(q + "dkv", m["kv_rank"] + m["rot_dim"], W, 1.7)
            norm(q + "dkv.norm", m["kv_rank"])
            mat(q + "uk", H * m["dim"], m["kv_rank"], 1.7)
            mat(q + "uv", H * m["vdim"], m["kv_rank"])
            mat(q + "g", H, W)
            mat(q + "o", W, H * m["vdim"])
        else:
            n = H * m["dim"]
            for s in "rkvgw":
                out[q + "mu." + s] = rng.uniform(size=W)
            for s in "rkvg":
                mat(q + s, n, W)
            mat(q + "w1", rank, W)
            mat(q + "w2", n, rank)
            out[q + "w0"] = rng.normal(size=n) - 2.0
            out[q + "u"] = rng.normal(size=(H, m["dim"]))
            norm(q + "norm", n)
            mat(q + "o", W, n)
        if f and f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
        elif f:
            r = f["router"]
            n = r["experts"] + r["identity"]
            for e in range(r["experts"]):
                glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
            mat(p + "mlp.router", n, W, 1.5)
            out[p + "mlp.correction"] = 1.25 * rng.permutation(n) - n / 2 if clear_choice else 0.1 * rng.normal(size=n)
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"])
                mat(p + "mlp.shared.sg", 1, W)
    norm("final.norm", W)
    mat("head", cfg["vocab"], W)
    return {k: bf16(v) for k, v in out.items()}
