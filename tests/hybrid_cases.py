"""Small layer-list models for the tests: configurations, random weights (rounded to bfloat16, as the
weight files hold them), files, and the error measure."""
import json
import struct

import numpy as np


def attention(heads, kv_heads, dim, chunk, rot_dims, base=1e4, scaling=None, scale=None):
    rot = {"dims": rot_dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "rot": rot,
            "scale": scale or dim ** -0.5}


def lightning(heads, dim, vdim, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.6 + 0.39 * i / max(heads - 1, 1) for i in range(heads)]}


def parallel(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def mlp(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def model(vocab, width, layers, eps=1e-5):
    return {"architecture": "Zutalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Grouped heads everywhere, sizes that are no multiples of anything, rotation of a part of the head with
# all three frequency bands, both orders of layers, a feed-forward on each mixer type and on neither.
GROUPED = model(130, 92, [
    parallel(attention(4, 2, 36, 24, 16, scaling=(4.0, 1.0, 4.0, 64)), lightning(3, 40, 24), mlp(150, 1.5)),
    delta(6, 3, 48, 20, 4),
    delta(2, 1, 20, 44, 4, mlp(70, 0.7)),
    parallel(attention(3, 1, 20, 7, 20, base=500.0), lightning(2, 12, 36)),
], eps=1e-3)
# One head of everything, tensor-core head sizes, another number of taps, no frequency scaling.
SINGLE = model(64, 64, [
    delta(1, 1, 128, 128, 3),
    parallel(attention(1, 1, 128, 40, 128), lightning(1, 128, 128, [0.97]), mlp(128, 3.0)),
    delta(2, 2, 64, 64, 4, mlp(64, 2.0)),
    parallel(attention(2, 2, 64, 128, 32), lightning(2, 64, 64)),
])
# Head sizes above the tile kernels' (token-by-token recurrences, fp32 attention), a chunk longer than the cache.
WIDE = model(72, 40, [
    parallel(attention(2, 1, 160, 1000, 48), lightning(2, 72, 136), mlp(40, 1.0)),
    delta(2, 1, 136, 40, 6),
    delta(1, 1, 24, 136, 1),
])
CONFIGS = {"grouped": GROUPED, "single": SINGLE, "wide": WIDE}


def bf16(a):
    """Rounds to bfloat16 (ties to even), kept as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32).reshape(np.shape(a))


def weights(cfg, seed, rank=(12, 20)):
    """Random weights by tensor name; low-rank widths of the delta layers from `rank`."""
    rng = np.random.default_rng(seed)
    W, out = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        out[name] = rng.normal(0.0, gain / np.sqrt(k), (n, k))

    def norm(name, n):
        out[name] = 1.0 + 0.2 * rng.normal(size=n)

    out["embed"] = rng.normal(size=(cfg["vocab"], W))
    norm("embed.norm", W)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        norm(p + "norm1", W)
        norm(p + "norm1b", W)
        if lay["type"] == "parallel":
            a, r, q = m["left"], m["right"], p + "mix.left."
            n, nk = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            mat(q + "q", n, W, 1.7)
            mat(q + "k", nk, W, 1.7)
            out[q + "q.b"], out[q + "k.b"] = 0.5 * rng.normal(size=n), 0.5 * rng.normal(size=nk)
            mat(q + "g", a["heads"], W)
            mat(q + "o", W, n)
            q, n, nv = p + "mix.right.", r["heads"] * r["dim"], r["heads"] * r["vdim"]
            mat(q + "q", n, W)
            mat(q + "k", n, W)
            mat(q + "v", nv, W)
            mat(q + "g", nv, W)
            mat(q + "o", W, nv)
            norm(q + "norm", nv)
            norm(p + "mix.left.out", W)
            norm(p + "mix.right.out", W)
        else:
            q, nq, nh, nv = p + "mix.", m["kv_heads"] * m["dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for t, n in (("q", nq), ("k", nq), ("v", nv)):
                mat(q + t, n, W)
                out[q + t + ".conv"] = 0.6 * rng.normal(size=(n, m["conv"]))
            mat(q + "b", m["heads"], W)
            out[q + "A_log"] = 0.5 * rng.normal(size=m["heads"]) - 1.0
            out[q + "dt_bias"] = rng.normal(size=nh) - 1.0
            norm(q + "norm", m["vdim"])
            mat(q + "a1", rank[0], W)
            mat(q + "a2", nh, rank[0])
            mat(q + "g1", rank[1], W)
            mat(q + "g2", nv, rank[1])
            mat(q + "o", W, nv)
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            norm(p + "norm2", W)
            norm(p + "norm2b", W)
            mat(p + "mlp.gate", ff, W, 1.5)
            mat(p + "mlp.up", ff, W, 1.5)
            mat(p + "mlp.down", W, ff)
    norm("final.norm", W)
    mat("head", cfg["vocab"], W)
    return {k: bf16(v) for k, v in out.items()}


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)


def error(got, want):
    """Root mean square difference of the rows, largest row, relative to the whole's root mean square."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = np.sqrt(np.mean((got - want) ** 2, axis=-1))
    return float(np.max(d) / np.sqrt(np.mean(want ** 2)))


def save_folder(path, cfg, w):
    """config.json and a bfloat16 model.safetensors."""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blobs, at = {}, [], 0
    for n, a in w.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[n] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + b"".join(blobs))
