"""Serving throughput (prefill and greedy decode, batch 1) of the layer-list designs beside the preset
decoder closest to them, at equal width, depth, (active) feed-forward width and vocabulary. Random weights.

  python -m emberlm_b200.serve_bench --size 0.6b            # one JSON line per model
  python -m emberlm_b200.serve_bench --size 1.7b --layers 4 # a short stack (per-kernel profiles)

Times are CUDA events on the decoder's stream. Weights (and for short stacks the activations) are
larger than L2."""
from __future__ import annotations

import argparse
import json

import torch

from . import engine as E
from . import lib

# preset, (attention heads, kv heads, head size, recurrent heads, recurrent head size, low rank)
SIZES = {"0.6b": ("qwen3_0_6b", (8, 4, 128, 8, 128, 128)), "1.7b": ("qwen3_1_7b", (16, 8, 128, 16, 128, 128))}


def zutalix_config(preset: dict, shape, layers: int, chunk: int = 1024) -> dict:
    """A Zutalix of the preset's width, feed-forward width, vocabulary and `layers` layers: one
    delta-rule layer in four, the rest chunked attention beside lightning attention."""
    H, G, D, R, RD, _ = shape
    rot = {"dims": D, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    mlp = {"kind": "dense", "ff": preset["intermediate_size"], "limit": 7.0}
    par = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": chunk}, "rot": rot},
           "right": {"heads": R, "dim": RD, "vdim": RD, "decay": [1.0 - 2.0 ** (-2 - 6.0 * i / R) for i in range(R)]}}
    delta = {"heads": R, "kv_heads": R, "dim": RD, "vdim": RD, "conv": 4}
    kinds = [("channel_delta", delta) if i % 4 == 0 else ("parallel", par) for i in range(layers)]
    return {"architecture": "Zutalix", "vocab": preset["vocab_size"], "width": preset["hidden_size"], "norm": {"eps": 1e-5},
            "layers": [{"type": t, "mixer": m, "mlp": mlp} for t, m in kinds]}


def zutalix_shapes(cfg: dict, rank: int) -> dict:
    W = cfg["width"]
    s = {"embed": [cfg["vocab"], W], "embed.norm": [W], "final.norm": [W], "head": [cfg["vocab"], W]}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        s[p + "norm1"] = s[p + "norm1b"] = [W]
        if lay["type"] == "parallel":
            a, r, q = m["left"], m["right"], p + "mix."
            n = a["heads"] * a["dim"]
            s |= {q + "left.q": [n, W], q + "left.q.b": [n], q + "left.k": [a["kv_heads"] * a["dim"], W],
                  q + "left.k.b": [a["kv_heads"] * a["dim"]], q + "left.g": [a["heads"], W], q + "left.o": [W, n]}
            n, nv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            s |= {q + "right.q": [n, W], q + "right.k": [n, W], q + "right.v": [nv, W], q + "right.g": [nv, W],
                  q + "right.o": [W, nv], q + "right.norm": [nv], q + "left.out": [W], q + "right.out": [W]}
        else:
            n, nq, nv, q = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], p + "mix."
            s |= {q + "q": [nq, W], q + "q.conv": [nq, m["conv"]], q + "k": [nq, W], q + "k.conv": [nq, m["conv"]],
                  q + "v": [nv, W], q + "v.conv": [nv, m["conv"]], q + "b": [m["heads"], W], q + "A_log": [m["heads"]],
                  q + "norm": [m["vdim"]], q + "a1": [rank, W], q + "a2": [n, rank], q + "dt_bias": [n], q + "g1": [rank, W],
                  q + "g2": [nv, rank], q + "o": [W, nv]}
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            s |= {p + "norm2": [W], p + "norm2b": [W], p + "mlp.gate": [ff, W], p + "mlp.up": [ff, W], p + "mlp.down": [W, ff]}
    return s


# (heads, dim, rot_dim, vdim, kv_rank, q_rank), (wkv heads, dim, rank); the active experts and the shared one
# add up to the preset's feed-forward width
DETATAR_SIZES = {"0.6b": ((16, 64, 32, 64, 256, 512), (16, 64, 64)), "1.7b": ((16, 128, 64, 128, 512, 1024), (32, 64, 64))}
EXPERTS, IDENTITY, TOP, GROUPS = 40, 8, 4, (8, 5)


def detatar_config(preset: dict, size: str, layers: int) -> dict:
    """A Detatar of the preset's width, vocabulary and `layers` layers: one time-mixing layer in four, the rest
    latent attention; a dense feed-forward in the first layer, mixtures of experts in the others."""
    (H, D, DR, DV, R, Q), (RH, RD, _) = DETATAR_SIZES[size]
    ff = preset["intermediate_size"]
    lat = {"heads": H, "dim": D, "rot_dim": DR, "vdim": DV, "kv_rank": R, "q_rank": Q, "scale": (D + DR) ** -0.5, "rot": {"base": 1e6, "dims": DR}}
    moe = {"kind": "moe", "expert": {"ff": ff // 6}, "shared": {"ff": ff - TOP * (ff // 6)},
           "router": {"experts": EXPERTS, "identity": IDENTITY, "top": TOP, "groups": {"count": GROUPS[0], "keep": GROUPS[1]}}}
    kinds = [("wkv", {"heads": RH, "dim": RD}) if i % 4 == 3 else ("latent_attention", lat) for i in range(layers)]
    return {"architecture": "Detatar", "vocab": preset["vocab_size"], "width": preset["hidden_size"], "embedding": {"scale": 1.0},
            "norm": {"eps": 1e-5, "groups": 2},
            "layers": [{"type": t, "mixer": m, "mlp": moe if i else {"kind": "dense", "ff": ff}} for i, (t, m) in enumerate(kinds)]}


def detatar_shapes(cfg: dict, rank: int) -> dict:
    W = cfg["width"]
    s = {"embed": [cfg["vocab"], W], "final.norm": [W], "head": [cfg["vocab"], W]}

    def glu(p, ff):
        return {p + "gate": [ff, W], p + "up": [ff, W], p + "down": [W, ff]}

    for i, lay in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", lay["mixer"], lay["mlp"]
        q, H = p + "mix.", m["heads"]
        s |= {p + "norm1": [W], p + "shift": [W], p + "rg1": [W, W], p + "rg1.b": [W], p + "rg2": [W, W], p + "rg2.b": [W]}
        if lay["type"] == "latent_attention":
            s |= {q + "dq": [m["q_rank"], W], q + "dq.norm": [m["q_rank"]], q + "uq": [H * (m["dim"] + m["rot_dim"]), m["q_rank"]],
                  q + "dkv": [m["kv_rank"] + m["rot_dim"], W], q + "dkv.norm": [m["kv_rank"]], q + "uk": [H * m["dim"], m["kv_rank"]],
                  q + "uv": [H * m["vdim"], m["kv_rank"]], q + "g": [H, W], q + "o": [W, H * m["vdim"]]}
        else:
            n = H * m["dim"]
            s |= {q + "mu." + x: [W] for x in "rkvgw"} | {q + x: [n, W] for x in "rkvg"}
            s |= {q + "w1": [rank, W], q + "w2": [n, rank], q + "w0": [n], q + "u": [H, m["dim"]], q + "norm": [n], q + "o": [W, n]}
        if f["kind"] == "dense":
            s |= glu(p + "mlp.", f["ff"])
        else:
            n = f["router"]["experts"] + f["router"]["identity"]
            for e in range(f["router"]["experts"]):
                s |= glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
            s |= {p + "mlp.router": [n, W], p + "mlp.correction": [n], p + "mlp.shared.sg": [1, W]} | glu(p + "mlp.shared.", f["shared"]["ff"])
    return s


def build_detatar(size: str, layers: int | None, max_seq: int, max_portion: int, dtype: str = "bf16"):
    preset = E.PRESETS[SIZES[size][0]]
    cfg = detatar_config(preset, size, layers or preset["num_hidden_layers"])
    model = E.HybridModel(cfg, detatar_shapes(cfg, DETATAR_SIZES[size][1][2]), dtype)
    dec = E.HybridDecoder(model, max_seq, max_portion)
    gen = torch.Generator(device="cuda").manual_seed(1234)
    views = dec.named_parameters()
    streamed = 0.0   # parameters a token reads: experts by the share of them that are chosen, no embedding
    for t in model.tensors:
        name = t.name.decode()
        v = views[name]
        if t.is_matrix:
            v.normal_(0.0, 0.02, generator=gen)
        elif name.endswith(("correction", ".b", "w0", ".u")):
            v.normal_(-1.0 if name.endswith("w0") else 0.0, 0.02 if name.endswith("correction") else 0.5, generator=gen)
        elif name.endswith("shift") or ".mu." in name:
            v.uniform_(0.0, 1.0, generator=gen)
        else:
            v.fill_(1.0)
        share = TOP / (EXPERTS + IDENTITY) if ".mlp.e" in name else (0.0 if name == "embed" else 1.0)
        streamed += share * t.rows * t.cols
    return dec, sum(t.rows * t.cols for t in model.tensors), int(streamed)


def build_zutalix(size: str, layers: int | None, max_seq: int, max_portion: int, dtype: str = "bf16"):
    preset = E.PRESETS[SIZES[size][0]]
    shape = SIZES[size][1]
    cfg = zutalix_config(preset, shape, layers or preset["num_hidden_layers"])
    model = E.HybridModel(cfg, zutalix_shapes(cfg, shape[5]), dtype)
    dec = E.HybridDecoder(model, max_seq, max_portion)
    gen = torch.Generator(device="cuda").manual_seed(1234)
    for t in model.tensors:
        v = dec.named_parameters()[t.name.decode()]
        if t.is_matrix or t.name.endswith(b".conv"):
            v.normal_(0.0, 0.02 if t.is_matrix else 0.3, generator=gen)
        elif t.name.endswith((b".b", b"A_log", b"dt_bias")):
            v.normal_(0.0, 0.5, generator=gen)
        else:
            v.fill_(1.0)
    return dec, sum(t.rows * t.cols for t in model.tensors)


def build_preset(size: str, layers: int | None, max_seq: int):
    preset = dict(E.PRESETS[SIZES[size][0]])
    if layers:
        preset["num_hidden_layers"] = layers
    dec = E.Decoder(E.make_config(**preset), max_seq)
    gen = torch.Generator(device="cuda").manual_seed(1234)
    for (_, v), dcy in zip(dec.named_parameters().items(), dec.layout.decay):
        v.normal_(0.0, 0.02, generator=gen) if dcy else v.fill_(1.0)
    return dec, sum(dec.layout.numels)


def measure(dec, vocab: int, prompt_len: int, new_tokens: int, steps: int, warmup: int, sampler=None) -> dict:
    """Milliseconds per prefill of prompt_len tokens and per greedy token after it. sampler: makes an object
    with start() / stop() that watches the clocks of the timed steps."""
    L, s = E._L, dec.stream
    gen = torch.Generator(device="cuda").manual_seed(7)
    ids = torch.randint(0, vocab, (prompt_len,), generator=gen, device="cuda")
    out = torch.zeros(new_tokens + 1, dtype=torch.int64, device="cuda")
    torch.cuda.synchronize()
    pre = dcd = 0.0
    watch, launches = sampler() if sampler else None, 0
    with torch.cuda.stream(s):
        for i in range(warmup + steps):
            if i == warmup:
                launches = L.ctdk_launch_count()
                if watch:
                    watch.start()
            e = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
            e[0].record(s)
            lib.check(L.ctdk_decode_prefill(dec._h, ids.data_ptr(), prompt_len, s.cuda_stream))
            e[1].record(s)
            lib.check(L.ctdk_decode_greedy(dec._h, new_tokens, out.data_ptr(), s.cuda_stream))
            e[2].record(s)
            lib.check(L.ctdk_device_status(s.cuda_stream, None))
            if i >= warmup:
                pre += e[0].elapsed_time(e[1])
                dcd += e[1].elapsed_time(e[2])
    launches = L.ctdk_launch_count() - launches
    extra = {"clocks": watch.stop()} if watch else {}
    return {**extra, "gpu_launches": launches, "prefill_ms": pre / steps, "prefill_tokens_per_s": prompt_len * steps / pre * 1e3, "token_ms": dcd / steps / new_tokens,
            "decode_tokens_per_s": new_tokens * steps / dcd * 1e3}


def run(size: str, layers: int | None = None, prompt_len: int = 4096, new_tokens: int = 128, steps: int = 5, warmup: int = 3,
        models=("zutalix", "preset"), sampler=None) -> list[dict]:
    rows = []
    for which in models:
        max_seq = prompt_len + new_tokens + 64
        preset = which == "preset"
        if which == "detatar":
            dec, params, streamed = build_detatar(size, layers, max_seq, prompt_len)
        else:
            dec, params = build_preset(size, layers, max_seq) if preset else build_zutalix(size, layers, max_seq, prompt_len)
            streamed = params
        r = measure(dec, dec.vocab, prompt_len, new_tokens, steps, warmup, sampler)
        rows.append({"model": SIZES[size][0] if preset else f"{which}-{size}", "dtype": "tf32 prefill, fp32 decode" if preset else "bf16",
                     "params": params, "streamed_params": streamed, "prompt_len": prompt_len, "new_tokens": new_tokens, **r,
                     "decode_weight_gbs": streamed * (4 if preset else 2) / r["token_ms"] / 1e6})
        del dec
        torch.cuda.empty_cache()
    return rows


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", choices=sorted(SIZES), default="0.6b")
    ap.add_argument("--layers", type=int, default=None)
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--new", type=int, default=128)
    ap.add_argument("--steps", type=int, default=5)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--models", default="detatar,zutalix,preset")
    a = ap.parse_args()
    for r in run(a.size, a.layers, a.prompt, a.new, a.steps, a.warmup, tuple(a.models.split(","))):
        print(json.dumps(r), flush=True)


if __name__ == "__main__":
    main()
