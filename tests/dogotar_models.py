"""Small Dogotar configurations and random weights of the tests' own making (no code of the package is used to draw or name a
tensor): config.json contents, a tensor dictionary by checkpoint name, and a folder writer."""

from __future__ import annotations

import json
from pathlib import Path

import torch
from safetensors.torch import save_file


def attention(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, cap=6.0, window=9, rot=(4, 900.0, 3.0), v_mix=True, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap is not None:
        m["softcap"] = cap
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        dims, base, factor = rot
        m["rot"] = {"base": base, "dims": dims}
        if factor is not None:
            m["rot"]["scaling"] = {"factor": factor}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": mlp}


def left(heads=3, kv_heads=1, dim=10, vdim=7, scale=0.35, cap=5.0, chunk=11):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap is not None:
        m["softcap"] = cap
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return m


def right(heads=2, dim=6, vdim=10, cap=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def parallel(a=None, b=None, scales=(0.7, 1.3), mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a or left(), "left_scale": scales[0], "right": b or right(), "right_scale": scales[1]}}


def dense(ff=20):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=61, width=24, eps=2e-5):
    return {"architecture": "Dogotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that differ wherever a model could happen to make them equal or 1: key and value sizes, query heads per key/value head
# (1, 2, 3), windows, chunks and neither, whole and partial rotations with and without scaling and none, caps and none, value
# mixing in some layers only (the first attention without it), factors below and above one, layers without a feed-forward, either
# mixer first and last, sizes that are no multiples of 8 and sizes of the tensor-core kernels.  The larger eps of the deep ones keep
# read-outs of a few numbers from being blown up where they happen to be tiny (and show whether eps is where it belongs).
CONFIGS = {
    "attention_only": config([attention(), attention(2, 2, 8, 6, v_mix=True, window=5, rot=(8, 50.0, None))], vocab=59),
    "parallel_only": config([parallel()], width=20, eps=1e-3),
    "mixed": config([
        attention(6, 3, 12, 5, 0.3, 4.0, 20, (6, 300.0, 2.0), v_mix=False, mlp=dense(30)),
        parallel(left(4, 2, 16, 10, 0.25, 7.0, 21), right(3, 12, 5, 3.0), (1.2, 0.6), dense(26)),
        attention(4, 1, 16, 9, 0.3, None, None, (16, 5000.0, None), v_mix=True, mlp=None),
        parallel(left(2, 2, 6, 14, 0.4, None, None), right(1, 9, 20, 12.0), (-0.5, 2.0), None),
        attention(2, 1, 10, 9, 0.33, 9.0, 33, None, v_mix=True, mlp=dense(17)),
        attention(9, 3, 8, 3, 0.5, 3.0, 14, (2, 40.0, 5.0), v_mix=True, mlp=dense(24)),
    ], vocab=131, width=40, eps=4e-3),
    # sizes in the multiples the tensor-core kernels and the wide accesses take, gaps and none between joined rows
    "wide": config([
        attention(4, 2, 64, 32, 0.12, 8.0, 50, (32, 2000.0, 2.5), mlp=dense(192)),
        parallel(left(4, 2, 64, 64, 0.125, 6.0, 70), right(2, 64, 72, 15.0), (0.6, 0.9), dense(128)),
        parallel(left(4, 1, 32, 64, 0.2, 5.0, 90), right(3, 40, 24, 6.0), (0.8, 0.7), None),
        attention(2, 2, 128, 32, 0.09, 10.0, 130, (64, 20000.0, 4.0), mlp=dense(256)),
        parallel(left(2, 2, 128, 40, 0.1, None, 128), right(2, 136, 136, 10.0), (0.5, 0.5), dense(64)),
    ], vocab=300, width=128, eps=2e-3),
}


def tensors(cfg, seed=0, dtype=torch.float32, std=0.5):
    """Checkpoint name -> tensor.  Matrices scaled so that activations stay of order one; norm gains around one; biases, gates
    and shares large enough to matter."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return torch.randn(*shape, generator=g) * s

    w = cfg["width"]
    out = {"embed": rnd(cfg["vocab"], w, s=0.8), "final.norm": 1 + rnd(w, s=0.1), "final.norm.b": rnd(w, s=0.2)}

    def normed_attention(p, m, gate):
        h, kv = m["heads"], m["kv_heads"]
        for n, rows in (("q", h * m["dim"]), ("k", kv * m["dim"]), ("v", kv * m["vdim"])):
            out[f"{p}{n}"] = rnd(rows, w, s=2 * std / w ** 0.5)
            out[f"{p}{n}.b"] = rnd(rows, s=0.4)
            if n != "v":
                out[f"{p}{n}.norm"] = 1 + rnd(m["dim"], s=0.3)
        if gate:
            out[p + "g"] = rnd(h * m["vdim"], w, s=3 * std / w ** 0.5)
        out[p + "o"] = rnd(w, h * m["vdim"], s=2 * std / (h * m["vdim"]) ** 0.5)

    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        for n in ("norm1",) + (("norm2",) if lay["mlp"] else ()):
            out[p + n] = 1 + rnd(w, s=0.2)
            out[p + n + ".b"] = rnd(w, s=0.2)
        if lay["type"] == "attention":
            normed_attention(p + "mix.", m, gate=True)
            if m.get("v_mix"):
                out[p + "mix.vmix"] = torch.tensor(0.35 + 0.1 * i)
        else:
            normed_attention(p + "mix.left.", m["left"], gate=False)
            b = m["right"]
            qk, v = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            for n, rows in (("q", qk), ("k", qk), ("v", v), ("g", v)):
                out[f"{p}mix.right.{n}"] = rnd(rows, w, s=2 * std / w ** 0.5)
            out[p + "mix.right.o"] = rnd(w, v, s=2 * std / v ** 0.5)
            out[p + "mix.right.norm"] = 1 + rnd(v, s=0.2)
            for n, at in (("i", -0.5), ("f", 2.0)):
                out[f"{p}mix.right.{n}"] = rnd(b["heads"], w, s=2.0 / w ** 0.5)
                out[f"{p}mix.right.{n}.b"] = at + rnd(b["heads"], s=1.0)
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            out[p + "mlp.up"] = rnd(ff, w, s=2 * std / w ** 0.5)
            out[p + "mlp.down"] = rnd(w, ff, s=2 * std / ff ** 0.5)
    return {k: v.to(dtype).contiguous() for k, v in out.items()}


def write_folder(folder, cfg, weights) -> Path:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return folder
