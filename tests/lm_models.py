"""Small decoder language models for the tests: configurations, random weights, model folders."""
import json
import os

import numpy as np


def bf16(a):
    """Round to nearest BF16, as uint16."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def delta(heads=3, kv_heads=1, dim=24, vdim=40, conv=3, ff=72):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


YARN = {"factor": 3.0, "original": 640, "fast": 24.0, "slow": 1.5}


def attention(heads=4, kv_heads=2, dim=32, vdim=48, window=17, keep=3, rot=16, base=5000.0, scaling=YARN, scale=0.21,
              softcap=15.0, ff=72):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = scaling
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=4, dim=24, rot_dim=8, vdim=40, kv_rank=48, q_rank=56, window=19, scale=0.3, base=3000.0, kv_from=None, ff=72, experts=0, top=2,
           rot=None):
    """A latent attention beside a squared-ReLU feed-forward, one or `experts` of size ff (0: none)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim if rot is None else rot}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    mlp = None
    if ff and experts:
        mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    elif ff:
        mlp = {"kind": "dense", "ff": ff}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers, width=136, vocab=203, loop=None, eps=2e-5):
    name = "Bupozen" if layers[0]["type"] == "latent_attention" else "Kegizen"
    c = {"architecture": name, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if cfg.get("loop"):
        s["loop.in"] = (W, 2 * W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}", l["mixer"]
        if l["type"] == "latent_attention":
            s.update(latent_shapes(l, p, W))
            continue
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        s[f"{p}.norm1"] = s[f"{p}.norm1b"] = (W,)
        if l["type"] == "delta":
            rows = {"q": G * d, "k": G * d, "v": H * vd}
            for n, r in rows.items():
                s[f"{p}.mix.{n}.conv"] = (r, m["conv"])
            rows.update(g=H * vd, b=H, a=H)
            s[f"{p}.mix.A_log"] = s[f"{p}.mix.dt_bias"] = (H,)
            s[f"{p}.mix.norm"] = (vd,)
        else:
            rows = {"q": H * d, "k": G * d, "v": G * vd}
            s[f"{p}.mix.q.norm"], s[f"{p}.mix.k.norm"] = (H * d,), (G * d,)
        for n, r in rows.items():
            s[f"{p}.mix.{n}"] = (r, W)
        s[f"{p}.mix.o"] = (W, H * vd)
        if l.get("mlp"):
            ff = l["mlp"]["ff"]
            s[f"{p}.norm2"] = s[f"{p}.norm2b"] = (W,)
            s[f"{p}.mlp.gate"] = s[f"{p}.mlp.up"] = (ff, W)
            s[f"{p}.mlp.down"] = (W, ff)
    return s


def latent_shapes(l, p, W):
    m, mlp = l["mixer"], l["mlp"]
    H, R, Q = m["heads"], m["kv_rank"], m["q_rank"]
    s = {f"{p}.norm1": (W,), f"{p}.mix.dq": (Q, W), f"{p}.mix.dq.norm": (Q,), f"{p}.mix.uq": (H * (m["dim"] + m["rot_dim"]), Q)}
    if m.get("kv_from") is None:
        s[f"{p}.mix.dkv"], s[f"{p}.mix.dkv.norm"] = (R + m["rot_dim"], W), (R,)
    s.update({f"{p}.mix.uk": (H * m["dim"], R), f"{p}.mix.uv": (H * m["vdim"], R), f"{p}.mix.g": (H, W), f"{p}.mix.o": (W, H * m["vdim"])})
    if mlp and mlp["kind"] == "moe":
        s[f"{p}.mlp.router"] = (mlp["router"]["experts"], W)
        for e in range(mlp["router"]["experts"]):
            s[f"{p}.mlp.e{e}.up"], s[f"{p}.mlp.e{e}.down"] = (mlp["expert"]["ff"], W), (W, mlp["expert"]["ff"])
    elif mlp:
        s[f"{p}.mlp.up"], s[f"{p}.mlp.down"] = (mlp["ff"], W), (W, mlp["ff"])
    return s


def weights(cfg, seed, qk_gain=1.6):
    """BF16 values (as uint16) by name. Routers choose clearly. Query and key gains are large enough that a softmax puts most
    of its weight on a few keys, decays range from almost none to almost all, gains are not one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        z = rng.standard_normal(shape)
        if name.endswith((".q.norm", ".k.norm", ".dq.norm")):
            a = qk_gain * (1.0 + 0.2 * z)
        elif "norm" in name:
            a = 1.0 + 0.2 * z
        elif name.endswith("A_log"):
            a = rng.uniform(-6.0, 1.0, shape)
        elif name.endswith("dt_bias"):
            a = 0.5 * z - 0.5
        elif name.endswith(".conv"):
            a = 0.6 * z
        elif name == "embed":
            a = z
        elif name.endswith(".router"):
            a = 3.0 * z / np.sqrt(shape[-1])
        else:
            a = z / np.sqrt(shape[-1]) * (2.0 if name == "head" else 1.0)
        out[name] = bf16(a)
    return out


LIMIT = {"float32": 2e-5, "bfloat16": 4e-4}      # summation order; two-term BF16 products of prompts
DTYPES = ("float32", "bfloat16")


class Case:
    """A model folder with its weights in double precision."""

    def __init__(self, mod, path, cfg, seed, **kw):
        self.mod, self.cfg = mod, cfg
        w = weights(cfg, seed, **kw)
        self.folder = write_folder(path, cfg, w)
        self.w = as_float(w)

    def rewrite(self):
        write_folder(self.folder, self.cfg, {n: bf16(a) for n, a in self.w.items()})
        self.w = as_float({n: bf16(a) for n, a in self.w.items()})

    def open(self, dtype, **kw):
        kw.setdefault("max_tokens", 2048)
        return self.mod.LanguageModel(self.folder, dtype=dtype, **kw)


def feed(lm, seq, toks, sizes):
    """Logits at every place, the tokens cut into portions of the given sizes (repeated)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - at)
        out.append(lm.step(seq, toks[at:at + n], range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)


def as_float(w):
    return {n: (a.astype(np.uint32) << 16).view(np.float32).astype(np.float64) for n, a in w.items()}


def write_folder(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, at = {"__metadata__": {"format": "pt"}}, 0
    for n, a in w.items():
        head[n] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    blob = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(blob).to_bytes(8, "little") + blob)
        for a in w.values():
            f.write(a.tobytes())
    return str(path)


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def error(got, want):
    """Largest root mean square over the vocabulary of a position's difference (means taken off), in units
    of the logits' own spread."""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=-1)).max() / np.std(want))
