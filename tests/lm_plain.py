"""Plain, slow statement of the decoder language models the library serves (the Kegizen and Bupozen
designs), in double precision, one function per mechanism. For tests only: it shares nothing with the product.

Weights are a dict name -> float64 array, the configuration is the dict of a model folder's
config.json. Sequences are processed one token at a time wherever a mechanism has memory, so what
these functions say about a prompt is what they say about decoding it."""
import json
import math
import os

import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def layer_norm(x, w, eps):
    """Centre, divide by the standard deviation (eps under the root), scale by w. No bias."""
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def swiglu(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def rope_frequencies(rot):
    """Angle per position of each rotated pair, and the factor on cos and sin."""
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turn(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turn(sc["fast"])), 0)
    hi = min(math.ceil(turn(sc["slow"])), dims - 1)
    r = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * r + f * (1.0 - r), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims dimensions of a head, i paired with i + dims/2."""
    if not rot:
        return x
    f, m = rope_frequencies(rot)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * f
    c, s = np.cos(a) * m, np.sin(a) * m
    half = rot["dims"] // 2
    u, v = x[..., :half], x[..., half:2 * half]
    out = x.copy()
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def visible(i, j, mask):
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


def attention(h, w, name, mix, eps):
    """Windowed softmax attention over a whole sequence h [T, width]."""
    T = h.shape[0]
    H, G, d, vd = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms_norm(h @ w[name + ".q"].T, w[name + ".q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ w[name + ".k"].T, w[name + ".k.norm"], eps).reshape(T, G, d)
    v = (h @ w[name + ".v"].T).reshape(T, G, vd)
    pos = np.arange(T)
    q, k = rotate(q, pos, mix.get("rot")), rotate(k, pos, mix.get("rot"))
    mask = np.array([[visible(i, j, mix.get("mask")) for j in range(T)] for i in range(T)])
    out = np.zeros((T, H, vd))
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * mix["scale"]
        if mix.get("softcap"):
            s = mix["softcap"] * np.tanh(s / mix["softcap"])
        s = np.where(mask, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hd] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out.reshape(T, H * vd) @ w[name + ".o"].T


def causal_conv_silu(x, taps):
    """x [T, channels], taps [channels, n] with the last column on the current token."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return silu(sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def delta_rule(q, k, v, beta, g, state=None):
    """Gated delta rule of one head, token by token: q, k [T, dim], v [T, vdim], beta, g [T].
    Returns the read-outs [T, vdim] and the final state [dim, vdim]."""
    S = np.zeros((k.shape[1], v.shape[1])) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def delta(h, w, name, mix, eps):
    """Gated delta-rule mixer over a whole sequence h [T, width]."""
    T = h.shape[0]
    H, G, d, vd = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q, k, v = (causal_conv_silu(h @ w[f"{name}.{c}"].T, w[f"{name}.{c}.conv"]) for c in "qkv")
    q, k, v = q.reshape(T, G, d), k.reshape(T, G, d), v.reshape(T, H, vd)
    q = q / np.sqrt((q * q).sum(axis=-1, keepdims=True) + 1e-6) * d ** -0.5
    k = k / np.sqrt((k * k).sum(axis=-1, keepdims=True) + 1e-6)
    beta = sigmoid(h @ w[name + ".b"].T)
    g = np.exp(-np.exp(w[name + ".A_log"]) * softplus(h @ w[name + ".a"].T + w[name + ".dt_bias"]))
    gate = silu(h @ w[name + ".g"].T).reshape(T, H, vd)
    out = np.zeros((T, H, vd))
    for hd in range(H):
        kv = hd // (H // G)
        o, _ = delta_rule(q[:, kv], k[:, kv], v[:, hd], beta[:, hd], g[:, hd])
        out[:, hd] = rms_norm(o, w[name + ".norm"], eps) * gate[:, hd]
    return out.reshape(T, H * vd) @ w[name + ".o"].T


def rotate_neighbours(x, positions, rot):
    """x [T, ..., dim]: the first rot.dims dimensions, 2i paired with 2i + 1."""
    if not rot:
        return x
    f, m = rope_frequencies(rot)
    n = rot["dims"]
    a = np.asarray(positions, dtype=np.float64).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    c, s = np.cos(a) * m, np.sin(a) * m
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.copy()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def latent_memory(h, w, name, mix, eps):
    """What a latent attention keeps of every token: the normed latent [T, kv_rank] and the rotated key part
    [T, rot_dim] that all heads share."""
    y = h @ w[name + ".dkv"].T
    r = mix["kv_rank"]
    return rms_norm(y[:, :r], w[name + ".dkv.norm"], eps), rotate_neighbours(y[:, r:], np.arange(h.shape[0]), mix.get("rot"))


def latent_attention(h, w, name, mix, eps, memory):
    """Attention whose keys and values are read out of a latent (c, shared key part), with a gate per head."""
    T = h.shape[0]
    H, d, e, vd = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    c, shared = memory
    q = (rms_norm(h @ w[name + ".dq"].T, w[name + ".dq.norm"], eps) @ w[name + ".uq"].T).reshape(T, H, d + e)
    q_plain, q_rot = q[..., :d], rotate_neighbours(q[..., d:], np.arange(T), mix.get("rot"))
    k = (c @ w[name + ".uk"].T).reshape(T, H, d)
    v = (c @ w[name + ".uv"].T).reshape(T, H, vd)
    gate = sigmoid(h @ w[name + ".g"].T)
    mask = np.array([[visible(i, j, mix.get("mask")) for j in range(T)] for i in range(T)])
    out = np.zeros((T, H, vd))
    for hd in range(H):
        s = (q_plain[:, hd] @ k[:, hd].T + q_rot[:, hd] @ shared.T) * mix["scale"]
        s = np.where(mask, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hd] = (p / p.sum(axis=1, keepdims=True)) @ v[:, hd] * gate[:, hd, None]
    return out.reshape(T, H * vd) @ w[name + ".o"].T


def relu2_mlp(h, up, down):
    return np.maximum(h @ up.T, 0.0) ** 2 @ down.T


def route(h, router, top):
    """Per token: the `top` experts with the largest logits, and the softmax over their logits."""
    z = h @ router.T
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=1)
    p = np.exp(zc - zc.max(axis=1, keepdims=True))
    return chosen, p / p.sum(axis=1, keepdims=True)


def experts_mlp(h, w, name, spec):
    chosen, weight = route(h, w[name + ".router"], spec["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(chosen[t], weight[t]):
            out[t] += p * relu2_mlp(h[t:t + 1], w[f"{name}.e{e}.up"], w[f"{name}.e{e}.down"])[0]
    return out


def parallel_layer(x, w, i, cfg, memories):
    """One norm feeds the mixer and the feed-forward; both are added to the stream. `memories`: what the
    latent attentions before this one keep, by layer; a layer with kv_from reads another layer's."""
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    mix, mlp = spec["mixer"], spec.get("mlp")
    h = rms_norm(x, w[f"l{i}.norm1"], eps)
    if mix.get("kv_from") is None:
        memories[i] = latent_memory(h, w, f"l{i}.mix", mix, eps)
        source = i
    else:
        source = mix["kv_from"]
    y = latent_attention(h, w, f"l{i}.mix", mix, eps, memories[source])
    if mlp and mlp["kind"] == "moe":
        y = y + experts_mlp(h, w, f"l{i}.mlp", mlp)
    elif mlp:
        y = y + relu2_mlp(h, w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"])
    return x + y


MIXERS = {"delta": delta, "attention": attention}


def layer(x, w, i, cfg):
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]

    def norm(y, which):
        return layer_norm(y, w[f"l{i}.{which}"], eps)

    x = x + norm(MIXERS[spec["type"]](norm(x, "norm1"), w, f"l{i}.mix", spec["mixer"], eps), "norm1b")
    if spec.get("mlp"):
        y = swiglu(norm(x, "norm2"), w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"])
        x = x + norm(y, "norm2b")
    return x


def layer_runs(cfg):
    """(layer, starts a pass) in execution order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for _ in range(loop["times"]):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(w, cfg, tokens):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width]."""
    x0 = w["embed"][np.asarray(tokens)]
    x, taps, memories = x0, [], {}
    if cfg["architecture"] == "Bupozen":
        for i in range(len(cfg["layers"])):
            x = parallel_layer(x, w, i, cfg, memories)
            taps.append(x)
        return rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T, np.stack(taps)
    for i, starts_pass in layer_runs(cfg):
        if starts_pass:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        x = layer(x, w, i, cfg)
        taps.append(x)
    return layer_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T, np.stack(taps)


def greedy(w, cfg, prompt, n):
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(np.argmax(forward(w, cfg, tokens)[0][-1])))
    return tokens[len(prompt):]


def load_folder(path):
    """(config, weights as float64) of a model folder: config.json + model.safetensors."""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    w = {}
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        head, data = json.loads(f.read(n)), f.read()
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        if t["dtype"] == "BF16":
            raw = np.frombuffer(data[lo:hi], dtype="<u2").astype(np.uint32) << 16
            a = raw.view(np.float32)
        else:
            a = np.frombuffer(data[lo:hi], dtype={"F32": "<f4", "I32": "<i4"}[t["dtype"]])
        w[name] = a.astype(np.float64).reshape(t["shape"])
    return cfg, w
