"""A plain, slow implementation of the Marotar decoder in f64 on the CPU, written from its equations: one function per
mechanism, whole sequences at once, every score of every pair computed and masked.  Nothing here is shared with the package.

Weights: a dict name -> f64 tensor, names as in a checkpoint.  `config` is the design's config.json as a dict.
"""
import math

import torch


def rms(x, eps):
    """x over its root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def pair_frequencies(rot):
    """(frequency of each pair, factor on cosine and sine)"""
    d, base = rot["dims"], float(rot["base"])
    freqs = [base ** (-2.0 * i / d) for i in range(d // 2)]
    s = rot.get("scaling")
    if not s:
        return freqs, 1.0

    def at(turns):
        return d * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), d - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append((f / s["factor"]) * r + f * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [tokens, ..., width]: pairs (2i, 2i + 1) of the first rot.dims dimensions turned by position * frequency."""
    freqs, mag = pair_frequencies(rot)
    y = x.clone()
    for i, f in enumerate(freqs):
        a = (positions.double() * f).reshape(-1, *[1] * (x.dim() - 2))
        c, s = torch.cos(a) * mag, torch.sin(a) * mag
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(n, window):
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def latent_attention(h, w, m, eps):
    """h [tokens, width] from position 0; w(name) the mixer's tensors; m its sizes."""
    n, heads, pos = h.shape[0], m["heads"], torch.arange(h.shape[0])
    q = (rms(h @ w("dq").T, eps) * w("dq.norm")) @ w("uq").T
    q = q.reshape(n, heads, m["dim"] + m["rot_dim"])
    down = h @ w("dkv").T
    c = rms(down[:, :m["kv_rank"]], eps) * w("dkv.norm")
    shared = rotate(down[:, m["kv_rank"]:], pos, m["rot"])
    k = (c @ w("uk").T).reshape(n, heads, m["dim"])
    v = (c @ w("uv").T).reshape(n, heads, m["vdim"])
    q_rot = rotate(q[..., m["dim"]:], pos, m["rot"])
    score = torch.einsum("ihd,jhd->hij", q[..., :m["dim"]], k) + torch.einsum("ihd,jd->hij", q_rot, shared)
    score = (score * m["scale"]).masked_fill(~visible(n, (m.get("mask") or {}).get("size")), -math.inf)
    o = torch.einsum("hij,jhd->ihd", torch.softmax(score, -1), v)
    return o.reshape(n, -1) @ w("o").T


def feed_forward(h, w):
    return (h @ w("up").T + w("up.b")).clamp_min(0).square() @ w("down").T + w("down.b")


def forward(config, weights, tokens, trace=None):
    """Logits [tokens, vocab]; trace receives the residual stream after every layer."""
    t = {k: v.double() for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(config["layers"]):
        j = i
        while config["layers"][j].get("weights_of") is not None:
            j = config["layers"][j]["weights_of"]
        y = latent_attention(zero_centred_norm(x, t[f"l{j}.norm1"], eps), lambda n: t[f"l{j}.mix.{n}"], layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + feed_forward(zero_centred_norm(x, t[f"l{j}.norm2"], eps), lambda n: t[f"l{j}.mlp.{n}"])
        x = x + y
        if trace is not None:
            trace.append(x)
    return zero_centred_norm(x, t["final.norm"], eps) @ t["embed"].T


def greedy(config, weights, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(config, weights, out)[-1].argmax()))
    return out[len(prompt):]


# ---------------------------------------------------------------------------------------------- small models

def mixer(heads=3, dim=24, rot_dim=8, vdim=40, q_rank=56, kv_rank=48, window=20, base=5000.0, rot_dims=None, scaling=True, scale=None):
    rot = {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}
    if scaling:
        rot["scaling"] = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 1.0}
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot": rot,
         "scale": scale if scale is not None else 1.5 * (dim + rot_dim) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return m


def layer(ff=88, weights_of=None, **kw):
    out = {"type": "latent_attention", "mixer": mixer(**kw), "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def model(*layers, width=72, vocab=131, eps=1e-5):
    return {"architecture": "Marotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": list(layers)}


def make_weights(config, seed=0, q_gain=1.0):
    """Random tensors with values bf16 can hold.  q_gain scales the query latent's norm weight: larger makes single keys stand
    out in the softmax."""
    g = torch.Generator().manual_seed(seed)
    width, out = config["width"], {}

    def put(name, *shape, std, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16).float()

    put("embed", config["vocab"], width, std=1.0)
    put("final.norm", width, std=0.2)
    for i, l in enumerate(config["layers"]):
        if l.get("weights_of") is not None:
            continue
        m, p = l["mixer"], f"l{i}."
        put(p + "norm1", width, std=0.2)
        put(p + "mix.dq", m["q_rank"], width, std=width ** -0.5)
        put(p + "mix.dq.norm", m["q_rank"], std=0.2 * q_gain, mean=q_gain)
        put(p + "mix.uq", m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], std=m["q_rank"] ** -0.5)
        put(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], width, std=width ** -0.5)
        put(p + "mix.dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
        put(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], std=m["kv_rank"] ** -0.5)
        put(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"], std=m["kv_rank"] ** -0.5)
        put(p + "mix.o", width, m["heads"] * m["vdim"], std=(m["heads"] * m["vdim"]) ** -0.5)
        if l.get("mlp"):
            ff = l["mlp"]["ff"]
            put(p + "norm2", width, std=0.2)
            put(p + "mlp.up", ff, width, std=width ** -0.5)
            put(p + "mlp.up.b", ff, std=0.3)
            put(p + "mlp.down", width, ff, std=0.5 * ff ** -0.5)
            put(p + "mlp.down.b", width, std=0.3)
    return out


def save(folder, config, weights):
    """config.json and model.safetensors as a checkpoint has them."""
    import json
    import os
    import struct

    header, data, at = {}, [], 0
    for name, w in weights.items():
        raw = w.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [at, at + len(raw)]}
        data.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(data))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
