"""A plain, slow implementation of the Videdra decoder in f64 on the CPU, written from its equations: one function per mechanism, whole
sequences at once, every score of every pair computed and masked, the recurrence token by token.  Nothing here is shared with the
package.

Weights: a dict name -> tensor, names as in a checkpoint.  `config` is the design's config.json as a dict.
"""
import math

import torch


def rms(x, eps):
    """x over its root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rotate_half(x, rot):
    """x [tokens, ..., width] from position 0: dimension i turns together with i + dims / 2."""
    y, half = x.clone(), rot["dims"] // 2
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(half):
        a = (pos * float(rot["base"]) ** (-2.0 * i / rot["dims"])).reshape(-1, *[1] * (x.dim() - 2))
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return y


def visible(n, mask):
    """[query, key]: not in the future, and near enough or among the first ones."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    if not mask:
        return j <= i
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def keys_and_values(h, w, m):
    """k [tokens, groups, 2, dim] (rotated), v [tokens, groups, vdim]"""
    n, g = h.shape[0], m["kv_heads"]
    k = (h @ w("k").T).reshape(n, g, 2, m["dim"])
    return rotate_half(k, m["rot"]), (h @ w("v").T).reshape(n, g, m["vdim"])


def attention_maps(q, k, v, m):
    """q [tokens, heads, 2, dim], rotated: the two maps' outputs [tokens, heads, 2, vdim]."""
    n, heads = q.shape[:2]
    out = torch.zeros(n, heads, 2, v.shape[-1], dtype=q.dtype)
    seen = visible(n, m.get("mask"))
    for h in range(heads):
        g = h // (heads // k.shape[1])
        for p in range(2):
            score = (q[:, h, p] @ k[:, g, p].T * m["scale"]).masked_fill(~seen, -math.inf)
            out[:, h, p] = torch.softmax(score, -1) @ v[:, g]
    return out


def difference(a, w, m, eps):
    """a [tokens, heads, 2, vdim] -> [tokens, heads, vdim]"""
    lam = torch.exp((w("lq1") * w("lk1")).sum()) - torch.exp((w("lq2") * w("lk2")).sum()) + m["diff"]
    return rms(a[:, :, 0] - lam * a[:, :, 1], eps) * (1 - m["diff"])


def differential_attention(h, w, m, eps, kv):
    n, heads = h.shape[0], m["heads"]
    q = rotate_half((h @ w("q").T).reshape(n, heads, 2, m["dim"]), m["rot"])
    o = difference(attention_maps(q, *kv, m), w, m, eps)
    o = o * sigmoid(h @ w("g").T)[:, :, None]
    return o.reshape(n, -1) @ w("o").T


def recurrence(q, k, v, decay, state=None):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim]: outputs [tokens, heads, vdim] and the state after them."""
    s = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    d = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for t in range(q.shape[0]):
        s = d * s + k[t][:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * s).sum(1))
    return torch.stack(out), s


def retention(h, w, m, eps):
    n, heads = h.shape[0], m["heads"]
    q = rotate_half((h @ w("q").T).reshape(n, heads, m["dim"]), m["rot"])
    k = rotate_half((h @ w("k").T).reshape(n, heads, m["dim"]), m["rot"]) * m["dim"] ** -0.5
    o, _ = recurrence(q, k, (h @ w("v").T).reshape(n, heads, m["vdim"]), m["decay"])
    return (rms(o, eps).reshape(n, -1) * silu(h @ w("g").T)) @ w("o").T


def gated(h, w, act):
    return (act(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def route(z, top):
    """Router logits -> weights [tokens, experts], zero for those that were not chosen."""
    out = torch.zeros_like(z)
    for t in range(z.shape[0]):
        chosen = torch.argsort(z[t], descending=True, stable=True)[:top]
        out[t, chosen] = torch.softmax(z[t, chosen], -1)
    return out


def experts(h, w, mlp):
    p = route(h @ w("router").T, mlp["router"]["top"])
    y = sum(p[:, e:e + 1] * gated(h, lambda n: w(f"e{e}.{n}"), silu) for e in range(mlp["router"]["experts"]))
    if mlp.get("shared"):
        y = y + sigmoid(h @ w("shared.sg").T) * gated(h, lambda n: w(f"shared.{n}"), silu)
    return y


def forward(config, weights, tokens, trace=None):
    """Logits [tokens, vocab]; trace receives the residual stream after every layer."""
    t = {k: v.double() for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)]
    held = {}
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        w = lambda n: t[f"l{i}.mix.{n}"]
        h = rms(x, eps) * t[f"l{i}.norm1"]
        if layer["type"] == "retention":
            y = retention(h, w, m, eps)
        else:
            if m.get("kv_from") is None:
                held[i] = keys_and_values(h, w, m)
            y = differential_attention(h, w, m, eps, held[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + rms(y, eps) * t[f"l{i}.norm1b"] * t[f"l{i}.ls1"]
        if mlp:
            w = lambda n: t[f"l{i}.mlp.{n}"]
            h = rms(x, eps) * t[f"l{i}.norm2"]
            y = gated(h, w, gelu_tanh) if mlp["kind"] == "dense" else experts(h, w, mlp)
            x = x + rms(y, eps) * t[f"l{i}.norm2b"] * t[f"l{i}.ls2"]
        if trace is not None:
            trace.append(x)
    return (rms(x, eps) * t["final.norm"]) @ t["head"].T


def greedy(config, weights, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(forward(config, weights, out)[-1].argmax()))
    return out[len(prompt):]


# ---------------------------------------------------------------------------------------------- small models

def attention_layer(heads=6, kv_heads=2, dim=24, vdim=40, diff=0.4, window=21, keep=5, rot_dims=16, base=3000.0, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "rot": {"base": base, "dims": rot_dims},
         "scale": dim ** -0.5 if scale is None else scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def retention_layer(heads=3, dim=20, vdim=28, decay=None, rot_dims=12, base=800.0, mlp=None):
    decay = [1 - 0.5 ** (i + 2.5) for i in range(heads)] if decay is None else decay
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims}}, "mlp": mlp}


def dense_mlp(ff=72):
    return {"kind": "dense", "ff": ff}


def moe_mlp(ff=24, experts=7, top=2, shared=40):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def model(*layers, width=56, vocab=131, eps=1e-5):
    return {"architecture": "Videdra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": list(layers)}


def make_weights(config, seed=0, q_gain=1.0, router_gain=3.0):
    """Random tensors with values bf16 can hold.  q_gain scales the queries: larger makes single keys stand out in the softmax;
    router_gain the router, so that no choice of experts is close."""
    g = torch.Generator().manual_seed(seed)
    width, out = config["width"], {}

    def put(name, *shape, std, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16).float()

    def gated(p, ff):
        put(p + "gate", ff, width, std=1.5 * width ** -0.5)
        put(p + "up", ff, width, std=width ** -0.5)
        put(p + "down", width, ff, std=ff ** -0.5)

    put("embed", config["vocab"], width, std=1.0)
    put("head", config["vocab"], width, std=width ** -0.5)
    put("final.norm", width, std=0.2, mean=1.0)
    for i, l in enumerate(config["layers"]):
        m, mlp, p = l["mixer"], l["mlp"], f"l{i}."
        for n in ("norm1", "norm1b", "ls1") + (("norm2", "norm2b", "ls2") if mlp else ()):
            put(p + n, width, std=0.2, mean=0.7 if n.startswith("ls") else 1.0)
        if l["type"] == "attention":
            put(p + "mix.q", m["heads"] * 2 * m["dim"], width, std=q_gain * width ** -0.5)
            if m.get("kv_from") is None:
                put(p + "mix.k", m["kv_heads"] * 2 * m["dim"], width, std=width ** -0.5)
                put(p + "mix.v", m["kv_heads"] * m["vdim"], width, std=width ** -0.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + "mix." + n, m["dim"], std=0.3)
            put(p + "mix.g", m["heads"], width, std=width ** -0.5)
        else:
            for n, d in (("q", "dim"), ("k", "dim"), ("v", "vdim"), ("g", "vdim")):
                put(p + "mix." + n, m["heads"] * m[d], width, std=width ** -0.5)
        put(p + "mix.o", width, m["heads"] * m["vdim"], std=(m["heads"] * m["vdim"]) ** -0.5)
        if mlp and mlp["kind"] == "dense":
            gated(p + "mlp.", mlp["ff"])
        elif mlp:
            put(p + "mlp.router", mlp["router"]["experts"], width, std=router_gain * width ** -0.5)
            for e in range(mlp["router"]["experts"]):
                gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                gated(p + "mlp.shared.", mlp["shared"]["ff"])
                put(p + "mlp.shared.sg", 1, width, std=width ** -0.5)
    return out
