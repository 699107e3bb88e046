"""Plain float64 restatement of the Povilorn design, one function per mechanism, token loops instead of batched
kernels.  Shares no code with the package: the tests compare the CUDA path with this.

A model is ``(config, tensors)``: ``config`` is the dict form of ``config.json`` (keys ``width``, ``vocab``,
``norm.eps``, ``embedding.scale``, ``loop``, ``layers``), ``tensors`` maps checkpoint names to arrays.
"""

from __future__ import annotations

import math

import numpy as np


def f64(t) -> np.ndarray:
    if hasattr(t, "detach"):
        t = t.detach().cpu().double().numpy()
    return np.asarray(t, dtype=np.float64)


# ------------------------------------------------------------------------------------------------- small pieces #
def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / math.sqrt(float(np.mean(x * x)) + eps)


def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


def squash(x: np.ndarray, alpha: float, w: np.ndarray, b: np.ndarray) -> np.ndarray:
    """The element-wise norm: no statistic, a scaled ``tanh`` with a weight and a shift per channel."""
    return np.tanh(alpha * x) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotation_plan(dims: int, base: float, scaling: dict | None):
    """(angle per position of every pair, factor on cos and sin).  With ``scaling`` the pairs that turn slowly over the
    original length are slowed further, the fast ones are left, and a ramp joins them."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0
    F, L = scaling["factor"], scaling["original"]

    def at(turns):
        return dims * math.log(L / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / F * r + f * (1.0 - r))
    return out, 0.1 * math.log(F) + 1.0


def rotate(x: np.ndarray, p: int, dims: int, base: float, scaling: dict | None) -> np.ndarray:
    """The first ``dims`` entries turned by position ``p``; entries ``2i`` and ``2i + 1`` are a pair."""
    freq, mag = rotation_plan(dims, base, scaling)
    y = x.copy()
    for i, f in enumerate(freq):
        c, s = mag * math.cos(p * f), mag * math.sin(p * f)
        u, v = x[2 * i], x[2 * i + 1]
        y[2 * i], y[2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def query_gain(p: int, q_temp: dict | None) -> float:
    if not q_temp or not q_temp.get("every"):
        return 1.0
    return 1.0 + q_temp["coef"] * math.log(math.floor((p + 1) / q_temp["every"]) + 1)


# ------------------------------------------------------------------------------------------------- mixers #
def softmax_sum(scores: np.ndarray, values: np.ndarray) -> np.ndarray:
    e = np.exp(scores - scores.max())
    return e @ values / e.sum()


def attention(h: np.ndarray, m: dict, w: dict, eps: float) -> np.ndarray:
    """Position-free attention whose values are the projected keys as they are before the key norm; one norm statistic
    per token over all query (key) heads; an element-wise logistic gate before the output projection."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w["q"].T + w["q.b"], h @ w["k"].T + w["k.b"]
    values = k.reshape(T, G, D)
    keys = np.stack([unit_rms(r, eps) * w["k.norm"] for r in k]).reshape(T, G, D)
    out = np.zeros((T, H, D))
    for t in range(T):
        qt = (unit_rms(q[t], eps) * w["q.norm"] * query_gain(t, m.get("q_temp"))).reshape(H, D)
        for a in range(H):
            g = a // (H // G)
            out[t, a] = softmax_sum(keys[:t + 1, g] @ qt[a] * m["scale"], values[:t + 1, g])
    return (out.reshape(T, H * D) * logistic(h @ w["g"].T)) @ w["o"].T


def latent_attention(h: np.ndarray, m: dict, w: dict, eps: float) -> np.ndarray:
    """Keys and values expanded per head from a normed latent, plus one rotated key part that all heads share."""
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = (m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (h @ w["q"].T).reshape(T, H, D + R)
    d = h @ w["dkv"].T
    c = np.stack([unit_rms(r, eps) for r in d[:, :K]]) * w["dkv.norm"]
    kr = np.stack([rotate(d[t, K:], t, *rot) for t in range(T)])
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, V)
    out = np.zeros((T, H, V))
    for t in range(T):
        for a in range(H):
            qr = rotate(q[t, a, D:], t, *rot)
            out[t, a] = softmax_sum((k[:t + 1, a] @ q[t, a, :D] + kr[:t + 1] @ qr) * m["scale"], v[:t + 1, a])
    return out.reshape(T, H * V) @ w["o"].T


# ------------------------------------------------------------------------------------------------- feed-forward #
def dense_ff(h: np.ndarray, w: dict) -> np.ndarray:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_unit(x: np.ndarray, w: dict, prefix: str, limit: float) -> np.ndarray:
    g = np.minimum(w[prefix + "gate"] @ x, limit)
    u = np.clip(w[prefix + "up"] @ x, -limit, limit)
    return w[prefix + "down"] @ (g * logistic(1.702 * g) * (u + 1.0))


def choose(x: np.ndarray, r: dict, w: dict):
    """(chosen ids, their weights): softmax scores, a correction that counts for the choice alone, only the best groups
    of neighbours (by their largest choice score) eligible."""
    z = w["router"] @ x
    e = np.exp(z - z.max())
    s = e / e.sum()
    c = s + w["correction"] if "correction" in w else s.copy()
    groups = r.get("groups") or {"count": 1, "keep": 1}
    per = len(s) // groups["count"]
    best = [c[g * per:(g + 1) * per].max() for g in range(groups["count"])]
    kept = np.argsort(-np.array(best), kind="stable")[:groups["keep"]]
    c = np.array([c[j] if j // per in kept else -np.inf for j in range(len(s))])
    pick = np.argsort(-c, kind="stable")[:r["top"]]
    return pick, s[pick] / (s[pick].sum() + 1e-20)


def routed_ff(h: np.ndarray, m: dict, w: dict) -> np.ndarray:
    """The chosen experts' weighted outputs; ids from ``experts`` on hand the input through; a shared expert times one
    logistic number per token joins."""
    out = np.zeros_like(h)
    for t, x in enumerate(h):
        for j, weight in zip(*choose(x, m["router"], w)):
            y = x if j >= m["router"]["experts"] else clamped_unit(x, w, f"e{j}.", m["expert"]["limit"])
            out[t] += weight * y
        if m.get("shared"):
            out[t] += clamped_unit(x, w, "shared.", m["shared"]["limit"]) * logistic(float((w["shared.sg"] @ x).reshape(())))
    return out


# ------------------------------------------------------------------------------------------------- whole model #
def layer_tensors(tensors: dict, i: int, part: str) -> dict:
    p = f"l{i}.{part}."
    return {k[len(p):]: f64(v) for k, v in tensors.items() if k.startswith(p)}


def named_squash(x: np.ndarray, tensors: dict, name: str) -> np.ndarray:
    return squash(x, float(f64(tensors[name + ".alpha"]).reshape(())), f64(tensors[name]), f64(tensors[name + ".b"]))


def run_order(config: dict) -> list[tuple[int, int | None]]:
    """(layer, pass number if it is the first layer of a pass, else None) in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(config: dict, tensors: dict, tokens, return_layers: bool = False):
    """``tokens`` of ONE sequence -> logits ``[T, vocab]`` (``return_layers``: also the residual after every layer run)."""
    eps = float(config["norm"]["eps"])
    start = f64(tensors["embed"])[list(tokens)] * config["embedding"]["scale"]
    x, layers = start, []
    for i, t in run_order(config):
        layer = config["layers"][i]
        if t is not None:
            if t > 0:
                x = x + start
            x = x + f64(tensors["loop.step"])[t]
        mixer = {"attention": attention, "latent_attention": latent_attention}[layer["type"]]
        x = x + mixer(named_squash(x, tensors, f"l{i}.norm1"), layer["mixer"], layer_tensors(tensors, i, "mix"), eps)
        if layer.get("mlp") is not None:
            h, w = named_squash(x, tensors, f"l{i}.norm2"), layer_tensors(tensors, i, "mlp")
            x = x + (dense_ff(h, w) if layer["mlp"]["kind"] == "dense" else routed_ff(h, layer["mlp"], w))
        layers.append(x)
    z = named_squash(x, tensors, "final.norm") @ f64(tensors["head"]).T
    return (z, layers) if return_layers else z


# ------------------------------------------------------------------------------------------- test model builders #
def dense_mlp(ff=9) -> dict:
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts=5, identity=3, top=3, ff=6, limit=0.9, groups=2, keep=1, shared_ff=7, shared_limit=0.6) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
           "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def attention_layer(heads=6, kv_heads=2, dim=5, coef=0.4, every=7, scale=0.5, mlp="moe") -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if every:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m, "mlp": moe_mlp() if mlp == "moe" else mlp}


def latent_layer(heads=3, dim=5, rot_dim=4, vdim=3, kv_rank=6, base=500.0, scaling=True, scale=0.5, mlp="dense") -> dict:
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = {"factor": 4.0, "original": 100, "fast": 9.0, "slow": 0.5} if scaling is True else scaling
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": rot},
            "mlp": dense_mlp() if mlp == "dense" else mlp}


def make_config(layers, width=24, vocab=50, eps=1e-5, embed_scale=3.0, loop=(0, 0, 0)) -> dict:
    start, stop, times = loop
    out = {"architecture": "Povilorn", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "embedding": {"scale": embed_scale}, "layers": list(layers)}
    if times:
        out["loop"] = {"start": start, "stop": stop, "times": times}
    return out


def norm_shapes(name: str, w: int) -> dict:
    return {name: (w,), name + ".b": (w,), name + ".alpha": ()}


def tensor_shapes(config: dict) -> dict:
    w = config["width"]
    out = {"embed": (config["vocab"], w), "head": (config["vocab"], w), **norm_shapes("final.norm", w)}
    if config.get("loop"):
        out["loop.step"] = (config["loop"]["times"], w)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        out.update(norm_shapes(f"l{i}.norm1", w))
        if layer["type"] == "attention":
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            out.update({p + "q": (nq, w), p + "q.b": (nq,), p + "k": (nk, w), p + "k.b": (nk,), p + "q.norm": (nq,),
                        p + "k.norm": (nk,), p + "g": (nq, w), p + "o": (w, nq)})
        else:
            H, D, R, V, K = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            out.update({p + "q": (H * (D + R), w), p + "dkv": (K + R, w), p + "dkv.norm": (K,), p + "uk": (H * D, K),
                        p + "uv": (H * V, K), p + "o": (w, H * V)})
        mlp, q = layer.get("mlp"), f"l{i}.mlp."
        if mlp is None:
            continue
        out.update(norm_shapes(f"l{i}.norm2", w))
        if mlp["kind"] == "dense":
            out.update({q + "gate": (mlp["ff"], w), q + "up": (mlp["ff"], w), q + "down": (w, mlp["ff"])})
            continue
        for name in [f"e{e}" for e in range(mlp["router"]["experts"])] + (["shared"] if mlp.get("shared") else []):
            f = mlp["shared"]["ff"] if name == "shared" else mlp["expert"]["ff"]
            out.update({f"{q}{name}.gate": (f, w), f"{q}{name}.up": (f, w), f"{q}{name}.down": (w, f)})
        ids = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
        out.update({q + "router": (ids, w), q + "correction": (ids,)})
        if mlp.get("shared"):
            out[q + "shared.sg"] = (1, w)
    return out


def random_model(config: dict, seed: int = 0, spread: float = 1.0) -> dict:
    """Random tensors (torch, fp32 holding bf16-exact values) with checkpoint names; ``spread`` widens the head so
    that greedy choices are decided by more than rounding."""
    import torch

    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        if name == "head":
            t = spread * torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf == "alpha":
            t = 0.3 + 0.3 * torch.rand(shape, generator=g)
        elif leaf == "router":
            t = 3.0 * torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf in ("gate", "up") and ".e" in name or name.endswith(("shared.gate", "shared.up")):
            t = 1.5 * torch.randn(shape, generator=g) / shape[1] ** 0.5       # some units reach their bound
        elif name == "embed":
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "loop.step":
            t = 0.5 * torch.randn(shape, generator=g)
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf == "correction":                           # some choice scores below zero
            t = 0.3 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        else:                                                # norm weights
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        out[name] = t.to(torch.bfloat16).float()
    return out
