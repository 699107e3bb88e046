"""Plain float64 restatement of the Torutar design, one function per mechanism, token loops instead of batched
kernels.  Shares no code with the package: the tests compare the CUDA path with this.

A model is ``(config, tensors)``: ``config`` is the dict form of ``config.json`` (keys ``width``, ``vocab``,
``norm.eps``, ``streams``, ``canon.taps``, ``logit_scale``, ``layers``), ``tensors`` maps checkpoint names to arrays.

Notation: ``n(x) = x / sqrt(mean(x^2) + eps)`` is the unit-RMS form of a vector, ``s(z)`` the logistic function.
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


def log_logistic(z):
    return -(np.log1p(np.exp(-np.abs(z))) + np.maximum(-z, 0.0))


def rotate(x: np.ndarray, p: int, dims: int, base: float, layout: str) -> np.ndarray:
    """The first ``dims`` entries turned by position ``p``; pair ``i`` turns by ``p * base^(-2i/dims)``.  ``layout``
    "halves": entries ``i`` and ``i + dims/2`` are a pair; "neighbours": ``2i`` and ``2i + 1``."""
    y = x.copy()
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if layout == "halves" else (2 * i, 2 * i + 1)
        t = p * base ** (-2.0 * i / dims)
        y[a] = x[a] * math.cos(t) - x[b] * math.sin(t)
        y[b] = x[b] * math.cos(t) + x[a] * math.sin(t)
    return y


def input_conv(h: np.ndarray, taps_w: np.ndarray) -> np.ndarray:
    """``h_t + sum_j w[:, j] h_(t - taps + 1 + j)`` per channel; zeros before the first token."""
    T, taps = h.shape[0], taps_w.shape[1]
    y = h.copy()
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1 - j)
            if src >= 0:
                y[t] += taps_w[:, j] * h[src]
    return y


def sees(i: int, j: int, mask: dict | None) -> bool:
    """Causal; with a mask also: fewer than ``size`` positions back, or among the ``keep_first`` first ones."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


# ------------------------------------------------------------------------------------------------- mixers #
def attention_keys_values(h: np.ndarray, m: dict, w: dict, eps: float):
    """Keys (normed, rotated) ``[T, G, dim]`` and values (divided by their root mean square) ``[T, G, vdim]``."""
    T, G, D, V = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, D)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, V)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    kk, vv = np.zeros_like(k), np.zeros_like(v)
    for t in range(T):
        for g in range(G):
            kk[t, g] = rotate(unit_rms(k[t, g], eps) * w["k.norm"], t, rot["dims"], rot["base"], "halves")
            vv[t, g] = unit_rms(v[t, g], eps)
    return kk, vv


def attention(h: np.ndarray, m: dict, w: dict, eps: float, kv) -> np.ndarray:
    """Softmax attention with a sink per head in the denominator, a window with kept first tokens and one logistic
    gate per head; ``kv`` are this layer's keys and values, or those of the layer it borrows them from."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, D)
    keys, values = kv
    gate = logistic(h @ w["g"].T)
    out = np.zeros((T, H, V))
    for t in range(T):
        seen = [j for j in range(t + 1) if sees(t, j, m.get("mask"))]
        for a in range(H):
            g = a // (H // G)
            qa = rotate(unit_rms(q[t, a], eps) * w["q.norm"], t, rot["dims"], rot["base"], "halves")
            sc = keys[seen, g] @ qa * m["scale"]
            top = max(float(sc.max()), float(w["sink"][a]))
            e = np.exp(sc - top)
            out[t, a] = (e @ values[seen, g]) / (e.sum() + math.exp(float(w["sink"][a]) - top)) * gate[t, a]
    return out.reshape(T, H * V) @ w["o"].T + w["o.b"]


def latent_attention(h: np.ndarray, m: dict, w: dict, eps: float) -> np.ndarray:
    """Queries through a latent; keys and values expanded per head from a normed latent, plus one rotated key part that
    all heads share; every earlier token is seen; an element-wise logistic gate before the output projection."""
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    cq = np.stack([unit_rms(r, eps) for r in h @ w["dq"].T]) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(T, H, D + R)
    d = h @ w["dkv"].T
    c = np.stack([unit_rms(r, eps) for r in d[:, :K]]) * w["dkv.norm"]
    kr = np.stack([rotate(d[t, K:], t, R, base, "neighbours") for t in range(T)])
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, V)
    out = np.zeros((T, H, V))
    for t in range(T):
        for a in range(H):
            qr = rotate(q[t, a, D:], t, R, base, "neighbours")
            sc = (k[:t + 1, a] @ q[t, a, :D] + kr[:t + 1] @ qr) * m["scale"]
            e = np.exp(sc - sc.max())
            out[t, a] = e @ v[:t + 1, a] / e.sum()
    return (out.reshape(T, H * V) * logistic(h @ w["g"].T)) @ w["o"].T


def mlstm(h: np.ndarray, m: dict, w: dict, eps: float) -> np.ndarray:
    """Matrix memory with exponential gates: per head a ``dim x vdim`` memory ``S``, a normaliser ``n`` and a running
    log scale ``mx`` that starts at 0."""
    T, H, D, V, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).reshape(T, H, D)
    v = (h @ w["v"].T).reshape(T, H, V)
    gi = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    gf = log_logistic(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    S, n, mx = np.zeros((H, D, V)), np.zeros((H, D)), np.zeros(H)
    o = np.zeros((T, H, V))
    for t in range(T):
        for a in range(H):
            new = max(gf[t, a] + mx[a], gi[t, a])
            keep, write = math.exp(gf[t, a] + mx[a] - new), math.exp(gi[t, a] - new)
            S[a] = keep * S[a] + write * np.outer(k[t, a], v[t, a])
            n[a] = keep * n[a] + write * k[t, a]
            mx[a] = new
            y = S[a].T @ q[t, a] / (max(abs(float(n[a] @ q[t, a])), math.exp(-new)) + 1e-6)
            o[t, a] = unit_rms(y, eps)
    return (o.reshape(T, H * V) * w["norm"] * logistic(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------------------- feed-forward #
def clamped_unit(x: np.ndarray, w: dict, prefix: str, limit: float) -> np.ndarray:
    g = np.minimum(w[prefix + "gate"] @ x, limit)
    u = np.clip(w[prefix + "up"] @ x, -limit, limit)
    return w[prefix + "down"] @ (g * logistic(1.702 * g) * (u + 1.0))


def routed_ff(h: np.ndarray, m: dict, w: dict) -> np.ndarray:
    """Softmax scores; the choice adds a correction, the weights do not; renormalised over the chosen, times a constant;
    a shared expert (its own size and limit) joins."""
    r = m["router"]
    out = np.zeros((h.shape[0], w["e0.down"].shape[0]))
    for t, x in enumerate(h):
        z = w["router"] @ x
        e = np.exp(z - z.max())
        s = e / e.sum()
        pick = np.argsort(-(s + w["correction"] if "correction" in w else s), kind="stable")[:r["top"]]
        total = s[pick].sum() + 1e-20
        for j in pick:
            out[t] += s[j] / total * r.get("scale", 1.0) * clamped_unit(x, w, f"e{j}.", m["expert"]["limit"])
        if m.get("shared"):
            out[t] += clamped_unit(x, w, "shared.", m["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------------------- whole model #
def layer_tensors(tensors: dict, i: int, part: str) -> dict:
    p = f"l{i}.{part}."
    return {k[len(p):]: f64(v) for k, v in tensors.items() if k.startswith(p)}


def sublayer(streams: np.ndarray, i: int, q: int, tensors: dict, eps: float, inner) -> np.ndarray:
    """One sublayer of layer ``i`` (q = 1: mixer, 2: feed-forward) on ``streams [s, T, width]``: read a weighted sum,
    norm it, convolve what the sublayer reads, gate its result, write all streams at once."""
    p = f"l{i}."
    u = np.einsum("s,std->td", f64(tensors[f"{p}hc{q}.in"]), streams)
    nw = f64(tensors[f"{p}norm{q}"])
    h = np.stack([unit_rms(r, eps) * nw for r in u])
    y = inner(input_conv(h, f64(tensors[f"{p}canon{q}"])))
    y = y * logistic(h @ f64(tensors[f"{p}rg{q}"]).T + f64(tensors[f"{p}rg{q}.b"]))
    mix, out = f64(tensors[f"{p}hc{q}.mix"]), f64(tensors[f"{p}hc{q}.out"])
    new = np.zeros_like(streams)
    for t in range(streams.shape[0]):
        for s in range(streams.shape[0]):
            new[t] += mix[s, t] * streams[s]
        new[t] += out[t] * y
    return new


def forward(config: dict, tensors: dict, tokens, return_layers: bool = False):
    """``tokens`` of ONE sequence -> logits ``[T, vocab]`` (``return_layers``: also the summed streams after every
    layer)."""
    eps = float(config["norm"]["eps"])
    e = f64(tensors["embed"])[list(tokens)]
    e = np.stack([unit_rms(r, eps) for r in e]) * f64(tensors["embed.norm"])
    x = np.stack([e] * config["streams"])
    layers, shared = [], {}
    for i, layer in enumerate(config["layers"]):
        m, w = layer["mixer"], layer_tensors(tensors, i, "mix")

        def mixer(h):
            if layer["type"] == "mlstm":
                return mlstm(h, m, w, eps)
            if layer["type"] == "latent_attention":
                return latent_attention(h, m, w, eps)
            if layer["type"] != "attention":
                raise ValueError(layer["type"])
            if m.get("kv_from") is None:
                shared[i] = attention_keys_values(h, m, w, eps)
                return attention(h, m, w, eps, shared[i])
            return attention(h, m, w, eps, shared[m["kv_from"]])

        x = sublayer(x, i, 1, tensors, eps, mixer)
        if layer.get("mlp") is not None:
            fw = layer_tensors(tensors, i, "mlp")
            x = sublayer(x, i, 2, tensors, eps, lambda h: routed_ff(h, layer["mlp"], fw))
        layers.append(x.sum(0))
    fn = f64(tensors["final.norm"])
    z = np.stack([unit_rms(r, eps) for r in x.sum(0)]) * fn @ f64(tensors["head"]).T
    z = z * float(config.get("logit_scale", 1.0))
    return (z, layers) if return_layers else z


# ------------------------------------------------------------------------------------------- test model builders #
def attention_layer(heads=3, kv_heads=1, dim=6, vdim=5, size=9, keep_first=2, rot=4, base=1000.0, scale=0.4, kv_from=None,
                    mlp="moe") -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size, "keep_first": keep_first}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": moe_mlp() if mlp == "moe" else mlp}


def latent_layer(heads=2, dim=5, rot_dim=4, vdim=3, q_rank=7, kv_rank=6, base=500.0, scale=0.5, mlp="moe") -> dict:
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim,
                                                  "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"dims": rot_dim, "base": base}},
            "mlp": moe_mlp() if mlp == "moe" else mlp}


def mlstm_layer(heads=2, dim=4, vdim=6, gate_cap=6.0, mlp="moe") -> dict:
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap},
            "mlp": moe_mlp() if mlp == "moe" else mlp}


def moe_mlp(experts=5, top=2, ff=6, limit=0.9, scale=1.7, shared_ff=7, shared_limit=0.6) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def make_config(layers, width=24, vocab=50, eps=1e-5, streams=2, taps=4, logit_scale=0.7) -> dict:
    return {"architecture": "Torutar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams,
            "canon": {"taps": taps}, "logit_scale": logit_scale, "layers": list(layers)}


def tensor_shapes(config: dict) -> dict:
    w, s, taps = config["width"], config["streams"], config["canon"]["taps"]
    out = {"embed": (config["vocab"], w), "embed.norm": (w,), "final.norm": (w,), "head": (config["vocab"], w)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "attention":
            parts = {"q": m["heads"] * m["dim"]}
            if m.get("kv_from") is None:
                parts.update({"k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]})
                out[p + "k.norm"] = (m["dim"],)
            for name, rows in parts.items():
                out.update({p + name: (rows, w), f"{p}{name}.b": (rows,)})
            out.update({p + "q.norm": (m["dim"],), p + "sink": (m["heads"],), p + "g": (m["heads"], w),
                        p + "o": (w, m["heads"] * m["vdim"]), p + "o.b": (w,)})
        elif layer["type"] == "latent_attention":
            H, D, R, V, K, Q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            out.update({p + "dq": (Q, w), p + "dq.norm": (Q,), p + "uq": (H * (D + R), Q), p + "dkv": (K + R, w),
                        p + "dkv.norm": (K,), p + "uk": (H * D, K), p + "uv": (H * V, K), p + "g": (H * V, w),
                        p + "o": (w, H * V)})
        else:
            H, D, V = m["heads"], m["dim"], m["vdim"]
            out.update({p + "q": (H * D, w), p + "k": (H * D, w), p + "v": (H * V, w), p + "g": (H * V, w),
                        p + "o": (w, H * V), p + "norm": (H * V,), p + "i": (H, w), p + "i.b": (H,), p + "f": (H, w),
                        p + "f.b": (H,)})
        for q in (1,) if layer.get("mlp") is None else (1, 2):
            a = f"l{i}."
            out.update({f"{a}norm{q}": (w,), f"{a}canon{q}": (w, taps), f"{a}rg{q}": (w, w), f"{a}rg{q}.b": (w,),
                        f"{a}hc{q}.in": (s,), f"{a}hc{q}.out": (s,), f"{a}hc{q}.mix": (s, s)})
        mlp, q = layer.get("mlp"), f"l{i}.mlp."
        if mlp is None:
            continue
        names = [f"e{e}" for e in range(mlp["router"]["experts"])] + (["shared"] if mlp.get("shared") else [])
        for name in names:
            f = mlp["shared"]["ff"] if name == "shared" else mlp["expert"]["ff"]
            out.update({f"{q}{name}.gate": (f, w), f"{q}{name}.up": (f, w), f"{q}{name}.down": (w, f)})
        out.update({q + "router": (mlp["router"]["experts"], w), q + "correction": (mlp["router"]["experts"],)})
    return out


def random_model(config: dict, seed: int = 0, spread: float = 1.0) -> dict:
    """Random tensors (torch, fp32 holding bf16-exact values) with checkpoint names; ``spread`` widens the head so
    that greedy choices are decided by more than rounding."""
    import torch

    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("canon1", "canon2"):
            t = 0.4 * torch.randn(shape, generator=g)
        elif leaf == "mix":
            t = 0.3 * torch.randn(shape, generator=g) + 0.7 * torch.eye(shape[0])
        elif leaf in ("in", "out"):
            t = 0.6 + 0.5 * torch.randn(shape, generator=g)
        elif name == "head":
            t = spread * torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf == "router":
            t = 3.0 * torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf in ("gate", "up"):                         # some units reach their bound
            t = 1.5 * torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf == "correction":
            t = 0.2 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            t = 1.5 * torch.randn(shape, generator=g)
        elif name.endswith(".f.b"):
            t = 2.0 + 1.5 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.4 * torch.randn(shape, generator=g)
        else:                                                # norm weights
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        out[name] = t.to(torch.bfloat16).float()
    return out
