"""Plain evaluation of the Vemepel design in f64, one function per mechanism, for the tests. Nothing here is shared with the package: every function
works on one sequence, recomputes everything from the first token and is written for reading, not for speed.

Notation: ``x`` and ``h`` are ``[tokens, width]``; a weight ``w`` is ``[out, in]``; ``W`` maps a mixer's or feed-forward's tensor names to weights.
"""
import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def norm_around_zero(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def token_shift(h, s):
    """Every column moves from its own value to the previous token's by the share ``s``; zeros come before the first token."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return (1.0 - s) * h + s * before


def depth_average(results, w):
    """``results``: the embedding output and every layer's result so far; one weight each."""
    return sum(c * r for c, r in zip(w, results))


# -- attention ------------------------------------------------------------------------------------------------------------------------------
def visible(tokens, chunk=None):
    """``[queries, keys]``: a query sees what came before, itself included; with chunks only what lies in its own chunk of the sequence."""
    i, j = np.arange(tokens)[:, None], np.arange(tokens)[None, :]
    return (j <= i) & ((i // chunk == j // chunk) if chunk else True)


def softmax_weights(q, k, scale, see):
    """One head: ``q`` ``[queries, dim]`` and ``k`` ``[keys, dim]``."""
    s = np.where(see, (q @ k.T) * scale, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def attend(q, k, v, scale, see):
    """Grouped-query attention; ``q`` ``[tokens, heads, dim]``, ``k`` / ``v`` ``[tokens, groups, .]``, ``see`` as :func:`visible` makes it."""
    H, G = q.shape[1], k.shape[1]
    return np.stack([softmax_weights(q[:, n], k[:, n // (H // G)], scale, see) @ v[:, n // (H // G)] for n in range(H)], 1)


def blend(lq1, lk1, lq2, lk2, diff):
    """The factor of the second map."""
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def differential(q, k, v, scale, see, factor, diff, eps):
    """``q`` ``[tokens, heads, 2, dim]``, ``k`` ``[tokens, groups, 2, dim]``: the first map's output less ``factor`` times the second's, normed per head."""
    a, b = (attend(q[:, :, m], k[:, :, m], v, scale, see) for m in range(2))
    return rms(a - factor * b, eps) * (1.0 - diff)


def keys_and_values(h, W, m):
    T, G = h.shape[0], m["kv_heads"]
    return (h @ W["k"].T).reshape(T, G, 2, m["dim"]), (h @ W["v"].T).reshape(T, G, m["vdim"])


def attention_mixer(h, W, m, eps, kv):
    """``kv``: this layer's keys and values or an earlier layer's."""
    T, H = h.shape[0], m["heads"]
    q = (h @ W["q"].T).reshape(T, H, 2, m["dim"])
    factor = blend(W["lq1"], W["lk1"], W["lq2"], W["lk2"], m["diff"])
    o = differential(q, *kv, m["scale"], visible(T, (m.get("mask") or {}).get("size")), factor, m["diff"], eps)
    return o.reshape(T, H * m["vdim"]) @ W["o"].T


# -- latent attention -----------------------------------------------------------------------------------------------------------------------
def rotate_pairs(x, positions, dims, base):
    """``x`` ``[tokens, heads, size]``: dimension 2 i below ``dims`` turns with dimension 2 i + 1, the rest stays."""
    out = x.copy()
    for i in range(dims // 2):
        a = (np.asarray(positions, dtype=np.float64) * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def latent_of(h, W, m, eps):
    """The normed latent and the rotated key part that all heads share (``[tokens, 0]`` where there is none)."""
    r, rot = m["kv_rank"], m.get("rot")
    x = h @ W["dkv"].T
    kr = x[:, None, r:]
    return rms(x[:, :r], eps) * W["dkv.norm"], (rotate_pairs(kr, np.arange(len(h)), rot["dims"], rot["base"]) if rot else kr)[:, 0]


def latent_mixer(h, W, m, eps):
    """One gate per head, or per element of the concatenated heads: as many as ``W["g"]`` has rows."""
    T, H, d, dv, rot = h.shape[0], m["heads"], m["dim"], m["vdim"], m.get("rot")
    q = (h @ W["q"].T).reshape(T, H, -1)
    if rot:
        q = np.concatenate([q[..., :d], rotate_pairs(q[..., d:], np.arange(T), rot["dims"], rot["base"])], -1)
    c, kr = latent_of(h, W, m, eps)
    k = np.concatenate([(c @ W["uk"].T).reshape(T, H, d), np.repeat(kr[:, None], H, 1)], -1)
    o = attend(q, k, (c @ W["uv"].T).reshape(T, H, dv), m["scale"], visible(T))
    g = sigmoid(h @ W["g"].T).reshape(T, H, -1)                      # one or ``vdim`` per head
    return (o * g).reshape(T, H * dv) @ W["o"].T


# -- feed-forward ---------------------------------------------------------------------------------------------------------------------------
def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, W, eps):
    return poly_norm(h @ W["up"].T, W["act"], eps) @ W["down"].T


def expert(h, W, name):
    return (silu(h @ W[name + ".gate"].T) * (h @ W[name + ".up"].T)) @ W[name + ".down"].T


def route(z, top):
    """Chosen experts of one token and their weights from router logits ``z``."""
    chosen = sorted(range(len(z)), key=lambda e: -z[e])[:top]
    w = np.exp(z[chosen] - z[chosen].max())
    return chosen, w / w.sum()


def mixture(h, W, mlp):
    out = np.zeros(h.shape)
    for t, z in enumerate(h @ W["router"].T + W["router.b"]):
        for e, w in zip(*route(z, mlp["router"]["top"])):
            out[t] += w * expert(h[t], W, f"e{e}")
    return out


# -- the model ------------------------------------------------------------------------------------------------------------------------------
def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``trace`` collects what every layer hands on."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    results, shared = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h, M = token_shift(norm_around_zero(x, W[p + "norm1"], eps), W[p + "shift"]), _sub(W, p + "mix.")
        if layer["type"] == "attention":
            if m.get("kv_from") is None:
                shared[i] = keys_and_values(h, M, m)
            y = attention_mixer(h, M, m, eps, shared[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = latent_mixer(h, M, m, eps)
        x = x + norm_around_zero(y, W[p + "norm1b"], eps)
        if mlp:
            h, F = norm_around_zero(x, W[p + "norm2"], eps), _sub(W, p + "mlp.")
            x = x + norm_around_zero(dense(h, F, eps) if mlp["kind"] == "dense" else mixture(h, F, mlp), W[p + "norm2b"], eps)
        results.append(x)
        x = depth_average(results, W[p + "dwa"])
        if trace is not None:
            trace.append(x)
    return norm_around_zero(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, new):
    """Greedy continuation by running the whole sequence again for every token."""
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(np.argmax(forward(cfg, weights, seq)[-1])))
    return seq[len(prompt):]


def bf16(a):
    """Values rounded to bf16."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return (((u.astype(np.uint64) + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).reshape(np.shape(a))


def random_model(seed, kinds="arl", vocab=90, width=56, logit_scale=0.7, eps=1e-5, heads=4, kv_heads=2, dim=12, vdim=20, scale=None, diff=0.35, chunk=24, kv_from=None, lat_heads=3,
                 lat_dim=16, lat_vdim=20, kv_rank=32, rot=8, base=10000.0, mlp="moe", ff=40, dense_ff=72, experts=8, top=3, overrides=None):
    """A configuration with one layer per letter of ``kinds`` (``a``: differential attention, ``l``: latent attention without positions, ``r``: with a rotated part) and random
    weights rounded to bf16. ``overrides[i]`` replaces keyword values for layer i; ``mlp`` is ``moe``, ``dense`` or ``None``; ``chunk=0`` leaves the chunks out."""
    rng = np.random.default_rng(seed)

    def mat(o, i, s=1.0):
        return bf16(rng.standard_normal((o, i)) * s / math.sqrt(i))

    def vec(n, mean=0.0, s=0.2):
        return bf16(mean + s * rng.standard_normal(n))
    W, layers = {"embed": bf16(rng.standard_normal((vocab, width)))}, []
    given = {k: v for k, v in locals().items() if k in ("heads kv_heads dim vdim scale diff chunk kv_from lat_heads lat_dim lat_vdim kv_rank rot base mlp ff dense_ff experts top").split()}
    for i, kind in enumerate(kinds):
        o, p = dict(given, **(overrides or {}).get(i, {})), f"l{i}."
        q = p + "mix."
        W.update({p + "norm1": vec(width), p + "norm1b": vec(width, -0.2), p + "shift": bf16(rng.uniform(0.0, 1.0, width)), p + "dwa": vec(i + 2, 0.1, 0.3)})
        W[p + "dwa"][-1] += 1.0
        W[p + "dwa"] = bf16(W[p + "dwa"])
        if kind == "a":
            H, G, d, dv = o["heads"], o["kv_heads"], o["dim"], o["vdim"]
            W.update({q + "q": mat(2 * H * d, width, 1.5), q + "o": mat(width, H * dv), **{q + n: vec(d, 0.0, 0.3) for n in ("lq1", "lk1", "lq2", "lk2")}})
            m = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=o["scale"] or d ** -0.5, diff=o["diff"])
            if o["kv_from"] is None:
                W.update({q + "k": mat(2 * G * d, width, 1.5), q + "v": mat(G * dv, width)})
            else:
                m["kv_from"] = o["kv_from"]
            if o["chunk"]:
                m["mask"] = dict(size=o["chunk"])
        else:
            H, d, dv, r, e = o["lat_heads"], o["lat_dim"], o["lat_vdim"], o["kv_rank"], o["rot"] if kind == "r" else 0
            W.update({q + "q": mat(H * (d + e), width, 1.5), q + "dkv": mat(r + e, width), q + "dkv.norm": vec(r, 1.0), q + "uk": mat(H * d, r, 1.5), q + "uv": mat(H * dv, r),
                      q + "g": mat(H * dv if e else H, width, 1.5), q + "o": mat(width, H * dv)})
            m = dict(heads=H, dim=d, vdim=dv, kv_rank=r, scale=o["scale"] or (d + e) ** -0.5)
            if e:
                m.update(rot_dim=e, rot=dict(base=o["base"], dims=e))
        f, F = p + "mlp.", None
        if o["mlp"]:
            W.update({p + "norm2": vec(width), p + "norm2b": vec(width, -0.2)})
        if o["mlp"] == "dense":
            F = dict(kind="dense", ff=o["dense_ff"])
            W.update({f + "up": mat(o["dense_ff"], width, 1.5), f + "down": mat(width, o["dense_ff"]), f + "act": vec(4, 0.3, 0.5)})
        elif o["mlp"] == "moe":
            F = dict(kind="moe", router=dict(experts=o["experts"], top=o["top"]), expert=dict(ff=o["ff"]))
            W.update({f + "router": mat(o["experts"], width, 2.0), f + "router.b": vec(o["experts"], 0.0, 0.5)})
            for n in range(o["experts"]):
                W.update({f"{f}e{n}.gate": mat(o["ff"], width, 1.5), f"{f}e{n}.up": mat(o["ff"], width), f"{f}e{n}.down": mat(width, o["ff"])})
        layers.append(dict(type=dict(a="attention", l="latent_attention", r="latent_attention_2")[kind], mixer=m, mlp=F))
    W["final.norm"], W["head"] = vec(width), mat(vocab, width, 2.0)
    return dict(architecture="Vemepel", vocab=vocab, width=width, norm=dict(eps=eps), logit_scale=logit_scale, layers=layers), W
