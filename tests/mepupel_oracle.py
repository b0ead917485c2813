"""Plain evaluation of the Mepupel design in f64, one function per mechanism, for the tests. Nothing here is shared with the package: every function
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


def softplus(x):
    return np.logaddexp(0.0, x)


# -- attention with partial rotation, window and kept first tokens --------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """Frequency of every pair, and the factor on cos and sin."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    s, orig = scaling["factor"], scaling["original"]

    def pair_that_turns(times):
        return dims * math.log(orig / (2.0 * math.pi * times)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_that_turns(scaling["fast"])), 0), min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        f[i] = f[i] / s * ramp + f[i] * (1.0 - ramp)
    return f, 0.1 * math.log(s) + 1.0


def rotate_halves(x, positions, dims, base, scaling=None):
    """``x`` ``[tokens, heads, size]``: dimension i below ``dims / 2`` turns with dimension i + dims / 2, the rest stays."""
    out, half = x.copy(), dims // 2
    if not dims:
        return out
    f, k = frequencies(dims, base, scaling)
    for i in range(half):
        a = (np.asarray(positions, dtype=np.float64) * f[i])[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = k * (u * np.cos(a) - v * np.sin(a))
        out[..., i + half] = k * (v * np.cos(a) + u * np.sin(a))
    return out


def visible(tokens, window=None, keep_first=0):
    """``[queries, keys]``: a query sees what came before, itself included; with a window the last ``window`` of those and the first ``keep_first`` tokens."""
    i, j = np.arange(tokens)[:, None], np.arange(tokens)[None, :]
    near = i - j < window if window else np.ones((tokens, tokens), dtype=bool)
    return (j <= i) & (near | (j < keep_first))


def attend(q, k, v, scale, see):
    """Grouped-query softmax attention; ``q`` ``[tokens, heads, dim]``, ``k`` / ``v`` ``[tokens, groups, .]``, ``see`` as :func:`visible` makes it."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for n in range(H):
        g = n // (H // G)
        s = np.where(see, (q[:, n] @ k[:, g].T) * scale, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, n] = (e / e.sum(-1, keepdims=True)) @ v[:, g]
    return out


def attention_mixer(h, W, m):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, mask = m.get("rot") or dict(dims=0, base=1.0), m.get("mask") or {}
    q, k, v = ((h @ W[n].T).reshape(T, heads, size) for n, heads, size in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = (rotate_halves(t, np.arange(T), rot["dims"], rot["base"], rot.get("scaling")) for t in (q, k))
    o = attend(q, k, v, m["scale"], visible(T, mask.get("size"), mask.get("keep_first", 0)))
    return o.reshape(T, H * dv) @ W["o"].T


# -- latent attention -----------------------------------------------------------------------------------------------------------------------
def latent_of(h, W, eps):
    return rms(h @ W["dkv"].T, eps) * W["dkv.norm"]


def latent_mixer(h, W, m, eps, c):
    """``c`` ``[tokens, kv_rank]``: this layer's latent or an earlier layer's."""
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ W["dq"].T, eps) * W["dq.norm"]
    q, k, v = (cq @ W["uq"].T).reshape(T, H, d), (c @ W["uk"].T).reshape(T, H, d), (c @ W["uv"].T).reshape(T, H, dv)
    return attend(q, k, v, m["scale"], visible(T)).reshape(T, H * dv) @ W["o"].T


# -- state-space mixer ----------------------------------------------------------------------------------------------------------------------
def causal_convolution(u, w, b):
    """``u`` ``[tokens, channels]``, ``w`` ``[channels, taps]`` with the current token's weight last; zeros ahead of the first token."""
    T, taps = u.shape[0], w.shape[1]
    out = np.tile(np.asarray(b, dtype=np.float64), (T, 1))
    for t in range(T):
        for k in range(taps):
            s = t - (taps - 1 - k)
            if s >= 0:
                out[t] += w[:, k] * u[s]
    return out


def state_space(x, B, C, dt, A_log, D):
    """``x`` ``[tokens, heads, vdim]``, ``B`` / ``C`` ``[tokens, groups, state]``, ``dt`` ``[tokens, heads]`` (positive): outputs and the last states
    ``[heads, state, vdim]``."""
    T, H, dv = x.shape
    per = H // B.shape[1]
    S, out = np.zeros((H, B.shape[2], dv)), np.zeros(x.shape)
    for t in range(T):
        b, c = np.repeat(B[t], per, 0), np.repeat(C[t], per, 0)
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        out[t] = (S * c[:, :, None]).sum(1) + D[:, None] * x[t]
    return out, S


def gated_group_norm(y, z, w, groups, eps):
    """``y silu(z)`` normed in ``groups`` equal parts of the columns."""
    g = y * silu(z)
    return rms(g.reshape(g.shape[0], groups, -1), eps).reshape(g.shape) * w


def mamba2_mixer(h, W, m, eps):
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = np.split(h @ W["in"].T, [inner, 2 * inner + 2 * G * N], 1)
    x, B, C = np.split(silu(causal_convolution(xbc, W["conv"], W["conv.b"])), [inner, inner + G * N], 1)
    y, _ = state_space(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W["dt_bias"]), W["A_log"], W["D"])
    return gated_group_norm(y.reshape(T, inner), z, W["norm"], m["norm_groups"], eps) @ W["o"].T


# -- feed-forward ---------------------------------------------------------------------------------------------------------------------------
def dense(h, W):
    return (silu(h @ W["gate"].T + W["gate.b"]) * (h @ W["up"].T + W["up.b"])) @ W["down"].T + W["down.b"]


def expert(h, W, name):
    return (silu(h @ W[name + ".gate"].T) * (h @ W[name + ".up"].T)) @ W[name + ".down"].T


def route(z, correction, r):
    """Chosen experts of one token and their weights from router logits ``z``."""
    s = sigmoid(z)
    choice = s + correction
    if r.get("groups"):
        n = r["groups"]["count"]
        size = len(z) // n
        best = [np.sort(choice[g * size: (g + 1) * size])[::-1][:2].sum() for g in range(n)]
        kept = sorted(range(n), key=lambda g: -best[g])[: r["groups"]["keep"]]
        choice = np.array([c if e // size in kept else -np.inf for e, c in enumerate(choice)])
    chosen = sorted(range(len(z)), key=lambda e: -choice[e])[: r["top"]]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * r["scale"]


def mixture(h, W, mlp):
    out = expert(h, W, "shared") if mlp.get("shared") else np.zeros(h.shape)
    for t, z in enumerate(h @ W["router"].T):
        for e, w in zip(*route(z, W["correction"], mlp["router"])):
            out[t] += w * expert(h[t], W, f"e{e}")
    return out


# -- the model ------------------------------------------------------------------------------------------------------------------------------
def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``trace`` collects the residual after every layer."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x, latents = W["embed"][np.asarray(tokens)], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h, M = rms(x, eps) * W[p + "norm1"], _sub(W, p + "mix.")
        if layer["type"] == "attention":
            y = attention_mixer(h, M, m)
        elif layer["type"] == "latent_attention":
            if m.get("kv_from") is None:
                latents[i] = latent_of(h, M, eps)
            y = latent_mixer(h, M, m, eps, latents[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = mamba2_mixer(h, M, m, eps)
        mlp = layer.get("mlp")
        if mlp:
            h2, F = rms(x, eps) * W[p + "norm2"], _sub(W, p + "mlp.")
            y = y + (dense(h2, F) if mlp["kind"] == "dense" else mixture(h2, F, mlp))
        x = x + cfg["residual_mult"] * y
        if trace is not None:
            trace.append(x)
    return rms(x, eps) * W["final.norm"] @ W["head"].T


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


def random_model(seed, kinds="mal", vocab=90, width=56, residual_mult=0.4, eps=1e-5, heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=10000.0, scaling=None, scale=None, window=20,
                 keep_first=3, lat_heads=3, lat_dim=16, lat_vdim=20, q_rank=24, kv_rank=32, kv_from=None, ssm_heads=4, ssm_vdim=16, state=24, groups=2, norm_groups=2, conv=4,
                 mlp="moe", ff=40, experts=8, top=3, group_count=4, group_keep=2, router_scale=1.7, shared=24, overrides=None):
    """A configuration with one layer per letter of ``kinds`` (``m``: state space, ``a``: attention, ``l``: latent attention) and random weights rounded to bf16.
    ``overrides[i]`` replaces keyword values for layer i; ``mlp`` is ``moe``, ``dense`` or ``None``; ``shared=0``, ``group_count=0``, ``window=0`` and ``rot=0``
    leave those parts out."""
    rng = np.random.default_rng(seed)

    def mat(o, i, s=1.0):
        return bf16(rng.standard_normal((o, i)) * s / math.sqrt(i))

    def vec(n, mean=1.0, s=0.2):
        return bf16(mean + s * rng.standard_normal(n))
    W, layers = {"embed": bf16(rng.standard_normal((vocab, width)))}, []
    given = {k: v for k, v in locals().items() if k in ("heads kv_heads dim vdim rot base scaling scale window keep_first lat_heads lat_dim lat_vdim q_rank kv_rank kv_from ssm_heads "
                                                        "ssm_vdim state groups norm_groups conv mlp ff experts top group_count group_keep router_scale shared").split()}
    for i, kind in enumerate(kinds):
        o, p = dict(given, **(overrides or {}).get(i, {})), f"l{i}."
        q = p + "mix."
        W[p + "norm1"] = vec(width)
        if kind == "a":
            H, G, d, dv = o["heads"], o["kv_heads"], o["dim"], o["vdim"]
            W.update({q + "q": mat(H * d, width, 1.5), q + "k": mat(G * d, width, 1.5), q + "v": mat(G * dv, width), q + "o": mat(width, H * dv)})
            m = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=o["scale"] or d ** -0.5)
            if o["rot"]:
                m["rot"] = dict(base=o["base"], dims=o["rot"], **(dict(scaling=o["scaling"]) if o["scaling"] else {}))
            if o["window"]:
                m["mask"] = dict(size=o["window"], keep_first=o["keep_first"])
        elif kind == "l":
            H, d, dv, r, qr = o["lat_heads"], o["lat_dim"], o["lat_vdim"], o["kv_rank"], o["q_rank"]
            W.update({q + "dq": mat(qr, width), q + "dq.norm": vec(qr), q + "uq": mat(H * d, qr, 1.5), q + "uk": mat(H * d, r, 1.5), q + "uv": mat(H * dv, r), q + "o": mat(width, H * dv)})
            m = dict(heads=H, dim=d, vdim=dv, q_rank=qr, kv_rank=r, scale=o["scale"] or d ** -0.5)
            if o["kv_from"] is None:
                W.update({q + "dkv": mat(r, width), q + "dkv.norm": vec(r)})
            else:
                m["kv_from"] = o["kv_from"]
        else:
            H, dv, N, G = o["ssm_heads"], o["ssm_vdim"], o["state"], o["groups"]
            ch = H * dv + 2 * G * N
            W.update({q + "in": mat(H * dv + ch + H, width), q + "conv": mat(ch, o["conv"], 1.2), q + "conv.b": vec(ch, 0.0), q + "dt_bias": vec(H, -1.0, 1.5),
                      q + "A_log": vec(H, 0.0, 1.0), q + "D": vec(H), q + "norm": vec(H * dv), q + "o": mat(width, H * dv)})
            m = dict(heads=H, vdim=dv, state=N, groups=G, norm_groups=o["norm_groups"], conv=o["conv"])
        f, F = p + "mlp.", None
        if o["mlp"]:
            W[p + "norm2"] = vec(width)
        if o["mlp"] == "dense":
            F = dict(kind="dense", ff=o["ff"])
            W.update({f + "gate": mat(o["ff"], width, 1.5), f + "up": mat(o["ff"], width), f + "down": mat(width, o["ff"]), f + "gate.b": vec(o["ff"], 0.0, 0.5),
                      f + "up.b": vec(o["ff"], 0.0, 0.5), f + "down.b": vec(width, 0.0, 0.5)})
        elif o["mlp"] == "moe":
            F = dict(kind="moe", router=dict(experts=o["experts"], top=o["top"], scale=o["router_scale"]), expert=dict(ff=o["ff"]))
            if o["group_count"]:
                F["router"]["groups"] = dict(count=o["group_count"], keep=o["group_keep"])
            if o["shared"]:
                F["shared"] = dict(ff=o["shared"])
            W.update({f + "router": mat(o["experts"], width, 2.0), f + "correction": vec(o["experts"], -0.1, 0.4)})
            for n, size in [(f"e{e}", o["ff"]) for e in range(o["experts"])] + ([("shared", o["shared"])] if o["shared"] else []):
                W.update({f"{f}{n}.gate": mat(size, width, 1.5), f"{f}{n}.up": mat(size, width), f"{f}{n}.down": mat(width, size)})
        layers.append(dict(type=dict(m="mamba2", a="attention", l="latent_attention")[kind], mixer=m, mlp=F))
    W["final.norm"], W["head"] = vec(width), mat(vocab, width, 2.0)
    return dict(architecture="Mepupel", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=residual_mult, layers=layers), W
