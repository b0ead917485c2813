"""Plain evaluation of the Pufevik design in f64, one function per mechanism, for the tests. Nothing here is shared with the package: every function
works on one sequence, recomputes everything from the first token and is written for reading, not for speed.

Notation: ``x`` and ``h`` are ``[tokens, width]``; a weight ``w`` is ``[out, in]``.
"""
import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_first_pairs(x, positions, dims, base):
    """``x`` ``[tokens, heads, size]``: pairs (0, 1), (2, 3), ... below ``dims`` turn by ``position * base ** (-2 i / dims)``, the rest stays."""
    out = x.copy()
    for i in range(dims // 2):
        a = (np.asarray(positions, dtype=np.float64) * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(tokens, window=None):
    """``[queries, keys]``: a query sees itself and what came before, with a window only the last ``window`` of those."""
    back = np.arange(tokens)[:, None] - np.arange(tokens)[None, :]
    return (back >= 0) & (back < (window or tokens))


def attend(q, k, v, scale, window=None, sink=None):
    """Grouped-query softmax attention; ``q`` ``[tokens, heads, dim]``, ``k`` / ``v`` ``[tokens, groups, .]``. ``sink[h]`` enters head h's denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    see = visible(T, window)
    out = np.zeros((T, H, v.shape[2]))
    for n in range(H):
        g = n // (H // G)
        s = np.where(see, (q[:, n] @ k[:, g].T) * scale, -np.inf)
        top = s.max(-1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[n])
        e = np.exp(s - top)
        den = e.sum(-1, keepdims=True)
        if sink is not None:
            den = den + np.exp(sink[n] - top)
        out[:, n] = (e / den) @ v[:, g]
    return out


def attention_full(h, W, m, eps, first=None):
    """Mixer 'attention'. ``first`` is a list that carries the values of the first value-mixing layer from layer to layer."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(T), m["rot"]
    q = rms_norm((h @ W["q"].T).reshape(T, H, d), W["q.norm"], eps)
    k = rms_norm((h @ W["k"].T).reshape(T, G, d), W["k.norm"], eps)
    v = (h @ W["v"].T).reshape(T, G, dv)
    q, k = (rotate_first_pairs(t, pos, rot["dims"], rot["base"]) for t in (q, k))
    if m.get("v_mix"):
        if first:
            lam = float(W["vmix"])
            v = (1.0 - lam) * v + lam * first[0]
        else:
            first.append(v)
    o = attend(q, k, v, m["scale"]).reshape(T, H * dv)
    return (o * sigmoid(h @ W["g"].T)) @ W["o"].T


def attention_window(h, W, m, eps):
    """Left half of mixer 'parallel'."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(T), m["rot"]
    q = rms_norm(h @ W["q"].T, W["q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ W["k"].T, W["k.norm"], eps).reshape(T, G, d)
    v = (h @ W["v"].T).reshape(T, G, dv)
    q, k = (rotate_first_pairs(t, pos, rot["dims"], rot["base"]) for t in (q, k))
    o = attend(q, k, v, m["scale"], window=m["mask"]["size"], sink=W["sink"])
    return (o * sigmoid(h @ W["g"].T)[:, :, None]).reshape(T, H * dv) @ W["o"].T


def matrix_memory(q, k, v, i, f):
    """The recurrence of one head: ``q`` (scaled), ``k`` ``[tokens, dim]``, ``v`` ``[tokens, vdim]``, log gates ``i``, ``f``. Returns outputs and the last
    state ``(S, n, m)``."""
    S, n, m = np.zeros((q.shape[1], v.shape[1])), np.zeros(q.shape[1]), 0.0
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        m_new = max(f[t] + m, i[t])
        keep, add = math.exp(f[t] + m - m_new), math.exp(i[t] - m_new)
        S = keep * S + add * np.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = m_new
        out[t] = (q[t] @ S) / (max(abs(n @ q[t]), math.exp(-m)) + 1e-6)
    return out, (S, n, m)


def memory_gates(h, W, cap):
    """Log input and log forget gates ``[tokens, heads]``."""
    def soft(z):
        return cap * np.tanh(z / cap)
    i = soft(h @ W["i"].T + W["i.b"])
    f = -np.logaddexp(0.0, -soft(h @ W["f"].T + W["f.b"]))
    return i, f


def memory_mixer(h, W, m, eps):
    """Right half of mixer 'parallel'."""
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ W["k"].T).reshape(T, H, d)
    v = (h @ W["v"].T).reshape(T, H, dv)
    i, f = memory_gates(h, W, m["gate_cap"])
    o = np.zeros((T, H, dv))
    for n in range(H):
        o[:, n] = rms_norm(matrix_memory(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n])[0], 1.0, eps)
    return (o.reshape(T, H * dv) * W["norm"] * sigmoid(h @ W["g"].T)) @ W["o"].T


def feed_forward(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``trace`` collects the residual after every layer."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    first = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            y = attention_full(x, _sub(W, p + "mix."), m, eps, first)
        else:
            y = (m["left_scale"] * attention_window(x, _sub(W, p + "mix.left."), m["left"], eps)
                 + m["right_scale"] * memory_mixer(x, _sub(W, p + "mix.right."), m["right"], eps))
        x = x + rms_norm(y, W[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(feed_forward(x, _sub(W, p + "mlp.")), W[p + "norm2"], eps)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


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


def random_model(seed, kinds="pa", vocab=90, width=56, ff=72, heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=10000.0, scale=None, v_mix=True, window=20, mem_heads=3,
                 mem_dim=16, mem_vdim=16, cap=6.0, left_scale=0.7, right_scale=0.6, sink=1.5, emb_scale=3.0, eps=1e-5, overrides=None):
    """A configuration with one layer per letter of ``kinds`` (``p``: two mixers side by side, ``a``: full attention) and random weights rounded to bf16.
    ``overrides[i]`` replaces keyword values for layer i; ``ff=0`` leaves the feed-forward out."""
    rng = np.random.default_rng(seed)

    def mat(o, i, s=1.0):
        return bf16(rng.standard_normal((o, i)) * s / math.sqrt(i))

    def vec(n, mean=1.0, s=0.2):
        return bf16(mean + s * rng.standard_normal(n))
    W, layers = {"embed": bf16(rng.standard_normal((vocab, width)) / emb_scale)}, []
    for i, kind in enumerate(kinds):
        o = dict(ff=ff, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=rot, base=base, scale=scale, v_mix=v_mix, window=window, mem_heads=mem_heads, mem_dim=mem_dim,
                 mem_vdim=mem_vdim, cap=cap, left_scale=left_scale, right_scale=right_scale, sink=sink)
        o.update((overrides or {}).get(i, {}))
        p, H, G, d, dv = f"l{i}.", o["heads"], o["kv_heads"], o["dim"], o["vdim"]
        att = dict(heads=H, kv_heads=G, dim=d, vdim=dv, rot=dict(base=o["base"], dims=o["rot"]), scale=o["scale"] if o["scale"] is not None else d ** -0.5)

        def attention(q, whole, gate_rows):
            W.update({q + "q": mat(H * d, width), q + "k": mat(G * d, width), q + "v": mat(G * dv, width), q + "g": mat(gate_rows, width), q + "o": mat(width, H * dv),
                      q + "q.norm": vec(H * d if whole else d, 1.4), q + "k.norm": vec(G * d if whole else d, 1.4)})
        if kind == "a":
            attention(p + "mix.", False, H * dv)
            mixer = dict(att, v_mix=o["v_mix"])
            if o["v_mix"]:
                W[p + "mix.vmix"] = bf16(np.float32(0.3 + 0.4 * rng.random()))
        else:
            attention(p + "mix.left.", True, H)
            W[p + "mix.left.sink"] = bf16(o["sink"] * rng.standard_normal(H))
            mh, md, mv, q = o["mem_heads"], o["mem_dim"], o["mem_vdim"], p + "mix.right."
            W.update({q + "q": mat(mh * md, width), q + "k": mat(mh * md, width), q + "v": mat(mh * mv, width), q + "g": mat(mh * mv, width), q + "o": mat(width, mh * mv),
                      q + "norm": vec(mh * mv), q + "i": mat(mh, width, 2.0), q + "f": mat(mh, width, 2.0), q + "i.b": vec(mh, -1.0, 1.0), q + "f.b": vec(mh, 3.0, 2.0)})
            mixer = dict(left=dict(att, mask=dict(size=o["window"])), right=dict(heads=mh, dim=md, vdim=mv, gate_cap=o["cap"]), left_scale=o["left_scale"],
                         right_scale=o["right_scale"])
        W[p + "norm1"] = vec(width)
        mlp = None
        if o["ff"]:
            mlp = dict(kind="dense", ff=o["ff"])
            W.update({p + "norm2": vec(width), p + "mlp.gate": mat(o["ff"], width, 1.5), p + "mlp.up": mat(o["ff"], width), p + "mlp.down": mat(width, o["ff"])})
        layers.append(dict(type="attention" if kind == "a" else "parallel", mixer=mixer, mlp=mlp))
    W["final.norm"], W["head"] = vec(width), mat(vocab, width, 2.0)
    return dict(architecture="Pufevik", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb_scale), layers=layers), W
