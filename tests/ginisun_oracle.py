"""Plain evaluation of the Ginisun design in f64, one function per mechanism, for the tests. Nothing here is shared with the package: every
function works on one sequence, recomputes everything from the first token and is written for reading, not for speed.

Notation: ``x`` is ``[tokens, width]``; ``streams`` is ``[count, tokens, width]``; a weight ``w`` is ``[out, in]``.
"""
import math

import numpy as np


def dynamic_tanh(x, alpha, w, b):
    return np.tanh(float(alpha) * x) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def rotate_pairs(x, positions, base):
    """Rotates the pairs (0, 1), (2, 3), ... of the last dimension; pair i turns by ``position * base ** (-2 i / dims)``."""
    dims = x.shape[-1]
    out = np.empty_like(x)
    for i in range(dims // 2):
        a = np.asarray(positions, dtype=np.float64) * base ** (-2.0 * i / dims)
        a = a.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def softmax(s):
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def latent_attention(h, W, m, eps):
    """``W``: q, dkv, dkv.norm, uk, uv, o; ``m``: the mixer's sizes and constants."""
    T, H, dn, dr, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (h @ W["q"].T).reshape(T, H, dn + dr)
    q_plain, q_rot = q[..., :dn], rotate_pairs(q[..., dn:], pos, m["rot"]["base"])
    down = h @ W["dkv"].T
    c = rms_norm(down[:, :rank], W["dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, rank:], pos, m["rot"]["base"])
    k = (c @ W["uk"].T).reshape(T, H, dn)
    v = (c @ W["uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for n in range(H):
        s = (q_plain[:, n] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]
        s[np.triu(np.ones((T, T), bool), 1)] = -np.inf
        out[:, n] = softmax(s) @ v[:, n]
    return out.reshape(T, H * dv) @ W["o"].T


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)) @ down.T


def route(h, router, top):
    """Chosen experts ``[tokens, top]`` and their sigmoid scores."""
    s = 1.0 / (1.0 + np.exp(-(h @ router.T)))
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, -1)


def mixture(h, W, m):
    """Sum over the chosen experts of ``expert(score * token)``, plus the shared expert if there is one."""
    chosen, score = route(h, W["router"], m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], score[t]):
            out[t] += clamped_expert(s * h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"], m["expert"]["limit"])
    if m.get("shared"):
        out = out + clamped_expert(h, W["shared.gate"], W["shared.up"], W["shared.down"], m["shared"]["limit"])
    return out


def connect_in(streams, weights):
    return sum(float(weights[s]) * streams[s] for s in range(streams.shape[0]))


def connect_out(streams, y, mix, out):
    n = streams.shape[0]
    return np.stack([sum(float(mix[s, t]) * streams[s] for s in range(n)) + float(out[t]) * y for t in range(n)])


def _sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[tokens, vocab]`` of one sequence; ``trace`` collects the sum of the streams after every layer."""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}

    def norm(x, name):
        return dynamic_tanh(x, W[name + ".alpha"], W[name], W[name + ".b"])
    eps = cfg["norm"]["eps"]
    x0 = norm(W["embed"][np.asarray(tokens)], "embed.norm")
    streams = np.stack([x0] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = latent_attention(norm(connect_in(streams, W[p + "hc1.in"]), p + "norm1"), _sub(W, p + "mix."), layer["mixer"], eps)
        streams = connect_out(streams, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if layer.get("mlp"):
            y = mixture(norm(connect_in(streams, W[p + "hc2.in"]), p + "norm2"), _sub(W, p + "mlp."), layer["mlp"])
            streams = connect_out(streams, y, W[p + "hc2.mix"], W[p + "hc2.out"])
        if trace is not None:
            trace.append(streams.sum(0))
    return norm(streams.sum(0), "final.norm") @ W["head"].T


def greedy(cfg, weights, prompt, new):
    """Greedy continuation by running the whole sequence again for every token."""
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(np.argmax(forward(cfg, weights, seq)[-1])))
    return seq[len(prompt):]


def random_model(seed, vocab=96, width=64, heads=(3, 2), dim=16, rot_dim=8, vdim=16, kv_rank=32, experts=5, top=2, ff=24, shared_ff=40, limit=1.25,
                 shared_limit=0.75, streams=3, base=10000.0, scale=None, mlp=True, eps=1e-5, overrides=None):
    """A configuration of ``len(heads)`` layers and random weights rounded to bf16 (returned as f32 torch-free arrays). ``overrides[i]`` replaces
    keyword values for layer i; ``mlp=False`` (there or here) leaves the feed-forward out."""
    rng = np.random.default_rng(seed)

    def bf16(a):
        u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
        return (((u.astype(np.uint64) + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).reshape(np.shape(a))

    def mat(o, i, s=1.0):
        return bf16(rng.standard_normal((o, i)) * s / math.sqrt(i))
    W, layers = {}, []

    def norm(name):
        W[name] = bf16(1.0 + 0.2 * rng.standard_normal(width))
        W[name + ".b"] = bf16(0.1 * rng.standard_normal(width))
        W[name + ".alpha"] = bf16(np.float32(0.6 + 0.3 * rng.random()))
    W["embed"] = bf16(rng.standard_normal((vocab, width)))
    norm("embed.norm")
    for i, H in enumerate(heads):
        o = dict(dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, experts=experts, top=top, ff=ff, shared_ff=shared_ff, limit=limit,
                 shared_limit=shared_limit, base=base, scale=scale, mlp=mlp)
        o.update((overrides or {}).get(i, {}))
        p = f"l{i}."
        dn, dr, dv, r = o["dim"], o["rot_dim"], o["vdim"], o["kv_rank"]
        mixer = dict(heads=H, dim=dn, rot_dim=dr, vdim=dv, kv_rank=r, rot=dict(base=o["base"], dims=dr),
                     scale=o["scale"] if o["scale"] is not None else (dn + dr) ** -0.5)
        norm(p + "norm1")
        W[p + "mix.q"] = mat(H * (dn + dr), width, 1.6)
        W[p + "mix.dkv"] = mat(r + dr, width, 1.3)
        W[p + "mix.dkv.norm"] = bf16(1.0 + 0.2 * rng.standard_normal(r))
        W[p + "mix.uk"] = mat(H * dn, r, 1.5)
        W[p + "mix.uv"] = mat(H * dv, r)
        W[p + "mix.o"] = mat(width, H * dv)
        n = 1
        ff_cfg = None
        if o["mlp"]:
            n = 2
            norm(p + "norm2")
            ff_cfg = dict(kind="moe", router=dict(experts=o["experts"], top=o["top"]), expert=dict(ff=o["ff"], limit=o["limit"]))
            W[p + "mlp.router"] = mat(o["experts"], width, 2.0)
            names = [(f"e{e}", o["ff"]) for e in range(o["experts"])]
            if o["shared_ff"]:
                ff_cfg["shared"] = dict(ff=o["shared_ff"], limit=o["shared_limit"])
                names.append(("shared", o["shared_ff"]))
            for nm, f in names:
                W[f"{p}mlp.{nm}.gate"], W[f"{p}mlp.{nm}.up"] = mat(f, width, 1.5), mat(f, width, 1.5)
                W[f"{p}mlp.{nm}.down"] = mat(width, f)
        for q in range(1, n + 1):
            W[f"{p}hc{q}.in"] = bf16(1.0 / streams + 0.3 * rng.standard_normal(streams))
            W[f"{p}hc{q}.out"] = bf16(1.0 + 0.3 * rng.standard_normal(streams))
            W[f"{p}hc{q}.mix"] = bf16(np.eye(streams) + 0.2 * rng.standard_normal((streams, streams)))
        layers.append(dict(type="latent_attention", mixer=mixer, mlp=ff_cfg))
    norm("final.norm")
    W["head"] = mat(vocab, width, 2.0)
    return dict(architecture="Ginisun", vocab=vocab, width=width, streams=streams, norm=dict(eps=eps), layers=layers), W
