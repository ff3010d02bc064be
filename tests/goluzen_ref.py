"""NumPy float64 oracle of the Goluzen design: whole sequences at once, no cache, no state, one function per mechanism, no code
shared with the package.  Notation: T tokens, W width, H heads, G key/value heads, D key size, Dv value size.

    layer             x += mixer(n1(x));  x += ff(n2(x));  n(v) = v / rms(v) * (1 + w)
    attention         q, k, v with biases;  q, k rotated (element i with i + dims/2 of the first `dims`, angle
                      p * base^(-2i/dims) / factor), then divided by their root mean square per head;  s_ij = cap tanh(scale
                      q_i.k_j / cap);  i sees j <= i with i - j < window or j < keep_first;  the softmax denominator gains
                      exp(sink_h);  W_o
    latent_attention  q = W_q h per head [plain | rotated];  W_dkv h = [c', r'], c = rms(c') w, key of head h = [W_uk c | rope(r')],
                      value W_uv c;  rotation of elements 2i, 2i + 1 with stretched frequencies and a factor on cosine and
                      sine;  window;  heads * sigmoid(W_g h), W_o.  A layer may read the c and rope(r') of an earlier one.
    gla               q = W_q h D^(-1/2), k, v;  a = sigmoid(W_a2 W_a1 h + b)^(1/tau) per head and key channel;
                      S_t = diag(a_t) S_(t-1) + k_t v_t^T, o = S^T q;  W_o (rms(o) per head * w * silu(W_g h))
    dense ff          W_down gelu_tanh(W_up h)
    moe               s = sigmoid(W_r h), choice s + correction;  groups of neighbours ranked by the sum of their two largest
                      choices, the members of the best `keep` compete, the `top` largest win;  weights factor * s;  expert
                      W_down max(W_up h, 0)^2;  + sigmoid(w_sg . h) * a shared expert of the same form
    output            head . n(x),  x starts as factor * embed[token]
"""
import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def plain_frequencies(rot):
    """angle per position of every pair, linear position scaling"""
    i = np.arange(rot["dims"] // 2)
    return rot["base"] ** (-2.0 * i / rot["dims"]) / float((rot.get("scaling") or {}).get("factor", 1.0))


def stretched_frequencies(rot):
    """-> (angle per position of every pair, factor on cosine and sine): fast pairs keep their frequency, slow ones are
    divided by the factor, those in between are mixed along a ramp over the pair index"""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = base ** (-2.0 * np.arange(n // 2) / n)
    if not sc:
        return f, 1.0

    def index_of(turns):
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, freq, pairs, mult=1.0):
    """x [T, heads, n]: the first 2 len(freq) elements turn by position * freq; pairs: element 2i with 2i + 1, else i with
    i + len(freq)"""
    out = np.array(x, np.float64)
    m = len(freq)
    ang = np.asarray(positions, np.float64)[:, None] * freq
    c, s = mult * np.cos(ang)[:, None, :], mult * np.sin(ang)[:, None, :]
    iu, iv = (np.arange(0, 2 * m, 2), np.arange(1, 2 * m, 2)) if pairs else (np.arange(m), np.arange(m, 2 * m))
    u, v = out[..., iu].copy(), out[..., iv].copy()
    out[..., iu] = u * c - v * s
    out[..., iv] = v * c + u * s
    return out


def seen(i, window, keep_first):
    """positions that i sees"""
    return [j for j in range(i + 1) if window <= 0 or i - j < window or j < keep_first]


def softmax_attention(q, k, v, scale, softcap=0.0, window=0, keep_first=0, sinks=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; head h reads key/value head h // (H / G)"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    g = np.arange(H) // (H // G)
    for i in range(T):
        js = seen(i, window, keep_first)
        s = np.einsum("hd,jhd->hj", q[i], k[js][:, g]) * scale
        if softcap > 0:
            s = softcap * np.tanh(s / softcap)
        top = s.max(-1) if sinks is None else np.maximum(s.max(-1), sinks)
        p = np.exp(s - top[:, None])
        den = p.sum(-1) + (0.0 if sinks is None else np.exp(sinks - top))
        out[i] = np.einsum("hj,jhd->hd", p / den[:, None], v[js][:, g])
    return out


def decayed_recurrence(q, k, v, a):
    """q, k, a [T, H, D], v [T, H, Dv] -> [T, H, Dv]"""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def route(z, correction, top, group_count, group_keep, factor):
    """router outputs z [T, E] -> (chosen [T, top], their weights)"""
    T, E = z.shape
    s = sigmoid(z)
    choice = s + correction
    if group_count > 1 and group_keep < group_count:
        members = choice.reshape(T, group_count, E // group_count)
        rank = np.sort(members, axis=-1)[..., -2:].sum(-1)
        best = np.argsort(-rank, axis=-1, kind="stable")[:, :group_keep]
        open_ = np.zeros((T, group_count), bool)
        np.put_along_axis(open_, best, True, -1)
        choice = np.where(np.repeat(open_, E // group_count, axis=1), choice, -np.inf)
    order = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    return order, factor * np.take_along_axis(s, order, -1)


# ---------------------------------------------------------------- mixers and feed-forwards from named tensors
def attention_mixer(h, P, pre, m, eps, positions):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ P[pre + n].T + P[pre + n + ".b"]).reshape(T, c, d) for n, c, d in (("q", H, D), ("k", G, D), ("v", G, Dv)))
    f = plain_frequencies(m["rot"])
    q, k = (unit_rms(rotate(x, positions, f, False), eps) for x in (q, k))
    mask = m.get("mask") or {}
    o = softmax_attention(q, k, v, m["scale"], m.get("softcap") or 0.0, mask.get("size") or 0, mask.get("keep_first") or 0, P[pre + "sink"])
    return o.reshape(T, H * Dv) @ P[pre + "o"].T


def latent_rows(h, P, pre, m, eps, positions):
    """-> (c [T, kv_rank], rotated key part [T, rot_dim])"""
    R = m["kv_rank"]
    y = h @ P[pre + "dkv"].T
    f, mult = stretched_frequencies(m["rot"])
    return unit_rms(y[:, :R], eps) * P[pre + "dkv.norm"], rotate(y[:, None, R:], positions, f, True, mult)[:, 0]


def latent_mixer(h, P, pre, m, positions, c, r):
    T = h.shape[0]
    H, D, Dr, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ P[pre + "q"].T).reshape(T, H, D + Dr)
    f, mult = stretched_frequencies(m["rot"])
    q = np.concatenate([q[..., :D], rotate(q[..., D:], positions, f, True, mult)], axis=-1)
    k = np.concatenate([(c @ P[pre + "uk"].T).reshape(T, H, D), np.repeat(r[:, None], H, axis=1)], axis=-1)
    v = (c @ P[pre + "uv"].T).reshape(T, H, Dv)
    o = softmax_attention(q, k, v, m["scale"], window=(m.get("mask") or {}).get("size") or 0).reshape(T, H * Dv)
    return (o * sigmoid(h @ P[pre + "g"].T)) @ P[pre + "o"].T


def gla_mixer(h, P, pre, m, eps):
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q, k = (h @ P[pre + "q"].T).reshape(T, H, D) * D ** -0.5, (h @ P[pre + "k"].T).reshape(T, H, D)
    z = (h @ P[pre + "a1"].T) @ P[pre + "a2"].T + P[pre + "a2.b"]
    a = sigmoid(z) ** (1.0 / m["tau"])
    o = decayed_recurrence(q, k, (h @ P[pre + "v"].T).reshape(T, H, Dv), a.reshape(T, H, D))
    o = (unit_rms(o, eps) * P[pre + "norm"]).reshape(T, H * Dv)
    return (o * silu(h @ P[pre + "g"].T)) @ P[pre + "o"].T


def expert(h, P, pre):
    return relu2(h @ P[pre + "up"].T) @ P[pre + "down"].T


def feed_forward(h, P, pre, f):
    if f["kind"] == "dense":
        return gelu_tanh(h @ P[pre + "up"].T) @ P[pre + "down"].T
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    chosen, wts = route(h @ P[pre + "router"].T, P[pre + "correction"], r["top"], g["count"], g["keep"], r.get("scale", 1.0))
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        rows, slot = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += wts[rows, slot][:, None] * expert(h[rows], P, f"{pre}e{e}.")
    if f.get("shared"):
        out += sigmoid(h @ P[pre + "shared.sg"].T) * expert(h, P, pre + "shared.")
    return out


def forward(cfg, P, tokens, want_layers=False):
    """-> logits [T, vocab] (and the residual stream after every layer, [layers, T, W])"""
    P = {n: np.asarray(a, np.float64) for n, a in P.items()}
    eps = cfg["norm"]["eps"]
    x = P["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    pos = np.arange(len(tokens))
    rows, latents = [], {}

    def norm(v, name):
        return unit_rms(v, eps) * (1.0 + P[name])

    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(x, p + "norm1")
        if L["type"] == "attention":
            y = attention_mixer(h, P, p + "mix.", m, eps, pos)
        elif L["type"] == "latent_attention":
            if m.get("kv_from") is None:
                latents[i] = latent_rows(h, P, p + "mix.", m, eps, pos)
            y = latent_mixer(h, P, p + "mix.", m, pos, *latents[i if m.get("kv_from") is None else m["kv_from"]])
        elif L["type"] == "gla":
            y = gla_mixer(h, P, p + "mix.", m, eps)
        else:
            raise ValueError(L["type"])
        x = x + y
        if L.get("mlp"):
            x = x + feed_forward(norm(x, p + "norm2"), P, p + "mlp.", L["mlp"])
        rows.append(x.copy())
    logits = norm(x, "final.norm") @ P["head"].T
    return (logits, np.stack(rows)) if want_layers else logits


# ---------------------------------------------------------------- small configurations and random weights for the tests
def attention_layer(heads=4, kv_heads=2, dim=12, vdim=10, dims=8, base=300.0, factor=3.0, scale=1.1, softcap=7.0, window=9,
                    keep_first=3, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                      "rot": {"dims": dims, "base": base, "scaling": {"factor": factor}}, "mask": {"size": window, "keep_first": keep_first}}}


def latent_layer(heads=3, dim=10, rot_dim=8, vdim=6, kv_rank=14, scale=0.5, window=11, base=400.0, factor=5.0, original=64, fast=6.0,
                 slow=1.0, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "mask": {"size": window},
         "rot": {"dims": rot_dim, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def gla_layer(heads=3, dim=8, vdim=6, tau=5.0, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense_ff(ff=24):
    return {"kind": "dense", "ff": ff}


def moe_ff(experts=6, top=2, ff=12, shared_ff=10, groups=(3, 2), scale=1.7):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def make_config(layers, vocab=90, width=40, eps=1e-5, embed_scale=1.6):
    return {"architecture": "Goluzen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}}


def bf16_round(a):
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    b = ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32)
    return b.view(np.float32)


def random_params(cfg, seed=0, rank=5):
    """{tensor name: float32 array}, rounded to bfloat16-representable values so that both modes load the same numbers; rank: the
    inner size of the decays' two products"""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    bf = bf16_round

    def mat(n, k, gain=1.0):
        return bf(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def small(n, s=0.1):
        return bf(s * rng.standard_normal(n))

    P = {"embed": bf(rng.standard_normal((V, W))), "final.norm": small(W), "head": mat(V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mp = p + "mix."
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        P[p + "norm1"] = small(W)
        P[mp + "o"] = mat(W, H * Dv)
        if L["type"] == "attention":
            G = m["kv_heads"]
            for n, c in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                P[mp + n], P[mp + n + ".b"] = mat(c, W), small(c, 0.5)
            P[mp + "sink"] = bf(rng.uniform(-1.0, 2.0, H))
        elif L["type"] == "latent_attention":
            R, Dr = m["kv_rank"], m["rot_dim"]
            P[mp + "q"], P[mp + "g"] = mat(H * (D + Dr), W), mat(H * Dv, W)
            P[mp + "uk"], P[mp + "uv"] = mat(H * D, R), mat(H * Dv, R)
            if m.get("kv_from") is None:
                P[mp + "dkv"], P[mp + "dkv.norm"] = mat(R + Dr, W), bf(1.0 + 0.2 * rng.standard_normal(R))
        else:
            P[mp + "q"], P[mp + "k"], P[mp + "v"], P[mp + "g"] = mat(H * D, W), mat(H * D, W), mat(H * Dv, W), mat(H * Dv, W)
            P[mp + "a1"], P[mp + "a2"], P[mp + "a2.b"] = mat(rank, W), mat(H * D, rank, 2.0), bf(rng.uniform(-1.0, 4.0, H * D))
            P[mp + "norm"] = bf(1.0 + 0.2 * rng.standard_normal(Dv))
        f = L.get("mlp")
        if not f:
            continue
        P[p + "norm2"] = small(W)
        q = p + "mlp."
        if f["kind"] == "dense":
            P[q + "up"], P[q + "down"] = mat(f["ff"], W), mat(W, f["ff"])
        else:
            E = f["router"]["experts"]
            for e in range(E):
                P[f"{q}e{e}.up"], P[f"{q}e{e}.down"] = mat(f["expert"]["ff"], W), mat(W, f["expert"]["ff"], 0.7)
            P[q + "router"], P[q + "correction"] = mat(E, W, 1.5), bf(rng.uniform(-0.9, 0.3, E))
            if f.get("shared"):
                P[q + "shared.up"], P[q + "shared.down"] = mat(f["shared"]["ff"], W), mat(W, f["shared"]["ff"])
                P[q + "shared.sg"] = mat(1, W)
    return P
