"""NumPy float64 oracle of the Vosolorn design: whole sequences at once, no cache, no state, one function per mechanism,
no code shared with the package.  Notation: T tokens, W width, H heads, G key/value heads, D key size, Dv value size.

    layer        x += ls1 * rms(mixer(x)) w1;  x += ls2 * rms(ff(x)) w2      (both sublayers read x itself)
    attention    q, k: rms per head with a weight, then rotated (elements 2i and 2i + 1 paired, the first `dims`, angle
                 p * base^(-2i/dims));  v rotated the same way over all Dv elements;  s_ij = scale q_i.k_j;  i sees the tokens
                 j with 0 <= i - j < window and, beside them, one key and one value per block of `pool` tokens that lies
                 wholly before the window, the means of the block's keys and values;  one softmax over both;  every head's
                 output is turned back by i;  W_o
    mlstm        q = W_q x D^(-1/2), k, v;  log gates i = c tanh((W_i x + b_i) / c), f = log sigmoid(c tanh((W_f x + b_f) / c));
                 S_t = exp(f) S_(t-1) + exp(i) k v^T and n_t likewise with k, both scaled by exp(-m_t) with the running
                 maximum m_t = max(f + m_(t-1), i), m = 0 at the start;  o = S^T q / (max(|n.q|, exp(-m)) + 1e-6);
                 W_o (rms(o) per head * w * sigmoid(W_g x))
    dense ff     W_down (gelu_tanh(W_gate x) * W_up x)
    moe          z = W_r x + b;  the `top` largest are chosen, weights softmax over the chosen;  expert W_down gelu_erf(W_up x);
                 + a shared expert of the same form
    output       logit_scale * embed . rms(x) w
"""
import math

import numpy as np

_erf = np.vectorize(math.erf, otypes=[np.float64])


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / np.sqrt(2.0)))


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotate_pairs(x, positions, dims, base, sign=1.0):
    """x [T, heads, n]: elements 2i and 2i + 1 of the first `dims` turn by sign * position * base^(-2i/dims)"""
    out = np.array(x, np.float64)
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    ang = sign * np.asarray(positions, np.float64)[:, None] * f
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    a, b = out[..., 0:dims:2].copy(), out[..., 1:dims:2].copy()
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def window_and_blocks(i, window, pool):
    """(tokens, blocks) that position i sees"""
    lo = max(0, i - window + 1) if window > 0 else 0
    blocks = [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - window] if pool > 0 and window > 0 else []
    return list(range(lo, i + 1)), blocks


def pooled_window_attention(q, k, v, scale, window, pool):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; head h reads key/value head h // (H / G)"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    nb = T // pool if pool > 0 else 0
    kb = np.stack([k[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]) if nb else np.zeros((0,) + k.shape[1:])
    vb = np.stack([v[b * pool:(b + 1) * pool].mean(0) for b in range(nb)]) if nb else np.zeros((0,) + v.shape[1:])
    for i in range(T):
        toks, blocks = window_and_blocks(i, window, pool)
        K, V = np.concatenate([kb[blocks], k[toks]]), np.concatenate([vb[blocks], v[toks]])
        for h in range(H):
            g = h // (H // G)
            s = K[:, g] @ q[i, h] * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ V[:, g]
    return out


def mlstm_recurrence(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, Dv], log gates i, f [T, H] -> [T, H, Dv]"""
    T, H, D = q.shape
    S, n, m = np.zeros((H, D, v.shape[2])), np.zeros((H, D)), np.zeros(H)
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        m_new = np.maximum(f[t] + m, i[t])
        a, b = np.exp(f[t] + m - m_new), np.exp(i[t] - m_new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = m_new
        den = np.maximum(np.abs((n * q[t]).sum(-1)), np.exp(-m)) + 1e-6
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


def route(z, top):
    """router outputs z [T, E] -> (chosen [T, top], their weights)"""
    order = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    s = np.take_along_axis(z, order, -1)
    s = np.exp(s - s.max(-1, keepdims=True))
    return order, s / s.sum(-1, keepdims=True)


# ---------------------------------------------------------------- mixers and feed-forwards from named tensors
def attention_mixer(x, P, pre, m, eps, positions):
    T = x.shape[0]
    H, G, D, Dv = m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q = unit_rms((x @ P[pre + "q"].T).reshape(T, H, D), eps) * P[pre + "q.norm"]
    k = unit_rms((x @ P[pre + "k"].T).reshape(T, G, D), eps) * P[pre + "k.norm"]
    v = (x @ P[pre + "v"].T).reshape(T, G, Dv)
    rot, mask = m["rot"], m.get("mask") or {}
    q, k = rotate_pairs(q, positions, rot["dims"], rot["base"]), rotate_pairs(k, positions, rot["dims"], rot["base"])
    v = rotate_pairs(v, positions, Dv, rot["base"])
    o = pooled_window_attention(q, k, v, m["scale"], int(mask.get("size") or 0), int(mask.get("pool") or 0))
    o = rotate_pairs(o, positions, Dv, rot["base"], -1.0)
    return o.reshape(T, H * Dv) @ P[pre + "o"].T


def mlstm_mixer(x, P, pre, m, eps):
    T = x.shape[0]
    H, D, Dv, cap = m["heads"], m["dim"], m.get("vdim") or m["dim"], m["gate_cap"]
    q = (x @ P[pre + "q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (x @ P[pre + "k"].T).reshape(T, H, D), (x @ P[pre + "v"].T).reshape(T, H, Dv)
    i = cap * np.tanh((x @ P[pre + "i"].T + P[pre + "i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((x @ P[pre + "f"].T + P[pre + "f.b"]) / cap))
    o = unit_rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * Dv)
    return (o * P[pre + "norm"] * sigmoid(x @ P[pre + "g"].T)) @ P[pre + "o"].T


def expert(x, P, pre):
    return gelu_erf(x @ P[pre + "up"].T) @ P[pre + "down"].T


def feed_forward(x, P, pre, f):
    if f["kind"] == "dense":
        return (gelu_tanh(x @ P[pre + "gate"].T) * (x @ P[pre + "up"].T)) @ P[pre + "down"].T
    chosen, wts = route(x @ P[pre + "router"].T + P[pre + "router.b"], f["router"]["top"])
    out = np.zeros_like(x)
    for e in range(f["router"]["experts"]):
        rows, slot = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += wts[rows, slot][:, None] * expert(x[rows], P, f"{pre}e{e}.")
    if f.get("shared"):
        out += expert(x, P, pre + "shared.")
    return out


def forward(cfg, P, tokens, want_layers=False):
    """-> logits [T, vocab] (and the residual stream after every layer, [layers, T, W])"""
    P = {n: np.asarray(a, np.float64) for n, a in P.items()}
    eps = cfg["norm"]["eps"]
    x = unit_rms(P["embed"][np.asarray(tokens)], eps) * P["embed.norm"]
    pos = np.arange(len(tokens))
    seen = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        if L["type"] == "attention":
            y = attention_mixer(x, P, p + "mix.", L["mixer"], eps, pos)
        elif L["type"] == "mlstm":
            y = mlstm_mixer(x, P, p + "mix.", L["mixer"], eps)
        else:
            raise ValueError(L["type"])
        x = x + P[p + "ls1"] * (unit_rms(y, eps) * P[p + "norm1"])
        if L.get("mlp"):
            x = x + P[p + "ls2"] * (unit_rms(feed_forward(x, P, p + "mlp.", L["mlp"]), eps) * P[p + "norm2"])
        seen.append(x.copy())
    logits = (unit_rms(x, eps) * P["final.norm"]) @ P["embed"].T * cfg["logit_scale"]
    return (logits, np.stack(seen)) if want_layers else logits


# ---------------------------------------------------------------- small configurations and random weights for the tests
def attention_layer(heads=4, kv_heads=2, dim=12, vdim=10, dims=8, base=300.0, scale=0.4, window=9, pool=4, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "rot": {"dims": dims, "base": base}, "mask": {"size": window, "pool": pool}}}


def mlstm_layer(heads=3, dim=8, vdim=6, gate_cap=9.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def dense_ff(ff=24):
    return {"kind": "dense", "ff": ff}


def moe_ff(experts=5, top=3, ff=12, shared_ff=10):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff}
    return f


def make_config(layers, vocab=90, width=40, eps=1e-5, logit_scale=0.6):
    return {"architecture": "Vosolorn", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "logit_scale": logit_scale}


def bf16_round(a):
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    b = ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32)
    return b.view(np.float32)


def random_params(cfg, seed=0):
    """{tensor name: float32 array}, rounded to bfloat16-representable values so that both modes load the same numbers"""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    bf = bf16_round

    def mat(n, k, gain=1.0):
        return bf(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def around_one(n):
        return bf(1.0 + 0.1 * rng.standard_normal(n))

    P = {"embed": bf(rng.standard_normal((V, W))), "embed.norm": around_one(W), "final.norm": around_one(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mp = p + "mix."
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        P[p + "norm1"], P[p + "ls1"] = around_one(W), bf(rng.uniform(0.3, 1.5, W))
        if L["type"] == "attention":
            G = m.get("kv_heads") or H
            P[mp + "q"], P[mp + "k"], P[mp + "v"], P[mp + "o"] = mat(H * D, W), mat(G * D, W), mat(G * Dv, W), mat(W, H * Dv)
            P[mp + "q.norm"], P[mp + "k.norm"] = bf(rng.uniform(0.5, 1.5, D)), bf(rng.uniform(0.5, 1.5, D))
        else:
            P[mp + "q"], P[mp + "k"], P[mp + "v"], P[mp + "g"] = mat(H * D, W, 2.0), mat(H * D, W, 2.0), mat(H * Dv, W), mat(H * Dv, W)
            P[mp + "i"], P[mp + "f"], P[mp + "o"] = mat(H, W, 2.0), mat(H, W), mat(W, H * Dv)
            P[mp + "i.b"], P[mp + "f.b"] = bf(rng.standard_normal(H)), bf(rng.uniform(1.0, 5.0, H))
            P[mp + "norm"] = around_one(H * Dv)
        f = L.get("mlp")
        if not f:
            continue
        P[p + "norm2"], P[p + "ls2"] = around_one(W), bf(rng.uniform(0.3, 1.5, W))
        q = p + "mlp."
        if f["kind"] == "dense":
            P[q + "gate"], P[q + "up"], P[q + "down"] = mat(f["ff"], W), mat(f["ff"], W), mat(W, f["ff"])
        else:
            E = f["router"]["experts"]
            for e in range(E):
                P[f"{q}e{e}.up"], P[f"{q}e{e}.down"] = mat(f["expert"]["ff"], W), mat(W, f["expert"]["ff"])
            P[q + "router"], P[q + "router.b"] = mat(E, W, 2.0), bf(0.5 * rng.standard_normal(E))
            if f.get("shared"):
                P[q + "shared.up"], P[q + "shared.down"] = mat(f["shared"]["ff"], W), mat(W, f["shared"]["ff"])
    return P
