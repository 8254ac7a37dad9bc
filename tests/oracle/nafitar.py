"""A slow, literal implementation of the Nafitar decoder for the tests: one function per mechanism, one token or one
score at a time where that is the clearest form, float64 by default.  It works on the checkpoint's own tensors (a plain
dict of name -> tensor) and on the configuration dict, and shares no code with ``gcore_b200``."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1 + w)


def token_embedding(W, tokens):
    return W["embed"][tokens] + W["pos"][torch.arange(len(tokens))]


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def window_attention(W, name, m, h):
    """Grouped-query attention whose values are its keys, with a distance penalty and a sliding window."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[name + ".q"].T + W[name + ".q.b"]).view(T, H, d)
    k = (h @ W[name + ".k"].T + W[name + ".k.b"]).view(T, G, d)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    sl = slopes(H)
    for t in range(T):
        lo = max(0, t - m["mask"]["size"] + 1)
        dist = torch.arange(t - lo, -1, -1, dtype=h.dtype)
        for a in range(H):
            keys = k[lo:t + 1, a // (H // G)]
            p = torch.softmax(keys @ q[t, a] * m["scale"] - sl[a] * dist, 0)
            out[t, a] = p @ keys
    return out.reshape(T, H * d) @ W[name + ".o"].T


def matrix_memory(W, name, m, h, eps, state=None, core=False):
    """The gated matrix memory, token by token.  ``state``: list of (S, n, m) per head, updated in place."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W[name + ".q"].T).view(T, H, d) * d ** -0.5
    k = (h @ W[name + ".k"].T).view(T, H, d)
    v = (h @ W[name + ".v"].T).view(T, H, dv)
    gi = cap * torch.tanh((h @ W[name + ".i"].T + W[name + ".i.b"]) / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ W[name + ".f"].T + W[name + ".f.b"]) / cap))
    if state is None:
        state = fresh_memory(m, h.dtype)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        S, n, mx = state[a]
        for t in range(T):
            new = torch.maximum(gf[t, a] + mx, gi[t, a])
            keep, put = torch.exp(gf[t, a] + mx - new), torch.exp(gi[t, a] - new)
            S = keep * S + put * torch.outer(k[t, a], v[t, a])
            n = keep * n + put * k[t, a]
            mx = new
            den = torch.maximum((n @ q[t, a]).abs(), torch.exp(-mx)) + 1e-6
            out[t, a] = (S.T @ q[t, a]) / den
        state[a] = (S, n, mx)
    if core:
        return out
    y = rms(out, eps).reshape(T, H * dv) * W[name + ".norm"] * torch.sigmoid(h @ W[name + ".g"].T)
    return y @ W[name + ".o"].T


def fresh_memory(m, dtype=torch.float64):
    return [(torch.zeros(m["dim"], m["vdim"], dtype=dtype), torch.zeros(m["dim"], dtype=dtype),
             torch.zeros((), dtype=dtype)) for _ in range(m["heads"])]


def side_by_side(W, name, mixer, h, eps):
    a = window_attention(W, name + ".left", mixer["left"], h)
    b = matrix_memory(W, name + ".right", mixer["right"], h, eps)
    return 0.5 * (rms(a, eps) * W[name + ".left.out"] + rms(b, eps) * W[name + ".right.out"])


def feed_forward(W, name, h):
    g = h @ W[name + ".gate"].T
    return (g * torch.sigmoid(g) * (h @ W[name + ".up"].T)) @ W[name + ".down"].T


def layer(W, i, spec, x, eps):
    n = f"l{i}"
    x = x + norm_around_zero(side_by_side(W, n + ".mix", spec["mixer"], norm_around_zero(x, W[n + ".norm1"], eps), eps),
                             W[n + ".norm1b"], eps)
    if spec.get("mlp") is not None:
        x = x + norm_around_zero(feed_forward(W, n + ".mlp", norm_around_zero(x, W[n + ".norm2"], eps)),
                                 W[n + ".norm2b"], eps)
    return x


def run_order(config):
    """[(layer, pass number or None for a layer outside the loop, first of its pass)]"""
    L, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None, False) for i in range(L)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t, i == a) for i in range(a, b)]
    return order + [(i, None, False) for i in range(b, L)]


def forward(W, config, tokens, dtype=torch.float64, collect=None):
    """Logits [T, vocab] of one whole sequence; ``collect`` (a list) receives the residual after every layer run."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = first = token_embedding(W, tokens)
    for i, t, opens in run_order(config):
        if opens:
            if t > 0:
                x = x + first
            x = x + W["loop.step"][t]
        x = layer(W, i, config["layers"][i], x, eps)
        if collect is not None:
            collect.append(x.clone())
    return norm_around_zero(x, W["final.norm"], eps) @ W["head"].T


def random_weights(config, seed=0, scale=1.0):
    """Small random weights for a configuration, in the checkpoint's layout and precision."""
    g = torch.Generator().manual_seed(seed)

    def r(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    w, V = config["width"], config["vocab"]
    W = {"embed": r(V, w), "pos": r(config["max_positions"], w, std=0.3), "final.norm": r(w, std=0.1),
         "head": r(V, w, std=1 / math.sqrt(w))}
    if config.get("loop"):
        W["loop.step"] = r(config["loop"]["times"], w, std=0.3)
    for i, sp in enumerate(config["layers"]):
        n, a, b = f"l{i}", sp["mixer"]["left"], sp["mixer"]["right"]
        for nm in ("norm1", "norm1b"):
            W[f"{n}.{nm}"] = r(w, std=0.1)
        s = scale / math.sqrt(w)
        qd, kd, vd = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], b["heads"] * b["vdim"]
        for nm, shape in (("left.q", (qd, w)), ("left.k", (kd, w)), ("right.q", (b["heads"] * b["dim"], w)),
                          ("right.k", (b["heads"] * b["dim"], w)), ("right.v", (vd, w)), ("right.g", (vd, w)),
                          ("right.i", (b["heads"], w)), ("right.f", (b["heads"], w))):
            W[f"{n}.mix.{nm}"] = r(*shape, std=s)
        W[f"{n}.mix.left.q.b"], W[f"{n}.mix.left.k.b"] = r(qd, std=0.2), r(kd, std=0.2)
        W[f"{n}.mix.left.o"] = r(w, qd, std=1 / math.sqrt(qd))
        W[f"{n}.mix.right.o"] = r(w, vd, std=1 / math.sqrt(vd))
        W[f"{n}.mix.right.norm"] = 1 + r(vd, std=0.1)
        W[f"{n}.mix.right.i.b"] = r(b["heads"], std=1.0)
        W[f"{n}.mix.right.f.b"] = 2 + r(b["heads"], std=2.0)
        W[f"{n}.mix.left.out"], W[f"{n}.mix.right.out"] = 1 + r(w, std=0.2), 1 + r(w, std=0.2)
        if sp.get("mlp") is not None:
            W[f"{n}.norm2"], W[f"{n}.norm2b"] = r(w, std=0.1), r(w, std=0.1)
            f = sp["mlp"]["ff"]
            W[f"{n}.mlp.gate"], W[f"{n}.mlp.up"] = r(f, w, std=s), r(f, w, std=s)
            W[f"{n}.mlp.down"] = r(w, f, std=1 / math.sqrt(f))
    return W
