"""Plain NumPy float64 oracle of the Vupitar decoder: one function per mechanism, token by token with explicit state,
written from the equations and sharing no code with the library.

A layer adds the results of its mixer and of its feed-forward to the residual stream at once, each read through a norm
of its own:  x <- x + mixer(n1(x)) + ff(n2(x)).  The norm is element-wise (dynamic tanh).  The mixer is a pair: softmax
attention inside chunks of the sequence (biased projections, normed and rotated queries and keys, a gate per head)
beside a matrix memory with exponential gates (mLSTM).  The feed-forward is a clamped gated unit or a mixture of gated
experts with a shared one.  A block of layers may run several times: ahead of a pass the embedding output (from the
second pass on) and the pass's step vector join the stream.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def dynamic_tanh(x, alpha, w, b):
    return np.tanh(alpha * x) * w + b


def rms_unit(v, eps):
    return v / np.sqrt((v * v).mean(-1, keepdims=True) + eps)


def rotate_halves(v, pos, dims, base):
    """Entries i and i + dims / 2 of the last axis turn by pos * base^(-2 i / dims); entries from `dims` on stay."""
    half = dims // 2
    if half == 0:
        return v.copy()
    ang = pos * base ** (-2.0 * np.arange(half) / dims)
    u, w = v[..., :half], v[..., half:dims]
    return np.concatenate([u * np.cos(ang) - w * np.sin(ang), w * np.cos(ang) + u * np.sin(ang), v[..., dims:]], -1)


def visible_in_chunk(i, j, size):
    """Position i sees j: not later than itself and in the same chunk of `size` positions (0: no chunks)."""
    return j <= i and (size <= 0 or i // size == j // size)


def softmax(z):
    e = np.exp(z - z.max())
    return e / e.sum()


def chunk_attention(h, mc, P, st, pos, eps):
    """One token of the left mixer.  st: lists 'k' and 'v' of every earlier position."""
    H, G, dk, dv = mc["heads"], mc.get("kv_heads", mc["heads"]), mc["dim"], mc["vdim"]
    rot = mc.get("rot") or {"dims": 0, "base": 1.0}
    q = (P["q"] @ h + P["q.b"]).reshape(H, dk)
    k = (P["k"] @ h + P["k.b"]).reshape(G, dk)
    v = (P["v"] @ h + P["v.b"]).reshape(G, dv)
    q = rotate_halves(rms_unit(q, eps) * P["q.norm"], pos, rot["dims"], rot["base"])
    k = rotate_halves(rms_unit(k, eps) * P["k.norm"], pos, rot["dims"], rot["base"])
    st.setdefault("k", []).append(k)
    st.setdefault("v", []).append(v)
    seen = [j for j in range(pos + 1) if visible_in_chunk(pos, j, (mc.get("mask") or {}).get("size", 0))]
    K, V = np.stack([st["k"][j] for j in seen]), np.stack([st["v"][j] for j in seen])
    gate = sigmoid(P["g"] @ h)
    out = np.zeros((H, dv))
    for a in range(H):
        g = a // (H // G)
        out[a] = gate[a] * (softmax(K[:, g] @ q[a] * mc["scale"]) @ V[:, g])
    return P["o"] @ out.reshape(-1) + P["o.b"]


def mlstm_gates(zi, zf, cap):
    """Log input gate and log forget gate."""
    return cap * np.tanh(zi / cap), log_sigmoid(cap * np.tanh(zf / cap))


def mlstm_update(S, n, m, q, k, v, i, f):
    """One head, one token: (S, n, m, output)."""
    m2 = max(f + m, i)
    a, b = np.exp(f + m - m2), np.exp(i - m2)
    S = a * S + b * np.outer(k, v)
    n = a * n + b * k
    return S, n, m2, (S.T @ q) / (max(abs(n @ q), np.exp(-m2)) + 1e-6)


def mlstm(h, mc, P, st, eps):
    """One token of the right mixer.  st: 'S' [H, dim, vdim], 'n' [H, dim], 'm' [H], zeros at first."""
    H, dk, dv = mc["heads"], mc["dim"], mc["vdim"]
    if "S" not in st:
        st.update(S=np.zeros((H, dk, dv)), n=np.zeros((H, dk)), m=np.zeros(H))
    q = (P["q"] @ h).reshape(H, dk) * dk ** -0.5
    k = (P["k"] @ h).reshape(H, dk)
    v = (P["v"] @ h).reshape(H, dv)
    i, f = mlstm_gates(P["i"] @ h + P["i.b"], P["f"] @ h + P["f.b"], mc["gate_cap"])
    o = np.zeros((H, dv))
    for a in range(H):
        st["S"][a], st["n"][a], st["m"][a], o[a] = mlstm_update(st["S"][a], st["n"][a], st["m"][a], q[a], k[a], v[a], i[a], f[a])
    o = rms_unit(o, eps).reshape(-1) * P["norm"] * sigmoid(P["g"] @ h)
    return P["o"] @ o


def clamped_unit(h, P, limit):
    g = np.minimum(P["gate"] @ h, limit)
    u = np.clip(P["up"] @ h, -limit, limit)
    return P["down"] @ (g * sigmoid(1.702 * g) * (u + 1.0))


def gated_expert(h, P):
    return P["down"] @ (silu(P["gate"] @ h) * (P["up"] @ h))


def route(z, top):
    """(chosen experts, their weights): the largest softmax scores, over their own sum."""
    s = softmax(z)
    best = np.argsort(-s, kind="stable")[:top]
    return best, s[best] / (s[best].sum() + 1e-20)


def mixture(h, mlp, P):
    best, w = route(P["router"] @ h, mlp["router"]["top"])
    y = sum(wk * gated_expert(h, sub(P, f"e{e}.")) for e, wk in zip(best, w))
    if mlp.get("shared"):
        y = y + sigmoid(P["shared.sg"] @ h) * gated_expert(h, sub(P, "shared."))
    return y


def sub(P, prefix):
    return {k[len(prefix):]: v for k, v in P.items() if k.startswith(prefix)}


class OracleVupitar:
    def __init__(self, config, tensors):
        self.c = config
        self.t = {k: np.asarray(v, np.float64) for k, v in tensors.items()}
        self.layers = [sub(self.t, f"l{i}.") for i in range(len(config["layers"]))]
        lp = config.get("loop")
        n = len(self.layers)
        if lp and lp["times"] > 0:
            block = range(lp["start"], lp["stop"])
            self.runs = [(i, -1) for i in range(lp["start"])]
            for p in range(lp["times"]):
                self.runs += [(i, p if i == lp["start"] else -1) for i in block]
            self.runs += [(i, -1) for i in range(lp["stop"], n)]
        else:
            self.runs = [(i, -1) for i in range(n)]
        self.reset()

    def reset(self):
        self.pos = 0
        self.state = [{"left": {}, "right": {}} for _ in self.runs]

    def norm(self, x, P, name):
        return dynamic_tanh(x, float(np.reshape(P[name + ".alpha"], -1)[0]), P[name], P[name + ".b"])

    def layer(self, i, x, st, pos):
        lc, P, eps = self.c["layers"][i], self.layers[i], self.c["norm"]["eps"]
        mc, mlp = lc["mixer"], lc.get("mlp")
        h = self.norm(x, P, "norm1")
        y = mc["left_scale"] * chunk_attention(h, mc["left"], sub(P, "mix.left."), st["left"], pos, eps)
        y = y + mc["right_scale"] * mlstm(h, mc["right"], sub(P, "mix.right."), st["right"], eps)
        if mlp is not None:
            h2, F = self.norm(x, P, "norm2"), sub(P, "mlp.")
            y = y + (mixture(h2, mlp, F) if mlp["kind"] == "moe" else clamped_unit(h2, F, mlp["limit"]))
        return x + y

    def step(self, token):
        x0 = self.t["embed"][token] * (self.c.get("embedding") or {}).get("scale", 1.0)
        x, trace = x0, []
        for r, (i, p) in enumerate(self.runs):
            if p >= 0:
                x = x + (x0 if p > 0 else 0.0) + self.t["loop.step"][p]
            x = self.layer(i, x, self.state[r], self.pos)
            trace.append(x)
        self.pos += 1
        return self.t["head"] @ self.norm(x, self.t, "final.norm"), np.stack(trace)

    def run(self, ids, want_residual=False):
        out = [self.step(int(t)) for t in ids]
        logits = np.stack([o[0] for o in out])
        return (logits, np.stack([o[1] for o in out], 1)) if want_residual else logits


def random_model(config, seed):
    """Random float32 tensors (rounded to bfloat16, so that both modes of the library load the same numbers)."""
    rng = np.random.default_rng(seed)
    W, V = config["width"], config["vocab"]
    t = {}

    def put(name, *shape, scale=None, bias=0.0):
        scale = 1.0 / np.sqrt(shape[-1]) if scale is None else scale
        a = (bias + scale * rng.standard_normal(shape)).astype(np.float32)
        t[name] = ((a.view(np.uint32) + 0x8000) & 0xFFFF0000).view(np.float32) if a.ndim else np.float32(round(float(a) * 64) / 64)

    def norm(name):
        put(name, W, scale=0.2, bias=1.0)
        put(name + ".b", W, scale=0.1)
        put(name + ".alpha", scale=0.15, bias=0.7)

    def unit(p, ff):
        put(p + "gate", ff, W)
        put(p + "up", ff, W)
        put(p + "down", W, ff)

    put("embed", V, W, scale=0.3)
    lp = config.get("loop")
    if lp and lp["times"] > 0:
        put("loop.step", lp["times"], W, scale=0.3)
    for i, lc in enumerate(config["layers"]):
        p, a, r = f"l{i}.", lc["mixer"]["left"], lc["mixer"]["right"]
        norm(p + "norm1")
        H, G, dk, dv = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a["vdim"]
        for nm, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            put(p + "mix.left." + nm, rows, W)
            put(p + "mix.left." + nm + ".b", rows, scale=0.3)
        put(p + "mix.left.q.norm", dk, scale=0.3, bias=1.2)
        put(p + "mix.left.k.norm", dk, scale=0.3, bias=1.2)
        put(p + "mix.left.g", H, W)
        put(p + "mix.left.o", W, H * dv)
        put(p + "mix.left.o.b", W, scale=0.2)
        H, dk, dv = r["heads"], r["dim"], r["vdim"]
        for nm, rows in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv), ("i", H), ("f", H)):
            put(p + "mix.right." + nm, rows, W, scale=(2.0 if nm in "if" else 1.0) / np.sqrt(W))
        put(p + "mix.right.o", W, H * dv)
        put(p + "mix.right.norm", H * dv, scale=0.2, bias=1.0)
        put(p + "mix.right.i.b", H, scale=0.5, bias=-1.0)
        put(p + "mix.right.f.b", H, scale=1.0, bias=2.5)
        mlp = lc.get("mlp")
        if mlp is None:
            continue
        norm(p + "norm2")
        if mlp["kind"] == "moe":
            put(p + "mlp.router", mlp["router"]["experts"], W, scale=2.0 / np.sqrt(W))
            for e in range(mlp["router"]["experts"]):
                unit(p + f"mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                unit(p + "mlp.shared.", mlp["shared"]["ff"])
                put(p + "mlp.shared.sg", 1, W)
        else:
            unit(p + "mlp.", mlp["ff"])
    norm("final.norm")
    put("head", V, W)
    return t
