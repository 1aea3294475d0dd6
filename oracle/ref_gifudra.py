"""Plain NumPy (float64) statement of the Gifudra decoder, one function per mechanism.

The oracle of `llama3_np_b200.gifudra`: it shares no code with the product path, runs token by token,
and keeps every intermediate in float64.  Nothing here is fast.

Notation: `X` holds the residual streams of one token, a row per stream [s, W]; `h` is a sublayer's
input row, `P` a dict of one layer's tensors with the `l<i>.` prefix removed, `st` the mutable
per-sequence state of one layer (the states of all layers are at hand for layers that share a cache).

    X_t = s_e * E[token] for every stream t
    sublayer q:  u = a_q . X;  y = ls_q * F_q(n_q * u / rms(u));  X_t <- sum_s M_q[s, t] X_s + b_q[t] y
    logits = s_l * E (n_f * x / rms(x)),  x = sum_t X_t
with a_q, b_q [s] and M_q [s, s] (indexed [from, to]) the layer's stream weights, F_1 the mixer and F_2
the feed-forward.  A configuration without streams has one row and plain sums.
"""
from __future__ import annotations

import numpy as np


# ------------------------------------------------------------------ scalar functions
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_halves(v, pos, dims, base):
    """Rotary position on the first `dims` entries of v, entry i paired with entry i + dims / 2; the angle of
    pair i at position pos is pos * base^(-2i / dims).  The remaining entries pass unchanged."""
    out = np.array(v, dtype=np.float64)
    half = dims // 2
    ang = pos * np.power(float(base), -2.0 * np.arange(half) / max(1, dims))
    c, s = np.cos(ang), np.sin(ang)
    a, b = out[:half].copy(), out[half:dims].copy()
    out[:half] = a * c - b * s
    out[half:dims] = b * c + a * s
    return out


def sink_softmax(z, sink):
    """Weights exp(z_i) / (exp(sink) + sum_j exp(z_j)): they add up to less than one."""
    m = max(np.max(z), sink)
    e = np.exp(z - m)
    return e / (e.sum() + np.exp(sink - m))


# ------------------------------------------------------------------ residual streams
def streams_in(X, P, q):
    """What sublayer q reads, ahead of its norm: a weighted sum of the streams."""
    return P[f"hc{q}.in"] @ X if f"hc{q}.in" in P else X[0]


def streams_out(X, y, P, q):
    """All streams at once from the old ones: new_t = sum_s mix[s, t] X_s + out[t] y."""
    if f"hc{q}.mix" not in P:
        return X + y[None]
    return P[f"hc{q}.mix"].T @ X + np.outer(P[f"hc{q}.out"], y)


# ------------------------------------------------------------------ mixer (one token)
def latent_rows(h, pos, P, mc, eps):
    """The cached row of one token: the normed latent and the rotated key part every head shares."""
    kv = P["mix.dkv"] @ h
    rank, rot = mc["kv_rank"], mc.get("rot") or {"dims": 0, "base": 1.0}
    return rms_unit(kv[:rank], eps) * P["mix.dkv.norm"], rotate_halves(kv[rank:], pos, rot["dims"], rot["base"])


def latent_attention_step(h, pos, P, mc, eps, st, owner=None):
    """Attention whose keys and values are expanded from one cached latent row per token.

    q-side: cq = w * unit(Wdq h); per head q = [q_c (dim) | q_r (rot_dim)] = rows of Wuq cq, q_r rotated.
    kv-side: rows [c | k_r] of every token so far - the layer's own (`owner` None: this token's row is
    appended first) or those of the layer whose state `owner` is.
    Head j: score(i) = scale * (q_c . (Wuk_j c_i) + q_r . k_r,i); weights over i <= pos with exp(sink_j) in the
    denominator; o_j = sum_i p_i Wuv_j c_i;  y = Wo (concat(o) * sigmoid(Wg h))."""
    H, dn, dr, dv, rank = mc["heads"], mc["dim"], mc["rot_dim"], mc["vdim"], mc["kv_rank"]
    rot = mc.get("rot") or {"dims": 0, "base": 1.0}
    cq = rms_unit(P["mix.dq"] @ h, eps) * P["mix.dq.norm"]
    q = (P["mix.uq"] @ cq).reshape(H, dn + dr)
    if owner is None:
        c, kr = latent_rows(h, pos, P, mc, eps)
        st.setdefault("c", []).append(c)
        st.setdefault("kr", []).append(kr)
        owner = st
    Wuk = P["mix.uk"].reshape(H, dn, rank)
    Wuv = P["mix.uv"].reshape(H, dv, rank)
    # this layer's expansion of the rows, token by token: [H, dn] keys and [H, dv] values
    st.setdefault("k", []).append(Wuk @ owner["c"][pos])
    st.setdefault("v", []).append(Wuv @ owner["c"][pos])
    K, V, KR = np.stack(st["k"]), np.stack(st["v"]), np.stack(owner["kr"])
    out = np.zeros((H, dv))
    st["p"] = []                   # the last token's attention weights, head by head (tests look at them)
    for j in range(H):
        qr = rotate_halves(q[j, dn:], pos, rot["dims"], rot["base"])
        p = sink_softmax((K[:, j] @ q[j, :dn] + KR @ qr) * mc["scale"], P["mix.sink"][j])
        st["p"].append(p)
        out[j] = p @ V[:, j]
    return P["mix.o"] @ (out.reshape(-1) * sigmoid(P["mix.g"] @ h))


# ------------------------------------------------------------------ feed-forward
def relu2_ff(h, P):
    """Wdown relu(Wup h)^2"""
    return P["mlp.down"] @ np.maximum(P["mlp.up"] @ h, 0.0) ** 2


# ------------------------------------------------------------------ the model
class OracleGifudra:
    def __init__(self, config, tensors):
        self.cfg = config
        self.T = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])
        self.per_layer = []
        for i in range(len(config["layers"])):
            pre = f"l{i}."
            self.per_layer.append({k[len(pre):]: v for k, v in self.T.items() if k.startswith(pre)})
        self.reset()

    def reset(self):
        self.state = [dict() for _ in self.cfg["layers"]]
        self.pos = 0

    def step(self, token, want_residual=False):
        """One token -> logits (and the sum of the streams after every layer)."""
        cfg, T, eps = self.cfg, self.T, self.eps
        x = T["embed"][int(token)] * float(cfg["embedding"]["scale"])
        X = np.tile(x, (int(cfg.get("streams") or 1), 1))
        trace = []
        for lc, P, st in zip(cfg["layers"], self.per_layer, self.state):
            mc = lc["mixer"]
            owner = self.state[mc["kv_from"]] if mc.get("kv_from") is not None else None
            h = rms_unit(streams_in(X, P, 1), eps) * P["norm1"]
            y = latent_attention_step(h, self.pos, P, mc, eps, st, owner) * P["ls1"]
            X = streams_out(X, y, P, 1)
            if lc.get("mlp") is not None:
                h = rms_unit(streams_in(X, P, 2), eps) * P["norm2"]
                X = streams_out(X, relu2_ff(h, P) * P["ls2"], P, 2)
            trace.append(X.sum(axis=0))
        self.pos += 1
        logits = (T["embed"] @ (rms_unit(X.sum(axis=0), eps) * T["final.norm"])) * float(cfg["logit_scale"])
        return (logits, np.stack(trace)) if want_residual else logits

    def run(self, tokens, want_residual=False):
        """Continue the sequence with `tokens`; logits [n, vocab] (and residuals [layers, n, W])."""
        outs = [self.step(t, want_residual) for t in tokens]
        if want_residual:
            return np.stack([o[0] for o in outs]), np.stack([o[1] for o in outs], axis=1)
        return np.stack(outs)


def to_bf16_grid(tensors):
    """Every array rounded to values a bfloat16 checkpoint can hold (as float64)."""
    out = {}
    for k, v in tensors.items():
        a = np.ascontiguousarray(v, dtype=np.float32)
        u = a.view(np.uint32)
        u = ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32)
        out[k] = u.view(np.float32).reshape(a.shape).astype(np.float64)
    return out


def random_model(config, seed, bf16_round=True):
    """Random tensors for a configuration (names and shapes as a checkpoint has them)."""
    rng = np.random.default_rng(seed)
    W, V, S = config["width"], config["vocab"], config.get("streams") or 0

    def mat(o, i, gain=1.0):
        return rng.standard_normal((o, i)) * gain / np.sqrt(i)

    def vec(n, mean, spread):
        return mean + spread * rng.standard_normal(n)

    t = {"embed": rng.standard_normal((V, W)) * 0.1, "final.norm": vec(W, 1.0, 0.1)}
    for i, lc in enumerate(config["layers"]):
        p, mc = f"l{i}.", lc["mixer"]
        H, dn, dr, dv = mc["heads"], mc["dim"], mc["rot_dim"], mc["vdim"]
        has_ff = lc.get("mlp") is not None
        t[p + "norm1"] = vec(W, 1.0, 0.1)
        t[p + "mix.dq"] = mat(mc["q_rank"], W)
        t[p + "mix.dq.norm"] = vec(mc["q_rank"], 1.0, 0.1)
        t[p + "mix.uq"] = mat(H * (dn + dr), mc["q_rank"], 1.2)
        if mc.get("kv_from") is None:
            t[p + "mix.dkv"] = mat(mc["kv_rank"] + dr, W, 1.2)
            t[p + "mix.dkv.norm"] = vec(mc["kv_rank"], 1.0, 0.1)
        t[p + "mix.uk"] = mat(H * dn, mc["kv_rank"], 1.2)
        t[p + "mix.uv"] = mat(H * dv, mc["kv_rank"])
        t[p + "mix.sink"] = vec(H, 0.5, 1.0)
        t[p + "mix.g"] = mat(H * dv, W)
        t[p + "mix.o"] = mat(W, H * dv)
        for q in (1, 2) if has_ff else (1,):
            t[p + f"ls{q}"] = vec(W, 0.7, 0.2)
            if not S:
                continue
            t[p + f"hc{q}.in"] = vec(S, 1.0 / S, 0.3 / S)
            t[p + f"hc{q}.out"] = vec(S, 1.0, 0.4)
            t[p + f"hc{q}.mix"] = np.eye(S) * 0.8 + (0.3 / S) * rng.standard_normal((S, S))
        if has_ff:
            ff = lc["mlp"]["ff"]
            t[p + "norm2"] = vec(W, 1.0, 0.1)
            t[p + "mlp.up"] = mat(ff, W)
            t[p + "mlp.down"] = mat(W, ff)
    return to_bf16_grid(t) if bf16_round else t
