"""Plain evaluation of the Rufusun decoder in numpy, one function per mechanism.

Everything is token by token and head by head in the order of the equations, in the float type of
the inputs (the tests use float64), with no code shared with the package under test.
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x) + eps)


def rms_norm(x, w, eps):
    """The stored weight counts from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def rotate_half(v, position, dims, base):
    """Rotates (v[i], v[i + dims/2]) by position * base^(-2i/dims) for i < dims/2; v[dims:] stays."""
    out = v.copy()
    half = dims // 2
    for i in range(half):
        a = position * base ** (-2.0 * i / dims)
        c, s = np.cos(a), np.sin(a)
        out[i] = v[i] * c - v[i + half] * s
        out[i + half] = v[i + half] * c + v[i] * s
    return out


def capped(s, cap):
    return cap * np.tanh(s / cap)


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def visible(n):
    """Which of the n keys so far the newest token sees."""
    return np.ones(n, bool)


def attention(h, w, m, state, position):
    """One token; state["k"] and state["v"] (lists) grow by this token's."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q, k, v = w["q"] @ h + w["q.b"], w["k"] @ h + w["k.b"], w["v"] @ h + w["v.b"]
    state["k"].append(np.stack([rotate_half(k[g * D:(g + 1) * D], position, rot["dims"], rot["base"]) for g in range(G)]))
    state["v"].append(v.reshape(G, E))
    keys, values = np.stack(state["k"]), np.stack(state["v"])
    see = visible(len(keys))
    out = []
    for n in range(H):
        g = n // (H // G)
        qn = rotate_half(q[n * D:(n + 1) * D], position, rot["dims"], rot["base"])
        s = capped((keys[:, g] @ qn) * m["scale"], m["softcap"])
        p = softmax(np.where(see, s, -np.inf))
        out.append(p @ values[:, g])
    return w["o"] @ np.concatenate(out) + w["o.b"]


def causal_conv(x, tail, w):
    """One token of a per-channel causal convolution. tail: [taps - 1, channels], oldest first, updated."""
    taps = np.concatenate([tail, x[None]], 0)
    if len(tail):
        tail[:] = taps[1:]
    return (taps * w.T).sum(0)


def unit(x):
    return x / np.sqrt(np.sum(x * x) + 1e-6)


def decay(a, A_log, dt_bias):
    return np.exp(-np.exp(A_log) * softplus(a + dt_bias))


def delta_state(S, k, v, g, beta):
    S = g * S
    u = beta * (v - S.T @ k)
    return S + np.outer(k, u)


def delta(h, w, m, eps, state):
    """One token of the gated delta rule. state["S"]: [heads, dim, vdim]; state["q" / "k" / "v"]: conv tails."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(w[n] @ h, state[n], w[n + ".conv"])) for n in "qkv")
    beta = sigmoid(w["b"] @ h)
    g = decay(w["a"] @ h, w["A_log"], w["dt_bias"])
    out = []
    for n in range(H):
        j = n // (H // G)
        qn = unit(q[j * D:(j + 1) * D]) * D ** -0.5
        kn = unit(k[j * D:(j + 1) * D])
        state["S"][n] = delta_state(state["S"][n], kn, v[n * E:(n + 1) * E], g[n], beta[n])
        out.append(rms(state["S"][n].T @ qn, eps) * w["norm"])
    return w["o"] @ (np.concatenate(out) * silu(w["g"] @ h))


def gated_ff(x, w):
    return w["down"] @ (silu(w["gate"] @ x) * (w["up"] @ x))


def clamped_ff(x, w, limit):
    g = np.minimum(w["gate"] @ x, limit)
    u = np.clip(w["up"] @ x, -limit, limit)
    return w["down"] @ (g * sigmoid(1.702 * g) * (u + 1.0))


def route(h, w, top):
    """The chosen experts and their weights."""
    s = sigmoid(w @ h)
    chosen = np.argsort(-s, kind="stable")[:top]
    return chosen, s[chosen]


def sub(w, name):
    return {k[len(name) + 1:]: v for k, v in w.items() if k.startswith(name + ".")}


def mixture(h, w, mlp):
    out = np.zeros_like(h)
    for e, s in zip(*route(h, w["router"], mlp["router"]["top"])):
        out = out + clamped_ff(s * h, sub(w, f"e{e}"), mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + clamped_ff(h, sub(w, "shared"), mlp["shared"]["limit"])
    return out


def new_state(layer, dtype=np.float64):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return {"k": [], "v": []}
    qk, v, taps = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["conv"] - 1
    return {"S": np.zeros((m["heads"], m["dim"], m["vdim"]), dtype), "q": np.zeros((taps, qk), dtype),
            "k": np.zeros((taps, qk), dtype), "v": np.zeros((taps, v), dtype)}


def run_order(config):
    """The layers in the order they run."""
    order = list(range(len(config["layers"])))
    loop = config.get("loop")
    if not loop:
        return order
    return order[:loop["start"]] + order[loop["start"]:loop["stop"]] * loop["times"] + order[loop["stop"]:]


class Model:
    """config: the parsed config.json; tensors: name -> array. `forward` continues where it stopped."""

    def __init__(self, config, tensors, dtype=np.float64):
        self.config = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.dtype = dtype
        self.eps = config["norm"]["eps"]
        self.order = run_order(config)
        self.parts = {(i, kind): sub(sub(self.t, f"l{i}"), kind) for i in set(self.order) for kind in ("mix", "mlp")}
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [new_state(self.config["layers"][i], self.dtype) for i in self.order]

    def layer(self, i, st, x):
        layer, l = self.config["layers"][i], f"l{i}."
        h = rms_norm(x, self.t[l + "norm1"], self.eps)
        w = self.parts[i, "mix"]
        if layer["type"] == "attention":
            y = attention(h, w, layer["mixer"], st, self.position)
        else:
            y = delta(h, w, layer["mixer"], self.eps, st)
        mlp = layer.get("mlp")
        if mlp:
            h2 = rms_norm(x, self.t[l + "norm2"], self.eps)
            w = self.parts[i, "mlp"]
            y = y + (gated_ff(h2, w) if mlp["kind"] == "dense" else mixture(h2, w, mlp))
        return x + y

    def forward(self, tokens, trace=None):
        """Logits of every token, [tokens, vocab]; trace (a list) receives [layer runs, width] per token."""
        out = []
        for tok in tokens:
            x = self.t["embed"][tok]
            rows = []
            for run, i in enumerate(self.order):
                x = self.layer(i, self.state[run], x)
                rows.append(x)
            if trace is not None:
                trace.append(np.stack(rows))
            out.append(self.t["head"] @ rms_norm(x, self.t["final.norm"], self.eps) * self.config["logit_scale"])
            self.position += 1
        return np.stack(out)
