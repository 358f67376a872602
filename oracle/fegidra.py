"""Plain restatement of the Fegidra design in numpy, one function per mechanism; test infrastructure only.

Everything is written token by token (or key by key) from the equations, in the float type of its inputs (float64 unless
the caller asks for another), and shares no code with the product path.  A model is a dict of arrays under the
checkpoint's tensor names plus the parsed config.

Notation: x residual row, h = norm of x that the mixer reads, n = norm of x that the feed-forward reads,
    x <- x + (mixer(h + conv(h)) + ff(n)).
"""
from __future__ import annotations

import math

import numpy as np


# ------------------------------------------------------------------------------------------------ element-wise

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis; weight None = no weight."""
    normalised = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps))
    return normalised if weight is None else normalised * weight


def linear(x, weight, bias=None):
    out = x @ weight.T
    return out if bias is None else out + bias


def poly_norm(z, coefficients, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e with N the unweighted RMS norm of the whole row."""
    a, b, c, e = (z.dtype.type(value) for value in coefficients)
    return a * rms_norm(z, None, eps) + b * rms_norm(z * z, None, eps) + c * rms_norm(z * z * z, None, eps) + e


# ------------------------------------------------------------------------------------------------ input convolution

def causal_convolution(h, taps, history):
    """y_t[c] = sum_j taps[c, j] * h_(t - J + 1 + j)[c]; `history` holds the J - 1 inputs before h[0], oldest first.
    Returns (y, the last J - 1 inputs)."""
    width = taps.shape[1]
    padded = np.concatenate([history, h], axis=0)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(width):
            out[t] += taps[:, j] * padded[t + j]
    return out, padded[padded.shape[0] - (width - 1):].copy()


# ------------------------------------------------------------------------------------------------ generalised delta rule

def delta_decay(h, w1, w2, w0):
    """Decay per channel: exp(-exp(-1/2) * sigmoid(w2 tanh(w1 h) + w0))."""
    logits = linear(np.tanh(linear(h, w1)), w2) + w0
    return np.exp(-h.dtype.type(math.exp(-0.5)) * sigmoid(logits))


def delta_step(state, r, k, v, decay, removal):
    """One token of one head.  state [key, value]; returns (new state, state^T r)."""
    unit = k / np.sqrt(np.sum(k * k) + k.dtype.type(1e-6))
    recalled = unit @ state
    new = decay[:, None] * state - np.outer(removal * unit, recalled) + np.outer(k, v)
    return new, new.T @ r


def general_delta(h, tensors, heads, dim, eps, state):
    """The whole mixer over a run of tokens; `state` [heads, dim, dim] is the state before the first of them."""
    r, k, v = (linear(h, tensors[name]).reshape(-1, heads, dim) for name in ("r", "k", "v"))
    gate = sigmoid(linear(h, tensors["g"]))
    removal = sigmoid(linear(h, tensors["a"]) + tensors["a.b"]).reshape(-1, heads, dim)
    decay = delta_decay(h, tensors["w1"], tensors["w2"], tensors["w0"]).reshape(-1, heads, dim)
    state = state.copy()
    out = np.zeros((h.shape[0], heads, dim), dtype=h.dtype)
    for t in range(h.shape[0]):
        for head in range(heads):
            state[head], out[t, head] = delta_step(state[head], r[t, head], k[t, head], v[t, head], decay[t, head],
                                                   removal[t, head])
    normalised = rms_norm(out, None, eps).reshape(h.shape[0], heads * dim)
    return linear(normalised * tensors["norm"] * gate, tensors["o"]), state


# ------------------------------------------------------------------------------------------------ attention

def rotate_half(x, positions, base, dims):
    """Rotary positions on the first `dims` entries of each head; entry i is paired with entry i + dims / 2."""
    out = x.copy()
    half = dims // 2
    for i in range(half):
        angle = positions.astype(x.dtype) * x.dtype.type(float(base) ** (-2.0 * i / dims))
        cosine, sine = np.cos(angle)[:, None], np.sin(angle)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * cosine - v * sine
        out[..., i + half] = v * cosine + u * sine
    return out


def visible(query_position, key_position, chunk):
    """Causal, and inside the query's own chunk when there are chunks (counted from position 0)."""
    return key_position <= query_position and (not chunk or query_position // chunk == key_position // chunk)


def softmax_attention(q, k, v, query_positions, scale, chunk):
    """q [T, H, D]; k [N, G, D], v [N, G, E] for key positions 0..N-1; returns [T, H, E]."""
    group = q.shape[1] // k.shape[1]
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]), dtype=q.dtype)
    for t, position in enumerate(query_positions):
        keys = [j for j in range(k.shape[0]) if visible(int(position), j, chunk)]
        for head in range(q.shape[1]):
            scores = k[keys, head // group] @ q[t, head] * q.dtype.type(scale)
            weights = np.exp(scores - scores.max())
            out[t, head] = (weights / weights.sum()) @ v[keys, head // group]
    return out


def attention_inputs(h, tensors, mixer, positions, eps):
    """Projections with biases, the norms over all rows of q and of k, rotation: q [T,H,D], k [T,G,D], v [T,G,E]."""
    heads, kv_heads, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = rms_norm(linear(h, tensors["q"], tensors["q.b"]), tensors["q.norm"], eps).reshape(-1, heads, dim)
    k = rms_norm(linear(h, tensors["k"], tensors["k.b"]), tensors["k.norm"], eps).reshape(-1, kv_heads, dim)
    v = linear(h, tensors["v"], tensors["v.b"]).reshape(-1, kv_heads, vdim)
    rot = mixer["rot"]
    return (rotate_half(q, positions, rot["base"], rot["dims"]), rotate_half(k, positions, rot["base"], rot["dims"]), v)


def attention(h, tensors, mixer, positions, eps, cached_k, cached_v):
    q, k, v = attention_inputs(h, tensors, mixer, positions, eps)
    keys = np.concatenate([cached_k, k])
    values = np.concatenate([cached_v, v])
    out = softmax_attention(q, keys, values, positions, mixer["scale"], mixer["mask"]["size"])
    return linear(out.reshape(h.shape[0], -1), tensors["o"]), keys, values


# ------------------------------------------------------------------------------------------------ the whole model

class Model:
    """`tensors`: name -> array; every array is converted to `dtype`."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.config, self.dtype = config, dtype
        self.tensors = {name: np.asarray(value).astype(dtype) for name, value in tensors.items()}

    def part(self, prefix: str) -> dict:
        return {name[len(prefix):]: value for name, value in self.tensors.items() if name.startswith(prefix)}

    def new_state(self) -> dict:
        """Everything one sequence carries: tokens seen, and per layer the convolution history and the mixer's state."""
        layers = []
        for entry in self.config["layers"]:
            mixer, width = entry["mixer"], self.config["width"]
            layer = {"history": np.zeros((self.config["canon"]["taps"] - 1, width), self.dtype)}
            if entry["type"] == "general_delta":
                layer["state"] = np.zeros((mixer["heads"], mixer["dim"], mixer["dim"]), self.dtype)
            else:
                layer["k"] = np.zeros((0, mixer["kv_heads"], mixer["dim"]), self.dtype)
                layer["v"] = np.zeros((0, mixer["kv_heads"], mixer["vdim"]), self.dtype)
            layers.append(layer)
        return {"seen": 0, "layers": layers}

    def forward(self, tokens, state: dict, residuals: list | None = None):
        """Logits of every token of the run; advances `state`.  `residuals` collects x after every layer."""
        eps = self.config["norm"]["eps"]
        x = self.tensors["embed"][np.asarray(tokens, dtype=np.int64)]
        positions = state["seen"] + np.arange(len(tokens))
        for index, entry in enumerate(self.config["layers"]):
            prefix, held = f"l{index}.", state["layers"][index]
            h = rms_norm(x, self.tensors[prefix + "norm1"], eps)
            convolved, held["history"] = causal_convolution(h, self.tensors[prefix + "canon1"], held["history"])
            h = h + convolved
            tensors, mixer = self.part(prefix + "mix."), entry["mixer"]
            if entry["type"] == "general_delta":
                update, held["state"] = general_delta(h, tensors, mixer["heads"], mixer["dim"], eps, held["state"])
            else:
                update, held["k"], held["v"] = attention(h, tensors, mixer, positions, eps, held["k"], held["v"])
            if entry.get("mlp") is not None:
                n = rms_norm(x, self.tensors[prefix + "norm2"], eps)
                up = linear(n, self.tensors[prefix + "mlp.up"])
                update = update + linear(poly_norm(up, self.tensors[prefix + "mlp.act"], eps),
                                         self.tensors[prefix + "mlp.down"])
            x = x + update
            if residuals is not None:
                residuals.append(x.copy())
        state["seen"] += len(tokens)
        return linear(rms_norm(x, self.tensors["final.norm"], eps), self.tensors["head"])

    def greedy(self, prompt, count: int) -> list[int]:
        state = self.new_state()
        logits = self.forward(prompt, state)[-1]
        produced = []
        for _ in range(count):
            produced.append(int(np.argmax(logits)))
            if len(produced) < count:
                logits = self.forward([produced[-1]], state)[-1]
        return produced
