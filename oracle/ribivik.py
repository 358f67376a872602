"""Plain restatement of the Ribivik design in numpy, one function per mechanism; test infrastructure only.

Written token by token from the equations, in the float type of its inputs, and without any code of the product path.  A
model is a dict of arrays under the checkpoint's tensor names plus the parsed config.

Notation: N(x) = x / sqrt(mean(x^2) + eps); Z(x; w) = N(x) (1 + w).  A layer is
    x <- x + Z(mixer(Z(x; norm1)); norm1b),   x <- x + Z(ff(Z(x; norm2)); norm2b)
with the second line left out where the layer has no feed-forward.
"""
from __future__ import annotations

import numpy as np

from .fegidra import causal_convolution, linear, rms_norm, rotate_half, sigmoid


def shifted_norm(x, weight, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms_norm(x, None, eps) * (1.0 + weight)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def squared_relu(z):
    return np.square(np.maximum(z, 0.0))


def softcap(logits, cap):
    return logits if not cap else cap * np.tanh(logits / cap)


# ------------------------------------------------------------------------------------------------ latent attention

def latent_query(h, tensors, heads, dim, rot_dim, eps):
    """[T, heads, dim + rot_dim] before rotation."""
    compressed = rms_norm(linear(h, tensors["dq"]), tensors["dq.norm"], eps)
    return linear(compressed, tensors["uq"]).reshape(len(h), heads, dim + rot_dim)


def rotate(x, positions, base, dims):
    """Rotation of the first `dims` entries of each of x's vectors [T, vectors, entries]."""
    return rotate_half(x, positions, base, dims) if dims else x


def latent_entries(h, tensors, kv_rank, positions, base, rot_dims, eps):
    """What the cache holds of each token: (normed latent [T, kv_rank], rotated key part [T, rot_dim])."""
    both = linear(h, tensors["dkv"])
    latent = rms_norm(both[:, :kv_rank], tensors["dkv.norm"], eps)
    return latent, rotate(both[:, None, kv_rank:], positions, base, rot_dims)[:, 0]


def expand(latents, up_key, up_value, heads):
    """Unrotated keys [heads, N, dim] and values [heads, N, vdim] of latents [N, rank]."""
    keys = [latents @ part.T for part in np.split(up_key, heads)]
    values = [latents @ part.T for part in np.split(up_value, heads)]
    return np.stack(keys), np.stack(values)


def softmax_over(query, rotated_query, keys, values, rotated_keys, scale):
    """One query position: query [heads, dim], rotated_query [heads, rot_dim], keys [heads, N, dim], values [heads, N, vdim],
    rotated_keys [N, rot_dim] shared by the heads.  Returns [heads, vdim]."""
    out = []
    for head in range(len(query)):
        scores = (keys[head] @ query[head] + rotated_keys @ rotated_query[head]) * scale
        weights = np.exp(scores - scores.max())
        out.append((weights / weights.sum()) @ values[head])
    return np.stack(out)


def latent_attention(h, tensors, sizes, eps, positions, cache):
    """The whole mixer over a run of tokens.  `cache` = [latents [n, rank], rotated keys [n, rot_dim]] of the tokens before
    them (with `kv_from`: of these as well, left by the owning layer), extended in place."""
    heads, dim, rot_dim = sizes["heads"], sizes["dim"], sizes["rot_dim"]
    rot = sizes.get("rot") or {"dims": 0, "base": 1.0}
    query = latent_query(h, tensors, heads, dim, rot_dim, eps)
    rotated_query = rotate(query[..., dim:], positions, rot["base"], rot["dims"])
    if sizes.get("kv_from") is None:
        latent, key = latent_entries(h, tensors, sizes["kv_rank"], positions, rot["base"], rot["dims"], eps)
        cache[0], cache[1] = np.concatenate([cache[0], latent]), np.concatenate([cache[1], key])
    keys, values = expand(cache[0], tensors["uk"], tensors["uv"], heads)
    out = np.stack([softmax_over(query[t, :, :dim], rotated_query[t], keys[:, :position + 1], values[:, :position + 1],
                                 cache[1][:position + 1], sizes["scale"])
                    for t, position in enumerate(positions)])
    gated = out.reshape(len(h), -1) * sigmoid(linear(h, tensors["g"]))
    return linear(gated, tensors["o"])


# ------------------------------------------------------------------------------------------------ state-space mixer

def ssd_step(state, x, b, c, step, rate, skip):
    """One token of one head: state [N, V] <- exp(-rate step) state + step b x^T; returns (state, state^T c + skip x)."""
    state = np.exp(-rate * step) * state + step * np.outer(b, x)
    return state, state.T @ c + skip * x


def gated_group_norm(y, z, weight, groups, eps):
    """RMS norm of y silu(z) in `groups` equal parts of each row."""
    gated = y * silu(z)
    parts = gated.reshape(len(y), groups, -1)
    return rms_norm(parts, None, eps).reshape(gated.shape) * weight


def mamba2(h, tensors, sizes, eps, state):
    """The whole mixer; `state` = [convolution inputs [taps - 1, channels], S [heads, N, V]], replaced in place."""
    heads, groups, size, vdim = sizes["heads"], sizes["groups"], sizes["state"], sizes["vdim"]
    inner = heads * vdim
    projected = linear(h, tensors["in"])
    z, channels, raw_step = np.split(projected, [inner, 2 * inner + 2 * groups * size], axis=1)
    convolved, state[0] = causal_convolution(channels, tensors["conv"], state[0])
    convolved = silu(convolved + tensors["conv.b"])
    x, b, c = np.split(convolved, [inner, inner + groups * size], axis=1)
    x, b, c = x.reshape(-1, heads, vdim), b.reshape(-1, groups, size), c.reshape(-1, groups, size)
    step = softplus(raw_step + tensors["dt_bias"])
    rate = np.exp(tensors["A_log"])
    y = np.zeros((len(h), heads, vdim), dtype=h.dtype)
    matrices = state[1].copy()
    for t in range(len(h)):
        for head in range(heads):
            group = head // (heads // groups)
            matrices[head], y[t, head] = ssd_step(matrices[head], x[t, head], b[t, group], c[t, group], step[t, head],
                                                  rate[head], tensors["D"][head])
    state[1] = matrices
    normed = gated_group_norm(y.reshape(len(h), inner), z, tensors["norm"], sizes["norm_groups"], eps)
    return linear(normed, tensors["o"])


# ------------------------------------------------------------------------------------------------ whole model

class Model:
    """Forward passes of a configuration with `tensors` (name -> array); state is explicit, see new_state()."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.config = config
        self.tensors = {name: np.asarray(value, dtype=dtype) for name, value in tensors.items()}
        self.dtype = dtype

    def new_state(self) -> dict:
        layers = []
        for entry in self.config["layers"]:
            sizes = entry["mixer"]
            if entry["type"] == "mamba2":
                channels = sizes["heads"] * sizes["vdim"] + 2 * sizes["groups"] * sizes["state"]
                layers.append([np.zeros((sizes["conv"] - 1, channels), self.dtype),
                               np.zeros((sizes["heads"], sizes["state"], sizes["vdim"]), self.dtype)])
            else:
                layers.append([np.zeros((0, sizes["kv_rank"]), self.dtype), np.zeros((0, sizes["rot_dim"]), self.dtype)])
        return {"position": 0, "layers": layers}

    def _mixer_tensors(self, index: int) -> dict:
        prefix = f"l{index}.mix."
        return {name[len(prefix):]: value for name, value in self.tensors.items() if name.startswith(prefix)}

    def forward(self, tokens, state: dict, residuals: list | None = None) -> np.ndarray:
        """Logits of every token; `residuals` collects the stream behind each layer."""
        eps = self.config["norm"]["eps"]
        positions = state["position"] + np.arange(len(tokens))
        x = self.tensors["embed"][np.asarray(tokens, dtype=np.int64)]
        for index, entry in enumerate(self.config["layers"]):
            named = {key: self.tensors.get(f"l{index}.{key}") for key in ("norm1", "norm1b", "norm2", "norm2b")}
            h = shifted_norm(x, named["norm1"], eps)
            mixer = self._mixer_tensors(index)
            if entry["type"] == "mamba2":
                update = mamba2(h, mixer, entry["mixer"], eps, state["layers"][index])
            else:
                owner = entry["mixer"].get("kv_from")
                update = latent_attention(h, mixer, entry["mixer"], eps, positions,
                                          state["layers"][index if owner is None else owner])
            x = x + shifted_norm(update, named["norm1b"], eps)
            if entry["mlp"] is not None:
                n = shifted_norm(x, named["norm2"], eps)
                hidden = squared_relu(linear(n, self.tensors[f"l{index}.mlp.up"]))
                x = x + shifted_norm(linear(hidden, self.tensors[f"l{index}.mlp.down"]), named["norm2b"], eps)
            if residuals is not None:
                residuals.append(x.copy())
        state["position"] += len(tokens)
        final = shifted_norm(x, self.tensors["final.norm"], eps)
        return softcap(linear(final, self.tensors["head"]), self.config.get("logit_softcap"))
