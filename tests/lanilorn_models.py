"""Small Lanilorn configurations for the tests, and folders of random weights for them.

The configurations differ from one another in every size and option: each mixer alone, one to ten residual
streams, windows that are no multiple of a page, a window of one and none, query heads per key/value head
from one to four, keys and values of the differential layers of equal and of unequal width, rotations
of a part of the head, of all of it, of nothing, scaled and not, temperatures that change every token and
hardly ever, recurrences of one head and of several with wide and narrow decays, layers with and
without a feed-forward, widths that are no multiple of eight.
"""

from __future__ import annotations

from pathlib import Path

import torch


def yarn(base, dims, factor, original, fast, slow):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}


def attention(heads, kv_heads, dim, window, scale, rot=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                         "mask": None if window is None else {"size": window}, "rot": rot}


def difference(heads, kv_heads, dim, vdim, scale, diff, coef, every):
    return "attention_2", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                           "diff": diff, "q_temp": {"coef": coef, "every": every}}


def gla(heads, dim, vdim, tau, rank):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def layer(mixer, ff=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, eps, streams, layers, embedding=1.5, logits=2.0):
    return {"architecture": "Lanilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "embedding": {"scale": embedding}, "logit_scale": logits, "layers": layers}


CONFIGS = {
    # each mixer alone: a window of 11 over pages of 16, three query heads per key/value head
    "window": model(83, 48, 1e-5, 2, [layer(attention(6, 2, 16, 11, 0.9, yarn(5000.0, 8, 4.0, 64, 8.0, 0.5)))]),
    # no window, no rotation, a single head, one stream; what the embedding and the logits are multiplied by is 1
    "sinks": model(97, 40, 1e-6, 1, [layer(attention(1, 1, 24, None, 0.6), 56)], embedding=1.0, logits=1.0),
    "difference": model(71, 48, 1e-5, 3, [layer(difference(4, 2, 12, 20, 2.5, 0.35, 0.4, 7))]),
    # keys and values of one width; a temperature that changes with every token; one key/value head
    "difference_even": model(64, 40, 1e-4, 2, [layer(difference(3, 1, 8, 16, 3.0, 0.8, 0.15, 1), 24)]),
    "recurrent": model(90, 40, 1e-5, 2, [layer(gla(3, 10, 14, 4.0, 5))]),
    # several layers of it, one head, a state wider than long
    "recurrent_deep": model(90, 48, 1e-5, 4, [layer(gla(1, 16, 40, 1.0, 16), 32), layer(gla(2, 24, 8, 20.0, 3), 40)]),
    # the feed-forward under the simplest mixer (a token sees itself only)
    "feed_forward": model(71, 32, 1e-6, 3, [layer(attention(1, 1, 8, 1, 1.0), 44)]),
    # everything in turn
    "all": model(131, 64, 1e-5, 4, [
        layer(difference(4, 4, 16, 24, 2.0, 0.5, 0.3, 16), 72),
        layer(attention(4, 1, 16, 21, 0.8, yarn(9000.0, 16, 3.0, 48, 16.0, 1.0)), 96),
        layer(gla(2, 16, 24, 8.0, 8)),
        layer(attention(6, 3, 12, 40, 0.9, {"base": 700.0, "dims": 4, "scaling": None}), 48),
        layer(gla(3, 8, 8, 16.0, 4), 40),
        layer(difference(2, 1, 20, 40, 1.6, 0.25, 0.2, 5))]),
    # sizes that are no multiple of eight or four; more streams than the unrolled kernels take
    "odd": model(61, 37, 1e-5, 9, [
        layer(attention(3, 1, 6, 7, 1.3, yarn(100.0, 2, 2.0, 32, 4.0, 1.0)), 21),
        layer(difference(3, 3, 5, 7, 2.2, 0.6, 0.5, 3), 13),
        layer(gla(3, 7, 5, 3.0, 1), 19)]),
    # head sizes of real models in small: long portions take the tcgen05 attention (rows of 64 and of 128
    # columns), the others the mma.sync forms; an eps that keeps the recurrence, whose normed output at the first
    # token is the sign of q . k, from turning on a rounding
    "wide": model(150, 128, 1e-3, 3, [
        layer(difference(4, 2, 32, 64, 1.2, 0.4, 0.2, 32), 192),
        layer(attention(4, 1, 64, 100, 0.35, yarn(20000.0, 32, 4.0, 128, 32.0, 1.0)), 256),
        layer(gla(2, 64, 64, 12.0, 24)),
        layer(difference(2, 1, 64, 128, 0.8, 0.7, 0.25, 80), 128),
        layer(attention(4, 2, 128, 56, 0.25, yarn(20000.0, 128, 2.0, 64, 32.0, 1.0)), 64),
        layer(difference(6, 3, 48, 96, 0.9, 0.5, 0.35, 20))]),
}


def write_model(root, name, seed=0, std=0.08, sharpen=True) -> Path:
    """A folder with config.json and random weights for CONFIGS[name].  The streams' coefficients and the
    scales of the outputs are drawn wide and of both signs, the norms' weights wide, the sinks large enough to take
    a good part of the weights, the narrow vectors of the differential layers so that neither exponential is near
    one, gates and decays so that no two heads or rows are alike.  Without `sharpen` the outputs' scales, gates and
    scores are small, the embedding rows large and no stream is subtracted: a rounding in one layer is not blown up
    by the next, which is what a comparison in bfloat16 needs."""
    from from_scratch_inference_engine_b200.config import config_from_dict
    from from_scratch_inference_engine_b200.weights import load_file, save_file, write_random_model

    folder = write_random_model(Path(root) / f"lanilorn_{name}", config_from_dict(CONFIGS[name]),
                                seed, std, torch.bfloat16)
    tensors = load_file(folder / "model.safetensors")
    generator = torch.Generator().manual_seed(seed + 1000)

    def uniform(shape, low, high):
        return torch.rand(shape, generator=generator) * (high - low) + low

    def normal(shape, scale):
        return torch.randn(shape, generator=generator) * scale

    for key in sorted(tensors):
        shape, last = tensors[key].shape, key.split(".", 1)[-1]
        if last in ("hc1.in", "hc2.in"):
            value = uniform(shape, 0.4, 1.4)
            value[-1] = value[-1] if shape[0] == 1 or not sharpen else -0.5 * value[-1]
        elif last in ("hc1.out", "hc2.out"):
            value = uniform(shape, 0.5, 1.5)
        elif last in ("hc1.mix", "hc2.mix"):
            kept, noise = (0.7, 0.4) if sharpen else (1.0, 0.2)
            value = kept * torch.eye(shape[0]) + normal(shape, noise / shape[0] ** 0.5)
        elif last in ("ls1", "ls2"):
            value = uniform(shape, 0.5, 1.5) * torch.where(uniform(shape, 0, 1) < 0.3, -1.0, 1.0) * (1.0 if sharpen else 0.4)
        elif last == "mix.sink":
            value = uniform(shape, 0.5, 3.0)
        elif last.startswith("mix.l"):
            value = normal(shape, (1.2 if last.endswith("1") else 0.9) * (1.0 if sharpen else 0.3) / shape[0] ** 0.25)
        elif last == "mix.a2.b":
            value = uniform(shape, -1.5, 3.0)
        elif last == "mix.a2":
            value = normal(shape, 1.5 / shape[1] ** 0.5)
        elif last == "mix.g":
            value = tensors[key].float() * (3.0 if sharpen else 1.0)
        elif not sharpen and (key == "embed" or last == "mix.q"):
            value = tensors[key].float() * (6.0 if key == "embed" else 0.5)
        elif last.endswith("norm") or last.startswith("norm"):
            value = uniform(shape, 0.5, 1.6)
        else:
            continue
        tensors[key] = value.to(torch.bfloat16)
    save_file(tensors, folder / "model.safetensors")
    return folder


def random_config(seed: int) -> dict:
    """A configuration drawn at random: one to four layers, every mixer, size, window, constant, feed-forward and
    the number of streams drawn anew."""
    import random
    rng = random.Random(seed)

    def draw_mixer():
        kind = rng.choice(["attention", "difference", "gla"])
        kv_heads = rng.choice([1, 2, 3])
        heads = kv_heads * rng.choice([1, 2, 4])
        if kind == "attention":
            dim = rng.choice([6, 8, 16, 24, 32, 48, 64])
            dims = rng.choice([0, 2, dim // 2 // 2 * 2, dim])
            rot = None
            if dims:
                rot = {"base": rng.choice([50.0, 3000.0, 1e5]), "dims": dims, "scaling": None}
                if rng.random() < 0.7:
                    rot = yarn(rot["base"], dims, rng.choice([1.0, 2.0, 6.5]), rng.choice([32, 100, 2048]),
                               rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0, 2.0]))
            return attention(heads, kv_heads, dim, rng.choice([None, 1, 3, 16, 21, 64, 100, 500]),
                             rng.choice([2.0, 3.5]) * dim ** -0.5, rot)
        if kind == "difference":
            dim = rng.choice([4, 8, 10, 16, 24, 32, 48])
            return difference(heads, kv_heads, dim, rng.choice([2 * dim, 6, 16, 40]), rng.choice([6.0, 9.0]) * dim ** -0.5,
                              rng.choice([0.2, 0.5, 0.8]), rng.choice([0.0, 0.1, 0.4]), rng.choice([1, 5, 64, 300]))
        return gla(rng.choice([1, 2, 5]), rng.choice([4, 7, 16, 40, 64, 130]), rng.choice([4, 10, 16, 32, 50]),
                   rng.choice([1.0, 5.5, 16.0]), rng.choice([1, 4, 16, 20]))

    layers = [layer(draw_mixer(), rng.choice([None, 12, 40, 64])) for _ in range(rng.randint(1, 4))]
    return model(rng.choice([50, 97, 128]), rng.choice([24, 36, 64, 128]), rng.choice([1e-4, 1e-5, 1e-6]),
                 rng.choice([1, 2, 3, 4, 6, 10]), layers, rng.choice([0.5, 1.0, 3.0]), rng.choice([0.25, 1.0, 2.0]))


def write_random(root, seed: int, sharpen=True) -> Path:
    """A folder for `random_config(seed)`, which is entered into CONFIGS as "random<seed>"."""
    CONFIGS[f"random{seed}"] = random_config(seed)
    return write_model(root, f"random{seed}", seed=seed, sharpen=sharpen)
