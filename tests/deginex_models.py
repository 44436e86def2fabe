"""Small Deginex configurations for the tests, and folders of random weights for them.

The configurations differ from one another in every size and option: one to nine residual streams, key
and value widths that differ, query heads per key/value head from one to four, chunks that are no
multiple of a page, a chunk of one, caps that bend the scores hard and hardly at all, layers without a
feed-forward, dense ones and experts (top 1, all of them, one expert), loops over the first layers, the
last ones, of one pass and none, widths that are no multiple of eight.
"""

from __future__ import annotations

from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, chunk, scale, softcap):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
            "scale": scale, "softcap": softcap}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, eps, streams, layers, loop=None):
    return {"architecture": "Deginex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": layers}


CONFIGS = {
    # the mixer alone: chunks of 11 over pages of 16, three query heads per key/value head, two streams
    "chunk": model(83, 48, 1e-5, 2, [layer(attention(6, 2, 16, 12, 11, 0.9, 7.0))]),
    # a cap far below the scores it meets, a single head, one stream
    "capped": model(97, 40, 1e-6, 1, [layer(attention(1, 1, 24, 8, 64, 1.5, 3.0), dense(56))]),
    # the experts alone under the simplest mixer (a token sees itself only): top 3 of 12
    "experts": model(71, 32, 1e-6, 3, [layer(attention(1, 1, 8, 8, 1, 1.0, 50.0), moe(20, 12, 3))]),
    # the loop: two passes over the two middle layers, each pass with its own cache; four streams
    "loop": model(131, 64, 1e-5, 4, [
        layer(attention(4, 2, 16, 8, 21, 0.8, 12.0), dense(72)),
        layer(attention(2, 2, 12, 20, 40, 0.7, 9.0), moe(24, 6, 2)),
        layer(attention(4, 1, 16, 16, 13, 1.0, 15.0)),
        layer(attention(4, 2, 16, 8, 21, 0.8, 12.0), moe(16, 5, 5))], loop=(1, 3, 2)),
    # a loop from the first layer on and of a single pass; a loop up to the last layer, three passes
    "loop_first": model(90, 40, 1e-5, 2, [
        layer(attention(2, 1, 8, 8, 9, 1.2, 6.0), moe(24, 4, 1)),
        layer(attention(2, 2, 8, 16, 30, 1.0, 20.0), dense(40))], loop=(0, 1, 1)),
    "loop_last": model(90, 40, 1e-4, 5, [
        layer(attention(2, 2, 8, 16, 17, 1.0, 5.0), dense(24)),
        layer(attention(4, 4, 8, 4, 5, 1.1, 30.0), moe(12, 1, 1))], loop=(1, 2, 3)),
    # sizes that are no multiple of eight or four; more streams than the unrolled kernels take
    "odd": model(61, 37, 1e-5, 9, [
        layer(attention(3, 1, 6, 10, 7, 1.3, 8.0), dense(21)),
        layer(attention(3, 3, 10, 6, 25, 0.9, 11.0), moe(13, 7, 4))], loop=(0, 2, 2)),
    # head sizes of real models in small: long portions take the tcgen05 attention (64 columns) and the
    # experts' grouped product, the second layer's unequal widths the mma.sync attention
    "wide": model(150, 128, 1e-6, 3, [
        layer(attention(4, 2, 64, 64, 100, 0.3, 18.0), dense(192)),
        layer(attention(4, 1, 48, 64, 56, 0.35, 14.0), moe(64, 8, 2)),
        layer(attention(2, 1, 64, 64, 72, 0.3, 25.0), moe(32, 4, 2))], loop=(0, 2, 2)),
}


def write_model(root, name, seed=0, std=0.08, sharpen=True) -> Path:
    """A folder with config.json and random weights for CONFIGS[name].  The streams' coefficients are
    drawn wide and of both signs, so that no two streams are alike and a swapped index shows.  With
    `sharpen` the routers are ten times as wide and their biases N(0, 1), so that every token chooses
    its own experts.  Without it the routers are drawn narrow and the biases half a unit apart: the
    choice rests on the biases alone and no rounding can turn it - which is what a comparison in
    bfloat16 needs; the weights still come from each token's own logits."""
    from from_scratch_inference_engine_b200.config import config_from_dict
    from from_scratch_inference_engine_b200.weights import load_file, save_file, write_random_model

    folder = write_random_model(Path(root) / f"deginex_{name}", config_from_dict(CONFIGS[name]),
                                seed, std, torch.bfloat16)
    tensors = load_file(folder / "model.safetensors")
    generator = torch.Generator().manual_seed(seed + 1000)

    def uniform(shape, low, high):
        return torch.rand(shape, generator=generator) * (high - low) + low

    for key in sorted(tensors):
        shape = tensors[key].shape
        if key.endswith((".hc1.in", ".hc2.in")):
            value = uniform(shape, 0.4, 1.4)
            value[-1] = value[-1] if shape[0] == 1 else -0.5 * value[-1]
        elif key.endswith((".hc1.out", ".hc2.out")):
            value = uniform(shape, 0.5, 1.5)
        elif key.endswith((".hc1.mix", ".hc2.mix")):
            count = shape[0]
            value = 0.7 * torch.eye(count) + torch.randn(shape, generator=generator) * 0.4 / count ** 0.5
        elif key.endswith(".router.b"):
            count = tensors[key].numel()
            value = torch.randn(shape, generator=generator) if sharpen else \
                0.5 * torch.randperm(count, generator=generator).float()
        elif key.endswith(".router"):
            value = tensors[key].float() * (10.0 if sharpen else 0.05)
        elif key.endswith(".b"):
            value = tensors[key].float() * 3.0                 # the norms' biases
        else:
            continue
        tensors[key] = value.to(torch.bfloat16)
    save_file(tensors, folder / "model.safetensors")
    return folder


def random_config(seed: int) -> dict:
    """A configuration drawn at random: one to four layers, every size, chunk, scale, cap, feed-forward,
    number of streams and the loop drawn anew."""
    import random
    rng = random.Random(seed)

    def draw_attention():
        kv_heads = rng.choice([1, 2, 3])
        dim = rng.choice([6, 8, 16, 24, 32, 48, 64])
        return attention(kv_heads * rng.choice([1, 2, 4]), kv_heads, dim, rng.choice([4, 8, 10, 16, 32, 48, 64]),
                         rng.choice([1, 3, 7, 16, 21, 40, 64, 100, 500]), rng.choice([2.0, 3.5]) * dim ** -0.5,
                         rng.choice([2.5, 8.0, 20.0, 50.0]))

    def draw_mlp():
        kind = rng.random()
        if kind < 0.2:
            return None
        if kind < 0.5:
            return dense(rng.choice([12, 40, 64]))
        experts = rng.choice([1, 3, 4, 6, 8, 40])
        return moe(rng.choice([8, 12, 16, 40]), experts, rng.randint(1, min(experts, 5)))

    layers = [layer(draw_attention(), draw_mlp()) for _ in range(rng.randint(1, 4))]
    loop = None
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return model(rng.choice([50, 97, 128]), rng.choice([24, 36, 64, 128]), rng.choice([1e-4, 1e-5, 1e-6]),
                 rng.choice([1, 2, 3, 4, 6, 10]), layers, loop)


def write_random(root, seed: int, sharpen=True) -> Path:
    """A folder for `random_config(seed)`, which is entered into CONFIGS as "random<seed>"."""
    CONFIGS[f"random{seed}"] = random_config(seed)
    return write_model(root, f"random{seed}", seed=seed, sharpen=sharpen)
