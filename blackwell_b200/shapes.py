"""Model shapes of the benchmark configurations and the algorithmic byte counts
the roofline figures are computed from."""
from __future__ import annotations

from dataclasses import dataclass


@dataclass(frozen=True)
class ModelShape:
    name: str
    layers: int
    hidden: int
    inter: int
    n_q_heads: int
    n_kv_heads: int
    head_dim: int
    vocab: int
    eps: float = 1e-6

    @property
    def q_dim(self) -> int:
        return self.n_q_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    def layer_gemvs(self):
        """(name, N, K) of the per-layer projections in the fused form the
        decode step launches: QKV, O, gate+up, down."""
        return [
            ("qkv", self.q_dim + 2 * self.kv_dim, self.hidden),
            ("o", self.hidden, self.q_dim),
            ("gate_up", 2 * self.inter, self.hidden),
            ("down", self.hidden, self.inter),
        ]

    def gemv_set(self):
        """The five matrices of the per-layer GEMV benchmark set."""
        return self.layer_gemvs() + [("lm_head", self.vocab, self.hidden)]


QWEN3_8B = ModelShape("qwen3-8b-shape", 36, 4096, 10944, 32, 8, 128, 151643)
QWEN3_32B = ModelShape("qwen3-32b-shape", 64, 5120, 25600, 64, 8, 128, 151643)


def gemv_bytes(N: int, K: int, M: int, w_scale_bytes: int = 2, x_kind: str = "f16") -> int:
    """Algorithmic bytes of one GEMV call: nibbles + weight scales once,
    activations once, fp32 outputs once.  x_kind: 'f16' (fused quantize),
    'i8' (int8 + f32 block scales), 'i4' (nibbles + f32 block scales), 'f32'."""
    w = N * K // 2 + N * (K // 16) * w_scale_bytes
    if x_kind == "f16":
        x = M * K * 2
    elif x_kind == "f32":
        x = M * K * 4
    elif x_kind == "i8":
        x = M * K + M * (K // 16) * 4
    elif x_kind == "i4":
        x = M * K // 2 + M * (K // 16) * 4
    else:
        raise ValueError(x_kind)
    return w + x + M * N * 4


def vifivik_config(width: int, ff: int, vocab: int, layers: int, head_scale: int) -> dict:
    """A Vifivik configuration with the layer sizes of a real model (random weights, benchmark only): the pattern mamba2,
    latent attention, latent attention on that cache, retention.  head_scale = width / 2048."""
    mamba = {"heads": 64 * head_scale, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8}
    latent = {"heads": 16 * head_scale, "dim": 128, "rot_dim": 64, "kv_rank": 512, "vdim": 128, "scale": 192 ** -0.5,
              "rot": {"base": 10000.0, "dims": 64}}
    ret = {"heads": 8 * head_scale, "dim": 256, "vdim": 512, "decay": [1 - 2.0 ** -(5 + i % 8) for i in range(8 * head_scale)]}
    out = []
    for i in range(layers):
        kind, mixer = [("mamba2", mamba), ("latent_attention", latent), ("latent_attention", {**latent, "kv_from": i - 1}),
                       ("retention", ret)][i % 4]
        out.append({"type": kind, "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Vifivik", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "logit_softcap": 25.0, "layers": out}


def lanedra_config(width: int, ff: int, vocab: int, layers: int, head_scale: int, window: int = 1024) -> dict:
    """A Lanedra configuration of the same width, depth, feed-forward and vocabulary: the pattern delta, attention, attention on
    that cache, delta."""
    delta = {"heads": 32 * head_scale, "kv_heads": 16 * head_scale, "dim": 128, "vdim": 128, "conv": 4}
    attn = {"heads": 16 * head_scale, "kv_heads": 4 * head_scale, "dim": 64, "vdim": 128, "diff": 0.5, "scale": 64 ** -0.5, "mask": {"size": window},
            "rot": {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    out = []
    for i in range(layers):
        kind, mixer = [("delta", delta), ("attention", attn), ("attention", {**attn, "kv_from": i - 1}), ("delta", delta)][i % 4]
        out.append({"type": kind, "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Lanedra", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "layers": out}


# name -> (config.json model, the INT4 decode model of the same width, feed-forward size, layer count and vocabulary)
VIFIVIK_BENCH = {
    "2k": (vifivik_config(2048, 5632, 32768, 8, 1), ModelShape("int4-2k", 8, 2048, 5632, 16, 4, 128, 32768)),
    "4k": (vifivik_config(4096, 12288, 65536, 8, 2), ModelShape("int4-4k", 8, 4096, 12288, 32, 8, 128, 65536)),
}
# the same sizes as Lanedra models
LANEDRA_BENCH = {"2k": lanedra_config(2048, 5632, 32768, 8, 1), "4k": lanedra_config(4096, 12288, 65536, 8, 2)}
