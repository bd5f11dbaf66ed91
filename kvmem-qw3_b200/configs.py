"""Model shapes of the benchmark configurations (qwen35 hybrid, one MTP layer)."""
from .binding import ModelConfig

MODEL_SEED = 0x5EED
PROMPT_SEED = 0xC0FFEE


def tiny():
    """4 layers (DeltaNet x3, attention), hidden 256, 4q/2kv x 64, DeltaNet 2k/4v x 64, FFN 512, vocab 4096."""
    return ModelConfig(n_layers=4, n_embd=256, n_ff=512, n_heads=4, n_kv_heads=2, head_dim=64, rope_dim=16,
                       rope_theta=1e7, rms_eps=1e-6, ssm_conv_kernel=4, ssm_num_k_heads=2, ssm_num_v_heads=4,
                       ssm_head_dim=64, full_attention_interval=4, vocab_size=4096, mtp_layers=1, weight_sigma=0.02)


def qwen27b(n_layers=64):
    """27B-class shape: 64 layers (every 4th full attention), hidden 5120, 24q/4kv x 256,
    DeltaNet 16k/48v x 128 conv 4, FFN 17408, vocab 151936."""
    return ModelConfig(n_layers=n_layers, n_embd=5120, n_ff=17408, n_heads=24, n_kv_heads=4, head_dim=256, rope_dim=64,
                       rope_theta=1e7, rms_eps=1e-6, ssm_conv_kernel=4, ssm_num_k_heads=16, ssm_num_v_heads=48,
                       ssm_head_dim=128, full_attention_interval=4, vocab_size=151936, mtp_layers=1, weight_sigma=0.02)


def kezilix_bench(width, ff, n_layers=8, vocab=32768, loop=None):
    """A Kezilix model with layers of a real model's size: heads of 128, every fourth layer latent attention (rank 512,
    64 rotated dimensions), a feed-forward in every layer."""
    H = width // 128
    ret = {"type": "retention", "mlp": {"kind": "dense", "ff": ff},
           "mixer": {"heads": H, "dim": 128, "vdim": 128, "rot": {"dims": 128, "base": 1e4},
                     "decay": [1.0 - 2.0 ** -(5.0 + 6.0 * i / H) for i in range(H)]}}
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff},
           "mixer": {"heads": H, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
                     "rot": {"dims": 64, "base": 1e4, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    return {"architecture": "Kezilix", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "loop": loop,
            "layers": [lat if (i + 1) % 4 == 0 else ret for i in range(n_layers)]}


def figonex_bench(width, ff, n_layers=8, vocab=32768, tied=False):
    """A Figonex model with layers of a real model's size: every fourth layer attention (heads of 128, 32 rotated dimensions,
    four query heads per key/value head), the others lightning (heads of 128) and mLSTM (128 x 256) by turns, a feed-forward in
    every layer.  tied: the second half of the layers uses the weights of the first."""
    H, dense = width // 128, {"kind": "dense", "ff": ff}
    att = {"type": "attention", "mlp": dense,
           "mixer": {"heads": H, "kv_heads": H // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "rot": {"dims": 32, "base": 1e4, "scaling": {"factor": 4.0}}}}
    lig = {"type": "lightning", "mlp": dense,
           "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** -(3.0 + 6.0 * i / H) for i in range(H)]}}
    mls = {"type": "mlstm", "mlp": dense, "mixer": {"heads": width // 256, "dim": 128, "vdim": 256, "gate_cap": 15.0}}
    layers = [att if i % 4 == 3 else mls if i % 4 == 1 else lig for i in range(n_layers)]
    if tied:
        layers = layers[:n_layers // 2] + [dict(l, weights_of=i) for i, l in enumerate(layers[:n_layers // 2])]
    return {"architecture": "Figonex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5}, "layers": layers}


def qwen35_bench(width, ff, n_layers=8, vocab=32768):
    """The qwen35 hybrid at the width, feed-forward size, depth and attention interval of kezilix_bench."""
    return ModelConfig(n_layers=n_layers, n_embd=width, n_ff=ff, n_heads=width // 256, n_kv_heads=4 if width % 1024 == 0 else 2, head_dim=256,
                       rope_dim=64, rope_theta=1e7, rms_eps=1e-6, ssm_conv_kernel=4, ssm_num_k_heads=width // 128,
                       ssm_num_v_heads=width // 128, ssm_head_dim=128, full_attention_interval=4, vocab_size=vocab, mtp_layers=0,
                       weight_sigma=0.02)
