"""Which compile-time variants of each CUDA source exist.

Most sources compile once.  Sources that are specialised by a macro (for instance the
head size of an attention kernel) are compiled for the sizes a model needs when the model
is built; ``default_variants`` lists what a full build compiles ahead of time.
"""
from __future__ import annotations

COMMON_HEAD_DIMS = (16, 32, 64, 128)

_SPECIALISED: dict[str, list[dict]] = {
    "attention_bf16": [{"TW_HEAD_DIM": d} for d in COMMON_HEAD_DIMS] + [{"TW_HEAD_DIM": 2 * v, "TW_V_DIM": v} for v in (32, 64)],
    "attention_tcgen05": [{"TW_HEAD_DIM": d} for d in (64, 128)] + [{"TW_HEAD_DIM": 2 * v, "TW_V_DIM": v} for v in (32, 64)],
    "attention_latent_tcgen05": [{"TW_HEAD_DIM": d, "TW_V_COLS": v, "TW_KEY_TILE": 96} for d, v in ((256, 192), (128, 96))],
    "attention_decode_tma": [{"TW_HEAD_DIM": d} for d in (64, 128)] + [{"TW_HEAD_DIM": 128, "TW_V_DIM": 64}],
    "sigmoid_attention_bf16": [{"TW_HEAD_DIM": d} for d in (64, 128)],
    "sigmoid_attention_tcgen05": [{"TW_HEAD_DIM": d, "TW_SIG_KEY_TILE": 128} for d in (64, 128)],
    "state_space": [{"TW_DK": d} for d in (32, 64, 128)],
    "linear_recurrence": [{"TW_DK": d} for d in (32, 64, 128)],       # the key size of a head: a column of the state in registers
}


def specialise(name: str, variants: list[dict]) -> None:
    _SPECIALISED[name] = variants


def default_variants(name: str) -> list[dict]:
    return _SPECIALISED.get(name, [{}])
