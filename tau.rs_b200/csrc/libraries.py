"""The list of CUDA libraries of this folder, for a build of everything at once."""
from __future__ import annotations

from typing import List, Sequence, Tuple


def all_libraries() -> List[Tuple[str, Sequence[str]]]:
    return [
        ("elementwise.cu", ()),
        ("gemm_simt.cu", ()),
        ("gemm_skinny.cu", ()),
        ("gemm_tc.cu", ()),
        ("attention_generic.cu", ()),
        ("sampling.cu", ()),
        ("random_init.cu", ()),
        ("stream32.cu", ()),
        ("latent_attention.cu", ()),
        ("moe.cu", ()),
        ("sublayer.cu", ()),
        ("diff_attention.cu", ()),
        ("masked_attention.cu", ()),
        ("short_conv.cu", ()),
        ("walk_prepare.cu", ()),
        *[("delta_rule.cu", (f"TAU_KEY_DIM={key_dim}",)) for key_dim in (16, 32, 64, 128)],
        *[("wkv.cu", (f"TAU_KEY_DIM={key_dim}",)) for key_dim in (16, 32, 64, 128)],
        *[("selective_scan.cu", (f"TAU_SCAN_STATES={states}",)) for states in (8, 16, 32)],
        *[("recurrence.cu", (f"TAU_KEY_DIM={key_dim}",)) for key_dim in (16, 32, 64, 128)],
        # Specialised libraries: the head sizes of the benchmark shape and of the tests' tiny models.
        *[("attention_decode.cu", (f"TAU_HEAD_DIM={head_dim}", f"TAU_DTYPE={dtype}"))
          for head_dim in (128, 64, 16, 32, 48, 80) for dtype in (0, 1)],
        *[("attention_prefill.cu", (f"TAU_HEAD_DIM={head_dim}",)) for head_dim in (128, 16, 32, 48, 80, 192)],
        *[("attention_prefill_tc.cu", (f"TAU_HEAD_DIM={head_dim}",)) for head_dim in (128, 64)],
    ]
