import os
import sys

import pytest

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))


def pytest_configure(config):
    config.addinivalue_line("markers", "gpu: needs a CUDA device (NVIDIA B200)")


def pytest_collection_modifyitems(config, items):
    import torch
    if torch.cuda.is_available():
        return
    skip = pytest.mark.skip(reason="no CUDA device")
    for item in items:
        if "gpu" in item.keywords:
            item.add_marker(skip)


@pytest.fixture
def cpu_kernels(monkeypatch):
    """Replace the CUDA kernel wrappers by their plain torch references so that the engine's
    host logic (step planning, cache addressing, block wiring) can run without a GPU."""
    import kernel_refs
    from dotllm_b200.kernels import ops
    for name in ("gather_rows", "add_rmsnorm", "rope_cache_write", "attention", "swiglu", "linear", "gated_linear",
                 "sample", "repetition_penalty", "add_normed_branch", "add_rows", "embed_positions", "gated_activation",
                 "gla_scan", "head_norm_gate", "route_topk", "expert_gate_up", "expert_down", "linear_per_head",
                 "unary_activation", "activated_linear", "softcap", "head_gate", "head_rmsnorm", "delta_rule", "stream_norm",
                 "stream_copies", "embed_copies", "group_rmsnorm", "pair_norm_sum", "scale_values", "StreamWrite", "post_norm",
                 "causal_conv", "ssd_scan", "gated_group_norm", "latent_rows", "latent_queries", "latent_values", "channel_gate", "PostNormed",
                 "embed_pairs", "add_bias", "qkv_rows"):
        monkeypatch.setattr(ops, name, getattr(kernel_refs, name))
    monkeypatch.setattr(ops, "experts_grouped_takes", lambda *a, **k: False)     # the tensor-core path is the GPU's
    # ops.rope_cache_attention composes the two patched functions above for anything but CUDA bfloat16
    return kernel_refs


def pytest_terminal_summary(terminalreporter):
    """The worst logit errors the parity tests saw, next to the bounds they were held to."""
    try:
        import engine_checks
    except ImportError:
        return
    for dtype, (rel_max, rel_rms, abs_max) in engine_checks.OBSERVED.items():
        terminalreporter.write_line(f"observed {dtype}: max |diff| {abs_max:.3e}, max |diff| / row rms {rel_max:.3e}, "
                                    f"row rms error / row rms {rel_rms:.3e}")
