"""Model designs: each module reads its configuration, names its tensors and registers a builder."""
